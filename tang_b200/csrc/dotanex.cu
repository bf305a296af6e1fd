// Dotanex: a decoder with several residual streams whose mixers are windowed attention (per-head norms, a sink per head, the raw
// keys as values), latent attention or lightning attention, each followed by a dense gated feed-forward or by routed experts with
// a shared one (include/tangq.h, tq_dotanex_*).
//
// A layer is
//   * `in`: all projections of the mixer that read its input as one weight; the epilogue puts raw keys straight into the value
//     cache and the activations on the recurrent ones;
//   * the mixer: norms and rotation, then attention or the recurrence (gates are applied in their last kernels);
//   * `out` -> f32, then one kernel that mixes the streams, forms the next sublayer's input and norms it;
//   * experts: router and the shared expert's gate/up as one product, routing, grouped gate/up, grouped down, shared down, and the
//     same stream kernel, which also sums a row's weighted experts (identity experts: its own input).
// The step takes any mix of sequences: each brings its next rows, from one to a whole prompt, at its own position in its
// own slot (cache rows of the attention layers, state of the recurrent ones).
#include <cuda_bf16.h>

#include <cmath>
#include <new>
#include <vector>

#include "dense.cuh"
#include "expert_ff.cuh"
#include "gla.cuh"
#include "latent_attention.cuh"
#include "ragged.h"
#include "rowops.cuh"
#include "window_attention.cuh"

using namespace tq;

namespace {

constexpr float kGluAlpha = 1.702f;
constexpr int kAllKeys = 0x7fffffff;
constexpr size_t kExpandBytes = 1ull << 30;      // of expanded keys and values at a time, unless the configuration says
constexpr size_t kExpandJobs = 32768;

size_t up16(size_t n) { return (n + 15) / 16 * 16; }
size_t up8(size_t n) { return (n + 7) / 8 * 8; }

struct Layer {
  tq_dotanex_layer c;
  size_t src = 0;                                             // the layer whose weights it uses
  // ---- weights (of layer src)
  tq_dweight *w_in = nullptr, *w_out = nullptr;
  float *norm[2] = {}, *hc_in[2] = {}, *hc_out[2] = {}, *hc_mix[2] = {};
  size_t q_rows = 0, k_rows = 0, v_rows = 0, g_rows = 0;      // rows that exist
  size_t k0 = 0, v0 = 0, g0 = 0;                              // first row of the sections of w_in (latent: k0 is dkv's)
  size_t kc = 0, vc = 0, gc = 0;                              // columns of the sections in the mixer's buffer
  void *q_gain = nullptr, *k_gain = nullptr;                  // attention: of the model's dtype
  float *sinks = nullptr, *freq = nullptr, *decay = nullptr, *o_norm = nullptr;
  float rot_mult = 1.f;
  LatentDims d;
  tq_dweight *w_uq = nullptr, *w_kv = nullptr, *w_ukt = nullptr, *w_uv = nullptr;   // w_kv: [uk | uv]; w_ukt, w_uv: per head
  float *dq_norm = nullptr, *c_norm = nullptr;
  size_t q_ld = 0, key_pad = 0, v_pad = 0, ukt_rows = 0, uv_rows = 0;
  bool absorb = false;
  tq_dweight *front = nullptr, *gate_up = nullptr, *down = nullptr, *shared_down = nullptr;   // front: [router | shared gate/up]
  float* correction = nullptr;
  size_t shared0 = 0, gu_rows = 0, down_rows = 0;             // first row of the shared gate/up; rows of one expert in the stacked weights
  unsigned long long have = 0;                                // bit per tensor put
  std::vector<unsigned char> have_expert;                     // bits gate, up, down
  // ---- of its own
  void *k_cache = nullptr, *v_cache = nullptr;                // latent: k_cache alone
  float* state = nullptr;
  size_t dim_pad = 0;
};

}  // namespace

struct tq_dotanex {
  tq_ctx* ctx = nullptr;
  tq_dotanex_config cfg{};
  std::vector<Layer> layers;
  tq_dweight *embed = nullptr, *head = nullptr;
  float* final_norm = nullptr;
  unsigned long long have = 0;
  size_t mix_ld = 0, att_ld = 0, act_ld = 0, shared_ld = 0, low_ld = 0, cq_ld = 0, lq_ld = 0, max_experts = 0, max_top = 0;
  bool latent = false, moe = false;
  size_t ws_rows = 0;
  float *x = nullptr, *xs = nullptr, *y = nullptr, *logits = nullptr, *yp = nullptr, *ys = nullptr, *low = nullptr;
  void *hn = nullptr, *mix = nullptr, *att = nullptr, *gathered = nullptr, *act = nullptr, *shared = nullptr, *cq = nullptr, *lq = nullptr;
  int *row_pos = nullptr, *cache_row = nullptr;
  Routing route;
  LatentPlan plan;
  // per-slot buffers of the absorbed form
  void *lqs = nullptr, *q_lat = nullptr, *o_lat = nullptr;
  int4* head_jobs = nullptr;
  int* n_head_jobs = nullptr;
  // expanded keys and values
  void *exp_k = nullptr, *exp_v = nullptr;
  size_t exp_k_bytes = 0, exp_v_bytes = 0;
  int planned = -1;                                           // first sequence, rows per job and least rows of the plan in place
  int planned_chunk = 0, planned_min = 0, planned_end = 0;
  float* trace = nullptr;
  std::vector<void*> owned;
};

namespace {

struct Workspace {
  void** p;
  size_t bytes;
};

std::vector<Workspace> workspaces(tq_dotanex* m, size_t n) {
  const size_t es = dtype_size(m->cfg.dtype), width = m->cfg.width, pairs = n * m->max_top, hn = m->embed ? m->embed->kpad : 0;
  const size_t moe = m->moe ? n : 0, lat = m->latent ? n : 0, act = pairs > n ? pairs : n;
  return {{(void**)&m->x, n * width * 4}, {(void**)&m->xs, n * m->cfg.streams * width * 4}, {(void**)&m->y, n * width * 4},
          {(void**)&m->logits, moe * m->max_experts * 4}, {(void**)&m->yp, pairs * width * 4}, {(void**)&m->ys, moe * width * 4},
          {(void**)&m->low, lat * m->low_ld * 4}, {&m->hn, n * hn * es}, {&m->mix, n * m->mix_ld * es}, {&m->att, n * m->att_ld * es},
          {&m->gathered, pairs * hn * es}, {&m->act, act * m->act_ld * es}, {&m->shared, moe * m->shared_ld * es}, {&m->cq, lat * m->cq_ld * es},
          {&m->lq, lat * m->lq_ld * es}, {(void**)&m->row_pos, n * 4}, {(void**)&m->cache_row, n * 4}, {(void**)&m->plan.exp_row, lat * 4},
          {(void**)&m->route.expert, pairs * 4}, {(void**)&m->route.weight, pairs * 4}, {(void**)&m->route.rank, pairs * 4},
          {(void**)&m->route.slot, pairs * 4}, {(void**)&m->route.slot_row, pairs * 4}, {(void**)&m->route.slot_weight, pairs * 4},
          {(void**)&m->route.jobs, m->moe ? (pairs + m->max_experts) * sizeof(int4) : 0}};
}

void release(tq_dotanex* m) {
  for (auto& L : m->layers)
    for (tq_dweight* w : {L.w_in, L.w_out, L.w_uq, L.w_kv, L.w_ukt, L.w_uv, L.front, L.gate_up, L.down, L.shared_down})
      if (w) tq_dweight_free(m->ctx, w);
  for (tq_dweight* w : {m->embed, m->head})
    if (w) tq_dweight_free(m->ctx, w);
  for (auto& w : workspaces(m, 0))
    if (*w.p) cudaFree(*w.p);
  if (m->exp_k) cudaFree(m->exp_k);
  if (m->exp_v) cudaFree(m->exp_v);
  for (void* p : m->owned) cudaFree(p);
  delete m;
  cudaGetLastError();
}

int zalloc(tq_dotanex* m, void** p, size_t bytes) {
  cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
  if (e == cudaErrorMemoryAllocation) {
    cudaGetLastError();
    return fail(m->ctx, TQ_ENOMEM, "dotanex: out of device memory (%zu bytes)", bytes);
  }
  TQ_CUDA(m->ctx, e);
  TQ_CUDA(m->ctx, cudaMemsetAsync(*p, 0, bytes, m->ctx->stream));
  return TQ_OK;
}

int before_resize(tq_dotanex* m) {
  tq_ctx* ctx = m->ctx;
  TQ_REQUIRE(ctx, !ctx->capturing, "tq_dotanex_step: workspaces must be sized before graph capture (run once eagerly)");
  TQ_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  ctx->ws_generation++;   // graphs recorded over the old buffers must not be replayed
  return TQ_OK;
}

int ensure_rows(tq_dotanex* m, size_t rows) {
  if (rows <= m->ws_rows) return TQ_OK;
  if (int st = before_resize(m)) return st;
  const size_t n = rows < 64 ? 64 : rows;
  m->ws_rows = 0;
  for (auto& w : workspaces(m, n)) {
    if (*w.p) cudaFree(*w.p);
    *w.p = nullptr;
    if (int st = zalloc(m, w.p, w.bytes)) return st;
  }
  m->ws_rows = n;
  return TQ_OK;
}

int ensure_expanded(tq_dotanex* m, size_t k_bytes, size_t v_bytes) {
  auto grow = [&](void** p, size_t* have, size_t need) -> int {
    if (need <= *have) return TQ_OK;
    if (int st = before_resize(m)) return st;
    if (*p) cudaFree(*p);
    *p = nullptr;
    *have = 0;
    if (int st = zalloc(m, p, need)) return st;
    *have = need;
    return TQ_OK;
  };
  if (int st = grow(&m->exp_k, &m->exp_k_bytes, k_bytes)) return st;
  return grow(&m->exp_v, &m->exp_v_bytes, v_bytes);
}

constexpr unsigned long long bit(int t) { return 1ull << t; }

unsigned long long needed(const Layer& L) {
  unsigned long long n = bit(TQ_DX_NORM1) | bit(TQ_DX_HC1_IN) | bit(TQ_DX_HC1_OUT) | bit(TQ_DX_HC1_MIX) | bit(TQ_DX_O);
  if (L.c.kind == TQ_DX_ATTENTION) n |= bit(TQ_DX_Q) | bit(TQ_DX_K) | bit(TQ_DX_Q_NORM) | bit(TQ_DX_K_NORM) | bit(TQ_DX_SINK);
  else if (L.c.kind == TQ_DX_LATENT)
    n |= bit(TQ_DX_DQ) | bit(TQ_DX_DQ_NORM) | bit(TQ_DX_UQ) | bit(TQ_DX_DKV) | bit(TQ_DX_DKV_NORM) | bit(TQ_DX_UK) | bit(TQ_DX_UV) | bit(TQ_DX_G);
  else n |= bit(TQ_DX_Q) | bit(TQ_DX_K) | bit(TQ_DX_V) | bit(TQ_DX_G) | bit(TQ_DX_O_NORM);
  if (L.c.ff_kind != TQ_DX_NONE) n |= bit(TQ_DX_NORM2) | bit(TQ_DX_HC2_IN) | bit(TQ_DX_HC2_OUT) | bit(TQ_DX_HC2_MIX);
  if (L.c.ff_kind == TQ_DX_MOE) {
    n |= bit(TQ_DX_ROUTER) | bit(TQ_DX_CORRECTION);
    if (L.c.shared_ff) n |= bit(TQ_DX_SHARED_GATE) | bit(TQ_DX_SHARED_UP) | bit(TQ_DX_SHARED_DOWN);
  }
  return n;
}

bool same_shape(const tq_dotanex_layer& a, const tq_dotanex_layer& b) {
  return a.kind == b.kind && a.heads == b.heads && a.kv_heads == b.kv_heads && a.dim == b.dim && a.vdim == b.vdim && a.q_rank == b.q_rank &&
         a.kv_rank == b.kv_rank && a.rot_dim == b.rot_dim && a.ff_kind == b.ff_kind && a.ff == b.ff && a.experts == b.experts && a.identity == b.identity &&
         a.shared_ff == b.shared_ff;
}

int check_layer(tq_ctx* ctx, const tq_dotanex_config& cfg, const tq_dotanex_layer* layers, uint32_t i) {
  const tq_dotanex_layer& c = layers[i];
  TQ_REQUIRE(ctx, c.weights_of < 0 || ((uint32_t)c.weights_of < cfg.n_layers && layers[c.weights_of].weights_of < 0 && same_shape(c, layers[c.weights_of])),
             "tq_dotanex_create: layer %u: weights_of must name a layer of the same shape with tensors of its own", i);
  TQ_REQUIRE(ctx, c.heads > 0 && c.heads <= 65535 && c.dim > 0 && c.vdim > 0, "tq_dotanex_create: layer %u: bad head sizes", i);
  TQ_REQUIRE(ctx, c.rot_dims % 2 == 0 && (c.rot_dims == 0 || c.rot_base > 1.0), "tq_dotanex_create: layer %u: bad rotation", i);
  if (c.kind == TQ_DX_ATTENTION) {
    TQ_REQUIRE(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "tq_dotanex_create: layer %u: heads must be a multiple of kv_heads", i);
    TQ_REQUIRE(ctx, c.vdim == c.dim, "tq_dotanex_create: layer %u: the values are the keys, so their sizes agree", i);
    TQ_REQUIRE(ctx, c.window > 0 && c.window <= 0x7fffffffu, "tq_dotanex_create: layer %u: bad window", i);
    TQ_REQUIRE(ctx, c.rot_dims <= c.dim, "tq_dotanex_create: layer %u: bad rotation", i);
    TQ_REQUIRE(ctx, !(c.rot_factor > 0) || (c.rot_original > 0 && c.rot_low > 0 && c.rot_high > c.rot_low), "tq_dotanex_create: layer %u: bad rotation scaling", i);
  } else if (c.kind == TQ_DX_LATENT) {
    TQ_REQUIRE(ctx, c.q_rank > 0 && c.kv_rank > 0 && c.rot_dims == c.rot_dim, "tq_dotanex_create: layer %u: bad latent sizes", i);
    TQ_REQUIRE(ctx, !(c.rot_factor > 0) || (c.rot_original > 0 && c.rot_fast > 0 && c.rot_slow > 0), "tq_dotanex_create: layer %u: bad rotation scaling", i);
  } else {
    TQ_REQUIRE(ctx, c.kind == TQ_DX_LIGHTNING, "tq_dotanex_create: layer %u: unknown mixer %u", i, c.kind);
    TQ_REQUIRE(ctx, c.decay != nullptr, "tq_dotanex_create: layer %u: no decays", i);
    for (uint32_t h = 0; h < c.heads; ++h) TQ_REQUIRE(ctx, c.decay[h] >= 0.f && c.decay[h] <= 1.f, "tq_dotanex_create: layer %u: decays must be in 0..1", i);
  }
  TQ_REQUIRE(ctx, c.ff_kind <= TQ_DX_MOE && (c.ff_kind == TQ_DX_NONE || c.ff > 0), "tq_dotanex_create: layer %u: bad feed-forward", i);
  TQ_REQUIRE(ctx, c.ff_kind != TQ_DX_MOE || (c.experts > 0 && c.experts + c.identity <= 1024 && c.top > 0 && c.top <= c.experts + c.identity && c.top <= 64),
             "tq_dotanex_create: layer %u: bad experts", i);
  return TQ_OK;
}

}  // namespace

extern "C" {

int tq_dotanex_create(tq_ctx* ctx, const tq_dotanex_config* cfg, const tq_dotanex_layer* layers, tq_dotanex** out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && layers && out, "tq_dotanex_create: null argument");
  *out = nullptr;
  TQ_REQUIRE(ctx, cfg->n_layers > 0 && cfg->width > 0 && cfg->width <= 49152 && cfg->vocab > 0, "tq_dotanex_create: width must be 1..49152, and there must be layers and a vocabulary");
  TQ_REQUIRE(ctx, cfg->streams > 0 && cfg->streams <= (uint32_t)kMaxStreams, "tq_dotanex_create: 1 to %d streams", kMaxStreams);
  TQ_REQUIRE(ctx, cfg->dtype == TQ_BF16 || cfg->dtype == TQ_F32, "tq_dotanex_create: dtype must be bf16 or f32");
  TQ_REQUIRE(ctx, cfg->max_seq > 0 && cfg->max_slots > 0 && (size_t)cfg->max_seq * cfg->max_slots < (1ull << 31), "tq_dotanex_create: cache empty or too large");
  for (uint32_t i = 0; i < cfg->n_layers; ++i)
    if (int st = check_layer(ctx, *cfg, layers, i)) return st;
  tq_dotanex* m = new (std::nothrow) tq_dotanex();
  if (!m) return fail(ctx, TQ_ENOMEM, "out of host memory");
  m->ctx = ctx;
  m->cfg = *cfg;
  m->layers.resize(cfg->n_layers);
  const size_t es = dtype_size(cfg->dtype), tokens = (size_t)cfg->max_slots * cfg->max_seq, width = cfg->width, streams = cfg->streams;
  int st = TQ_OK;
  auto A = [&](auto** p, size_t bytes) {
    if (st != TQ_OK) return;
    st = zalloc(m, (void**)p, bytes);
    if (st == TQ_OK) m->owned.push_back(*p);
  };
  auto W = [&](size_t rows, size_t cols, tq_dweight** w) {
    if (st == TQ_OK) st = tq_dweight_create(ctx, rows, cols, cfg->dtype, w);
  };
  auto U = [&](float** p, const std::vector<float>& v) {
    A(p, v.size() * 4);
    if (st == TQ_OK && !v.empty() &&
        (cudaMemcpyAsync(*p, v.data(), v.size() * 4, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess || cudaStreamSynchronize(ctx->stream) != cudaSuccess))
      st = fail(ctx, TQ_ECUDA, "tq_dotanex_create: copying constants failed");
  };
  auto most = [](size_t& a, size_t b) { a = a > b ? a : b; };
  size_t q_lat = 0, lqs = 0, head_jobs = 0;
  A(&m->final_norm, width * 4);
  W(cfg->vocab, width, &m->embed);
  W(cfg->vocab, width, &m->head);
  for (uint32_t i = 0; i < cfg->n_layers && st == TQ_OK; ++i) {
    Layer& L = m->layers[i];
    L.c = layers[i];
    L.c.decay = nullptr;
    const tq_dotanex_layer& c = layers[i];
    L.src = c.weights_of < 0 ? i : (size_t)c.weights_of;
    const bool own = c.weights_of < 0;
    L.q_rows = (size_t)c.heads * c.dim;
    size_t in_rows = 0;
    if (c.kind == TQ_DX_ATTENTION) {
      L.k_rows = (size_t)c.kv_heads * c.dim;
      L.k0 = up16(L.q_rows);
      in_rows = L.k0 + L.k_rows;
      L.dim_pad = up8(c.dim);
      A(&L.k_cache, tokens * c.kv_heads * L.dim_pad * es);
      A(&L.v_cache, tokens * c.kv_heads * L.dim_pad * es);
      most(m->mix_ld, up8(L.q_rows));
      if (own) {
        A(&L.q_gain, c.dim * es);
        A(&L.k_gain, c.dim * es);
        A(&L.sinks, c.heads * 4);
        std::vector<float> f(c.rot_dims / 2);
        banded_frequencies((int)c.rot_dims, c.rot_base, c.rot_factor, c.rot_low, c.rot_high, c.rot_original, f.data());
        U(&L.freq, f);
      }
    } else if (c.kind == TQ_DX_LATENT) {
      m->latent = true;
      L.d = latent_dims((int)c.heads, (int)c.dim, (int)c.rot_dim, (int)c.vdim, (int)c.kv_rank);
      L.absorb = cfg->dtype == TQ_BF16 && latent_absorb_supported(L.d);
      L.q_rows = (size_t)c.heads * (c.dim + c.rot_dim);
      L.k_rows = (size_t)c.kv_rank + c.rot_dim;
      L.g_rows = (size_t)c.heads * c.vdim;
      L.k0 = up16(c.q_rank);
      L.g0 = L.k0 + up16(L.k_rows);
      in_rows = L.g0 + L.g_rows;
      L.q_ld = up8(c.dim + c.rot_dim);
      L.key_pad = L.q_ld;
      L.v_pad = up8(c.vdim);
      L.ukt_rows = up16(c.kv_rank);
      L.uv_rows = up16(c.vdim);
      L.v0 = up16((size_t)c.heads * c.dim);                  // of w_kv
      A(&L.k_cache, tokens * L.d.row() * es);
      most(m->mix_ld, up8(L.g_rows));
      most(m->low_ld, c.q_rank + L.k_rows);
      most(m->lq_ld, c.heads * L.q_ld);
      if (L.absorb) {
        most(q_lat, (size_t)c.heads * L.d.c_pad);
        most(lqs, c.heads * L.q_ld);
        most(head_jobs, (size_t)c.heads * (cfg->max_slots / 8 + 1));
      }
      if (own) {
        A(&L.dq_norm, c.q_rank * 4);
        A(&L.c_norm, c.kv_rank * 4);
        std::vector<float> f(c.rot_dims / 2);
        yarn_frequencies((int)c.rot_dims, c.rot_base, c.rot_factor, c.rot_original, c.rot_fast, c.rot_slow, f.data(), &L.rot_mult);
        U(&L.freq, f);
        W(L.q_rows, c.q_rank, &L.w_uq);
        W(L.v0 + L.g_rows, c.kv_rank, &L.w_kv);
        if (L.absorb) {
          W(c.heads * L.ukt_rows, c.dim, &L.w_ukt);
          W(c.heads * L.uv_rows, c.kv_rank, &L.w_uv);
        }
        if (st == TQ_OK) most(m->cq_ld, L.w_uq->kpad);
      }
    } else {
      L.k_rows = L.q_rows;
      L.v_rows = L.g_rows = (size_t)c.heads * c.vdim;
      L.k0 = up16(L.q_rows);
      L.v0 = L.k0 + up16(L.k_rows);
      L.g0 = L.v0 + up16(L.v_rows);
      in_rows = L.g0 + L.g_rows;
      L.kc = up8(L.q_rows);
      L.vc = L.kc + up8(L.k_rows);
      L.gc = L.vc + up8(L.v_rows);
      most(m->mix_ld, L.gc + up8(L.g_rows));
      A(&L.state, (size_t)cfg->max_slots * c.heads * c.dim * c.vdim * 4);
      if (own) {
        A(&L.o_norm, L.v_rows * 4);
        U(&L.decay, std::vector<float>(c.decay, c.decay + c.heads));
      }
    }
    if (c.ff_kind == TQ_DX_MOE) {
      m->moe = true;
      most(m->max_experts, c.experts + c.identity);
      most(m->max_top, c.top);
    }
    if (!own) continue;
    for (int q = 0; q < (c.ff_kind == TQ_DX_NONE ? 1 : 2); ++q) {
      A(&L.norm[q], width * 4);
      A(&L.hc_in[q], streams * 4);
      A(&L.hc_out[q], streams * 4);
      A(&L.hc_mix[q], streams * streams * 4);
    }
    W(in_rows, width, &L.w_in);
    W(width, (size_t)c.heads * c.vdim, &L.w_out);
    if (st == TQ_OK) most(m->att_ld, L.w_out->kpad);
    if (c.ff_kind == TQ_DX_NONE) continue;
    const size_t n = c.ff_kind == TQ_DX_MOE ? c.experts : 1;
    L.gu_rows = 2 * up8(c.ff);
    L.down_rows = up16(width);
    L.have_expert.assign(n, 0);
    W(n * L.gu_rows, width, &L.gate_up);
    W(n * L.down_rows, c.ff, &L.down);
    if (st == TQ_OK) most(m->act_ld, L.down->kpad);
    if (c.ff_kind == TQ_DX_MOE) {
      L.shared0 = up16(c.experts + c.identity);
      A(&L.correction, (c.experts + c.identity) * 4);
      W(L.shared0 + 2 * up8(c.shared_ff), width, &L.front);
      if (c.shared_ff) {
        W(width, c.shared_ff, &L.shared_down);
        if (st == TQ_OK) most(m->shared_ld, L.shared_down->kpad);
      }
    }
  }
  A(&m->route.counts, m->max_experts * 4);
  A(&m->route.offsets, m->max_experts * 4);
  A(&m->route.n_jobs, 16);
  if (m->latent) {
    A(&m->plan.off, cfg->max_slots * 4);
    A(&m->plan.single, cfg->max_slots * 4);
    A(&m->plan.jobs, kExpandJobs * sizeof(int4));
    A(&m->plan.n_jobs, 16);
    A(&m->lqs, cfg->max_slots * lqs * es);
    A(&m->q_lat, cfg->max_slots * q_lat * es);
    A(&m->o_lat, cfg->max_slots * q_lat * es);
    A(&m->head_jobs, head_jobs * sizeof(int4));
    A(&m->n_head_jobs, 16);
  }
  if (st != TQ_OK) {
    release(m);
    return st;
  }
  *out = m;
  return TQ_OK;
}

int tq_dotanex_destroy(tq_dotanex* m) {
  if (!m) return TQ_OK;
  bind(m->ctx);
  cudaStreamSynchronize(m->ctx->stream);
  release(m);
  return TQ_OK;
}

int tq_dotanex_put(tq_dotanex* m, int which, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src != nullptr && (src_dtype == TQ_BF16 || src_dtype == TQ_F32), "tq_dotanex_put: the source must be bf16 or f32");
  TQ_REQUIRE(ctx, which >= TQ_DX_EMBED && which <= TQ_DX_SHARED_DOWN, "tq_dotanex_put: unknown tensor %d", which);
  const size_t width = m->cfg.width, streams = m->cfg.streams;
  const int dt = m->cfg.dtype;
  int st = TQ_OK;
  auto shape = [&](size_t r, size_t c) -> bool {
    if (rows == r && cols == c) return true;
    st = fail(ctx, TQ_EINVAL, "tq_dotanex_put: tensor %d of layer %zu must be [%zu, %zu], got [%zu, %zu]", which, layer, r, c, rows, cols);
    return false;
  };
  auto table = [&](size_t r, size_t c, void* dst, int dst_dtype) {
    if (shape(r, c)) st = put_vector(ctx, src, src_dtype, dst, dst_dtype, r * c, 0.f);
  };
  auto vec = [&](size_t n, void* dst, int dst_dtype = TQ_F32) { table(1, n, dst, dst_dtype); };
  auto mat = [&](size_t r, size_t c, tq_dweight* w, size_t row0, int interleave = 0) {
    if (st == TQ_OK && shape(r, c)) st = tq_dweight_put(ctx, w, src, src_dtype, r, c, row0, 0, interleave);
  };
  if (which <= TQ_DX_HEAD) {
    if (which == TQ_DX_FINAL_NORM) vec(width, m->final_norm);
    else mat(m->cfg.vocab, width, which == TQ_DX_EMBED ? m->embed : m->head, 0);
    if (st == TQ_OK) m->have |= bit(which);
    return st;
  }
  TQ_REQUIRE(ctx, layer < m->layers.size(), "tq_dotanex_put: layer %zu out of range", layer);
  Layer& L = m->layers[layer];
  const tq_dotanex_layer& c = L.c;
  TQ_REQUIRE(ctx, L.src == layer, "tq_dotanex_put: layer %zu uses the weights of layer %zu", layer, L.src);
  if (which == TQ_DX_GATE || which == TQ_DX_UP || which == TQ_DX_DOWN) {
    TQ_REQUIRE(ctx, expert < L.have_expert.size(), "tq_dotanex_put: layer %zu has %zu experts", layer, L.have_expert.size());
    if (which == TQ_DX_DOWN) mat(width, c.ff, L.down, expert * L.down_rows);
    else mat(c.ff, width, L.gate_up, expert * L.gu_rows, which == TQ_DX_GATE ? 1 : 2);
    if (st == TQ_OK) L.have_expert[expert] |= 1u << (which - TQ_DX_GATE);
    return st;
  }
  TQ_REQUIRE(ctx, needed(L) & bit(which), "tq_dotanex_put: layer %zu has no tensor %d", layer, which);
  const size_t all = (size_t)c.experts + c.identity;
  switch (which) {
    case TQ_DX_NORM1: case TQ_DX_NORM2: vec(width, L.norm[which - TQ_DX_NORM1]); break;
    case TQ_DX_HC1_IN: case TQ_DX_HC2_IN: vec(streams, L.hc_in[which == TQ_DX_HC2_IN]); break;
    case TQ_DX_HC1_OUT: case TQ_DX_HC2_OUT: vec(streams, L.hc_out[which == TQ_DX_HC2_OUT]); break;
    case TQ_DX_HC1_MIX: case TQ_DX_HC2_MIX: table(streams, streams, L.hc_mix[which == TQ_DX_HC2_MIX], TQ_F32); break;
    case TQ_DX_Q: mat(L.q_rows, width, L.w_in, 0); break;
    case TQ_DX_K: mat(L.k_rows, width, L.w_in, L.k0); break;
    case TQ_DX_V: mat(L.v_rows, width, L.w_in, L.v0); break;
    case TQ_DX_G: mat(L.g_rows, width, L.w_in, L.g0); break;
    case TQ_DX_O: mat(width, (size_t)c.heads * c.vdim, L.w_out, 0); break;
    case TQ_DX_Q_NORM: vec(c.dim, L.q_gain, dt); break;
    case TQ_DX_K_NORM: vec(c.dim, L.k_gain, dt); break;
    case TQ_DX_SINK: vec(c.heads, L.sinks); break;
    case TQ_DX_O_NORM: vec(L.v_rows, L.o_norm); break;
    case TQ_DX_DQ: mat(c.q_rank, width, L.w_in, 0); break;
    case TQ_DX_DQ_NORM: vec(c.q_rank, L.dq_norm); break;
    case TQ_DX_UQ: mat(L.q_rows, c.q_rank, L.w_uq, 0); break;
    case TQ_DX_DKV: mat(L.k_rows, width, L.w_in, L.k0); break;
    case TQ_DX_DKV_NORM: vec(c.kv_rank, L.c_norm); break;
    case TQ_DX_UK:
      mat((size_t)c.heads * c.dim, c.kv_rank, L.w_kv, 0);
      if (st == TQ_OK && L.absorb) st = dweight_put_head_transposed(ctx, L.w_ukt, src, src_dtype, c.heads, c.dim, c.kv_rank, L.ukt_rows);
      break;
    case TQ_DX_UV:
      mat(L.g_rows, c.kv_rank, L.w_kv, L.v0);
      if (L.absorb)
        for (size_t h = 0; h < c.heads && st == TQ_OK; ++h)
          st = tq_dweight_put(ctx, L.w_uv, static_cast<const char*>(src) + h * c.vdim * c.kv_rank * dtype_size(src_dtype), src_dtype, c.vdim, c.kv_rank, h * L.uv_rows, 0, 0);
      break;
    case TQ_DX_ROUTER: mat(all, width, L.front, 0); break;
    case TQ_DX_CORRECTION: vec(all, L.correction); break;
    case TQ_DX_SHARED_GATE: mat(c.shared_ff, width, L.front, L.shared0, 1); break;
    case TQ_DX_SHARED_UP: mat(c.shared_ff, width, L.front, L.shared0, 2); break;
    default: mat(width, c.shared_ff, L.shared_down, 0); break;
  }
  if (st == TQ_OK) L.have |= bit(which);
  return st;
}

int tq_dotanex_trace(tq_dotanex* m, float* sums_dev_or_null) {
  if (!m) return TQ_EINVAL;
  m->trace = sums_dev_or_null;
  return TQ_OK;
}

}  // extern "C"

#define TQ_STEP(expr) \
  if (int st = (expr)) return st;

// In what follows L is the layer (its caches and state), W the layer whose weights it uses.

static int attention_layer(tq_dotanex* m, const Layer& L, const Layer& W, const RaggedBatch& b) {
  tq_ctx* ctx = m->ctx;
  const tq_dotanex_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, W.k0, W.q_rows, DENSE_ROW, f32, m->mix, m->mix_ld);
  DenseSection& k = dense_section(e, W.w_in->rpad, W.k_rows, DENSE_CACHE, f32, L.v_cache, (size_t)c.kv_heads * L.dim_pad);
  k.inner = (int)c.dim;
  k.inner_pad = (int)L.dim_pad;
  e.cache_row = m->cache_row;
  TQ_STEP(launch_dense(ctx, W.w_in, in, b.rows, e));
  HeadNormRope n;
  n.r.heads = (int)c.heads;
  n.r.kv_heads = (int)c.kv_heads;
  n.r.dim = (int)c.dim;
  n.r.raw_pad = n.r.key_pad = (int)L.dim_pad;
  n.r.q = m->mix;
  n.r.ldq = m->mix_ld;
  n.r.raw = L.v_cache;
  n.r.keys = L.k_cache;
  n.r.q_gain = W.q_gain;
  n.r.k_gain = W.k_gain;
  n.r.rot.dims = (int)c.rot_dims;
  n.r.rot.freq = W.freq;
  n.r.eps = m->cfg.eps;
  TQ_STEP(launch_head_norm_rope(ctx, n, b, dt));
  WindowAttn a;
  a.heads = (int)c.heads;
  a.kv_heads = (int)c.kv_heads;
  a.dim = a.vdim = (int)c.dim;
  a.dim_pad = a.vdim_pad = (int)L.dim_pad;
  a.window = (int)c.window;
  a.scale = c.scale;
  a.sinks = W.sinks;
  return launch_window_attention(ctx, a, b, dt, m->mix, m->mix_ld, nullptr, 0, L.k_cache, L.v_cache, m->att, m->att_ld);
}

static int lightning_layer(tq_dotanex* m, const Layer& L, const Layer& W, const RaggedBatch& b) {
  const tq_dotanex_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt);
  char* mix = static_cast<char*>(m->mix);
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, W.k0, W.q_rows, DENSE_ROW, f32, mix, m->mix_ld).act = DENSE_SILU;
  dense_section(e, W.v0, W.k_rows, DENSE_ROW, f32, mix + W.kc * es, m->mix_ld).act = DENSE_SILU;
  dense_section(e, W.g0, W.v_rows, DENSE_ROW, f32, mix + W.vc * es, m->mix_ld).act = DENSE_SILU;
  dense_section(e, W.w_in->rpad, W.g_rows, DENSE_ROW, f32, mix + W.gc * es, m->mix_ld);
  TQ_STEP(launch_dense(m->ctx, W.w_in, in, b.rows, e));
  Gla g;
  g.heads = (int)c.heads;
  g.dim = (int)c.dim;
  g.vdim = (int)c.vdim;
  g.eps = m->cfg.eps;
  g.norm = W.o_norm;
  g.head_decay = W.decay;
  g.state = L.state;
  g.max_seq = (int)m->cfg.max_seq;
  GlaRows r;
  r.q = mix;
  r.k = mix + W.kc * es;
  r.v = mix + W.vc * es;
  r.gate = mix + W.gc * es;
  r.ld = m->mix_ld;
  r.out = m->att;
  r.ldo = m->att_ld;
  return launch_gla(m->ctx, g, r, b, dt);
}

// Sequences that bring several rows (at least min_q): keys and values of their positions, then windowed attention without a window.
static int latent_expanded(tq_dotanex* m, const Layer& L, const Layer& W, const RaggedBatch& b, int min_q, const Rotation& rot) {
  tq_ctx* ctx = m->ctx;
  const tq_dotanex_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt), q_head = (size_t)b.rows * L.q_ld;
  HeadNormRope n;
  n.r.heads = (int)c.heads;
  n.r.dim = (int)(c.dim + c.rot_dim);
  n.r.q = m->lq;
  n.r.ldq = L.q_ld;
  n.r.rot = rot;
  n.q_head = q_head;
  TQ_STEP(launch_head_norm_rope(ctx, n, b, dt));
  // as many sequences at a time as fit the budget, every one as long as the longest
  const size_t k_row = c.heads * L.key_pad * es, v_row = c.heads * L.v_pad * es;
  const int chunk = f32 ? 64 : (int)(b.max_len >= 256 ? 256 : up16(b.max_len));
  const size_t seq_jobs = ((size_t)b.max_len + chunk - 1) / chunk;
  size_t per = (m->cfg.expand_bytes ? m->cfg.expand_bytes : kExpandBytes) / ((k_row + v_row) * b.max_len);
  if (per > kExpandJobs / seq_jobs) per = kExpandJobs / seq_jobs;
  if (per > (size_t)b.n_seqs) per = b.n_seqs;
  if (per < 1) per = 1;
  TQ_REQUIRE(ctx, seq_jobs <= kExpandJobs, "tq_dotanex_step: sequences of %d positions are too long", b.max_len);
  const size_t exp_rows = per * b.max_len;
  TQ_STEP(ensure_expanded(m, exp_rows * k_row, exp_rows * v_row));
  DenseEpilogue e;
  DenseSection& k = dense_section(e, W.v0, (size_t)c.heads * c.dim, DENSE_ROW, f32, m->exp_k, c.heads * L.key_pad);
  k.inner = (int)c.dim;
  k.inner_pad = (int)L.key_pad;
  DenseSection& v = dense_section(e, W.w_kv->rpad, W.g_rows, DENSE_ROW, f32, m->exp_v, c.heads * L.v_pad);
  v.inner = (int)c.vdim;
  v.inner_pad = (int)L.v_pad;
  DenseGroups g;
  g.jobs = m->plan.jobs;
  g.n_jobs = m->plan.n_jobs;
  g.max_jobs = (int)(per * seq_jobs);
  g.chunk = chunk;
  g.group_rows = W.w_kv->rpad;
  WindowAttn a;
  a.heads = a.kv_heads = (int)c.heads;
  a.dim = (int)(c.dim + c.rot_dim);
  a.vdim = (int)c.vdim;
  a.dim_pad = (int)L.key_pad;
  a.vdim_pad = (int)L.v_pad;
  a.window = kAllKeys;
  a.scale = c.scale;
  a.sink = -INFINITY;
  a.q_head = q_head;
  RaggedBatch x = b;
  x.cache_row = m->plan.exp_row;
  x.cache_rows = exp_rows;
  for (int s0 = 0; s0 < b.n_seqs; s0 += (int)per) {
    const int s1 = s0 + (int)per < b.n_seqs ? s0 + (int)per : b.n_seqs;
    if (m->planned != s0 || m->planned_end != s1 || m->planned_chunk != chunk || m->planned_min != min_q) {
      TQ_STEP(launch_latent_plan(ctx, b, s0, s1, min_q, chunk, g.max_jobs, m->plan));
      m->planned = s0;
      m->planned_end = s1;
      m->planned_chunk = chunk;
      m->planned_min = min_q;
    }
    TQ_STEP(launch_dense_grouped(ctx, W.w_kv, L.k_cache, L.d.row(), b.cache_rows, g, e));
    TQ_STEP(launch_latent_place(ctx, L.d, b, m->plan, L.k_cache, m->exp_k, (int)L.key_pad, dt));
    TQ_STEP(launch_window_attention(ctx, a, x, dt, m->lq, L.q_ld, m->mix, m->mix_ld, m->exp_k, m->exp_v, m->att, m->att_ld));
  }
  return TQ_OK;
}

static int latent_layer(tq_dotanex* m, const Layer& L, const Layer& W, const RaggedBatch& b) {
  tq_ctx* ctx = m->ctx;
  const tq_dotanex_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const bool all_single = b.max_q == 1, some_single = all_single || (long long)b.rows < (long long)b.n_seqs * b.max_q;
  const bool absorb = L.absorb && some_single;
  TQ_REQUIRE(ctx, (size_t)b.rows * L.q_ld < (1ull << 31), "tq_dotanex_step: too many rows for these heads");
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, W.k0, c.q_rank, DENSE_ROW, 1, m->low, m->low_ld);
  dense_section(e, W.g0, W.k_rows, DENSE_ROW, 1, m->low + c.q_rank, m->low_ld);
  dense_section(e, W.w_in->rpad, W.g_rows, DENSE_ROW, f32, m->mix, m->mix_ld);
  TQ_STEP(launch_dense(ctx, W.w_in, in, b.rows, e));
  Rotation rot;
  rot.dims = (int)c.rot_dims;
  rot.freq = W.freq;
  rot.mult = W.rot_mult;
  rot.interleaved = true;
  LatentIn li;
  li.d = L.d;
  li.low = m->low;
  li.ld_low = m->low_ld;
  li.q_rank = li.c0 = (int)c.q_rank;
  li.q_gain = W.dq_norm;
  li.c_gain = W.c_norm;
  li.cq = m->cq;
  li.ld_cq = m->cq_ld;
  li.cache = L.k_cache;
  li.rot = rot;
  li.eps = m->cfg.eps;
  if (absorb) {
    const size_t kpad = W.w_ukt->kpad > W.w_uv->kpad ? W.w_ukt->kpad : W.w_uv->kpad;
    li.head_jobs = m->head_jobs;
    li.n_head_jobs = m->n_head_jobs;
    li.n_head_rows = b.n_seqs;
    li.head_chunk = dense_even_chunk(dt, kpad, b.n_seqs);
  }
  TQ_STEP(launch_latent_in(ctx, li, b, dt));
  DenseInput cq;
  cq.x = m->cq;
  cq.ldx = m->cq_ld;
  DenseEpilogue q;                                           // head by head: [head][row][q_ld]
  DenseSection& qs = dense_section(q, W.w_uq->rpad, W.q_rows, DENSE_ROW, f32, m->lq, L.q_ld);
  qs.inner = (int)(c.dim + c.rot_dim);
  qs.inner_pad = (int)(b.rows * L.q_ld);
  TQ_STEP(launch_dense(ctx, W.w_uq, cq, b.rows, q));
  rot.first = (int)c.dim;
  if (!all_single || !L.absorb) TQ_STEP(latent_expanded(m, L, W, b, L.absorb ? 2 : 1, rot));
  if (!absorb) return TQ_OK;
  const int* single = all_single ? nullptr : m->plan.single;
  const void* query = m->lq;
  if (single) {
    TQ_STEP(launch_latent_gather(ctx, b, single, m->lq, (int)c.heads, L.q_ld, m->lqs));
    query = m->lqs;
  }
  const size_t pairs = (size_t)c.heads * b.n_seqs;
  DenseGroups g;
  g.jobs = m->head_jobs;
  g.n_jobs = m->n_head_jobs;
  g.chunk = li.head_chunk;
  g.max_jobs = (int)(c.heads * (((size_t)b.n_seqs + g.chunk - 1) / g.chunk));
  g.group_rows = W.ukt_rows;
  DenseEpilogue ql;
  dense_section(ql, W.ukt_rows, c.kv_rank, DENSE_ROW, f32, m->q_lat, L.d.c_pad);
  TQ_STEP(launch_dense_grouped(ctx, W.w_ukt, query, L.q_ld, pairs, g, ql));
  TQ_STEP(launch_latent_decode(ctx, L.d, b, single, c.scale, rot, single == nullptr, m->q_lat, query, L.q_ld, L.k_cache, m->o_lat));
  DenseEpilogue o;
  dense_section(o, W.uv_rows, c.vdim, DENSE_HEADS, f32, m->att, m->att_ld).inner_pad = (int)c.vdim;
  o.head_rows = b.n_seqs;
  o.head_row = single;
  o.gate = m->mix;
  o.ldg = (long long)m->mix_ld;
  g.group_rows = W.uv_rows;
  return launch_dense_grouped(ctx, W.w_uv, m->o_lat, L.d.c_pad, pairs, g, o);
}

// Leaves its output to the stream kernel: y rows and how they are summed.
static int feed_forward(tq_dotanex* m, const Layer& W, size_t rows, StreamMix& mix) {
  tq_ctx* ctx = m->ctx;
  const tq_dotanex_layer& c = W.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t width = m->cfg.width, hn_ld = m->embed->kpad;
  DenseInput in;
  in.x = m->hn;
  in.ldx = hn_ld;
  if (c.ff_kind == TQ_DX_DENSE) {
    DenseEpilogue u;
    dense_section(u, W.gate_up->rpad, c.ff, DENSE_GLU, f32, m->act, m->act_ld);
    u.glu = DENSE_GLU_SILU;
    TQ_STEP(launch_dense(ctx, W.gate_up, in, rows, u));
    DenseInput a;
    a.x = m->act;
    a.ldx = m->act_ld;
    DenseEpilogue d;
    dense_section(d, W.down->rpad, width, DENSE_ROW, 1, m->y, width);
    mix.y = m->y;
    return launch_dense(ctx, W.down, a, rows, d);
  }
  ExpertFf f;
  f.front = W.front;
  f.gate_up = W.gate_up;
  f.down = W.down;
  f.shared_down = W.shared_down;
  f.logits = (size_t)c.experts + c.identity;
  f.logit_end = W.shared0;
  f.experts = c.experts;
  f.identity = c.identity;
  f.top = c.top;
  f.ff = c.ff;
  f.shared_ff = c.shared_ff;
  f.gu_rows = W.gu_rows;
  f.down_rows = W.down_rows;
  f.rule.score = ROUTE_SOFTMAX;
  f.rule.renorm = true;
  f.rule.correction = W.correction;
  f.rule.identity = (int)c.identity;
  f.limit = c.limit;
  f.alpha = kGluAlpha;
  f.shared_limit = c.shared_limit;
  ExpertBuffers b;
  b.logits = m->logits;
  b.ld_logits = m->max_experts;
  b.route = m->route;
  b.gathered = m->gathered;
  b.act = m->act;
  b.act_ld = m->act_ld;
  b.shared = m->shared;
  b.shared_ld = m->shared_ld;
  b.y = m->yp;
  b.y_shared = m->ys;
  return launch_expert_ff(ctx, f, b, m->hn, hn_ld, rows, width, dt, mix);
}

extern "C" int tq_dotanex_step(tq_dotanex* m, const int* token_ids_dev, size_t rows, const int* seq_rows_dev, const int* starts_dev, const int* slots_dev,
                               size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev, size_t n_logits, float* logits_dev) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  const tq_dotanex_config& c = m->cfg;
  TQ_REQUIRE(ctx, token_ids_dev && starts_dev && rows > 0 && n_seqs > 0, "tq_dotanex_step: null pointer or empty step");
  TQ_REQUIRE(ctx, rows < (1ull << 24), "tq_dotanex_step: too many rows");
  TQ_REQUIRE(ctx, seq_rows_dev || rows == n_seqs, "tq_dotanex_step: without row offsets every sequence brings one row");
  TQ_REQUIRE(ctx, max_q > 0 && max_q <= rows && (seq_rows_dev || max_q == 1), "tq_dotanex_step: max_q must bound the sequences' rows");
  TQ_REQUIRE(ctx, n_seqs <= c.max_slots && max_len > 0 && max_len <= c.max_seq, "tq_dotanex_step: at most %u sequences of %u positions", c.max_slots, c.max_seq);
  TQ_REQUIRE(ctx, n_logits == 0 || logits_dev, "tq_dotanex_step: null logits");
  TQ_REQUIRE(ctx, logit_rows_dev || n_logits == 0 || n_logits == rows, "tq_dotanex_step: without a row list every row has logits");
  TQ_REQUIRE(ctx, m->have == (bit(TQ_DX_EMBED) | bit(TQ_DX_FINAL_NORM) | bit(TQ_DX_HEAD)), "tq_dotanex_step: the embedding, the final norm or the head is missing");
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer& L = m->layers[i];
    bool all = L.src != i || L.have == needed(L);
    for (unsigned char e : L.have_expert) all = all && e == 7;
    TQ_REQUIRE(ctx, all, "tq_dotanex_step: layer %zu has tensors missing", i);
  }
  TQ_STEP(ensure_rows(m, rows));
  TQ_REQUIRE(ctx, n_logits <= m->ws_rows, "tq_dotanex_step: more logits than rows");
  m->planned = -1;
  TQ_STEP(launch_embedding_pos(ctx, m->embed->data, m->embed->kpad, nullptr, c.dtype, token_ids_dev, seq_rows_dev, starts_dev, slots_dev, (int)n_seqs, rows,
                               (int)c.width, (int)c.vocab, (int)c.max_seq, (int)c.max_seq, (int)c.max_slots, m->x, m->row_pos, m->cache_row));
  RaggedBatch b;
  b.n_seqs = (int)n_seqs;
  b.rows = (int)rows;
  b.max_q = (int)max_q;
  b.max_len = (int)max_len;
  b.seq_rows = seq_rows_dev;
  b.row_pos = m->row_pos;
  b.cache_row = m->cache_row;
  b.cache_rows = (size_t)c.max_slots * c.max_seq;
  // the streams are all equal to the embedding until the first sublayer is done
  StreamMix s;
  s.streams = (int)c.streams;
  s.src = m->x;
  s.dst = m->xs;
  s.out = m->hn;
  s.out_dtype = c.dtype;
  s.ld_out = m->embed->kpad;
  s.eps = c.eps;
  auto read = [&](StreamMix& mix, const Layer* next, int q) {
    mix.w_in = next ? next->hc_in[q] : nullptr;
    mix.gain = next ? next->norm[q] : nullptr;
  };
  auto write = [&](StreamMix& mix, const Layer& W, int q) {
    mix.mix = W.hc_mix[q];
    mix.w_out = W.hc_out[q];
  };
  read(s, &m->layers[m->layers[0].src], 0);
  TQ_STEP(launch_stream_mix(ctx, s, rows, c.width));
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer &L = m->layers[i], &W = m->layers[L.src];
    const Layer* next = i + 1 < m->layers.size() ? &m->layers[m->layers[i + 1].src] : nullptr;
    const bool ff = L.c.ff_kind != TQ_DX_NONE;
    float* sum = m->trace ? m->trace + i * rows * c.width : nullptr;
    TQ_STEP(L.c.kind == TQ_DX_ATTENTION ? attention_layer(m, L, W, b) : L.c.kind == TQ_DX_LATENT ? latent_layer(m, L, W, b) : lightning_layer(m, L, W, b));
    DenseInput att;
    att.x = m->att;
    att.ldx = m->att_ld;
    DenseEpilogue o;
    dense_section(o, W.w_out->rpad, c.width, DENSE_ROW, 1, m->y, c.width);
    TQ_STEP(launch_dense(ctx, W.w_out, att, rows, o));
    StreamMix mix = s;
    mix.y = m->y;
    mix.sum = ff ? nullptr : sum;
    write(mix, W, 0);
    read(mix, ff ? &W : next, ff ? 1 : 0);
    TQ_STEP(launch_stream_mix(ctx, mix, rows, c.width));
    s.src = m->xs;
    s.src_streams = (int)c.streams;
    if (!ff) continue;
    StreamMix after = s;
    TQ_STEP(feed_forward(m, W, rows, after));
    after.sum = sum;
    write(after, W, 1);
    read(after, next, 0);
    TQ_STEP(launch_stream_mix(ctx, after, rows, c.width));
  }
  if (n_logits) {
    s.dst = nullptr;
    s.src_rows = logit_rows_dev;
    s.w_in = nullptr;
    s.gain = m->final_norm;
    TQ_STEP(launch_stream_mix(ctx, s, n_logits, c.width));
    DenseInput h;
    h.x = m->hn;
    h.ldx = m->embed->kpad;
    DenseEpilogue e;
    dense_section(e, m->head->rpad, c.vocab, DENSE_ROW, 1, logits_dev, c.vocab);
    TQ_STEP(launch_dense(ctx, m->head, h, n_logits, e));
  }
  return TQ_OK;
}
#undef TQ_STEP
