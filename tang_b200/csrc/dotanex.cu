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

#include <new>
#include <vector>

#include "dense.cuh"
#include "expert_route.cuh"
#include "gla.cuh"
#include "latent_attention.cuh"
#include "ragged.h"
#include "rowops.cuh"
#include "window_attention.cuh"

using namespace tq;

namespace {

constexpr float kGluAlpha = 1.702f;
constexpr int kAllKeys = 0x7fffffff;
constexpr size_t kExpandBytes = 1ull << 30;      // of expanded keys and values at a time
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
