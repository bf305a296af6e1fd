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
