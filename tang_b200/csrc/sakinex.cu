// Sakinex: a decoder with one residual stream whose mixers run windowed attention (convolved queries, keys and values, pooled blocks
// behind the window) and a minGRU on the same input, each followed by routed experts with a gated shared one; every
// sublayer's input passes a short convolution, and a stretch of layers may run several times (include/tangq.h, tq_sakinex_*).
//
// A run of a layer is
//   * `in`: the projections of both branches as one weight, raw rows [q | k | v | z | u | g];
//   * convolution, rotation and norm of the heads into the caches, pooled blocks, attention; beside it the recurrence;
//   * `out`: both output projections as one weight over [attention | recurrence] (the branches' factors are in those rows) -> f32;
//   * the stream kernel: residual, next norm, and in steps of one row per sequence the next convolution;
//   * the experts (expert_ff.cuh) and the stream kernel again.
// In other steps the normed rows leave the stream kernel for a convolution of their own, and one kernel at the end of the run moves
// the states of its three convolutions on.
#include <cuda_bf16.h>

#include <new>
#include <vector>

#include "dense.cuh"
#include "expert_ff.cuh"
#include "min_gru.cuh"
#include "ragged.h"
#include "rowops.cuh"
#include "short_conv.cuh"
#include "window_attention.cuh"

using namespace tq;

namespace {

size_t up16(size_t n) { return (n + 15) / 16 * 16; }
size_t up8(size_t n) { return (n + 7) / 8 * 8; }

struct Layer {
  tq_sakinex_layer c;
  size_t src = 0;                                             // the run whose weights it uses
  size_t q_rows = 0, k_rows = 0, v_rows = 0;                  // rows that exist
  size_t k0 = 0, v0 = 0, z0 = 0, u0 = 0, g0 = 0, in_rows = 0; // sections of w_in, and columns of the raw rows
  size_t right0 = 0;                                          // first column of the recurrence in w_out
  size_t key_pad = 0, val_pad = 0, pool_rows = 0;
  // ---- weights (of run src)
  tq_dweight *w_in = nullptr, *w_out = nullptr;
  float *norm[2] = {}, *canon[2] = {}, *conv = nullptr, *freq = nullptr, *z_bias = nullptr, *x_bias = nullptr;
  float rot_mult = 1.f;
  tq_dweight *front = nullptr, *gate_up = nullptr, *down = nullptr, *shared_down = nullptr;   // front: [router, shared switch | shared gate/up]
  float* router_bias = nullptr;
  size_t shared0 = 0, gu_rows = 0, down_rows = 0;             // first row of the shared gate/up; rows of one expert in the stacked weights
  unsigned long long have = 0;                                // bit per tensor put
  std::vector<unsigned char> have_expert;                     // bits gate, up, down
  // ---- of its own
  void *k_cache = nullptr, *v_cache = nullptr, *pooled_k = nullptr, *pooled_v = nullptr;
  void *canon_state[2] = {}, *conv_state = nullptr;
  float* state = nullptr;
};

}  // namespace

struct tq_sakinex {
  tq_ctx* ctx = nullptr;
  tq_sakinex_config cfg{};
  std::vector<Layer> layers;
  tq_dweight *embed = nullptr, *head = nullptr;
  float *final_norm = nullptr, *one = nullptr, *mult = nullptr;   // one, mult: the factors of the stream kernel
  unsigned long long have = 0;
  size_t mix_ld = 0, q_ld = 0, att_ld = 0, act_ld = 0, shared_ld = 0, max_experts = 0, max_top = 0;
  size_t ws_rows = 0;
  float *x = nullptr, *xs = nullptr, *y = nullptr, *logits = nullptr, *yp = nullptr, *ys = nullptr;
  void *hn = nullptr, *raw_hn[2] = {}, *mix = nullptr, *q = nullptr, *att = nullptr, *gathered = nullptr, *act = nullptr, *shared = nullptr;
  int *row_pos = nullptr, *cache_row = nullptr;
  Routing route;
  float* trace = nullptr;
  std::vector<void*> owned;
};

namespace {

struct Workspace {
  void** p;
  size_t bytes;
};

std::vector<Workspace> workspaces(tq_sakinex* m, size_t n) {
  const size_t es = dtype_size(m->cfg.dtype), width = m->cfg.width, pairs = n * m->max_top, hn = m->embed ? m->embed->kpad : 0;
  const size_t moe = m->max_experts ? n : 0;
  return {{(void**)&m->x, n * width * 4}, {(void**)&m->xs, n * width * 4}, {(void**)&m->y, n * width * 4}, {(void**)&m->logits, moe * (m->max_experts + 1) * 4},
          {(void**)&m->yp, pairs * width * 4}, {(void**)&m->ys, moe * width * 4}, {&m->hn, n * hn * es}, {&m->raw_hn[0], n * hn * es}, {&m->raw_hn[1], n * hn * es},
          {&m->mix, n * m->mix_ld * es}, {&m->q, n * m->q_ld * es}, {&m->att, n * m->att_ld * es}, {&m->gathered, pairs * hn * es}, {&m->act, pairs * m->act_ld * es},
          {&m->shared, moe * m->shared_ld * es}, {(void**)&m->row_pos, n * 4}, {(void**)&m->cache_row, n * 4}, {(void**)&m->route.expert, pairs * 4},
          {(void**)&m->route.weight, pairs * 4}, {(void**)&m->route.rank, pairs * 4}, {(void**)&m->route.slot, pairs * 4}, {(void**)&m->route.slot_row, pairs * 4},
          {(void**)&m->route.slot_weight, pairs * 4}, {(void**)&m->route.jobs, moe ? (pairs + m->max_experts) * sizeof(int4) : 0}};
}

void release(tq_sakinex* m) {
  for (auto& L : m->layers)
    for (tq_dweight* w : {L.w_in, L.w_out, L.front, L.gate_up, L.down, L.shared_down})
      if (w) tq_dweight_free(m->ctx, w);
  for (tq_dweight* w : {m->embed, m->head})
    if (w) tq_dweight_free(m->ctx, w);
  for (auto& w : workspaces(m, 0))
    if (*w.p) cudaFree(*w.p);
  for (void* p : m->owned) cudaFree(p);
  delete m;
  cudaGetLastError();
}

int zalloc(tq_sakinex* m, void** p, size_t bytes) {
  cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
  if (e == cudaErrorMemoryAllocation) {
    cudaGetLastError();
    return fail(m->ctx, TQ_ENOMEM, "sakinex: out of device memory (%zu bytes)", bytes);
  }
  TQ_CUDA(m->ctx, e);
  TQ_CUDA(m->ctx, cudaMemsetAsync(*p, 0, bytes, m->ctx->stream));
  return TQ_OK;
}

int ensure_rows(tq_sakinex* m, size_t rows) {
  if (rows <= m->ws_rows) return TQ_OK;
  tq_ctx* ctx = m->ctx;
  TQ_REQUIRE(ctx, !ctx->capturing, "tq_sakinex_step: workspaces must be sized before graph capture (run once eagerly)");
  TQ_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  ctx->ws_generation++;   // graphs recorded over the old buffers must not be replayed
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

constexpr unsigned long long bit(int t) { return 1ull << t; }

unsigned long long needed(const Layer& L) {
  unsigned long long n = bit(TQ_SX_NORM1) | bit(TQ_SX_CANON1) | bit(TQ_SX_Q) | bit(TQ_SX_K) | bit(TQ_SX_V) | bit(TQ_SX_LEFT_O) | bit(TQ_SX_Z) | bit(TQ_SX_Z_BIAS) |
                         bit(TQ_SX_X) | bit(TQ_SX_X_BIAS) | bit(TQ_SX_G) | bit(TQ_SX_RIGHT_O);
  if (L.c.taps) n |= bit(TQ_SX_Q_CONV) | bit(TQ_SX_K_CONV) | bit(TQ_SX_V_CONV);
  if (L.c.experts) {
    n |= bit(TQ_SX_NORM2) | bit(TQ_SX_CANON2) | bit(TQ_SX_ROUTER) | bit(TQ_SX_ROUTER_BIAS);
    if (L.c.shared_ff) n |= bit(TQ_SX_SHARED_GATE) | bit(TQ_SX_SHARED_UP) | bit(TQ_SX_SHARED_DOWN) | bit(TQ_SX_SHARED_SWITCH);
  }
  return n;
}

bool same_shape(const tq_sakinex_layer& a, const tq_sakinex_layer& b) {
  return a.heads == b.heads && a.kv_heads == b.kv_heads && a.dim == b.dim && a.vdim == b.vdim && a.taps == b.taps && a.rot_dims == b.rot_dims &&
         a.state_width == b.state_width && a.experts == b.experts && a.ff == b.ff && a.shared_ff == b.shared_ff;
}

int check_layer(tq_ctx* ctx, const tq_sakinex_config& cfg, const tq_sakinex_layer* layers, uint32_t i) {
  const tq_sakinex_layer& c = layers[i];
  TQ_REQUIRE(ctx, c.weights_of < 0 || ((uint32_t)c.weights_of < i && layers[c.weights_of].weights_of < 0 && same_shape(c, layers[c.weights_of])),
             "tq_sakinex_create: run %u: weights_of must name an earlier run of the same shape with tensors of its own", i);
  TQ_REQUIRE(ctx, i > 0 || !c.add_embedding, "tq_sakinex_create: the first run starts from the embedding");
  TQ_REQUIRE(ctx, c.heads > 0 && c.heads <= 65535 && c.dim > 0 && c.vdim > 0, "tq_sakinex_create: run %u: bad head sizes", i);
  TQ_REQUIRE(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "tq_sakinex_create: run %u: heads must be a multiple of kv_heads", i);
  TQ_REQUIRE(ctx, c.window > 0 && c.window <= 0x7fffffffu && c.pool <= 0x7fffffffu, "tq_sakinex_create: run %u: bad window", i);
  TQ_REQUIRE(ctx, c.taps <= 256, "tq_sakinex_create: run %u: bad convolution", i);
  TQ_REQUIRE(ctx, c.rot_dims % 2 == 0 && c.rot_dims <= c.dim && (c.rot_dims == 0 || c.rot_base > 1.0), "tq_sakinex_create: run %u: bad rotation", i);
  TQ_REQUIRE(ctx, !(c.rot_factor > 0) || (c.rot_original > 0 && c.rot_fast > 0 && c.rot_slow > 0), "tq_sakinex_create: run %u: bad rotation scaling", i);
  TQ_REQUIRE(ctx, c.state_width > 0, "tq_sakinex_create: run %u: the recurrence is empty", i);
  TQ_REQUIRE(ctx, c.experts == 0 || (c.experts <= 1023 && c.ff > 0 && c.top > 0 && c.top <= c.experts && c.top <= 64), "tq_sakinex_create: run %u: bad experts", i);
  return TQ_OK;
}

}  // namespace

extern "C" {

int tq_sakinex_create(tq_ctx* ctx, const tq_sakinex_config* cfg, const tq_sakinex_layer* layers, tq_sakinex** out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && layers && out, "tq_sakinex_create: null argument");
  *out = nullptr;
  TQ_REQUIRE(ctx, cfg->n_layers > 0 && cfg->width > 0 && cfg->width <= 49152 && cfg->vocab > 0, "tq_sakinex_create: width must be 1..49152, and there must be layers and a vocabulary");
  TQ_REQUIRE(ctx, cfg->taps >= 1 && cfg->taps <= 256, "tq_sakinex_create: 1 to 256 taps");
  TQ_REQUIRE(ctx, cfg->dtype == TQ_BF16 || cfg->dtype == TQ_F32, "tq_sakinex_create: dtype must be bf16 or f32");
  TQ_REQUIRE(ctx, cfg->max_seq > 0 && cfg->max_slots > 0 && (size_t)cfg->max_seq * cfg->max_slots < (1ull << 31), "tq_sakinex_create: cache empty or too large");
  for (uint32_t i = 0; i < cfg->n_layers; ++i)
    if (int st = check_layer(ctx, *cfg, layers, i)) return st;
  tq_sakinex* m = new (std::nothrow) tq_sakinex();
  if (!m) return fail(ctx, TQ_ENOMEM, "out of host memory");
  m->ctx = ctx;
  m->cfg = *cfg;
  m->layers.resize(cfg->n_layers);
  const size_t es = dtype_size(cfg->dtype), slots = cfg->max_slots, tokens = slots * cfg->max_seq, width = cfg->width;
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
      st = fail(ctx, TQ_ECUDA, "tq_sakinex_create: copying constants failed");
  };
  auto most = [](size_t& a, size_t b) { a = a > b ? a : b; };
  A(&m->final_norm, width * 4);
  U(&m->one, {1.f});
  U(&m->mult, {cfg->residual_mult});
  W(cfg->vocab, width, &m->embed);
  W(cfg->vocab, width, &m->head);
  for (uint32_t i = 0; i < cfg->n_layers && st == TQ_OK; ++i) {
    Layer& L = m->layers[i];
    L.c = layers[i];
    const tq_sakinex_layer& c = L.c;
    L.src = c.weights_of < 0 ? i : (size_t)c.weights_of;
    L.q_rows = (size_t)c.heads * c.dim;
    L.k_rows = (size_t)c.kv_heads * c.dim;
    L.v_rows = (size_t)c.kv_heads * c.vdim;
    L.k0 = up16(L.q_rows);
    L.v0 = L.k0 + up16(L.k_rows);
    L.z0 = L.v0 + up16(L.v_rows);
    L.u0 = L.z0 + up16(c.state_width);
    L.g0 = L.u0 + up16(c.state_width);
    L.in_rows = L.g0 + c.state_width;
    L.right0 = up16((size_t)c.heads * c.vdim);
    L.key_pad = up8(c.dim);
    L.val_pad = up8(c.vdim);
    A(&L.k_cache, tokens * c.kv_heads * L.key_pad * es);
    A(&L.v_cache, tokens * c.kv_heads * L.val_pad * es);
    if (c.pool) {
      L.pool_rows = cfg->max_seq / c.pool;
      A(&L.pooled_k, slots * L.pool_rows * c.kv_heads * L.key_pad * es);
      A(&L.pooled_v, slots * L.pool_rows * c.kv_heads * L.val_pad * es);
    }
    if (c.taps > 1) A(&L.conv_state, slots * (c.taps - 1) * L.z0 * es);
    for (int q = 0; q < (c.experts ? 2 : 1); ++q) A(&L.canon_state[q], slots * (cfg->taps - 1) * width * es);
    A(&L.state, slots * ((c.state_width + 1) / 2 * 2) * 4);
    most(m->mix_ld, up16(L.in_rows));
    most(m->q_ld, up8(L.q_rows));
    most(m->max_experts, c.experts);
    most(m->max_top, c.top);
    if (c.weights_of >= 0) continue;
    std::vector<float> f(c.rot_dims / 2);
    yarn_frequencies((int)c.rot_dims, c.rot_base, c.rot_factor, c.rot_original, c.rot_fast, c.rot_slow, f.data(), &L.rot_mult);
    U(&L.freq, f);
    U(&L.conv, std::vector<float>((c.taps ? c.taps : 1) * L.z0, c.taps ? 0.f : 1.f));
    A(&L.z_bias, up8(c.state_width) * 4);
    A(&L.x_bias, up8(c.state_width) * 4);
    for (int q = 0; q < (c.experts ? 2 : 1); ++q) {
      A(&L.norm[q], width * 4);
      A(&L.canon[q], cfg->taps * width * 4);
    }
    W(L.in_rows, width, &L.w_in);
    W(width, L.right0 + c.state_width, &L.w_out);
    if (st == TQ_OK) most(m->att_ld, L.w_out->kpad);
    if (!c.experts) continue;
    L.gu_rows = 2 * up8(c.ff);
    L.down_rows = up16(width);
    L.have_expert.assign(c.experts, 0);
    W(c.experts * L.gu_rows, width, &L.gate_up);
    W(c.experts * L.down_rows, c.ff, &L.down);
    if (st == TQ_OK) most(m->act_ld, L.down->kpad);
    L.shared0 = up16((size_t)c.experts + 1);
    A(&L.router_bias, c.experts * 4);
    W(L.shared0 + 2 * up8(c.shared_ff), width, &L.front);
    if (c.shared_ff) {
      W(width, c.shared_ff, &L.shared_down);
      if (st == TQ_OK) most(m->shared_ld, L.shared_down->kpad);
    }
  }
  A(&m->route.counts, m->max_experts * 4);
  A(&m->route.offsets, m->max_experts * 4);
  A(&m->route.n_jobs, 16);
  if (st != TQ_OK) {
    release(m);
    return st;
  }
  *out = m;
  return TQ_OK;
}

int tq_sakinex_destroy(tq_sakinex* m) {
  if (!m) return TQ_OK;
  bind(m->ctx);
  cudaStreamSynchronize(m->ctx->stream);
  release(m);
  return TQ_OK;
}

int tq_sakinex_put(tq_sakinex* m, int which, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src != nullptr && (src_dtype == TQ_BF16 || src_dtype == TQ_F32), "tq_sakinex_put: the source must be bf16 or f32");
  TQ_REQUIRE(ctx, which >= TQ_SX_EMBED && which <= TQ_SX_SHARED_SWITCH, "tq_sakinex_put: unknown tensor %d", which);
  const size_t width = m->cfg.width;
  int st = TQ_OK;
  auto shape = [&](size_t r, size_t c) -> bool {
    if (rows == r && cols == c) return true;
    st = fail(ctx, TQ_EINVAL, "tq_sakinex_put: tensor %d of layer %zu must be [%zu, %zu], got [%zu, %zu]", which, layer, r, c, rows, cols);
    return false;
  };
  auto vec = [&](size_t n, void* dst) {
    if (shape(1, n)) st = put_vector(ctx, src, src_dtype, dst, TQ_F32, n, 0.f);
  };
  auto mat = [&](size_t r, size_t c, tq_dweight* w, size_t row0, int interleave = 0, size_t col0 = 0) {
    if (shape(r, c)) st = tq_dweight_put(ctx, w, src, src_dtype, r, c, row0, col0, interleave);
  };
  auto conv = [&](size_t n, size_t taps, float* dst, size_t ld, size_t col0) {
    if (shape(n, taps)) st = put_conv_weights(ctx, src, src_dtype, dst, n, taps, ld, col0);
  };
  if (which <= TQ_SX_HEAD) {
    if (which == TQ_SX_FINAL_NORM) vec(width, m->final_norm);
    else mat(m->cfg.vocab, width, which == TQ_SX_EMBED ? m->embed : m->head, 0);
    if (st == TQ_OK) m->have |= bit(which);
    return st;
  }
  TQ_REQUIRE(ctx, layer < m->layers.size(), "tq_sakinex_put: layer %zu out of range", layer);
  Layer& L = m->layers[layer];
  const tq_sakinex_layer& c = L.c;
  TQ_REQUIRE(ctx, L.src == layer, "tq_sakinex_put: run %zu uses the weights of run %zu", layer, L.src);
  if (which == TQ_SX_GATE || which == TQ_SX_UP || which == TQ_SX_DOWN) {
    TQ_REQUIRE(ctx, expert < L.have_expert.size(), "tq_sakinex_put: layer %zu has %zu experts", layer, L.have_expert.size());
    if (which == TQ_SX_DOWN) mat(width, c.ff, L.down, expert * L.down_rows);
    else mat(c.ff, width, L.gate_up, expert * L.gu_rows, which == TQ_SX_GATE ? 1 : 2);
    if (st == TQ_OK) L.have_expert[expert] |= 1u << (which - TQ_SX_GATE);
    return st;
  }
  TQ_REQUIRE(ctx, needed(L) & bit(which), "tq_sakinex_put: layer %zu has no tensor %d", layer, which);
  switch (which) {
    case TQ_SX_NORM1: case TQ_SX_NORM2: vec(width, L.norm[which - TQ_SX_NORM1]); break;
    case TQ_SX_CANON1: case TQ_SX_CANON2: conv(width, m->cfg.taps, L.canon[which - TQ_SX_CANON1], width, 0); break;
    case TQ_SX_Q: mat(L.q_rows, width, L.w_in, 0); break;
    case TQ_SX_K: mat(L.k_rows, width, L.w_in, L.k0); break;
    case TQ_SX_V: mat(L.v_rows, width, L.w_in, L.v0); break;
    case TQ_SX_Q_CONV: conv(L.q_rows, c.taps, L.conv, L.z0, 0); break;
    case TQ_SX_K_CONV: conv(L.k_rows, c.taps, L.conv, L.z0, L.k0); break;
    case TQ_SX_V_CONV: conv(L.v_rows, c.taps, L.conv, L.z0, L.v0); break;
    case TQ_SX_LEFT_O: mat(width, (size_t)c.heads * c.vdim, L.w_out, 0); break;
    case TQ_SX_Z: mat(c.state_width, width, L.w_in, L.z0); break;
    case TQ_SX_Z_BIAS: vec(c.state_width, L.z_bias); break;
    case TQ_SX_X: mat(c.state_width, width, L.w_in, L.u0); break;
    case TQ_SX_X_BIAS: vec(c.state_width, L.x_bias); break;
    case TQ_SX_G: mat(c.state_width, width, L.w_in, L.g0); break;
    case TQ_SX_RIGHT_O: mat(width, c.state_width, L.w_out, 0, 0, L.right0); break;
    case TQ_SX_ROUTER: mat(c.experts, width, L.front, 0); break;
    case TQ_SX_ROUTER_BIAS: vec(c.experts, L.router_bias); break;
    case TQ_SX_SHARED_GATE: mat(c.shared_ff, width, L.front, L.shared0, 1); break;
    case TQ_SX_SHARED_UP: mat(c.shared_ff, width, L.front, L.shared0, 2); break;
    case TQ_SX_SHARED_DOWN: mat(width, c.shared_ff, L.shared_down, 0); break;
    default: mat(1, width, L.front, c.experts); break;
  }
  if (st == TQ_OK) L.have |= bit(which);
  return st;
}

int tq_sakinex_trace(tq_sakinex* m, float* streams_dev_or_null) {
  if (!m) return TQ_EINVAL;
  m->trace = streams_dev_or_null;
  return TQ_OK;
}

}  // extern "C"

#define TQ_STEP(expr) \
  if (int st = (expr)) return st;

// In what follows L is the run (its caches and states), W the run whose weights it uses.

static ShortConv canon(const tq_sakinex* m, const Layer& L, const Layer& W, int q) {
  ShortConv c;
  c.taps = (int)m->cfg.taps;
  c.channels = (int)m->cfg.width;
  c.w = W.canon[q];
  c.state = L.canon_state[q];
  c.max_seq = (int)m->cfg.max_seq;
  return c;
}

static ShortConv head_conv(const tq_sakinex* m, const Layer& L, const Layer& W) {
  ShortConv c;
  c.taps = L.c.taps ? (int)L.c.taps : 1;
  c.channels = (int)L.z0;
  c.w = W.conv;
  c.state = L.conv_state;
  c.max_seq = (int)m->cfg.max_seq;
  return c;
}

static int mixer(tq_sakinex* m, const Layer& L, const Layer& W, const RaggedBatch& b) {
  tq_ctx* ctx = m->ctx;
  const tq_sakinex_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt);
  char* mix = static_cast<char*>(m->mix);
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, W.w_in->rpad, L.in_rows, DENSE_ROW, f32, mix, m->mix_ld);
  TQ_STEP(launch_dense(ctx, W.w_in, in, b.rows, e));
  ConvHeads h;
  h.heads = (int)c.heads;
  h.kv_heads = (int)c.kv_heads;
  h.dim = (int)c.dim;
  h.vdim = (int)c.vdim;
  h.key_pad = (int)L.key_pad;
  h.val_pad = (int)L.val_pad;
  h.raw = mix;
  h.ld = m->mix_ld;
  h.k0 = (int)L.k0;
  h.v0 = (int)L.v0;
  h.conv = head_conv(m, L, W);
  h.rot.dims = (int)c.rot_dims;
  h.rot.freq = W.freq;
  h.rot.mult = W.rot_mult;
  h.eps = m->cfg.eps;
  h.q = m->q;
  h.ldq = m->q_ld;
  h.keys = L.k_cache;
  h.values = L.v_cache;
  h.pool = (int)c.pool;
  h.pool_rows = (int)L.pool_rows;
  h.pooled_keys = L.pooled_k;
  h.pooled_values = L.pooled_v;
  TQ_STEP(launch_conv_heads(ctx, h, b, dt));
  WindowAttn a;
  a.heads = (int)c.heads;
  a.kv_heads = (int)c.kv_heads;
  a.dim = (int)c.dim;
  a.vdim = (int)c.vdim;
  a.dim_pad = (int)L.key_pad;
  a.vdim_pad = (int)L.val_pad;
  a.window = (int)c.window;
  a.scale = c.scale;
  a.sink = -INFINITY;
  a.out_scale = c.left_scale;
  a.pool = (int)c.pool;
  a.pool_rows = (int)L.pool_rows;
  a.max_seq = (int)m->cfg.max_seq;
  a.pooled_keys = L.pooled_k;
  a.pooled_values = L.pooled_v;
  TQ_STEP(launch_window_attention(ctx, a, b, dt, m->q, m->q_ld, nullptr, 0, L.k_cache, L.v_cache, m->att, m->att_ld));
  MinGru g;
  g.width = (int)c.state_width;
  g.z_bias = W.z_bias;
  g.u_bias = W.x_bias;
  g.out_scale = c.right_scale;
  g.state = L.state;
  g.max_seq = (int)m->cfg.max_seq;
  MinGruRows r;
  r.z = mix + L.z0 * es;
  r.u = mix + L.u0 * es;
  r.gate = mix + L.g0 * es;
  r.ld = m->mix_ld;
  r.out = static_cast<char*>(m->att) + L.right0 * es;
  r.ldo = m->att_ld;
  TQ_STEP(launch_min_gru(ctx, g, r, b, dt));
  DenseInput att;
  att.x = m->att;
  att.ldx = m->att_ld;
  DenseEpilogue o;
  dense_section(o, W.w_out->rpad, m->cfg.width, DENSE_ROW, 1, m->y, m->cfg.width);
  return launch_dense(ctx, W.w_out, att, b.rows, o);
}

// Leaves its output to the stream kernel.
static int feed_forward(tq_sakinex* m, const Layer& W, size_t rows, StreamMix& mix) {
  const tq_sakinex_layer& c = W.c;
  ExpertFf f;
  f.front = W.front;
  f.gate_up = W.gate_up;
  f.down = W.down;
  f.shared_down = W.shared_down;
  f.logits = (size_t)c.experts + (c.shared_ff ? 1 : 0);
  f.logit_end = W.shared0;
  f.experts = c.experts;
  f.top = c.top;
  f.ff = c.ff;
  f.shared_ff = c.shared_ff;
  f.gu_rows = W.gu_rows;
  f.down_rows = W.down_rows;
  f.rule.score = ROUTE_SOFTMAX;
  f.rule.renorm = true;
  f.rule.bias = W.router_bias;
  f.glu = DENSE_GLU_SILU;
  ExpertBuffers b;
  b.logits = m->logits;
  b.ld_logits = m->max_experts + 1;
  b.route = m->route;
  b.gathered = m->gathered;
  b.act = m->act;
  b.act_ld = m->act_ld;
  b.shared = m->shared;
  b.shared_ld = m->shared_ld;
  b.y = m->yp;
  b.y_shared = m->ys;
  if (c.shared_ff) {
    mix.y_more_gate = m->logits + c.experts;
    mix.ld_gate = b.ld_logits;
  }
  return launch_expert_ff(m->ctx, f, b, m->hn, m->embed->kpad, rows, m->cfg.width, m->cfg.dtype, mix);
}

extern "C" int tq_sakinex_step(tq_sakinex* m, const int* token_ids_dev, size_t rows, const int* seq_rows_dev, const int* starts_dev, const int* slots_dev,
                               size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev, size_t n_logits, float* logits_dev) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  const tq_sakinex_config& c = m->cfg;
  TQ_REQUIRE(ctx, token_ids_dev && starts_dev && rows > 0 && n_seqs > 0, "tq_sakinex_step: null pointer or empty step");
  TQ_REQUIRE(ctx, rows < (1ull << 24), "tq_sakinex_step: too many rows");
  TQ_REQUIRE(ctx, seq_rows_dev || rows == n_seqs, "tq_sakinex_step: without row offsets every sequence brings one row");
  TQ_REQUIRE(ctx, max_q > 0 && max_q <= rows && (seq_rows_dev || max_q == 1), "tq_sakinex_step: max_q must bound the sequences' rows");
  TQ_REQUIRE(ctx, n_seqs <= c.max_slots && max_len > 0 && max_len <= c.max_seq, "tq_sakinex_step: at most %u sequences of %u positions", c.max_slots, c.max_seq);
  TQ_REQUIRE(ctx, n_logits == 0 || logits_dev, "tq_sakinex_step: null logits");
  TQ_REQUIRE(ctx, logit_rows_dev || n_logits == 0 || n_logits == rows, "tq_sakinex_step: without a row list every row has logits");
  TQ_REQUIRE(ctx, m->have == (bit(TQ_SX_EMBED) | bit(TQ_SX_FINAL_NORM) | bit(TQ_SX_HEAD)), "tq_sakinex_step: the embedding, the final norm or the head is missing");
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer& L = m->layers[i];
    bool all = L.src != i || L.have == needed(L);
    for (unsigned char e : L.have_expert) all = all && e == 7;
    TQ_REQUIRE(ctx, all, "tq_sakinex_step: layer %zu has tensors missing", i);
  }
  TQ_STEP(ensure_rows(m, rows));
  TQ_REQUIRE(ctx, n_logits <= m->ws_rows, "tq_sakinex_step: more logits than rows");
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
  const bool single = b.max_q == 1;
  const size_t hn_ld = m->embed->kpad;
  StreamMix s;
  s.src = m->x;
  s.dst = m->xs;
  s.mix = m->one;
  s.w_out = m->mult;
  s.out = m->hn;
  s.out_dtype = c.dtype;
  s.ld_out = hn_ld;
  s.eps = c.eps;
  // The stream kernel, and the convolved input of sublayer q of run `next` (null: none).
  auto pass = [&](StreamMix mix, const Layer* next, int q) -> int {
    if (!next) return launch_stream_mix(ctx, mix, rows, c.width);
    const Layer& W = m->layers[next->src];
    const ShortConv conv = canon(m, *next, W, q);
    mix.gain = W.norm[q];
    if (q == 0 && next->c.add_embedding) mix.inject = m->x;
    if (single) {
      mix.conv_w = conv.w;
      mix.conv_state = conv.state;
      mix.conv_taps = conv.taps;
      mix.max_seq = conv.max_seq;
      mix.row_pos = m->row_pos;
      mix.cache_row = m->cache_row;
      return launch_stream_mix(ctx, mix, rows, c.width);
    }
    mix.out = m->raw_hn[q];
    TQ_STEP(launch_stream_mix(ctx, mix, rows, c.width));
    return launch_conv_residual(ctx, conv, b, c.dtype, m->raw_hn[q], hn_ld, m->hn, hn_ld);
  };
  TQ_STEP(pass(s, &m->layers[0], 0));
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer &L = m->layers[i], &W = m->layers[L.src];
    const Layer* next = i + 1 < m->layers.size() ? &m->layers[i + 1] : nullptr;
    float* sum = m->trace ? m->trace + i * rows * c.width : nullptr;
    TQ_STEP(mixer(m, L, W, b));
    StreamMix mix = s;
    mix.y = m->y;
    s.src = m->xs;
    if (L.c.experts) {
      TQ_STEP(pass(mix, &L, 1));
      mix = s;
      TQ_STEP(feed_forward(m, W, rows, mix));
    }
    if (!single) {
      const ConvTail tails[] = {{canon(m, L, W, 0), m->raw_hn[0], hn_ld}, {head_conv(m, L, W), m->mix, m->mix_ld}, {canon(m, L, W, 1), m->raw_hn[1], hn_ld}};
      TQ_STEP(launch_conv_tails(ctx, tails, L.c.experts ? 3 : 2, b, c.dtype));
    }
    mix.sum = sum;
    TQ_STEP(pass(mix, next, 0));
  }
  if (n_logits) {
    s.dst = nullptr;
    s.src_rows = logit_rows_dev;
    s.gain = m->final_norm;
    TQ_STEP(launch_stream_mix(ctx, s, n_logits, c.width));
    DenseInput h;
    h.x = m->hn;
    h.ldx = hn_ld;
    DenseEpilogue e;
    dense_section(e, m->head->rpad, c.vocab, DENSE_ROW, 1, logits_dev, c.vocab);
    TQ_STEP(launch_dense(ctx, m->head, h, n_logits, e));
  }
  return TQ_OK;
}
#undef TQ_STEP
