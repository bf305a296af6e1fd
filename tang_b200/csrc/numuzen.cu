// Numuzen: a decoder whose layers are sliding-window attention (whole-projection query/key norm, YaRN rotation, capped scores, a
// sink, an output gate, values that are the raw keys) or gated linear attention, each followed by sigmoid-routed experts, with a
// norm before and after every sublayer and tied embeddings (include/tangq.h, tq_numuzen_*).
//
// A layer is
//   * `in`: all projections of the mixer as one weight; its epilogue puts raw keys straight into the value cache;
//   * the mixer: norm + rotation and attention, or the recurrence (gates are applied in their last kernels);
//   * `out` -> f32, then one kernel for post-norm, stream update and the next norm;
//   * experts: router product, routing, grouped gate/up (weight and clamped GLU in the epilogue), grouped down, and the same
//     norm kernel, which also sums a row's experts.
// The step takes any mix of sequences: each brings its next rows, from one to a whole prompt, at its own position in its
// own slot (cache rows of the attention layers, state of the recurrent ones).
#include <cuda_bf16.h>

#include <new>
#include <vector>

#include "dense.cuh"
#include "expert_route.cuh"
#include "gla.cuh"
#include "ragged.h"
#include "rowops.cuh"
#include "window_attention.cuh"

using namespace tq;

namespace {

constexpr float kGluAlpha = 1.702f;

size_t up16(size_t n) { return (n + 15) / 16 * 16; }
size_t up8(size_t n) { return (n + 7) / 8 * 8; }

struct Layer {
  tq_numuzen_layer c;
  tq_dweight *w_in = nullptr, *w_out = nullptr;
  float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;   // one plus the stored weights
  size_t q_rows = 0, k_rows = 0, v_rows = 0, g_rows = 0;      // rows that exist (attention: no v)
  size_t k0 = 0, v0 = 0, g0 = 0, a0 = 0;                      // first row of the sections of w_in
  size_t kc = 0, vc = 0, gc = 0;                              // columns of the sections in the mixer's buffer
  // attention
  void *k_cache = nullptr, *v_cache = nullptr, *q_gain = nullptr, *k_gain = nullptr;
  size_t dim_pad = 0;
  float* freq = nullptr;
  float rot_mult = 1.f;
  // recurrent
  float *a2 = nullptr, *a2_bias = nullptr, *o_norm = nullptr, *state = nullptr;
  // experts
  tq_dweight *router = nullptr, *gate_up = nullptr, *down = nullptr;
  size_t gu_rows = 0, down_rows = 0;                          // rows of one expert in the stacked weights
  unsigned have = 0;                                          // bit per tensor put
  std::vector<unsigned char> have_expert;                     // bits gate, up, down
};

}  // namespace

struct tq_numuzen {
  tq_ctx* ctx = nullptr;
  tq_numuzen_config cfg{};
  std::vector<Layer> layers;
  tq_dweight* embed = nullptr;
  float* final_norm = nullptr;
  unsigned have = 0;
  size_t mix_ld = 0, att_ld = 0, act_ld = 0, rank_ld = 0, max_experts = 0, max_top = 0;
  size_t ws_rows = 0;
  float *x = nullptr, *y = nullptr, *a1 = nullptr, *logits = nullptr, *yp = nullptr;
  void *hn = nullptr, *mix = nullptr, *att = nullptr, *xs = nullptr, *act = nullptr;
  int *row_pos = nullptr, *cache_row = nullptr;
  Routing route;
  float* trace = nullptr;
  std::vector<void*> owned;
};

static std::vector<void**> workspaces(tq_numuzen* m) {
  return {(void**)&m->x, (void**)&m->y, (void**)&m->a1, (void**)&m->logits, (void**)&m->yp, &m->hn, &m->mix, &m->att, &m->xs, &m->act,
          (void**)&m->row_pos, (void**)&m->cache_row, (void**)&m->route.expert, (void**)&m->route.weight, (void**)&m->route.rank, (void**)&m->route.slot,
          (void**)&m->route.slot_row, (void**)&m->route.slot_weight, (void**)&m->route.jobs};
}

static void release(tq_numuzen* m) {
  for (auto& L : m->layers)
    for (tq_dweight* w : {L.w_in, L.w_out, L.router, L.gate_up, L.down})
      if (w) tq_dweight_free(m->ctx, w);
  if (m->embed) tq_dweight_free(m->ctx, m->embed);
  for (void** p : workspaces(m))
    if (*p) cudaFree(*p);
  for (void* p : m->owned) cudaFree(p);
  delete m;
  cudaGetLastError();
}

static int zalloc(tq_numuzen* m, void** p, size_t bytes) {
  cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
  if (e == cudaErrorMemoryAllocation) {
    cudaGetLastError();
    return fail(m->ctx, TQ_ENOMEM, "numuzen: out of device memory (%zu bytes)", bytes);
  }
  TQ_CUDA(m->ctx, e);
  TQ_CUDA(m->ctx, cudaMemsetAsync(*p, 0, bytes, m->ctx->stream));
  return TQ_OK;
}

static int ensure_rows(tq_numuzen* m, size_t rows) {
  if (rows <= m->ws_rows) return TQ_OK;
  tq_ctx* ctx = m->ctx;
  TQ_REQUIRE(ctx, !ctx->capturing, "tq_numuzen_step: workspaces must be sized before graph capture (run once eagerly)");
  TQ_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  ctx->ws_generation++;   // graphs recorded over the old buffers must not be replayed
  const size_t es = dtype_size(m->cfg.dtype), n = rows < 64 ? 64 : rows, pairs = n * m->max_top, width = m->cfg.width;
  const size_t bytes[] = {n * width * 4, n * width * 4, n * m->rank_ld * 4, n * m->max_experts * 4, pairs * width * 4, n * m->embed->kpad * es,
                          n * m->mix_ld * es, n * m->att_ld * es, m->max_top ? pairs * m->embed->kpad * es : 0, pairs * m->act_ld * es, n * 4, n * 4,
                          pairs * 4, pairs * 4, pairs * 4, pairs * 4, pairs * 4, pairs * 4, (pairs + m->max_experts) * sizeof(int4)};
  m->ws_rows = 0;
  const auto slots = workspaces(m);
  for (size_t i = 0; i < slots.size(); ++i) {
    if (*slots[i]) cudaFree(*slots[i]);
    *slots[i] = nullptr;
    if (int st = zalloc(m, slots[i], bytes[i])) return st;
  }
  m->ws_rows = n;
  return TQ_OK;
}

static unsigned needed(const Layer& L) {
  auto bit = [](int t) { return 1u << t; };
  unsigned n = bit(TQ_NZ_NORM1) | bit(TQ_NZ_NORM1B) | bit(TQ_NZ_Q) | bit(TQ_NZ_K) | bit(TQ_NZ_G) | bit(TQ_NZ_O);
  if (L.c.kind == TQ_NZ_ATTENTION) n |= bit(TQ_NZ_Q_NORM) | bit(TQ_NZ_K_NORM);
  else n |= bit(TQ_NZ_V) | bit(TQ_NZ_A1) | bit(TQ_NZ_A2) | bit(TQ_NZ_A2_BIAS) | bit(TQ_NZ_O_NORM);
  if (L.c.experts) n |= bit(TQ_NZ_NORM2) | bit(TQ_NZ_NORM2B) | bit(TQ_NZ_ROUTER);
  return n;
}

extern "C" {

int tq_numuzen_create(tq_ctx* ctx, const tq_numuzen_config* cfg, const tq_numuzen_layer* layers, tq_numuzen** out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && layers && out, "tq_numuzen_create: null argument");
  *out = nullptr;
  TQ_REQUIRE(ctx, cfg->n_layers > 0 && cfg->width > 0 && cfg->width <= 8192 && cfg->vocab > 0, "tq_numuzen_create: width must be 1..8192, and there must be layers and a vocabulary");
  TQ_REQUIRE(ctx, cfg->dtype == TQ_BF16 || cfg->dtype == TQ_F32, "tq_numuzen_create: dtype must be bf16 or f32");
  TQ_REQUIRE(ctx, cfg->max_seq > 0 && cfg->max_slots > 0 && (size_t)cfg->max_seq * cfg->max_slots < (1ull << 31), "tq_numuzen_create: cache empty or too large");
  for (uint32_t i = 0; i < cfg->n_layers; ++i) {
    const tq_numuzen_layer& c = layers[i];
    TQ_REQUIRE(ctx, c.heads > 0 && c.dim > 0, "tq_numuzen_create: layer %u: bad head sizes", i);
    if (c.kind == TQ_NZ_ATTENTION) {
      TQ_REQUIRE(ctx, c.kv_heads > 0 && c.heads % c.kv_heads == 0, "tq_numuzen_create: layer %u: heads must be a multiple of kv_heads", i);
      TQ_REQUIRE(ctx, c.vdim == c.dim, "tq_numuzen_create: layer %u: the values are the keys, so their sizes agree", i);
      TQ_REQUIRE(ctx, c.window > 0 && c.window <= 0x7fffffffu, "tq_numuzen_create: layer %u: bad window", i);
      TQ_REQUIRE(ctx, c.rot_dims % 2 == 0 && c.rot_dims <= c.dim && (c.rot_dims == 0 || c.rot_base > 1.0), "tq_numuzen_create: layer %u: bad rotation", i);
      TQ_REQUIRE(ctx, !(c.rot_factor > 0) || (c.rot_original > 0 && c.rot_fast > 0 && c.rot_slow > 0), "tq_numuzen_create: layer %u: bad rotation scaling", i);
      TQ_REQUIRE(ctx, c.softcap >= 0.f, "tq_numuzen_create: layer %u: bad score cap", i);
    } else {
      TQ_REQUIRE(ctx, c.kind == TQ_NZ_GLA, "tq_numuzen_create: layer %u: unknown mixer %u", i, c.kind);
      TQ_REQUIRE(ctx, c.vdim > 0 && c.rank > 0 && c.tau > 0.f, "tq_numuzen_create: layer %u: bad recurrent mixer", i);
    }
    TQ_REQUIRE(ctx, c.experts == 0 || (c.experts <= 1024 && c.top > 0 && c.top <= c.experts && c.top <= 64 && c.ff > 0), "tq_numuzen_create: layer %u: bad experts", i);
  }
  tq_numuzen* m = new (std::nothrow) tq_numuzen();
  if (!m) return fail(ctx, TQ_ENOMEM, "out of host memory");
  m->ctx = ctx;
  m->cfg = *cfg;
  m->layers.resize(cfg->n_layers);
  const size_t es = dtype_size(cfg->dtype), tokens = (size_t)cfg->max_slots * cfg->max_seq, width = cfg->width;
  int st = TQ_OK;
  auto A = [&](auto** p, size_t bytes) {
    if (st != TQ_OK) return;
    st = zalloc(m, (void**)p, bytes);
    if (st == TQ_OK) m->owned.push_back(*p);
  };
  auto W = [&](size_t rows, size_t cols, tq_dweight** w) {
    if (st == TQ_OK) st = tq_dweight_create(ctx, rows, cols, cfg->dtype, w);
  };
  auto most = [](size_t& a, size_t b) { a = a > b ? a : b; };
  A(&m->final_norm, width * 4);
  W(cfg->vocab, width, &m->embed);
  for (uint32_t i = 0; i < cfg->n_layers && st == TQ_OK; ++i) {
    Layer& L = m->layers[i];
    L.c = layers[i];
    const tq_numuzen_layer& c = L.c;
    for (float** g : {&L.norm1, &L.norm1b, &L.norm2, &L.norm2b}) A(g, width * 4);
    L.q_rows = (size_t)c.heads * c.dim;
    size_t in_rows;
    if (c.kind == TQ_NZ_ATTENTION) {
      L.k_rows = (size_t)c.kv_heads * c.dim;
      L.g_rows = L.q_rows;
      L.k0 = up16(L.q_rows);
      L.g0 = L.k0 + up16(L.k_rows);
      in_rows = L.g0 + L.g_rows;
      L.gc = up8(L.q_rows);
      L.dim_pad = up8(c.dim);
      A(&L.k_cache, tokens * c.kv_heads * L.dim_pad * es);
      A(&L.v_cache, tokens * c.kv_heads * L.dim_pad * es);
      A(&L.q_gain, L.q_rows * es);
      A(&L.k_gain, L.k_rows * es);
      A(&L.freq, (c.rot_dims / 2) * 4);
      if (st == TQ_OK && c.rot_dims) {
        std::vector<float> f(c.rot_dims / 2);
        yarn_frequencies((int)c.rot_dims, c.rot_base, c.rot_factor, c.rot_original, c.rot_fast, c.rot_slow, f.data(), &L.rot_mult);
        if (cudaMemcpyAsync(L.freq, f.data(), f.size() * 4, cudaMemcpyHostToDevice, ctx->stream) != cudaSuccess || cudaStreamSynchronize(ctx->stream) != cudaSuccess)
          st = fail(ctx, TQ_ECUDA, "tq_numuzen_create: copying the frequencies failed");
      }
    } else {
      L.k_rows = L.q_rows;
      L.v_rows = L.g_rows = (size_t)c.heads * c.vdim;
      L.k0 = up16(L.q_rows);
      L.v0 = L.k0 + up16(L.k_rows);
      L.g0 = L.v0 + up16(L.v_rows);
      L.a0 = L.g0 + up16(L.g_rows);
      in_rows = L.a0 + c.rank;
      L.kc = up8(L.q_rows);
      L.vc = L.kc + up8(L.k_rows);
      L.gc = L.vc + up8(L.v_rows);
      A(&L.a2, L.q_rows * c.rank * 4);
      A(&L.a2_bias, L.q_rows * 4);
      A(&L.o_norm, (size_t)c.vdim * 4);
      A(&L.state, (size_t)cfg->max_slots * c.heads * c.dim * c.vdim * 4);
      most(m->rank_ld, c.rank);
    }
    most(m->mix_ld, L.gc + up8(L.g_rows));
    W(in_rows, width, &L.w_in);
    W(width, (size_t)c.heads * c.vdim, &L.w_out);
    if (c.experts) {
      L.gu_rows = 2 * up8(c.ff);
      L.down_rows = up16(width);
      L.have_expert.assign(c.experts, 0);
      W(c.experts, width, &L.router);
      W(c.experts * L.gu_rows, width, &L.gate_up);
      W(c.experts * L.down_rows, c.ff, &L.down);
      most(m->max_experts, c.experts);
      most(m->max_top, c.top);
      if (st == TQ_OK) most(m->act_ld, L.down->kpad);
    }
    if (st == TQ_OK) most(m->att_ld, L.w_out->kpad);
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

int tq_numuzen_destroy(tq_numuzen* m) {
  if (!m) return TQ_OK;
  bind(m->ctx);
  cudaStreamSynchronize(m->ctx->stream);
  release(m);
  return TQ_OK;
}

int tq_numuzen_put(tq_numuzen* m, int which, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src != nullptr && (src_dtype == TQ_BF16 || src_dtype == TQ_F32), "tq_numuzen_put: the source must be bf16 or f32");
  TQ_REQUIRE(ctx, which >= TQ_NZ_EMBED && which <= TQ_NZ_DOWN, "tq_numuzen_put: unknown tensor %d", which);
  const size_t width = m->cfg.width;
  const int dt = m->cfg.dtype;
  int st = TQ_OK;
  auto shape = [&](size_t r, size_t c) -> bool {
    if (rows == r && cols == c) return true;
    st = fail(ctx, TQ_EINVAL, "tq_numuzen_put: tensor %d of layer %zu must be [%zu, %zu], got [%zu, %zu]", which, layer, r, c, rows, cols);
    return false;
  };
  auto vec = [&](size_t n, void* dst, int dst_dtype, float add) {
    if (shape(1, n)) st = put_vector(ctx, src, src_dtype, dst, dst_dtype, n, add);
  };
  auto mat = [&](size_t r, size_t c, tq_dweight* w, size_t row0, int interleave = 0) {
    if (shape(r, c)) st = tq_dweight_put(ctx, w, src, src_dtype, r, c, row0, 0, interleave);
  };
  if (which == TQ_NZ_EMBED || which == TQ_NZ_FINAL_NORM) {
    if (which == TQ_NZ_EMBED) mat(m->cfg.vocab, width, m->embed, 0);
    else vec(width, m->final_norm, TQ_F32, 1.f);
    if (st == TQ_OK) m->have |= 1u << which;
    return st;
  }
  TQ_REQUIRE(ctx, layer < m->layers.size(), "tq_numuzen_put: layer %zu out of range", layer);
  Layer& L = m->layers[layer];
  const tq_numuzen_layer& c = L.c;
  if (which == TQ_NZ_GATE || which == TQ_NZ_UP || which == TQ_NZ_DOWN) {
    TQ_REQUIRE(ctx, expert < c.experts, "tq_numuzen_put: layer %zu has %u experts", layer, c.experts);
    if (which == TQ_NZ_DOWN) mat(width, c.ff, L.down, expert * L.down_rows);
    else mat(c.ff, width, L.gate_up, expert * L.gu_rows, which == TQ_NZ_GATE ? 1 : 2);
    if (st == TQ_OK) L.have_expert[expert] |= 1u << (which - TQ_NZ_GATE);
    return st;
  }
  TQ_REQUIRE(ctx, (needed(L) >> which) & 1u, "tq_numuzen_put: layer %zu has no tensor %d", layer, which);
  switch (which) {
    case TQ_NZ_NORM1: vec(width, L.norm1, TQ_F32, 1.f); break;
    case TQ_NZ_NORM1B: vec(width, L.norm1b, TQ_F32, 1.f); break;
    case TQ_NZ_NORM2: vec(width, L.norm2, TQ_F32, 1.f); break;
    case TQ_NZ_NORM2B: vec(width, L.norm2b, TQ_F32, 1.f); break;
    case TQ_NZ_Q: mat(L.q_rows, width, L.w_in, 0); break;
    case TQ_NZ_K: mat(L.k_rows, width, L.w_in, L.k0); break;
    case TQ_NZ_V: mat(L.v_rows, width, L.w_in, L.v0); break;
    case TQ_NZ_G: mat(L.g_rows, width, L.w_in, L.g0); break;
    case TQ_NZ_O: mat(width, (size_t)c.heads * c.vdim, L.w_out, 0); break;
    case TQ_NZ_Q_NORM: vec(L.q_rows, L.q_gain, dt, 0.f); break;
    case TQ_NZ_K_NORM: vec(L.k_rows, L.k_gain, dt, 0.f); break;
    case TQ_NZ_O_NORM: vec(c.vdim, L.o_norm, TQ_F32, 0.f); break;
    case TQ_NZ_A1: mat(c.rank, width, L.w_in, L.a0); break;
    case TQ_NZ_A2:
      if (shape(L.q_rows, c.rank)) st = put_vector(ctx, src, src_dtype, L.a2, TQ_F32, rows * cols, 0.f);
      break;
    case TQ_NZ_A2_BIAS: vec(L.q_rows, L.a2_bias, TQ_F32, 0.f); break;
    default: mat(c.experts, width, L.router, 0); break;
  }
  if (st == TQ_OK) L.have |= 1u << which;
  return st;
}

int tq_numuzen_hidden(tq_numuzen* m, float** hidden_dev) {
  if (!m || !hidden_dev || !m->x) return TQ_EINVAL;
  *hidden_dev = m->x;
  return TQ_OK;
}

int tq_numuzen_trace(tq_numuzen* m, float* streams_dev_or_null) {
  if (!m) return TQ_EINVAL;
  m->trace = streams_dev_or_null;
  return TQ_OK;
}

}  // extern "C"

#define TQ_STEP(expr) \
  if (int st = (expr)) return st;

static int attention_layer(tq_numuzen* m, const Layer& L, const RaggedBatch& b) {
  tq_ctx* ctx = m->ctx;
  const tq_numuzen_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt);
  char* mix = static_cast<char*>(m->mix);
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, L.k0, L.q_rows, DENSE_ROW, f32, mix, m->mix_ld);
  DenseSection& k = dense_section(e, L.g0, L.k_rows, DENSE_CACHE, f32, L.v_cache, (size_t)c.kv_heads * L.dim_pad);
  k.inner = (int)c.dim;
  k.inner_pad = (int)L.dim_pad;
  dense_section(e, L.w_in->rpad, L.g_rows, DENSE_ROW, f32, mix + L.gc * es, m->mix_ld);
  e.cache_row = m->cache_row;
  TQ_STEP(launch_dense(ctx, L.w_in, in, b.rows, e));
  QkNormRope n;
  n.heads = (int)c.heads;
  n.kv_heads = (int)c.kv_heads;
  n.dim = (int)c.dim;
  n.raw_pad = n.key_pad = (int)L.dim_pad;
  n.q = mix;
  n.ldq = m->mix_ld;
  n.raw = L.v_cache;
  n.keys = L.k_cache;
  n.q_gain = L.q_gain;
  n.k_gain = L.k_gain;
  n.rot.dims = (int)c.rot_dims;
  n.rot.freq = L.freq;
  n.rot.mult = L.rot_mult;
  n.eps = m->cfg.eps;
  TQ_STEP(launch_qk_norm_rope(ctx, n, b, dt));
  WindowAttn a;
  a.heads = (int)c.heads;
  a.kv_heads = (int)c.kv_heads;
  a.dim = a.vdim = (int)c.dim;
  a.dim_pad = a.vdim_pad = (int)L.dim_pad;
  a.window = (int)c.window;
  a.scale = c.scale;
  a.softcap = c.softcap;
  a.sink = 0.f;
  return launch_window_attention(ctx, a, b, dt, mix, m->mix_ld, mix + L.gc * es, m->mix_ld, L.k_cache, L.v_cache, m->att, m->att_ld);
}

static int gla_layer(tq_numuzen* m, const Layer& L, const RaggedBatch& b) {
  const tq_numuzen_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt);
  char* mix = static_cast<char*>(m->mix);
  DenseInput in;
  in.x = m->hn;
  in.ldx = m->embed->kpad;
  DenseEpilogue e;
  dense_section(e, L.k0, L.q_rows, DENSE_ROW, f32, mix, m->mix_ld);
  dense_section(e, L.v0, L.k_rows, DENSE_ROW, f32, mix + L.kc * es, m->mix_ld);
  dense_section(e, L.g0, L.v_rows, DENSE_ROW, f32, mix + L.vc * es, m->mix_ld);
  dense_section(e, L.a0, L.g_rows, DENSE_ROW, f32, mix + L.gc * es, m->mix_ld);
  dense_section(e, L.w_in->rpad, c.rank, DENSE_ROW, 1, m->a1, m->rank_ld);
  TQ_STEP(launch_dense(m->ctx, L.w_in, in, b.rows, e));
  Gla g;
  g.heads = (int)c.heads;
  g.dim = (int)c.dim;
  g.vdim = (int)c.vdim;
  g.rank = (int)c.rank;
  g.tau = c.tau;
  g.q_scale = c.scale;
  g.eps = m->cfg.eps;
  g.a2 = L.a2;
  g.a2_bias = L.a2_bias;
  g.norm = L.o_norm;
  g.state = L.state;
  g.max_seq = (int)m->cfg.max_seq;
  GlaRows r;
  r.q = mix;
  r.k = mix + L.kc * es;
  r.v = mix + L.vc * es;
  r.gate = mix + L.gc * es;
  r.ld = m->mix_ld;
  r.a1 = m->a1;
  r.ld_a1 = m->rank_ld;
  r.out = m->att;
  r.ldo = m->att_ld;
  return launch_gla(m->ctx, g, r, b, dt);
}

static int expert_layer(tq_numuzen* m, const Layer& L, size_t rows) {
  tq_ctx* ctx = m->ctx;
  const tq_numuzen_layer& c = L.c;
  const int dt = m->cfg.dtype, f32 = dt == TQ_F32;
  const size_t es = dtype_size(dt), pairs = rows * c.top, width = m->cfg.width, hn_ld = m->embed->kpad;
  DenseInput in;
  in.x = m->hn;
  in.ldx = hn_ld;
  DenseEpilogue z;
  dense_section(z, L.router->rpad, c.experts, DENSE_ROW, 1, m->logits, m->max_experts);
  TQ_STEP(launch_dense(ctx, L.router, in, rows, z));
  DenseGroups g;
  g.jobs = m->route.jobs;
  g.n_jobs = m->route.n_jobs;
  g.chunk = dense_group_chunk(dt, L.gate_up->kpad > L.down->kpad ? L.gate_up->kpad : L.down->kpad, pairs, c.experts);
  g.max_jobs = (int)route_max_jobs(pairs, c.experts, g.chunk);
  // the tcgen05 kernel copies boxes of consecutive rows, the others follow the slots' row numbers
  const bool gather = !f32 && g.chunk > 8;
  TQ_STEP(launch_route(ctx, m->logits, m->max_experts, rows, c.experts, c.top, RouteRule(), g.chunk, m->route, m->hn, hn_ld * es, up8(width) * es,
                       gather ? m->xs : nullptr, hn_ld * es));
  DenseEpilogue u;
  dense_section(u, L.gu_rows, c.ff, DENSE_GLU, f32, m->act, m->act_ld);
  u.glu_limit = c.limit;
  u.glu_alpha = kGluAlpha;
  u.row_scale = m->route.slot_weight;
  g.group_rows = L.gu_rows;
  g.x_rows = gather ? nullptr : m->route.slot_row;
  TQ_STEP(launch_dense_grouped(ctx, L.gate_up, gather ? m->xs : m->hn, hn_ld, pairs, g, u));
  DenseEpilogue d;
  dense_section(d, L.down_rows, width, DENSE_ROW, 1, m->yp, width);
  g.group_rows = L.down_rows;
  g.x_rows = nullptr;
  return launch_dense_grouped(ctx, L.down, m->act, m->act_ld, pairs, g, d);
}

extern "C" int tq_numuzen_step(tq_numuzen* m, const int* token_ids_dev, size_t rows, const int* seq_rows_dev, const int* starts_dev, const int* slots_dev,
                               size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev, size_t n_logits, float* logits_dev) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  const tq_numuzen_config& c = m->cfg;
  TQ_REQUIRE(ctx, token_ids_dev && starts_dev && rows > 0 && n_seqs > 0, "tq_numuzen_step: null pointer or empty step");
  TQ_REQUIRE(ctx, rows < (1ull << 24), "tq_numuzen_step: too many rows");
  TQ_REQUIRE(ctx, seq_rows_dev || rows == n_seqs, "tq_numuzen_step: without row offsets every sequence brings one row");
  TQ_REQUIRE(ctx, max_q > 0 && max_q <= rows && (seq_rows_dev || max_q == 1), "tq_numuzen_step: max_q must bound the sequences' rows");
  TQ_REQUIRE(ctx, n_seqs <= c.max_slots && max_len > 0 && max_len <= c.max_seq, "tq_numuzen_step: at most %u sequences of %u positions", c.max_slots, c.max_seq);
  TQ_REQUIRE(ctx, n_logits == 0 || logits_dev, "tq_numuzen_step: null logits");
  TQ_REQUIRE(ctx, logit_rows_dev || n_logits == 0 || n_logits == rows, "tq_numuzen_step: without a row list every row has logits");
  TQ_REQUIRE(ctx, m->have == ((1u << TQ_NZ_EMBED) | (1u << TQ_NZ_FINAL_NORM)), "tq_numuzen_step: the embedding or the final norm is missing");
  for (size_t i = 0; i < m->layers.size(); ++i) {
    bool all = m->layers[i].have == needed(m->layers[i]);
    for (unsigned char e : m->layers[i].have_expert) all = all && e == 7;
    TQ_REQUIRE(ctx, all, "tq_numuzen_step: layer %zu has tensors missing", i);
  }
  TQ_STEP(ensure_rows(m, rows));
  TQ_REQUIRE(ctx, n_logits <= m->ws_rows, "tq_numuzen_step: more logits than rows");
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
  AddNorm n;
  n.x = m->x;
  n.out = m->hn;
  n.out_dtype = c.dtype;
  n.ld_out = m->embed->kpad;
  n.eps = c.eps;
  n.gain_next = m->layers[0].norm1;
  TQ_STEP(launch_add_norm(ctx, n, rows, c.width));
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer& L = m->layers[i];
    const float* next = i + 1 < m->layers.size() ? m->layers[i + 1].norm1 : nullptr;
    TQ_STEP(L.c.kind == TQ_NZ_ATTENTION ? attention_layer(m, L, b) : gla_layer(m, L, b));
    DenseInput att;
    att.x = m->att;
    att.ldx = m->att_ld;
    DenseEpilogue o;
    dense_section(o, L.w_out->rpad, c.width, DENSE_ROW, 1, m->y, c.width);
    TQ_STEP(launch_dense(ctx, L.w_out, att, rows, o));
    n.y = m->y;
    n.y_rows = nullptr;
    n.n_y = 1;
    n.gain_post = L.norm1b;
    n.gain_next = L.c.experts ? L.norm2 : next;
    TQ_STEP(launch_add_norm(ctx, n, rows, c.width));
    if (L.c.experts) {
      TQ_STEP(expert_layer(m, L, rows));
      n.y = m->yp;
      n.y_rows = m->route.slot;
      n.n_y = (int)L.c.top;
      n.gain_post = L.norm2b;
      n.gain_next = next;
      TQ_STEP(launch_add_norm(ctx, n, rows, c.width));
    }
    if (m->trace)
      TQ_CUDA(ctx, cudaMemcpyAsync(m->trace + i * rows * c.width, m->x, rows * c.width * sizeof(float), cudaMemcpyDeviceToDevice, ctx->stream));
  }
  if (n_logits) {
    DenseInput h;
    h.h = m->x;
    h.ldh = c.width;
    h.h_rows = logit_rows_dev;
    h.gain = m->final_norm;
    h.gain_dtype = TQ_F32;
    h.eps = c.eps;
    h.xn_tmp = m->hn;
    DenseEpilogue e;
    dense_section(e, m->embed->rpad, c.vocab, DENSE_ROW, 1, logits_dev, c.vocab);
    TQ_STEP(launch_dense(ctx, m->embed, h, n_logits, e));
  }
  return TQ_OK;
}
#undef TQ_STEP
