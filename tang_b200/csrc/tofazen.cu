// Tofazen: a decoder with learned absolute positions, parallel layers (one norm feeds the mixer and the feed-forward),
// differential attention with a sliding window and kept first tokens, layers that read another layer's keys and values,
// and a clamped gated feed-forward (include/tangq.h, tq_tofazen_*).
//
// A layer is two dense products around the attention:
//   * `in`  [q | k | v | gate/up] x width: the layer's norm is its prologue (few rows) and its epilogue sends q to a
//     buffer, keys and values straight into their cache rows (nothing rotates them) and gate/up through the clamped GLU;
//   * `out` width x [heads * vdim | ff]: W_o and W_down side by side along k, since both results enter the stream with the
//     same factor; its operand is one buffer that the attention and the GLU fill, its epilogue adds to the f32 stream.
// A decode step is three kernels per layer (four when the attention splits its keys over CTAs).
// The step takes any mix of sequences: each brings its next rows, from one to a whole prompt, at its own position in its
// own cache slot.
#include <cuda_bf16.h>

#include <new>
#include <vector>

#include "dense.cuh"
#include "diff_attention.cuh"

using namespace tq;

namespace {

constexpr float kGluAlpha = 1.702f;

struct Layer {
  tq_tofazen_layer c;
  tq_dweight *w_in = nullptr, *w_out = nullptr;
  void* norm = nullptr;
  void *k_cache = nullptr, *v_cache = nullptr;     // null: another layer's
  size_t dim_pad = 0, vdim_pad = 0;
  size_t q_rows = 0, k_rows = 0, v_rows = 0;       // rows that exist
  size_t k0 = 0, v0 = 0, gu0 = 0;                  // first row of the sections of w_in
  unsigned have = 0;                               // bit per tensor put
};

size_t up16(size_t n) { return (n + 15) / 16 * 16; }
size_t up8(size_t n) { return (n + 7) / 8 * 8; }

}  // namespace

struct tq_tofazen {
  tq_ctx* ctx = nullptr;
  tq_tofazen_config cfg{};
  std::vector<Layer> layers;
  void *embed = nullptr, *pos = nullptr, *final_norm = nullptr;
  tq_dweight* head = nullptr;
  unsigned have = 0;
  size_t q_ld = 0, cat_ld = 0;
  size_t ws_rows = 0;
  float* x = nullptr;
  void *xn = nullptr, *q = nullptr, *cat = nullptr;
  int *row_pos = nullptr, *cache_row = nullptr;
  size_t last_rows = 0;
  float* trace = nullptr;
  std::vector<void*> owned;
};

static void release(tq_tofazen* m) {
  for (auto& L : m->layers) {
    if (L.w_in) tq_dweight_free(m->ctx, L.w_in);
    if (L.w_out) tq_dweight_free(m->ctx, L.w_out);
  }
  if (m->head) tq_dweight_free(m->ctx, m->head);
  for (void* p : {(void*)m->x, m->xn, m->q, m->cat, (void*)m->row_pos, (void*)m->cache_row})
    if (p) cudaFree(p);
  for (void* p : m->owned) cudaFree(p);
  delete m;
  cudaGetLastError();
}

static int zalloc(tq_tofazen* m, void** p, size_t bytes) {
  cudaError_t e = cudaMalloc(p, bytes);
  if (e == cudaErrorMemoryAllocation) {
    cudaGetLastError();
    return fail(m->ctx, TQ_ENOMEM, "tofazen: out of device memory (%zu bytes)", bytes);
  }
  TQ_CUDA(m->ctx, e);
  TQ_CUDA(m->ctx, cudaMemsetAsync(*p, 0, bytes, m->ctx->stream));
  return TQ_OK;
}

static int ensure_rows(tq_tofazen* m, size_t rows) {
  if (rows <= m->ws_rows) return TQ_OK;
  tq_ctx* ctx = m->ctx;
  TQ_REQUIRE(ctx, !ctx->capturing, "tq_tofazen_step: workspaces must be sized before graph capture (run once eagerly)");
  TQ_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  ctx->ws_generation++;   // graphs recorded over the old buffers must not be replayed
  const size_t es = dtype_size(m->cfg.dtype), want = rows < 64 ? 64 : rows;
  void** slots[] = {(void**)&m->x, &m->xn, &m->q, &m->cat, (void**)&m->row_pos, (void**)&m->cache_row};
  const size_t bytes[] = {want * m->cfg.width * 4, want * m->head->kpad * es, want * m->q_ld * es, want * m->cat_ld * es, want * 4, want * 4};
  m->ws_rows = 0;
  for (int i = 0; i < 6; ++i) {
    if (*slots[i]) cudaFree(*slots[i]);
    *slots[i] = nullptr;
    if (int st = zalloc(m, slots[i], bytes[i])) return st;
  }
  m->ws_rows = want;
  return TQ_OK;
}

extern "C" {

int tq_tofazen_create(tq_ctx* ctx, const tq_tofazen_config* cfg, const tq_tofazen_layer* layers, tq_tofazen** out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && layers && out, "tq_tofazen_create: null argument");
  *out = nullptr;
  TQ_REQUIRE(ctx, cfg->n_layers > 0 && cfg->width > 0 && cfg->width <= 8192 && cfg->vocab > 0, "tq_tofazen_create: width must be 1..8192, and there must be layers and a vocabulary");
  TQ_REQUIRE(ctx, cfg->dtype == TQ_BF16 || cfg->dtype == TQ_F32, "tq_tofazen_create: dtype must be bf16 or f32");
  TQ_REQUIRE(ctx, cfg->max_seq > 0 && cfg->max_seq <= cfg->max_positions && cfg->max_slots > 0, "tq_tofazen_create: max_seq must be 1..max_positions, max_slots at least 1");
  TQ_REQUIRE(ctx, (size_t)cfg->max_seq * cfg->max_slots < (1ull << 31), "tq_tofazen_create: cache too large");
  for (uint32_t i = 0; i < cfg->n_layers; ++i) {
    const tq_tofazen_layer& c = layers[i];
    TQ_REQUIRE(ctx, c.heads > 0 && c.kv_heads > 0 && c.heads % c.kv_heads == 0 && c.dim > 0 && c.vdim > 0,
               "tq_tofazen_create: layer %u: heads must be a multiple of kv_heads", i);
    TQ_REQUIRE(ctx, c.window > 0 && c.window <= 0x7fffffffu && c.keep_first <= 0x7fffffffu, "tq_tofazen_create: layer %u: bad window", i);
    if (c.kv_from >= 0) {
      TQ_REQUIRE(ctx, (uint32_t)c.kv_from < i && layers[c.kv_from].kv_from < 0, "tq_tofazen_create: layer %u: kv_from must name an earlier layer with keys of its own", i);
      const tq_tofazen_layer& s = layers[c.kv_from];
      TQ_REQUIRE(ctx, s.kv_heads == c.kv_heads && s.dim == c.dim && s.vdim == c.vdim, "tq_tofazen_create: layer %u: shape differs from layer %d, whose keys it reads", i, c.kv_from);
    }
  }
  tq_tofazen* m = new (std::nothrow) tq_tofazen();
  if (!m) return fail(ctx, TQ_ENOMEM, "out of host memory");
  m->ctx = ctx;
  m->cfg = *cfg;
  m->layers.resize(cfg->n_layers);
  const size_t es = dtype_size(cfg->dtype), tokens = (size_t)cfg->max_slots * cfg->max_seq;
  int st = TQ_OK;
  auto A = [&](void** p, size_t bytes) {
    if (st != TQ_OK) return;
    st = zalloc(m, p, bytes);
    if (st == TQ_OK) m->owned.push_back(*p);
  };
  A(&m->embed, (size_t)cfg->vocab * cfg->width * es);
  A(&m->pos, (size_t)cfg->max_positions * cfg->width * es);
  A(&m->final_norm, cfg->width * es);
  if (st == TQ_OK) st = tq_dweight_create(ctx, cfg->vocab, cfg->width, cfg->dtype, &m->head);
  for (uint32_t i = 0; i < cfg->n_layers && st == TQ_OK; ++i) {
    Layer& L = m->layers[i];
    L.c = layers[i];
    L.dim_pad = up8(L.c.dim);
    L.vdim_pad = up8(L.c.vdim);
    L.q_rows = (size_t)L.c.heads * 2 * L.c.dim;
    if (L.c.kv_from < 0) {
      L.k_rows = (size_t)L.c.kv_heads * 2 * L.c.dim;
      L.v_rows = (size_t)L.c.kv_heads * L.c.vdim;
      A(&L.k_cache, tokens * L.c.kv_heads * 2 * L.dim_pad * es);
      A(&L.v_cache, tokens * L.c.kv_heads * L.vdim_pad * es);
    }
    L.k0 = up16(L.q_rows);
    L.v0 = L.k0 + up16(L.k_rows);
    L.gu0 = L.v0 + up16(L.v_rows);
    const size_t in_rows = L.gu0 + 2 * up8(L.c.ff), cat = (size_t)L.c.heads * L.c.vdim + L.c.ff;
    A(&L.norm, cfg->width * es);
    if (st == TQ_OK) st = tq_dweight_create(ctx, in_rows, cfg->width, cfg->dtype, &L.w_in);
    if (st == TQ_OK) st = tq_dweight_create(ctx, cfg->width, cat, cfg->dtype, &L.w_out);
    if (st != TQ_OK) break;
    if (up8(L.q_rows) > m->q_ld) m->q_ld = up8(L.q_rows);
    if (L.w_out->kpad > m->cat_ld) m->cat_ld = L.w_out->kpad;
  }
  if (st != TQ_OK) {
    release(m);
    return st;
  }
  *out = m;
  return TQ_OK;
}

int tq_tofazen_destroy(tq_tofazen* m) {
  if (!m) return TQ_OK;
  bind(m->ctx);
  cudaStreamSynchronize(m->ctx->stream);
  release(m);
  return TQ_OK;
}

int tq_tofazen_put(tq_tofazen* m, int which, size_t layer, const void* src, int src_dtype, size_t rows, size_t cols) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src != nullptr && (src_dtype == TQ_BF16 || src_dtype == TQ_F32), "tq_tofazen_put: the source must be bf16 or f32");
  const size_t width = m->cfg.width;
  auto shape = [&](size_t r, size_t c) -> int {
    if (rows == r && cols == c) return TQ_OK;
    return fail(ctx, TQ_EINVAL, "tq_tofazen_put: tensor %d of layer %zu must be [%zu, %zu], got [%zu, %zu]", which, layer, r, c, rows, cols);
  };
  // a plain array: the embedding tables and the gains
  auto plain = [&](void* dst) -> int {
    const size_t n = rows * cols;
    if (src_dtype == m->cfg.dtype) {
      TQ_CUDA(ctx, cudaMemcpyAsync(dst, src, n * dtype_size(src_dtype), cudaMemcpyDefault, ctx->stream));
    } else {
      void* tmp = nullptr;
      TQ_CUDA(ctx, cudaMalloc(&tmp, n * dtype_size(src_dtype)));
      cudaError_t e = cudaMemcpyAsync(tmp, src, n * dtype_size(src_dtype), cudaMemcpyDefault, ctx->stream);
      int st = e == cudaSuccess ? tq_convert(ctx, tmp, src_dtype, dst, m->cfg.dtype, n) : fail(ctx, TQ_ECUDA, "tq_tofazen_put: %s", cudaGetErrorString(e));
      cudaStreamSynchronize(ctx->stream);
      cudaFree(tmp);
      if (st) return st;
    }
    TQ_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    return TQ_OK;
  };
  int st = TQ_OK;
  switch (which) {
    case TQ_TZ_EMBED:
      if ((st = shape(m->cfg.vocab, width)) == TQ_OK) st = plain(m->embed);
      break;
    case TQ_TZ_POS:
      if ((st = shape(m->cfg.max_positions, width)) == TQ_OK) st = plain(m->pos);
      break;
    case TQ_TZ_FINAL_NORM:
      if ((st = shape(1, width)) == TQ_OK) st = plain(m->final_norm);
      break;
    case TQ_TZ_HEAD:
      if ((st = shape(m->cfg.vocab, width)) == TQ_OK) st = tq_dweight_put(ctx, m->head, src, src_dtype, rows, cols, 0, 0, 0);
      break;
    default: {
      TQ_REQUIRE(ctx, which >= TQ_TZ_NORM && which <= TQ_TZ_DOWN, "tq_tofazen_put: unknown tensor %d", which);
      TQ_REQUIRE(ctx, layer < m->layers.size(), "tq_tofazen_put: layer %zu out of range", layer);
      Layer& L = m->layers[layer];
      const size_t o_cols = (size_t)L.c.heads * L.c.vdim, ff = L.c.ff;
      TQ_REQUIRE(ctx, !(which == TQ_TZ_K || which == TQ_TZ_V) || L.c.kv_from < 0, "tq_tofazen_put: layer %zu reads another layer's keys and values", layer);
      TQ_REQUIRE(ctx, !(which == TQ_TZ_GATE || which == TQ_TZ_UP || which == TQ_TZ_DOWN) || ff > 0, "tq_tofazen_put: layer %zu has no feed-forward", layer);
      if (which == TQ_TZ_NORM) {
        if ((st = shape(1, width)) == TQ_OK) st = plain(L.norm);
      } else if (which == TQ_TZ_Q) {
        if ((st = shape(L.q_rows, width)) == TQ_OK) st = tq_dweight_put(ctx, L.w_in, src, src_dtype, rows, cols, 0, 0, 0);
      } else if (which == TQ_TZ_K) {
        if ((st = shape(L.k_rows, width)) == TQ_OK) st = tq_dweight_put(ctx, L.w_in, src, src_dtype, rows, cols, L.k0, 0, 0);
      } else if (which == TQ_TZ_V) {
        if ((st = shape(L.v_rows, width)) == TQ_OK) st = tq_dweight_put(ctx, L.w_in, src, src_dtype, rows, cols, L.v0, 0, 0);
      } else if (which == TQ_TZ_O) {
        if ((st = shape(width, o_cols)) == TQ_OK) st = tq_dweight_put(ctx, L.w_out, src, src_dtype, rows, cols, 0, 0, 0);
      } else if (which == TQ_TZ_DOWN) {
        if ((st = shape(width, ff)) == TQ_OK) st = tq_dweight_put(ctx, L.w_out, src, src_dtype, rows, cols, 0, o_cols, 0);
      } else {
        if ((st = shape(ff, width)) == TQ_OK) st = tq_dweight_put(ctx, L.w_in, src, src_dtype, rows, cols, L.gu0, 0, which == TQ_TZ_GATE ? 1 : 2);
      }
      if (st == TQ_OK) L.have |= 1u << which;
      return st;
    }
  }
  if (st == TQ_OK) m->have |= 1u << which;
  return st;
}

int tq_tofazen_hidden(tq_tofazen* m, float** hidden_dev) {
  if (!m || !hidden_dev || !m->x) return TQ_EINVAL;
  *hidden_dev = m->x;
  return TQ_OK;
}

int tq_tofazen_trace(tq_tofazen* m, float* streams_dev_or_null) {
  if (!m) return TQ_EINVAL;
  m->trace = streams_dev_or_null;
  return TQ_OK;
}

int tq_tofazen_step(tq_tofazen* m, const int* token_ids_dev, size_t rows, const int* seq_rows_dev, const int* starts_dev, const int* slots_dev,
                    size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev, size_t n_logits, float* logits_dev) {
  if (!m) return TQ_EINVAL;
  tq_ctx* ctx = m->ctx;
  if (int st = bind(ctx)) return st;
  const tq_tofazen_config& c = m->cfg;
  TQ_REQUIRE(ctx, token_ids_dev && starts_dev && rows > 0 && n_seqs > 0, "tq_tofazen_step: null pointer or empty step");
  TQ_REQUIRE(ctx, rows < (1ull << 24), "tq_tofazen_step: too many rows");
  TQ_REQUIRE(ctx, seq_rows_dev || rows == n_seqs, "tq_tofazen_step: without row offsets every sequence brings one row");
  TQ_REQUIRE(ctx, max_q > 0 && max_q <= rows && (seq_rows_dev || max_q == 1), "tq_tofazen_step: max_q must bound the sequences' rows");
  TQ_REQUIRE(ctx, n_seqs <= c.max_slots && max_len > 0 && max_len <= c.max_seq, "tq_tofazen_step: at most %u sequences of %u positions", c.max_slots, c.max_seq);
  TQ_REQUIRE(ctx, n_logits == 0 || logits_dev, "tq_tofazen_step: null logits");
  TQ_REQUIRE(ctx, logit_rows_dev || n_logits == 0 || n_logits == rows, "tq_tofazen_step: without a row list every row has logits");
  const unsigned all = (1u << TQ_TZ_EMBED) | (1u << TQ_TZ_POS) | (1u << TQ_TZ_FINAL_NORM) | (1u << TQ_TZ_HEAD);
  TQ_REQUIRE(ctx, m->have == all, "tq_tofazen_step: an embedding, the final norm or the head is missing");
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer& L = m->layers[i];
    unsigned need = (1u << TQ_TZ_NORM) | (1u << TQ_TZ_Q) | (1u << TQ_TZ_O);
    if (L.c.kv_from < 0) need |= (1u << TQ_TZ_K) | (1u << TQ_TZ_V);
    if (L.c.ff) need |= (1u << TQ_TZ_GATE) | (1u << TQ_TZ_UP) | (1u << TQ_TZ_DOWN);
    TQ_REQUIRE(ctx, L.have == need, "tq_tofazen_step: layer %zu has tensors missing", i);
  }
  if (int st = ensure_rows(m, rows)) return st;
#define TQ_STEP(expr) \
  if (int st = (expr)) return st;
  TQ_STEP(launch_embedding_pos(ctx, m->embed, c.width, m->pos, c.dtype, token_ids_dev, seq_rows_dev, starts_dev, slots_dev, (int)n_seqs, rows, (int)c.width,
                               (int)c.vocab, (int)c.max_positions, (int)c.max_seq, (int)c.max_slots, m->x, m->row_pos, m->cache_row));
  const int f32 = c.dtype == TQ_F32;
  RaggedBatch batch;
  batch.n_seqs = (int)n_seqs;
  batch.rows = (int)rows;
  batch.max_q = (int)max_q;
  batch.max_len = (int)max_len;
  batch.seq_rows = seq_rows_dev;
  batch.row_pos = m->row_pos;
  batch.cache_row = m->cache_row;
  batch.cache_rows = (size_t)c.max_slots * c.max_seq;
  DenseInput normed;
  normed.h = m->x;
  normed.ldh = c.width;
  normed.gain_dtype = c.dtype;
  normed.eps = c.eps;
  normed.xn_tmp = m->xn;
  for (size_t i = 0; i < m->layers.size(); ++i) {
    const Layer& L = m->layers[i];
    const Layer& src = L.c.kv_from < 0 ? L : m->layers[L.c.kv_from];
    const size_t o_cols = (size_t)L.c.heads * L.c.vdim;
    const size_t cat_ld = L.w_out->kpad, es = dtype_size(c.dtype);
    DenseEpilogue e;
    auto section = [&](size_t end, size_t real, int kind, void* out, size_t ld) -> DenseSection& {
      DenseSection& s = e.s[e.n++];
      s.row_end = (int)end;
      s.rows = (int)real;
      s.kind = kind;
      s.f32 = f32;
      s.out = out;
      s.ld = (long long)ld;
      return s;
    };
    section(L.k0, L.q_rows, DENSE_ROW, m->q, m->q_ld);
    if (L.c.kv_from < 0) {
      DenseSection& k = section(L.v0, L.k_rows, DENSE_CACHE, L.k_cache, (size_t)L.c.kv_heads * 2 * L.dim_pad);
      k.inner = (int)L.c.dim;
      k.inner_pad = (int)L.dim_pad;
      DenseSection& v = section(L.gu0, L.v_rows, DENSE_CACHE, L.v_cache, (size_t)L.c.kv_heads * L.vdim_pad);
      v.inner = (int)L.c.vdim;
      v.inner_pad = (int)L.vdim_pad;
    }
    if (L.c.ff) section(L.w_in->rpad, L.c.ff, DENSE_GLU, static_cast<char*>(m->cat) + o_cols * es, cat_ld);
    e.cache_row = m->cache_row;
    e.glu_limit = L.c.limit;
    e.glu_alpha = kGluAlpha;
    normed.gain = L.norm;
    TQ_STEP(launch_dense(ctx, L.w_in, normed, rows, e));
    DiffAttn a;
    a.heads = (int)L.c.heads;
    a.kv_heads = (int)L.c.kv_heads;
    a.dim = (int)L.c.dim;
    a.vdim = (int)L.c.vdim;
    a.dim_pad = (int)src.dim_pad;
    a.vdim_pad = (int)src.vdim_pad;
    a.window = (int)L.c.window;
    a.keep_first = (int)L.c.keep_first;
    a.scale = L.c.scale;
    a.lambda = L.c.lambda;
    a.out_scale = L.c.out_scale;
    a.eps = c.eps;
    TQ_STEP(launch_diff_attention(ctx, a, batch, c.dtype, m->q, m->q_ld, src.k_cache, src.v_cache, m->cat, cat_ld));
    DenseEpilogue r;
    r.n = 1;
    r.s[0].row_end = (int)L.w_out->rpad;
    r.s[0].rows = (int)c.width;
    r.s[0].kind = DENSE_RESID;
    r.s[0].f32 = 1;
    r.s[0].ld = c.width;
    r.s[0].out = m->x;
    r.mult = c.residual_mult;
    DenseInput cat;
    cat.x = m->cat;
    cat.ldx = cat_ld;
    TQ_STEP(launch_dense(ctx, L.w_out, cat, rows, r));
    if (m->trace)
      TQ_CUDA(ctx, cudaMemcpyAsync(m->trace + i * rows * c.width, m->x, rows * c.width * sizeof(float), cudaMemcpyDeviceToDevice, ctx->stream));
  }
  if (n_logits) {
    DenseEpilogue h;
    h.n = 1;
    h.s[0].row_end = (int)m->head->rpad;
    h.s[0].rows = (int)c.vocab;
    h.s[0].f32 = 1;
    h.s[0].ld = c.vocab;
    h.s[0].out = logits_dev;
    normed.gain = m->final_norm;
    normed.h_rows = logit_rows_dev;
    TQ_STEP(launch_dense(ctx, m->head, normed, n_logits, h));
  }
#undef TQ_STEP
  return TQ_OK;
}

int tq_embedding_pos(tq_ctx* ctx, const void* table_dev, const void* pos_table_dev, int dtype, const int* ids_dev, const int* seq_rows_dev,
                     const int* starts_dev, const int* slots_dev, size_t n_seqs, size_t rows, size_t dim, size_t vocab, size_t n_pos,
                     size_t max_seq, size_t n_slots, float* out_dev, int* row_pos_dev, int* cache_row_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_BF16 || dtype == TQ_F32, "tq_embedding_pos: tables must be bf16 or f32");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, table_dev && pos_table_dev && ids_dev && starts_dev && out_dev && row_pos_dev && cache_row_dev && n_seqs > 0, "tq_embedding_pos: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || rows == n_seqs, "tq_embedding_pos: without row offsets every sequence brings one row");
  return launch_embedding_pos(ctx, table_dev, dim, pos_table_dev, dtype, ids_dev, seq_rows_dev, starts_dev, slots_dev, (int)n_seqs, rows, (int)dim,
                              (int)vocab, (int)n_pos, (int)max_seq, (int)n_slots, out_dev, row_pos_dev, cache_row_dev);
}

int tq_diff_attention(tq_ctx* ctx, const tq_diff_attn_config* cfg, int dtype, const void* q_dev, size_t ldq, const void* k_cache_dev,
                      const void* v_cache_dev, size_t cache_rows, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev,
                      size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && (dtype == TQ_BF16 || dtype == TQ_F32), "tq_diff_attention: dtype must be bf16 or f32");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, q_dev && k_cache_dev && v_cache_dev && row_pos_dev && cache_row_dev && out_dev, "tq_diff_attention: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || (rows == n_seqs && max_q == 1), "tq_diff_attention: without row offsets every sequence brings one row");
  DiffAttn a;
  a.heads = (int)cfg->heads;
  a.kv_heads = (int)cfg->kv_heads;
  a.dim = (int)cfg->dim;
  a.vdim = (int)cfg->vdim;
  a.dim_pad = (int)up8(cfg->dim);
  a.vdim_pad = (int)up8(cfg->vdim);
  a.window = (int)cfg->window;
  a.keep_first = (int)cfg->keep_first;
  a.scale = cfg->scale;
  a.lambda = cfg->lambda;
  a.out_scale = cfg->out_scale;
  a.eps = cfg->eps;
  RaggedBatch b;
  b.n_seqs = (int)n_seqs;
  b.rows = (int)rows;
  b.max_q = (int)max_q;
  b.max_len = (int)max_len;
  b.seq_rows = seq_rows_dev;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  return launch_diff_attention(ctx, a, b, dtype, q_dev, ldq, k_cache_dev, v_cache_dev, out_dev, ldo);
}

}  // extern "C"
