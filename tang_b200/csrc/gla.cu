// Gated linear attention (see gla.cuh).
//
//   * gla_decode_kernel: one row per sequence.  A cluster of CTAs shares a head's state by value columns, streams it through
//     registers once and exchanges the sums of squares of the head norm through distributed shared memory;
//   * gla_scan_kernel + gla_out_kernel: any number of rows, token by token, the state in shared memory: the exact f32 form;
//   * prompts in bf16: csrc/gla_chunk.cu.
// Lightning attention runs through the first two, which then leave f32 outputs for launch_norm_gate; prompts: csrc/lightning.cu.
#include "gla.cuh"

#include <cooperative_groups.h>
#include <cuda_bf16.h>

#include "common.cuh"
#include "gla_device.cuh"
#include "rowops.cuh"

namespace tq {

namespace cg = cooperative_groups;

// ------------------------------------------------------------------------------------------------ one row per sequence
constexpr int kGdThreads = 256;
constexpr int kGdWarps = kGdThreads / 32;

// blockIdx.x: head * splits + part (a cluster is one head's parts); part owns vdim / splits columns.
template <typename T>
__global__ void __launch_bounds__(kGdThreads) gla_decode_kernel(Gla g, GlaRows r, RaggedBatch b, int splits, float* o_out) {
  extern __shared__ float gd_smem[];
  __shared__ float sums[2];
  const int cw = g.vdim / splits;
  float* alpha = gd_smem;                 // [dim]
  float* ks = alpha + g.dim;
  float* qs = ks + g.dim;
  float* part = qs + g.dim;               // [warps][cw]
  __shared__ float red[kGdWarps];
  const int head = blockIdx.x / splits, c0 = (blockIdx.x % splits) * cw;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  const bool ok = gl_sequence(g, b, blockIdx.y, s);
  const T* base_v = nullptr;
  if (ok) {
    const size_t row = s.row0;
    base_v = static_cast<const T*>(r.v) + row * r.ld + (size_t)head * g.vdim + c0;
    for (int d = threadIdx.x; d < g.dim; d += kGdThreads) {
      const int ch = head * g.dim + d;
      alpha[d] = s.fresh ? 0.f : gl_decay(g, head, ch, r.a1 + row * r.ld_a1);
      ks[d] = gl_load(static_cast<const T*>(r.k) + row * r.ld + ch);
      qs[d] = gl_load(static_cast<const T*>(r.q) + row * r.ld + ch) * g.q_scale;
    }
  }
  __syncthreads();
  float sq = 0.f;
  if (ok) {
    float* S = g.state + ((s.slot * g.heads + head) * g.dim) * g.vdim + c0;
    for (int cb = lane; cb < cw; cb += 32) {
      const float v = gl_load(base_v + cb);
      float acc = 0.f;
      float* col = S + cb;
      int d = warp;
      if (!s.fresh) {
        for (; d + 7 * kGdWarps < g.dim; d += 8 * kGdWarps) {
          float st[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) st[i] = __ldcs(col + (size_t)(d + i * kGdWarps) * g.vdim);
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int dd = d + i * kGdWarps;
            st[i] = fmaf(alpha[dd], st[i], ks[dd] * v);
            acc = fmaf(qs[dd], st[i], acc);
            __stcs(col + (size_t)dd * g.vdim, st[i]);
          }
        }
      }
      for (; d < g.dim; d += kGdWarps) {
        // (a fresh state is not read: what the slot held before may be anything)
        const float x = (s.fresh ? 0.f : alpha[d] * col[(size_t)d * g.vdim]) + ks[d] * v;
        acc = fmaf(qs[d], x, acc);
        col[(size_t)d * g.vdim] = x;
      }
      part[warp * cw + cb] = acc;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < cw; c += kGdThreads) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kGdWarps; ++w) o += part[w * cw + c];
      if (g.head_decay) {
        o_out[((size_t)s.row0 * g.heads + head) * g.vdim + c0 + c] = o;
        continue;
      }
      part[c] = o;              // (column c is read and written by this thread alone)
      sq += o * o;
    }
    if (g.head_decay) return;   // (no clusters then)
    sq = warp_sum(sq);
    if (lane == 0) red[warp] = sq;
    __syncthreads();
    sq = 0.f;
#pragma unroll
    for (int w = 0; w < kGdWarps; ++w) sq += red[w];
  }
  if (splits > 1) {
    // (every CTA of a cluster serves the same sequence: all of them come here or none has work)
    cg::cluster_group cl = cg::this_cluster();
    if (threadIdx.x == 0) sums[0] = sq;
    cl.sync();
    if (threadIdx.x == 0) {
      float tot = 0.f;
      for (int i = 0; i < splits; ++i) tot += *cl.map_shared_rank(&sums[0], i);
      sums[1] = tot;
    }
    cl.sync();
    sq = sums[1];
  }
  if (!ok) return;
  const float inv = 1.0f / sqrtf(sq / (float)g.vdim + g.eps);
  const T* gate = static_cast<const T*>(r.gate) + (size_t)s.row0 * r.ld + (size_t)head * g.vdim + c0;
  T* out = static_cast<T*>(r.out) + (size_t)s.row0 * r.ldo + (size_t)head * g.vdim + c0;
  for (int c = threadIdx.x; c < cw; c += kGdThreads) gl_store(out + c, part[c] * inv * g.norm[c0 + c] * gl_silu(gl_load(gate + c)));
}

// ------------------------------------------------------------------------------------------------ token by token
constexpr int kGsThreads = 128, kGsWarps = kGsThreads / 32;
constexpr int kGsCols = 32;           // value columns of a CTA
constexpr int kGsRows = 16;           // tokens staged at a time

template <typename T>
__global__ void __launch_bounds__(kGsThreads) gla_scan_kernel(Gla g, GlaRows r, RaggedBatch b, float* o_out) {
  extern __shared__ float gs_smem[];
  float* S = gs_smem;                             // [dim][kGsCols]
  float* al = S + (size_t)g.dim * kGsCols;        // [kGsRows][dim] decays, keys, queries
  float* ks = al + kGsRows * g.dim;
  float* qs = ks + kGsRows * g.dim;
  float* part = qs + kGsRows * g.dim;             // [warps][kGsRows][kGsCols]
  const int head = blockIdx.y, c = blockIdx.z * kGsCols + (threadIdx.x & 31);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.x, s)) return;
  const bool col = c < g.vdim;
  float* state = g.state + ((s.slot * g.heads + head) * g.dim) * g.vdim;
  for (int d = warp; d < g.dim; d += kGsWarps) S[d * kGsCols + lane] = col && !s.fresh ? state[(size_t)d * g.vdim + c] : 0.f;
  for (int t0 = 0; t0 < s.n; t0 += kGsRows) {
    const int n = min(kGsRows, s.n - t0);
    for (int i = threadIdx.x; i < n * g.dim; i += kGsThreads) {
      const int t = i / g.dim, d = i - t * g.dim, ch = head * g.dim + d;
      const size_t row = s.row0 + t0 + t;
      al[i] = gl_decay(g, head, ch, r.a1 + row * r.ld_a1);
      ks[i] = gl_load(static_cast<const T*>(r.k) + row * r.ld + ch);
      qs[i] = gl_load(static_cast<const T*>(r.q) + row * r.ld + ch) * g.q_scale;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = col ? gl_load(static_cast<const T*>(r.v) + (size_t)(s.row0 + t0 + t) * r.ld + (size_t)head * g.vdim + c) : 0.f;
      float acc = 0.f;
      for (int d = warp; d < g.dim; d += kGsWarps) {
        const float x = fmaf(al[t * g.dim + d], S[d * kGsCols + lane], ks[t * g.dim + d] * v);
        S[d * kGsCols + lane] = x;
        acc = fmaf(qs[t * g.dim + d], x, acc);
      }
      part[(warp * kGsRows + t) * kGsCols + lane] = acc;
    }
    __syncthreads();
    for (int t = warp; t < n; t += kGsWarps) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < kGsWarps; ++w) o += part[(w * kGsRows + t) * kGsCols + lane];
      if (col) o_out[(size_t)(s.row0 + t0 + t) * g.heads * g.vdim + (size_t)head * g.vdim + c] = o;
    }
  }
  for (int d = warp; d < g.dim; d += kGsWarps)
    if (col) state[(size_t)d * g.vdim + c] = S[d * kGsCols + lane];
}

// Head norm and gate: a warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) gla_out_kernel(Gla g, GlaRows r, const int* cache_row, int rows, const float* o) {
  pdl_wait();
  pdl_launch_dependents();
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= (long long)rows * g.heads) return;
  const int lane = threadIdx.x & 31;
  const size_t row = i / g.heads, head = i % g.heads;
  if (cache_row[row] < 0) return;
  const float* src = o + (row * g.heads + head) * g.vdim;
  float sq = 0.f;
  for (int c = lane; c < g.vdim; c += 32) sq += src[c] * src[c];
  const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)g.vdim + g.eps);
  const T* gate = static_cast<const T*>(r.gate) + row * r.ld + head * g.vdim;
  T* out = static_cast<T*>(r.out) + row * r.ldo + head * g.vdim;
  for (int c = lane; c < g.vdim; c += 32) gl_store(out + c, src[c] * inv * g.norm[c] * gl_silu(gl_load(gate + c)));
}

// ------------------------------------------------------------------------------------------------ launch
template <typename T>
static int launch_decode(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, float* o) {
  // columns over a cluster until about two CTAs per SM are busy, at least 32 columns each
  int splits = 1;
  while (splits < 8 && g.vdim % (64 * splits) == 0 && (long long)b.n_seqs * g.heads * splits < 2ll * ctx->sm_count) splits *= 2;
  const size_t smem = ((size_t)3 * g.dim + kGdWarps * (g.vdim / splits)) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 200 * 1024, "gated linear attention: head sizes %d / %d are too large", g.dim, g.vdim);
  auto kern = gla_decode_kernel<T>;
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)(g.heads * splits), (unsigned)b.n_seqs);
  if (g.head_decay) TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3(kGdThreads), smem, g, r, b, splits, o));
  else TQ_CUDA(ctx, launch_k_cluster(ctx, kern, grid, dim3(kGdThreads), smem, splits, g, r, b, splits, o));
  return TQ_OK;
}

template <typename T>
static int launch_scan(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, float* o) {
  const size_t smem = ((size_t)g.dim * kGsCols + (size_t)3 * kGsRows * g.dim + kGsWarps * kGsRows * kGsCols) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 226 * 1024, "gated linear attention: key size %d is too large", g.dim);
  auto kern = gla_scan_kernel<T>;
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.n_seqs, (unsigned)g.heads, (unsigned)((g.vdim + kGsCols - 1) / kGsCols)), dim3(kGsThreads), smem, g,
                        r, b, o));
  if (g.head_decay) return TQ_OK;
  TQ_CUDA(ctx, launch_k(ctx, gla_out_kernel<T>, dim3((unsigned)(((long long)b.rows * g.heads + 7) / 8)), dim3(256), 0, g, r, b.cache_row, b.rows,
                        (const float*)o));
  return TQ_OK;
}

int launch_gla(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, g.heads > 0 && g.dim > 0 && g.vdim > 0 && (g.head_decay || (g.rank > 0 && g.tau > 0.f)) && g.max_seq > 0, "gated linear attention: bad sizes");
  if (b.rows == 0 || b.n_seqs == 0) return TQ_OK;
  TQ_REQUIRE(ctx, g.heads <= 65535 && b.n_seqs <= 65535, "gated linear attention: too many heads or sequences");
  const bool decode = b.max_q <= 1, prompts = dtype == TQ_BF16 && b.max_q >= 8;
  if (!g.head_decay && prompts && gla_chunked_supported(g, r)) return launch_gla_chunked(ctx, g, r, b);
  float* o = nullptr;
  auto rows = [&]() -> int {
    if (decode) return dtype == TQ_F32 ? launch_decode<float>(ctx, g, r, b, o) : launch_decode<__nv_bfloat16>(ctx, g, r, b, o);
    return dtype == TQ_F32 ? launch_scan<float>(ctx, g, r, b, o) : launch_scan<__nv_bfloat16>(ctx, g, r, b, o);
  };
  const size_t width = (size_t)g.heads * g.vdim;
  if (!g.head_decay) {
    if (!decode) {
      if (int st = ensure_scratch(ctx, (size_t)b.rows * width * sizeof(float))) return st;
      o = static_cast<float*>(ctx->scratch);
    }
    return rows();
  }
  const bool chunked = prompts && lightning_chunked_supported(g, r);
  if (int st = ensure_scratch(ctx, ((size_t)b.rows * width + (chunked ? lightning_chunk_floats(g, b) : 0)) * sizeof(float))) return st;
  o = static_cast<float*>(ctx->scratch);
  if (int st = chunked ? launch_lightning_chunked(ctx, g, r, b, o, o + (size_t)b.rows * width) : rows()) return st;
  return launch_norm_gate(ctx, o, width, g.norm, r.gate, r.ld, r.out, r.ldo, b.cache_row, (size_t)b.rows, width, g.eps, dtype);
}

}  // namespace tq

using namespace tq;

extern "C" int tq_gla(tq_ctx* ctx, const tq_gla_config* cfg, int dtype, const void* q_dev, const void* k_dev, const void* v_dev, const void* gate_dev,
                      size_t ld, const float* a1_dev, size_t ld_a1, const float* a2_dev, const float* a2_bias_dev, const float* norm_dev,
                      float* state_dev, size_t max_seq, size_t cache_rows, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev,
                      size_t n_seqs, size_t rows, size_t max_q, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && (dtype == TQ_BF16 || dtype == TQ_F32), "tq_gla: dtype must be bf16 or f32");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, q_dev && k_dev && v_dev && gate_dev && a1_dev && a2_dev && a2_bias_dev && norm_dev && state_dev && row_pos_dev && cache_row_dev && out_dev,
             "tq_gla: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || (rows == n_seqs && max_q == 1), "tq_gla: without row offsets every sequence brings one row");
  Gla g;
  g.heads = (int)cfg->heads;
  g.dim = (int)cfg->dim;
  g.vdim = (int)cfg->vdim;
  g.rank = (int)cfg->rank;
  g.tau = cfg->tau;
  g.q_scale = cfg->q_scale;
  g.eps = cfg->eps;
  g.a2 = a2_dev;
  g.a2_bias = a2_bias_dev;
  g.norm = norm_dev;
  g.state = state_dev;
  g.max_seq = (int)max_seq;
  GlaRows r;
  r.q = q_dev;
  r.k = k_dev;
  r.v = v_dev;
  r.gate = gate_dev;
  r.ld = ld;
  r.a1 = a1_dev;
  r.ld_a1 = ld_a1;
  r.out = out_dev;
  r.ldo = ldo;
  RaggedBatch b;
  b.n_seqs = (int)n_seqs;
  b.rows = (int)rows;
  b.max_q = (int)max_q;
  b.seq_rows = seq_rows_dev;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  return launch_gla(ctx, g, r, b, dtype);
}
