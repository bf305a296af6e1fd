// Latent attention (see latent_attention.cuh).
//
// latent_decode_kernel: grid = (splits, head tiles, sequences).  A CTA owns one or two tiles of 16 heads (the rows of an
// mma.sync m16n8k16 tile), four warps each, and streams 64-position cache tiles, shared by its head tiles, through a cp.async
// double buffer.  Warp w of a head tile scores positions 16w .. 16w + 15, the four agree on the row maxima through shared memory,
// write the weights as two bf16 terms, and warp w then accumulates its quarter of the latent columns for all 64 positions.
// Splits are merged by latent_combine_kernel.
#include "latent_attention.cuh"

#include <cuda_bf16.h>

#include <cfloat>

#include "attn_mma.cuh"
#include "common.cuh"

namespace tq {

__device__ __forceinline__ float la_load(const float* p) { return *p; }
__device__ __forceinline__ float la_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void la_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void la_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

LatentDims latent_dims(int heads, int dim, int rot, int vdim, int rank) {
  LatentDims d;
  d.heads = heads;
  d.dim = dim;
  d.rot = rot;
  d.vdim = vdim;
  d.rank = rank;
  d.c_pad = (rank + 15) / 16 * 16;
  d.r_pad = (rot + 15) / 16 * 16;
  return d;
}

// ------------------------------------------------------------------------------------------------ norms and rotation of a row
constexpr int kLiThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kLiThreads) latent_in_kernel(LatentIn a, const int* row_pos, const int* cache_row, size_t cache_rows) {
  __shared__ float red[2][kLiThreads / 32];
  const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  if (m == 0 && a.head_jobs) {
    const int per = (a.n_head_rows + a.head_chunk - 1) / a.head_chunk;
    for (int i = threadIdx.x; i < per * a.d.heads; i += kLiThreads) {
      const int h = i / per, at = (i - h * per) * a.head_chunk;
      a.head_jobs[i] = make_int4(h, h * a.n_head_rows + at, min(a.head_chunk, a.n_head_rows - at), 0);
    }
    if (threadIdx.x == 0) *a.n_head_jobs = per * a.d.heads;
  }
  const float* low = a.low + (size_t)m * a.ld_low;
  const float* c = low + a.c0;
  float sq = 0.f, sc = 0.f;
  for (int i = threadIdx.x; i < a.q_rank; i += kLiThreads) sq += low[i] * low[i];
  for (int i = threadIdx.x; i < a.d.rank; i += kLiThreads) sc += c[i] * c[i];
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sc;
  }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < kLiThreads / 32; ++w) {
    sq += red[0][w];
    sc += red[1][w];
  }
  const float qi = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps), ci = 1.0f / sqrtf(sc / (float)a.d.rank + a.eps);
  T* cq = static_cast<T*>(a.cq) + (size_t)m * a.ld_cq;
  for (int i = threadIdx.x; i < a.q_rank; i += kLiThreads) la_store(cq + i, low[i] * qi * a.q_gain[i]);
  const int crow = cache_row[m];
  if (crow < 0 || (size_t)crow >= cache_rows) return;
  T* row = static_cast<T*>(a.cache) + (size_t)crow * a.d.row();
  for (int i = threadIdx.x; i < a.d.c_pad; i += kLiThreads) la_store(row + i, i < a.d.rank ? c[i] * ci * a.c_gain[i] : 0.f);
  const float* r = c + a.d.rank;
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < a.d.r_pad / 2; i += kLiThreads) {
    float u = 2 * i < a.d.rot ? r[2 * i] : 0.f, v = 2 * i + 1 < a.d.rot ? r[2 * i + 1] : 0.f;
    if (2 * i < a.rot.dims) {
      float s, co;
      sincosf(pos * a.rot.freq[i], &s, &co);
      s *= a.rot.mult;
      co *= a.rot.mult;
      const float x = u * co - v * s;
      v = v * co + u * s;
      u = x;
    }
    la_store(row + a.d.c_pad + 2 * i, u);
    la_store(row + a.d.c_pad + 2 * i + 1, v);
  }
}

int launch_latent_in(tq_ctx* ctx, const LatentIn& a, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, a.d.rank > 0 && a.q_rank > 0 && a.d.rot >= 0 && a.rot.dims % 2 == 0 && a.rot.dims <= a.d.rot, "latent attention: bad sizes");
  if (b.rows == 0) return TQ_OK;
  if (dtype == TQ_F32) TQ_CUDA(ctx, launch_k(ctx, latent_in_kernel<float>, dim3((unsigned)b.rows), dim3(kLiThreads), 0, a, b.row_pos, b.cache_row, b.cache_rows));
  else TQ_CUDA(ctx, launch_k(ctx, latent_in_kernel<__nv_bfloat16>, dim3((unsigned)b.rows), dim3(kLiThreads), 0, a, b.row_pos, b.cache_row, b.cache_rows));
  return TQ_OK;
}

// ------------------------------------------------------------------------------------------------ expansion plan
struct LatentSeq {
  int row0, n, len;
  int seq0;          // cache row of position 0; negative: not in the cache
};
__device__ __forceinline__ LatentSeq latent_seq(const RaggedBatch& b, int seq) {
  LatentSeq s;
  s.row0 = b.seq_rows ? b.seq_rows[seq] : seq;
  s.n = b.seq_rows ? b.seq_rows[seq + 1] - s.row0 : 1;
  s.len = 0;
  s.seq0 = -1;
  if (s.n <= 0 || s.row0 < 0 || s.row0 + s.n > b.rows) {
    s.n = 0;
    return s;
  }
  const int last = s.row0 + s.n - 1, c0 = b.cache_row[s.row0], c1 = b.cache_row[last], p0 = b.row_pos[s.row0];
  if (c0 < p0 || c1 != c0 + s.n - 1 || (size_t)c1 >= b.cache_rows) return s;      // (reported by the embedding kernel)
  s.seq0 = c0 - p0;
  s.len = p0 + s.n;
  return s;
}

constexpr int kLpThreads = 1024;

__global__ void __launch_bounds__(kLpThreads) latent_plan_kernel(RaggedBatch b, int first_seq, int end_seq, int min_q, int chunk, int max_jobs, LatentPlan p) {
  __shared__ int wl[32], wj[32];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int base_len = 0, base_jobs = 0;
  for (int s0 = 0; s0 < b.n_seqs; s0 += kLpThreads) {
    const int seq = s0 + threadIdx.x;
    LatentSeq s = {};
    bool mine = false;
    if (seq < b.n_seqs) {
      s = latent_seq(b, seq);
      mine = seq >= first_seq && seq < end_seq && s.n >= min_q && s.seq0 >= 0;
      p.single[seq] = s.n == 1 && s.seq0 >= 0 ? s.row0 : -1;
    }
    const int len = mine ? s.len : 0, jobs = (len + chunk - 1) / chunk;
    int sl = len, sj = jobs;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int x = __shfl_up_sync(0xffffffffu, sl, o), y = __shfl_up_sync(0xffffffffu, sj, o);
      if (lane >= o) {
        sl += x;
        sj += y;
      }
    }
    if (lane == 31) {
      wl[warp] = sl;
      wj[warp] = sj;
    }
    __syncthreads();
    int bl = base_len, bj = base_jobs;
    for (int w = 0; w < 32; ++w) {
      if (w < warp) {
        bl += wl[w];
        bj += wj[w];
      }
      base_len += wl[w];
      base_jobs += wj[w];
    }
    const int off = bl + sl - len, at = bj + sj - jobs;
    if (seq < b.n_seqs) p.off[seq] = mine ? off : -1;
    for (int i = 0; i < jobs; ++i)
      if (at + i < max_jobs) p.jobs[at + i] = make_int4(0, s.seq0 + i * chunk, min(chunk, len - i * chunk), off - s.seq0);
    __syncthreads();
  }
  if (threadIdx.x == 0) *p.n_jobs = min(base_jobs, max_jobs);
  for (int seq = 0; seq < b.n_seqs; ++seq) {
    const int row0 = b.seq_rows ? b.seq_rows[seq] : seq, end = min(b.seq_rows ? b.seq_rows[seq + 1] : seq + 1, b.rows), off = p.off[seq];
    for (int m = row0 + threadIdx.x; m < end; m += kLpThreads) p.exp_row[m] = off < 0 ? -1 : off + b.row_pos[m];
  }
}

int launch_latent_plan(tq_ctx* ctx, const RaggedBatch& b, int first_seq, int end_seq, int min_q, int chunk, int max_jobs, const LatentPlan& p) {
  TQ_REQUIRE(ctx, chunk > 0 && max_jobs > 0, "latent attention: bad plan");
  TQ_CUDA(ctx, launch_k(ctx, latent_plan_kernel, dim3(1), dim3(kLpThreads), 0, b, first_seq, end_seq, min_q, chunk, max_jobs, p));
  return TQ_OK;
}

// blockIdx: 16 positions, sequence.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) latent_place_kernel(LatentDims d, RaggedBatch b, const int* off, const T* cache, T* keys, int key_pad) {
  constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
  pdl_wait();
  pdl_launch_dependents();
  const int o = off[blockIdx.y];
  if (o < 0) return;
  const LatentSeq s = latent_seq(b, blockIdx.y);
  const int p0 = blockIdx.x * 16, n = min(16, s.len - p0), per = (key_pad - d.dim) / V;
  if (n <= 0) return;
  for (int i = threadIdx.x; i < n * d.heads * per; i += 256) {
    const int p = i / (d.heads * per), h = i / per % d.heads, j = i % per * V;
    const T* src = cache + (size_t)(s.seq0 + p0 + p) * d.row() + d.c_pad + j;
    T* dst = keys + ((size_t)(o + p0 + p) * d.heads + h) * key_pad + d.dim + j;
    if constexpr (VEC) *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
    else la_store(dst, j < d.rot ? la_load(src) : 0.f);
  }
}

int launch_latent_place(tq_ctx* ctx, const LatentDims& d, const RaggedBatch& b, const LatentPlan& p, const void* cache, void* keys, int key_pad, int dtype) {
  const dim3 grid((unsigned)((b.max_len + 15) / 16), (unsigned)b.n_seqs);
  TQ_REQUIRE(ctx, grid.y <= 65535, "latent attention: too many sequences");
  auto go = [&](auto kern, auto* tag) -> int {
    using T = std::remove_pointer_t<decltype(tag)>;
    TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3(256), 0, d, b, (const int*)p.off, static_cast<const T*>(cache), static_cast<T*>(keys), key_pad));
    return TQ_OK;
  };
  const int v = dtype == TQ_F32 ? 4 : 8;
  const bool vec = d.dim % v == 0 && key_pad == d.dim + d.rot && d.rot % v == 0;
  if (dtype == TQ_F32) return vec ? go(latent_place_kernel<float, true>, (float*)nullptr) : go(latent_place_kernel<float, false>, (float*)nullptr);
  return vec ? go(latent_place_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)nullptr) : go(latent_place_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)nullptr);
}

__global__ void __launch_bounds__(128) latent_gather_kernel(const int* single, const __nv_bfloat16* q, int rows, int n_seqs, size_t ld, __nv_bfloat16* out) {
  pdl_wait();
  pdl_launch_dependents();
  const int row = single[blockIdx.x];
  if (row < 0) return;
  const __nv_bfloat16* src = q + ((size_t)blockIdx.y * rows + row) * ld;
  __nv_bfloat16* dst = out + ((size_t)blockIdx.y * n_seqs + blockIdx.x) * ld;
  for (size_t i = threadIdx.x; i < ld; i += 128) dst[i] = src[i];
}

int launch_latent_gather(tq_ctx* ctx, const RaggedBatch& b, const int* single, const void* q, int heads, size_t ld, void* out) {
  TQ_REQUIRE(ctx, heads <= 65535, "latent attention: too many heads");
  TQ_CUDA(ctx, launch_k(ctx, latent_gather_kernel, dim3((unsigned)b.n_seqs, (unsigned)heads), dim3(128), 0, single, static_cast<const __nv_bfloat16*>(q), b.rows,
                        b.n_seqs, ld, static_cast<__nv_bfloat16*>(out)));
  return TQ_OK;
}
