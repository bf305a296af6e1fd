// Row operators (see rowops.cuh).
#include "rowops.cuh"

#include <cuda_bf16.h>

#include <cmath>
#include <type_traits>

#include "common.cuh"

namespace tq {

constexpr int kRoThreads = 256;
constexpr int kRoWarps = kRoThreads / 32;

__device__ __forceinline__ float ro_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRoWarps; ++i) t += red[i];
  return t;
}

__device__ __forceinline__ void ro_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ro_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float ro_load(const float* p) { return *p; }
__device__ __forceinline__ float ro_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ro_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ro_store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// One CTA per row, the row in registers.  width % 4 == 0, aligned rows, NV * 1024 >= width.
template <typename OT, int NV>
__global__ void __launch_bounds__(kRoThreads) add_norm_vec_kernel(AddNorm a, int width) {
  __shared__ float red[2][kRoWarps];
  const size_t m = blockIdx.x;
  float4 gp[NV], gn[NV];
  // (gains are weights: read before the wait)
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * kRoThreads);
    gp[i] = gn[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (d < width) {
      if (a.y) gp[i] = *reinterpret_cast<const float4*>(a.gain_post + d);
      if (a.gain_next) gn[i] = *reinterpret_cast<const float4*>(a.gain_next + d);
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  float4 x[NV], y[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * kRoThreads);
    x[i] = y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (d < width) x[i] = *reinterpret_cast<const float4*>(a.x + m * width + d);
  }
  if (a.y) {
    for (int k = 0; k < a.n_y; ++k) {
      const int r = a.y_rows ? a.y_rows[m * a.n_y + k] : (int)m;
      if (r < 0) continue;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = 4 * (threadIdx.x + i * kRoThreads);
        if (d < width) {
          const float4 v = *reinterpret_cast<const float4*>(a.y + (size_t)r * width + d);
          y[i].x += v.x;
          y[i].y += v.y;
          y[i].z += v.z;
          y[i].w += v.w;
        }
      }
    }
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) sq += y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
    const float inv = 1.0f / sqrtf(ro_block_sum(sq, red[0]) / (float)width + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = 4 * (threadIdx.x + i * kRoThreads);
      x[i].x += y[i].x * inv * gp[i].x;
      x[i].y += y[i].y * inv * gp[i].y;
      x[i].z += y[i].z * inv * gp[i].z;
      x[i].w += y[i].w * inv * gp[i].w;
      if (d < width) *reinterpret_cast<float4*>(a.x + m * width + d) = x[i];
    }
  }
  if (!a.gain_next) return;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) sq += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
  const float inv = 1.0f / sqrtf(ro_block_sum(sq, red[1]) / (float)width + a.eps);
  OT* out = static_cast<OT*>(a.out) + m * a.ld_out;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * kRoThreads);
    if (d < width) ro_store4(out + d, make_float4(x[i].x * inv * gn[i].x, x[i].y * inv * gn[i].y, x[i].z * inv * gn[i].z, x[i].w * inv * gn[i].w));
  }
}

// Any width and alignment.
template <typename OT>
__global__ void __launch_bounds__(kRoThreads) add_norm_kernel(AddNorm a, int width) {
  extern __shared__ float ro_row[];
  __shared__ float red[2][kRoWarps];
  pdl_wait();
  pdl_launch_dependents();
  const size_t m = blockIdx.x;
  float* x = a.x + m * width;
  float sq = 0.f;
  if (a.y) {
    for (int d = threadIdx.x; d < width; d += kRoThreads) {
      float y = 0.f;
      for (int k = 0; k < a.n_y; ++k) {
        const int r = a.y_rows ? a.y_rows[m * a.n_y + k] : (int)m;
        if (r >= 0) y += a.y[(size_t)r * width + d];
      }
      ro_row[d] = y;
      sq += y * y;
    }
  }
  const float inv_y = a.y ? 1.0f / sqrtf(ro_block_sum(sq, red[0]) / (float)width + a.eps) : 0.f;
  sq = 0.f;
  for (int d = threadIdx.x; d < width; d += kRoThreads) {
    float v = x[d];
    if (a.y) {
      v += ro_row[d] * inv_y * a.gain_post[d];
      x[d] = v;
    }
    ro_row[d] = v;
    sq += v * v;
  }
  if (!a.gain_next) return;
  const float inv = 1.0f / sqrtf(ro_block_sum(sq, red[1]) / (float)width + a.eps);
  OT* out = static_cast<OT*>(a.out) + m * a.ld_out;
  for (int d = threadIdx.x; d < width; d += kRoThreads) ro_store(out + d, ro_row[d] * inv * a.gain_next[d]);
}

template <typename OT>
static int add_norm_typed(tq_ctx* ctx, const AddNorm& a, size_t rows, size_t width) {
  const dim3 grid((unsigned)rows), block(kRoThreads);
  const uintptr_t bits = (uintptr_t)a.x | (uintptr_t)a.y | (uintptr_t)a.gain_post | (uintptr_t)a.gain_next | (uintptr_t)a.out;
  if (width % 4 || a.ld_out % 4 || (bits & 15)) {
    TQ_CUDA(ctx, launch_k(ctx, add_norm_kernel<OT>, grid, block, width * sizeof(float), a, (int)width));
  } else if (width <= 2048) {
    TQ_CUDA(ctx, launch_k(ctx, add_norm_vec_kernel<OT, 2>, grid, block, 0, a, (int)width));
  } else if (width <= 4096) {
    TQ_CUDA(ctx, launch_k(ctx, add_norm_vec_kernel<OT, 4>, grid, block, 0, a, (int)width));
  } else {
    TQ_CUDA(ctx, launch_k(ctx, add_norm_vec_kernel<OT, 8>, grid, block, 0, a, (int)width));
  }
  return TQ_OK;
}

int launch_add_norm(tq_ctx* ctx, const AddNorm& a, size_t rows, size_t width) {
  TQ_REQUIRE(ctx, width > 0 && width <= 8192, "add_norm: width must be in 1..8192");
  if (rows == 0) return TQ_OK;
  return a.out_dtype == TQ_F32 ? add_norm_typed<float>(ctx, a, rows, width) : add_norm_typed<__nv_bfloat16>(ctx, a, rows, width);
}

// ------------------------------------------------------------------------------------------------ query / key norm, rotation
// One CTA per row; the row's queries and keys pass through shared memory as f32 (a pair's halves sit in different places).
// VEC: everything in 16-byte pieces; a thread then handles one piece of a row at a time.
constexpr int kQkMaxThreads = 640;

template <typename T, bool VEC>
__global__ void __launch_bounds__(kQkMaxThreads) qk_norm_rope_kernel(QkNormRope a, const int* row_pos, const int* cache_row, size_t cache_rows) {
  extern __shared__ __align__(16) float qr_smem[];
  __shared__ float red[2][kQkMaxThreads / 32];
  constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, half = a.rot.dims / 2, per = a.dim / V;
  const int n_pieces = (nq + nk) / V;
  float* vals = qr_smem;                     // [nq + nk]: queries, then keys
  float* cs = vals + nq + nk;                // [half] cosine, then [half] sine
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, crow = cache_row[m];
  if (crow < 0 || (size_t)crow >= cache_rows) return;
  T* q = static_cast<T*>(a.q) + (size_t)m * a.ldq;
  const T* raw = static_cast<const T*>(a.raw) + (size_t)crow * a.kv_heads * a.raw_pad;
  T* keys = static_cast<T*>(a.keys) + (size_t)crow * a.kv_heads * a.key_pad;
  auto unpack = [](const uint4& u, float (&f)[V]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = V == 4 ? __uint_as_float(w[j & 3]) : bf16_bits_to_float(j & 1 ? w[(j >> 1) & 3] >> 16 : w[(j >> 1) & 3] & 0xFFFFu);
  };
  auto load = [&](const T* p, float (&f)[V]) {
    if constexpr (VEC) unpack(*reinterpret_cast<const uint4*>(p), f);
    else f[0] = ro_load(p);
  };
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < n_pieces; i += blockDim.x) {
    const bool is_q = i < nq / V;
    const int c = is_q ? i : i - nq / V;
    float f[V], s = 0.f;
    if (is_q) {
      load(q + c * V, f);
    } else {
      const int head = (int)((unsigned)c / (unsigned)per);
      load(raw + head * a.raw_pad + (c - head * per) * V, f);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s += f[j] * f[j];
    if constexpr (VEC) {
#pragma unroll
      for (int j = 0; j < V; j += 4) *reinterpret_cast<float4*>(vals + (size_t)i * V + j) = make_float4(f[j], f[j + 1], f[j + 2], f[j + 3]);
    } else {
      vals[i] = f[0];
    }
    if (is_q) sq += s;
    else sk += s;
  }
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * a.rot.freq[i], &s, &c);
    cs[i] = c * a.rot.mult;
    cs[half + i] = s * a.rot.mult;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();
  const bool has = (threadIdx.x & 31) < (blockDim.x >> 5);
  sq = warp_sum(has ? red[0][threadIdx.x & 31] : 0.f);
  sk = warp_sum(has ? red[1][threadIdx.x & 31] : 0.f);
  const float qi = 1.0f / sqrtf(sq / (float)nq + a.eps), ki = 1.0f / sqrtf(sk / (float)nk + a.eps);
  for (int i = threadIdx.x; i < n_pieces; i += blockDim.x) {
    const bool is_q = i < nq / V;
    const int c = is_q ? i : i - nq / V, head = (int)((unsigned)c / (unsigned)per), d0 = (c - head * per) * V;
    const float inv = is_q ? qi : ki;
    const T* gain = static_cast<const T*>(is_q ? a.q_gain : a.k_gain);
    // V values of the row from vals[at], normed
    auto piece = [&](int at, float (&f)[V]) {
      float gf[V];
      load(gain + at, gf);
      const float* src = vals + (is_q ? 0 : nq) + at;
      if constexpr (VEC) {
#pragma unroll
        for (int j = 0; j < V; j += 4) {
          const float4 v = *reinterpret_cast<const float4*>(src + j);
          f[j] = v.x, f[j + 1] = v.y, f[j + 2] = v.z, f[j + 3] = v.w;
        }
      } else {
        f[0] = *src;
      }
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= inv * gf[j];
    };
    float f[V];
    piece(c * V, f);
    if (d0 < 2 * half) {
      if (half % V == 0) {                   // whole pieces turn with whole pieces
        const bool first = d0 < half;
        const int r = first ? d0 : d0 - half;
        float o[V];
        piece(c * V + (first ? half : -half), o);
#pragma unroll
        for (int j = 0; j < V; ++j) f[j] = f[j] * cs[r + j] + (first ? -o[j] : o[j]) * cs[half + r + j];
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const int d = d0 + j;
          if (d < 2 * half) {
            const bool first = d < half;
            const int shift = first ? half : -half, r = first ? d : d - half;
            const float other = vals[i * V + j + shift] * inv * ro_load(gain + c * V + j + shift);
            f[j] = f[j] * cs[r] + (first ? -other : other) * cs[half + r];
          }
        }
      }
    }
    T* dst = is_q ? q + c * V : keys + head * a.key_pad + d0;
    if constexpr (VEC) {
#pragma unroll
      for (int j = 0; j < V; j += 4) ro_store4(dst + j, make_float4(f[j], f[j + 1], f[j + 2], f[j + 3]));
    } else {
      ro_store(dst, f[0]);
    }
  }
}

int launch_qk_norm_rope(tq_ctx* ctx, const QkNormRope& a, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.rot.dims >= 0 && a.rot.dims % 2 == 0 && a.rot.dims <= a.dim,
             "query/key norm: the rotated dimensions must be even and at most the head size");
  if (b.rows == 0) return TQ_OK;
  const size_t smem = ((size_t)(a.heads + a.kv_heads) * a.dim + a.rot.dims) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 200 * 1024, "query/key norm: %d + %d heads of %d values are too many", a.heads, a.kv_heads, a.dim);
  auto go = [&](auto kern, int v) -> int {
    // one round of pieces when there are few rows, several rounds per thread when the rows fill the GPU anyway
    const int pieces = (a.heads + a.kv_heads) * a.dim / v, most = b.rows >= 4 * ctx->sm_count ? 256 : kQkMaxThreads;
    const int threads = pieces >= most ? most : (pieces + 31) / 32 * 32;
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.rows), dim3((unsigned)threads), smem, a, b.row_pos, b.cache_row, b.cache_rows));
    return TQ_OK;
  };
  const int v = dtype == TQ_F32 ? 4 : 8;
  const uintptr_t bits = (uintptr_t)a.q | (uintptr_t)a.raw | (uintptr_t)a.keys | (uintptr_t)a.q_gain | (uintptr_t)a.k_gain;
  const bool vec = a.dim % v == 0 && a.ldq % v == 0 && a.raw_pad % v == 0 && a.key_pad % v == 0 && (bits & 15) == 0;
  if (dtype == TQ_F32) return vec ? go(qk_norm_rope_kernel<float, true>, v) : go(qk_norm_rope_kernel<float, false>, 1);
  return vec ? go(qk_norm_rope_kernel<__nv_bfloat16, true>, v) : go(qk_norm_rope_kernel<__nv_bfloat16, false>, 1);
}

// ------------------------------------------------------------------------------------------------ per-head norm, rotation
// blockIdx.x: row; the CTA's warps (and blockIdx.y's CTAs) share its heads, queries first.  The row's cosines and sines are formed
// once per CTA.  Two forms: a head's 16-byte pieces in the registers of up to 32 lanes, which pass the other half of a pair through
// shuffles; any size and alignment, the head in its warp's shared memory.
template <typename T>
__global__ void __launch_bounds__(256) head_norm_rope_reg_kernel(HeadNormRope a, int lanes, const int* row_pos, const int* cache_row, size_t cache_rows) {
  extern __shared__ __align__(16) float hr_smem[];
  constexpr int V = 16 / (int)sizeof(T);
  const QkNormRope& r = a.r;
  const int half = r.rot.dims / 2, dim = r.dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  float* cs = hr_smem;                                    // [half rounded to 4] cosine, then sine
  float* sn = hr_smem + (half + 3) / 4 * 4;
  const int l = lane & (lanes - 1), d0 = l * V, i0 = d0 - r.rot.first, per_warp = 32 / lanes;
  const bool live = d0 < dim;
  auto unpack = [](const uint4& u, float (&f)[V]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = V == 4 ? __uint_as_float(w[j & 3]) : bf16_bits_to_float(j & 1 ? w[(j >> 1) & 3] >> 16 : w[(j >> 1) & 3] & 0xFFFFu);
  };
  uint4 qg = make_uint4(0u, 0u, 0u, 0u), kg = qg;         // (weights: before the wait)
  if (live && r.q_gain) qg = *reinterpret_cast<const uint4*>(static_cast<const T*>(r.q_gain) + d0);
  if (live && r.k_gain) kg = *reinterpret_cast<const uint4*>(static_cast<const T*>(r.k_gain) + d0);
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, crow = cache_row[m];
  if (crow < 0 || (size_t)crow >= cache_rows) return;
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * r.rot.freq[i], &s, &c);
    cs[i] = c * r.rot.mult;
    sn[i] = s * r.rot.mult;
  }
  __syncthreads();
  const bool turns = live && i0 >= 0 && i0 < 2 * half, lead = i0 < half;
  // this lane's cosines and sines (the same for every head), and where its pairs' other halves are
  float c[V], s[V];
  const int other = r.rot.interleaved || !turns ? lane : lead ? lane + half / V : lane - half / V;
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int p = r.rot.interleaved ? (i0 + j) >> 1 : lead ? i0 + j : i0 + j - half;
    const bool on = turns && p < half;
    c[j] = on ? cs[p] : 1.f;
    s[j] = on ? ((r.rot.interleaved ? !(j & 1) : lead) ? -sn[p] : sn[p]) : 0.f;
  }
  const int total = r.heads + r.kv_heads;
  for (int h0 = (blockIdx.y * warps + warp) * per_warp; h0 < total; h0 += warps * gridDim.y * per_warp) {
    const int h = h0 + lane / lanes, g = h - r.heads;
    const bool is_q = h < r.heads, on = live && h < total;
    const T* src = is_q ? static_cast<const T*>(r.q) + (size_t)m * r.ldq + (size_t)h * a.q_head
                        : static_cast<const T*>(r.raw) + ((size_t)crow * r.kv_heads + g) * r.raw_pad;
    T* dst = is_q ? static_cast<T*>(r.q) + (size_t)m * r.ldq + (size_t)h * a.q_head : static_cast<T*>(r.keys) + ((size_t)crow * r.kv_heads + g) * r.key_pad;
    float f[V];
    unpack(on ? *reinterpret_cast<const uint4*>(src + d0) : make_uint4(0u, 0u, 0u, 0u), f);
    if (is_q ? r.q_gain != nullptr : r.k_gain != nullptr) {
      float sq = 0.f, gf[V];
#pragma unroll
      for (int j = 0; j < V; ++j) sq += f[j] * f[j];
      for (int o = lanes / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      const float inv = 1.0f / sqrtf(sq / (float)dim + r.eps);
      unpack(is_q ? qg : kg, gf);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= inv * gf[j];
    }
    float out[V];
    if (r.rot.interleaved) {
#pragma unroll
      for (int j = 0; j < V; ++j) out[j] = f[j] * c[j] + f[j ^ 1] * s[j];
    } else {
#pragma unroll
      for (int j = 0; j < V; ++j) out[j] = f[j] * c[j] + __shfl_sync(0xffffffffu, f[j], other) * s[j];
    }
    if (on) {
#pragma unroll
      for (int j = 0; j < V; j += 4) ro_store4(dst + d0 + j, make_float4(out[j], out[j + 1], out[j + 2], out[j + 3]));
    }
  }
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) head_norm_rope_kernel(HeadNormRope a, const int* row_pos, const int* cache_row, size_t cache_rows) {
  extern __shared__ __align__(16) float hr_smem[];
  constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
  const QkNormRope& r = a.r;
  const int half = r.rot.dims / 2, dim = r.dim, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  float* cs = hr_smem;                                    // [half] cosine, then [half] sine
  float* vals = hr_smem + (2 * half + 3) / 4 * 4 + (size_t)warp * ((dim + 3) / 4 * 4);
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, crow = cache_row[m];
  if (crow < 0 || (size_t)crow >= cache_rows) return;
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(pos * r.rot.freq[i], &s, &c);
    cs[i] = c * r.rot.mult;
    cs[half + i] = s * r.rot.mult;
  }
  __syncthreads();
  for (int h = blockIdx.y * warps + warp; h < r.heads + r.kv_heads; h += warps * gridDim.y) {
    const bool is_q = h < r.heads;
    const int g = h - r.heads;
    const T* src = is_q ? static_cast<const T*>(r.q) + (size_t)m * r.ldq + (size_t)h * a.q_head
                        : static_cast<const T*>(r.raw) + ((size_t)crow * r.kv_heads + g) * r.raw_pad;
    T* dst = is_q ? static_cast<T*>(r.q) + (size_t)m * r.ldq + (size_t)h * a.q_head : static_cast<T*>(r.keys) + ((size_t)crow * r.kv_heads + g) * r.key_pad;
    const T* gain = static_cast<const T*>(is_q ? r.q_gain : r.k_gain);
    float sq = 0.f;
    for (int d = lane * V; d < dim; d += 32 * V) {
      if constexpr (VEC) {
        const uint4 u = *reinterpret_cast<const uint4*>(src + d);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int j = 0; j < V; ++j) {
          const float f = V == 4 ? __uint_as_float(w[j & 3]) : bf16_bits_to_float(j & 1 ? w[(j >> 1) & 3] >> 16 : w[(j >> 1) & 3] & 0xFFFFu);
          vals[d + j] = f;
          sq += f * f;
        }
      } else {
        vals[d] = ro_load(src + d);
        sq += vals[d] * vals[d];
      }
    }
    const float inv = gain ? 1.0f / sqrtf(warp_sum(sq) / (float)dim + r.eps) : 1.0f;
    __syncwarp();
    auto normed = [&](int d) { return gain ? vals[d] * inv * ro_load(gain + d) : vals[d]; };
    for (int d0 = lane * V; d0 < dim; d0 += 32 * V) {
      float f[V];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const int d = d0 + j, i = d - r.rot.first;
        f[j] = normed(d);
        if (i >= 0 && i < 2 * half) {
          const bool lead = r.rot.interleaved ? !(i & 1) : i < half;
          const int shift = r.rot.interleaved ? 1 : half, p = r.rot.interleaved ? i >> 1 : lead ? i : i - half;
          const float other = normed(lead ? d + shift : d - shift);
          f[j] = f[j] * cs[p] + (lead ? -other : other) * cs[half + p];
        }
      }
      if constexpr (VEC) {
#pragma unroll
        for (int j = 0; j < V; j += 4) ro_store4(dst + d0 + j, make_float4(f[j], f[j + 1], f[j + 2], f[j + 3]));
      } else {
        ro_store(dst + d0, f[0]);
      }
    }
    __syncwarp();
  }
}

int launch_head_norm_rope(tq_ctx* ctx, const HeadNormRope& a0, const RaggedBatch& b, int dtype) {
  HeadNormRope a = a0;
  if (!a.q_head) a.q_head = (size_t)a.r.dim;
  QkNormRope& r = a.r;
  TQ_REQUIRE(ctx, r.heads >= 0 && r.kv_heads >= 0 && r.heads + r.kv_heads > 0 && r.dim > 0 && r.rot.first >= 0 && r.rot.dims >= 0 && r.rot.dims % 2 == 0 &&
                      r.rot.first + r.rot.dims <= r.dim,
             "head norm: the rotated dimensions must be even and inside the head");
  if (b.rows == 0) return TQ_OK;
  if (!r.q_gain && r.kv_heads == 0) {          // only what turns is touched
    if (r.rot.dims == 0) return TQ_OK;
    r.q = static_cast<char*>(r.q) + (size_t)r.rot.first * dtype_size(dtype);
    r.dim = r.rot.dims;
    r.rot.first = 0;
  }
  const int total = r.heads + r.kv_heads;
  int warps = total < 8 ? total : 8;
  const size_t smem = ((size_t)r.rot.dims + 3 + (size_t)warps * ((r.dim + 3) / 4 * 4)) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 200 * 1024, "head norm: heads of %d values are too large", r.dim);
  int parts = 1;
  while (parts * warps < total && (long long)b.rows * parts < 2ll * ctx->sm_count) ++parts;
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.rows, (unsigned)parts), dim3((unsigned)(32 * warps)), smem, a, b.row_pos, b.cache_row, b.cache_rows));
    return TQ_OK;
  };
  const int v = dtype == TQ_F32 ? 4 : 8;
  const uintptr_t bits = (uintptr_t)r.q | (uintptr_t)r.raw | (uintptr_t)r.keys;
  const bool vec = r.dim % v == 0 && r.ldq % v == 0 && a.q_head % v == 0 && r.raw_pad % v == 0 && r.key_pad % v == 0 && (bits & 15) == 0;
  const bool gains = (((uintptr_t)r.q_gain | (uintptr_t)r.k_gain) & 15) == 0 && (r.kv_heads == 0 || !r.q_gain == !r.k_gain);
  if (vec && gains && r.dim / v <= 32 && r.rot.first % v == 0 && (r.rot.interleaved || r.rot.dims % (2 * v) == 0)) {
    int lanes = 1;
    while (lanes < r.dim / v) lanes *= 2;
    const int units = (total + 32 / lanes - 1) / (32 / lanes), w = units < 8 ? units : 8;      // warps of heads
    int y = 1;
    while (y * w < units && (long long)b.rows * y < 2ll * ctx->sm_count) ++y;
    const size_t cs = ((size_t)r.rot.dims + 8) * sizeof(float);
    auto reg = [&](auto kern) -> int {
      TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.rows, (unsigned)y), dim3((unsigned)(32 * w)), cs, a, lanes, b.row_pos, b.cache_row, b.cache_rows));
      return TQ_OK;
    };
    return dtype == TQ_F32 ? reg(head_norm_rope_reg_kernel<float>) : reg(head_norm_rope_reg_kernel<__nv_bfloat16>);
  }
  if (dtype == TQ_F32) return vec ? go(head_norm_rope_kernel<float, true>) : go(head_norm_rope_kernel<float, false>);
  return vec ? go(head_norm_rope_kernel<__nv_bfloat16, true>) : go(head_norm_rope_kernel<__nv_bfloat16, false>);
}

// ------------------------------------------------------------------------------------------------ row norm and gate
template <typename T, bool VEC>
__global__ void __launch_bounds__(kRoThreads) norm_gate_kernel(const float* o, size_t ld_o, const float* norm, const T* gate, size_t ldg, T* out, size_t ldo,
                                                               const int* cache_row, int width, float eps) {
  __shared__ float red[kRoWarps];
  constexpr int V = VEC ? 4 : 1;
  pdl_wait();
  pdl_launch_dependents();
  const size_t m = blockIdx.x;
  if (cache_row && cache_row[m] < 0) return;
  o += m * ld_o;
  gate += m * ldg;
  out += m * ldo;
  float sq = 0.f;
#pragma unroll 4
  for (int d = V * threadIdx.x; d < width; d += V * kRoThreads) {
    if constexpr (VEC) {
      const float4 v = *reinterpret_cast<const float4*>(o + d);
      sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    } else {
      sq += o[d] * o[d];
    }
  }
  const float inv = 1.0f / sqrtf(ro_block_sum(sq, red) / (float)width + eps);
  auto open = [](float z) { return 1.0f / (1.0f + expf(-z)); };
#pragma unroll 4
  for (int d = V * threadIdx.x; d < width; d += V * kRoThreads) {
    if constexpr (VEC) {
      const float4 v = *reinterpret_cast<const float4*>(o + d), w = *reinterpret_cast<const float4*>(norm + d);
      ro_store4(out + d, make_float4(v.x * inv * w.x * open(ro_load(gate + d)), v.y * inv * w.y * open(ro_load(gate + d + 1)),
                                     v.z * inv * w.z * open(ro_load(gate + d + 2)), v.w * inv * w.w * open(ro_load(gate + d + 3))));
    } else {
      ro_store(out + d, o[d] * inv * norm[d] * open(ro_load(gate + d)));
    }
  }
}

int launch_norm_gate(tq_ctx* ctx, const float* o, size_t ld_o, const float* norm, const void* gate, size_t ldg, void* out, size_t ldo, const int* cache_row,
                     size_t rows, size_t width, float eps, int dtype) {
  if (rows == 0) return TQ_OK;
  const bool vec = width % 4 == 0 && ld_o % 4 == 0 && ldo % 4 == 0 && (((uintptr_t)o | (uintptr_t)norm | (uintptr_t)out) & 15) == 0;
  auto go = [&](auto kern, auto* tag) -> int {
    using T = std::remove_pointer_t<decltype(tag)>;
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)rows), dim3(kRoThreads), 0, o, ld_o, norm, static_cast<const T*>(gate), ldg, static_cast<T*>(out), ldo,
                          cache_row, (int)width, eps));
    return TQ_OK;
  };
  if (dtype == TQ_F32) return vec ? go(norm_gate_kernel<float, true>, (float*)nullptr) : go(norm_gate_kernel<float, false>, (float*)nullptr);
  return vec ? go(norm_gate_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)nullptr) : go(norm_gate_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)nullptr);
}

void banded_frequencies(int dims, double base, double factor, double low, double high, double original, float* freq) {
  const double pi = 3.14159265358979323846;
  for (int i = 0; i < dims / 2; ++i) {
    const double f = std::pow(base, -2.0 * i / dims), wave = 2 * pi / f;
    double g = f;
    if (factor > 0) {
      if (wave > original / low) {
        g = f / factor;
      } else if (wave >= original / high) {
        const double s = (original / wave - low) / (high - low);
        g = (1 - s) * f / factor + s * f;
      }
    }
    freq[i] = (float)g;
  }
}

void yarn_frequencies(int dims, double base, double factor, double original, double fast, double slow, float* freq, float* mult) {
  const double pi = 3.14159265358979323846;
  *mult = factor > 0 ? (float)(0.1 * std::log(factor) + 1.0) : 1.0f;
  // the dimension whose pair makes `turns` turns over the original context
  auto at = [&](double turns) { return dims * std::log(original / (2 * pi * turns)) / (2 * std::log(base)); };
  const double lo = factor > 0 ? std::fmax(std::floor(at(fast)), 0.0) : 0.0, hi = factor > 0 ? std::fmin(std::ceil(at(slow)), dims - 1.0) : 0.0;
  for (int i = 0; i < dims / 2; ++i) {
    const double f = std::pow(base, -2.0 * i / dims);
    const double ramp = factor > 0 ? std::fmin(std::fmax((i - lo) / std::fmax(hi - lo, 0.001), 0.0), 1.0) : 0.0;
    freq[i] = (float)(factor > 0 ? f / factor * ramp + f * (1 - ramp) : f);
  }
}

}  // namespace tq

using namespace tq;

extern "C" {

int tq_yarn_frequencies(size_t dims, double base, double factor, double original, double fast, double slow, float* freq_host, float* mult_host) {
  if (!freq_host || !mult_host || dims % 2 || dims == 0 || !(base > 1.0)) return TQ_EINVAL;
  if (factor > 0 && !(original > 0 && fast > 0 && slow > 0)) return TQ_EINVAL;
  yarn_frequencies((int)dims, base, factor, original, fast, slow, freq_host, mult_host);
  return TQ_OK;
}

int tq_banded_frequencies(size_t dims, double base, double factor, double low, double high, double original, float* freq_host) {
  if (!freq_host || dims % 2 || dims == 0 || !(base > 1.0)) return TQ_EINVAL;
  if (factor > 0 && !(original > 0 && low > 0 && high > low)) return TQ_EINVAL;
  banded_frequencies((int)dims, base, factor, low, high, original, freq_host);
  return TQ_OK;
}

int tq_add_norm(tq_ctx* ctx, float* x_dev, const float* y_dev, const int* y_rows_dev, size_t n_y, const float* gain_post_dev,
                const float* gain_next_dev, size_t rows, size_t width, float eps, void* out_dev, int out_dtype, size_t ld_out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, out_dtype == TQ_F32 || out_dtype == TQ_BF16, "tq_add_norm: out must be f32 or bf16");
  TQ_REQUIRE(ctx, x_dev && (!y_dev || gain_post_dev) && (!gain_next_dev || out_dev) && (y_dev || gain_next_dev), "tq_add_norm: null pointer");
  AddNorm a;
  a.x = x_dev;
  a.y = y_dev;
  a.y_rows = y_rows_dev;
  a.n_y = y_rows_dev ? (int)n_y : 1;
  a.gain_post = gain_post_dev;
  a.gain_next = gain_next_dev;
  a.out = out_dev;
  a.out_dtype = out_dtype;
  a.ld_out = ld_out ? ld_out : width;
  a.eps = eps;
  return launch_add_norm(ctx, a, rows, width);
}

int tq_qk_norm_rope(tq_ctx* ctx, int dtype, size_t heads, size_t kv_heads, size_t dim, void* q_dev, size_t ldq, const void* raw_dev,
                    void* keys_dev, size_t cache_rows, const void* q_gain_dev, const void* k_gain_dev, size_t rot_dims, const float* freq_dev,
                    float rot_mult, float eps, const int* row_pos_dev, const int* cache_row_dev, size_t rows) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_F32 || dtype == TQ_BF16, "tq_qk_norm_rope: dtype must be f32 or bf16");
  TQ_REQUIRE(ctx, q_dev && raw_dev && keys_dev && q_gain_dev && k_gain_dev && (freq_dev || rot_dims == 0) && row_pos_dev && cache_row_dev,
             "tq_qk_norm_rope: null pointer");
  QkNormRope a;
  a.heads = (int)heads;
  a.kv_heads = (int)kv_heads;
  a.dim = (int)dim;
  a.raw_pad = a.key_pad = (int)((dim + 7) / 8 * 8);
  a.q = q_dev;
  a.ldq = ldq;
  a.raw = raw_dev;
  a.keys = keys_dev;
  a.q_gain = q_gain_dev;
  a.k_gain = k_gain_dev;
  a.rot.dims = (int)rot_dims;
  a.rot.freq = freq_dev;
  a.rot.mult = rot_mult;
  a.eps = eps;
  RaggedBatch b;
  b.rows = (int)rows;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  return launch_qk_norm_rope(ctx, a, b, dtype);
}

int tq_head_norm_rope(tq_ctx* ctx, int dtype, size_t heads, size_t kv_heads, size_t dim, void* q_dev, size_t ldq, size_t q_head, const void* raw_dev,
                      void* keys_dev, size_t cache_rows, const void* q_gain_dev, const void* k_gain_dev, size_t rot_first, size_t rot_dims, int interleaved,
                      const float* freq_dev, float rot_mult, float eps, const int* row_pos_dev, const int* cache_row_dev, size_t rows) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_F32 || dtype == TQ_BF16, "tq_head_norm_rope: dtype must be f32 or bf16");
  TQ_REQUIRE(ctx, (q_dev || !heads) && ((raw_dev && keys_dev) || !kv_heads) && (freq_dev || rot_dims == 0) && row_pos_dev && cache_row_dev,
             "tq_head_norm_rope: null pointer");
  HeadNormRope a;
  a.q_head = q_head;
  a.r.heads = (int)heads;
  a.r.kv_heads = (int)kv_heads;
  a.r.dim = (int)dim;
  a.r.raw_pad = a.r.key_pad = (int)((dim + 7) / 8 * 8);
  a.r.q = q_dev;
  a.r.ldq = ldq;
  a.r.raw = raw_dev;
  a.r.keys = keys_dev;
  a.r.q_gain = q_gain_dev;
  a.r.k_gain = k_gain_dev;
  a.r.rot.first = (int)rot_first;
  a.r.rot.dims = (int)rot_dims;
  a.r.rot.interleaved = interleaved != 0;
  a.r.rot.freq = freq_dev;
  a.r.rot.mult = rot_mult;
  a.r.eps = eps;
  RaggedBatch b;
  b.rows = (int)rows;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  return launch_head_norm_rope(ctx, a, b, dtype);
}

}  // extern "C"
