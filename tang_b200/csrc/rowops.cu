// Row operators (see rowops.cuh).
#include "rowops.cuh"

#include <cuda_bf16.h>

#include <cmath>

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
template <typename T>
__global__ void __launch_bounds__(kRoThreads) qk_norm_rope_kernel(QkNormRope a, const int* row_pos, const int* cache_row, size_t cache_rows) {
  extern __shared__ float qr_smem[];
  __shared__ float red[2][kRoWarps];
  const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, half = a.rot.dims / 2;
  float* qs = qr_smem;
  float* ks = qs + nq;
  float* cs = ks + nk;             // [half] cosine, then [half] sine
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, crow = cache_row[m];
  if (crow < 0 || (size_t)crow >= cache_rows) return;
  T* q = static_cast<T*>(a.q) + (size_t)m * a.ldq;
  const T* raw = static_cast<const T*>(a.raw) + (size_t)crow * a.kv_heads * a.raw_pad;
  T* keys = static_cast<T*>(a.keys) + (size_t)crow * a.kv_heads * a.key_pad;
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < half; i += kRoThreads) {
    float s, c;
    sincosf(pos * a.rot.freq[i], &s, &c);
    cs[i] = c * a.rot.mult;
    cs[half + i] = s * a.rot.mult;
  }
  float sq = 0.f, sk = 0.f;
  constexpr int V = 16 / sizeof(T);
  const bool vec = a.dim % V == 0 && a.ldq % V == 0 && a.raw_pad % V == 0 && a.key_pad % V == 0;
  auto unpack = [](const uint4& u, float (&f)[V]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = V == 4 ? __uint_as_float(w[j & 3]) : bf16_bits_to_float(j & 1 ? w[(j >> 1) & 3] >> 16 : w[(j >> 1) & 3] & 0xFFFFu);
  };
  if (vec) {
    const int per = a.dim / V;
    for (int i = threadIdx.x; i < (nq + nk) / V; i += kRoThreads) {
      const bool is_q = i < nq / V;
      const int c = is_q ? i : i - nq / V;
      float f[V];
      unpack(*reinterpret_cast<const uint4*>(is_q ? q + c * V : raw + (c / per) * a.raw_pad + (c % per) * V), f);
      float* dst = (is_q ? qs : ks) + c * V;
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < V; ++j) {
        dst[j] = f[j];
        s += f[j] * f[j];
      }
      if (is_q) sq += s;
      else sk += s;
    }
  } else {
    for (int i = threadIdx.x; i < nq; i += kRoThreads) {
      const float v = ro_load(q + i);
      qs[i] = v;
      sq += v * v;
    }
    for (int i = threadIdx.x; i < nk; i += kRoThreads) {
      const float v = ro_load(raw + (i / a.dim) * a.raw_pad + i % a.dim);
      ks[i] = v;
      sk += v * v;
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < kRoWarps; ++i) {
    sq += red[0][i];
    sk += red[1][i];
  }
  const float qi = 1.0f / sqrtf(sq / (float)nq + a.eps), ki = 1.0f / sqrtf(sk / (float)nk + a.eps);
  const T *qg = static_cast<const T*>(a.q_gain), *kg = static_cast<const T*>(a.k_gain);
  // value i of a row, normed and rotated
  auto value = [&](const float* row, const T* gain, float inv, int i) -> float {
    const int d = i % a.dim;
    const float own = row[i] * inv * ro_load(gain + i);
    if (d >= 2 * half) return own;
    const bool first = d < half;
    const int o = first ? i + half : i - half, f = first ? d : d - half;
    const float other = row[o] * inv * ro_load(gain + o);
    return first ? own * cs[f] - other * cs[half + f] : own * cs[f] + other * cs[half + f];
  };
  if (vec) {
    const int per = a.dim / V;
    for (int i = threadIdx.x; i < (nq + nk) / V; i += kRoThreads) {
      const bool is_q = i < nq / V;
      const int c = is_q ? i : i - nq / V;
      float f[V];
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = is_q ? value(qs, qg, qi, c * V + j) : value(ks, kg, ki, c * V + j);
      T* dst = is_q ? q + c * V : keys + (c / per) * a.key_pad + (c % per) * V;
      ro_store4(dst, make_float4(f[0], f[1], f[2], f[3]));
      if constexpr (V == 8) ro_store4(dst + 4, make_float4(f[4], f[5], f[6], f[7]));
    }
  } else {
    for (int i = threadIdx.x; i < nq; i += kRoThreads) ro_store(q + i, value(qs, qg, qi, i));
    for (int i = threadIdx.x; i < nk; i += kRoThreads) ro_store(keys + (i / a.dim) * a.key_pad + i % a.dim, value(ks, kg, ki, i));
  }
}

int launch_qk_norm_rope(tq_ctx* ctx, const QkNormRope& a, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.rot.dims >= 0 && a.rot.dims % 2 == 0 && a.rot.dims <= a.dim,
             "query/key norm: the rotated dimensions must be even and at most the head size");
  if (b.rows == 0) return TQ_OK;
  const size_t smem = ((size_t)(a.heads + a.kv_heads) * a.dim + a.rot.dims) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 200 * 1024, "query/key norm: %d + %d heads of %d values are too many", a.heads, a.kv_heads, a.dim);
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.rows), dim3(kRoThreads), smem, a, b.row_pos, b.cache_row, b.cache_rows));
    return TQ_OK;
  };
  return dtype == TQ_F32 ? go(qk_norm_rope_kernel<float>) : go(qk_norm_rope_kernel<__nv_bfloat16>);
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

}  // extern "C"
