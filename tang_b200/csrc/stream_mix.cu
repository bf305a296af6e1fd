// Hyper-connections (StreamMix in rowops.cuh): one pass over a row's streams takes a sublayer's output in -- summing the rows of
// its chosen experts on the way --, mixes the streams, forms the next sublayer's input from them and norms it.
#include <cuda_bf16.h>

#include <type_traits>

#include "common.cuh"
#include "rowops.cuh"

namespace tq {

constexpr int kSmMaxRows = 64;       // rows of y per row of the batch

template <int V>
struct SmVec {
  float v[V];
};
template <int V>
__device__ __forceinline__ SmVec<V> sm_load(const float* p) {
  SmVec<V> r;
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    r.v[0] = f.x, r.v[1] = f.y, r.v[2] = f.z, r.v[3] = f.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ SmVec<V> sm_load(const __nv_bfloat16* p) {
  SmVec<V> r;
  if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    r.v[0] = bf16_bits_to_float(u.x & 0xFFFFu), r.v[1] = bf16_bits_to_float(u.x >> 16);
    r.v[2] = bf16_bits_to_float(u.y & 0xFFFFu), r.v[3] = bf16_bits_to_float(u.y >> 16);
  } else {
    r.v[0] = __bfloat162float(*p);
  }
  return r;
}
template <int V>
__device__ __forceinline__ void sm_store(float* p, const SmVec<V>& r) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
template <int V>
__device__ __forceinline__ void sm_store(__nv_bfloat16* p, const SmVec<V>& r) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  } else {
    *p = __float2bfloat16_rn(r.v[0]);
  }
}

template <int S, int V>
__device__ __forceinline__ SmVec<V> sm_sum(const SmVec<V> (&x)[S], int n) {
  SmVec<V> r;
#pragma unroll
  for (int j = 0; j < V; ++j) r.v[j] = 0.f;
#pragma unroll
  for (int s = 0; s < S; ++s)
    if (s < n) {
#pragma unroll
      for (int j = 0; j < V; ++j) r.v[j] += x[s].v[j];
    }
  return r;
}

// The value of an output type, as the next reader of a stored vector sees it.
template <typename OT, int V>
__device__ __forceinline__ void sm_round(SmVec<V>& r) {
  if constexpr (sizeof(OT) == 2) {
#pragma unroll
    for (int j = 0; j < V; ++j) r.v[j] = __bfloat162float(__float2bfloat16_rn(r.v[j]));
  }
}

// One CTA per row; a thread owns V columns at a time in every stream, so that the streams and `self` may be overwritten in place.
// S: streams, or (above 4) the most of them.
template <typename OT, int S, int V>
__global__ void __launch_bounds__(512) stream_mix_kernel(StreamMix a, int width) {
  extern __shared__ __align__(16) float sm_u[];           // [width] the next input before its norm
  __shared__ float mix[S * S], w_out[S], w_in[S], red[32], yw[kSmMaxRows];
  __shared__ int yr[kSmMaxRows];
  const int n = S > 4 ? a.streams : S;
  // (weights: before the wait)
  if (a.y && (int)threadIdx.x < n * n) mix[threadIdx.x] = a.mix[threadIdx.x];
  if ((int)threadIdx.x < n) {
    if (a.y) w_out[threadIdx.x] = a.w_out[threadIdx.x];
    w_in[threadIdx.x] = a.w_in ? a.w_in[threadIdx.x] : 1.f;
  }
  pdl_wait();
  pdl_launch_dependents();
  const size_t m = blockIdx.x, row = a.src_rows ? (size_t)a.src_rows[m] : m;
  if (a.y && (int)threadIdx.x < a.n_y) {
    yr[threadIdx.x] = a.y_rows ? a.y_rows[m * a.n_y + threadIdx.x] : (int)m;
    yw[threadIdx.x] = a.y_weight ? a.y_weight[m * a.n_y + threadIdx.x] : 1.f;
  }
  __syncthreads();
  const float* src = a.src + row * a.src_streams * width;
  const size_t src_ld = a.src_streams == 1 ? 0 : width;
  float* dst = a.dst + m * n * width;
  OT* out = static_cast<OT*>(a.out) + m * a.ld_out;
  const OT* self = static_cast<const OT*>(a.self) + m * a.ld_out;
  const float more = a.y_more_gate ? 1.0f / (1.0f + expf(-a.y_more_gate[m * a.ld_gate])) : 1.f;
  float sq = 0.f;
#pragma unroll(S > 4 ? 1 : 2)
  for (int d = V * threadIdx.x; d < width; d += V * blockDim.x) {
    SmVec<V> x[S], u;
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s < n) x[s] = sm_load<V>(src + s * src_ld + d);
    if (a.y) {
      SmVec<V> y;
#pragma unroll
      for (int j = 0; j < V; ++j) y.v[j] = 0.f;
      for (int k = 0; k < a.n_y; ++k) {
        const int r = yr[k];
        const float w = yw[k];
        SmVec<V> part;
        if (r >= 0) part = sm_load<V>(a.y + (size_t)r * width + d);
        else if (a.self) part = sm_load<V>(self + d);
        else continue;
#pragma unroll
        for (int j = 0; j < V; ++j) y.v[j] = fmaf(w, part.v[j], y.v[j]);
      }
      if (a.y_more) {
        const SmVec<V> part = sm_load<V>(a.y_more + m * width + d);
#pragma unroll
        for (int j = 0; j < V; ++j) y.v[j] = fmaf(more, part.v[j], y.v[j]);
      }
      SmVec<V> old[S];
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s < n) old[s] = x[s];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < V; ++j) x[t].v[j] = w_out[t] * y.v[j];
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s < n) {
#pragma unroll
            for (int j = 0; j < V; ++j) x[t].v[j] = fmaf(mix[s * n + t], old[s].v[j], x[t].v[j]);
          }
      }
      if (a.inject) {
        if (a.sum) sm_store<V>(a.sum + m * width + d, sm_sum<S, V>(x, n));
        const SmVec<V> part = sm_load<V>(a.inject + m * width + d);
#pragma unroll
        for (int t = 0; t < S; ++t)
          if (t < n) {
#pragma unroll
            for (int j = 0; j < V; ++j) x[t].v[j] += part.v[j];
          }
      }
#pragma unroll
      for (int t = 0; t < S; ++t)
        if (t < n) sm_store<V>(dst + (size_t)t * width + d, x[t]);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) u.v[j] = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s < n) {
#pragma unroll
        for (int j = 0; j < V; ++j) u.v[j] = fmaf(w_in[s], x[s].v[j], u.v[j]);
      }
    if (a.sum && !a.inject) sm_store<V>(a.sum + m * width + d, sm_sum<S, V>(x, n));
    if (a.gain) {
#pragma unroll
      for (int j = 0; j < V; ++j) sq += u.v[j] * u.v[j];
      sm_store<V>(sm_u + d, u);
    }
  }
  if (!a.gain) return;
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
  const float inv = 1.0f / sqrtf(sq / (float)width + a.eps);
  const int crow = a.conv_w ? a.cache_row[m] : 0, pos = a.conv_w ? a.row_pos[m] : 0;
  OT* st_row = static_cast<OT*>(a.conv_state) + (size_t)(crow < 0 ? 0 : crow / a.max_seq) * (a.conv_taps - 1) * width;   // (a row without a slot reads slot 0's)
  for (int d = V * threadIdx.x; d < width; d += V * blockDim.x) {
    const SmVec<V> g = sm_load<V>(a.gain + d);
    SmVec<V> u = sm_load<V>(sm_u + d);
#pragma unroll
    for (int j = 0; j < V; ++j) u.v[j] *= inv * g.v[j];
    if (a.conv_w) {
      // (the state holds what a prompt's rows hold: values of the output type)
      sm_round<OT, V>(u);
      const SmVec<V> h = u;
      OT* st = st_row + d;
      for (int t = 0; t < a.conv_taps; ++t) {
        const SmVec<V> w = sm_load<V>(a.conv_w + (size_t)t * width + d);
        SmVec<V> in = h;
        if (t + 1 < a.conv_taps) {
          in = sm_load<V>(st + (size_t)t * width);
          if (t > 0 && crow >= 0) sm_store<V>(st + (size_t)(t - 1) * width, in);
          if (pos < a.conv_taps - 1 - t) {                 // before the sequence's start, whatever the slot still holds
#pragma unroll
            for (int j = 0; j < V; ++j) in.v[j] = 0.f;
          }
        } else if (t > 0 && crow >= 0) {
          sm_store<V>(st + (size_t)(t - 1) * width, h);
        }
#pragma unroll
        for (int j = 0; j < V; ++j) u.v[j] = fmaf(w.v[j], in.v[j], u.v[j]);
      }
    }
    sm_store<V>(out + d, u);
  }
}

// A decode step's form of one stream with a convolution: the row, its norm's gain, the convolution's weights and inputs in registers,
// NV vectors of four columns per thread.  Weights are read before the wait, everything else right behind it.
template <typename OT>
using SmRaw = std::conditional_t<sizeof(OT) == 2, uint2, float4>;
__device__ __forceinline__ SmVec<4> sm_unpack(uint2 u) {
  SmVec<4> r;
  r.v[0] = bf16_bits_to_float(u.x & 0xFFFFu), r.v[1] = bf16_bits_to_float(u.x >> 16);
  r.v[2] = bf16_bits_to_float(u.y & 0xFFFFu), r.v[3] = bf16_bits_to_float(u.y >> 16);
  return r;
}
__device__ __forceinline__ SmVec<4> sm_unpack(float4 f) {
  SmVec<4> r;
  r.v[0] = f.x, r.v[1] = f.y, r.v[2] = f.z, r.v[3] = f.w;
  return r;
}

constexpr int kSmStepThreads = 512;

template <typename OT, int NV, int TAPS>
__global__ void __launch_bounds__(kSmStepThreads) stream_step_kernel(StreamMix a, int width) {
  using Raw = SmRaw<OT>;
  __shared__ float red[32];
  SmVec<4> gain[NV], w[TAPS][NV], x[NV];
  const int n_thr = blockDim.x;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * n_thr);
    const bool on = d < width;
    gain[i] = on ? sm_load<4>(a.gain + d) : SmVec<4>{};
#pragma unroll
    for (int t = 0; t < TAPS; ++t) w[t][i] = on ? sm_load<4>(a.conv_w + (size_t)t * width + d) : SmVec<4>{};
  }
  const float keep = a.y ? a.mix[0] : 1.f, mult = a.y ? a.w_out[0] : 0.f;
  pdl_wait();
  pdl_launch_dependents();
  const size_t m = blockIdx.x;
  const int crow = a.cache_row[m], pos = a.row_pos[m];
  const float logit = a.y_more_gate ? a.y_more_gate[m * a.ld_gate] : 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = 4 * (threadIdx.x + i * n_thr);
    x[i] = d < width ? sm_load<4>(a.src + m * width + d) : SmVec<4>{};
  }
  Raw* st = static_cast<Raw*>(a.conv_state) + ((size_t)(crow < 0 ? 0 : crow / a.max_seq) * (TAPS - 1) * width) / 4;   // (a row without a slot reads slot 0's)
  Raw hist[TAPS > 1 ? TAPS - 1 : 1][NV];
#pragma unroll
  for (int t = 0; t < TAPS - 1; ++t)
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int v = threadIdx.x + i * n_thr;
      if (4 * v < width) hist[t][i] = st[(size_t)t * (width / 4) + v];
      else hist[t][i] = Raw{};
    }
  if (a.y) {
    SmVec<4> y[NV] = {};
    for (int k0 = 0; k0 < a.n_y; k0 += 4) {
      int r[4];
      float wy[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const bool on = k0 + k < a.n_y;
        r[k] = !on ? -1 : a.y_rows ? a.y_rows[m * a.n_y + k0 + k] : (int)m;
        wy[k] = on && a.y_weight ? a.y_weight[m * a.n_y + k0 + k] : 1.f;
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = 4 * (threadIdx.x + i * n_thr);
        SmVec<4> part[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) part[k] = r[k] >= 0 && d < width ? sm_load<4>(a.y + (size_t)r[k] * width + d) : SmVec<4>{};
#pragma unroll
        for (int k = 0; k < 4; ++k)
#pragma unroll
          for (int j = 0; j < 4; ++j) y[i].v[j] = fmaf(wy[k], part[k].v[j], y[i].v[j]);
      }
    }
    const float more = a.y_more_gate ? 1.0f / (1.0f + expf(-logit)) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = 4 * (threadIdx.x + i * n_thr);
      if (d >= width) continue;
      if (a.y_more) {
        const SmVec<4> part = sm_load<4>(a.y_more + m * width + d);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[i].v[j] = fmaf(more, part.v[j], y[i].v[j]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) x[i].v[j] = fmaf(keep, x[i].v[j], mult * y[i].v[j]);
      if (a.sum) sm_store<4>(a.sum + m * width + d, x[i]);
      if (a.inject) {
        const SmVec<4> part = sm_load<4>(a.inject + m * width + d);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[i].v[j] += part.v[j];
      }
      sm_store<4>(a.dst + m * width + d, x[i]);
    }
  }
  const float u_mult = a.w_in ? a.w_in[0] : 1.f;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      x[i].v[j] *= u_mult;
      sq += x[i].v[j] * x[i].v[j];
    }
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
  const float inv = 1.0f / sqrtf(sq / (float)width + a.eps);
  OT* out = static_cast<OT*>(a.out) + m * a.ld_out;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * n_thr, d = 4 * v;
    if (d >= width) continue;
    SmVec<4> h;
#pragma unroll
    for (int j = 0; j < 4; ++j) h.v[j] = x[i].v[j] * inv * gain[i].v[j];
    sm_round<OT, 4>(h);
    SmVec<4> o = h;
#pragma unroll
    for (int t = 0; t < TAPS - 1; ++t) {
      const SmVec<4> in = sm_unpack(hist[t][i]);
#pragma unroll
      for (int j = 0; j < 4; ++j) o.v[j] = fmaf(w[t][i].v[j], pos < TAPS - 1 - t ? 0.f : in.v[j], o.v[j]);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) o.v[j] = fmaf(w[TAPS - 1][i].v[j], h.v[j], o.v[j]);
    sm_store<4>(out + d, o);
    if (TAPS > 1 && crow >= 0) {
#pragma unroll
      for (int t = 0; t + 2 < TAPS; ++t) st[(size_t)t * (width / 4) + v] = hist[t + 1][i];
      sm_store<4>(reinterpret_cast<OT*>(st + (size_t)(TAPS - 2) * (width / 4) + v), h);
    }
  }
}

template <typename OT>
static int stream_step_typed(tq_ctx* ctx, const StreamMix& a, size_t rows, size_t width) {
  auto go = [&](auto taps) -> int {
    constexpr int T = decltype(taps)::value;
    const size_t vecs = width / 4;
    auto kern = vecs <= kSmStepThreads ? stream_step_kernel<OT, 1, T> : stream_step_kernel<OT, 2, T>;
    const size_t per = vecs <= kSmStepThreads ? vecs : (vecs + 1) / 2;
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)rows), dim3((unsigned)((per + 31) / 32 * 32)), 0, a, (int)width));
    return TQ_OK;
  };
  switch (a.conv_taps) {
    case 1: return go(std::integral_constant<int, 1>());
    case 2: return go(std::integral_constant<int, 2>());
    case 3: return go(std::integral_constant<int, 3>());
    default: return go(std::integral_constant<int, 4>());
  }
}

template <typename OT>
static int stream_mix_typed(tq_ctx* ctx, const StreamMix& a, size_t rows, size_t width) {
  const uintptr_t bits = (uintptr_t)a.src | (uintptr_t)a.dst | (uintptr_t)a.y | (uintptr_t)a.y_more | (uintptr_t)a.gain | (uintptr_t)a.out | (uintptr_t)a.self |
                         (uintptr_t)a.sum | (uintptr_t)a.inject | (uintptr_t)a.conv_w | (uintptr_t)a.conv_state;
  const bool vec = a.streams <= 4 && width % 4 == 0 && a.ld_out % 4 == 0 && (bits & 15) == 0;
  if (vec && a.conv_w && a.conv_taps <= 4 && a.streams == 1 && !a.self && !a.src_rows && width <= 8 * (size_t)kSmStepThreads) return stream_step_typed<OT>(ctx, a, rows, width);
  const size_t smem = a.gain ? width * sizeof(float) : 0;
  size_t threads = vec ? width / 4 : width;
  const size_t most = rows >= 2 * (size_t)ctx->sm_count ? 256 : 512, least = a.streams > 4 ? 256 : 64;
  threads = threads > most ? most : threads < least ? least : (threads + 31) / 32 * 32;
  auto go = [&](auto s) -> int {
    constexpr int S = decltype(s)::value;
    auto kern = vec ? stream_mix_kernel<OT, S, S <= 4 ? 4 : 1> : stream_mix_kernel<OT, S, 1>;
    if (smem > 40 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)rows), dim3((unsigned)threads), smem, a, (int)width));
    return TQ_OK;
  };
  switch (a.streams) {
    case 1: return go(std::integral_constant<int, 1>());
    case 2: return go(std::integral_constant<int, 2>());
    case 3: return go(std::integral_constant<int, 3>());
    case 4: return go(std::integral_constant<int, 4>());
    default: return go(std::integral_constant<int, kMaxStreams>());
  }
}

int launch_stream_mix(tq_ctx* ctx, const StreamMix& a, size_t rows, size_t width) {
  TQ_REQUIRE(ctx, a.streams >= 1 && a.streams <= kMaxStreams && (a.src_streams == 1 || a.src_streams == a.streams), "stream mix: 1 to %d streams", kMaxStreams);
  TQ_REQUIRE(ctx, width > 0 && width <= 49152, "stream mix: rows of 1 to 49152 values");
  TQ_REQUIRE(ctx, !a.y || (a.dst && a.mix && a.w_out && a.n_y >= 1 && a.n_y <= kSmMaxRows && !a.src_rows && (a.y_rows || a.n_y == 1)),
             "stream mix: bad sublayer output (at most %d rows each)", kSmMaxRows);
  TQ_REQUIRE(ctx, !a.gain || a.out, "stream mix: nowhere to put the norm");
  TQ_REQUIRE(ctx, !a.inject || a.y, "stream mix: rows are added to the streams together with a sublayer's output");
  TQ_REQUIRE(ctx, !a.conv_w || (a.gain && a.row_pos && a.cache_row && a.conv_taps >= 1 && a.max_seq > 0 && (a.conv_state || a.conv_taps == 1)), "stream mix: bad convolution");
  if (rows == 0) return TQ_OK;
  return a.out_dtype == TQ_F32 ? stream_mix_typed<float>(ctx, a, rows, width) : stream_mix_typed<__nv_bfloat16>(ctx, a, rows, width);
}

}  // namespace tq

using namespace tq;

extern "C" int tq_stream_mix(tq_ctx* ctx, size_t streams, size_t src_streams, const float* src_dev, float* dst_dev, const float* y_dev, const int* y_rows_dev,
                             const float* y_weight_dev, size_t n_y, const void* self_dev, const float* y_more_dev, const float* mix_dev,
                             const float* w_out_dev, const float* w_in_dev, const float* gain_dev, size_t rows, size_t width, float eps, void* out_dev,
                             int out_dtype, size_t ld_out, float* sum_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src_dev && (out_dtype == TQ_F32 || out_dtype == TQ_BF16), "tq_stream_mix: no streams, or out is neither f32 nor bf16");
  StreamMix a;
  a.streams = (int)streams;
  a.src_streams = (int)src_streams;
  a.src = src_dev;
  a.dst = dst_dev;
  a.y = y_dev;
  a.y_rows = y_rows_dev;
  a.y_weight = y_weight_dev;
  a.n_y = y_rows_dev ? (int)n_y : 1;
  a.self = self_dev;
  a.y_more = y_more_dev;
  a.mix = mix_dev;
  a.w_out = w_out_dev;
  a.w_in = w_in_dev;
  a.gain = gain_dev;
  a.out = out_dev;
  a.out_dtype = out_dtype;
  a.ld_out = ld_out ? ld_out : width;
  a.eps = eps;
  a.sum = sum_dev;
  return launch_stream_mix(ctx, a, rows, width);
}

extern "C" int tq_stream_step(tq_ctx* ctx, const float* src_dev, float* dst_dev, const float* y_dev, const int* y_rows_dev, const float* y_weight_dev, size_t n_y,
                              const float* y_more_dev, const float* y_more_gate_dev, size_t ld_gate, const float* inject_dev, const float* mix_one_dev,
                              const float* w_out_dev, const float* gain_dev, size_t rows, size_t width, float eps, const float* conv_w_dev, void* conv_state_dev,
                              size_t taps, size_t max_seq, const int* row_pos_dev, const int* cache_row_dev, void* out_dev, int out_dtype, size_t ld_out,
                              float* sum_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, src_dev && dst_dev && y_dev && mix_one_dev && w_out_dev && gain_dev && out_dev && (out_dtype == TQ_F32 || out_dtype == TQ_BF16),
             "tq_stream_step: null pointer, or out is neither f32 nor bf16");
  StreamMix a;
  a.src = src_dev;
  a.dst = dst_dev;
  a.y = y_dev;
  a.y_rows = y_rows_dev;
  a.y_weight = y_weight_dev;
  a.n_y = y_rows_dev ? (int)n_y : 1;
  a.y_more = y_more_dev;
  a.y_more_gate = y_more_gate_dev;
  a.ld_gate = ld_gate;
  a.inject = inject_dev;
  a.mix = mix_one_dev;
  a.w_out = w_out_dev;
  a.gain = gain_dev;
  a.out = out_dev;
  a.out_dtype = out_dtype;
  a.ld_out = ld_out ? ld_out : width;
  a.eps = eps;
  a.sum = sum_dev;
  a.conv_w = conv_w_dev;
  a.conv_state = conv_state_dev;
  a.conv_taps = (int)taps;
  a.max_seq = (int)max_seq;
  a.row_pos = row_pos_dev;
  a.cache_row = cache_row_dev;
  return launch_stream_mix(ctx, a, rows, width);
}
