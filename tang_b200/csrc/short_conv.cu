// Short causal convolutions (see short_conv.cuh).
//
// Row m's predecessor m - k is in the batch when its cache row is the one k before (a slot brings one run of rows per step);
// otherwise the input comes from the slot's state, or is zero when it would lie before position 0.
#include "short_conv.cuh"

#include <cuda_bf16.h>

#include <type_traits>

#include "common.cuh"

namespace tq {

namespace {

constexpr int kScThreads = 128;
constexpr int kMaxFixedTaps = 4;    // convolutions up to here keep their window in registers

template <typename T, int V>
__device__ __forceinline__ void sc_load(const T* p, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = (float)*p;
  } else {
    static_assert(V * sizeof(T) == 16, "one 16-byte piece");
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = V == 4 ? __uint_as_float(w[j & 3]) : bf16_bits_to_float(j & 1 ? w[(j >> 1) & 3] >> 16 : w[(j >> 1) & 3] & 0xFFFFu);
  }
}

template <typename T, int V>
__device__ __forceinline__ void sc_store(T* p, const float (&f)[V]) {
  if constexpr (V == 1) {
    *p = (T)f[0];
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    uint32_t w[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
      w[j] = *reinterpret_cast<const uint32_t*>(&v);
    }
    *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
}

// (channels and columns are multiples of V)
template <int V>
__device__ __forceinline__ void sc_weights(const float* p, bool live, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = live ? *p : 0.f;
  } else {
#pragma unroll
    for (int j = 0; j < V; j += 4) {
      const float4 v = live ? *reinterpret_cast<const float4*>(p + j) : make_float4(0.f, 0.f, 0.f, 0.f);
      f[j] = v.x, f[j + 1] = v.y, f[j + 2] = v.z, f[j + 3] = v.w;
    }
  }
}

// Input k rows before row m (k > 0), V channels from `col` on.
template <typename T, int V>
__device__ __forceinline__ void sc_before(const ShortConv& c, const T* x, size_t ldx, int col, int m, int k, int pos, int crow, const int* cache_row, float (&f)[V]) {
  if (pos < k) {                                       // before the sequence's start, whatever the slot still holds
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = 0.f;
    return;
  }
  int n = 0;                                           // how many of the k predecessors are in the batch
  while (n < k && n < m && cache_row[m - n - 1] == crow - n - 1) ++n;
  if (n == k) sc_load<T, V>(x + (size_t)(m - k) * ldx + col, f);
  else sc_load<T, V>(static_cast<const T*>(c.state) + ((size_t)(crow / c.max_seq) * (c.taps - 1) + c.taps - 1 - (k - n)) * c.channels + col, f);
}

// The state after one row: everything moves up by one, `cur` is the latest input.  (What another sequence left moves along; sc_before
// never looks before position 0.)
template <typename T, int V>
__device__ __forceinline__ void sc_push(const ShortConv& c, int col, int crow, const float (&cur)[V]) {
  if (c.taps < 2) return;
  T* st = static_cast<T*>(c.state) + (size_t)(crow / c.max_seq) * (c.taps - 1) * c.channels + col;
  for (int j = 0; j + 2 < c.taps; ++j) {
    float f[V];
    sc_load<T, V>(st + (size_t)(j + 1) * c.channels, f);
    sc_store<T, V>(st + (size_t)j * c.channels, f);
  }
  sc_store<T, V>(st + (size_t)(c.taps - 2) * c.channels, cur);
}

// y = conv at row m for V channels, whose input is cur; any number of taps, every input read again.
template <typename T, int V>
__device__ __forceinline__ void conv_any(const ShortConv& c, const T* x, size_t ldx, int col, int m, int pos, int crow, const int* cache_row, const float (&cur)[V],
                                         float (&y)[V]) {
#pragma unroll
  for (int j = 0; j < V; ++j) y[j] = 0.f;
  for (int t = 0; t < c.taps; ++t) {
    float f[V], wt[V];
    if (t == c.taps - 1) {
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = cur[j];
    } else {
      sc_before<T, V>(c, x, ldx, col, m, c.taps - 1 - t, pos, crow, cache_row, f);
    }
    sc_weights<V>(c.w + (size_t)t * c.channels + col, true, wt);
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] = fmaf(wt[j], f[j], y[j]);
  }
}

// Up to kMaxFixedTaps taps: R consecutive rows and the TAPS - 1 rows ahead of them, V channels per thread, all loaded at once.  STEP:
// one row per sequence, whose predecessors are all in the state.
//   cr[TAPS - 1 + r]: cache row of row r of the run, cr[TAPS - 2 - k] of the row k + 1 before the run; impossible values where there is none
template <typename T, int V, int TAPS, int R, bool STEP>
struct ConvWindow {
  static constexpr int H = TAPS - 1, N = STEP ? 1 : R + H;      // rows of x in registers
  float w[TAPS][V];
  uint4 x[N];

  __device__ __forceinline__ void weights(const ShortConv& c, int col, bool on) {
#pragma unroll
    for (int t = 0; t < TAPS; ++t) sc_weights<V>(c.w + (size_t)t * c.channels + col, on, w[t]);
  }
  // (rows of the batch that are no predecessors are loaded all the same, rows outside it are not)
  __device__ __forceinline__ void load(const T* src, size_t ld, int col, int m0, int rows, bool on) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int m = m0 + i - (STEP ? 0 : H);
      x[i] = on && m >= 0 && m < rows ? *reinterpret_cast<const uint4*>(src + (size_t)m * ld + col) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  static __device__ __forceinline__ void unpack(const uint4& u, float (&f)[V]) {
    const uint32_t b[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int j = 0; j < V; ++j) f[j] = V == 4 ? __uint_as_float(b[j & 3]) : bf16_bits_to_float(j & 1 ? b[(j >> 1) & 3] >> 16 : b[(j >> 1) & 3] & 0xFFFFu);
  }
  __device__ __forceinline__ void add(int t, const uint4& u, float (&y)[V]) {
    float f[V];
    unpack(u, f);
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] = fmaf(w[t][j], f[j], y[j]);
  }
  // Row r's input and convolution; STEP moves the state on.
  __device__ __forceinline__ void row(const ShortConv& c, int col, int r, int pos, const int* cr, bool on, float (&cur)[V], float (&y)[V]) {
    unpack(x[STEP ? 0 : r + H], cur);
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] = w[H][j] * cur[j];
    if constexpr (H > 0) {
      const int crow = cr[r + H];
      int n = 0;                                         // predecessors in the batch
      if constexpr (!STEP) {
        while (n < H && cr[r + H - 1 - n] == crow - 1 - n) ++n;
        if (n > pos) n = pos;
        if (n == H) {
#pragma unroll
          for (int t = 0; t < H; ++t) add(t, x[r + t], y);
          return;
        }
      }
      uint4* st = reinterpret_cast<uint4*>(static_cast<T*>(c.state) + (size_t)(crow / c.max_seq) * H * c.channels + col);
      const int ld = c.channels / V;
      uint4 old[H];
#pragma unroll
      for (int t = 0; t < H; ++t) {
        const int k = H - t;                             // rows before row r
        old[t] = on && k > n && pos >= k ? st[(H - (k - n)) * ld] : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int t = 0; t < H; ++t) {
        if constexpr (STEP) add(t, old[t], y);
        else add(t, H - t <= n ? x[r + t] : old[t], y);
      }
      if (STEP && on) {
#pragma unroll
        for (int t = 0; t + 1 < H; ++t) st[t * ld] = old[t + 1];
        st[(H - 1) * ld] = x[0];
      }
    }
  }
};

// The metadata of a run of R rows: cache rows (see ConvWindow) and positions; rows that are skipped have a negative cache row.
template <int R, int H>
__device__ __forceinline__ void run_rows(const RaggedBatch& b, int m0, int* cr, int* pos) {
  const int i = threadIdx.x;
  if (i < R + H) {
    const int m = m0 + i - H;
    int c = m >= 0 && m < b.rows ? b.cache_row[m] : -1;
    if (c < 0 || (size_t)c >= b.cache_rows) c = -0x40000000;
    cr[i] = c;
    if (i >= H) pos[i - H] = m < b.rows ? b.row_pos[m] : 0;
  }
}

constexpr int kScRun = 8, kScShortRun = 4;     // rows per thread in prompts, when there are many and when there are some

// A thread owns V channels of R consecutive rows.
template <typename T, int TAPS, int R, bool STEP>
__global__ void __launch_bounds__(kScThreads) conv_residual_kernel(ShortConv c, RaggedBatch b, const T* x, size_t ldx, T* out, size_t ldo) {
  constexpr int V = 16 / (int)sizeof(T), H = TAPS - 1;
  __shared__ int cr[R + H], ps[R];
  const int col = (blockIdx.y * kScThreads + threadIdx.x) * V;
  const bool on = col < c.channels;
  ConvWindow<T, V, TAPS, R, STEP> win;
  win.weights(c, on ? col : 0, on);
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.x * R;
  win.load(x, ldx, col, m0, b.rows, on);
  run_rows<R, H>(b, m0, cr, ps);
  __syncthreads();
#pragma unroll
  for (int r = 0; r < R; ++r) {
    if (cr[r + H] < 0) continue;
    float cur[V], y[V];
    win.row(c, col, r, ps[r], cr, on, cur, y);
#pragma unroll
    for (int j = 0; j < V; ++j) y[j] += cur[j];
    if (on) sc_store<T, V>(out + (size_t)(m0 + r) * ldo + col, y);
  }
}

// The same for any number of taps, size and alignment; a thread per V channels of a row.
template <typename T, int V>
__global__ void __launch_bounds__(kScThreads) conv_residual_any_kernel(ShortConv c, RaggedBatch b, int push, const T* x, size_t ldx, T* out, size_t ldo) {
  pdl_wait();
  pdl_launch_dependents();
  const int col = (blockIdx.y * kScThreads + threadIdx.x) * V, m = blockIdx.x;
  const int crow = b.cache_row[m], pos = b.row_pos[m];
  if (col >= c.channels || crow < 0 || (size_t)crow >= b.cache_rows) return;
  float cur[V], y[V];
  sc_load<T, V>(x + (size_t)m * ldx + col, cur);
  conv_any<T, V>(c, x, ldx, col, m, pos, crow, b.cache_row, cur, y);
#pragma unroll
  for (int j = 0; j < V; ++j) y[j] += cur[j];
  sc_store<T, V>(out + (size_t)m * ldo + col, y);
  if (push) sc_push<T, V>(c, col, crow, cur);
}

// Mean over the block's cache rows, one V-piece of one cache (keys, then values) per thread and turn.
template <typename T, int V>
__device__ __forceinline__ void pool_block(const ConvHeads& a, size_t seq0, size_t slot, int block, int first, int step) {
  const int kw = a.kv_heads * a.key_pad / V, vw = a.kv_heads * a.val_pad / V;
  const float inv = 1.0f / (float)a.pool;
  for (int i = first; i < kw + vw; i += step) {
    const bool is_v = i >= kw;
    const int w = is_v ? vw : kw, c = is_v ? i - kw : i;
    const T* src = static_cast<const T*>(is_v ? a.values : a.keys) + (seq0 + (size_t)block * a.pool) * (size_t)w * V + (size_t)c * V;
    float s[V];
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] = 0.f;
    for (int t0 = 0; t0 < a.pool; t0 += 8) {              // eight rows in flight
      float f[8][V];
#pragma unroll
      for (int t = 0; t < 8; ++t) {
        if (t0 + t < a.pool) sc_load<T, V>(src + (size_t)(t0 + t) * w * V, f[t]);
        else
#pragma unroll
          for (int j = 0; j < V; ++j) f[t][j] = 0.f;
      }
#pragma unroll
      for (int t = 0; t < 8; ++t)
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] += f[t][j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s[j] *= inv;
    sc_store<T, V>(static_cast<T*>(is_v ? a.pooled_values : a.pooled_keys) + (slot * a.pool_rows + block) * (size_t)w * V + (size_t)c * V, s);
  }
}

// Cosines and sines of `n` rows: [row][half] each.
__device__ __forceinline__ void row_angles(const Rotation& rot, const int* pos, int n, float* cs, float* sn) {
  const int half = rot.dims / 2;
  for (int i = threadIdx.x; i < n * half; i += blockDim.x) {
    const int r = i / half, d = i - r * half;
    float s, c;
    sincosf((float)pos[r] * rot.freq[d], &s, &c);
    cs[i] = c * rot.mult;
    sn[i] = s * rot.mult;
  }
}

// blockIdx.x: R consecutive rows; the CTA's lane groups (and blockIdx.y's CTAs) share the heads: queries, keys, values.  A head's
// 16-byte pieces sit in the registers of up to 32 lanes, which pass the other half of a pair through shuffles.
template <typename T, int TAPS, int R, bool STEP>
__global__ void __launch_bounds__(256) conv_heads_reg_kernel(ConvHeads a, RaggedBatch b, int lanes) {
  extern __shared__ __align__(16) float sc_smem[];
  constexpr int V = 16 / (int)sizeof(T), H = TAPS - 1;
  __shared__ int cr[R + H], ps[R];
  const int half = a.rot.dims / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  float *cs = sc_smem, *sn = sc_smem + R * half;
  const int l = lane & (lanes - 1), d0 = l * V, per_warp = 32 / lanes, total = a.heads + 2 * a.kv_heads, stride = warps * gridDim.y * per_warp;
  const int m0 = blockIdx.x * R;
  const T* raw = static_cast<const T*>(a.raw);
  const float inv_dim = 1.0f / (float)a.dim;
  const bool turns = d0 < 2 * half, lead = d0 < half;
  const int other = !turns ? lane : lead ? lane + half / V : lane - half / V, p0 = !turns ? 0 : lead ? d0 : d0 - half;
  ConvWindow<T, V, TAPS, R, STEP> win;
  // the lane's head, its kind, its number among the kind, and its first raw column
  int h = (blockIdx.y * warps + warp) * per_warp + lane / lanes;
  bool is_q, is_v, on;
  int col;
  T* dst;                                                 // of row 0 (queries) or cache row 0
  size_t dst_ld;
  auto locate = [&]() {
    is_q = h < a.heads;
    is_v = h >= a.heads + a.kv_heads;
    on = h < total && d0 < (is_v ? a.vdim : a.dim);
    const int g = is_q ? h : is_v ? h - a.heads - a.kv_heads : h - a.heads;
    col = !on ? 0 : is_q ? g * a.dim + d0 : is_v ? a.v0 + g * a.vdim + d0 : a.k0 + g * a.dim + d0;
    dst = d0 + (is_q ? static_cast<T*>(a.q) + (size_t)g * a.dim : is_v ? static_cast<T*>(a.values) + (size_t)g * a.val_pad : static_cast<T*>(a.keys) + (size_t)g * a.key_pad);
    dst_ld = is_q ? a.ldq : (size_t)a.kv_heads * (is_v ? a.val_pad : a.key_pad);
  };
  locate();
  win.weights(a.conv, col, on);
  pdl_wait();
  pdl_launch_dependents();
  win.load(raw, a.ld, col, m0, b.rows, on);
  run_rows<R, H>(b, m0, cr, ps);
  __syncthreads();
  row_angles(a.rot, ps, R, cs, sn);
  __syncthreads();
  for (int first = h - lane / lanes; first < total; first += stride) {     // (the same number of turns for every lane)
    if (first != h - lane / lanes) {
      h = first + lane / lanes;
      locate();
      win.weights(a.conv, col, on);
      win.load(raw, a.ld, col, m0, b.rows, on);
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int crow = cr[r + H];
      if (crow < 0) continue;
      const bool rotates = turns && !is_v;
      float cur[V], y[V], out[V], sq = 0.f;
      win.row(a.conv, col, r, ps[r], cr, on, cur, y);
#pragma unroll
      for (int j = 0; j < V; j += 4) {
        const float4 c4 = *reinterpret_cast<const float4*>(cs + r * half + p0 + j), s4 = *reinterpret_cast<const float4*>(sn + r * half + p0 + j);
        const float c[4] = {c4.x, c4.y, c4.z, c4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float o = __shfl_sync(0xffffffffu, y[j + i], other);
          out[j + i] = rotates ? fmaf(o, lead ? -s[i] : s[i], y[j + i] * c[i]) : y[j + i];
          sq += out[j + i] * out[j + i];
        }
      }
      if (a.norm) {
        for (int o = lanes / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        const float inv = is_v ? 1.0f : rsqrtf(sq * inv_dim + a.eps);
#pragma unroll
        for (int j = 0; j < V; ++j) out[j] *= inv;
      }
      if (on) sc_store<T, V>(dst + (size_t)(is_q ? m0 + r : crow) * dst_ld, out);
    }
  }
  if constexpr (STEP) {
    const int crow = cr[H], pos = ps[0];
    if (a.pool && crow >= 0 && pos > 0 && pos % a.pool == 0)
      pool_block<T, V>(a, (size_t)(crow - pos), (size_t)(crow / a.conv.max_seq), pos / a.pool - 1, blockIdx.y * blockDim.x + threadIdx.x, gridDim.y * blockDim.x);
  }
}

// Any size and alignment: a warp per (row, head), the head in its shared memory.
template <typename T>
__global__ void __launch_bounds__(256) conv_heads_kernel(ConvHeads a, RaggedBatch b, int push) {
  extern __shared__ __align__(16) float sc_smem[];
  const int half = a.rot.dims / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int widest = a.dim > a.vdim ? a.dim : a.vdim;
  float *cs = sc_smem, *sn = cs + half, *vals = sn + half + (size_t)warp * widest;
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, crow = b.cache_row[m], pos = b.row_pos[m];
  if (crow < 0 || (size_t)crow >= b.cache_rows) return;
  row_angles(a.rot, b.row_pos + m, 1, cs, sn);
  __syncthreads();
  const T* raw = static_cast<const T*>(a.raw);
  for (int h = blockIdx.y * warps + warp; h < a.heads + 2 * a.kv_heads; h += warps * gridDim.y) {
    const bool is_q = h < a.heads, is_v = h >= a.heads + a.kv_heads;
    const int g = is_q ? h : is_v ? h - a.heads - a.kv_heads : h - a.heads, dim = is_v ? a.vdim : a.dim;
    const int col0 = is_q ? g * a.dim : is_v ? a.v0 + g * a.vdim : a.k0 + g * a.dim;
    float sq = 0.f;
    for (int d = lane; d < dim; d += 32) {
      float cur[1], y[1];
      sc_load<T, 1>(raw + (size_t)m * a.ld + col0 + d, cur);
      if (a.conv.w) {
        conv_any<T, 1>(a.conv, raw, a.ld, col0 + d, m, pos, crow, b.cache_row, cur, y);
        if (push) sc_push<T, 1>(a.conv, col0 + d, crow, cur);
      } else {
        y[0] = cur[0];
      }
      vals[d] = y[0];
    }
    __syncwarp();
    auto turned = [&](int d) {
      if (is_v || d >= 2 * half) return vals[d];
      const bool lead = d < half;
      const int p = lead ? d : d - half;
      return vals[d] * cs[p] + (lead ? -vals[d + half] : vals[d - half]) * sn[p];
    };
    for (int d = lane; d < dim; d += 32) sq += turned(d) * turned(d);
    const float inv = a.norm && !is_v ? 1.0f / sqrtf(warp_sum(sq) / (float)dim + a.eps) : 1.0f;
    T* dst = is_q ? static_cast<T*>(a.q) + (size_t)m * a.ldq + (size_t)g * a.dim
                  : is_v ? static_cast<T*>(a.values) + ((size_t)crow * a.kv_heads + g) * a.val_pad : static_cast<T*>(a.keys) + ((size_t)crow * a.kv_heads + g) * a.key_pad;
    for (int d = lane; d < dim; d += 32) dst[d] = (T)(turned(d) * inv);
    __syncwarp();
  }
  if (push && a.pool && pos > 0 && pos % a.pool == 0)
    pool_block<T, 1>(a, (size_t)(crow - pos), (size_t)(crow / a.conv.max_seq), pos / a.pool - 1, blockIdx.y * blockDim.x + threadIdx.x, gridDim.y * blockDim.x);
}

// blockIdx: (block of the sequence's share, part of the row, sequence).
template <typename T, int V>
__global__ void __launch_bounds__(128) pool_blocks_kernel(ConvHeads a, RaggedBatch b) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.z, row0 = b.seq_rows[seq], n = b.seq_rows[seq + 1] - row0;
  if (n <= 0 || row0 < 0 || row0 + n > b.rows) return;
  const int c0 = b.cache_row[row0], c1 = b.cache_row[row0 + n - 1], s = b.row_pos[row0];
  if (c0 < s || c1 != c0 + n - 1 || (size_t)c1 >= b.cache_rows) return;
  const int first = s > 0 ? (s + a.pool - 1) / a.pool - 1 : 0, block = first + blockIdx.x;
  if (block >= (s + n - 1) / a.pool) return;
  pool_block<T, V>(a, (size_t)(c0 - s), (size_t)(c0 / a.conv.max_seq), block, blockIdx.y * 128 + threadIdx.x, gridDim.y * 128);
}

struct TailList {
  ConvTail t[kMaxConvTails];
  int n;
};

// A thread per (sequence, channel): reads what it overwrites in ascending order.
template <typename T>
__global__ void __launch_bounds__(kScThreads) conv_tails_kernel(TailList list, RaggedBatch b) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, row0 = b.seq_rows ? b.seq_rows[seq] : seq, n = b.seq_rows ? b.seq_rows[seq + 1] - row0 : 1;
  if (n <= 0 || row0 < 0 || row0 + n > b.rows) return;
  const int c0 = b.cache_row[row0], c1 = b.cache_row[row0 + n - 1], pos = b.row_pos[row0];
  if (c0 < pos || c1 != c0 + n - 1 || (size_t)c1 >= b.cache_rows) return;
  int ch = blockIdx.x * kScThreads + threadIdx.x;
  for (int i = 0; i < list.n; ++i) {
    const ConvTail& t = list.t[i];
    if (ch >= t.c.channels) {
      ch -= t.c.channels;
      continue;
    }
    const int keep = t.c.taps - 1;
    T* st = static_cast<T*>(t.c.state) + (size_t)(c0 / t.c.max_seq) * keep * t.c.channels + ch;
    for (int j = 0; j < keep; ++j) {
      const int at = n - keep + j;                        // the step's row that state row j becomes; negative: an earlier input
      T v;
      if (at >= 0) v = static_cast<const T*>(t.x)[(size_t)(row0 + at) * t.ldx + ch];
      else v = pos + at >= 0 ? st[(size_t)(j + n) * t.c.channels] : (T)0.f;
      st[(size_t)j * t.c.channels] = v;
    }
    return;
  }
}

__global__ void put_conv_kernel(const void* src, int s_dt, float* w, size_t channels, size_t taps, size_t ld, size_t col0) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= channels * taps) return;
  const float v = s_dt == TQ_F32 ? static_cast<const float*>(src)[i] : __bfloat162float(static_cast<const __nv_bfloat16*>(src)[i]);
  w[(i % taps) * ld + col0 + i / taps] = v;
}

template <typename T>
int conv_residual_typed(tq_ctx* ctx, const ShortConv& c, const RaggedBatch& b, const void* x, size_t ldx, void* out, size_t ldo) {
  constexpr int V = 16 / (int)sizeof(T);
  const uintptr_t bits = (uintptr_t)x | (uintptr_t)out | (uintptr_t)c.state;
  const bool vec = c.channels % V == 0 && ldx % V == 0 && ldo % V == 0 && (bits & 15) == 0, step = b.max_q <= 1;
  auto cols = [&](int v) { return (unsigned)((c.channels + v * kScThreads - 1) / (v * kScThreads)); };
  if (!vec || c.taps > kMaxFixedTaps) {
    auto any = [&](auto kern, int v) -> int {
      TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)b.rows, cols(v)), dim3(kScThreads), 0, c, b, (int)step, static_cast<const T*>(x), ldx, static_cast<T*>(out), ldo));
      return TQ_OK;
    };
    return vec ? any(conv_residual_any_kernel<T, V>, V) : any(conv_residual_any_kernel<T, 1>, 1);
  }
  // a few CTAs per SM before a thread takes several rows
  auto fills = [&](int rows) { return !step && (long long)b.rows / rows * cols(V) >= 2ll * ctx->sm_count; };
  const int rows = fills(kScRun) ? kScRun : fills(kScShortRun) ? kScShortRun : 1;
  auto go = [&](auto taps) -> int {
    constexpr int N = decltype(taps)::value;
    auto kern = step ? conv_residual_kernel<T, N, 1, true> : rows == kScRun ? conv_residual_kernel<T, N, kScRun, false>
                : rows == kScShortRun ? conv_residual_kernel<T, N, kScShortRun, false> : conv_residual_kernel<T, N, 1, false>;
    TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)((b.rows + rows - 1) / rows), cols(V)), dim3(kScThreads), 0, c, b, static_cast<const T*>(x), ldx, static_cast<T*>(out), ldo));
    return TQ_OK;
  };
  switch (c.taps) {
    case 1: return go(std::integral_constant<int, 1>());
    case 2: return go(std::integral_constant<int, 2>());
    case 3: return go(std::integral_constant<int, 3>());
    default: return go(std::integral_constant<int, 4>());
  }
}

template <typename T>
int conv_heads_typed(tq_ctx* ctx, const ConvHeads& a, const RaggedBatch& b) {
  constexpr int V = 16 / (int)sizeof(T);
  const int push = b.max_q <= 1, total = a.heads + 2 * a.kv_heads, widest = a.dim > a.vdim ? a.dim : a.vdim, half = a.rot.dims / 2;
  const uintptr_t bits = (uintptr_t)a.raw | (uintptr_t)a.q | (uintptr_t)a.keys | (uintptr_t)a.values | (uintptr_t)a.conv.state;
  const bool vec = a.dim % V == 0 && a.vdim % V == 0 && a.rot.dims % (2 * V) == 0 && a.ld % V == 0 && a.ldq % V == 0 && a.k0 % V == 0 && a.v0 % V == 0 &&
                   a.conv.channels % V == 0 && widest / V <= 32 && (bits & 15) == 0 && a.conv.w && a.conv.taps <= kMaxFixedTaps;
  if (vec) {
    int lanes = 1;
    while (lanes < widest / V) lanes *= 2;
    const int units = (total + 32 / lanes - 1) / (32 / lanes);
    auto fills = [&](int n, int per_sm) { return !push && (long long)b.rows / n * units >= (long long)per_sm * ctx->sm_count; };
    const int rows = fills(kScRun, 8) ? kScRun : fills(kScShortRun, 6) ? kScShortRun : 1;
    const int parts = (units + 7) / 8, warps = (units + parts - 1) / parts;      // up to eight warps, all of them with heads
    const long long blocks = (b.rows + rows - 1) / rows;
    int y = 1;                                            // a head per warp when the rows alone do not fill the GPU
    while (y * warps < units && blocks * y < 4ll * ctx->sm_count) ++y;
    const size_t smem = ((size_t)rows * a.rot.dims + V) * sizeof(float);
    auto go = [&](auto taps) -> int {
      constexpr int N = decltype(taps)::value;
      auto kern = push ? conv_heads_reg_kernel<T, N, 1, true> : rows == kScRun ? conv_heads_reg_kernel<T, N, kScRun, false>
                  : rows == kScShortRun ? conv_heads_reg_kernel<T, N, kScShortRun, false> : conv_heads_reg_kernel<T, N, 1, false>;
      TQ_CUDA(ctx, launch_k(ctx, kern, dim3((unsigned)blocks, (unsigned)y), dim3((unsigned)(32 * warps)), smem, a, b, lanes));
      return TQ_OK;
    };
    switch (a.conv.taps) {
      case 1: return go(std::integral_constant<int, 1>());
      case 2: return go(std::integral_constant<int, 2>());
      case 3: return go(std::integral_constant<int, 3>());
      default: return go(std::integral_constant<int, 4>());
    }
  }
  const int warps = total < 8 ? total : 8;
  int y = 1;
  while (y * warps < total && (long long)b.rows * y < 2ll * ctx->sm_count) ++y;
  const size_t smem = ((size_t)2 * half + (size_t)warps * widest) * sizeof(float);
  TQ_REQUIRE(ctx, smem <= 200 * 1024, "convolved heads: heads of %d values are too large", widest);
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(conv_heads_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, conv_heads_kernel<T>, dim3((unsigned)b.rows, (unsigned)y), dim3((unsigned)(32 * warps)), smem, a, b, push));
  return TQ_OK;
}

}  // namespace

int put_conv_weights(tq_ctx* ctx, const void* src, int src_dtype, float* w, size_t channels, size_t taps, size_t ld, size_t col0) {
  const size_t bytes = channels * taps * dtype_size(src_dtype);
  void* tmp = nullptr;
  TQ_CUDA(ctx, cudaMalloc(&tmp, bytes));
  cudaError_t e = cudaMemcpyAsync(tmp, src, bytes, cudaMemcpyDefault, ctx->stream);
  if (e == cudaSuccess) {
    put_conv_kernel<<<(unsigned)((channels * taps + 255) / 256), 256, 0, ctx->stream>>>(tmp, src_dtype, w, channels, taps, ld, col0);
    ctx->launches++;
    e = cudaGetLastError();
  }
  if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
  cudaFree(tmp);
  TQ_CUDA(ctx, e);
  return TQ_OK;
}

int launch_conv_residual(tq_ctx* ctx, const ShortConv& c, const RaggedBatch& b, int dtype, const void* x, size_t ldx, void* out, size_t ldo) {
  TQ_REQUIRE(ctx, c.taps >= 1 && c.channels > 0 && c.w && (c.state || c.taps == 1) && c.max_seq > 0 && x != out, "short convolution: bad sizes");
  if (b.rows == 0) return TQ_OK;
  return dtype == TQ_F32 ? conv_residual_typed<float>(ctx, c, b, x, ldx, out, ldo) : conv_residual_typed<__nv_bfloat16>(ctx, c, b, x, ldx, out, ldo);
}

int launch_conv_heads(tq_ctx* ctx, const ConvHeads& a, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, a.heads > 0 && a.kv_heads > 0 && a.dim > 0 && a.vdim > 0 && a.key_pad >= a.dim && a.val_pad >= a.vdim && a.key_pad % 8 == 0 && a.val_pad % 8 == 0,
             "convolved heads: bad head sizes");
  TQ_REQUIRE(ctx, a.rot.dims >= 0 && a.rot.dims % 2 == 0 && a.rot.dims <= a.dim, "convolved heads: the rotated dimensions must be even and inside the head");
  TQ_REQUIRE(ctx, a.conv.taps >= 1 && a.conv.max_seq > 0 && (!a.conv.w || a.conv.taps == 1 || a.conv.state), "convolved heads: bad convolution");
  TQ_REQUIRE(ctx, a.pool == 0 || (a.pool > 0 && a.pooled_keys && a.pooled_values), "convolved heads: nowhere to put the pooled blocks");
  if (b.rows == 0) return TQ_OK;
  if (int st = dtype == TQ_F32 ? conv_heads_typed<float>(ctx, a, b) : conv_heads_typed<__nv_bfloat16>(ctx, a, b)) return st;
  if (!a.pool || b.max_q <= 1 || b.max_len <= a.pool) return TQ_OK;
  // (16-byte pieces: the padded heads are multiples of eight values and the caches come from the allocator)
  const int pieces = a.kv_heads * (a.key_pad + a.val_pad) / (dtype == TQ_F32 ? 4 : 8);
  const dim3 grid((unsigned)(b.max_q / a.pool + 2), (unsigned)((pieces + 127) / 128), (unsigned)b.n_seqs);
  if (dtype == TQ_F32) TQ_CUDA(ctx, launch_k(ctx, pool_blocks_kernel<float, 4>, grid, dim3(128), 0, a, b));
  else TQ_CUDA(ctx, launch_k(ctx, pool_blocks_kernel<__nv_bfloat16, 8>, grid, dim3(128), 0, a, b));
  return TQ_OK;
}

int launch_conv_tails(tq_ctx* ctx, const ConvTail* tails, int n, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, n >= 0 && n <= kMaxConvTails, "convolution states: at most %d at a time", kMaxConvTails);
  TailList list;
  list.n = 0;
  int channels = 0;
  for (int i = 0; i < n; ++i)
    if (tails[i].c.w && tails[i].c.taps > 1) {
      list.t[list.n++] = tails[i];
      channels += tails[i].c.channels;
    }
  if (list.n == 0 || b.n_seqs == 0) return TQ_OK;
  TQ_REQUIRE(ctx, b.n_seqs <= 65535, "convolution states: too many sequences");
  const dim3 grid((unsigned)((channels + kScThreads - 1) / kScThreads), (unsigned)b.n_seqs);
  if (dtype == TQ_F32) TQ_CUDA(ctx, launch_k(ctx, conv_tails_kernel<float>, grid, dim3(kScThreads), 0, list, b));
  else TQ_CUDA(ctx, launch_k(ctx, conv_tails_kernel<__nv_bfloat16>, grid, dim3(kScThreads), 0, list, b));
  return TQ_OK;
}

}  // namespace tq

using namespace tq;

static RaggedBatch conv_batch(const int* seq_rows, const int* row_pos, const int* cache_row, size_t n_seqs, size_t rows, size_t max_q, size_t max_len, size_t cache_rows) {
  RaggedBatch b;
  b.n_seqs = (int)n_seqs;
  b.rows = (int)rows;
  b.max_q = (int)max_q;
  b.max_len = (int)max_len;
  b.seq_rows = seq_rows;
  b.row_pos = row_pos;
  b.cache_row = cache_row;
  b.cache_rows = cache_rows;
  return b;
}

extern "C" int tq_conv_residual(tq_ctx* ctx, int dtype, size_t channels, size_t taps, const float* w_dev, void* state_dev, size_t max_seq, size_t cache_rows,
                                const void* x_dev, size_t ldx, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs,
                                size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_F32 || dtype == TQ_BF16, "tq_conv_residual: dtype must be f32 or bf16");
  TQ_REQUIRE(ctx, x_dev && out_dev && row_pos_dev && cache_row_dev && (seq_rows_dev || (rows == n_seqs && max_q == 1)), "tq_conv_residual: null pointer");
  ConvTail t;
  t.c.taps = (int)taps;
  t.c.channels = (int)channels;
  t.c.w = w_dev;
  t.c.state = state_dev;
  t.c.max_seq = (int)max_seq;
  t.x = x_dev;
  t.ldx = ldx;
  const RaggedBatch b = conv_batch(seq_rows_dev, row_pos_dev, cache_row_dev, n_seqs, rows, max_q, max_len, cache_rows);
  if (int st = launch_conv_residual(ctx, t.c, b, dtype, x_dev, ldx, out_dev, ldo)) return st;
  return b.max_q > 1 ? launch_conv_tails(ctx, &t, 1, b, dtype) : TQ_OK;
}

extern "C" int tq_conv_heads(tq_ctx* ctx, const tq_conv_heads_config* cfg, int dtype, const void* raw_dev, size_t ld, const float* w_dev, void* state_dev,
                             const float* freq_dev, size_t max_seq, size_t cache_rows, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev,
                             size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* q_dev, size_t ldq, void* keys_dev, void* values_dev,
                             void* pooled_keys_dev, void* pooled_values_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && (dtype == TQ_F32 || dtype == TQ_BF16), "tq_conv_heads: dtype must be f32 or bf16");
  TQ_REQUIRE(ctx, raw_dev && q_dev && keys_dev && values_dev && row_pos_dev && cache_row_dev && (freq_dev || cfg->rot_dims == 0) &&
                      (seq_rows_dev || (rows == n_seqs && max_q == 1)),
             "tq_conv_heads: null pointer");
  ConvHeads a;
  a.heads = (int)cfg->heads;
  a.kv_heads = (int)cfg->kv_heads;
  a.dim = (int)cfg->dim;
  a.vdim = (int)cfg->vdim;
  a.key_pad = (int)((cfg->dim + 7) / 8 * 8);
  a.val_pad = (int)((cfg->vdim + 7) / 8 * 8);
  a.raw = raw_dev;
  a.ld = ld;
  a.k0 = (int)cfg->k0;
  a.v0 = (int)cfg->v0;
  a.conv.taps = w_dev ? (int)cfg->taps : 1;
  a.conv.channels = (int)cfg->channels;
  a.conv.w = w_dev;
  a.conv.state = state_dev;
  a.conv.max_seq = (int)max_seq;
  a.rot.dims = (int)cfg->rot_dims;
  a.rot.freq = freq_dev;
  a.rot.mult = cfg->rot_mult;
  a.norm = cfg->norm != 0;
  a.eps = cfg->eps;
  a.q = q_dev;
  a.ldq = ldq;
  a.keys = keys_dev;
  a.values = values_dev;
  a.pool = (int)cfg->pool;
  a.pool_rows = (int)cfg->pool_rows;
  a.pooled_keys = pooled_keys_dev;
  a.pooled_values = pooled_values_dev;
  ConvTail t;
  t.c = a.conv;
  t.x = raw_dev;
  t.ldx = ld;
  const RaggedBatch b = conv_batch(seq_rows_dev, row_pos_dev, cache_row_dev, n_seqs, rows, max_q, max_len, cache_rows);
  if (int st = launch_conv_heads(ctx, a, b, dtype)) return st;
  return b.max_q > 1 ? launch_conv_tails(ctx, &t, 1, b, dtype) : TQ_OK;
}
