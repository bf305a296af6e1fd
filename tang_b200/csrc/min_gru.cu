// minGRU (see min_gru.cuh).  A thread owns two neighbouring channels.
//   * one row per sequence: one pass over the state;
//   * prompts: a CTA owns 16 channels of a sequence and walks it in tiles of 256 rows.  Each of its 64 row groups reads four rows
//     once, reduces them to an affine map of the state, a warp per channel scans the 64 maps through shuffles, and every group
//     finishes its rows from the state ahead of them, still in registers.
#include "min_gru.cuh"

#include <cuda_bf16.h>

#include "common.cuh"

namespace tq {

namespace {

constexpr int kMgLanes = 8, kMgGroups = 64, kMgRows = 4;         // channel pairs, row groups of a CTA, rows of a group
constexpr int kMgThreads = kMgLanes * kMgGroups, kMgChannels = 2 * kMgLanes, kMgTile = kMgGroups * kMgRows;
static_assert(kMgGroups == 64 && kMgThreads >= 32 * kMgChannels, "a warp scans a channel's 64 maps");

// sigmoid(z), sigmoid(u) and sigmoid(g).  bf16 models take approximate exponentials and one quotient for the three (about 2^-21, the
// arguments carry 2^-9); its denominator stays finite because below -28 a sigmoid is 7e-13 all the same.
template <typename T>
__device__ __forceinline__ void mg_sigmoids(float z, float u, float g, float& sz, float& su, float& sg) {
  if constexpr (sizeof(T) == 4) {
    sz = 1.0f / (1.0f + expf(-z));
    su = 1.0f / (1.0f + expf(-u));
    sg = 1.0f / (1.0f + expf(-g));
  } else {
    const float a = 1.0f + __expf(fminf(-z, 28.f)), b = 1.0f + __expf(fminf(-u, 28.f)), c = 1.0f + __expf(fminf(-g, 28.f));
    const float ab = a * b, r = __fdividef(1.0f, ab * c), rc = r * c;
    sz = rc * b;
    su = rc * a;
    sg = r * ab;
  }
}

// A pair of channels as it is stored, and its values (the second is 0 if there is none).
__device__ __forceinline__ float2 mg_raw(const float* p, bool two) { return two ? *reinterpret_cast<const float2*>(p) : make_float2(*p, 0.f); }
__device__ __forceinline__ uint32_t mg_raw(const __nv_bfloat16* p, bool two) {
  return two ? *reinterpret_cast<const uint32_t*>(p) : (uint32_t)*reinterpret_cast<const uint16_t*>(p);
}
__device__ __forceinline__ float2 mg_pair(float2 v) { return v; }
__device__ __forceinline__ float2 mg_pair(uint32_t w) { return make_float2(bf16_bits_to_float(w & 0xFFFFu), bf16_bits_to_float(w >> 16)); }
template <typename T>
__device__ __forceinline__ float2 mg_load(const T* p, bool two) {
  return mg_pair(mg_raw(p, two));
}
__device__ __forceinline__ void mg_store(float* p, float2 v, bool two) {
  if (two) *reinterpret_cast<float2*>(p) = v;
  else *p = v.x;
}
__device__ __forceinline__ void mg_store(__nv_bfloat16* p, float2 v, bool two) {
  if (two) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
  else *p = __float2bfloat16_rn(v.x);
}

// One row as an affine map of the state, S <- a S + b, and the factor q of its output.
template <typename T>
__device__ __forceinline__ void mg_row(float z, float u, float g, float scale, float& a, float& b, float& q) {
  float sz, su, sg;
  mg_sigmoids<T>(z, u, g, sz, su, sg);
  a = 1.0f - sz;
  b = sz * (u >= 0.f ? u + 0.5f : su);
  q = g * sg * scale;
}

struct MgSeq {
  int row0, n;
  size_t slot;
  bool fresh;
};
__device__ __forceinline__ bool mg_sequence(const MinGru& g, const RaggedBatch& b, int seq, MgSeq& s) {
  s.row0 = b.seq_rows ? b.seq_rows[seq] : seq;
  s.n = b.seq_rows ? b.seq_rows[seq + 1] - s.row0 : 1;
  if (s.n <= 0 || s.row0 < 0 || s.row0 + s.n > b.rows) return false;
  const int c0 = b.cache_row[s.row0], c1 = b.cache_row[s.row0 + s.n - 1];
  if (c0 < 0 || c1 != c0 + s.n - 1 || (size_t)c1 >= b.cache_rows) return false;    // (reported by the embedding kernel)
  s.slot = (size_t)(c0 / g.max_seq);
  s.fresh = b.row_pos[s.row0] == 0;
  return true;
}

template <typename T>
__global__ void __launch_bounds__(128) min_gru_step_kernel(MinGru g, MinGruRows r, RaggedBatch b) {
  const int c = 2 * (blockIdx.x * 128 + threadIdx.x);
  const bool on = c < g.width, two = c + 1 < g.width;
  float2 zb = make_float2(0.f, 0.f), ub = zb;
  if (on) zb = mg_load(g.z_bias + c, two), ub = mg_load(g.u_bias + c, two);       // (weights: before the wait)
  pdl_wait();
  pdl_launch_dependents();
  MgSeq s;
  if (!on || !mg_sequence(g, b, blockIdx.y, s)) return;
  const size_t at = (size_t)s.row0 * r.ld + c;
  const float2 z = mg_load(static_cast<const T*>(r.z) + at, two), u = mg_load(static_cast<const T*>(r.u) + at, two), gt = mg_load(static_cast<const T*>(r.gate) + at, two);
  float2* st = reinterpret_cast<float2*>(g.state + s.slot * ((g.width + 1) / 2 * 2) + c);
  float2 S = s.fresh ? make_float2(0.f, 0.f) : *st;
  float a0, b0, q0, a1, b1, q1;
  mg_row<T>(z.x + zb.x, u.x + ub.x, gt.x, g.out_scale, a0, b0, q0);
  mg_row<T>(z.y + zb.y, u.y + ub.y, gt.y, g.out_scale, a1, b1, q1);
  S.x = fmaf(a0, S.x, b0);
  S.y = fmaf(a1, S.y, b1);
  *st = S;
  mg_store(static_cast<T*>(r.out) + (size_t)s.row0 * r.ldo + c, make_float2(S.x * q0, S.y * q1), two);
}

// EVEN: an even width, so that no pair of channels is cut.
template <typename T, bool EVEN>
__global__ void __launch_bounds__(kMgThreads, 2) min_gru_scan_kernel(MinGru g, MinGruRows r, RaggedBatch b) {
  // [group][channel]: the group's map, then the state ahead of the group
  __shared__ float ma[kMgGroups][kMgChannels + 1], mb[kMgGroups][kMgChannels + 1], carry[kMgChannels];
  const int pair = threadIdx.x % kMgLanes, group = threadIdx.x / kMgLanes, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cl = 2 * pair, c = blockIdx.x * kMgChannels + cl;
  const bool on = c < g.width, two = EVEN || c + 1 < g.width;
  float2 zb = make_float2(0.f, 0.f), ub = zb;
  if (on) zb = mg_load(g.z_bias + c, two), ub = mg_load(g.u_bias + c, two);
  pdl_wait();
  pdl_launch_dependents();
  MgSeq s;
  if (!mg_sequence(g, b, blockIdx.y, s)) return;
  float* st = g.state + s.slot * ((g.width + 1) / 2 * 2) + blockIdx.x * kMgChannels;
  const int n_ch = min(kMgChannels, g.width - (int)blockIdx.x * kMgChannels);
  if ((int)threadIdx.x < kMgChannels) carry[threadIdx.x] = (int)threadIdx.x < n_ch && !s.fresh ? st[threadIdx.x] : 0.f;
  // (idle lanes read the first pair's rows)
  const size_t col = on ? c : 0;
  const T *zp = static_cast<const T*>(r.z) + col, *up = static_cast<const T*>(r.u) + col, *gp = static_cast<const T*>(r.gate) + col;
  T* op = static_cast<T*>(r.out) + c;
  decltype(mg_raw(zp, true)) z[kMgRows], u[kMgRows], gt[kMgRows];
  auto load = [&](int t0) {
#pragma unroll
    for (int i = 0; i < kMgRows; ++i) {                   // (rows behind the end: the last one again)
      const size_t at = (size_t)(s.row0 + min(t0 + group * kMgRows + i, s.n - 1)) * r.ld;
      z[i] = mg_raw(zp + at, two);
      u[i] = mg_raw(up + at, two);
      gt[i] = mg_raw(gp + at, two);
    }
  };
  load(0);
  for (int t0 = 0; t0 < s.n; t0 += kMgTile) {
    float2 a[kMgRows], d[kMgRows], q[kMgRows], A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < kMgRows; ++i) {
      const float2 zi = mg_pair(z[i]), ui = mg_pair(u[i]), gi = mg_pair(gt[i]);
      mg_row<T>(zi.x + zb.x, ui.x + ub.x, gi.x, g.out_scale, a[i].x, d[i].x, q[i].x);
      mg_row<T>(zi.y + zb.y, ui.y + ub.y, gi.y, g.out_scale, a[i].y, d[i].y, q[i].y);
      if (t0 + group * kMgRows + i >= s.n) {              // rows behind the end leave the state alone
        a[i] = make_float2(1.f, 1.f);
        d[i] = make_float2(0.f, 0.f);
      }
      A.x *= a[i].x;
      A.y *= a[i].y;
      B.x = fmaf(a[i].x, B.x, d[i].x);
      B.y = fmaf(a[i].y, B.y, d[i].y);
    }
    if (t0 + kMgTile < s.n) load(t0 + kMgTile);           // under the scan
    ma[group][cl] = A.x, ma[group][cl + 1] = A.y;
    mb[group][cl] = B.x, mb[group][cl + 1] = B.y;
    __syncthreads();
    if (warp < kMgChannels) {                             // a warp per channel, a lane per two groups
      const float a0 = ma[2 * lane][warp], b0 = mb[2 * lane][warp], a1 = ma[2 * lane + 1][warp], b1 = mb[2 * lane + 1][warp], S0 = carry[warp];
      float sa = a1 * a0, sb = fmaf(a1, b0, b1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {                  // maps up to this lane's, composed
        const float pa = __shfl_up_sync(0xffffffffu, sa, o), pb = __shfl_up_sync(0xffffffffu, sb, o);
        if (lane >= o) {
          sb = fmaf(sa, pb, sb);
          sa *= pa;
        }
      }
      const float S = fmaf(sa, S0, sb);
      float ahead = __shfl_up_sync(0xffffffffu, S, 1);
      if (lane == 0) ahead = S0;
      __syncwarp();
      mb[2 * lane][warp] = ahead;
      mb[2 * lane + 1][warp] = fmaf(a0, ahead, b0);
      if (lane == 31) carry[warp] = S;
    }
    __syncthreads();
    float2 S = make_float2(mb[group][cl], mb[group][cl + 1]);
#pragma unroll
    for (int i = 0; i < kMgRows; ++i) {
      const int row = t0 + group * kMgRows + i;
      S.x = fmaf(a[i].x, S.x, d[i].x);
      S.y = fmaf(a[i].y, S.y, d[i].y);
      if (on && row < s.n) mg_store(op + (size_t)(s.row0 + row) * r.ldo, make_float2(S.x * q[i].x, S.y * q[i].y), two);
    }
    __syncthreads();                                      // the maps are rewritten by the next tile
  }
  if ((int)threadIdx.x < n_ch) st[threadIdx.x] = carry[threadIdx.x];
}

template <typename T>
int min_gru_typed(tq_ctx* ctx, const MinGru& g, const MinGruRows& r, const RaggedBatch& b) {
  if (b.max_q <= 1)
    TQ_CUDA(ctx, launch_k(ctx, min_gru_step_kernel<T>, dim3((unsigned)((g.width + 255) / 256), (unsigned)b.n_seqs), dim3(128), 0, g, r, b));
  else
    TQ_CUDA(ctx, launch_k(ctx, g.width % 2 ? min_gru_scan_kernel<T, false> : min_gru_scan_kernel<T, true>,
                          dim3((unsigned)((g.width + kMgChannels - 1) / kMgChannels), (unsigned)b.n_seqs), dim3(kMgThreads), 0, g, r, b));
  return TQ_OK;
}

}  // namespace

int launch_min_gru(tq_ctx* ctx, const MinGru& g, const MinGruRows& r, const RaggedBatch& b, int dtype) {
  TQ_REQUIRE(ctx, g.width > 0 && g.max_seq > 0 && g.z_bias && g.u_bias && g.state, "minGRU: bad sizes");
  const size_t es = dtype_size(dtype);
  TQ_REQUIRE(ctx, r.ld % 2 == 0 && r.ldo % 2 == 0 && (((uintptr_t)r.z | (uintptr_t)r.u | (uintptr_t)r.gate | (uintptr_t)r.out) & (2 * es - 1)) == 0,
             "minGRU: rows must start on even elements");
  TQ_REQUIRE(ctx, b.n_seqs <= 65535, "minGRU: too many sequences");
  if (b.rows == 0 || b.n_seqs == 0) return TQ_OK;
  return dtype == TQ_F32 ? min_gru_typed<float>(ctx, g, r, b) : min_gru_typed<__nv_bfloat16>(ctx, g, r, b);
}

}  // namespace tq

using namespace tq;

extern "C" int tq_min_gru(tq_ctx* ctx, int dtype, size_t width, const void* z_dev, const void* u_dev, const void* gate_dev, size_t ld, const float* z_bias_dev,
                          const float* u_bias_dev, float out_scale, float* state_dev, size_t max_seq, size_t cache_rows, const int* seq_rows_dev, const int* row_pos_dev,
                          const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_F32 || dtype == TQ_BF16, "tq_min_gru: dtype must be f32 or bf16");
  TQ_REQUIRE(ctx, z_dev && u_dev && gate_dev && row_pos_dev && cache_row_dev && out_dev, "tq_min_gru: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || (rows == n_seqs && max_q == 1), "tq_min_gru: without row offsets every sequence brings one row");
  MinGru g;
  g.width = (int)width;
  g.z_bias = z_bias_dev;
  g.u_bias = u_bias_dev;
  g.out_scale = out_scale;
  g.state = state_dev;
  g.max_seq = (int)max_seq;
  MinGruRows r;
  r.z = z_dev;
  r.u = u_dev;
  r.gate = gate_dev;
  r.ld = ld;
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
  return launch_min_gru(ctx, g, r, b, dtype);
}
