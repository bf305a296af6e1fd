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
#include <type_traits>

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
    const int row0 = max(b.seq_rows ? b.seq_rows[seq] : seq, 0), end = min(b.seq_rows ? b.seq_rows[seq + 1] : seq + 1, b.rows), off = p.off[seq];
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

// ------------------------------------------------------------------------------------------------ one query per sequence
constexpr int kLdTile = 64, kLdThreads = 128;             // positions of a cache tile; threads per head tile
constexpr int kLdPRow = kLdTile * 2 + 16;                 // bytes of a row of weights
constexpr int kLdMaxSplits = 64;

struct LatentDecodeParams {
  LatentDims d;
  RaggedBatch b;
  const int* single;
  const __nv_bfloat16 *q_lat, *q, *cache;
  size_t ldq;
  __nv_bfloat16* out;
  float scale;
  Rotation rot;
  int rotate, n_splits;
  float* part_o;                                          // [n_seqs][heads][n_splits][c_pad]
  float* part_ml;                                         // [n_seqs][heads][n_splits][2]
};

// VT: 8-column tiles of latents per warp (c_pad <= 32 VT); HT: head tiles per CTA; FULL: c_pad = 32 VT; ROW: elements of a cache row (0: any).
template <int VT, int HT, bool FULL, int ROW = 0>
__global__ void __launch_bounds__(kLdThreads * HT) latent_decode_kernel(const __grid_constant__ LatentDecodeParams p) {
  extern __shared__ __align__(128) uint8_t ld_smem[];
  static_assert(kLdTile * (ROW / 8) % (kLdThreads * HT) == 0, "whole rounds of copies");
  constexpr int kThreads = kLdThreads * HT;
  const int row_el = ROW ? ROW : p.d.row();
  const int row_bytes = row_el * 2 + 16;               // an odd number of 16-byte groups: ldmatrix rows do not meet in a bank
  const int ht = threadIdx.x >> 7, warp = (threadIdx.x >> 5) & 3, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  uint8_t* q_s = ld_smem + (size_t)ht * 16 * row_bytes;
  uint8_t* kv_s = ld_smem + (size_t)HT * 16 * row_bytes;
  uint8_t* p_s = kv_s + (size_t)2 * kLdTile * row_bytes + (size_t)ht * 2 * 16 * kLdPRow;      // [terms][16][kLdPRow]
  float* mw = reinterpret_cast<float*>(kv_s + (size_t)2 * kLdTile * row_bytes + (size_t)HT * 2 * 16 * kLdPRow) + ht * 64;   // [4 warps][16] maxima
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.z, head0 = (blockIdx.y * HT + ht) * 16;
  const int row = p.single ? p.single[seq] : seq;
  if (row < 0) return;
  const int pos = p.b.row_pos[row], crow = p.b.cache_row[row];
  if (crow < pos || (size_t)crow >= p.b.cache_rows) return;
  const __nv_bfloat16* base = p.cache + (size_t)(crow - pos) * row_el;
  const int tiles = pos / kLdTile + 1, per = (tiles + p.n_splits - 1) / p.n_splits;
  const int t0 = min((int)blockIdx.x * per, tiles), t1 = min(t0 + per, tiles);
  const int chunks = row_el / 8;
  const int step_r = kThreads / chunks, step_c = kThreads % chunks, first_r = threadIdx.x / chunks, first_c = threadIdx.x % chunks;
  const uint32_t kv_u = smem_u32(kv_s);

  auto load_tile = [&](int tile, int buf) {
    const int n_valid = pos + 1 - tile * kLdTile;          // rows at or beyond it become zeros
    const __nv_bfloat16* src = base + (size_t)tile * kLdTile * row_el;
    const uint32_t dst = kv_u + (uint32_t)(buf * kLdTile * row_bytes);
    if constexpr (ROW != 0) {
#pragma unroll
      for (int i = 0; i < kLdTile * (ROW / 8) / kThreads; ++i) {
        const int at = i * kThreads + threadIdx.x, r = at / (ROW / 8), c = at % (ROW / 8);
        const bool ok = r < n_valid;
        cp_async16(dst + (uint32_t)(r * row_bytes + c * 16), ok ? src + at * 8 : base, ok);
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
      return;
    }
    int r = first_r, c = first_c;
    while (r < kLdTile) {
      const bool ok = r < n_valid;
      cp_async16(dst + (uint32_t)(r * row_bytes + c * 16), ok ? src + r * row_el + c * 8 : base, ok);
      r += step_r;
      c += step_c;
      if (c >= chunks) {
        c -= chunks;
        ++r;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 < t1) load_tile(t0, 0);

  // ---- queries: [latent | rotated part] of 16 heads
  for (int i = threadIdx.x & 127; i < 16 * p.d.c_pad / 2; i += kLdThreads) {
    const int r = i / (p.d.c_pad / 2), c = 2 * (i - r * (p.d.c_pad / 2));
    uint32_t v = 0u;
    if (head0 + r < p.d.heads) {
      v = *reinterpret_cast<const uint32_t*>(p.q_lat + ((size_t)(head0 + r) * p.b.n_seqs + seq) * p.d.c_pad + c);
      if (c + 1 >= p.d.rank) v = c < p.d.rank ? v & 0xFFFFu : 0u;
    }
    *reinterpret_cast<uint32_t*>(q_s + (size_t)r * row_bytes + 2 * c) = v;
  }
  for (int i = threadIdx.x & 127; i < 16 * p.d.r_pad / 2; i += kLdThreads) {
    const int r = i / (p.d.r_pad / 2), c = 2 * (i - r * (p.d.r_pad / 2));
    float u = 0.f, v = 0.f;
    if (head0 + r < p.d.heads) {
      const __nv_bfloat16* src = p.q + ((size_t)(head0 + r) * p.b.n_seqs + seq) * p.ldq + p.d.dim;
      if (c < p.d.rot) u = __bfloat162float(src[c]);
      if (c + 1 < p.d.rot) v = __bfloat162float(src[c + 1]);
      if (p.rotate && c < p.rot.dims) {
        float s, co;
        sincosf((float)pos * p.rot.freq[c / 2], &s, &co);
        s *= p.rot.mult;
        co *= p.rot.mult;
        const float x = u * co - v * s;
        v = v * co + u * s;
        u = x;
      }
    }
    *reinterpret_cast<uint32_t*>(q_s + (size_t)r * row_bytes + 2 * (p.d.c_pad + c)) = pack_bf16(u, v);
  }

  float o[VT][4];                                         // latent columns 8 (VT warp + j) + 2t, +1; heads g, then g + 8
#pragma unroll
  for (int j = 0; j < VT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  const float scale2 = p.scale * kLog2e;
  const int nks = row_el / 16, col0 = 8 * VT * warp;
  const int n_vt = max(0, min(VT, (p.d.c_pad - col0) / 8));   // this warp's tiles (an even number)

  for (int tile = t0; tile < t1; ++tile) {
    const int buf = (tile - t0) & 1;
    if (tile + 1 < t1) {
      load_tile(tile + 1, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint8_t* kt = kv_s + (size_t)buf * kLdTile * row_bytes;
    const int key0 = tile * kLdTile + 16 * warp;
    float s[2][4] = {};
    {
      const uint8_t* qa = q_s + (size_t)(lane & 15) * row_bytes + 16 * (lane >> 4);
      const uint8_t* ka = kt + (size_t)(16 * warp + 8 * (lane >> 4) + (lane & 7)) * row_bytes + 16 * ((lane >> 3) & 1);
#pragma unroll 4
      for (int ks = 0; ks < nks; ++ks) {
        uint32_t a[4], kb[4];
        ldmatrix4(a, qa + 32 * ks);
        ldmatrix4(kb, ka + 32 * ks);
        mma_bf16_16816(s[0], a[0], a[1], a[2], a[3], kb[0], kb[1]);
        mma_bf16_16816(s[1], a[0], a[1], a[2], a[3], kb[2], kb[3]);
      }
    }
    float mx[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        s[n][c] = key0 + 8 * n + 2 * t + (c & 1) <= pos ? s[n][c] * scale2 : -FLT_MAX;
        mx[c >> 1] = fmaxf(mx[c >> 1], s[n][c]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
    }
    if (t == 0) {
      mw[warp * 16 + g] = mx[0];
      mw[warp * 16 + g + 8] = mx[1];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int hr = g + 8 * r;
      const float mn = fmaxf(m_run[r], fmaxf(fmaxf(mw[hr], mw[16 + hr]), fmaxf(mw[32 + hr], mw[48 + hr])));   // (finite: a tile has a visible key)
      alpha[r] = ex2_ftz(m_run[r] - mn);
      m_run[r] = mn;
      float w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) w[i] = ex2_ftz(s[i >> 1][2 * r + (i & 1)] - mn);
      l_run[r] = l_run[r] * alpha[r] + ((w[0] + w[1]) + (w[2] + w[3]));
      uint32_t hi, lo;
      uint8_t* pr = p_s + (size_t)hr * kLdPRow + 2 * (16 * warp + 2 * t);
      split_bf16(w[0], w[1], hi, lo);
      *reinterpret_cast<uint32_t*>(pr) = hi;
      *reinterpret_cast<uint32_t*>(pr + 16 * kLdPRow) = lo;
      split_bf16(w[2], w[3], hi, lo);
      *reinterpret_cast<uint32_t*>(pr + 16) = hi;
      *reinterpret_cast<uint32_t*>(pr + 16 * kLdPRow + 16) = lo;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < VT; ++j) {
      o[j][0] *= alpha[0];
      o[j][1] *= alpha[0];
      o[j][2] *= alpha[1];
      o[j][3] *= alpha[1];
    }
    const uint8_t* pa = p_s + (size_t)(lane & 15) * kLdPRow + 16 * (lane >> 4);
    const uint8_t* va = kt + (size_t)(lane & 15) * row_bytes + 16 * (lane >> 4) + 2 * col0;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t ah[4], al[4];
      ldmatrix4(ah, pa + 32 * ks);
      ldmatrix4(al, pa + 16 * kLdPRow + 32 * ks);
#pragma unroll
      for (int j = 0; j < VT; j += 2) {
        if (FULL || j < n_vt) {
          uint32_t vb[4];
          ldmatrix4_t(vb, va + (size_t)16 * ks * row_bytes + 16 * j);
          mma_bf16_16816(o[j], ah[0], ah[1], ah[2], ah[3], vb[0], vb[1]);
          mma_bf16_16816(o[j + 1], ah[0], ah[1], ah[2], ah[3], vb[2], vb[3]);
          mma_bf16_16816(o[j], al[0], al[1], al[2], al[3], vb[0], vb[1]);
          mma_bf16_16816(o[j + 1], al[0], al[1], al[2], al[3], vb[2], vb[3]);
        }
      }
    }
    __syncthreads();                                      // the tile's buffer and the weights may be overwritten
  }
  // ---- sums: lanes of a quad, then the four warps (all share the running maxima)
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
  }
  if (t == 0) {
    mw[warp * 16 + g] = l_run[0];
    mw[warp * 16 + g + 8] = l_run[1];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int hr = g + 8 * r, head = head0 + hr;
    if (head >= p.d.heads) continue;
    const float L = (mw[hr] + mw[16 + hr]) + (mw[32 + hr] + mw[48 + hr]);
    if (p.n_splits == 1) {
      const float inv = 1.0f / L;
      __nv_bfloat16* dst = p.out + ((size_t)head * p.b.n_seqs + seq) * p.d.c_pad + col0 + 2 * t;
#pragma unroll
      for (int j = 0; j < VT; ++j)
        if (FULL || j < n_vt) *reinterpret_cast<uint32_t*>(dst + 8 * j) = pack_bf16(o[j][2 * r] * inv, o[j][2 * r + 1] * inv);
    } else {
      const size_t at = ((size_t)seq * p.d.heads + head) * p.n_splits + blockIdx.x;
      float* dst = p.part_o + at * p.d.c_pad + col0 + 2 * t;
#pragma unroll
      for (int j = 0; j < VT; ++j)
        if (FULL || j < n_vt) *reinterpret_cast<float2*>(dst + 8 * j) = make_float2(o[j][2 * r], o[j][2 * r + 1]);
      if (warp == 0 && t == 0) {
        p.part_ml[2 * at] = m_run[r];
        p.part_ml[2 * at + 1] = L;
      }
    }
  }
}

// One CTA per (head, sequence): a thread owns two columns at a time.
__global__ void __launch_bounds__(256) latent_combine_kernel(const int* single, const int* cache_row, int n_splits, int heads, int n_seqs, int c_pad,
                                                             const float* part_o, const float* part_ml, __nv_bfloat16* out) {
  __shared__ float wgt[kLdMaxSplits];
  pdl_wait();
  pdl_launch_dependents();
  const int head = blockIdx.x, seq = blockIdx.y, row = single ? single[seq] : seq, lane = threadIdx.x & 31;
  if (row < 0 || cache_row[row] < 0) return;
  const size_t at = ((size_t)seq * heads + head) * n_splits;
  if (threadIdx.x < 32) {
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      m[i] = s < n_splits ? part_ml[2 * (at + s)] : -FLT_MAX;
      l[i] = s < n_splits ? part_ml[2 * (at + s) + 1] : 0.f;
    }
    const float M = warp_max(fmaxf(m[0], m[1])), w0 = ex2_ftz(m[0] - M), w1 = ex2_ftz(m[1] - M);
    const float f = 1.0f / warp_sum(l[0] * w0 + l[1] * w1);
    wgt[lane] = w0 * f;
    wgt[lane + 32] = w1 * f;
  }
  __syncthreads();
  for (int c = 2 * threadIdx.x; c < c_pad; c += 512) {
    float x = 0.f, y = 0.f;
#pragma unroll 8
    for (int s = 0; s < n_splits; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(part_o + (at + s) * c_pad + c);
      x = fmaf(wgt[s], v.x, x);
      y = fmaf(wgt[s], v.y, y);
    }
    *reinterpret_cast<uint32_t*>(out + ((size_t)head * n_seqs + seq) * c_pad + c) = pack_bf16(x, y);
  }
}

static size_t decode_smem(const LatentDims& d, int ht) {
  const size_t row_bytes = (size_t)d.row() * 2 + 16;
  return (size_t)(16 * ht + 2 * kLdTile) * row_bytes + (size_t)ht * (2 * 16 * kLdPRow + 64 * sizeof(float));
}

bool latent_absorb_supported(const LatentDims& d) { return d.c_pad <= 512 && decode_smem(d, 2) <= 226 * 1024; }

int launch_latent_decode(tq_ctx* ctx, const LatentDims& d, const RaggedBatch& b, const int* single, float scale, const Rotation& rot, bool rotate,
                         const void* q_lat, const void* q, size_t ldq, const void* cache, void* out) {
  TQ_REQUIRE(ctx, latent_absorb_supported(d), "latent attention: a latent of %d values is too large for the absorbed form", d.rank);
  const long long tiles = (b.max_len + kLdTile - 1) / kLdTile;
  // two head tiles share a CTA's cache tiles unless that leaves the GPU half empty
  const int HT = d.heads > 16 && (d.heads + 31) / 32 * (tiles + 1) / 2 * b.n_seqs >= ctx->sm_count ? 2 : 1, hg = (d.heads + 16 * HT - 1) / (16 * HT);
  TQ_REQUIRE(ctx, hg <= 65535 && b.n_seqs <= 65535, "latent attention: too many heads or sequences");
  LatentDecodeParams p;
  p.d = d;
  p.b = b;
  p.single = single;
  p.q_lat = static_cast<const __nv_bfloat16*>(q_lat);
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.ldq = ldq;
  p.cache = static_cast<const __nv_bfloat16*>(cache);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.scale = scale;
  p.rot = rot;
  p.rotate = rotate;
  p.part_o = p.part_ml = nullptr;
  // about two CTAs per SM
  const long long ctas = (long long)hg * b.n_seqs;
  long long n = (2ll * ctx->sm_count + ctas - 1) / ctas;
  if (n > tiles) n = tiles;
  if (n > kLdMaxSplits) n = kLdMaxSplits;
  if (n < 1) n = 1;
  const long long per = (tiles + n - 1) / n;               // (no split without a tile)
  p.n_splits = (int)((tiles + per - 1) / per);
  if (p.n_splits > 1) {
    const size_t parts = (size_t)b.n_seqs * d.heads * p.n_splits;
    if (int st = ensure_scratch(ctx, parts * (d.c_pad + 2) * sizeof(float))) return st;
    p.part_o = static_cast<float*>(ctx->scratch);
    p.part_ml = p.part_o + parts * d.c_pad;
  }
  const size_t smem = decode_smem(d, HT);
  const dim3 grid((unsigned)p.n_splits, (unsigned)hg, (unsigned)b.n_seqs);
  auto go = [&](auto kern) -> int {
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3((unsigned)(kLdThreads * HT)), smem, p));
    return TQ_OK;
  };
  int st;
  if (d.c_pad <= 128) st = HT == 2 ? go(latent_decode_kernel<4, 2, false>) : go(latent_decode_kernel<4, 1, false>);
  else if (d.c_pad < 256) st = HT == 2 ? go(latent_decode_kernel<8, 2, false>) : go(latent_decode_kernel<8, 1, false>);
  else if (d.c_pad == 256) st = HT == 2 ? go(latent_decode_kernel<8, 2, true>) : go(latent_decode_kernel<8, 1, true>);
  else if (d.c_pad < 512) st = HT == 2 ? go(latent_decode_kernel<16, 2, false>) : go(latent_decode_kernel<16, 1, false>);
  else if (d.row() == 576) st = HT == 2 ? go(latent_decode_kernel<16, 2, true, 576>) : go(latent_decode_kernel<16, 1, true, 576>);
  else st = HT == 2 ? go(latent_decode_kernel<16, 2, true>) : go(latent_decode_kernel<16, 1, true>);
  if (st != TQ_OK) return st;
  if (p.n_splits > 1)
    TQ_CUDA(ctx, launch_k(ctx, latent_combine_kernel, dim3((unsigned)d.heads, (unsigned)b.n_seqs), dim3(256), 0, single, b.cache_row, p.n_splits, d.heads, b.n_seqs,
                          d.c_pad, (const float*)p.part_o, (const float*)p.part_ml, p.out));
  return TQ_OK;
}

}  // namespace tq

using namespace tq;

extern "C" int tq_latent_decode(tq_ctx* ctx, size_t heads, size_t dim, size_t rot, size_t rank, float scale, size_t rot_dims, const float* freq_dev,
                                float rot_mult, int rotate, const void* q_lat_dev, const void* q_dev, size_t ldq, const void* cache_dev, size_t cache_rows,
                                const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t max_len, void* out_dev) {
  if (int st = bind(ctx)) return st;
  if (n_seqs == 0) return TQ_OK;
  TQ_REQUIRE(ctx, heads > 0 && rank > 0 && max_len > 0 && rot_dims <= rot && rot_dims % 2 == 0, "tq_latent_decode: bad sizes");
  TQ_REQUIRE(ctx, q_lat_dev && (q_dev || rot == 0) && cache_dev && row_pos_dev && cache_row_dev && out_dev && (freq_dev || rot_dims == 0 || !rotate),
             "tq_latent_decode: null pointer");
  RaggedBatch b;
  b.n_seqs = b.rows = (int)n_seqs;
  b.max_len = (int)max_len;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  Rotation r;
  r.dims = (int)rot_dims;
  r.freq = freq_dev;
  r.mult = rot_mult;
  r.interleaved = true;
  return launch_latent_decode(ctx, latent_dims((int)heads, (int)dim, (int)rot, 0, (int)rank), b, nullptr, scale, r, rotate != 0, q_lat_dev, q_dev, ldq, cache_dev,
                              out_dev);
}
