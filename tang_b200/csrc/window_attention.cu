// Windowed grouped-query attention (see window_attention.cuh).
//
// bf16, head sizes up to 256: one kernel body in two forms.  The 16 rows of an mma.sync m16n8k16 tile are 16 (position, head)
// pairs of one KV head, so that a group of any size fills the tile with few positions.
//   * SPLIT = false (prompts): a CTA's eight warps own 16 pairs each and walk the same key tiles, each warp only the steps
//     that its own pairs' windows reach;
//   * SPLIT = true (one query per sequence): a CTA's four warps own the same 16 pairs and take 16 of a tile's 64 keys each;
//     the tiles are also split over CTAs, and window_combine_kernel merges the splits.
// Scores, weights and their sums are f32; a weight enters the tensor core as two bf16 terms (16 significant bits).  The sink
// starts the running maximum and sum.  Key tiles of 64 rows arrive by cp.async, two in flight.
//
// window_attention_simt_kernel is the exact f32 form (and takes bf16 heads of any size).
#include "window_attention.cuh"

#include <cuda_bf16.h>

#include <cfloat>

#include "attn_mma.cuh"
#include "common.cuh"

namespace tq {

constexpr int kWaKeys = 64;
constexpr int kWaMaxSplits = 64;
constexpr int kWaPairs = 128;      // pairs of a prompt CTA

struct WinParams {
  const __nv_bfloat16 *q, *k, *v, *gate;
  __nv_bfloat16* out;
  long long ldq, ldg, ldo;
  WindowAttn a;
  RaggedBatch b;
  int group, gb, n_hb;         // heads per KV head; heads per block; blocks per KV head
  int dp;                      // dim rounded up to 16
  int stages;
  int n_splits;                // SPLIT only
  float* part_o;               // [rows][heads][n_splits][16-column padded vdim]
  float* part_ml;              // [rows][heads][n_splits][2]
};

__device__ __forceinline__ float sigmoid_gate(float g) { return 1.0f / (1.0f + expf(-g)); }

// Base-2 logarithm of the weight of a raw score: scaled, capped.  tanh(x) = 1 - 2 / (1 + e^2x).
struct CapScore {
  float in, out;               // capped: 2 log2(e) scale / softcap, softcap log2(e); else scale log2(e), unused
  bool capped;
  __device__ __forceinline__ CapScore(const WindowAttn& a) {
    capped = a.softcap > 0.f;
    in = capped ? 2.f * kLog2e * a.scale / a.softcap : a.scale * kLog2e;
    out = a.softcap * kLog2e;
  }
  __device__ __forceinline__ float operator()(float s) const {
    const float x = s * in;
    if (!capped) return x;
    return out - __fdividef(2.f * out, 1.f + ex2_ftz(fminf(x, 100.f)));
  }
};

// DVT: value columns / 8 (padded to 16 columns, so even).  POOL: key tiles of pooled blocks come first, then the window's.
template <int DVT, bool SPLIT, bool POOL>
__global__ void __launch_bounds__(SPLIT ? 128 : 256, DVT > 16 ? 1 : SPLIT ? 3 : 2) window_attention_kernel(const __grid_constant__ WinParams p) {
  constexpr int kThreads = SPLIT ? 128 : 256;
  constexpr int kWarps = kThreads / 32;
  constexpr int NT = SPLIT ? 2 : 4;                 // 8-key tiles of scores a warp forms at a time
  constexpr int kSub = SPLIT ? 1 : kWaKeys / (8 * NT);   // such steps per key tile
  extern __shared__ __align__(128) uint8_t wa_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int k_row = p.dp * 2 + 16;                  // bytes; one bank group of shift per row
  constexpr int v_row = DVT * 16 + 16;
  const int q_rows = SPLIT ? 16 : kWaPairs;
  uint8_t* q_s = wa_smem;
  uint8_t* k_s = q_s + (size_t)q_rows * k_row;
  uint8_t* v_s = k_s + (size_t)p.stages * kWaKeys * k_row;

  pdl_wait();
  pdl_launch_dependents();

  const int kvh = blockIdx.y / p.n_hb, hb = blockIdx.y % p.n_hb, b = blockIdx.z;
  const int gb = min(p.gb, p.group - hb * p.gb);    // heads of this block
  const int head0 = kvh * p.group + hb * p.gb;
  const int row0 = p.b.seq_rows ? p.b.seq_rows[b] : b;
  const int n_q = p.b.seq_rows ? p.b.seq_rows[b + 1] - row0 : 1;
  const int pos_per_cta = SPLIT ? 1 : kWaPairs / p.gb;
  // first query of this CTA inside the sequence; the last queries go first (they may see the most keys)
  const int i0 = SPLIT ? 0 : ((int)gridDim.x - 1 - (int)blockIdx.x) * pos_per_cta;
  if (i0 >= n_q || row0 < 0 || row0 + n_q > p.b.rows) return;
  const int i1 = min(i0 + pos_per_cta, n_q) - 1;
  const int p0 = p.b.row_pos[row0 + i0], p1 = p0 + (i1 - i0);
  const int crow = p.b.cache_row[row0 + i0];
  // every row of the range has to be in the cache (the embedding kernel has reported one that is not)
  const bool in_cache = crow >= p0 && p.b.cache_row[row0 + i1] == crow + (i1 - i0) && (size_t)(crow + (i1 - i0)) < p.b.cache_rows;
  if (!in_cache) return;
  const size_t seq0 = (size_t)(crow - p0);                 // cache row of the sequence's position 0
  const size_t ke = (size_t)p.a.kv_heads * p.a.dim_pad, ve = (size_t)p.a.kv_heads * p.a.vdim_pad;
  const __nv_bfloat16* kb = p.k + seq0 * ke + (size_t)kvh * p.a.dim_pad;
  const __nv_bfloat16* vb = p.v + seq0 * ve + (size_t)kvh * p.a.vdim_pad;

  const int lo = max(0, p0 - p.a.window + 1);
  // tiles below `lo_t` are the pooled ones, counted from lo_t - pool_t
  const int lo_t = lo / kWaKeys, hi_t = p1 / kWaKeys;
  const int n_pool = POOL ? min(seen_blocks(p1, p.a.window, p.a.pool), p.a.pool_rows) : 0, pool_t = (n_pool + kWaKeys - 1) / kWaKeys, first_t = lo_t - pool_t;
  int t0 = first_t, t1 = hi_t + 1;
  if constexpr (SPLIT) {
    const int per = (hi_t - first_t + p.n_splits) / p.n_splits;
    t0 = min(first_t + (int)blockIdx.x * per, hi_t + 1);
    t1 = min(t0 + per, hi_t + 1);
  }

  // ---- padding columns of shared memory must hold numbers
  const bool pad = p.dp != p.a.dim_pad || p.a.dim != p.a.dim_pad || DVT * 8 != p.a.vdim_pad;
  if (pad) {
    const int words = (int)(((size_t)q_rows * k_row + (size_t)p.stages * kWaKeys * (k_row + v_row)) / 16);
    for (int i = threadIdx.x; i < words; i += kThreads) reinterpret_cast<uint4*>(wa_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
  }
  const int kcm = p.a.dim_pad / 8, vcm = p.a.vdim_pad / 8;   // 16-byte pieces per key / value row
  // This thread copies piece `pc` of every row_step-th row of a tile (at most 64 pieces).
  const int per_row = kcm + vcm;
  const int row_step = kThreads / per_row;
  const int row_first = threadIdx.x / per_row, pc = threadIdx.x - row_first * per_row;
  const bool copies = row_first < row_step, is_v = pc >= kcm;
  const __nv_bfloat16* src_c = is_v ? vb + (pc - kcm) * 8 : kb + pc * 8;
  const __nv_bfloat16* pool_c = nullptr;
  if constexpr (POOL) {
    const size_t row = seq0 / (size_t)p.a.max_seq * p.a.pool_rows;
    pool_c = is_v ? static_cast<const __nv_bfloat16*>(p.a.pooled_values) + row * ve + (size_t)kvh * p.a.vdim_pad + (pc - kcm) * 8
                  : static_cast<const __nv_bfloat16*>(p.a.pooled_keys) + row * ke + (size_t)kvh * p.a.dim_pad + pc * 8;
  }
  const size_t src_ld = is_v ? ve : ke;
  const int dst_ld = is_v ? v_row : k_row;
  const uint32_t dst_c = smem_u32(is_v ? v_s + (pc - kcm) * 16 : k_s + pc * 16);
  auto load_tile = [&](int tile, int buf) {
    const bool pooled = POOL && tile < lo_t;
    const int key0 = (pooled ? tile - first_t : tile) * kWaKeys;
    if (copies) {
      const __nv_bfloat16* src = (pooled ? pool_c : src_c) + (size_t)(key0 + row_first) * src_ld;
      uint32_t dst = dst_c + (uint32_t)((buf * kWaKeys + row_first) * dst_ld);
      const int n_valid = (pooled ? n_pool : p1 + 1) - key0;   // rows at or beyond it become zeros
#pragma unroll 4
      for (int row = row_first; row < kWaKeys; row += row_step) {
        cp_async16(dst, row < n_valid ? src : src_c, row < n_valid);
        src += row_step * src_ld;
        dst += (uint32_t)(row_step * dst_ld);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (t0 < t1) load_tile(t0, 0);

  // ---- queries: pair r = position * gb + head
  auto q_src = [&](int r) -> const __nv_bfloat16* {
    const int qi = SPLIT ? 0 : r / p.gb, hh = SPLIT ? r : r % p.gb;
    if (i0 + qi > i1 || (!SPLIT && r >= pos_per_cta * p.gb) || hh >= gb) return nullptr;
    return p.q + (size_t)(row0 + i0 + qi) * p.ldq + (size_t)(head0 + hh) * p.a.q_head;
  };
  if ((p.a.dim & 7) == 0 && (p.ldq & 7) == 0 && (p.a.q_head & 7) == 0) {
    const int pm = p.a.dim / 8;
    for (int i = threadIdx.x; i < q_rows * pm; i += kThreads) {
      const int r = i / pm, c = i - r * pm;
      const __nv_bfloat16* src = q_src(r);
      *reinterpret_cast<uint4*>(q_s + (size_t)r * k_row + c * 16) = src ? *reinterpret_cast<const uint4*>(src + c * 8) : make_uint4(0u, 0u, 0u, 0u);
    }
  } else {
    for (int i = threadIdx.x; i < q_rows * p.a.dim; i += kThreads) {
      const int r = i / p.a.dim, d = i - r * p.a.dim;
      const __nv_bfloat16* src = q_src(r);
      *reinterpret_cast<__nv_bfloat16*>(q_s + (size_t)r * k_row + d * 2) = src ? src[d] : __float2bfloat16_rn(0.f);
    }
  }

  // this lane's two pairs: rows g and g + 8 of the warp's tile
  const int base_pair = SPLIT ? 0 : 16 * warp;
  bool live[2];
  int qpos[2], qrow[2], qhead[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int pr = base_pair + g + 8 * h;
    const int pqi = SPLIT ? 0 : pr / p.gb, phh = SPLIT ? pr : pr % p.gb;
    live[h] = i0 + pqi <= i1 && (SPLIT || pr < pos_per_cta * p.gb) && phh < gb;
    qpos[h] = p0 + pqi;
    qrow[h] = row0 + i0 + pqi;
    qhead[h] = head0 + phh;
  }
  // positions of the warp's pairs
  const int w_first = SPLIT ? p0 : p0 + base_pair / p.gb, w_last = SPLIT ? p0 : min(p1, p0 + (base_pair + 15) / p.gb);
  const bool w_live = SPLIT || w_first <= p1;

  float o[DVT][4];                                         // [columns 8j + 2t, +1] of pair g, then of pair g + 8
#pragma unroll
  for (int j = 0; j < DVT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // one lane of a row (one warp and split of a pair) carries the sink's term
  const bool owns_sink = t == 0 && (!SPLIT || (warp == 0 && blockIdx.x == 0));
  float m_run[2], l_run[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const float sink = p.a.sinks ? (live[h] ? p.a.sinks[qhead[h]] : 0.f) : p.a.sink;
    m_run[h] = sink * kLog2e;
    l_run[h] = owns_sink && sink > -FLT_MAX ? 1.f : 0.f;
  }
  const CapScore cap(p.a);
  const int nks = p.dp / 16;
  int seen[2] = {0, 0}, w_seen_first = 0, w_seen_last = 0;   // pooled blocks that the two pairs, the warp's first and its last one see
  if constexpr (POOL) {
    seen[0] = seen_blocks(qpos[0], p.a.window, p.a.pool);
    seen[1] = seen_blocks(qpos[1], p.a.window, p.a.pool);
    w_seen_first = seen_blocks(w_first, p.a.window, p.a.pool);
    w_seen_last = seen_blocks(w_last, p.a.window, p.a.pool);
  }

  for (int tile = t0; tile < t1; ++tile) {
    const int buf = p.stages == 2 ? (tile - t0) & 1 : 0;
    if (p.stages == 2 && tile + 1 < t1) {
      load_tile(tile + 1, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    for (int sub = 0; sub < kSub; ++sub) {
      const int w0 = SPLIT ? 16 * warp : 8 * NT * sub;     // first key of the tile for this warp's step
      const bool pooled = POOL && tile < lo_t;
      const int key0 = (pooled ? tile - first_t : tile) * kWaKeys + w0;
      if (!w_live || (pooled ? key0 >= w_seen_last : key0 > w_last || w_first - (key0 + 8 * NT - 1) >= p.a.window)) continue;
      const uint8_t* kt = k_s + (buf * kWaKeys + w0) * k_row;
      const uint8_t* vt = v_s + (buf * kWaKeys + w0) * v_row;
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const uint8_t* qaddr = q_s + (size_t)(base_pair + (lane & 15)) * k_row + 16 * (lane >> 4);
      // lanes 0..7 / 8..15: the two k halves of the first eight keys, lanes 16..31: of the next eight
      const uint8_t* kaddr = kt + (size_t)((lane & 7) + 8 * (lane >> 4)) * k_row + ((lane >> 3) & 1) * 16;
      for (int ks = 0; ks < nks; ++ks) {
        uint32_t qf[4], kf[NT / 2][4];
        ldmatrix4(qf, qaddr + 32 * ks);
#pragma unroll
        for (int n = 0; n < NT / 2; ++n) ldmatrix4(kf[n], kaddr + 16 * n * k_row + 32 * ks);
#pragma unroll
        for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n], qf[0], qf[1], qf[2], qf[3], kf[n >> 1][2 * (n & 1)], kf[n >> 1][2 * (n & 1) + 1]);
      }
      // a step whose keys every pair of the warp sees needs no mask (rows without a query are never stored)
      const bool full = pooled ? key0 + 8 * NT <= w_seen_first : key0 + 8 * NT - 1 <= w_first && w_last - key0 < p.a.window;
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float v = cap(s[n][c]);
          if (!full) {
            const int key = key0 + 8 * n + 2 * t + (c & 1);
            const bool ok = live[c >> 1] && (pooled ? key < seen[c >> 1] : key <= qpos[c >> 1] && qpos[c >> 1] - key < p.a.window);
            v = ok ? v : -INFINITY;
          }
          s[n][c] = v;
          mx[c >> 1] = fmaxf(mx[c >> 1], v);
        }
      float alpha[2], base[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        const float mn = fmaxf(m_run[h], mx[h]);
        base[h] = mn == -INFINITY ? 0.f : mn;              // (nothing seen yet: every weight below becomes zero)
        alpha[h] = ex2_ftz(m_run[h] - base[h]);
        m_run[h] = mn;
      }
      float ps[2] = {0.f, 0.f};
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          s[n][c] = ex2_ftz(s[n][c] - base[c >> 1]);
          ps[c >> 1] += s[n][c];
        }
      l_run[0] = l_run[0] * alpha[0] + ps[0];
      l_run[1] = l_run[1] * alpha[1] + ps[1];
      if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
        for (int j = 0; j < DVT; ++j) {
          o[j][0] *= alpha[0];
          o[j][1] *= alpha[0];
          o[j][2] *= alpha[1];
          o[j][3] *= alpha[1];
        }
      }
#pragma unroll
      for (int kk = 0; kk < NT / 2; ++kk) {
        uint32_t h0, h1, h2, h3, r0, r1, r2, r3;
        split_bf16(s[2 * kk][0], s[2 * kk][1], h0, r0);
        split_bf16(s[2 * kk][2], s[2 * kk][3], h1, r1);
        split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], h2, r2);
        split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], h3, r3);
        const uint8_t* vaddr = vt + (size_t)(16 * kk + (lane & 15)) * v_row + 16 * (lane >> 4);
        // two column pairs at a time, the four leading terms before the four residual ones: no product waits for the last
#pragma unroll
        for (int j = 0; j < DVT / 2; j += 2) {
          uint32_t vf[2][4];
          ldmatrix4_t(vf[0], vaddr + 32 * j);
          ldmatrix4_t(vf[1], vaddr + 32 * j + 32);
#pragma unroll
          for (int i = 0; i < 4; ++i) mma_bf16_16816(o[2 * j + i], h0, h1, h2, h3, vf[i >> 1][2 * (i & 1)], vf[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
          for (int i = 0; i < 4; ++i) mma_bf16_16816(o[2 * j + i], r0, r1, r2, r3, vf[i >> 1][2 * (i & 1)], vf[i >> 1][2 * (i & 1) + 1]);
        }
      }
    }
    __syncthreads();
    if (p.stages == 1 && tile + 1 < t1) load_tile(tile + 1, 0);
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
  }
  const int vd = p.a.vdim;

  if constexpr (!SPLIT) {
    const bool even = ((p.ldo | p.ldg | vd) & 1) == 0;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (!live[h]) continue;
      const float inv = p.a.out_scale / l_run[h];
      __nv_bfloat16* dst = p.out + (size_t)qrow[h] * p.ldo + (size_t)qhead[h] * vd;
      const __nv_bfloat16* gate = p.gate ? p.gate + (size_t)qrow[h] * p.ldg + (size_t)qhead[h] * vd : nullptr;
#pragma unroll
      for (int j = 0; j < DVT; ++j) {
        const int d = 8 * j + 2 * t;
        if (d >= vd) continue;
        float v0 = o[j][2 * h] * inv, v1 = o[j][2 * h + 1] * inv;
        if (even) {
          if (gate) {
            const uint32_t gw = *reinterpret_cast<const uint32_t*>(gate + d);
            v0 *= sigmoid_gate(bf16_bits_to_float(gw & 0xFFFFu));
            v1 *= sigmoid_gate(bf16_bits_to_float(gw >> 16));
          }
          *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(v0, v1);
        } else {
          dst[d] = __float2bfloat16_rn(gate ? v0 * sigmoid_gate(__bfloat162float(gate[d])) : v0);
          if (d + 1 < vd) dst[d + 1] = __float2bfloat16_rn(gate ? v1 * sigmoid_gate(__bfloat162float(gate[d + 1])) : v1);
        }
      }
    }
  } else {
    // ---- merge the four warps: [warp][16 pairs][DVT * 8]
    constexpr int W = DVT * 8;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // (a CTA without tiles has not met one since it wrote q_s)
    float* mo = reinterpret_cast<float*>(wa_smem);
    float* mml = mo + kWarps * 16 * W;
#pragma unroll
    for (int j = 0; j < DVT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) mo[((size_t)warp * 16 + g + 8 * (c >> 1)) * W + 8 * j + 2 * t + (c & 1)] = o[j][c];
    if (t == 0) {
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        // (a finite stand-in for "no key seen": its weight is zero beside any real maximum)
        mml[(warp * 16 + g + 8 * h) * 2] = fmaxf(m_run[h], -FLT_MAX);
        mml[(warp * 16 + g + 8 * h) * 2 + 1] = l_run[h];
      }
    }
    __syncthreads();
    for (int h = warp; h < gb; h += kWarps) {              // a warp finishes a head
      float wt[kWarps], L = 0.f, M = -FLT_MAX;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) M = fmaxf(M, mml[(w * 16 + h) * 2]);
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        wt[w] = exp2f(mml[(w * 16 + h) * 2] - M);
        L += mml[(w * 16 + h) * 2 + 1] * wt[w];
      }
      float acc[(W + 31) / 32];
#pragma unroll
      for (int i = 0; i < (W + 31) / 32; ++i) {
        const int d = lane + 32 * i;
        float v = 0.f;
        if (d < W) {
#pragma unroll
          for (int w = 0; w < kWarps; ++w) v += mo[((size_t)w * 16 + h) * W + d] * wt[w];
        }
        acc[i] = v;
      }
      if (p.n_splits > 1) {
        const size_t pi = ((size_t)row0 * p.a.heads + head0 + h) * p.n_splits + blockIdx.x;
#pragma unroll
        for (int i = 0; i < (W + 31) / 32; ++i)
          if (lane + 32 * i < W) p.part_o[pi * W + lane + 32 * i] = acc[i];
        if (lane == 0) {
          p.part_ml[pi * 2] = M;
          p.part_ml[pi * 2 + 1] = L;
        }
      } else {
        const float inv = p.a.out_scale / L;
        __nv_bfloat16* dst = p.out + (size_t)row0 * p.ldo + (size_t)(head0 + h) * vd;
        const __nv_bfloat16* gate = p.gate ? p.gate + (size_t)row0 * p.ldg + (size_t)(head0 + h) * vd : nullptr;
#pragma unroll
        for (int i = 0; i < (W + 31) / 32; ++i) {
          const int d = lane + 32 * i;
          if (d < vd) dst[d] = __float2bfloat16_rn(acc[i] * inv * (gate ? sigmoid_gate(__bfloat162float(gate[d])) : 1.f));
        }
      }
    }
  }
}

// Merges the splits of one (row, head).  One CTA per head, a thread per column.
__global__ void __launch_bounds__(256) window_combine_kernel(const float* part_o, const float* part_ml, int n_splits, int W, int heads, int vdim,
                                                             const int* cache_row, float out_scale, const __nv_bfloat16* gate, long long ldg,
                                                             __nv_bfloat16* out, long long ldo) {
  __shared__ float wgt[kWaMaxSplits];
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31, d = threadIdx.x;
  const size_t rh = blockIdx.x;                            // row * heads + head
  const int row = (int)(rh / heads), head = (int)(rh % heads);
  if (cache_row[row] < 0) return;
  if (threadIdx.x < 32) {
    const float* ml = part_ml + rh * n_splits * 2;
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      m[i] = s < n_splits ? ml[2 * s] : -FLT_MAX;
      l[i] = s < n_splits ? ml[2 * s + 1] : 0.f;
    }
    const float M = warp_max(fmaxf(m[0], m[1]));
    const float w0 = exp2f(m[0] - M), w1 = exp2f(m[1] - M);
    const float f = out_scale / warp_sum(l[0] * w0 + l[1] * w1);
    wgt[lane] = w0 * f;
    wgt[lane + 32] = w1 * f;
  }
  __syncthreads();
  if (d >= vdim) return;
  float v = 0.f;
  const float* src = part_o + rh * n_splits * W + d;
#pragma unroll 8
  for (int s = 0; s < n_splits; ++s) v += src[(size_t)s * W] * wgt[s];
  if (gate) v *= sigmoid_gate(__bfloat162float(gate[(size_t)row * ldg + (size_t)head * vdim + d]));
  out[(size_t)row * ldo + (size_t)head * vdim + d] = __float2bfloat16_rn(v);
}

// ------------------------------------------------------------------------------------------------ f32 / any size
__device__ __forceinline__ float wa_load(const float* p) { return *p; }
__device__ __forceinline__ float wa_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void wa_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void wa_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// One CTA per (row, head); 128 keys at a time, one per thread; then every thread owns value columns.
template <typename T>
__global__ void __launch_bounds__(128) window_attention_simt_kernel(const T* q, long long ldq, const T* gate, long long ldg, const T* k, const T* v,
                                                                    T* out, long long ldo, WindowAttn a, RaggedBatch b) {
  extern __shared__ float ws_smem[];
  float* qs = ws_smem;                       // [dim]
  float* acc = qs + a.dim;                   // [vdim]
  float* pr = acc + a.vdim;                  // [128]
  __shared__ float red[4];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = b.row_pos[row], crow = b.cache_row[row];
  if (crow < pos || (size_t)crow >= b.cache_rows) return;
  const int kvh = head / (a.heads / a.kv_heads);
  const size_t seq0 = (size_t)(crow - pos);
  const size_t ke = (size_t)a.kv_heads * a.dim_pad, ve = (size_t)a.kv_heads * a.vdim_pad;
  const T* kb = k + seq0 * ke + (size_t)kvh * a.dim_pad;
  const T* vb = v + seq0 * ve + (size_t)kvh * a.vdim_pad;
  for (int i = tid; i < a.dim; i += 128) qs[i] = wa_load(q + (size_t)row * ldq + (size_t)head * a.q_head + i);
  for (int i = tid; i < a.vdim; i += 128) acc[i] = 0.f;
  __syncthreads();
  auto block_reduce = [&](float x, bool is_max) {
    x = is_max ? warp_max(x) : warp_sum(x);
    if (lane == 0) red[warp] = x;
    __syncthreads();
    const float r = is_max ? fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])) : (red[0] + red[1]) + (red[2] + red[3]);
    __syncthreads();
    return r;
  };
  const int lo = max(0, pos - a.window + 1);
  const int n_pool = a.pool ? min(seen_blocks(pos, a.window, a.pool), a.pool_rows) : 0, n_vis = n_pool + pos - lo + 1;   // pooled blocks first
  const size_t pool0 = a.pool ? seq0 / (size_t)a.max_seq * a.pool_rows : 0;
  const T* pk = static_cast<const T*>(a.pooled_keys) + pool0 * ke + (size_t)kvh * a.dim_pad;
  const T* pv = static_cast<const T*>(a.pooled_values) + pool0 * ve + (size_t)kvh * a.vdim_pad;
  auto key_row = [&](int c) { return c < n_pool ? pk + (size_t)c * ke : kb + (size_t)(lo + c - n_pool) * ke; };
  auto value_row = [&](int c) { return c < n_pool ? pv + (size_t)c * ve : vb + (size_t)(lo + c - n_pool) * ve; };
  const float sink = a.sinks ? a.sinks[head] : a.sink;
  const bool has_sink = sink > -FLT_MAX;
  float m_run = has_sink ? sink : -FLT_MAX, l_run = has_sink ? 1.f : 0.f;
  for (int c0 = 0; c0 < n_vis; c0 += 128) {
    const int c = c0 + tid, n = min(128, n_vis - c0);
    float sc = -FLT_MAX;
    if (c < n_vis) {
      const T* kr = key_row(c);
      float s = 0.f;
      for (int d = 0; d < a.dim; ++d) s = fmaf(qs[d], wa_load(kr + d), s);
      s *= a.scale;
      sc = a.softcap > 0.f ? a.softcap * tanhf(s / a.softcap) : s;
    }
    const float mn = fmaxf(m_run, block_reduce(sc, true));
    const float alpha = expf(m_run - mn);
    m_run = mn;
    const float w = c < n_vis ? expf(sc - mn) : 0.f;
    pr[tid] = w;
    l_run = l_run * alpha + block_reduce(w, false);   // (its barriers also publish pr)
    for (int d = tid; d < a.vdim; d += 128) {
      float x = acc[d] * alpha;
      for (int j = 0; j < n; ++j) x = fmaf(pr[j], wa_load(value_row(c0 + j) + d), x);
      acc[d] = x;
    }
    __syncthreads();
  }
  for (int d = tid; d < a.vdim; d += 128) {
    float o = acc[d] / l_run * a.out_scale;
    if (gate) o *= sigmoid_gate(wa_load(gate + (size_t)row * ldg + (size_t)head * a.vdim + d));
    wa_store(out + (size_t)row * ldo + (size_t)head * a.vdim + d, o);
  }
}

// ------------------------------------------------------------------------------------------------ launch
template <typename T>
static int launch_simt(tq_ctx* ctx, const WindowAttn& a, const RaggedBatch& b, const void* q, size_t ldq, const void* gate, size_t ldg, const void* k,
                       const void* v, void* out, size_t ldo) {
  const size_t smem = ((size_t)a.dim + a.vdim + 128) * sizeof(float);
  if (smem > 200 * 1024) return fail(ctx, TQ_EUNSUPPORTED, "window attention: head sizes %d / %d are too large", a.dim, a.vdim);
  if (smem > 48 * 1024)
    TQ_CUDA(ctx, cudaFuncSetAttribute(window_attention_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, window_attention_simt_kernel<T>, dim3((unsigned)b.rows, (unsigned)a.heads), dim3(128), smem, static_cast<const T*>(q),
                        (long long)ldq, static_cast<const T*>(gate), (long long)ldg, static_cast<const T*>(k), static_cast<const T*>(v),
                        static_cast<T*>(out), (long long)ldo, a, b));
  return TQ_OK;
}

template <int DVT>
static int launch_mma(tq_ctx* ctx, WinParams& p, bool split, size_t smem, dim3 grid) {
  auto go = [&](auto kern, int threads) -> int {
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3((unsigned)threads), smem, p));
    return TQ_OK;
  };
  if (p.a.pool) return split ? go(window_attention_kernel<DVT, true, true>, 128) : go(window_attention_kernel<DVT, false, true>, 256);
  return split ? go(window_attention_kernel<DVT, true, false>, 128) : go(window_attention_kernel<DVT, false, false>, 256);
}

int launch_window_attention(tq_ctx* ctx, const WindowAttn& attn, const RaggedBatch& b, int dtype, const void* q, size_t ldq, const void* gate,
                            size_t ldg, const void* k_cache, const void* v_cache, void* out, size_t ldo) {
  WindowAttn a = attn;
  if (!a.q_head) a.q_head = (size_t)a.dim;
  TQ_REQUIRE(ctx, a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0, "window attention: heads must be a multiple of kv_heads");
  TQ_REQUIRE(ctx, a.dim > 0 && a.vdim > 0 && a.dim_pad >= a.dim && a.vdim_pad >= a.vdim && a.dim_pad % 8 == 0 && a.vdim_pad % 8 == 0,
             "window attention: bad head sizes");
  TQ_REQUIRE(ctx, a.window > 0 && a.softcap >= 0.f, "window attention: bad window or cap");
  TQ_REQUIRE(ctx, a.pool >= 0 && (a.pool == 0 || (a.pooled_keys && a.pooled_values && a.max_seq > 0 && a.pool_rows >= 0)), "window attention: bad pooled blocks");
  if (b.rows == 0 || b.n_seqs == 0) return TQ_OK;
  if (dtype == TQ_F32) return launch_simt<float>(ctx, a, b, q, ldq, gate, ldg, k_cache, v_cache, out, ldo);
  if (a.dim > 256 || a.vdim > 256) return launch_simt<__nv_bfloat16>(ctx, a, b, q, ldq, gate, ldg, k_cache, v_cache, out, ldo);
  WinParams p;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k_cache);
  p.v = static_cast<const __nv_bfloat16*>(v_cache);
  p.gate = static_cast<const __nv_bfloat16*>(gate);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.ldq = (long long)ldq;
  p.ldg = (long long)ldg;
  p.ldo = (long long)ldo;
  p.a = a;
  p.b = b;
  p.group = a.heads / a.kv_heads;
  p.dp = (a.dim + 15) / 16 * 16;
  p.part_o = p.part_ml = nullptr;
  p.n_splits = 1;
  const bool split = b.max_q <= 1;
  const int most = split ? 16 : kWaPairs;
  p.gb = p.group < most ? p.group : most;
  p.n_hb = (p.group + p.gb - 1) / p.gb;
  const int widths[] = {4, 8, 12, 16, 24, 32};
  int dvt = 32;
  for (int w : widths)
    if (8 * w >= a.vdim_pad) {
      dvt = w;
      break;
    }
  const int W = dvt * 8;
  const size_t k_row = (size_t)p.dp * 2 + 16, v_row = (size_t)W * 2 + 16, q_bytes = (split ? 16 : kWaPairs) * k_row;
  p.stages = 2;
  size_t smem = q_bytes + 2 * kWaKeys * (k_row + v_row);
  if (smem > 226 * 1024) {
    p.stages = 1;
    smem = q_bytes + kWaKeys * (k_row + v_row);
  }
  if (split) {
    const size_t merge = (size_t)4 * 16 * (W + 2) * sizeof(float);
    if (smem < merge) smem = merge;
  }
  TQ_REQUIRE(ctx, smem <= 226 * 1024, "window attention: %zu bytes of shared memory needed", smem);
  dim3 grid(1, (unsigned)(a.kv_heads * p.n_hb), (unsigned)b.n_seqs);
  TQ_REQUIRE(ctx, grid.y <= 65535 && grid.z <= 65535, "window attention: too many heads or sequences");
  if (split) {
    // about four CTAs per SM, at least two key tiles each
    long long tiles = (b.max_len + kWaKeys - 1) / kWaKeys;
    const long long win_tiles = ((long long)a.window - 1 + kWaKeys - 1) / kWaKeys + 1;
    if (win_tiles < tiles) tiles = win_tiles;
    if (a.pool) tiles += (seen_blocks(b.max_len - 1, a.window, a.pool) + kWaKeys - 1) / kWaKeys;
    const long long ctas = (long long)a.kv_heads * p.n_hb * b.n_seqs;
    long long n = (4ll * ctx->sm_count + ctas - 1) / ctas;
    if (n > tiles / 2) n = tiles / 2;
    if (n > kWaMaxSplits) n = kWaMaxSplits;
    if (n < 1) n = 1;
    p.n_splits = (int)n;
    grid.x = (unsigned)n;
    if (n > 1) {
      const size_t n_part = (size_t)b.rows * a.heads * n;
      if (int st = ensure_scratch(ctx, n_part * (W + 2) * sizeof(float))) return st;
      p.part_o = static_cast<float*>(ctx->scratch);
      p.part_ml = p.part_o + n_part * W;
    }
  } else {
    const int ppc = kWaPairs / p.gb;
    grid.x = (unsigned)((b.max_q + ppc - 1) / ppc);
  }
  int st;
  switch (dvt) {
    case 4: st = launch_mma<4>(ctx, p, split, smem, grid); break;
    case 8: st = launch_mma<8>(ctx, p, split, smem, grid); break;
    case 12: st = launch_mma<12>(ctx, p, split, smem, grid); break;
    case 16: st = launch_mma<16>(ctx, p, split, smem, grid); break;
    case 24: st = launch_mma<24>(ctx, p, split, smem, grid); break;
    default: st = launch_mma<32>(ctx, p, split, smem, grid); break;
  }
  if (st != TQ_OK) return st;
  if (p.n_splits > 1)
    TQ_CUDA(ctx, launch_k(ctx, window_combine_kernel, dim3((unsigned)((size_t)b.rows * a.heads)), dim3((unsigned)((a.vdim + 31) / 32 * 32)), 0,
                          (const float*)p.part_o, (const float*)p.part_ml, p.n_splits, W, a.heads, a.vdim, b.cache_row, a.out_scale, p.gate, p.ldg, p.out, p.ldo));
  return TQ_OK;
}

}  // namespace tq

using namespace tq;

extern "C" int tq_window_attention(tq_ctx* ctx, const tq_window_attn_config* cfg, int dtype, const void* q_dev, size_t ldq, const void* gate_dev,
                                   size_t ldg, const void* k_cache_dev, const void* v_cache_dev, size_t cache_rows, const int* seq_rows_dev,
                                   const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, size_t max_len,
                                   void* out_dev, size_t ldo) {
  return tq_window_attention_sinks(ctx, cfg, nullptr, dtype, q_dev, ldq, gate_dev, ldg, k_cache_dev, v_cache_dev, cache_rows, seq_rows_dev, row_pos_dev,
                                   cache_row_dev, n_seqs, rows, max_q, max_len, out_dev, ldo);
}

extern "C" int tq_window_attention_sinks(tq_ctx* ctx, const tq_window_attn_config* cfg, const float* sinks_dev, int dtype, const void* q_dev, size_t ldq,
                                         const void* gate_dev, size_t ldg, const void* k_cache_dev, const void* v_cache_dev, size_t cache_rows,
                                         const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows,
                                         size_t max_q, size_t max_len, void* out_dev, size_t ldo) {
  return tq_window_attention_pooled(ctx, cfg, sinks_dev, dtype, q_dev, ldq, gate_dev, ldg, k_cache_dev, v_cache_dev, cache_rows, 0, nullptr, nullptr, 0, 0, 1.f,
                                    seq_rows_dev, row_pos_dev, cache_row_dev, n_seqs, rows, max_q, max_len, out_dev, ldo);
}

extern "C" int tq_window_attention_pooled(tq_ctx* ctx, const tq_window_attn_config* cfg, const float* sinks_dev, int dtype, const void* q_dev, size_t ldq,
                                          const void* gate_dev, size_t ldg, const void* k_cache_dev, const void* v_cache_dev, size_t cache_rows,
                                          size_t pool, const void* pooled_keys_dev, const void* pooled_values_dev, size_t pool_rows, size_t max_seq,
                                          float out_scale, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs,
                                          size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, cfg && (dtype == TQ_BF16 || dtype == TQ_F32), "tq_window_attention: dtype must be bf16 or f32");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, q_dev && k_cache_dev && v_cache_dev && row_pos_dev && cache_row_dev && out_dev, "tq_window_attention: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || (rows == n_seqs && max_q == 1), "tq_window_attention: without row offsets every sequence brings one row");
  WindowAttn a;
  a.heads = (int)cfg->heads;
  a.kv_heads = (int)cfg->kv_heads;
  a.dim = (int)cfg->dim;
  a.vdim = (int)cfg->vdim;
  a.dim_pad = (int)((cfg->dim + 7) / 8 * 8);
  a.vdim_pad = (int)((cfg->vdim + 7) / 8 * 8);
  a.window = (int)cfg->window;
  a.scale = cfg->scale;
  a.softcap = cfg->softcap;
  a.sink = cfg->sink;
  a.sinks = sinks_dev;
  a.out_scale = out_scale;
  a.pool = (int)pool;
  a.pool_rows = (int)pool_rows;
  a.max_seq = (int)max_seq;
  a.pooled_keys = pooled_keys_dev;
  a.pooled_values = pooled_values_dev;
  RaggedBatch b;
  b.n_seqs = (int)n_seqs;
  b.rows = (int)rows;
  b.max_q = (int)max_q;
  b.max_len = (int)max_len;
  b.seq_rows = seq_rows_dev;
  b.row_pos = row_pos_dev;
  b.cache_row = cache_row_dev;
  b.cache_rows = cache_rows;
  return launch_window_attention(ctx, a, b, dtype, q_dev, ldq, gate_dev, ldg, k_cache_dev, v_cache_dev, out_dev, ldo);
}
