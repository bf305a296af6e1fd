// Differential attention (see diff_attention.cuh).
//
// bf16, head sizes up to 256: one kernel body in two forms.  The 16 rows of an mma.sync m16n8k16 tile are EIGHT
// (position, head) pairs in both maps: tile rows 0..7 are map 1, rows 8..15 map 2 of the same pairs.  Scores take one
// product per map (the other map's rows of A are zero), both into the same accumulator; the product with the values then
// serves both maps at once, and a lane ends up holding a1 and a2 of the same head and columns, so that the difference and
// the head norm need no exchange beyond the four lanes of a row.
//   * SPLIT = false (prefill): a CTA's eight warps own eight pairs each and all walk the same key tiles;
//   * SPLIT = true (one query per sequence): a CTA's four warps own the same eight pairs and take 16 of a tile's 64 keys
//     each; the tiles are also split over CTAs, and diff_combine_kernel merges the splits.
// Scores, softmax weights and their sums are f32; a weight enters the tensor core as two bf16 terms (16 significant bits).
// Key tiles of 64 rows arrive by cp.async, two in flight.  Only tiles with visible keys are visited: those of the kept
// first tokens, then those of the window.
//
// diff_attention_simt_kernel is the exact f32 form (and takes bf16 heads of any size).
#include "diff_attention.cuh"

#include <cuda_bf16.h>

#include <cfloat>

#include "attn_mma.cuh"
#include "common.cuh"

namespace tq {

constexpr int kDaKeys = 64;
constexpr int kDaMaxSplits = 64;

struct DiffParams {
  const __nv_bfloat16 *q, *k, *v;
  __nv_bfloat16* out;
  long long ldq, ldo;
  DiffAttn a;
  RaggedBatch b;
  int group, gb, n_hb;         // heads per KV head; heads per block; blocks per KV head
  int dp;                      // dim rounded up to 16
  int stages;
  int n_splits;                // SPLIT only
  float* part_o;               // [rows][heads][2][n_splits][16-column padded vdim]
  float* part_ml;              // [rows][heads][2][n_splits][2]
  int* err;
};

// DVT: value columns / 8 (padded to 16 columns, so even).
template <int DVT, bool SPLIT>
__global__ void __launch_bounds__(SPLIT ? 128 : 256, DVT > 16 ? 1 : SPLIT ? 3 : 2) diff_attention_kernel(const __grid_constant__ DiffParams p) {
  constexpr int kThreads = SPLIT ? 128 : 256;
  constexpr int kWarps = kThreads / 32;
  constexpr int NT = SPLIT ? 2 : 4;                 // 8-key tiles of scores a warp forms at a time
  constexpr int kSub = SPLIT ? 1 : kDaKeys / (8 * NT);   // such steps per key tile
  extern __shared__ __align__(128) uint8_t da_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int k_row = p.dp * 4 + 16;                  // bytes: both maps of a key, then a shift of one bank group per row
  constexpr int v_row = DVT * 16 + 16;
  const int q_rows = SPLIT ? 8 : 64;
  uint8_t* q_s = da_smem;
  uint8_t* k_s = q_s + (size_t)q_rows * k_row;
  uint8_t* v_s = k_s + (size_t)p.stages * kDaKeys * k_row;

  pdl_wait();
  pdl_launch_dependents();

  const int kvh = blockIdx.y / p.n_hb, hb = blockIdx.y % p.n_hb, b = blockIdx.z;
  const int gb = min(p.gb, p.group - hb * p.gb);    // heads of this block
  const int head0 = kvh * p.group + hb * p.gb;
  const int row0 = p.b.seq_rows ? p.b.seq_rows[b] : b;
  const int n_q = p.b.seq_rows ? p.b.seq_rows[b + 1] - row0 : 1;
  const int pos_per_cta = SPLIT ? 1 : 64 / p.gb;
  // first query of this CTA inside the sequence; the last queries see the most keys and go first
  const int i0 = SPLIT ? 0 : ((int)gridDim.x - 1 - (int)blockIdx.x) * pos_per_cta;
  if (i0 >= n_q || row0 < 0 || row0 + n_q > p.b.rows) return;
  const int i1 = min(i0 + pos_per_cta, n_q) - 1;
  const int p0 = p.b.row_pos[row0 + i0], p1 = p0 + (i1 - i0);
  const int crow = p.b.cache_row[row0 + i0];
  // every row of the range has to be in the cache (the embedding kernel has reported one that is not)
  const bool in_cache = crow >= p0 && p.b.cache_row[row0 + i1] == crow + (i1 - i0) && (size_t)(crow + (i1 - i0)) < p.b.cache_rows;
  if (!in_cache) return;
  const size_t seq0 = (size_t)(crow - p0);                 // cache row of the sequence's position 0
  const size_t ke = (size_t)p.a.kv_heads * 2 * p.a.dim_pad, ve = (size_t)p.a.kv_heads * p.a.vdim_pad;
  const __nv_bfloat16* kb = p.k + seq0 * ke + (size_t)kvh * 2 * p.a.dim_pad;
  const __nv_bfloat16* vb = p.v + seq0 * ve + (size_t)kvh * p.a.vdim_pad;

  // visible key tiles: the kept tokens' tiles that lie before the window's, then the window's
  const int lo = max(0, p0 - p.a.window + 1);
  const int lo_t = lo / kDaKeys, hi_t = p1 / kDaKeys;
  const int n_kept = min((min(p.a.keep_first, p1 + 1) + kDaKeys - 1) / kDaKeys, lo_t);
  const int n_list = n_kept + hi_t - lo_t + 1;
  int li0 = 0, li1 = n_list;
  if constexpr (SPLIT) {
    const int per = (n_list + p.n_splits - 1) / p.n_splits;
    li0 = min((int)blockIdx.x * per, n_list);
    li1 = min(li0 + per, n_list);
  }

  // ---- padding columns of shared memory must hold numbers
  const bool pad = p.dp != p.a.dim_pad || p.a.dim != p.a.dim_pad || DVT * 8 != p.a.vdim_pad;
  if (pad) {
    const int words = (int)(((size_t)q_rows * k_row + (size_t)p.stages * kDaKeys * (k_row + v_row)) / 16);
    for (int i = threadIdx.x; i < words; i += kThreads) reinterpret_cast<uint4*>(da_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
    __syncthreads();
  }
  const int kcm = p.a.dim_pad / 8, vcm = p.a.vdim_pad / 8;   // 16-byte pieces per map / value row
  // This thread copies piece `pc` of every row_step-th row of a tile (at most 96 pieces: a row has 2 * 32 + 32).
  const int per_row = 2 * kcm + vcm;
  const int row_step = kThreads / per_row;
  const int row_first = threadIdx.x / per_row, pc = threadIdx.x - row_first * per_row;
  const bool copies = row_first < row_step, is_v = pc >= 2 * kcm;
  const int mp_c = pc >= kcm ? 1 : 0;
  const __nv_bfloat16* src_c = is_v ? vb + (pc - 2 * kcm) * 8 : kb + pc * 8;
  const size_t src_ld = is_v ? ve : ke;
  const int dst_ld = is_v ? v_row : k_row;
  const uint32_t dst_c = smem_u32(is_v ? v_s + (pc - 2 * kcm) * 16 : k_s + mp_c * p.dp * 2 + (pc - mp_c * kcm) * 16);
  auto load_tile = [&](int li, int buf) {
    const int key0 = (li < n_kept ? li : lo_t + li - n_kept) * kDaKeys;
    if (copies) {
      const __nv_bfloat16* src = src_c + (size_t)(key0 + row_first) * src_ld;
      uint32_t dst = dst_c + (uint32_t)((buf * kDaKeys + row_first) * dst_ld);
      const int n_valid = p1 + 1 - key0;                   // rows at or beyond it become zeros
#pragma unroll 4
      for (int row = row_first; row < kDaKeys; row += row_step) {
        cp_async16(dst, row < n_valid ? src : src_c, row < n_valid);
        src += row_step * src_ld;
        dst += (uint32_t)(row_step * dst_ld);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (li0 < li1) load_tile(li0, 0);

  // ---- queries: pair r = 8 * warp + g (prefill) or g; both maps side by side like a key row
  if ((p.a.dim & 7) == 0 && (p.ldq & 7) == 0) {
    const int pm = p.a.dim / 8;                            // 16-byte pieces per map
    for (int i = threadIdx.x; i < q_rows * 2 * pm; i += kThreads) {
      const int r = i / (2 * pm), c = i - r * 2 * pm;
      const int mp = c >= pm;
      const int qi = SPLIT ? 0 : r / p.gb, hh = SPLIT ? r : r % p.gb;
      uint4 x = make_uint4(0u, 0u, 0u, 0u);
      if (i0 + qi <= i1 && (SPLIT || r < pos_per_cta * p.gb) && hh < gb)
        x = *reinterpret_cast<const uint4*>(p.q + (size_t)(row0 + i0 + qi) * p.ldq + (size_t)2 * (head0 + hh) * p.a.dim + c * 8);
      *reinterpret_cast<uint4*>(q_s + (size_t)r * k_row + mp * p.dp * 2 + (c - mp * pm) * 16) = x;
    }
  } else {
    for (int i = threadIdx.x; i < q_rows * 2 * p.a.dim; i += kThreads) {
      const int r = i / (2 * p.a.dim), c = i - r * 2 * p.a.dim;
      const int mp = c >= p.a.dim, d = c - mp * p.a.dim;
      const int qi = SPLIT ? 0 : r / p.gb, hh = SPLIT ? r : r % p.gb;
      __nv_bfloat16 x = __float2bfloat16_rn(0.f);
      if (i0 + qi <= i1 && (SPLIT || r < pos_per_cta * p.gb) && hh < gb)
        x = p.q[(size_t)(row0 + i0 + qi) * p.ldq + (size_t)(2 * (head0 + hh) + mp) * p.a.dim + d];
      *reinterpret_cast<__nv_bfloat16*>(q_s + (size_t)r * k_row + (mp * p.dp + d) * 2) = x;
    }
  }

  const int pr = SPLIT ? g : 8 * warp + g;                 // this lane's pair
  const int pqi = SPLIT ? 0 : pr / p.gb, phh = SPLIT ? pr : pr % p.gb;
  const bool live = i0 + pqi <= i1 && (SPLIT || pr < pos_per_cta * p.gb) && phh < gb;
  const int qpos = p0 + pqi;
  const uint8_t* qrow = q_s + (size_t)pr * k_row + 4 * t;

  float o[DVT][4];                                         // [columns 8j + 2t, +1] of map 1, then of map 2
#pragma unroll
  for (int j = 0; j < DVT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const float sl2 = p.a.scale * kLog2e;
  const int nks = p.dp / 16;

  for (int li = li0; li < li1; ++li) {
    const int buf = p.stages == 2 ? (li - li0) & 1 : 0;
    if (p.stages == 2 && li + 1 < li1) {
      load_tile(li + 1, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int tile = li < n_kept ? li : lo_t + li - n_kept;
    for (int sub = 0; sub < kSub; ++sub) {
      const int w0 = SPLIT ? 16 * warp : 8 * NT * sub;     // first key of the tile for this warp's step
      const int key0 = tile * kDaKeys + w0;
      if (key0 > p1) break;
      const uint8_t* kt = k_s + (buf * kDaKeys + w0) * k_row;
      const uint8_t* vt = v_s + (buf * kDaKeys + w0) * v_row;
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      // lanes 0..7 / 8..15 address the two k halves of map 1, lanes 16..23 / 24..31 those of map 2
      const uint8_t* kaddr = kt + (size_t)(lane & 7) * k_row + ((lane >> 3) & 1) * 16 + (lane >> 4) * p.dp * 2;
      for (int ks = 0; ks < nks; ++ks) {
        const uint32_t q10 = *reinterpret_cast<const uint32_t*>(qrow + 32 * ks), q11 = *reinterpret_cast<const uint32_t*>(qrow + 32 * ks + 16);
        const uint32_t q20 = *reinterpret_cast<const uint32_t*>(qrow + p.dp * 2 + 32 * ks), q21 = *reinterpret_cast<const uint32_t*>(qrow + p.dp * 2 + 32 * ks + 16);
        uint32_t kf[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n) ldmatrix4(kf[n], kaddr + 8 * n * k_row + 32 * ks);
#pragma unroll
        for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n], q10, 0u, q11, 0u, kf[n][0], kf[n][1]);
#pragma unroll
        for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n], 0u, q20, 0u, q21, kf[n][2], kf[n][3]);
      }
      // a step whose keys every query of the CTA sees needs no mask (rows without a query are never stored)
      const bool full = key0 + 8 * NT - 1 <= p0 && (p1 - key0 < p.a.window || key0 + 8 * NT <= p.a.keep_first);
      float mx[2] = {-INFINITY, -INFINITY};
      if (full) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            s[n][c] *= sl2;
            mx[c >> 1] = fmaxf(mx[c >> 1], s[n][c]);
          }
      } else {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int key = key0 + 8 * n + 2 * t + (c & 1);
            const bool ok = live && key <= qpos && (qpos - key < p.a.window || key < p.a.keep_first);
            s[n][c] = ok ? s[n][c] * sl2 : -INFINITY;
            mx[c >> 1] = fmaxf(mx[c >> 1], s[n][c]);
          }
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
    if (p.stages == 1 && li + 1 < li1) load_tile(li + 1, 0);
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
  }
  const int vd = p.a.vdim;

  if constexpr (!SPLIT) {
    if (!live) return;      // (a row's four lanes agree; the shuffles below stay inside them)
    const float w1 = 1.0f / l_run[0], w2 = p.a.lambda / l_run[1];
    float sq = 0.f;
#pragma unroll
    for (int j = 0; j < DVT; ++j)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const float v = o[j][c] * w1 - o[j][2 + c] * w2;
        o[j][c] = v;
        if (8 * j + 2 * t + c < vd) sq += v * v;
      }
    const uint32_t quad = 0xFu << (lane & 28);
    sq += __shfl_xor_sync(quad, sq, 1);
    sq += __shfl_xor_sync(quad, sq, 2);
    const float inv = p.a.out_scale / sqrtf(sq / (float)vd + p.a.eps);
    __nv_bfloat16* dst = p.out + (size_t)(row0 + i0 + pqi) * p.ldo + (size_t)(head0 + phh) * vd;
    const bool even = ((p.ldo | vd) & 1) == 0;
#pragma unroll
    for (int j = 0; j < DVT; ++j) {
      const int d = 8 * j + 2 * t;
      if (even) {
        if (d < vd) *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(o[j][0] * inv, o[j][1] * inv);
      } else {
        if (d < vd) dst[d] = __float2bfloat16_rn(o[j][0] * inv);
        if (d + 1 < vd) dst[d + 1] = __float2bfloat16_rn(o[j][1] * inv);
      }
    }
  } else {
    // ---- merge the four warps: [warp][16 rows][DVT * 8], rows 0..7 map 1, 8..15 map 2
    constexpr int W = DVT * 8;
    __syncthreads();                                       // (a CTA without tiles has not met one since it wrote q_s)
    float* mo = reinterpret_cast<float*>(da_smem);
    float* mml = mo + kWarps * 16 * W;
#pragma unroll
    for (int j = 0; j < DVT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) mo[((size_t)warp * 16 + g + 8 * (c >> 1)) * W + 8 * j + 2 * t + (c & 1)] = o[j][c];
    if (t == 0) {
      // (a finite stand-in for "no key seen": its weight is zero beside any real maximum)
      mml[(warp * 16 + g) * 2] = fmaxf(m_run[0], -FLT_MAX);
      mml[(warp * 16 + g) * 2 + 1] = l_run[0];
      mml[(warp * 16 + g + 8) * 2] = fmaxf(m_run[1], -FLT_MAX);
      mml[(warp * 16 + g + 8) * 2 + 1] = l_run[1];
    }
    __syncthreads();
    for (int h = warp; h < gb; h += kWarps) {              // a warp finishes a head
      float wt[2][kWarps], L[2], M[2];
#pragma unroll
      for (int mp = 0; mp < 2; ++mp) {
        M[mp] = -FLT_MAX;
        L[mp] = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) M[mp] = fmaxf(M[mp], mml[(w * 16 + h + 8 * mp) * 2]);
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
          wt[mp][w] = exp2f(mml[(w * 16 + h + 8 * mp) * 2] - M[mp]);
          L[mp] += mml[(w * 16 + h + 8 * mp) * 2 + 1] * wt[mp][w];
        }
      }
      float a[2][(W + 31) / 32];
#pragma unroll
      for (int i = 0; i < (W + 31) / 32; ++i)
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
          const int d = lane + 32 * i;
          float v = 0.f;
          if (d < W) {
#pragma unroll
            for (int w = 0; w < kWarps; ++w) v += mo[((size_t)w * 16 + h + 8 * mp) * W + d] * wt[mp][w];
          }
          a[mp][i] = v;
        }
      if (p.n_splits > 1) {
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
          const size_t pi = (((size_t)row0 * p.a.heads + head0 + h) * 2 + mp) * p.n_splits + blockIdx.x;
#pragma unroll
          for (int i = 0; i < (W + 31) / 32; ++i)
            if (lane + 32 * i < W) p.part_o[pi * W + lane + 32 * i] = a[mp][i];
          if (lane == 0) {
            p.part_ml[pi * 2] = M[mp];
            p.part_ml[pi * 2 + 1] = L[mp];
          }
        }
      } else {
        const float w1 = 1.0f / L[0], w2 = p.a.lambda / L[1];
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < (W + 31) / 32; ++i) {
          a[0][i] = a[0][i] * w1 - a[1][i] * w2;
          if (lane + 32 * i < vd) sq += a[0][i] * a[0][i];
        }
        sq = warp_sum(sq);
        const float inv = p.a.out_scale / sqrtf(sq / (float)vd + p.a.eps);
        __nv_bfloat16* dst = p.out + (size_t)row0 * p.ldo + (size_t)(head0 + h) * vd;
#pragma unroll
        for (int i = 0; i < (W + 31) / 32; ++i)
          if (lane + 32 * i < vd) dst[lane + 32 * i] = __float2bfloat16_rn(a[0][i] * inv);
      }
    }
  }
}

// Merges the splits of one (row, head), forms the difference and the head norm.  One CTA per head, a thread per column.
__global__ void __launch_bounds__(256) diff_combine_kernel(const float* part_o, const float* part_ml, int n_splits, int W, DiffAttn a,
                                                           const int* cache_row, __nv_bfloat16* out, long long ldo) {
  __shared__ float wgt[2][kDaMaxSplits];                   // weight of each split in the head's result, 1 / l and lambda in it
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, d = threadIdx.x;
  const size_t rh = blockIdx.x;                            // row * heads + head
  const int row = (int)(rh / a.heads), head = (int)(rh % a.heads);
  if (cache_row[row] < 0) return;
  for (int mp = warp; mp < 2; mp += (int)(blockDim.x >> 5)) {
    const float* ml = part_ml + (rh * 2 + mp) * n_splits * 2;
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      m[i] = s < n_splits ? ml[2 * s] : -FLT_MAX;
      l[i] = s < n_splits ? ml[2 * s + 1] : 0.f;
    }
    const float M = warp_max(fmaxf(m[0], m[1]));
    const float w0 = exp2f(m[0] - M), w1 = exp2f(m[1] - M);
    const float L = warp_sum(l[0] * w0 + l[1] * w1);
    const float f = (mp ? -a.lambda : 1.0f) / L;
    wgt[mp][lane] = w0 * f;
    wgt[mp][lane + 32] = w1 * f;
  }
  __syncthreads();
  float v = 0.f;
  if (d < a.vdim) {
    float acc[2] = {0.f, 0.f};
    const float* src = part_o + rh * 2 * n_splits * W + d;
#pragma unroll 8
    for (int s = 0; s < n_splits; ++s) {
      acc[0] += src[(size_t)s * W] * wgt[0][s];
      acc[1] += src[(size_t)(n_splits + s) * W] * wgt[1][s];
    }
    v = acc[0] + acc[1];
  }
  const float sq = warp_sum(v * v);
  if (lane == 0) red[warp] = sq;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += red[i];
  const float inv = a.out_scale / sqrtf(tot / (float)a.vdim + a.eps);
  if (d < a.vdim) out[(size_t)row * ldo + (size_t)head * a.vdim + d] = __float2bfloat16_rn(v * inv);
}

// ------------------------------------------------------------------------------------------------ f32 / any size
__device__ __forceinline__ float da_load(const float* p) { return *p; }
__device__ __forceinline__ float da_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void da_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void da_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// One CTA per (row, head); 128 keys at a time, one per thread; then every thread owns value columns.
template <typename T>
__global__ void __launch_bounds__(128) diff_attention_simt_kernel(const T* q, long long ldq, const T* k, const T* v, T* out, long long ldo,
                                                                  DiffAttn a, RaggedBatch b) {
  extern __shared__ float ds_smem[];
  float* qs = ds_smem;                       // [2][dim]
  float* acc = qs + 2 * a.dim;               // [2][vdim]
  float* pr = acc + 2 * a.vdim;              // [2][128]
  __shared__ float red[4];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = b.row_pos[row], crow = b.cache_row[row];
  if (crow < pos || (size_t)crow >= b.cache_rows) return;
  const int kvh = head / (a.heads / a.kv_heads);
  const size_t seq0 = (size_t)(crow - pos);
  const size_t ke = (size_t)a.kv_heads * 2 * a.dim_pad, ve = (size_t)a.kv_heads * a.vdim_pad;
  const T* kb = k + seq0 * ke + (size_t)kvh * 2 * a.dim_pad;
  const T* vb = v + seq0 * ve + (size_t)kvh * a.vdim_pad;
  for (int i = tid; i < 2 * a.dim; i += 128) qs[i] = da_load(q + (size_t)row * ldq + (size_t)2 * head * a.dim + i);
  for (int i = tid; i < 2 * a.vdim; i += 128) acc[i] = 0.f;
  __syncthreads();
  auto block_reduce = [&](float x, bool is_max) {
    x = is_max ? warp_max(x) : warp_sum(x);
    if (lane == 0) red[warp] = x;
    __syncthreads();
    const float r = is_max ? fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])) : (red[0] + red[1]) + (red[2] + red[3]);
    __syncthreads();
    return r;
  };
  const int lo = max(0, pos - a.window + 1), kept = min(a.keep_first, lo);
  const int n_vis = kept + pos - lo + 1;     // visible keys, in order: 0 .. kept-1, lo .. pos
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f};
  for (int c0 = 0; c0 < n_vis; c0 += 128) {
    const int c = c0 + tid, n = min(128, n_vis - c0);
    float sc[2] = {-FLT_MAX, -FLT_MAX};
    if (c < n_vis) {
      const int key = c < kept ? c : lo + c - kept;
      const T* kr = kb + (size_t)key * ke;
      for (int mp = 0; mp < 2; ++mp) {
        float s = 0.f;
        for (int d = 0; d < a.dim; ++d) s = fmaf(qs[mp * a.dim + d], da_load(kr + mp * a.dim_pad + d), s);
        sc[mp] = s * a.scale;
      }
    }
    float alpha[2];
    for (int mp = 0; mp < 2; ++mp) {
      const float mn = fmaxf(m_run[mp], block_reduce(sc[mp], true));
      alpha[mp] = expf(m_run[mp] - mn);
      m_run[mp] = mn;
      const float w = c < n_vis ? expf(sc[mp] - mn) : 0.f;
      pr[mp * 128 + tid] = w;
      l_run[mp] = l_run[mp] * alpha[mp] + block_reduce(w, false);   // (its barriers also publish pr)
    }
    for (int d = tid; d < a.vdim; d += 128) {
      float a1 = acc[d] * alpha[0], a2 = acc[a.vdim + d] * alpha[1];
      for (int j = 0; j < n; ++j) {
        const int cj = c0 + j, key = cj < kept ? cj : lo + cj - kept;
        const float x = da_load(vb + (size_t)key * ve + d);
        a1 = fmaf(pr[j], x, a1);
        a2 = fmaf(pr[128 + j], x, a2);
      }
      acc[d] = a1;
      acc[a.vdim + d] = a2;
    }
    __syncthreads();
  }
  float sq = 0.f;
  for (int d = tid; d < a.vdim; d += 128) {
    const float o = acc[d] / l_run[0] - a.lambda * (acc[a.vdim + d] / l_run[1]);
    acc[d] = o;
    sq += o * o;
  }
  const float inv = a.out_scale / sqrtf(block_reduce(sq, false) / (float)a.vdim + a.eps);
  for (int d = tid; d < a.vdim; d += 128) da_store(out + (size_t)row * ldo + (size_t)head * a.vdim + d, acc[d] * inv);
}

// ------------------------------------------------------------------------------------------------ launch
template <typename T>
static int launch_simt(tq_ctx* ctx, const DiffAttn& a, const RaggedBatch& b, const void* q, size_t ldq, const void* k, const void* v,
                       void* out, size_t ldo) {
  const size_t smem = ((size_t)2 * a.dim + 2 * a.vdim + 256) * sizeof(float);
  if (smem > 200 * 1024) return fail(ctx, TQ_EUNSUPPORTED, "differential attention: head sizes %d / %d are too large", a.dim, a.vdim);
  if (smem > 48 * 1024)
    TQ_CUDA(ctx, cudaFuncSetAttribute(diff_attention_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, diff_attention_simt_kernel<T>, dim3((unsigned)b.rows, (unsigned)a.heads), dim3(128), smem, static_cast<const T*>(q),
                        (long long)ldq, static_cast<const T*>(k), static_cast<const T*>(v), static_cast<T*>(out), (long long)ldo, a, b));
  return TQ_OK;
}

template <int DVT>
static int launch_mma(tq_ctx* ctx, DiffParams& p, bool split, size_t smem, dim3 grid) {
  auto go = [&](auto kern, int threads) -> int {
    if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3((unsigned)threads), smem, p));
    return TQ_OK;
  };
  return split ? go(diff_attention_kernel<DVT, true>, 128) : go(diff_attention_kernel<DVT, false>, 256);
}

int launch_diff_attention(tq_ctx* ctx, const DiffAttn& a, const RaggedBatch& b, int dtype, const void* q, size_t ldq, const void* k_cache,
                          const void* v_cache, void* out, size_t ldo) {
  TQ_REQUIRE(ctx, a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0, "differential attention: heads must be a multiple of kv_heads");
  TQ_REQUIRE(ctx, a.dim > 0 && a.vdim > 0 && a.dim_pad >= a.dim && a.vdim_pad >= a.vdim && a.dim_pad % 8 == 0 && a.vdim_pad % 8 == 0,
             "differential attention: bad head sizes");
  TQ_REQUIRE(ctx, a.window > 0 && a.keep_first >= 0, "differential attention: bad window");
  if (b.rows == 0 || b.n_seqs == 0) return TQ_OK;
  if (dtype == TQ_F32) return launch_simt<float>(ctx, a, b, q, ldq, k_cache, v_cache, out, ldo);
  if (a.dim > 256 || a.vdim > 256) return launch_simt<__nv_bfloat16>(ctx, a, b, q, ldq, k_cache, v_cache, out, ldo);
  DiffParams p;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.k = static_cast<const __nv_bfloat16*>(k_cache);
  p.v = static_cast<const __nv_bfloat16*>(v_cache);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.ldq = (long long)ldq;
  p.ldo = (long long)ldo;
  p.a = a;
  p.b = b;
  p.err = ctx->dev_err;
  p.group = a.heads / a.kv_heads;
  p.dp = (a.dim + 15) / 16 * 16;
  p.part_o = p.part_ml = nullptr;
  p.n_splits = 1;
  const bool split = b.max_q <= 1;
  p.gb = split ? (p.group < 8 ? p.group : 8) : (p.group < 64 ? p.group : 64);
  p.n_hb = (p.group + p.gb - 1) / p.gb;
  const int widths[] = {4, 8, 12, 16, 24, 32};
  int dvt = 32;
  for (int w : widths)
    if (8 * w >= a.vdim_pad) {
      dvt = w;
      break;
    }
  const int W = dvt * 8;
  const size_t k_row = (size_t)p.dp * 4 + 16, v_row = (size_t)W * 2 + 16, q_bytes = (split ? 8 : 64) * k_row;
  p.stages = 2;
  size_t smem = q_bytes + 2 * kDaKeys * (k_row + v_row);
  if (smem > 226 * 1024) {
    p.stages = 1;
    smem = q_bytes + kDaKeys * (k_row + v_row);
  }
  if (split) {
    const size_t merge = (size_t)4 * 16 * (W + 2) * sizeof(float);
    if (smem < merge) smem = merge;
  }
  TQ_REQUIRE(ctx, smem <= 226 * 1024, "differential attention: %zu bytes of shared memory needed", smem);
  dim3 grid(1, (unsigned)(a.kv_heads * p.n_hb), (unsigned)b.n_seqs);
  if (split) {
    // about four CTAs per SM, at least two key tiles each
    const int kept_tiles = (a.keep_first + kDaKeys - 1) / kDaKeys;
    long long tiles = (b.max_len + kDaKeys - 1) / kDaKeys;
    const long long win_tiles = ((long long)a.window - 1 + kDaKeys - 1) / kDaKeys + 1 + kept_tiles;
    if (win_tiles < tiles) tiles = win_tiles;
    const long long ctas = (long long)a.kv_heads * p.n_hb * b.n_seqs;
    long long n = (4ll * ctx->sm_count + ctas - 1) / ctas;
    if (n > tiles / 2) n = tiles / 2;
    if (n > kDaMaxSplits) n = kDaMaxSplits;
    if (n < 1) n = 1;
    p.n_splits = (int)n;
    grid.x = (unsigned)n;
    if (n > 1) {
      const size_t n_part = (size_t)b.rows * a.heads * 2 * n;
      if (int st = ensure_scratch(ctx, n_part * (W + 2) * sizeof(float))) return st;
      p.part_o = static_cast<float*>(ctx->scratch);
      p.part_ml = p.part_o + n_part * W;
    }
  } else {
    const int ppc = 64 / p.gb;
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
    TQ_CUDA(ctx, launch_k(ctx, diff_combine_kernel, dim3((unsigned)((size_t)b.rows * a.heads)), dim3((unsigned)((a.vdim + 31) / 32 * 32)), 0,
                          (const float*)p.part_o, (const float*)p.part_ml, p.n_splits, W, a, b.cache_row, p.out, p.ldo));
  return TQ_OK;
}

}  // namespace tq
