// Dense linear layers (see dense.cuh): GEMV for few rows, tcgen05 GEMM for many, f32 GEMM, weight handles and the
// C entry points tq_dweight_* / tq_dlinear / tq_clamped_glu.
#include "dense.cuh"

#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "qgemm_umma.cuh"
#include "tensormap.h"

namespace tq {

// ------------------------------------------------------------------------------------------------ GEMV, 1..8 rows
constexpr int kGvWarps = 8;
constexpr int kGvThreads = 32 * kGvWarps;
constexpr int kGvPad = 128;         // weight rows are padded to this many columns

struct GemvParams {
  const __nv_bfloat16* w;
  int kpad, n_rb;                   // n_rb: 16-row blocks
  const __nv_bfloat16* x;
  long long ldx;
  int m, cols;
  const float* h;                   // RMSNorm prologue (x is null then)
  long long ldh;
  const int* h_rows;
  const __nv_bfloat16* gain;
  float eps;
  DenseGroups grp;                  // GROUPED only
  DenseEpilogue epi;
};

// 32 bytes of a weight row: read once, not kept in L1, first to leave L2.
struct Frag32 {
  uint32_t v[8];
};
__device__ __forceinline__ Frag32 ldg_stream(const void* p) {
  Frag32 f;
  asm volatile("ld.global.nc.L1::no_allocate.L2::evict_first.v8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
               : "=r"(f.v[0]), "=r"(f.v[1]), "=r"(f.v[2]), "=r"(f.v[3]), "=r"(f.v[4]), "=r"(f.v[5]), "=r"(f.v[6]), "=r"(f.v[7])
               : "l"(p));
  return f;
}

// The first n (at most 8) of eight bf16 values, zeros behind them.
__device__ __forceinline__ uint4 x_tail(const void* src, int n) {
  const uint16_t* e = static_cast<const uint16_t*>(src);
  uint32_t w[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) w[j] = (2 * j < n ? (uint32_t)e[2 * j] : 0u) | (2 * j + 1 < n ? (uint32_t)e[2 * j + 1] << 16 : 0u);
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// A CTA walks 16-row blocks (grid-stride); its eight warps take the k chunks of a block in turn and meet
// in shared memory.  Lane 4g + t holds bytes 32t .. 32t + 31 of rows g and g + 8 of every 64-k step (a row's four lanes
// read one 128-byte line): words 2i, 2i + 1 are the two k halves of MMA i; the activations are read the same way.  The loads of
// the next step -- of the next block too -- are issued before the current step is multiplied, and the first ones before
// the kernel waits for its predecessor (weights do not change).  The activations sit in shared memory.
// GROUPED: a CTA walks a contiguous range of (job, 16-row block) pairs and stages a job's activations when it comes to it.
template <bool GROUPED>
__global__ void __launch_bounds__(kGvThreads, 2) dgemv_kernel(const __grid_constant__ GemvParams p) {
  constexpr int U = 2;                               // 64-k loads per row and step: 32 registers in flight
  constexpr int kGvChunk = 64 * U;                   // k per warp step
  extern __shared__ __align__(16) uint8_t gv_smem[];
  __shared__ float red[2][kGvWarps][128];
  __shared__ float ssq[kGvWarps];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n_ch = p.kpad / kGvChunk;
  const size_t row_bytes = (size_t)p.kpad * 2;
  const uint8_t* wb = reinterpret_cast<const uint8_t*>(p.w) + (size_t)g * row_bytes + 32 * t;

  Frag32 nxt[U][2];
  auto load = [&](int rb, int c) {
    const uint8_t* src = wb + (size_t)rb * 16 * row_bytes + (size_t)c * (kGvChunk * 2);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      nxt[u][0] = ldg_stream(src + 128 * u);
      nxt[u][1] = ldg_stream(src + 8 * row_bytes + 128 * u);
    }
  };
  // tile -> 16-row block of the weight
  int tile = blockIdx.x, tile_end = p.n_rb;
  const int tile_step = GROUPED ? 1 : gridDim.x;
  auto row_block = [&](int tl) {
    if constexpr (!GROUPED) return tl;
    return p.grp.jobs[tl / p.n_rb].x * (int)(p.grp.group_rows / 16) + tl % p.n_rb;
  };
  if constexpr (GROUPED) {
    pdl_wait();
    pdl_launch_dependents();
    const long long n = (long long)min(*p.grp.n_jobs, p.grp.max_jobs) * p.n_rb;
    tile = (int)(n * blockIdx.x / gridDim.x);
    tile_end = (int)(n * (blockIdx.x + 1) / gridDim.x);
    if (tile >= tile_end) return;
  }
  if (tile < tile_end && warp < n_ch) load(row_block(tile), warp);

  if constexpr (!GROUPED) {
    pdl_wait();
    pdl_launch_dependents();
  }

  const size_t xs_stride = row_bytes + 16;   // bytes; 16 mod 32: two rows' reads, 32 bytes apart, do not meet in a bank
  int m_rows = p.m, m_first = 0, m_shift = 0, job = -1;
  if constexpr (!GROUPED) {
    if (p.h) {
      int wpr = kGvWarps;                        // warps per row
      while (wpr * p.m > kGvWarps) wpr >>= 1;
      const int row = warp / wpr, part = warp % wpr;
      const bool mine = row < p.m;
      const float* src = p.h + (size_t)(mine ? (p.h_rows ? p.h_rows[row] : row) : 0) * p.ldh;
      const bool vec = (p.cols & 3) == 0 && (p.ldh & 3) == 0;
      float sq = 0.f;
      if (mine) {
        if (vec) {
#pragma unroll 4
          for (int d = 4 * (part * 32 + lane); d < p.cols; d += 128 * wpr) {
            const float4 v = *reinterpret_cast<const float4*>(src + d);
            sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
          }
        } else {
          for (int d = part * 32 + lane; d < p.cols; d += 32 * wpr) sq += src[d] * src[d];
        }
      }
      sq = warp_sum(sq);
      if (lane == 0) ssq[warp] = sq;
      __syncthreads();
      if (mine) {
        float tot = 0.f;
        for (int i = 0; i < wpr; ++i) tot += ssq[row * wpr + i];
        const float inv = 1.0f / sqrtf(tot / (float)p.cols + p.eps);
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(gv_smem + row * xs_stride);
        if (vec) {
#pragma unroll 4
          for (int d = 4 * (part * 32 + lane); d < p.cols; d += 128 * wpr) {
            const float4 v = *reinterpret_cast<const float4*>(src + d);
            const uint2 gr = *reinterpret_cast<const uint2*>(p.gain + d);
            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x * inv * bf16_bits_to_float(gr.x & 0xFFFFu), v.y * inv * bf16_bits_to_float(gr.x >> 16));
            const __nv_bfloat162 b = __floats2bfloat162_rn(v.z * inv * bf16_bits_to_float(gr.y & 0xFFFFu), v.w * inv * bf16_bits_to_float(gr.y >> 16));
            *reinterpret_cast<uint2*>(dst + d) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
          }
        } else {
          for (int d = part * 32 + lane; d < p.cols; d += 32 * wpr) dst[d] = __float2bfloat16_rn(src[d] * inv * __bfloat162float(p.gain[d]));
        }
        for (int d = p.cols + part * 32 + lane; d < p.kpad; d += 32 * wpr) dst[d] = __float2bfloat16_rn(0.f);
      }
    } else {
      const int vpr = p.kpad / 8;
      for (int i = threadIdx.x; i < p.m * vpr; i += kGvThreads) {
        const int row = i / vpr, c = i % vpr;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        const __nv_bfloat16* src = p.x + (size_t)row * p.ldx + 8 * c;
        if (8 * c + 8 <= p.cols) v = *reinterpret_cast<const uint4*>(src);
        else if (8 * c < p.cols) v = x_tail(src, p.cols - 8 * c);
        *reinterpret_cast<uint4*>(gv_smem + row * xs_stride + 16 * c) = v;
      }
    }
    __syncthreads();
  }
  bool live = g < m_rows;
  const uint8_t* xrow = gv_smem + (live ? g : 0) * xs_stride + 32 * t;

  int buf = 0;
  for (; tile < tile_end; tile += tile_step) {
    if constexpr (GROUPED) {
      if (tile / p.n_rb != job) {                // (the barrier of the previous block was behind its last read of the activations)
        job = tile / p.n_rb;
        const int4 jb = p.grp.jobs[job];
        m_first = jb.y;
        m_shift = jb.w;
        m_rows = min(jb.z, p.grp.chunk);
        const int vpr = p.kpad / 8;
        for (int i = threadIdx.x; i < m_rows * vpr; i += kGvThreads) {
          const int row = i / vpr, c = i % vpr;
          const int xr = p.grp.x_rows ? p.grp.x_rows[m_first + row] : m_first + row;
          uint4 v = make_uint4(0u, 0u, 0u, 0u);
          const __nv_bfloat16* src = p.x + (size_t)xr * p.ldx + 8 * c;
          if (8 * c + 8 <= p.cols) v = *reinterpret_cast<const uint4*>(src);
          else if (8 * c < p.cols) v = x_tail(src, p.cols - 8 * c);
          *reinterpret_cast<uint4*>(gv_smem + row * xs_stride + 16 * c) = v;
        }
        __syncthreads();
        live = g < m_rows;
        xrow = gv_smem + (live ? g : 0) * xs_stride + 32 * t;
      }
    }
    const bool last_tile = tile + tile_step >= tile_end;
    const int rb = row_block(tile), rb_next = last_tile ? 0 : row_block(tile + tile_step);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int c = warp; c < n_ch; c += kGvWarps) {
      Frag32 cur[U][2];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        cur[u][0] = nxt[u][0];
        cur[u][1] = nxt[u][1];
      }
      const bool more = c + kGvWarps < n_ch;
      if (more || !last_tile) load(more ? rb : rb_next, more ? c + kGvWarps : warp);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        uint4 xa = make_uint4(0u, 0u, 0u, 0u), xb = xa;
        if (live) {
          const uint8_t* xp = xrow + (size_t)c * (kGvChunk * 2) + 128 * u;
          xa = *reinterpret_cast<const uint4*>(xp);
          xb = *reinterpret_cast<const uint4*>(xp + 16);
        }
        const uint32_t xw[8] = {xa.x, xa.y, xa.z, xa.w, xb.x, xb.y, xb.z, xb.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
          mma_bf16_16816(acc, cur[u][0].v[2 * i], cur[u][1].v[2 * i], cur[u][0].v[2 * i + 1], cur[u][1].v[2 * i + 1], xw[2 * i], xw[2 * i + 1]);
      }
    }
    // rows g, g + 8 x activation rows 2t, 2t + 1
    float* part = red[buf][warp];
    part[g * 8 + 2 * t] = acc[0];
    part[g * 8 + 2 * t + 1] = acc[1];
    part[(g + 8) * 8 + 2 * t] = acc[2];
    part[(g + 8) * 8 + 2 * t + 1] = acc[3];
    __syncthreads();
    const int row = threadIdx.x >> 3, m = threadIdx.x & 7;
    if (row < 16 && m < m_rows) {
      const DenseDst d = dense_dst(p.epi, (GROUPED ? tile % p.n_rb : rb) * 16 + row);
      if (d.kind != DENSE_GLU || row < 8) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kGvWarps; ++w) v += red[buf][w][row * 8 + m];
        const float scale = p.epi.row_scale ? p.epi.row_scale[m_first + m_shift + m] : 1.f;
        v *= scale;
        if (d.kind == DENSE_GLU) {
          float up = 0.f;
#pragma unroll
          for (int w = 0; w < kGvWarps; ++w) up += red[buf][w][(row + 8) * 8 + m];
          v = dense_glu(p.epi, v, up * scale);
        }
        dense_store(p.epi, d, m_first + m_shift + m, v);
      }
    }
    buf ^= 1;
  }
}

// ------------------------------------------------------------------------------------------------ tcgen05 GEMM
// The weights are the UMMA M operand (128 features per tile), the activation rows the N operand (16..256), both K-major
// in the 128-byte swizzle; D[128 x rows] in tensor memory.  Warp 0 copies, warp 1 multiplies, warps 4..11 store.
constexpr int kDuThreads = 384;
constexpr int kDuEpiWarp0 = 4, kDuEpiWarps = 8;
constexpr int kDuMaxStages = 12;
constexpr int kDuHeader = 1024;

struct DUmmaParams {
  int m, ntok, stages;
  int n_ft, n_tt, splits, n_tiles;   // feature tiles, row tiles, K splits; n_tiles = product
  int kb_total, kb_per_split;        // 64-k steps
  int n_acc, acc_stride, tmem_cols;
  float* partial;                    // [splits][m][n_ft * 128], splits > 1
  int* counters;                     // one per (feature tile, row tile), zero between launches
  int grouped;                       // tiles are (job, feature tile), listed by grp (n_tiles bounds them)
  DenseGroups grp;
  DenseEpilogue epi;
  int* err;
};

__global__ void __launch_bounds__(kDuThreads, 1)
dgemm_umma_kernel(const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map, const __grid_constant__ DUmmaParams p) {
  extern __shared__ uint8_t du_smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(du_smem);
  uint64_t* empty = full + kDuMaxStages;
  uint64_t* acc_full = empty + kDuMaxStages;
  uint64_t* acc_empty = acc_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* failed = reinterpret_cast<volatile int*>(tmem_slot + 1);
  volatile int* last_flag = failed + 1;
  const uint32_t base_u32 = smem_u32(du_smem);
  uint8_t* tiles_s = du_smem + kDuHeader + ((1024 - ((base_u32 + kDuHeader) & 1023)) & 1023);
  const uint32_t stage_bytes = (uint32_t)(kUmmaRows + p.ntok) * 128u;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int S = p.stages;

  if (threadIdx.x == 0) {
    for (int s = 0; s < S; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(&acc_full[a], 1);
      mbar_init(&acc_empty[a], kDuEpiWarps);
    }
    *failed = 0;
    mbar_init_fence();
  }
  if (warp == 2) tmem_alloc(tmem_slot, (uint32_t)p.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_d = *tmem_slot;

  auto give_up = [&](int code) {
    *failed = 1;
    atomicCAS(p.err, 0, code);
  };
  // tile -> (feature tile, row tile, K split): splits fastest, then row tiles, so that the CTAs of a wave share weights
  // (grouped: tt is the job)
  auto coords = [&](int tile, int& ft, int& tt, int& kb0, int& kbn, int& z) {
    if (p.grouped) {
      z = kb0 = 0;
      kbn = p.kb_total;
      tt = tile / p.n_ft;
      ft = tile % p.n_ft;
      return;
    }
    z = tile % p.splits;
    const int q = tile / p.splits;
    tt = q % p.n_tt;
    ft = q / p.n_tt;
    kb0 = z * p.kb_per_split;
    kbn = min(p.kb_per_split, p.kb_total - kb0);
  };

  // the number of tiles and a tile's first weight row / activation row; grouped: only behind the wait
  auto tiles_total = [&]() { return p.grouped ? min(*p.grp.n_jobs, p.grp.max_jobs) * p.n_ft : p.n_tiles; };
  auto w_row = [&](int ft, int tt) { return ft * kUmmaRows + (p.grouped ? p.grp.jobs[tt].x * (int)p.grp.group_rows : 0); };
  auto x_row = [&](int tt) { return p.grouped ? p.grp.jobs[tt].y : tt * p.ntok; };

  if (warp == 0) {
    if (lane == 0) {
      // The weights of the first stages do not depend on the previous kernel: their copies start before the wait.
      int ft, tt, kb0, kbn, z;
      int pre = 0;
      if (!p.grouped && (int)blockIdx.x < p.n_tiles) {
        coords(blockIdx.x, ft, tt, kb0, kbn, z);
        pre = min(S, kbn);
        for (int s = 0; s < pre; ++s) {
          mbar_arrive_expect_tx(&full[s], stage_bytes);
          tma_load_2d(tiles_s + (size_t)s * stage_bytes, &w_map, (kb0 + s) * kUmmaK, ft * kUmmaRows, &full[s]);
        }
      }
      pdl_wait();
      int s = 0;
      uint32_t ph = 0;
      bool ok = true;
      const int n_tiles = tiles_total();
      for (int tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x) {
        coords(tile, ft, tt, kb0, kbn, z);
        const int wr = w_row(ft, tt), xr = x_row(tt);
        for (int kb = 0; kb < kbn; ++kb) {
          uint8_t* st = tiles_s + (size_t)s * stage_bytes;
          if (pre > 0) {
            --pre;
          } else {
            ok = !*failed && mbar_wait_spin(&empty[s], ph ^ 1u);
            if (!ok) { give_up(DERR_EMPTY_WAIT); break; }
            mbar_arrive_expect_tx(&full[s], stage_bytes);
            tma_load_2d(st, &w_map, (kb0 + kb) * kUmmaK, wr, &full[s]);
          }
          tma_load_2d(st + kUmmaRows * 128, &x_map, (kb0 + kb) * kUmmaK, xr, &full[s]);
          if (++s == S) {
            s = 0;
            ph ^= 1u;
          }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (p.grouped) pdl_wait();
    const int n_tiles = tiles_total();
    const bool leader = elect_one();
    const uint32_t idesc = umma_idesc_bf16(p.ntok);
    const uint64_t desc0 = umma_desc_sw128(tiles_s);
    const uint32_t stage_u = stage_bytes >> 4, b_off = (uint32_t)(kUmmaRows * 128) >> 4;
    int s = 0, a = 0;
    uint32_t ph = 0, aph = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x) {
      int ft, tt, kb0, kbn, z;
      coords(tile, ft, tt, kb0, kbn, z);
      ok = !*failed && mbar_wait_spin(&acc_empty[a], aph ^ 1u);
      if (!ok) { give_up(DERR_TMEM); break; }
      tc_fence_after();
      const uint32_t acc = tmem_d + (uint32_t)(a * p.acc_stride);
      for (int kb = 0; kb < kbn; ++kb) {
        ok = !*failed && mbar_wait_spin(&full[s], ph);
        if (!ok) { give_up(DERR_FULL_WAIT); break; }
        tc_fence_after();
        if (leader) {
          const uint64_t ad = desc0 + (uint64_t)((uint32_t)s * stage_u);
#pragma unroll
          for (int k16 = 0; k16 < kUmmaK / 16; ++k16) umma_f16(acc, ad + 2 * k16, ad + b_off + 2 * k16, idesc, (kb | k16) != 0);
          umma_commit(&empty[s]);
        }
        __syncwarp();
        if (++s == S) {
          s = 0;
          ph ^= 1u;
        }
      }
      if (!ok) break;
      if (leader) umma_commit(&acc_full[a]);
      __syncwarp();
      if (++a == p.n_acc) {
        a = 0;
        aph ^= 1u;
      }
    }
  } else if (warp >= kDuEpiWarp0) {
    pdl_wait();
    pdl_launch_dependents();
    const int q = warp & 3, half = (warp - kDuEpiWarp0) >> 2;
    const int et = threadIdx.x - 32 * kDuEpiWarp0;     // 0..255
    int a = 0;
    uint32_t aph = 0;
    const int n_pad = p.n_ft * kUmmaRows;
    const int n_tiles = tiles_total();
    for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x) {
      int ft, tt, kb0, kbn, z;
      coords(tile, ft, tt, kb0, kbn, z);
      // (after a failure every warp still walks all tiles, without touching memory: the named barriers below stay matched)
      const bool good = __all_sync(0xffffffffu, !*failed && mbar_wait_spin(&acc_full[a], aph));
      if (!good) give_up(DERR_TMEM);
      tc_fence_after();
      const int row = ft * kUmmaRows + 32 * q + lane;
      const int m0 = x_row(tt) + (p.grouped ? p.grp.jobs[tt].w : 0), m_n = good ? min(p.ntok, p.grouped ? p.grp.jobs[tt].z : p.m - m0) : 0;
      const uint32_t t_addr = tmem_d + (uint32_t)(a * p.acc_stride) + ((uint32_t)(32 * q) << 16);
      const DenseDst dst = dense_dst(p.epi, row);
      for (int c0 = 16 * half; c0 < m_n; c0 += 32) {
        float v[16];
        tmem_ld16(t_addr + (uint32_t)c0, v);
        const int n = min(16, m_n - c0), mb = m0 + c0;
        if (p.splits > 1) {
          float* pp = p.partial + ((size_t)z * p.m + mb) * n_pad + row;
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (j < n && dst.base) __stcg(pp + (size_t)j * n_pad, v[j]);
          continue;
        }
        if (p.epi.row_scale) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (j < n) v[j] *= p.epi.row_scale[mb + j];
        }
        // a half-warp's rows share a section, so the shuffles below are only ever needed by lanes that agree on the kind
        const bool glu = dst.kind == DENSE_GLU;
        if (__any_sync(0xffffffffu, glu)) {
          // lanes with (row & 8) == 0 hold gates, the others the matching ups: of every two columns the gate lanes
          // finish the first and the up lanes the second
          const bool upper = lane & 8;
#pragma unroll
          for (int j = 0; j < 16; j += 2) {
            const float give = upper ? v[j] : v[j + 1];
            const float got = __shfl_xor_sync(0xffffffffu, give, 8);
            if (glu) {
              const float val = upper ? dense_glu(p.epi, got, v[j + 1]) : dense_glu(p.epi, v[j], got);
              const int jj = upper ? j + 1 : j;
              if (jj < n) dense_store(p.epi, dst, mb + jj, val);
            }
          }
          if (glu) continue;
        }
        if (dst.kind == DENSE_RESID) {
          if (dst.base) {
            float old[16];
#pragma unroll
            for (int j = 0; j < 16; ++j)
              if (j < n) old[j] = *reinterpret_cast<const float*>(dst.base + (long long)(mb + j) * dst.ld);
#pragma unroll
            for (int j = 0; j < 16; ++j)
              if (j < n) *reinterpret_cast<float*>(dst.base + (long long)(mb + j) * dst.ld) = old[j] + p.epi.mult * v[j];
          }
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (j < n) dense_store(p.epi, dst, mb + j, v[j]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[a]);
      if (++a == p.n_acc) {
        a = 0;
        aph ^= 1u;
      }
      if (p.splits > 1) {
        // the CTA that counts in last adds the tile's partials in split order (the same bits whichever CTA that is)
        __threadfence();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (et == 0) {
          int* c = p.counters + ft * p.n_tt + tt;
          const int seen = atomicAdd(c, 1);
          *last_flag = seen == p.splits - 1;
          if (seen == p.splits - 1) *c = 0;
          __threadfence();
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (*last_flag) {
          __threadfence();
          const size_t plane = (size_t)p.m * n_pad;
          // the 256 threads: F features (as many as the tile has) x 256 / F groups of four rows
          int F = kUmmaRows;
          while (F > 16 && ft * kUmmaRows + F / 2 >= p.epi.s[p.epi.n - 1].row_end) F >>= 1;
          const int mrow = ft * kUmmaRows + (et & (F - 1)), rows_step = 4 * (256 / F);
          const DenseDst md = dense_dst(p.epi, mrow);
          const bool upper = et & 8;
          for (int r0 = 0; r0 < m_n; r0 += rows_step) {       // (the same number of turns for every lane: they exchange below)
            const int c0 = r0 + 4 * (et / F);
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            const int n = md.base ? min(4, m_n - c0) : 0, mb = m0 + c0;
            const float* src = p.partial + (size_t)mb * n_pad + mrow;
            for (int z0 = 0; z0 < p.splits; z0 += 4) {        // sixteen loads in flight, added in split order
              float part[4][4];
#pragma unroll
              for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) part[i][j] = z0 + i < p.splits && j < n ? __ldcg(src + (size_t)(z0 + i) * plane + (size_t)j * n_pad) : 0.f;
#pragma unroll
              for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) v[j] += part[i][j];
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const float other = __shfl_xor_sync(0xffffffffu, v[j], 8);
              if (j >= n) continue;
              if (md.kind == DENSE_GLU) {
                if (!upper) dense_store(p.epi, md, mb + j, dense_glu(p.epi, v[j], other));
              } else {
                dense_store(p.epi, md, mb + j, v[j]);
              }
            }
          }
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");     // last_flag is read before the next tile rewrites it
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*failed && threadIdx.x == 0) {
    // copies and products that are still in flight target this CTA's memories: give them time to land before leaving
    for (int i = 0; i < 10000; ++i) __nanosleep(1000);
  }
  __syncthreads();
  if (warp == 2) tmem_dealloc(tmem_d, (uint32_t)p.tmem_cols);
}

// ------------------------------------------------------------------------------------------------ f32 GEMM
// 64 activation rows x 64 features per CTA, 16 k per step; every operation is an f32 FMA in ascending k.
constexpr int kDfTile = 64, kDfK = 16;

// Grouped (jobs given): blockIdx.y is the job, rpad a group's rows.
__global__ void __launch_bounds__(256) dgemm_f32_kernel(const float* w, int kpad, int rpad, const float* x, long long ldx, int m, int cols,
                                                        const __grid_constant__ DenseGroups grp, const __grid_constant__ DenseEpilogue epi) {
  __shared__ __align__(16) float xs[kDfK][kDfTile + 4], ws[kDfK][kDfTile + 4];
  __shared__ float ys[kDfTile][kDfTile + 1];
  pdl_wait();
  pdl_launch_dependents();
  const int n0 = blockIdx.x * kDfTile;
  int m0 = blockIdx.y * kDfTile, shift = 0;
  if (grp.jobs) {
    if ((int)blockIdx.y >= *grp.n_jobs) return;
    const int4 job = grp.jobs[blockIdx.y];
    w += (size_t)job.x * grp.group_rows * kpad;
    m0 = job.y;
    shift = job.w;
    m = min(m, m0 + min(job.z, kDfTile));
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;      // features 4 tx.., rows 4 ty..
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4; // this thread's share of the loads
  float acc[4][4] = {};
  const float* xrow = x + (size_t)(m0 + lr < m ? (grp.x_rows ? grp.x_rows[m0 + lr] : m0 + lr) : 0) * ldx;
  for (int k0 = 0; k0 < cols; k0 += kDfK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      xs[lk + i][lr] = m0 + lr < m && k < cols ? xrow[k] : 0.f;
      ws[lk + i][lr] = n0 + lr < rpad && k < cols ? w[(size_t)(n0 + lr) * kpad + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kDfK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][4 * ty]), b = *reinterpret_cast<const float4*>(&ws[k][4 * tx]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) ys[4 * ty + i][4 * tx + j] = acc[i][j];
  __syncthreads();
  const int n = threadIdx.x & 63;
  const DenseDst d = dense_dst(epi, n0 + n);
  if (d.kind == DENSE_GLU && (n & 8)) return;
  for (int r = threadIdx.x >> 6; r < kDfTile && m0 + r < m; r += 4) {
    const float scale = epi.row_scale ? epi.row_scale[m0 + shift + r] : 1.f;
    float v = ys[r][n] * scale;
    if (d.kind == DENSE_GLU) v = dense_glu(epi, v, ys[r][n + 8] * scale);
    dense_store(epi, d, m0 + shift + r, v);
  }
}

// ------------------------------------------------------------------------------------------------ launches
constexpr size_t kGvSmemMax = 100 * 1024;   // activations of the GEMV in shared memory (two CTAs per SM)
constexpr size_t kGvRows = 8;
constexpr size_t kGvNormRows = 2;           // up to here every CTA of the GEMV norms the rows itself; above, a kernel of its own does

template <typename K>
static int set_smem(tq_ctx* ctx, K kern, size_t bytes) {
  if (bytes > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
  return TQ_OK;
}

static int launch_gemv(tq_ctx* ctx, const tq_dweight* w, const DenseInput& in, size_t m, const DenseEpilogue& epi) {
  GemvParams p;
  p.w = static_cast<const __nv_bfloat16*>(w->data);
  p.kpad = (int)w->kpad;
  p.n_rb = (int)(w->rpad / 16);
  p.x = static_cast<const __nv_bfloat16*>(in.x);
  p.ldx = (long long)in.ldx;
  p.m = (int)m;
  p.cols = (int)w->cols;
  p.h = in.h;
  p.ldh = (long long)in.ldh;
  p.h_rows = in.h_rows;
  p.gain = static_cast<const __nv_bfloat16*>(in.gain);
  p.eps = in.eps;
  p.grp = DenseGroups();
  p.epi = epi;
  const size_t smem = m * (w->kpad * 2 + 16);
  int grid = ctx->sm_count * 2;
  if (grid > p.n_rb) grid = p.n_rb;
  if (int st = set_smem(ctx, dgemv_kernel<false>, smem)) return st;
  TQ_CUDA(ctx, launch_k(ctx, dgemv_kernel<false>, dim3((unsigned)grid), dim3(kGvThreads), smem, p));
  return TQ_OK;
}

static int launch_umma(tq_ctx* ctx, const tq_dweight* w, const void* x, size_t ldx, size_t m, const DenseEpilogue& epi, const DenseGroups* groups = nullptr) {
  if (!w->has_map) return fail(ctx, TQ_EUNSUPPORTED, "cuTensorMapEncodeTiled is not available from this driver");
  TQ_REQUIRE(ctx, ((uintptr_t)x & 15) == 0 && ldx % 8 == 0, "dense linear: activation rows must be 16-byte aligned");
  DUmmaParams p;
  p.m = (int)m;
  p.grouped = groups != nullptr;
  p.grp = groups ? *groups : DenseGroups();
  p.n_ft = (int)(((groups ? groups->group_rows : w->rpad) + kUmmaRows - 1) / kUmmaRows);
  p.kb_total = (int)((w->cols + kUmmaK - 1) / kUmmaK);
  int ntok = 16;
  if (groups) {
    ntok = groups->chunk;
    p.n_tt = groups->max_jobs;
    p.splits = 1;
    p.kb_per_split = p.kb_total;
    TQ_REQUIRE(ctx, (long long)p.n_ft * p.n_tt < (1ll << 31), "dense linear: too many jobs");
    p.n_tiles = p.n_ft * p.n_tt;
  } else {
    // Row tile: the width that makes (waves of CTAs) x (width) smallest; the wider one on a tie.
    long long best = 0;
    for (int cand = 256; cand >= 16; cand -= 16) {
      if (cand > 16 && (size_t)(cand - 15) > m && cand - 16 >= (int)m) continue;     // wider than the rows need
      const long long tiles = (long long)p.n_ft * (long long)((m + cand - 1) / cand);
      const long long waves = (tiles + ctx->sm_count - 1) / ctx->sm_count;
      const long long cost = waves * (cand < 96 ? 96 : cand);   // (below about 96 rows a step costs the same)
      if (best == 0 || cost < best) {
        best = cost;
        ntok = cand;
      }
    }
    p.n_tt = (int)((m + ntok - 1) / ntok);
    const int base = p.n_ft * p.n_tt;
    int splits = 1;
    if (base <= ctx->sm_count / 2 && base <= kTileCounters && !epi.row_scale) {
      splits = ctx->sm_count / base;
      if (splits > p.kb_total / 4) splits = p.kb_total / 4;    // at least four 64-k steps each
      if (splits > 16) splits = 16;
      if (splits < 1) splits = 1;
    }
    p.kb_per_split = (p.kb_total + splits - 1) / splits;
    p.splits = (p.kb_total + p.kb_per_split - 1) / p.kb_per_split;
    p.n_tiles = base * p.splits;
  }
  p.ntok = ntok;
  p.acc_stride = ntok <= 32 ? 32 : ntok <= 64 ? 64 : ntok <= 128 ? 128 : 256;
  p.n_acc = 2;
  p.tmem_cols = 2 * p.acc_stride;
  const size_t stage = (size_t)(kUmmaRows + ntok) * 128, budget = 227 * 1024 - kDuHeader - 1024;
  p.stages = (int)(budget / stage);
  if (p.stages > kDuMaxStages) p.stages = kDuMaxStages;
  p.epi = epi;
  p.err = ctx->dev_err;
  p.counters = ctx->dev_err + 1;
  p.partial = nullptr;
  if (p.splits > 1) {
    if (int st = ensure_splitk(ctx, (size_t)p.splits * m * p.n_ft * kUmmaRows * sizeof(float))) return st;
    p.partial = static_cast<float*>(ctx->splitk);
  }
  CUtensorMap xmap;
  if (!encode_bf16_k64(&xmap, x, m, w->cols, ldx, (unsigned)ntok)) return fail(ctx, TQ_ECUDA, "cuTensorMapEncodeTiled failed");
  const size_t smem = kDuHeader + 1024 + (size_t)p.stages * stage;
  if (int st = set_smem(ctx, dgemm_umma_kernel, smem)) return st;
  const int grid = p.n_tiles < ctx->sm_count ? p.n_tiles : ctx->sm_count;
  TQ_CUDA(ctx, launch_k(ctx, dgemm_umma_kernel, dim3((unsigned)grid), dim3(kDuThreads), smem, w->map, xmap, p));
  return TQ_OK;
}

int dense_group_chunk(int dtype, size_t kpad, size_t rows, size_t n_groups) {
  if (dtype == TQ_F32) return kDfTile;
  const size_t mean = (rows + n_groups - 1) / n_groups;
  size_t gv = kGvSmemMax / (kpad * 2 + 16);
  if (gv > kGvRows) gv = kGvRows;
  if (mean <= 4 && gv > 0) return (int)gv;
  // a group of two standard deviations above the mean (rows spread at random) still fills its jobs: ntok is paid in full
  const size_t need = mean + 2 * (size_t)std::ceil(std::sqrt((double)mean)), jobs = (need + 255) / 256;
  return (int)(((need + jobs - 1) / jobs + 15) / 16 * 16);
}

int dense_even_chunk(int dtype, size_t kpad, size_t rows) {
  if (dtype == TQ_F32) return kDfTile;
  if (rows <= kGvRows && kGvRows * (kpad * 2 + 16) <= kGvSmemMax) return (int)kGvRows;
  const size_t jobs = (rows + 255) / 256;
  return (int)(((rows + jobs - 1) / jobs + 15) / 16 * 16);
}

int launch_dense_grouped(tq_ctx* ctx, const tq_dweight* w, const void* x, size_t ldx, size_t rows, const DenseGroups& g, const DenseEpilogue& epi) {
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, g.jobs && g.n_jobs && g.max_jobs > 0 && g.chunk > 0 && g.group_rows > 0 && g.group_rows % 16 == 0, "grouped dense linear: bad groups");
  TQ_REQUIRE(ctx, epi.n >= 1 && epi.n <= kDenseMaxSections && epi.s[epi.n - 1].row_end <= (int)g.group_rows, "grouped dense linear: bad output sections");
  if (w->dtype == TQ_F32) {
    TQ_REQUIRE(ctx, g.chunk == kDfTile && g.max_jobs <= 65535, "grouped dense linear: f32 jobs have up to %d rows", kDfTile);
    TQ_CUDA(ctx, launch_k(ctx, dgemm_f32_kernel, dim3((unsigned)((g.group_rows + kDfTile - 1) / kDfTile), (unsigned)g.max_jobs), dim3(256), 0,
                          static_cast<const float*>(w->data), (int)w->kpad, (int)g.group_rows, static_cast<const float*>(x), (long long)ldx, (int)rows,
                          (int)w->cols, g, epi));
    return TQ_OK;
  }
  TQ_REQUIRE(ctx, ((uintptr_t)x & 15) == 0 && ldx % 8 == 0, "dense linear: activation rows must be 16-byte aligned");
  if (g.chunk > (int)kGvRows) {
    TQ_REQUIRE(ctx, g.chunk % 16 == 0 && g.chunk <= 256 && !g.x_rows, "grouped dense linear: bad job size");
    return launch_umma(ctx, w, x, ldx, rows, epi, &g);
  }
  GemvParams p = {};
  p.w = static_cast<const __nv_bfloat16*>(w->data);
  p.kpad = (int)w->kpad;
  p.n_rb = (int)(g.group_rows / 16);
  p.x = static_cast<const __nv_bfloat16*>(x);
  p.ldx = (long long)ldx;
  p.m = g.chunk;
  p.cols = (int)w->cols;
  p.grp = g;
  p.epi = epi;
  const size_t smem = g.chunk * (w->kpad * 2 + 16);
  TQ_REQUIRE(ctx, smem <= kGvSmemMax, "grouped dense linear: rows too long for the job size");
  const long long tiles = (long long)p.n_rb * g.max_jobs;
  TQ_REQUIRE(ctx, tiles < (1ll << 31), "dense linear: too many jobs");
  const int grid = (int)(tiles < ctx->sm_count * 2 ? tiles : ctx->sm_count * 2);
  if (int st = set_smem(ctx, dgemv_kernel<true>, smem)) return st;
  TQ_CUDA(ctx, launch_k(ctx, dgemv_kernel<true>, dim3((unsigned)grid), dim3(kGvThreads), smem, p));
  return TQ_OK;
}

int launch_dense(tq_ctx* ctx, const tq_dweight* w, const DenseInput& in, size_t m, const DenseEpilogue& epi) {
  if (m == 0) return TQ_OK;
  TQ_REQUIRE(ctx, epi.n >= 1 && epi.n <= kDenseMaxSections && epi.s[epi.n - 1].row_end <= (int)w->rpad, "dense linear: bad output sections");
  const bool bf = w->dtype == TQ_BF16;
  const bool fits = m <= kGvRows && m * (w->kpad * 2 + 16) <= kGvSmemMax;
  DenseInput x = in;
  if (in.h && !(bf && fits && m <= kGvNormRows && in.gain_dtype == TQ_BF16)) {
    TQ_REQUIRE(ctx, in.xn_tmp != nullptr, "dense linear: no buffer for the normalised rows");
    if (int st = launch_rms_norm_rows(ctx, in.h, in.ldh, in.h_rows, in.gain, in.gain_dtype, m, w->cols, in.eps, in.xn_tmp,
                                      bf ? TQ_BF16 : TQ_F32, w->kpad)) return st;
    x = DenseInput();
    x.x = in.xn_tmp;
    x.ldx = w->kpad;
  }
  if (!bf) {
    TQ_CUDA(ctx, launch_k(ctx, dgemm_f32_kernel, dim3((unsigned)((w->rpad + kDfTile - 1) / kDfTile), (unsigned)((m + kDfTile - 1) / kDfTile)),
                          dim3(256), 0, static_cast<const float*>(w->data), (int)w->kpad, (int)w->rpad, static_cast<const float*>(x.x),
                          (long long)x.ldx, (int)m, (int)w->cols, DenseGroups(), epi));
    return TQ_OK;
  }
  if (!x.h) TQ_REQUIRE(ctx, ((uintptr_t)x.x & 15) == 0 && x.ldx % 8 == 0, "dense linear: activation rows must be 16-byte aligned");
  if (fits) return launch_gemv(ctx, w, x, m, epi);
  return launch_umma(ctx, w, x.x, x.ldx, m, epi);
}

__global__ void dweight_put_kernel(const void* src, int s_dt, void* dst, int d_dt, size_t rows, size_t cols, size_t kpad, size_t row0,
                                   size_t col0, int interleave) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows * cols) return;
  const size_t r = i / cols, c = i % cols;
  const float v = s_dt == TQ_F32 ? reinterpret_cast<const float*>(src)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(src)[i]);
  const size_t dr = row0 + (interleave ? (r / 8) * 16 + (interleave == 2 ? 8 : 0) + r % 8 : r);
  const size_t o = dr * kpad + col0 + c;
  if (d_dt == TQ_F32) reinterpret_cast<float*>(dst)[o] = v;
  else reinterpret_cast<__nv_bfloat16*>(dst)[o] = __float2bfloat16_rn(v);
}

// dst = src + add, to f32 or bf16.
__global__ void put_vector_kernel(const void* src, int s_dt, void* dst, int d_dt, size_t n, float add) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = (s_dt == TQ_F32 ? static_cast<const float*>(src)[i] : __bfloat162float(static_cast<const __nv_bfloat16*>(src)[i])) + add;
  if (d_dt == TQ_F32) static_cast<float*>(dst)[i] = v;
  else static_cast<__nv_bfloat16*>(dst)[i] = __float2bfloat16_rn(v);
}

int put_vector(tq_ctx* ctx, const void* src, int src_dtype, void* dst, int dst_dtype, size_t n, float add) {
  void* tmp = nullptr;
  TQ_CUDA(ctx, cudaMalloc(&tmp, n * dtype_size(src_dtype)));
  cudaError_t e = cudaMemcpyAsync(tmp, src, n * dtype_size(src_dtype), cudaMemcpyDefault, ctx->stream);
  if (e == cudaSuccess) {
    put_vector_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(tmp, src_dtype, dst, dst_dtype, n, add);
    ctx->launches++;
    e = cudaGetLastError();
  }
  if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
  cudaFree(tmp);
  TQ_CUDA(ctx, e);
  return TQ_OK;
}

__global__ void dweight_put_head_t_kernel(const void* src, int s_dt, void* dst, int d_dt, size_t heads, size_t dim, size_t rank, size_t group_rows, size_t kpad) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= heads * dim * rank) return;
  const size_t r = i / rank, c = i % rank, o = (r / dim * group_rows + c) * kpad + r % dim;
  const float v = s_dt == TQ_F32 ? reinterpret_cast<const float*>(src)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(src)[i]);
  if (d_dt == TQ_F32) reinterpret_cast<float*>(dst)[o] = v;
  else reinterpret_cast<__nv_bfloat16*>(dst)[o] = __float2bfloat16_rn(v);
}

int dweight_put_head_transposed(tq_ctx* ctx, tq_dweight* w, const void* src, int src_dtype, size_t heads, size_t dim, size_t rank, size_t group_rows) {
  TQ_REQUIRE(ctx, rank <= group_rows && heads * group_rows <= w->rpad && dim <= w->kpad, "dense weight: transposed heads outside the weight");
  const size_t n = heads * dim * rank, bytes = n * dtype_size(src_dtype);
  void* tmp = nullptr;
  TQ_CUDA(ctx, cudaMalloc(&tmp, bytes));
  cudaError_t e = cudaMemcpyAsync(tmp, src, bytes, cudaMemcpyDefault, ctx->stream);
  if (e == cudaSuccess) {
    dweight_put_head_t_kernel<<<(unsigned)((n + 255) / 256), 256, 0, ctx->stream>>>(tmp, src_dtype, w->data, w->dtype, heads, dim, rank, group_rows, w->kpad);
    ctx->launches++;
    e = cudaGetLastError();
  }
  if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
  cudaFree(tmp);
  TQ_CUDA(ctx, e);
  return TQ_OK;
}

__global__ void clamped_glu_kernel(const void* gate, const void* up, int dt, size_t n, float limit, float alpha, void* out, int out_dt) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float g = dt == TQ_F32 ? reinterpret_cast<const float*>(gate)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(gate)[i]);
  const float u = dt == TQ_F32 ? reinterpret_cast<const float*>(up)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(up)[i]);
  const float v = clamped_glu(g, u, limit, alpha);
  if (out_dt == TQ_F32) reinterpret_cast<float*>(out)[i] = v;
  else reinterpret_cast<__nv_bfloat16*>(out)[i] = __float2bfloat16_rn(v);
}

}  // namespace tq

using namespace tq;

extern "C" {

int tq_dweight_create(tq_ctx* ctx, size_t rows, size_t cols, int dtype, tq_dweight** out) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, out && rows > 0 && cols > 0, "tq_dweight_create: empty weight");
  *out = nullptr;
  TQ_REQUIRE(ctx, dtype == TQ_BF16 || dtype == TQ_F32, "tq_dweight_create: dtype must be bf16 or f32");
  TQ_REQUIRE(ctx, rows < (1ull << 30) && cols < (1ull << 30), "tq_dweight_create: weight too large");
  tq_dweight* w = new (std::nothrow) tq_dweight();
  if (!w) return fail(ctx, TQ_ENOMEM, "out of host memory");
  w->dtype = dtype;
  w->rows = rows;
  w->cols = cols;
  w->rpad = (rows + 15) / 16 * 16;
  w->kpad = (cols + kGvPad - 1) / kGvPad * kGvPad;
  const size_t bytes = w->rpad * w->kpad * dtype_size(dtype);
  cudaError_t e = cudaMalloc(&w->data, bytes);
  if (e == cudaSuccess) e = cudaMemsetAsync(w->data, 0, bytes, ctx->stream);
  if (e != cudaSuccess) {
    if (w->data) cudaFree(w->data);
    delete w;
    cudaGetLastError();
    return fail(ctx, e == cudaErrorMemoryAllocation ? TQ_ENOMEM : TQ_ECUDA, "tq_dweight_create: %s", cudaGetErrorString(e));
  }
  if (dtype == TQ_BF16) w->has_map = encode_bf16_k64(&w->map, w->data, w->rpad, w->kpad, w->kpad, kUmmaRows);
  *out = w;
  return TQ_OK;
}

int tq_dweight_put(tq_ctx* ctx, tq_dweight* w, const void* src, int src_dtype, size_t rows, size_t cols, size_t row0, size_t col0,
                   int interleave) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, w && src && rows > 0 && cols > 0, "tq_dweight_put: null argument");
  TQ_REQUIRE(ctx, src_dtype == TQ_BF16 || src_dtype == TQ_F32, "tq_dweight_put: the source must be bf16 or f32");
  TQ_REQUIRE(ctx, interleave >= 0 && interleave <= 2 && (!interleave || row0 % 16 == 0), "tq_dweight_put: bad row order");
  const size_t last = interleave ? ((rows - 1) / 8) * 16 + 8 * (interleave - 1) + (rows - 1) % 8 : rows - 1;
  TQ_REQUIRE(ctx, row0 + last < w->rpad && col0 + cols <= w->kpad, "tq_dweight_put: block outside the weight");
  const size_t bytes = rows * cols * dtype_size(src_dtype);
  void* tmp = nullptr;
  TQ_CUDA(ctx, cudaMalloc(&tmp, bytes));
  cudaError_t e = cudaMemcpyAsync(tmp, src, bytes, cudaMemcpyDefault, ctx->stream);
  if (e == cudaSuccess) {
    dweight_put_kernel<<<(unsigned)((rows * cols + 255) / 256), 256, 0, ctx->stream>>>(tmp, src_dtype, w->data, w->dtype, rows, cols, w->kpad,
                                                                                      row0, col0, interleave);
    ctx->launches++;
    e = cudaGetLastError();
  }
  if (e == cudaSuccess) e = cudaStreamSynchronize(ctx->stream);
  cudaFree(tmp);
  TQ_CUDA(ctx, e);
  return TQ_OK;
}

int tq_dweight_free(tq_ctx* ctx, tq_dweight* w) {
  if (!w) return TQ_OK;
  if (int st = bind(ctx)) return st;
  cudaStreamSynchronize(ctx->stream);
  cudaFree(w->data);
  delete w;
  return TQ_OK;
}

int tq_dweight_data(const tq_dweight* w, void** dev, size_t* rows_padded, size_t* cols_padded) {
  if (!w) return TQ_EINVAL;
  if (dev) *dev = w->data;
  if (rows_padded) *rows_padded = w->rpad;
  if (cols_padded) *cols_padded = w->kpad;
  return TQ_OK;
}

int tq_dlinear(tq_ctx* ctx, const tq_dweight* w, const void* x_dev, size_t ldx, size_t m, void* y_dev, int y_dtype, size_t ldy) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, w && x_dev && y_dev, "tq_dlinear: null pointer");
  TQ_REQUIRE(ctx, y_dtype == TQ_F32 || y_dtype == TQ_BF16, "tq_dlinear: y must be f32 or bf16");
  DenseInput in;
  in.x = x_dev;
  in.ldx = ldx ? ldx : w->cols;
  DenseEpilogue e;
  e.n = 1;
  e.s[0].row_end = (int)w->rpad;
  e.s[0].rows = (int)w->rows;
  e.s[0].f32 = y_dtype == TQ_F32;
  e.s[0].ld = (long long)(ldy ? ldy : w->rows);
  e.s[0].out = y_dev;
  return launch_dense(ctx, w, in, m, e);
}

size_t tq_dense_group_chunk(int dtype, size_t cols, size_t rows, size_t n_groups) {
  if (cols == 0 || n_groups == 0) return 0;
  return (size_t)dense_group_chunk(dtype, (cols + kGvPad - 1) / kGvPad * kGvPad, rows, n_groups);
}

int tq_dlinear_grouped(tq_ctx* ctx, const tq_dweight* w, const void* x_dev, size_t ldx, size_t rows, const int* jobs_dev, const int* n_jobs_dev,
                       size_t max_jobs, size_t chunk, size_t group_rows, const int* x_rows_dev, const float* row_scale_dev, float glu_limit,
                       float glu_alpha, void* y_dev, int y_dtype, size_t ldy) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, w && x_dev && y_dev && jobs_dev && n_jobs_dev, "tq_dlinear_grouped: null pointer");
  TQ_REQUIRE(ctx, y_dtype == TQ_F32 || y_dtype == TQ_BF16, "tq_dlinear_grouped: y must be f32 or bf16");
  DenseGroups g;
  g.jobs = reinterpret_cast<const int4*>(jobs_dev);
  g.n_jobs = n_jobs_dev;
  g.max_jobs = (int)max_jobs;
  g.chunk = (int)chunk;
  g.group_rows = group_rows;
  g.x_rows = x_rows_dev;
  DenseEpilogue e;
  e.n = 1;
  e.s[0].row_end = (int)group_rows;
  e.s[0].rows = (int)(glu_alpha != 0.f ? group_rows / 2 : group_rows);
  e.s[0].kind = glu_alpha != 0.f ? DENSE_GLU : DENSE_ROW;
  e.s[0].f32 = y_dtype == TQ_F32;
  e.s[0].ld = (long long)(ldy ? ldy : (size_t)e.s[0].rows);
  e.s[0].out = y_dev;
  e.glu_limit = glu_limit;
  e.glu_alpha = glu_alpha;
  e.row_scale = row_scale_dev;
  return launch_dense_grouped(ctx, w, x_dev, ldx ? ldx : w->cols, rows, g, e);
}

int tq_clamped_glu(tq_ctx* ctx, const void* gate_dev, const void* up_dev, int in_dtype, size_t n, float limit, float alpha, void* out_dev,
                   int out_dtype) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, (in_dtype == TQ_F32 || in_dtype == TQ_BF16) && (out_dtype == TQ_F32 || out_dtype == TQ_BF16),
             "tq_clamped_glu: dtypes must be f32 or bf16");
  if (n == 0) return TQ_OK;
  TQ_REQUIRE(ctx, gate_dev && up_dev && out_dev, "tq_clamped_glu: null pointer");
  TQ_CUDA(ctx, launch_k(ctx, clamped_glu_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, gate_dev, up_dev, in_dtype, n, limit, alpha,
                        out_dev, out_dtype));
  return TQ_OK;
}

}  // extern "C"
