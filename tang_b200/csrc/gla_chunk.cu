// Gated linear attention over prompts in bf16, in chunks of 64 tokens on the tensor cores (see gla.cuh for the recurrence).
// With L_t the running sum of a chunk's log decays (per key channel) and S the state before the chunk,
//     o_t = (q_t e^{L_t})^T S + sum_{s <= t} (sum_d q_td k_sd e^{L_td - L_sd}) v_s
//     S'  = diag(e^{L_end}) S + sum_s (k_s e^{L_end - L_s}) v_s^T.
//   1. gla_chunk_state_kernel  (chunk, head): L, the chunk's own contribution to the state and its total decay;
//   2. gla_chunk_carry_kernel: walks the chunks of a sequence, leaves every chunk the state before it, updates the slot;
//   3. gla_chunk_out_kernel    (chunk, head): the outputs, head norm and gate.
// Every exponent is at most zero: token pairs in different 16-token blocks meet through the running sum at the later block's
// start, pairs of one block are formed directly.  Operands that are not bf16 already (everything with a decay in it, states,
// token-pair weights) enter the products as two bf16 terms each, with f32 accumulation.
#include "attn_mma.cuh"
#include "gla_device.cuh"

namespace tq {

constexpr int kGcTokens = 64, kGcBlock = 16;
constexpr int kGcThreads = 256, kGcWarps = kGcThreads / 32;
constexpr int kGcPad = 8;            // bf16 elements of padding per shared-memory row (one bank group)

// First chunk of a sequence in the workspaces (at most rows / 64 + sequences chunks in all).
__device__ __forceinline__ size_t gc_first_chunk(const GlaSeq& s, int seq) { return (size_t)(s.row0 / kGcTokens) + seq; }

// cp.async of n_rows rows of `cols` bf16 (a multiple of 8) into rows of `ld` elements; rows up to 64 become zeros.
__device__ __forceinline__ void gc_copy(__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, size_t ld_src, int n_rows, int cols) {
  const int per = cols / 8;
  for (int i = threadIdx.x; i < kGcTokens * per; i += kGcThreads) {
    const int t = i / per, c = i - t * per;
    const bool ok = t < n_rows;
    cp_async16(smem_u32(dst + t * ld + 8 * c), ok ? src + (size_t)t * ld_src + 8 * c : src, ok);
  }
}

// log2 of a channel's decay from its logit
__device__ __forceinline__ float gc_log2_decay(float z, float inv_tau) {
  const float y = z * kLog2e;
  return (fminf(y, 0.f) - __log2f(1.0f + ex2_ftz(-fabsf(y)))) * inv_tau;
}

__device__ __forceinline__ void ldmatrix2_t(uint32_t (&r)[2], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(smem_u32(p)));
}

// ------------------------------------------------------------------------------------------------ 1. contributions
__global__ void __launch_bounds__(kGcThreads) gla_chunk_state_kernel(Gla g, GlaRows r, RaggedBatch b, float* logs, float* upd, float* total) {
  extern __shared__ __align__(16) uint8_t gc_smem[];
  const int kld = g.dim + kGcPad, vld = g.vdim + kGcPad;
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(gc_smem);     // [64][kld] raw keys, then their leading terms
  __nv_bfloat16* kl = kh + kGcTokens * kld;
  __nv_bfloat16* vs = kl + kGcTokens * kld;                          // [64][vld]
  float* L = reinterpret_cast<float*>(vs + kGcTokens * vld);         // [64][dim]
  float* a1s = L + kGcTokens * g.dim;                                // [64][rank]
  float* a2s = a1s + kGcTokens * g.rank;                             // [rank][dim]
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ch0 = head * g.dim;
  for (int i = threadIdx.x; i < g.dim * g.rank; i += kGcThreads) {   // (weights: before the wait)
    const int d = i / g.rank, k = i - d * g.rank;
    a2s[k * g.dim + d] = g.a2[(size_t)ch0 * g.rank + i];
  }
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.z, s)) return;
  const int t0 = blockIdx.x * kGcTokens, n = min(kGcTokens, s.n - t0);
  if (n <= 0) return;
  const size_t row = s.row0 + t0, chunk = gc_first_chunk(s, blockIdx.z) + blockIdx.x;
  gc_copy(kh, kld, static_cast<const __nv_bfloat16*>(r.k) + row * r.ld + ch0, r.ld, n, g.dim);
  gc_copy(vs, vld, static_cast<const __nv_bfloat16*>(r.v) + row * r.ld + (size_t)head * g.vdim, r.ld, n, g.vdim);
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = threadIdx.x; i < n * g.rank; i += kGcThreads) a1s[i] = r.a1[(row + i / g.rank) * r.ld_a1 + i % g.rank];
  __syncthreads();
  const float inv_tau = 1.0f / g.tau;
  // a thread forms four tokens of a channel at a time: the channel's weights are read once for them
  for (int i = threadIdx.x; i < (kGcTokens / 4) * g.dim; i += kGcThreads) {
    const int tq = i / g.dim, d = i - tq * g.dim, t = 4 * tq;
    float z[4];
    z[0] = z[1] = z[2] = z[3] = g.a2_bias[ch0 + d];
    for (int k = 0; k < g.rank; ++k) {
      const float w = a2s[k * g.dim + d];
#pragma unroll
      for (int j = 0; j < 4; ++j) z[j] = fmaf(w, a1s[min(t + j, n - 1) * g.rank + k], z[j]);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) L[(t + j) * g.dim + d] = t + j < n ? gc_log2_decay(z[j], inv_tau) : 0.f;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < g.dim; d += kGcThreads) {
    float run = 0.f;
#pragma unroll 16
    for (int t = 0; t < kGcTokens; ++t) {
      run += L[t * g.dim + d];
      L[t * g.dim + d] = run;
    }
    total[(chunk * g.heads + head) * g.dim + d] = ex2_ftz(run);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  float* lg = logs + row * g.heads * g.dim + ch0;
  for (int i = threadIdx.x; i < kGcTokens * g.dim / 2; i += kGcThreads) {
    const int t = 2 * i / g.dim, d = 2 * i - t * g.dim;
    const float2 l = *reinterpret_cast<const float2*>(L + t * g.dim + d), e = *reinterpret_cast<const float2*>(L + (kGcTokens - 1) * g.dim + d);
    if (t < n) *reinterpret_cast<float2*>(lg + (size_t)t * g.heads * g.dim + d) = l;
    const uint32_t kw = *reinterpret_cast<const uint32_t*>(kh + t * kld + d);
    uint32_t hi, lo;
    split_bf16(bf16_bits_to_float(kw & 0xFFFFu) * ex2_ftz(e.x - l.x), bf16_bits_to_float(kw >> 16) * ex2_ftz(e.y - l.y), hi, lo);
    *reinterpret_cast<uint32_t*>(kh + t * kld + d) = hi;
    *reinterpret_cast<uint32_t*>(kl + t * kld + d) = lo;
  }
  __syncthreads();
  // [dim x 64] x [64 x vdim]: a warp takes units of 16 channels x 64 columns
  const int n_mt = g.dim / 16, n_cb = (g.vdim + 63) / 64;
  float* out = upd + ((chunk * g.heads + head) * g.dim) * g.vdim;
  for (int u = warp; u < n_mt * n_cb; u += kGcWarps) {
    const int mt = u % n_mt, c0 = (u / n_mt) * 64, nt = min(8, (g.vdim - c0) / 8);
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int k = 0; k < kGcTokens / 16; ++k) {
      uint32_t ah[4], al[4];
      const int off = (16 * k + (lane & 7) + 8 * (lane >> 4)) * kld + 16 * mt + 8 * ((lane >> 3) & 1);
      ldmatrix4_t(ah, kh + off);
      ldmatrix4_t(al, kl + off);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (j < nt) {                                    // (vdim is a multiple of 16)
          uint32_t vf[4];
          ldmatrix4_t(vf, vs + (16 * k + (lane & 15)) * vld + c0 + 8 * j + 8 * (lane >> 4));
          mma_bf16_16816(acc[j], ah[0], ah[1], ah[2], ah[3], vf[0], vf[1]);
          mma_bf16_16816(acc[j + 1], ah[0], ah[1], ah[2], ah[3], vf[2], vf[3]);
          mma_bf16_16816(acc[j], al[0], al[1], al[2], al[3], vf[0], vf[1]);
          mma_bf16_16816(acc[j + 1], al[0], al[1], al[2], al[3], vf[2], vf[3]);
        }
      }
    }
    float* dst = out + (size_t)(16 * mt + (lane >> 2)) * g.vdim + c0 + 2 * (lane & 3);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (j < nt) {
        *reinterpret_cast<float2*>(dst + 8 * j) = make_float2(acc[j][0], acc[j][1]);
        *reinterpret_cast<float2*>(dst + (size_t)8 * g.vdim + 8 * j) = make_float2(acc[j][2], acc[j][3]);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ 2. states
__global__ void __launch_bounds__(256) gla_chunk_carry_kernel(Gla g, RaggedBatch b, float* upd, const float* total) {
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.y, s)) return;
  const size_t per = (size_t)g.heads * g.dim * g.vdim, i = 4 * ((size_t)blockIdx.x * 256 + threadIdx.x);
  if (i >= per) return;
  const int chunks = (s.n + kGcTokens - 1) / kGcTokens;
  const size_t c0 = gc_first_chunk(s, blockIdx.y), ch = i / g.vdim, chs = (size_t)g.heads * g.dim;
  float* st = g.state + s.slot * per + i;
  float4 S = s.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  float* u = upd + c0 * per + i;
  const float* d = total + c0 * chs + ch;
  constexpr int U = 8;
  for (int c = 0; c < chunks; c += U) {
    float4 x[U];
    float f[U];
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c + j < chunks) {
        x[j] = *reinterpret_cast<const float4*>(u + (size_t)(c + j) * per);
        f[j] = d[(size_t)(c + j) * chs];
      }
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c + j < chunks) {
        *reinterpret_cast<float4*>(u + (size_t)(c + j) * per) = S;
        S.x = fmaf(f[j], S.x, x[j].x);
        S.y = fmaf(f[j], S.y, x[j].y);
        S.z = fmaf(f[j], S.z, x[j].z);
        S.w = fmaf(f[j], S.w, x[j].w);
      }
  }
  *reinterpret_cast<float4*>(st) = S;
}

// ------------------------------------------------------------------------------------------------ 3. outputs
// NTW: 8-column tiles per warp (vdim <= 64 NTW).
template <int NTW>
__global__ void __launch_bounds__(kGcThreads, 2) gla_chunk_out_kernel(Gla g, GlaRows r, RaggedBatch b, const float* logs, const float* states) {
  extern __shared__ __align__(16) uint8_t gc_smem[];
  constexpr int kPld = kGcTokens + kGcPad;
  const int kld = g.dim + kGcPad, vld = g.vdim + kGcPad;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(gc_smem);      // [64][kld] queries, then the leading terms of q e^L
  __nv_bfloat16* ks = qs + kGcTokens * kld;                           // keys, then the second terms of q e^L
  __nv_bfloat16* ph = ks + kGcTokens * kld;                           // [64][kPld] token-pair weights, two terms
  __nv_bfloat16* pl = ph + kGcTokens * kPld;
  float* L = reinterpret_cast<float*>(pl + kGcTokens * kPld);         // [64][dim]; later the values [64][vld]
  __nv_bfloat16* vs = reinterpret_cast<__nv_bfloat16*>(L);
  __shared__ float sq_s[kGcWarps][kGcTokens];
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tl = lane & 3;
  const int ch0 = head * g.dim;
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.z, s)) return;
  const int t0 = blockIdx.x * kGcTokens, n = min(kGcTokens, s.n - t0);
  if (n <= 0) return;
  const size_t row = s.row0 + t0, chunk = gc_first_chunk(s, blockIdx.z) + blockIdx.x;
  gc_copy(qs, kld, static_cast<const __nv_bfloat16*>(r.q) + row * r.ld + ch0, r.ld, n, g.dim);
  gc_copy(ks, kld, static_cast<const __nv_bfloat16*>(r.k) + row * r.ld + ch0, r.ld, n, g.dim);
  {
    // rows without a token repeat the last one's sums: their keys are zero
    const int per = g.dim / 4;
    for (int i = threadIdx.x; i < kGcTokens * per; i += kGcThreads) {
      const int t = i / per, c = i - t * per;
      cp_async16(smem_u32(L + t * g.dim + 4 * c), logs + (row + min(t, n - 1)) * g.heads * g.dim + ch0 + 4 * c, true);
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int i = threadIdx.x; i < 2 * kGcTokens * kPld / 8; i += kGcThreads) reinterpret_cast<uint4*>(ph)[i] = make_uint4(0u, 0u, 0u, 0u);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();

  // ---- token pairs of different blocks: (I, J) with J < I through the sums at the start of block I
  if (warp < 6) {
    const int I = warp < 1 ? 1 : warp < 3 ? 2 : 3, J = warp - (I == 1 ? 0 : I == 2 ? 1 : 3);
    const float* ref = L + (kGcBlock * I - 1) * g.dim;
    float acc[2][4] = {};
    for (int k0 = 0; k0 < g.dim; k0 += 16) {
      uint32_t ah[4], al[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {                      // rows g, g + 8; channels 2t, 2t + 8
        const int t = kGcBlock * I + gq + 8 * (i & 1), d = k0 + 2 * tl + 8 * (i >> 1);
        const float2 l = *reinterpret_cast<const float2*>(L + t * g.dim + d), rf = *reinterpret_cast<const float2*>(ref + d);
        const uint32_t w = *reinterpret_cast<const uint32_t*>(qs + t * kld + d);
        split_bf16(bf16_bits_to_float(w & 0xFFFFu) * ex2_ftz(l.x - rf.x), bf16_bits_to_float(w >> 16) * ex2_ftz(l.y - rf.y), ah[i], al[i]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = kGcBlock * J + 8 * j + gq, d = k0 + 2 * tl + 8 * i;
          const float2 l = *reinterpret_cast<const float2*>(L + t * g.dim + d), rf = *reinterpret_cast<const float2*>(ref + d);
          const uint32_t w = *reinterpret_cast<const uint32_t*>(ks + t * kld + d);
          split_bf16(bf16_bits_to_float(w & 0xFFFFu) * ex2_ftz(rf.x - l.x), bf16_bits_to_float(w >> 16) * ex2_ftz(rf.y - l.y), bh[i], bl[i]);
        }
        mma_bf16_16816(acc[j], ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
        mma_bf16_16816(acc[j], ah[0], ah[1], ah[2], ah[3], bl[0], bl[1]);
        mma_bf16_16816(acc[j], al[0], al[1], al[2], al[3], bh[0], bh[1]);
      }
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        uint32_t hi, lo;
        split_bf16(acc[j][2 * h] * g.q_scale, acc[j][2 * h + 1] * g.q_scale, hi, lo);
        const int off = (kGcBlock * I + gq + 8 * h) * kPld + kGcBlock * J + 8 * j + 2 * tl;
        *reinterpret_cast<uint32_t*>(ph + off) = hi;
        *reinterpret_cast<uint32_t*>(pl + off) = lo;
      }
  }
  // ---- pairs of one block, term by term: a warp takes a query, its lanes the channels
  for (int t = warp; t < n; t += kGcWarps) {
    const int s0 = t & ~(kGcBlock - 1);
    float sum[kGcBlock];
#pragma unroll
    for (int j = 0; j < kGcBlock; ++j) sum[j] = 0.f;
    for (int d = 2 * lane; d < g.dim; d += 64) {
      const float2 lt = *reinterpret_cast<const float2*>(L + t * g.dim + d);
      const uint32_t qw = *reinterpret_cast<const uint32_t*>(qs + t * kld + d);
      const float q0 = bf16_bits_to_float(qw & 0xFFFFu), q1 = bf16_bits_to_float(qw >> 16);
#pragma unroll
      for (int j = 0; j < kGcBlock; ++j) {
        if (s0 + j <= t) {
          const float2 ls = *reinterpret_cast<const float2*>(L + (s0 + j) * g.dim + d);
          const uint32_t kw = *reinterpret_cast<const uint32_t*>(ks + (s0 + j) * kld + d);
          sum[j] = fmaf(q0 * bf16_bits_to_float(kw & 0xFFFFu), ex2_ftz(lt.x - ls.x), sum[j]);
          sum[j] = fmaf(q1 * bf16_bits_to_float(kw >> 16), ex2_ftz(lt.y - ls.y), sum[j]);
        }
      }
    }
    // sixteen sums over 32 lanes: halve the sums while exchanging lanes; lane l ends up with sum (l >> 1)
#pragma unroll
    for (int w = kGcBlock / 2, o = 16; w >= 1; w >>= 1, o >>= 1) {
      const bool upper = lane & o;
#pragma unroll
      for (int j = 0; j < w; ++j) {
        const float give = upper ? sum[j] : sum[j + w], keep = upper ? sum[j + w] : sum[j];
        sum[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
      }
    }
    sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 1);
    const int sj = s0 + (lane >> 1);
    if (!(lane & 1) && sj <= t) {
      const float v = sum[0] * g.q_scale;
      const __nv_bfloat16 hi = __float2bfloat16_rn(v);
      ph[t * kPld + sj] = hi;
      pl[t * kPld + sj] = __float2bfloat16_rn(v - __bfloat162float(hi));
    }
  }
  __syncthreads();
  // ---- q e^L in place
  for (int i = threadIdx.x; i < kGcTokens * g.dim / 2; i += kGcThreads) {
    const int t = 2 * i / g.dim, d = 2 * i - t * g.dim;
    const float2 l = *reinterpret_cast<const float2*>(L + t * g.dim + d);
    const uint32_t w = *reinterpret_cast<const uint32_t*>(qs + t * kld + d);
    uint32_t hi, lo;
    split_bf16(bf16_bits_to_float(w & 0xFFFFu) * g.q_scale * ex2_ftz(l.x), bf16_bits_to_float(w >> 16) * g.q_scale * ex2_ftz(l.y), hi, lo);
    *reinterpret_cast<uint32_t*>(qs + t * kld + d) = hi;
    *reinterpret_cast<uint32_t*>(ks + t * kld + d) = lo;
  }
  __syncthreads();
  gc_copy(vs, vld, static_cast<const __nv_bfloat16*>(r.v) + row * r.ld + (size_t)head * g.vdim, r.ld, n, g.vdim);
  asm volatile("cp.async.commit_group;" ::: "memory");

  // ---- [64 x dim] x state: a warp owns NTW column tiles for all 64 tokens
  float o[4][NTW][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int j = 0; j < NTW; ++j) o[m][j][0] = o[m][j][1] = o[m][j][2] = o[m][j][3] = 0.f;
  const int c0 = 8 * NTW * warp;
  const float* S = states + ((chunk * g.heads + head) * g.dim) * g.vdim;
  const bool carried = !(s.fresh && blockIdx.x == 0);                 // else the state is zero
  if (carried && c0 < g.vdim) {
    for (int k0 = 0; k0 < g.dim; k0 += 16) {
      uint32_t bh[NTW][2], bl[NTW][2];
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        const int c = c0 + 8 * j;
        const float* src = S + (size_t)(k0 + 2 * tl) * g.vdim + (c < g.vdim ? c : 0) + gq;
        split_bf16(src[0], src[g.vdim], bh[j][0], bl[j][0]);
        split_bf16(src[(size_t)8 * g.vdim], src[(size_t)9 * g.vdim], bh[j][1], bl[j][1]);
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        uint32_t ah[4], al[4];
        const int off = (16 * m + (lane & 15)) * kld + k0 + 8 * (lane >> 4);
        ldmatrix4(ah, qs + off);
        ldmatrix4(al, ks + off);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], ah[0], ah[1], ah[2], ah[3], bh[j][0], bh[j][1]);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], ah[0], ah[1], ah[2], ah[3], bl[j][0], bl[j][1]);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], al[0], al[1], al[2], al[3], bh[j][0], bh[j][1]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // ---- token-pair weights x values
  if (c0 < g.vdim) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t vf[NTW][2];
#pragma unroll
      for (int j = 0; j < NTW; ++j) ldmatrix2_t(vf[j], vs + (16 * k + (lane & 15)) * vld + (c0 + 8 * j < g.vdim ? c0 + 8 * j : 0));
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (m < k) continue;
        uint32_t ah[4], al[4];
        const int off = (16 * m + (lane & 15)) * kPld + 16 * k + 8 * (lane >> 4);
        ldmatrix4(ah, ph + off);
        ldmatrix4(al, pl + off);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], ah[0], ah[1], ah[2], ah[3], vf[j][0], vf[j][1]);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], al[0], al[1], al[2], al[3], vf[j][0], vf[j][1]);
      }
    }
  }
  // ---- head norm and gate
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float sq = 0.f;
#pragma unroll
      for (int j = 0; j < NTW; ++j)
        if (c0 + 8 * j < g.vdim) sq += o[m][j][2 * h] * o[m][j][2 * h] + o[m][j][2 * h + 1] * o[m][j][2 * h + 1];
      sq += __shfl_xor_sync(0xffffffffu, sq, 1);
      sq += __shfl_xor_sync(0xffffffffu, sq, 2);
      if (tl == 0) sq_s[warp][16 * m + gq + 8 * h] = sq;
    }
  __syncthreads();
  if (c0 >= g.vdim) return;
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = 16 * m + gq + 8 * h;
      if (t >= n) continue;
      float sq = 0.f;
#pragma unroll
      for (int w = 0; w < kGcWarps; ++w) sq += sq_s[w][t];
      const float inv = 1.0f / sqrtf(sq / (float)g.vdim + g.eps);
      const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(r.gate) + (row + t) * r.ld + (size_t)head * g.vdim + 2 * tl;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(r.out) + (row + t) * r.ldo + (size_t)head * g.vdim + 2 * tl;
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        const int c = c0 + 8 * j;
        if (c < g.vdim) {
          const uint32_t gw = *reinterpret_cast<const uint32_t*>(gate + c);
          const float2 w = *reinterpret_cast<const float2*>(g.norm + c + 2 * tl);
          *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[m][j][2 * h] * inv * w.x * gl_silu(bf16_bits_to_float(gw & 0xFFFFu)),
                                                            o[m][j][2 * h + 1] * inv * w.y * gl_silu(bf16_bits_to_float(gw >> 16)));
        }
      }
    }
}

// ------------------------------------------------------------------------------------------------ launch
static size_t state_smem(const Gla& g) {
  return (size_t)kGcTokens * (2 * (g.dim + kGcPad) + g.vdim + kGcPad) * 2 + ((size_t)kGcTokens * (g.dim + g.rank) + (size_t)g.rank * g.dim) * 4;
}

bool gla_chunked_supported(const Gla& g, const GlaRows& r) {
  const uintptr_t bits = (uintptr_t)r.q | (uintptr_t)r.k | (uintptr_t)r.v | (uintptr_t)r.gate;
  return g.dim % 16 == 0 && g.vdim % 16 == 0 && g.dim <= 256 && g.vdim <= 256 && r.ld % 8 == 0 && (bits & 15) == 0 && r.ldo % 2 == 0 &&
         ((uintptr_t)r.out & 3) == 0 && ((uintptr_t)g.state & 15) == 0 && ((uintptr_t)g.norm & 7) == 0 && state_smem(g) <= 226 * 1024;
}

template <int NTW>
static int launch_out(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, dim3 grid, const float* logs, const float* states) {
  size_t tail = (size_t)kGcTokens * g.dim * 4;
  if (tail < (size_t)kGcTokens * (g.vdim + kGcPad) * 2) tail = (size_t)kGcTokens * (g.vdim + kGcPad) * 2;
  const size_t smem = (size_t)kGcTokens * (2 * (g.dim + kGcPad) + 2 * (kGcTokens + kGcPad)) * 2 + tail;
  auto kern = gla_chunk_out_kernel<NTW>;
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3(kGcThreads), smem, g, r, b, logs, states));
  return TQ_OK;
}

int launch_gla_chunked(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b) {
  const size_t chunks = (size_t)b.rows / kGcTokens + b.n_seqs, channels = (size_t)g.heads * g.dim, per = channels * g.vdim;
  if (int st = ensure_scratch(ctx, (chunks * (per + channels) + (size_t)b.rows * channels) * sizeof(float))) return st;
  float* upd = static_cast<float*>(ctx->scratch);
  float* total = upd + chunks * per;
  float* logs = total + chunks * channels;
  const dim3 grid((unsigned)((b.max_q + kGcTokens - 1) / kGcTokens), (unsigned)g.heads, (unsigned)b.n_seqs);
  const size_t smem = state_smem(g);
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(gla_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, gla_chunk_state_kernel, grid, dim3(kGcThreads), smem, g, r, b, logs, upd, total));
  TQ_CUDA(ctx, launch_k(ctx, gla_chunk_carry_kernel, dim3((unsigned)((per / 4 + 255) / 256), (unsigned)b.n_seqs), dim3(256), 0, g, b, upd, (const float*)total));
  const float* l = logs;
  const float* st = upd;
  if (g.vdim <= 64) return launch_out<1>(ctx, g, r, b, grid, l, st);
  if (g.vdim <= 128) return launch_out<2>(ctx, g, r, b, grid, l, st);
  return launch_out<4>(ctx, g, r, b, grid, l, st);
}

}  // namespace tq
