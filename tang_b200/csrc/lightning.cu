// Lightning attention over prompts in bf16, in chunks of 64 tokens on the tensor cores (see gla.cuh for the recurrence).  With d
// the head's decay, t and s counted inside a chunk of n tokens and S the state before it,
//     o_t = d^(t+1) q_t^T S + sum_{s <= t} d^(t-s) (q_t . k_s) v_s
//     S'  = d^n S + sum_s (d^(n-1-s) k_s) v_s^T.
//   1. lightning_state_kernel  (chunk, head): the chunk's own contribution to the state;
//   2. lightning_carry_kernel: walks the chunks of a sequence, leaves every chunk the state before it, updates the slot;
//   3. lightning_out_kernel    (chunk, head): the outputs.
// Queries, keys and values are bf16 already and the decay of a token pair is a factor on its score, so only decayed keys, states
// and token-pair weights enter the products as two bf16 terms; all sums are f32.
#include "attn_mma.cuh"
#include "gla_device.cuh"

namespace tq {

constexpr int kLnTokens = 64;
constexpr int kLnThreads = 256, kLnWarps = kLnThreads / 32;
constexpr int kLnPad = 8;            // bf16 elements of padding per shared-memory row (one bank group)

// d^0 .. d^64 into shared memory
__device__ __forceinline__ void ln_powers(float decay, float* pw) {
  if (threadIdx.x <= kLnTokens) pw[threadIdx.x] = threadIdx.x == 0 ? 1.0f : exp2f((float)threadIdx.x * log2f(decay));
}

__device__ __forceinline__ void ln_copy(__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, size_t ld_src, int n_rows, int cols) {
  const int per = cols / 8;
  for (int i = threadIdx.x; i < kLnTokens * per; i += kLnThreads) {
    const int t = i / per, c = i - t * per;
    const bool ok = t < n_rows;
    cp_async16(smem_u32(dst + t * ld + 8 * c), ok ? src + (size_t)t * ld_src + 8 * c : src, ok);
  }
}

// First chunk of a sequence in the workspace (at most rows / 64 + sequences chunks in all).
__device__ __forceinline__ size_t ln_first_chunk(const GlaSeq& s, int seq) { return (size_t)(s.row0 / kLnTokens) + seq; }

// ------------------------------------------------------------------------------------------------ 1. contributions
__global__ void __launch_bounds__(kLnThreads) lightning_state_kernel(Gla g, GlaRows r, RaggedBatch b, float* upd) {
  extern __shared__ __align__(16) uint8_t ln_smem[];
  __shared__ float pw[kLnTokens + 1];
  const int kld = g.dim + kLnPad, vld = g.vdim + kLnPad;
  __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(ln_smem);     // [64][kld] keys, then the leading terms of the decayed keys
  __nv_bfloat16* kl = kh + kLnTokens * kld;
  __nv_bfloat16* vs = kl + kLnTokens * kld;                          // [64][vld]
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  ln_powers(g.head_decay[head], pw);                                 // (weights: before the wait)
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.z, s)) return;
  const int t0 = blockIdx.x * kLnTokens, n = min(kLnTokens, s.n - t0);
  if (n <= 0) return;
  const size_t row = s.row0 + t0, chunk = ln_first_chunk(s, blockIdx.z) + blockIdx.x;
  ln_copy(kh, kld, static_cast<const __nv_bfloat16*>(r.k) + row * r.ld + (size_t)head * g.dim, r.ld, n, g.dim);
  ln_copy(vs, vld, static_cast<const __nv_bfloat16*>(r.v) + row * r.ld + (size_t)head * g.vdim, r.ld, n, g.vdim);
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  for (int i = threadIdx.x; i < kLnTokens * g.dim / 2; i += kLnThreads) {
    const int t = 2 * i / g.dim, d = 2 * i - t * g.dim;
    const uint32_t kw = *reinterpret_cast<const uint32_t*>(kh + t * kld + d);
    const float f = t < n ? pw[n - 1 - t] : 0.f;
    uint32_t hi, lo;
    split_bf16(bf16_bits_to_float(kw & 0xFFFFu) * f, bf16_bits_to_float(kw >> 16) * f, hi, lo);
    *reinterpret_cast<uint32_t*>(kh + t * kld + d) = hi;
    *reinterpret_cast<uint32_t*>(kl + t * kld + d) = lo;
  }
  __syncthreads();
  // [dim x 64] x [64 x vdim]: a warp takes units of 16 channels x 64 columns
  const int n_mt = g.dim / 16, n_cb = (g.vdim + 63) / 64;
  float* out = upd + ((chunk * g.heads + head) * g.dim) * g.vdim;
  for (int u = warp; u < n_mt * n_cb; u += kLnWarps) {
    const int mt = u % n_mt, c0 = (u / n_mt) * 64, nt = min(8, (g.vdim - c0) / 8);
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int k = 0; k < kLnTokens / 16; ++k) {
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
__global__ void __launch_bounds__(256) lightning_carry_kernel(Gla g, RaggedBatch b, float* upd) {
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.y, s)) return;
  const size_t per = (size_t)g.heads * g.dim * g.vdim, i = 4 * ((size_t)blockIdx.x * 256 + threadIdx.x);
  if (i >= per) return;
  const int chunks = (s.n + kLnTokens - 1) / kLnTokens, last = s.n - (chunks - 1) * kLnTokens;
  const float l2 = log2f(g.head_decay[i / ((size_t)g.dim * g.vdim)]), whole = exp2f((float)kLnTokens * l2), tail = exp2f((float)last * l2);
  float* st = g.state + s.slot * per + i;
  float4 S = s.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(st);
  float* u = upd + ln_first_chunk(s, blockIdx.y) * per + i;
  constexpr int U = 8;
  for (int c = 0; c < chunks; c += U) {
    float4 x[U];
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c + j < chunks) x[j] = *reinterpret_cast<const float4*>(u + (size_t)(c + j) * per);
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c + j < chunks) {
        const float f = c + j == chunks - 1 ? tail : whole;
        *reinterpret_cast<float4*>(u + (size_t)(c + j) * per) = S;
        S.x = fmaf(f, S.x, x[j].x);
        S.y = fmaf(f, S.y, x[j].y);
        S.z = fmaf(f, S.z, x[j].z);
        S.w = fmaf(f, S.w, x[j].w);
      }
  }
  *reinterpret_cast<float4*>(st) = S;
}

// ------------------------------------------------------------------------------------------------ 3. outputs
// NTW: 8-column tiles per warp (vdim <= 64 NTW).
template <int NTW>
__global__ void __launch_bounds__(kLnThreads, 2) lightning_out_kernel(Gla g, GlaRows r, RaggedBatch b, const float* states, float* o_out) {
  extern __shared__ __align__(16) uint8_t ln_smem[];
  __shared__ float pw[kLnTokens + 1];
  constexpr int kPld = kLnTokens + kLnPad;
  const int kld = g.dim + kLnPad, vld = g.vdim + kLnPad;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(ln_smem);      // [64][kld]
  __nv_bfloat16* ks = qs + kLnTokens * kld;
  __nv_bfloat16* vs = ks + kLnTokens * kld;                           // [64][vld]
  __nv_bfloat16* ph = vs + kLnTokens * vld;                           // [64][kPld] token-pair weights, two terms
  __nv_bfloat16* pl = ph + kLnTokens * kPld;
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tl = lane & 3;
  ln_powers(g.head_decay[head], pw);
  pdl_wait();
  pdl_launch_dependents();
  GlaSeq s;
  if (!gl_sequence(g, b, blockIdx.z, s)) return;
  const int t0 = blockIdx.x * kLnTokens, n = min(kLnTokens, s.n - t0);
  if (n <= 0) return;
  const size_t row = s.row0 + t0, chunk = ln_first_chunk(s, blockIdx.z) + blockIdx.x;
  ln_copy(qs, kld, static_cast<const __nv_bfloat16*>(r.q) + row * r.ld + (size_t)head * g.dim, r.ld, n, g.dim);
  ln_copy(ks, kld, static_cast<const __nv_bfloat16*>(r.k) + row * r.ld + (size_t)head * g.dim, r.ld, n, g.dim);
  asm volatile("cp.async.commit_group;" ::: "memory");
  ln_copy(vs, vld, static_cast<const __nv_bfloat16*>(r.v) + row * r.ld + (size_t)head * g.vdim, r.ld, n, g.vdim);
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();

  // ---- token pairs: a warp forms 16 queries x 32 keys
  {
    const int mt = warp & 3, s0 = 32 * (warp >> 2);
    if (s0 <= 16 * mt + 15) {
      float acc[4][4] = {};
      const __nv_bfloat16* qa = qs + (16 * mt + (lane & 15)) * kld + 8 * (lane >> 4);
      const __nv_bfloat16* ka = ks + (s0 + (lane & 7) + 8 * (lane >> 4)) * kld + 8 * ((lane >> 3) & 1);
      for (int k0 = 0; k0 < g.dim; k0 += 16) {
        uint32_t qf[4], kf[2][4];
        ldmatrix4(qf, qa + k0);
        ldmatrix4(kf[0], ka + k0);
        ldmatrix4(kf[1], ka + 16 * kld + k0);
#pragma unroll
        for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[j], qf[0], qf[1], qf[2], qf[3], kf[j >> 1][2 * (j & 1)], kf[j >> 1][2 * (j & 1) + 1]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = 16 * mt + gq + 8 * h, sj = s0 + 8 * j + 2 * tl;
          const float f0 = sj <= t ? acc[j][2 * h] * pw[t - sj] : 0.f, f1 = sj + 1 <= t ? acc[j][2 * h + 1] * pw[t - sj - 1] : 0.f;
          uint32_t hi, lo;
          split_bf16(f0, f1, hi, lo);
          *reinterpret_cast<uint32_t*>(ph + t * kPld + sj) = hi;
          *reinterpret_cast<uint32_t*>(pl + t * kPld + sj) = lo;
        }
    }
  }
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
        uint32_t a[4];
        ldmatrix4(a, qs + (16 * m + (lane & 15)) * kld + k0 + 8 * (lane >> 4));
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], a[0], a[1], a[2], a[3], bh[j][0], bh[j][1]);
#pragma unroll
        for (int j = 0; j < NTW; ++j) mma_bf16_16816(o[m][j], a[0], a[1], a[2], a[3], bl[j][0], bl[j][1]);
      }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const float f0 = pw[16 * m + gq + 1], f1 = pw[16 * m + gq + 9];
#pragma unroll
      for (int j = 0; j < NTW; ++j) {
        o[m][j][0] *= f0;
        o[m][j][1] *= f0;
        o[m][j][2] *= f1;
        o[m][j][3] *= f1;
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (c0 >= g.vdim) return;
  // ---- token-pair weights x values
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    uint32_t vf[NTW][2];
#pragma unroll
    for (int j = 0; j < NTW; ++j) {
      const void* p = vs + (16 * k + (lane & 15)) * vld + (c0 + 8 * j < g.vdim ? c0 + 8 * j : 0);
      asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(vf[j][0]), "=r"(vf[j][1]) : "r"(smem_u32(p)));
    }
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
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = 16 * m + gq + 8 * h;
      if (t >= n) continue;
      float* dst = o_out + ((row + t) * g.heads + head) * g.vdim + 2 * tl;
#pragma unroll
      for (int j = 0; j < NTW; ++j)
        if (c0 + 8 * j < g.vdim) *reinterpret_cast<float2*>(dst + c0 + 8 * j) = make_float2(o[m][j][2 * h], o[m][j][2 * h + 1]);
    }
}

// ------------------------------------------------------------------------------------------------ launch
static size_t out_smem(const Gla& g) {
  return (size_t)kLnTokens * (2 * (g.dim + kLnPad) + g.vdim + kLnPad + 2 * (kLnTokens + kLnPad)) * 2;
}

bool lightning_chunked_supported(const Gla& g, const GlaRows& r) {
  const uintptr_t bits = (uintptr_t)r.q | (uintptr_t)r.k | (uintptr_t)r.v;
  return g.dim % 16 == 0 && g.vdim % 16 == 0 && g.dim <= 256 && g.vdim <= 256 && r.ld % 8 == 0 && (bits & 15) == 0 && ((uintptr_t)g.state & 15) == 0;
}

size_t lightning_chunk_floats(const Gla& g, const RaggedBatch& b) {
  return ((size_t)b.rows / kLnTokens + b.n_seqs) * g.heads * g.dim * g.vdim;
}

template <int NTW>
static int launch_out(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, dim3 grid, const float* states, float* o) {
  const size_t smem = out_smem(g);
  auto kern = lightning_out_kernel<NTW>;
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, kern, grid, dim3(kLnThreads), smem, g, r, b, states, o));
  return TQ_OK;
}

int launch_lightning_chunked(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, float* o, float* work) {
  const size_t per = (size_t)g.heads * g.dim * g.vdim;
  const dim3 grid((unsigned)((b.max_q + kLnTokens - 1) / kLnTokens), (unsigned)g.heads, (unsigned)b.n_seqs);
  const size_t smem = (size_t)kLnTokens * (2 * (g.dim + kLnPad) + g.vdim + kLnPad) * 2;
  if (smem > 48 * 1024) TQ_CUDA(ctx, cudaFuncSetAttribute(lightning_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  TQ_CUDA(ctx, launch_k(ctx, lightning_state_kernel, grid, dim3(kLnThreads), smem, g, r, b, work));
  TQ_CUDA(ctx, launch_k(ctx, lightning_carry_kernel, dim3((unsigned)((per / 4 + 255) / 256), (unsigned)b.n_seqs), dim3(256), 0, g, b, work));
  if (g.vdim <= 64) return launch_out<1>(ctx, g, r, b, grid, work, o);
  if (g.vdim <= 128) return launch_out<2>(ctx, g, r, b, grid, work, o);
  return launch_out<4>(ctx, g, r, b, grid, work, o);
}

}  // namespace tq

using namespace tq;

extern "C" int tq_lightning(tq_ctx* ctx, int dtype, size_t heads, size_t dim, size_t vdim, float eps, const float* decay_dev, const void* q_dev,
                            const void* k_dev, const void* v_dev, const void* gate_dev, size_t ld, const float* norm_dev, float* state_dev, size_t max_seq,
                            size_t cache_rows, const int* seq_rows_dev, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows,
                            size_t max_q, void* out_dev, size_t ldo) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, dtype == TQ_BF16 || dtype == TQ_F32, "tq_lightning: dtype must be bf16 or f32");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, decay_dev && q_dev && k_dev && v_dev && gate_dev && norm_dev && state_dev && row_pos_dev && cache_row_dev && out_dev, "tq_lightning: null pointer");
  TQ_REQUIRE(ctx, seq_rows_dev || (rows == n_seqs && max_q == 1), "tq_lightning: without row offsets every sequence brings one row");
  Gla g;
  g.heads = (int)heads;
  g.dim = (int)dim;
  g.vdim = (int)vdim;
  g.eps = eps;
  g.norm = norm_dev;
  g.head_decay = decay_dev;
  g.state = state_dev;
  g.max_seq = (int)max_seq;
  GlaRows r;
  r.q = q_dev;
  r.k = k_dev;
  r.v = v_dev;
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
  return launch_gla(ctx, g, r, b, dtype);
}
