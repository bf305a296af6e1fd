// Device pieces shared by the gated-linear-attention kernels.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"
#include "gla.cuh"

namespace tq {

__device__ __forceinline__ float gl_load(const float* p) { return *p; }
__device__ __forceinline__ float gl_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void gl_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void gl_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// log of a channel's decay: log(sigmoid(z)) / tau
__device__ __forceinline__ float gl_log_decay(float z, float inv_tau) { return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau; }

__device__ __forceinline__ float gl_decay_logit(const Gla& g, int channel, const float* a1) {
  float z = g.a2_bias[channel];
  const float* w = g.a2 + (size_t)channel * g.rank;
  for (int r = 0; r < g.rank; ++r) z = fmaf(w[r], a1[r], z);
  return z;
}

// Decay of a channel at a row whose a1 values are given (null: constant decays).
__device__ __forceinline__ float gl_decay(const Gla& g, int head, int channel, const float* a1) {
  return g.head_decay ? g.head_decay[head] : expf(gl_log_decay(gl_decay_logit(g, channel, a1), 1.0f / g.tau));
}

__device__ __forceinline__ float gl_silu(float x) { return x / (1.0f + expf(-x)); }

// The rows of a sequence and its state; false: nothing to do.
struct GlaSeq {
  int row0, n;
  size_t slot;
  bool fresh;          // the sequence starts here
};
__device__ __forceinline__ bool gl_sequence(const Gla& g, const RaggedBatch& b, int seq, GlaSeq& s) {
  s.row0 = b.seq_rows ? b.seq_rows[seq] : seq;
  s.n = b.seq_rows ? b.seq_rows[seq + 1] - s.row0 : 1;
  if (s.n <= 0 || s.row0 < 0 || s.row0 + s.n > b.rows) return false;
  const int c0 = b.cache_row[s.row0], c1 = b.cache_row[s.row0 + s.n - 1];
  if (c0 < 0 || c1 != c0 + s.n - 1 || (size_t)c1 >= b.cache_rows) return false;    // (reported by the embedding kernel)
  s.slot = (size_t)(c0 / g.max_seq);
  s.fresh = b.row_pos[s.row0] == 0;
  return true;
}

}  // namespace tq
