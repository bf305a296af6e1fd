// Grouped-query attention under a sliding window, with capped scores, a sink and an output gate:
//     s = (q . k) * scale;  s <- softcap * tanh(s / softcap)          (softcap 0: no cap)
//     p_j = exp(s_j) / (exp(sink) + sum exp(s))                       (one sink, or one per head; -infinity: none; it has no value)
//     out = (sum p_j v_j) * sigmoid(gate)                             (no gate pointer: 1)
// Mask: the query at position i sees key j when j <= i and i - j < window.
//
// Pooled blocks (pool > 0): positions b pool .. b pool + pool - 1 have an averaged key and value, which are one more term of the
// softmax once the window has moved past all of them, b pool + pool - 1 <= i - window.  Until then the positions that the window
// has dropped count for nothing.
#pragma once

#include "internal.h"
#include "ragged.h"

namespace tq {

// Cache rows: keys [kv_heads][dim_pad], values [kv_heads][vdim_pad]; the padding (to 8 elements) is zero.
struct WindowAttn {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dim_pad = 0, vdim_pad = 0;
  int window = 0;
  float scale = 0.f, softcap = 0.f, sink = 0.f;
  const float* sinks = nullptr;        // [heads], instead of `sink`
  size_t q_head = 0;                   // elements between the heads of a query row; 0: dim
  float out_scale = 1.f;               // factor on the result
  int pool = 0, pool_rows = 0, max_seq = 0;            // pooled rows and cache rows per slot
  const void *pooled_keys = nullptr, *pooled_values = nullptr;   // [slot * pool_rows + block], rows as in the caches
};

// Pooled blocks that the query at position `pos` sees.
__host__ __device__ inline int seen_blocks(int pos, int window, int pool) { return pos >= window ? (pos - window + 1) / pool : 0; }

// q [rows][ldq], head h at column h * dim (q_head); gate [rows][ldg] and out [rows][ldo], head h at column h * vdim.  dtype (TQ_BF16 or
// TQ_F32) is that of q, gate, caches and out; scores, weights and sums are f32, in TQ_F32 every operation is.
int launch_window_attention(tq_ctx* ctx, const WindowAttn& a, const RaggedBatch& b, int dtype, const void* q, size_t ldq, const void* gate,
                            size_t ldg, const void* k_cache, const void* v_cache, void* out, size_t ldo);

}  // namespace tq
