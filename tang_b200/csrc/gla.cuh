// Gated linear attention: a recurrent state S [dim][vdim] per head with a decay per key channel,
//     alpha_t = sigmoid(z_t)^(1/tau),  z_t = a2 a1_t + bias            (a1_t: `rank` values per row)
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T (q_t * q_scale)
//     out_t = o_t / sqrt(mean(o_t^2) + eps) * norm * silu(gate_t)       (mean over the head's vdim values)
// The state starts at zero with a sequence's position 0 and is kept in f32 from step to step, one per cache slot.
//
// Lightning attention is the same recurrence with one constant decay per head, and its output is normed over all heads together
// and gated by a sigmoid:
//     out_t = o_t / sqrt(mean(o_t^2) + eps) * norm * sigmoid(gate_t)    (o_t: the heads' vdim values side by side)
#pragma once

#include "internal.h"
#include "ragged.h"

namespace tq {

struct Gla {
  int heads = 0, dim = 0, vdim = 0, rank = 0;
  float tau = 1.f, q_scale = 1.f, eps = 0.f;
  const float *a2 = nullptr, *a2_bias = nullptr;   // [heads * dim][rank], [heads * dim]
  const float* norm = nullptr;                     // [vdim]; lightning: [heads * vdim]
  const float* head_decay = nullptr;               // [heads]: lightning; rank, tau, a2, a2_bias and rows of a1 are not used then
  float* state = nullptr;                          // [slots][heads][dim][vdim]
  int max_seq = 0;                                 // cache rows per slot: a row's slot is cache_row / max_seq
};

// Rows of q, k (heads * dim values each), v and gate (heads * vdim), all with `ld` elements between rows; a1 [rows][ld_a1] f32;
// out [rows][ldo].  dtype (TQ_BF16 or TQ_F32) is that of q, k, v, gate and out; everything else is f32.
struct GlaRows {
  const void *q = nullptr, *k = nullptr, *v = nullptr, *gate = nullptr;
  size_t ld = 0;
  const float* a1 = nullptr;
  size_t ld_a1 = 0;
  void* out = nullptr;
  size_t ldo = 0;
};

// Prompts in bf16 on the tensor cores (csrc/gla_chunk.cu): head sizes that are multiples of 16 up to 256, rows and sections on
// 16-byte boundaries.
bool gla_chunked_supported(const Gla& g, const GlaRows& r);
int launch_gla_chunked(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b);

// The same for lightning attention (csrc/lightning.cu): o [rows][heads * vdim] f32 (16-byte aligned), before norm and gate; work:
// lightning_chunk_floats values.
bool lightning_chunked_supported(const Gla& g, const GlaRows& r);
size_t lightning_chunk_floats(const Gla& g, const RaggedBatch& b);
int launch_lightning_chunked(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, float* o, float* work);

int launch_gla(tq_ctx* ctx, const Gla& g, const GlaRows& r, const RaggedBatch& b, int dtype);

}  // namespace tq
