// minGRU: per channel, a leaky average whose rate and input depend on the current row alone,
//     z = sigmoid(z_t + z_bias);  u = u_t + u_bias;  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//     S_t = (1 - z) S_(t-1) + z c;   out_t = S_t * silu(gate_t) * out_scale
// The state starts at zero with a sequence's position 0 and is kept in f32 from step to step, one per cache slot.
#pragma once

#include "internal.h"
#include "ragged.h"

namespace tq {

struct MinGru {
  int width = 0;
  const float *z_bias = nullptr, *u_bias = nullptr;   // [width]
  float out_scale = 1.f;
  float* state = nullptr;                             // [slots][width rounded up to 2]
  int max_seq = 0;                                    // cache rows per slot: a row's slot is cache_row / max_seq
};

// Rows of z, u and gate with `ld` elements between rows, out [rows][ldo]; dtype (TQ_BF16 or TQ_F32) is that of all four, the
// gates and the recurrence are f32.  All `ld`, `ldo` and the pointers are even multiples of the element size.
struct MinGruRows {
  const void *z = nullptr, *u = nullptr, *gate = nullptr;
  size_t ld = 0;
  void* out = nullptr;
  size_t ldo = 0;
};
int launch_min_gru(tq_ctx* ctx, const MinGru& g, const MinGruRows& r, const RaggedBatch& b, int dtype);

}  // namespace tq
