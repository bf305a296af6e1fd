// Operators on activation rows between the matrix products: sublayer output -> norm -> stream -> next norm, and the norm and
// rotation of queries and keys.
#pragma once

#include "internal.h"
#include "ragged.h"

namespace tq {

// For every row:  y = sum of its sublayer's outputs;  x += y / rms(y) * gain_post;  out = x / rms(x) * gain_next,
// rms(v) = sqrt(mean(v^2) + eps).  Gains are f32.
struct AddNorm {
  float* x = nullptr;              // [rows][width] f32 stream, updated in place
  const float* y = nullptr;        // f32 rows of `width` values; null: the stream stays and only the second norm is formed
  const int* y_rows = nullptr;     // rows of y that belong to row m: y_rows[m * n_y + i] (negative: none); null: row m
  int n_y = 1;
  const float* gain_post = nullptr;
  const float* gain_next = nullptr;   // null: no second norm
  void* out = nullptr;             // [rows][ld_out] of out_dtype
  int out_dtype = TQ_BF16;
  size_t ld_out = 0;
  float eps = 0.f;
};
int launch_add_norm(tq_ctx* ctx, const AddNorm& a, size_t rows, size_t width);

// Rotation of the first `dims` dimensions of every head in the "rotate half" pairing: dimension i turns with i + dims / 2 by
// position * freq[i]; cosine and sine are multiplied by `mult`.
struct Rotation {
  int dims = 0;
  const float* freq = nullptr;     // [dims / 2]
  float mult = 1.f;
};
// q [rows][ldq] (heads * dim values) is divided by the root mean square over the whole row, multiplied by q_gain, rotated and
// written back.  The keys come from `raw` (a cache row's [kv_heads][raw_pad]), get the same treatment over kv_heads * dim
// values and go to `keys` ([kv_heads][key_pad]).  Everything but storage is f32; dtype is that of q, gains and caches.
struct QkNormRope {
  int heads = 0, kv_heads = 0, dim = 0;
  int raw_pad = 0, key_pad = 0;
  void* q = nullptr;
  size_t ldq = 0;
  const void* raw = nullptr;
  void* keys = nullptr;
  const void *q_gain = nullptr, *k_gain = nullptr;
  Rotation rot;
  float eps = 0.f;
};
int launch_qk_norm_rope(tq_ctx* ctx, const QkNormRope& a, const RaggedBatch& b, int dtype);

// Frequencies of a rotation with base `base`, stretched by YaRN when factor > 0 (interpolated by `factor` below `slow`
// turns over `original` positions, left alone above `fast`, blended between); *mult receives the factor on cos and sin.
void yarn_frequencies(int dims, double base, double factor, double original, double fast, double slow, float* freq, float* mult);

}  // namespace tq
