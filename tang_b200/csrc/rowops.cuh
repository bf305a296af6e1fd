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

// Rotation of `dims` dimensions of every head, from `first` on, in the "rotate half" pairing: dimension i turns with i + dims / 2 by
// position * freq[i]; interleaved: dimension 2i turns with 2i + 1.  Cosine and sine are multiplied by `mult`.
struct Rotation {
  int dims = 0;
  const float* freq = nullptr;     // [dims / 2]
  float mult = 1.f;
  int first = 0;                   // per-head norms only, as `interleaved`
  bool interleaved = false;
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

// The same per head: every head is normed over its own dim values with gains of size dim shared by all heads (null: no norm), and
// head h of a query row starts at q_head * h.
struct HeadNormRope {
  QkNormRope r;
  size_t q_head = 0;
};
int launch_head_norm_rope(tq_ctx* ctx, const HeadNormRope& a, const RaggedBatch& b, int dtype);

// Hyper-connections: `streams` residual rows per row of the batch.
//     x'_t = sum_s mix[s][t] x_s + w_out[t] y;   u = sum_s w_in[s] x'_s;   out = u / rms(u) * gain
// y gathers a sublayer's output: the weighted rows of its chosen experts (a negative row: the sublayer's own input, `self`) and
// one more row, multiplied by a sigmoid if there is a gate.
// Steps of one row per sequence may add a short convolution: out <- out + conv(out), whose states move on by the row.
constexpr int kMaxStreams = 16;
struct StreamMix {
  int streams = 1, src_streams = 1;
  const float* src = nullptr;        // [rows][src_streams][width]; src_streams 1: all streams are equal
  const int* src_rows = nullptr;     // row of src of output row m; null: m.  Not with y
  float* dst = nullptr;              // [rows][streams][width], may be src; with y
  const float* y = nullptr;          // f32 rows of `width`; null: the streams stay
  const int* y_rows = nullptr;       // [rows * n_y]; null: row m
  const float* y_weight = nullptr;   // [rows * n_y], with y_rows
  int n_y = 1;
  const void* self = nullptr;        // of out_dtype, ld_out; may be out
  const float* y_more = nullptr;
  const float* y_more_gate = nullptr;   // row m's logit at m * ld_gate; null: no gate
  size_t ld_gate = 0;
  const float* inject = nullptr;     // [rows][width], added to every x' after `sum`; with y
  const float *mix = nullptr, *w_out = nullptr, *w_in = nullptr;   // w_in null: ones
  const float* gain = nullptr;       // null: no norm, no out
  void* out = nullptr;
  int out_dtype = TQ_BF16;
  size_t ld_out = 0;
  float eps = 0.f;
  float* sum = nullptr;              // [rows][width] sum of the streams
  const float* conv_w = nullptr;     // [conv_taps][width]; null: no convolution
  void* conv_state = nullptr;        // [slots][conv_taps - 1][width] of out_dtype
  int conv_taps = 0, max_seq = 1;    // cache rows per slot
  const int *row_pos = nullptr, *cache_row = nullptr;   // of the convolution
};
int launch_stream_mix(tq_ctx* ctx, const StreamMix& a, size_t rows, size_t width);

// out = o / rms(o) * norm * sigmoid(gate) over whole rows of `width` values; o f32, gate and out of dtype.
int launch_norm_gate(tq_ctx* ctx, const float* o, size_t ld_o, const float* norm, const void* gate, size_t ldg, void* out, size_t ldo, const int* cache_row,
                     size_t rows, size_t width, float eps, int dtype);

// Frequencies stretched by wavelength (factor > 0): 2 pi / f below original / high stays, above original / low is divided by
// `factor`, between them the two are blended.
void banded_frequencies(int dims, double base, double factor, double low, double high, double original, float* freq);

// Frequencies of a rotation with base `base`, stretched by YaRN when factor > 0 (interpolated by `factor` below `slow`
// turns over `original` positions, left alone above `fast`, blended between); *mult receives the factor on cos and sin.
void yarn_frequencies(int dims, double base, double factor, double original, double fast, double slow, float* freq, float* mult);

}  // namespace tq
