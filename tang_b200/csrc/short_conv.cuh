// Short causal convolutions over time on every channel of a sequence's rows,
//     y_t = sum_j w[j] u_(t - taps + 1 + j)         (zeros before the sequence's position 0),
// as a row operator (h + conv(h)) and fused with what follows the projections of queries, keys and values.  The last taps - 1 inputs
// of a sequence stay in its cache slot from step to step.
//
// Steps of one row per sequence update that state inside the kernels that use it.  In other steps a row's predecessors are in the
// batch too, other CTAs still read the old state while the rows are worked off, and launch_conv_tails moves it on afterwards.
#pragma once

#include "internal.h"
#include "ragged.h"
#include "rowops.cuh"

namespace tq {

struct ShortConv {
  int taps = 1;
  int channels = 0;
  const float* w = nullptr;        // [taps][channels]; null: y = u
  void* state = nullptr;           // [slots][taps - 1][channels] of the model's dtype; the last row is the latest input
  int max_seq = 1;                 // cache rows per slot
};

// Source [channels, taps] (bf16 or f32, host or device) to columns col0 ... of w [taps][ld].
int put_conv_weights(tq_ctx* ctx, const void* src, int src_dtype, float* w, size_t channels, size_t taps, size_t ld, size_t col0);

// out = x + conv(x) for rows of c.channels values; x and out are different buffers.
int launch_conv_residual(tq_ctx* ctx, const ShortConv& c, const RaggedBatch& b, int dtype, const void* x, size_t ldx, void* out, size_t ldo);

// What follows the projections of attention: raw rows hold queries, keys and values at columns 0, k0 and v0 (the convolution's
// channels are the raw columns); queries and keys are convolved, rotated and rms-normed per head (no gain; norm
// false: not); values are only convolved.  Queries go to q, keys and values to the row's cache row.
// Blocks of `pool` tokens (0: none) get one pooled row each, the mean of their keys and of their values as the cache holds them.
// A step forms the rows of the blocks whose last position is at least its first one minus 1 and lies before its last one: a
// block is complete in the cache one row before any query behind it can see it.
struct ConvHeads {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int key_pad = 0, val_pad = 0;    // of one head in the caches, multiples of 8; the padding stays zero
  const void* raw = nullptr;
  size_t ld = 0;
  int k0 = 0, v0 = 0;
  ShortConv conv;
  Rotation rot;                    // in halves, from dimension 0
  bool norm = true;
  float eps = 0.f;
  void* q = nullptr;               // [rows][ldq], head h at column h * dim
  size_t ldq = 0;
  void *keys = nullptr, *values = nullptr;                 // [cache row][kv_heads][key_pad / val_pad]
  int pool = 0, pool_rows = 0;     // pooled rows per slot
  void *pooled_keys = nullptr, *pooled_values = nullptr;   // [slot * pool_rows + block][kv_heads][key_pad / val_pad]
};
int launch_conv_heads(tq_ctx* ctx, const ConvHeads& a, const RaggedBatch& b, int dtype);

// Moves the states of up to kMaxConvTails convolutions on by a step's rows.
constexpr int kMaxConvTails = 4;
struct ConvTail {
  ShortConv c;
  const void* x = nullptr;         // the step's inputs
  size_t ldx = 0;
};
int launch_conv_tails(tq_ctx* ctx, const ConvTail* tails, int n, const RaggedBatch& b, int dtype);

}  // namespace tq
