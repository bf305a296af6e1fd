// Differential attention over a key/value cache: every query head has two query maps and every key head two key maps;
// each map is a softmax attention of its own over the same values, and a head's output is
//     o = a1 - lambda * a2;   o <- o / sqrt(mean(o^2) + eps) * out_scale       (mean over the head's vdim values).
// Mask: the query at position i sees key j when j <= i and (i - j < window or j < keep_first).
#pragma once

#include "internal.h"
#include "ragged.h"

namespace tq {

// One layer's keys and values: row r of slot s is row s * max_seq + r of both matrices.  A key row is [kv_heads][2][dim_pad],
// a value row [kv_heads][vdim_pad]; the padding (to 8 elements) is zero.
struct DiffAttn {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0, dim_pad = 0, vdim_pad = 0;
  int window = 0, keep_first = 0;
  float scale = 0.f, lambda = 0.f, out_scale = 1.f, eps = 0.f;
};

// q [rows][ldq], head h's map m at column (2h + m) * dim; out [rows][ldo], head h at column h * vdim.  dtype (TQ_BF16 or
// TQ_F32) is that of q, keys, values and out; in TQ_F32 every operation is f32.
int launch_diff_attention(tq_ctx* ctx, const DiffAttn& a, const RaggedBatch& b, int dtype, const void* q, size_t ldq, const void* k_cache,
                          const void* v_cache, void* out, size_t ldo);

}  // namespace tq
