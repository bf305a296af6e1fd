// Latent attention: keys and values of all heads come from one latent c (rank values) and one rotated part r (rot values) per
// position, and only those are cached:
//     c = rmsnorm(c_raw), r = rotate(r_raw);   score_h = (q_h . W_uk,h c + q'_h . r) * scale;   out_h = sum softmax_j W_uv,h c_j
// Two forms share the cache:
//   * expanded (sequences that bring several rows, and everything in f32): keys and values of the sequence's positions are formed
//     with one grouped product over its cache rows and attended by the windowed kernel;
//   * absorbed (sequences that bring one row): q_h W_uk,h is a query over the latents themselves, so all heads read the same cache
//     rows; W_uv,h follows the weighted sum of latents.
#pragma once

#include "internal.h"
#include "ragged.h"
#include "rowops.cuh"

namespace tq {

// A cache row: [latent padded to 16][rotated part padded to 16], the padding zero.
struct LatentDims {
  int heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;
  int c_pad = 0, r_pad = 0;
  __host__ __device__ int row() const { return c_pad + r_pad; }
};
LatentDims latent_dims(int heads, int dim, int rot, int vdim, int rank);

// low: f32 rows [q_rank | latent | rotated part] (first columns 0, c0, c0 + rank).  cq = rmsnorm(q_rank values) * q_gain; the row's
// cache row receives rmsnorm(latent) * c_gain and the rotated part.  head_jobs (may be null): filled with the jobs of per-head
// products over n_head_rows rows each, at most `chunk` per job (group h, rows h * n_head_rows ...).
struct LatentIn {
  LatentDims d;
  const float* low = nullptr;
  size_t ld_low = 0;
  int q_rank = 0, c0 = 0;
  const float *q_gain = nullptr, *c_gain = nullptr;
  void* cq = nullptr;
  size_t ld_cq = 0;
  void* cache = nullptr;
  Rotation rot;
  float eps = 0.f;
  int4* head_jobs = nullptr;
  int* n_head_jobs = nullptr;
  int n_head_rows = 0, head_chunk = 0;
};
int launch_latent_in(tq_ctx* ctx, const LatentIn& a, const RaggedBatch& b, int dtype);

// Which positions are expanded where.  Sequences first_seq .. end_seq - 1 that bring at least min_q rows get consecutive rows.
struct LatentPlan {
  int* off = nullptr;         // [n_seqs] first expanded row; negative: none
  int* exp_row = nullptr;     // [rows] expanded row of every row's position; negative: none
  int* single = nullptr;      // [n_seqs] row of a sequence that brings one row; negative: it brings more
  int4* jobs = nullptr;       // (0, cache row, rows, shift to the expanded row)
  int* n_jobs = nullptr;
};
int launch_latent_plan(tq_ctx* ctx, const RaggedBatch& b, int first_seq, int end_seq, int min_q, int chunk, int max_jobs, const LatentPlan& p);

// keys [expanded row][heads][key_pad]: columns dim .. dim + rot - 1 of every head receive the position's rotated part, the rest zero.
int launch_latent_place(tq_ctx* ctx, const LatentDims& d, const RaggedBatch& b, const LatentPlan& p, const void* cache, void* keys, int key_pad, int dtype);

// Rows of q [head][row][ld] of the sequences that bring one row, to out [head][sequence][ld].
int launch_latent_gather(tq_ctx* ctx, const RaggedBatch& b, const int* single, const void* q, int heads, size_t ld, void* out);

// The absorbed form in bf16, one query per sequence: q_lat and out [head][n_seqs][c_pad] (the padding of out is not written), q
// [head][n_seqs][ldq] with the rotated part from column dim on, still to be rotated if rotate.  single null: sequence b's row is b.
bool latent_absorb_supported(const LatentDims& d);
int launch_latent_decode(tq_ctx* ctx, const LatentDims& d, const RaggedBatch& b, const int* single, float scale, const Rotation& rot, bool rotate,
                         const void* q_lat, const void* q, size_t ldq, const void* cache, void* out);

}  // namespace tq
