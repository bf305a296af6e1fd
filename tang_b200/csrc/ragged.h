// A step's rows: the next tokens of several sequences, packed (csrc/ops.cu, embedding_pos_kernel leaves positions and cache rows).
#pragma once

#include <stddef.h>

#include "internal.h"

namespace tq {

struct RaggedBatch {
  int n_seqs = 0, rows = 0, max_q = 1;   // rows in total; the longest sequence's rows
  int max_len = 0;                       // bounds every position + 1
  const int* seq_rows = nullptr;         // [n_seqs + 1] first row of each sequence; null: one row each
  const int* row_pos = nullptr;          // [rows] position of each row
  const int* cache_row = nullptr;        // [rows] its cache row (slot * max_seq + position); negative: the row is skipped
  size_t cache_rows = 0;                 // rows of the cache: nothing at or beyond is read
};

// x rows = table rows (ld_table elements apart) of the tokens, plus pos_table rows of their positions unless it is null; every
// row's position and cache row are left for the kernels that follow.
int launch_embedding_pos(tq_ctx* ctx, const void* table, size_t ld_table, const void* pos_table, int dt, const int* ids, const int* seq_rows,
                         const int* starts, const int* slots, int n_seqs, size_t rows, int dim, int vocab, int n_pos, int max_seq,
                         int n_slots, float* out, int* row_pos, int* cache_row);

}  // namespace tq
