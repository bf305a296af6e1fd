// Dense (unquantised) linear layers: weights bf16 or f32 in HBM, one weight matrix holding several projections
// stacked by rows, and an epilogue that sends every section of the rows where the next kernel reads it.
//
//   y[m, n] = sum_k x[m, k] * w[n, k]
//
// Three kernels share the epilogue description below:
//   * dgemv_kernel      1..8 activation rows, bound by the HBM stream of the weights (mma.sync on fragments loaded straight
//                       from global memory: a warp's lanes hold 16 consecutive bytes of a row, and the same permutation
//                       of k is used for the activations, so no layout change and no shared-memory pass is needed);
//   * dgemm_umma_kernel more rows: TMA -> shared memory -> tcgen05.mma, accumulators in tensor memory, persistent CTAs with
//                       two accumulators so that one tile's epilogue runs under the next tile's products;
//   * dgemm_f32_kernel  f32 weights and activations, every product and sum in f32 (no reduced-precision mode).
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>

#include "common.cuh"
#include "internal.h"

// A dense weight [rows, cols]; rows padded to 16, columns to 128 with zeros.
struct tq_dweight {
  int dtype = 0;               // TQ_BF16 or TQ_F32
  size_t rows = 0, cols = 0;   // as given by the caller
  size_t rpad = 0, kpad = 0;
  void* data = nullptr;        // [rpad][kpad]
  bool has_map = false;
  CUtensorMap map;             // bf16 only: 128-row x 64-column boxes
};

namespace tq {

constexpr int kDenseMaxSections = 5;

enum DenseOutKind : int {
  DENSE_ROW = 0,     // out[m * ld + column]
  DENSE_CACHE = 1,   // out[cache_row[m] * ld + column]; a negative cache row is skipped
  DENSE_GLU = 2,     // 16-row blocks of eight gate rows and the matching eight up rows -> eight outputs, gated (DenseEpilogue::glu)
  DENSE_RESID = 3,   // out[m * ld + column] += mult * value (f32)
  DENSE_HEADS = 4,   // row m is head m / head_rows of sequence b = m % head_rows: out[row(b) * ld + head * inner_pad + column] =
                     // value * sigmoid(gate at the same place), row(b) = head_row[b] (null: b; negative: skipped)
};

enum DenseAct : int { DENSE_LINEAR = 0, DENSE_SILU = 1 };        // on what a DENSE_ROW section stores
enum DenseGlu : int { DENSE_GLU_CLAMPED = 0, DENSE_GLU_SILU = 1 };   // clamped_glu, or silu(gate) * up

// Rows [previous row_end, row_end) of the weight.  Row r of the section (r < rows) goes to column
// (r / inner) * inner_pad + r % inner: heads of `inner` values may be spaced `inner_pad` apart.
struct DenseSection {
  int row_end = 0;             // multiple of 16
  int rows = 0;                // rows of the section that exist (the rest of the last 16-row block is padding)
  int kind = DENSE_ROW;
  int act = DENSE_LINEAR;
  int f32 = 0;                 // element type of out: f32 or bf16
  int inner = 1 << 30, inner_pad = 0;
  long long ld = 0;
  void* out = nullptr;
};

struct DenseEpilogue {
  int n = 0;
  DenseSection s[kDenseMaxSections];
  const int* cache_row = nullptr;
  float mult = 1.f;                       // DENSE_RESID
  const float* row_scale = nullptr;       // factor on the products of every activation row (before the GLU); not with K splits
  int glu = DENSE_GLU_CLAMPED;            // DENSE_GLU
  float glu_limit = 0.f, glu_alpha = 0.f; // of the clamped form
  int head_rows = 0;                      // DENSE_HEADS
  const int* head_row = nullptr;
  const void* gate = nullptr;             // of the type of out; null: 1
  long long ldg = 0;
};

// Appends a section of weight rows [previous end, end), of which `real` exist.
inline DenseSection& dense_section(DenseEpilogue& e, size_t end, size_t real, int kind, int f32, void* out, size_t ld) {
  DenseSection& s = e.s[e.n++];
  s.row_end = (int)end;
  s.rows = (int)real;
  s.kind = kind;
  s.f32 = f32;
  s.out = out;
  s.ld = (long long)ld;
  return s;
}

// Where one output feature goes; constant over the activation rows.
struct DenseDst {
  char* base;        // null: a padding row
  long long ld;      // bytes
  int kind, f32, act;
  int col, head_ld;  // DENSE_HEADS: column inside a head, elements between heads
};

__device__ __forceinline__ DenseDst dense_dst(const DenseEpilogue& e, int row) {
  DenseDst d;
  d.base = nullptr;
  d.ld = 0;
  d.kind = -1;
  d.f32 = d.act = d.col = d.head_ld = 0;
  int start = 0;
#pragma unroll
  for (int i = 0; i < kDenseMaxSections; ++i) {
    if (i < e.n && row >= start && row < e.s[i].row_end) {
      const DenseSection& s = e.s[i];
      const int r = row - start;
      const int es = s.f32 ? 4 : 2;
      d.kind = s.kind;
      d.f32 = s.f32;
      d.act = s.act;
      d.col = r;
      d.head_ld = s.inner_pad;
      d.ld = s.ld * es;
      if (s.kind == DENSE_GLU) {
        const int o = (r >> 4) * 8 + (r & 7);
        if (o < s.rows) d.base = static_cast<char*>(s.out) + (long long)o * es;
      } else if (r < s.rows) {
        d.base = static_cast<char*>(s.out) + ((long long)(r / s.inner) * s.inner_pad + r % s.inner) * es;
      }
    }
    if (i < e.n) start = e.s[i].row_end;
  }
  return d;
}

// min(gate, limit) * sigmoid(alpha * .) * (clamp(up, -limit, limit) + 1)
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g * (1.0f / (1.0f + expf(-alpha * g))) * (u + 1.0f);
}

__device__ __forceinline__ float dense_glu(const DenseEpilogue& e, float gate, float up) {
  return e.glu == DENSE_GLU_SILU ? gate / (1.0f + expf(-gate)) * up : clamped_glu(gate, up, e.glu_limit, e.glu_alpha);
}

__device__ __forceinline__ void dense_store(const DenseEpilogue& e, const DenseDst& d, int m, float v) {
  if (!d.base) return;
  long long idx = m;
  if (d.kind == DENSE_CACHE) {
    idx = e.cache_row[m];
    if (idx < 0) return;
  }
  char* p = d.base + idx * d.ld;
  if (d.kind == DENSE_HEADS) {
    const int head = m / e.head_rows, b = m - head * e.head_rows, row = e.head_row ? e.head_row[b] : b;
    if (row < 0) return;
    if (e.gate) {
      const long long at = row * e.ldg + (long long)head * d.head_ld + d.col;
      const float g = d.f32 ? static_cast<const float*>(e.gate)[at] : __bfloat162float(static_cast<const __nv_bfloat16*>(e.gate)[at]);
      v *= 1.0f / (1.0f + expf(-g));
    }
    p = d.base + row * d.ld + (long long)head * d.head_ld * (d.f32 ? 4 : 2);
  } else if (d.act == DENSE_SILU) {
    v = v / (1.0f + expf(-v));
  }
  if (d.kind == DENSE_RESID) {
    float* f = reinterpret_cast<float*>(p);
    *f = *f + e.mult * v;
  } else if (d.f32) {
    *reinterpret_cast<float*>(p) = v;
  } else {
    *reinterpret_cast<__nv_bfloat16*>(p) = __float2bfloat16_rn(v);
  }
}

// Activations of a dense linear: rows x [m][ldx] (the weight's dtype), or -- `h` set -- rms_norm of f32 rows
// h[h_rows ? h_rows[m] : m] times `gain`, formed by the GEMV itself for few rows and through xn_tmp [m][kpad] otherwise.
struct DenseInput {
  const void* x = nullptr;
  size_t ldx = 0;
  const float* h = nullptr;
  size_t ldh = 0;
  const int* h_rows = nullptr;
  const void* gain = nullptr;
  int gain_dtype = TQ_BF16;
  float eps = 0.f;
  void* xn_tmp = nullptr;
};

int launch_dense(tq_ctx* ctx, const tq_dweight* w, const DenseInput& in, size_t m, const DenseEpilogue& epi);

// Several weights of one shape stacked by rows in one handle (experts): a job multiplies rows first .. first + n - 1 of the
// activations with group g's rows g * group_rows ...  The job list is written on the device by an earlier kernel.
struct DenseGroups {
  const int4* jobs = nullptr;      // (group, first row, rows, shift); rows <= chunk; the epilogue sees row first + shift + i
  const int* n_jobs = nullptr;
  int max_jobs = 0;                // bounds *n_jobs
  int chunk = 0;                   // dense_group_chunk
  size_t group_rows = 0;           // multiple of 16
  const int* x_rows = nullptr;     // where activation row i is in x; null: row i.  Not with chunks above 8 of bf16 weights
};

// Rows per job that suit `rows` activation rows spread over n_groups, for weights with these padded columns: up to 8 the
// GEMV runs, above the tcgen05 kernel; f32 weights always take 64.
int dense_group_chunk(int dtype, size_t kpad, size_t rows, size_t n_groups);
// Rows per job where every group multiplies exactly `rows` rows.
int dense_even_chunk(int dtype, size_t kpad, size_t rows);
// The epilogue's sections describe one group's rows; its row indices are activation rows (`first` + `shift` of a job onwards).
int launch_dense_grouped(tq_ctx* ctx, const tq_dweight* w, const void* x, size_t ldx, size_t rows, const DenseGroups& groups, const DenseEpilogue& epi);

// dst = src + add over a vector of n values (host or device memory, bf16 or f32); for loading weights.
int put_vector(tq_ctx* ctx, const void* src, int src_dtype, void* dst, int dst_dtype, size_t n, float add);

// Per-head transposition for absorbed products: row-major src [heads * dim][rank] becomes, group by group,
// w[h * group_rows + c][d] = src[h * dim + d][c].
int dweight_put_head_transposed(tq_ctx* ctx, tq_dweight* w, const void* src, int src_dtype, size_t heads, size_t dim, size_t rank, size_t group_rows);

// rms_norm of rows of an f32 matrix, output row stride ld_out (csrc/ops.cu).
int launch_rms_norm_rows(tq_ctx* ctx, const float* x, size_t ldx, const int* rows, const void* gain, int gain_dtype, size_t n,
                         size_t dim, float eps, void* out, int out_dtype, size_t ld_out);

}  // namespace tq
