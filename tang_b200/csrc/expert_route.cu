// Routing to dense experts (see expert_route.cuh).  Up to kErSmall pairs one CTA does everything; above, a selection kernel
// (a warp per row), a plan kernel (one CTA: offsets and jobs) and a placement kernel that also gathers the rows.
#include "expert_route.cuh"

#include "common.cuh"

namespace tq {

constexpr int kErMaxExperts = 1024, kErMaxTop = 64;
constexpr int kErThreads = 1024;
constexpr int kErSmall = 2048;      // pairs of the one-CTA form

// Selection of one row by a warp: lane l owns experts l, l + 32, ...  Lane 0 calls emit(i, expert, weight).
template <typename Emit>
__device__ __forceinline__ void choose_experts(const float* z, int experts, int top, int score, bool renorm, Emit emit) {
  const int lane = threadIdx.x & 31;
  float mx = -INFINITY, sum = 0.f;
  if (score == ROUTE_SOFTMAX) {
    for (int e = lane; e < experts; e += 32) mx = fmaxf(mx, z[e]);
    mx = warp_max(mx);
    for (int e = lane; e < experts; e += 32) sum += expf(z[e] - mx);
    sum = warp_sum(sum);
  }
  auto weight = [&](float v) { return score == ROUTE_SIGMOID ? 1.0f / (1.0f + expf(-v)) : expf(v - mx) / sum; };
  unsigned taken = 0;
  float chosen = 0.f;
  const int passes = renorm ? 2 : 1;
  for (int pass = 0; pass < passes; ++pass) {
    taken = 0;
    float total = 0.f;
    for (int i = 0; i < top; ++i) {
      float bv = -INFINITY;
      int be = -1;
      for (int j = 0, e = lane; e < experts; ++j, e += 32) {
        const float v = z[e];
        if (!((taken >> j) & 1u) && (be < 0 || v > bv)) {        // ascending: '>' keeps the lower index
          bv = v;
          be = e;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (oe >= 0 && (be < 0 || ov > bv || (!(bv > ov) && oe < be))) {
          bv = ov;
          be = oe;
        }
      }
      be = __shfl_sync(0xffffffffu, be, 0);                        // (a NaN has no order: all lanes go with lane 0)
      bv = __shfl_sync(0xffffffffu, bv, 0);
      if ((be & 31) == lane) taken |= 1u << (be >> 5);
      const float w = weight(bv);
      total += w;
      if (pass == passes - 1 && lane == 0) emit(i, be, renorm ? w / chosen : w);
    }
    chosen = total;
  }
}

// Offsets and jobs from the counts (in shared memory) of up to 1024 experts, one thread each; all threads of the CTA come here.
__device__ __forceinline__ void plan_jobs(int count, int experts, int chunk, int max_jobs, int4* jobs, int* n_jobs, int& offset) {
  __shared__ int ws[32], wj[32];
  const int e = threadIdx.x, warp = e >> 5, lane = e & 31;
  const int c = e < experts ? count : 0, nj = (c + chunk - 1) / chunk;
  int sc = c, sj = nj;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int a = __shfl_up_sync(0xffffffffu, sc, o), b = __shfl_up_sync(0xffffffffu, sj, o);
    if (lane >= o) {
      sc += a;
      sj += b;
    }
  }
  if (lane == 31) {
    ws[warp] = sc;
    wj[warp] = sj;
  }
  __syncthreads();
  int bc = 0, bj = 0;
  for (int w = 0; w < warp; ++w) {
    bc += ws[w];
    bj += wj[w];
  }
  offset = bc + sc - c;
  int at = bj + sj - nj;
  for (int i = 0; i < nj; ++i, ++at)
    if (at < max_jobs) jobs[at] = make_int4(e, offset + i * chunk, min(chunk, c - i * chunk), 0);
  if (e == blockDim.x - 1) *n_jobs = min(bj + sj, max_jobs);
}

__global__ void __launch_bounds__(kErThreads) route_small_kernel(const float* logits, size_t ld, int rows, int experts, int top, int score, bool renorm,
                                                                 int chunk, int max_jobs, Routing r, const uint8_t* x, size_t ldx, int row_vecs,
                                                                 uint8_t* gathered, size_t ldg) {
  __shared__ int counts[kErMaxExperts], offs[kErMaxExperts];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, pairs = rows * top;
  for (int e = threadIdx.x; e < experts; e += kErThreads) counts[e] = 0;
  __syncthreads();
  for (int m = warp; m < rows; m += kErThreads / 32)
    choose_experts(logits + (size_t)m * ld, experts, top, score, renorm, [&](int i, int e, float w) {
      const int p = m * top + i;
      r.expert[p] = e;
      r.weight[p] = w;
      r.rank[p] = atomicAdd(&counts[e], 1);
    });
  __syncthreads();
  int offset = 0;
  plan_jobs(threadIdx.x < (unsigned)experts ? counts[threadIdx.x] : 0, experts, chunk, max_jobs, r.jobs, r.n_jobs, offset);
  if (threadIdx.x < (unsigned)experts) {
    offs[threadIdx.x] = offset;
    r.offsets[threadIdx.x] = offset;
  }
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += kErThreads) {
    const int s = offs[r.expert[p]] + r.rank[p];      // (written above by this CTA, before the barriers)
    r.slot[p] = s;
    r.slot_row[s] = p / top;
    r.slot_weight[s] = r.weight[p];
  }
  if (gathered) {
    for (int i = threadIdx.x; i < pairs * row_vecs; i += kErThreads) {
      const int p = i / row_vecs, v = i - p * row_vecs;
      const int s = offs[r.expert[p]] + r.rank[p];
      *reinterpret_cast<uint4*>(gathered + (size_t)s * ldg + 16 * (size_t)v) = *reinterpret_cast<const uint4*>(x + (size_t)(p / top) * ldx + 16 * (size_t)v);
    }
  }
}

__global__ void __launch_bounds__(256) route_choose_kernel(const float* logits, size_t ld, int rows, int experts, int top, int score, bool renorm, Routing r) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (m >= rows) return;
  choose_experts(logits + (size_t)m * ld, experts, top, score, renorm, [&](int i, int e, float w) {
    const size_t p = (size_t)m * top + i;
    r.expert[p] = e;
    r.weight[p] = w;
    r.rank[p] = atomicAdd(&r.counts[e], 1);
  });
}

__global__ void __launch_bounds__(kErThreads) route_plan_kernel(int experts, int chunk, int max_jobs, Routing r) {
  pdl_wait();
  pdl_launch_dependents();
  const bool mine = threadIdx.x < (unsigned)experts;
  const int count = mine ? r.counts[threadIdx.x] : 0;
  int offset = 0;
  plan_jobs(count, experts, chunk, max_jobs, r.jobs, r.n_jobs, offset);
  if (mine) {
    r.offsets[threadIdx.x] = offset;
    r.counts[threadIdx.x] = 0;
  }
}

// One CTA per pair.
__global__ void __launch_bounds__(128) route_place_kernel(int top, Routing r, const uint8_t* x, size_t ldx, int row_vecs, uint8_t* gathered, size_t ldg) {
  pdl_wait();
  pdl_launch_dependents();
  const int p = blockIdx.x;
  const int s = r.offsets[r.expert[p]] + r.rank[p];
  if (threadIdx.x == 0) {
    r.slot[p] = s;
    r.slot_row[s] = p / top;
    r.slot_weight[s] = r.weight[p];
  }
  if (gathered)
    for (int v = threadIdx.x; v < row_vecs; v += 128)
      *reinterpret_cast<uint4*>(gathered + (size_t)s * ldg + 16 * (size_t)v) = *reinterpret_cast<const uint4*>(x + (size_t)(p / top) * ldx + 16 * (size_t)v);
}

size_t route_max_jobs(size_t pairs, size_t experts, size_t chunk) {
  const size_t n = experts + pairs / chunk;
  return n < pairs ? n : pairs;
}

int launch_route(tq_ctx* ctx, const float* logits, size_t ld, size_t rows, size_t experts, size_t top, int score, bool renorm, size_t chunk,
                 const Routing& r, const void* x, size_t ldx_bytes, size_t row_bytes, void* gathered, size_t ldg_bytes) {
  TQ_REQUIRE(ctx, experts > 0 && experts <= kErMaxExperts && top > 0 && top <= experts && top <= kErMaxTop, "routing: 1..%d experts, at most %d of them per row",
             kErMaxExperts, kErMaxTop);
  TQ_REQUIRE(ctx, chunk > 0 && rows * top < (1ull << 31), "routing: bad sizes");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, !gathered || (row_bytes % 16 == 0 && ldx_bytes % 16 == 0 && ldg_bytes % 16 == 0), "routing: gathered rows must be 16-byte aligned");
  const int pairs = (int)(rows * top), mj = (int)route_max_jobs(pairs, experts, chunk), vecs = (int)(row_bytes / 16);
  const uint8_t* xb = static_cast<const uint8_t*>(x);
  uint8_t* gb = static_cast<uint8_t*>(gathered);
  if (pairs <= (gathered ? 64 : kErSmall)) {
    TQ_CUDA(ctx, launch_k(ctx, route_small_kernel, dim3(1), dim3(kErThreads), 0, logits, ld, (int)rows, (int)experts, (int)top, score, renorm, (int)chunk, mj,
                          r, xb, ldx_bytes, vecs, gb, ldg_bytes));
    return TQ_OK;
  }
  TQ_CUDA(ctx, launch_k(ctx, route_choose_kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, logits, ld, (int)rows, (int)experts, (int)top, score, renorm, r));
  TQ_CUDA(ctx, launch_k(ctx, route_plan_kernel, dim3(1), dim3(kErThreads), 0, (int)experts, (int)chunk, mj, r));
  TQ_CUDA(ctx, launch_k(ctx, route_place_kernel, dim3((unsigned)pairs), dim3(128), 0, (int)top, r, xb, ldx_bytes, vecs, gb, ldg_bytes));
  return TQ_OK;
}

}  // namespace tq

using namespace tq;

extern "C" int tq_route(tq_ctx* ctx, const float* logits_dev, size_t rows, size_t experts, size_t top, int score, int renorm, size_t chunk,
                        int* expert_dev, float* weight_dev, int* slot_dev, int* slot_row_dev, int* jobs_dev, int* n_jobs_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, score == ROUTE_SIGMOID || score == ROUTE_SOFTMAX, "tq_route: unknown score");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, logits_dev && expert_dev && weight_dev && slot_dev && slot_row_dev && jobs_dev && n_jobs_dev, "tq_route: null pointer");
  const size_t pairs = rows * top;
  if (int st = ensure_scratch(ctx, (pairs * 2 + 2 * kErMaxExperts) * sizeof(int))) return st;
  Routing r;
  r.expert = expert_dev;
  r.weight = weight_dev;
  r.slot = slot_dev;
  r.slot_row = slot_row_dev;
  r.jobs = reinterpret_cast<int4*>(jobs_dev);
  r.n_jobs = n_jobs_dev;
  r.rank = static_cast<int*>(ctx->scratch);
  r.slot_weight = reinterpret_cast<float*>(r.rank + pairs);
  r.counts = r.rank + 2 * pairs;
  r.offsets = r.counts + kErMaxExperts;
  TQ_CUDA(ctx, cudaMemsetAsync(r.counts, 0, kErMaxExperts * sizeof(int), ctx->stream));
  return launch_route(ctx, logits_dev, experts, rows, experts, top, score, renorm != 0, chunk, r, nullptr, 0, 0, nullptr, 0);
}
