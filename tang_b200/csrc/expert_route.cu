// Routing to dense experts (see expert_route.cuh).  Up to kErSmall pairs one CTA does everything; above, a selection kernel
// (a warp per row), a plan kernel (one CTA: offsets and jobs) and a placement kernel that also gathers the rows.
#include "expert_route.cuh"

#include <type_traits>

#include "common.cuh"

namespace tq {

constexpr int kErMaxExperts = 1024, kErMaxTop = 64;
constexpr int kErThreads = 1024;
constexpr int kErSmall = 2048;      // pairs of the one-CTA form

// Selection of one row by a warp: lane l owns experts l, l + 32, ... (NR of them at most, in registers).  The lanes call
// emit(i, expert, weight) for their choices.
template <int NR, typename Emit>
__device__ __forceinline__ void choose_experts(const float* z, int experts, int top, const RouteRule& rule, Emit emit) {
  const int score = rule.score;
  const int lane = threadIdx.x & 31;
  float v[NR];
  unsigned key[NR];            // order of the values as integers; 0: taken or none
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int e = lane + 32 * j;
    v[j] = e < experts ? z[e] + (rule.bias ? rule.bias[e] : 0.f) : -INFINITY;
  }
  float mx = -INFINITY, sum = 0.f;
  if (score == ROUTE_SOFTMAX) {
#pragma unroll
    for (int j = 0; j < NR; ++j) mx = fmaxf(mx, v[j]);
    mx = warp_max(mx);
#pragma unroll
    for (int j = 0; j < NR; ++j) sum += expf(v[j] - mx);
    sum = warp_sum(sum);
  }
  auto weigh = [&](float logit) { return score == ROUTE_SIGMOID ? 1.0f / (1.0f + expf(-logit)) : expf(logit - mx) / sum; };
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int e = lane + 32 * j;
    const unsigned u = __float_as_uint(rule.correction && e < experts ? weigh(v[j]) + rule.correction[e] : v[j]);
    key[j] = e < experts ? max(u ^ ((u >> 31) ? 0xFFFFFFFFu : 0x80000000u), 1u) : 0u;
  }
  float mine[kErMaxTop / 32];  // lane l keeps choices l and l + 32
  int chosen[kErMaxTop / 32];
  float total = 0.f;
  for (int i = 0; i < top; ++i) {
    unsigned best = 0u;
    float bv = 0.f;
    int be = 0x7FFFFFFF;
#pragma unroll
    for (int j = 0; j < NR; ++j)
      if (key[j] > best) {                               // ascending: '>' keeps the lower index
        best = key[j];
        bv = v[j];
        be = lane + 32 * j;
      }
    const unsigned mxk = __reduce_max_sync(0xffffffffu, best);
    const int e = (int)__reduce_min_sync(0xffffffffu, best == mxk ? (unsigned)be : 0x7FFFFFFFu);
    bv = __shfl_sync(0xffffffffu, bv, e & 31);
#pragma unroll
    for (int j = 0; j < NR; ++j)
      if (e == lane + 32 * j) key[j] = 0u;
    const float w = weigh(bv);
    total += w;
#pragma unroll
    for (int h = 0; h < kErMaxTop / 32; ++h)
      if (i == lane + 32 * h) {
        mine[h] = w;
        chosen[h] = e;
      }
  }
#pragma unroll
  for (int h = 0; h < kErMaxTop / 32; ++h)
    if (lane + 32 * h < top) emit(lane + 32 * h, chosen[h], rule.renorm ? mine[h] / (total + 1e-20f) : mine[h]);
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

template <int NR>
__global__ void __launch_bounds__(kErThreads) route_small_kernel(const float* logits, size_t ld, int rows, int experts, int top, RouteRule rule,
                                                                 int chunk, int max_jobs, Routing r, const uint8_t* x, size_t ldx, int row_vecs,
                                                                 uint8_t* gathered, size_t ldg) {
  __shared__ int counts[32 * NR], offs[32 * NR];
  __shared__ unsigned short pe[kErSmall], pk[kErSmall];   // expert of every pair and its place among the expert's
  __shared__ float pw[kErSmall];
  const int real = experts - rule.identity;
  for (int e = threadIdx.x; e < experts; e += blockDim.x) counts[e] = 0;
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, pairs = rows * top;
  __syncthreads();
  for (int m = warp; m < rows; m += blockDim.x >> 5)
    choose_experts<NR>(logits + (size_t)m * ld, experts, top, rule, [&](int i, int e, float w) {
      const int p = m * top + i;
      pe[p] = (unsigned short)e;
      pw[p] = w;
      if (e < real) pk[p] = (unsigned short)atomicAdd(&counts[e], 1);
    });
  __syncthreads();
  int offset = 0;
  plan_jobs(threadIdx.x < (unsigned)experts ? counts[threadIdx.x] : 0, experts, chunk, max_jobs, r.jobs, r.n_jobs, offset);
  if (threadIdx.x < (unsigned)experts) offs[threadIdx.x] = offset;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int s = pe[p] < real ? offs[pe[p]] + pk[p] : -1;
    r.expert[p] = pe[p];
    r.weight[p] = pw[p];
    r.slot[p] = s;
    if (s < 0) continue;
    r.slot_row[s] = p / top;
    r.slot_weight[s] = pw[p];
  }
  if (gathered) {
    for (int i = threadIdx.x; i < pairs * row_vecs; i += blockDim.x) {
      const int p = i / row_vecs, v = i - p * row_vecs;
      if (pe[p] >= real) continue;
      const int s = offs[pe[p]] + pk[p];
      *reinterpret_cast<uint4*>(gathered + (size_t)s * ldg + 16 * (size_t)v) = *reinterpret_cast<const uint4*>(x + (size_t)(p / top) * ldx + 16 * (size_t)v);
    }
  }
}

template <int NR>
__global__ void __launch_bounds__(256) route_choose_kernel(const float* logits, size_t ld, int rows, int experts, int top, RouteRule rule, Routing r) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (m >= rows) return;
  const int real = experts - rule.identity;
  choose_experts<NR>(logits + (size_t)m * ld, experts, top, rule, [&](int i, int e, float w) {
    const size_t p = (size_t)m * top + i;
    r.expert[p] = e;
    r.weight[p] = w;
    if (e < real) r.rank[p] = atomicAdd(&r.counts[e], 1);
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
__global__ void __launch_bounds__(128) route_place_kernel(int top, int real, Routing r, const uint8_t* x, size_t ldx, int row_vecs, uint8_t* gathered, size_t ldg) {
  pdl_wait();
  pdl_launch_dependents();
  const int p = blockIdx.x;
  if (r.expert[p] >= real) {
    if (threadIdx.x == 0) r.slot[p] = -1;
    return;
  }
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

int launch_route(tq_ctx* ctx, const float* logits, size_t ld, size_t rows, size_t experts, size_t top, const RouteRule& rule, size_t chunk,
                 const Routing& r, const void* x, size_t ldx_bytes, size_t row_bytes, void* gathered, size_t ldg_bytes) {
  TQ_REQUIRE(ctx, experts > 0 && experts <= kErMaxExperts && top > 0 && top <= experts && top <= kErMaxTop, "routing: 1..%d experts, at most %d of them per row",
             kErMaxExperts, kErMaxTop);
  TQ_REQUIRE(ctx, rule.identity >= 0 && rule.identity < (int)experts, "routing: some of the experts must have weights");
  TQ_REQUIRE(ctx, chunk > 0 && rows * top < (1ull << 31), "routing: bad sizes");
  if (rows == 0) return TQ_OK;
  TQ_REQUIRE(ctx, !gathered || (row_bytes % 16 == 0 && ldx_bytes % 16 == 0 && ldg_bytes % 16 == 0), "routing: gathered rows must be 16-byte aligned");
  const int pairs = (int)(rows * top), mj = (int)route_max_jobs(pairs, experts - rule.identity, chunk), vecs = (int)(row_bytes / 16);
  const uint8_t* xb = static_cast<const uint8_t*>(x);
  uint8_t* gb = static_cast<uint8_t*>(gathered);
  auto go = [&](auto nr) -> int {
    constexpr int NR = decltype(nr)::value;
    if (pairs <= (gathered ? 64 : kErSmall)) {
      int threads = (int)(experts > 32 * rows ? experts : 32 * rows);
      threads = threads < 256 ? 256 : threads > kErThreads ? kErThreads : (threads + 31) / 32 * 32;
      TQ_CUDA(ctx, launch_k(ctx, route_small_kernel<NR>, dim3(1), dim3((unsigned)threads), 0, logits, ld, (int)rows, (int)experts, (int)top, rule,
                            (int)chunk, mj, r, xb, ldx_bytes, vecs, gb, ldg_bytes));
      return TQ_OK;
    }
    TQ_CUDA(ctx, launch_k(ctx, route_choose_kernel<NR>, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, logits, ld, (int)rows, (int)experts, (int)top, rule, r));
    TQ_CUDA(ctx, launch_k(ctx, route_plan_kernel, dim3(1), dim3(kErThreads), 0, (int)experts - rule.identity, (int)chunk, mj, r));
    TQ_CUDA(ctx, launch_k(ctx, route_place_kernel, dim3((unsigned)pairs), dim3(128), 0, (int)top, (int)experts - rule.identity, r, xb, ldx_bytes, vecs, gb, ldg_bytes));
    return TQ_OK;
  };
  if (experts <= 32) return go(std::integral_constant<int, 1>());
  if (experts <= 64) return go(std::integral_constant<int, 2>());
  if (experts <= 128) return go(std::integral_constant<int, 4>());
  if (experts <= 256) return go(std::integral_constant<int, 8>());
  return go(std::integral_constant<int, kErMaxExperts / 32>());
}

}  // namespace tq

using namespace tq;

extern "C" int tq_route_rule(tq_ctx* ctx, const float* logits_dev, size_t rows, size_t experts, size_t top, int score, int renorm,
                             const float* correction_dev, size_t identity, size_t chunk, int* expert_dev, float* weight_dev, int* slot_dev,
                             int* slot_row_dev, int* jobs_dev, int* n_jobs_dev) {
  return tq_route_biased(ctx, logits_dev, experts, rows, experts, top, score, renorm, nullptr, correction_dev, identity, chunk, expert_dev, weight_dev, slot_dev,
                         slot_row_dev, jobs_dev, n_jobs_dev);
}

extern "C" int tq_route_biased(tq_ctx* ctx, const float* logits_dev, size_t ld, size_t rows, size_t experts, size_t top, int score, int renorm, const float* bias_dev,
                               const float* correction_dev, size_t identity, size_t chunk, int* expert_dev, float* weight_dev, int* slot_dev,
                               int* slot_row_dev, int* jobs_dev, int* n_jobs_dev) {
  if (int st = bind(ctx)) return st;
  TQ_REQUIRE(ctx, (score == ROUTE_SIGMOID || score == ROUTE_SOFTMAX) && ld >= experts, "tq_route: unknown score, or rows of logits that overlap");
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
  RouteRule rule;
  rule.score = score;
  rule.renorm = renorm != 0;
  rule.bias = bias_dev;
  rule.correction = correction_dev;
  rule.identity = (int)identity;
  return launch_route(ctx, logits_dev, ld, rows, experts, top, rule, chunk, r, nullptr, 0, 0, nullptr, 0);
}

extern "C" int tq_route(tq_ctx* ctx, const float* logits_dev, size_t rows, size_t experts, size_t top, int score, int renorm, size_t chunk,
                        int* expert_dev, float* weight_dev, int* slot_dev, int* slot_row_dev, int* jobs_dev, int* n_jobs_dev) {
  return tq_route_rule(ctx, logits_dev, rows, experts, top, score, renorm, nullptr, 0, chunk, expert_dev, weight_dev, slot_dev, slot_row_dev, jobs_dev,
                       n_jobs_dev);
}
