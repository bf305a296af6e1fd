// The feed-forward of routed dense experts with a shared one, as a sequence of launches: [router (and other logits) | shared
// gate/up] as one product, routing, grouped gate/up, grouped down, shared down.  Its output is left to launch_stream_mix, which
// sums a row's weighted experts.
#pragma once

#include "dense.cuh"
#include "expert_route.cuh"
#include "internal.h"
#include "rowops.cuh"

namespace tq {

struct ExpertFf {
  const tq_dweight *front = nullptr, *gate_up = nullptr, *down = nullptr, *shared_down = nullptr;
  size_t logits = 0, logit_end = 0;      // rows of `front` that give logits, and its first row of the shared gate/up
  size_t experts = 0, identity = 0, top = 0, ff = 0, shared_ff = 0;   // experts: with weights; shared_ff 0: no shared expert
  size_t gu_rows = 0, down_rows = 0;     // rows of one expert in the stacked weights
  RouteRule rule;
  int glu = DENSE_GLU_CLAMPED;
  float limit = 0.f, alpha = 0.f, shared_limit = 0.f;   // of the clamped form
};

// Work space; every row count is the step's.
struct ExpertBuffers {
  float* logits = nullptr;               // [rows][ld_logits]
  size_t ld_logits = 0;
  Routing route;
  void* gathered = nullptr;              // [rows * top][ldx]
  void* act = nullptr;                   // [rows * top][act_ld]
  size_t act_ld = 0;
  void* shared = nullptr;                // [rows][shared_ld]
  size_t shared_ld = 0;
  float *y = nullptr, *y_shared = nullptr;   // [rows * top][width], [rows][width]
};

// x rows of `width` values, ldx apart, of `dtype`; fills y, y_rows, y_weight, n_y, y_more and, for identity experts, self of `mix`.
int launch_expert_ff(tq_ctx* ctx, const ExpertFf& f, const ExpertBuffers& b, const void* x, size_t ldx, size_t rows, size_t width, int dtype, StreamMix& mix);

}  // namespace tq
