// Routing of activation rows to dense experts: selection from f32 router logits and the grouped layout that
// launch_dense_grouped walks.
#pragma once

#include "dense.cuh"
#include "internal.h"

namespace tq {

enum RouteScore : int { ROUTE_SIGMOID = 0, ROUTE_SOFTMAX = 1 };

// How a row's experts are chosen and weighed.  The bias is part of the logits.  Scores are sigmoid(logit), or softmax over all experts.  The `top` experts with
// the largest logits -- with a correction, the largest score + correction[expert] -- are chosen (the lower index among equals);
// weights are the scores, divided by their sum if `renorm`.  The last `identity` of the experts have no weights: their pairs
// take no slot.
struct RouteRule {
  int score = ROUTE_SIGMOID;
  bool renorm = false;
  const float* bias = nullptr;         // [experts]; null: 0
  const float* correction = nullptr;
  int identity = 0;
};

// Device arrays of a routing; pair p = row * top + i is the i-th choice of a row, and the pairs of one expert occupy
// consecutive slots.
struct Routing {
  int* expert = nullptr;      // [rows * top] chosen expert of every pair
  float* weight = nullptr;    // [rows * top] its weight
  int* rank = nullptr;        // [rows * top] place among the expert's pairs
  int* slot = nullptr;        // [rows * top] slot of every pair; -1: an identity expert
  int* slot_row = nullptr;    // [rows * top] row of every slot
  float* slot_weight = nullptr;   // [rows * top]
  int* counts = nullptr;      // [experts], zero between launches
  int* offsets = nullptr;     // [experts] first slot
  int4* jobs = nullptr;       // [route_max_jobs] (expert, first slot, rows, 0)
  int* n_jobs = nullptr;
};

// Upper bound of the number of jobs of at most `chunk` slots.
size_t route_max_jobs(size_t pairs, size_t experts, size_t chunk);

// Fills every array of `r`; when gathered is set, it also copies row slot_row[s] of x (row bytes, a multiple of 16) to row s of
// gathered.
int launch_route(tq_ctx* ctx, const float* logits, size_t ld, size_t rows, size_t experts, size_t top, const RouteRule& rule, size_t chunk,
                 const Routing& r, const void* x, size_t ldx_bytes, size_t row_bytes, void* gathered, size_t ldg_bytes);

}  // namespace tq
