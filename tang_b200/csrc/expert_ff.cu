// Feed-forward of routed dense experts (see expert_ff.cuh).
#include "expert_ff.cuh"

namespace tq {

int launch_expert_ff(tq_ctx* ctx, const ExpertFf& f, const ExpertBuffers& b, const void* x, size_t ldx, size_t rows, size_t width, int dtype, StreamMix& mix) {
  const int f32 = dtype == TQ_F32;
  const size_t es = dtype_size(dtype), pairs = rows * f.top, all = f.experts + f.identity;
  DenseInput in;
  in.x = x;
  in.ldx = ldx;
  DenseEpilogue e;
  dense_section(e, f.logit_end, f.logits, DENSE_ROW, 1, b.logits, b.ld_logits);
  if (f.shared_ff) dense_section(e, f.front->rpad, f.shared_ff, DENSE_GLU, f32, b.shared, b.shared_ld);
  e.glu = f.glu;
  e.glu_limit = f.shared_limit;
  e.glu_alpha = f.alpha;
  if (int st = launch_dense(ctx, f.front, in, rows, e)) return st;
  DenseGroups g;
  g.jobs = b.route.jobs;
  g.n_jobs = b.route.n_jobs;
  g.chunk = dense_group_chunk(dtype, f.gate_up->kpad > f.down->kpad ? f.gate_up->kpad : f.down->kpad, pairs * f.experts / all + 1, f.experts);
  g.max_jobs = (int)route_max_jobs(pairs, f.experts, g.chunk);
  // the tcgen05 kernel copies boxes of consecutive rows, the others follow the slots' row numbers
  const bool gather = !f32 && g.chunk > 8;
  if (int st = launch_route(ctx, b.logits, b.ld_logits, rows, all, f.top, f.rule, g.chunk, b.route, x, ldx * es, (width + 7) / 8 * 8 * es, gather ? b.gathered : nullptr,
                            ldx * es))
    return st;
  DenseEpilogue u;
  dense_section(u, f.gu_rows, f.ff, DENSE_GLU, f32, b.act, b.act_ld);
  u.glu = f.glu;
  u.glu_limit = f.limit;
  u.glu_alpha = f.alpha;
  g.group_rows = f.gu_rows;
  g.x_rows = gather ? nullptr : b.route.slot_row;
  if (int st = launch_dense_grouped(ctx, f.gate_up, gather ? b.gathered : x, ldx, pairs, g, u)) return st;
  DenseEpilogue d;
  dense_section(d, f.down_rows, width, DENSE_ROW, 1, b.y, width);
  g.group_rows = f.down_rows;
  g.x_rows = nullptr;
  if (int st = launch_dense_grouped(ctx, f.down, b.act, b.act_ld, pairs, g, d)) return st;
  if (f.shared_ff) {
    DenseInput s;
    s.x = b.shared;
    s.ldx = b.shared_ld;
    DenseEpilogue y;
    dense_section(y, f.shared_down->rpad, width, DENSE_ROW, 1, b.y_shared, width);
    if (int st = launch_dense(ctx, f.shared_down, s, rows, y)) return st;
    mix.y_more = b.y_shared;
  }
  mix.y = b.y;
  mix.y_rows = b.route.slot;
  mix.y_weight = b.route.weight;
  mix.n_y = (int)f.top;
  if (f.identity) mix.self = x;
  return TQ_OK;
}

}  // namespace tq
