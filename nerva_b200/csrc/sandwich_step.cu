// Layers of sandwich blocks (a norm in front of and a norm behind each sublayer,
// x += norm1b(mixer(norm1(x))), x += norm2b(mlp(norm2(x)))) for the session's two step functions.  The
// plan, the weights and the cache are those of parallel_step.cu; mixers are attention or a state space.
//
// What a sublayer returns is normalised as a whole before it joins the stream, so it stays pending and the
// next norm adds it.  Decode step, per layer: norms + input projection -> mixer -> output projection ->
// norms + gate/up -> down: five launches, for either mixer (a state space's grouped norm is the prologue of
// its output projection).  Block step: the same with the norms as launches of their own.
#include <algorithm>

#include "common.cuh"
#include "session.h"

namespace nb {
namespace {

typedef NervaCudaHfDecodeSequenceSession Session;

const uint16_t *step_vector(const ParallelPlan &plan, const ParallelRun &run) {
  return plan.loop_vectors + static_cast<uint64_t>(run.step) * plan.width_pad;
}

StateSpaceParams layer_state_space(const Session *s, const ParallelLayerPlan &l, const ParallelRun &run) {
  const LayerLayout &L = s->layout.layers[run.layer];
  const uint16_t *arena = s->weights->arena;
  StateSpaceParams p{};
  p.s = l.space;
  p.in_stride = l.qkv_pad;
  p.out_stride = l.attn_pad;
  p.conv = arena + L.conv;
  p.conv_bias = arena + L.conv_bias;
  p.step_bias = arena + L.step_bias;
  p.a_log = arena + L.a_log;
  p.skip = arena + L.skip;
  p.state_offset = run.state_offset;
  p.history_offset = run.history_offset;
  p.f32 = s->parallel->f32 ? 1u : 0u;
  p.pdl = s->use_pdl ? 1u : 0u;
  return p;
}

ParallelProjectionParams matrix(const uint16_t *w, uint32_t rows, uint32_t cols, float *out) {
  ParallelProjectionParams p{};
  p.w0 = w;
  p.rows0 = rows;
  p.cols0 = cols;
  p.out_f32 = out;
  return p;
}
ParallelProjectionParams gate_up(const ParallelPlan &plan, const ParallelLayerPlan &l, void *out) {
  ParallelProjectionParams p{};
  p.w1 = l.w_in + static_cast<uint64_t>(l.qkv_pad) * plan.width_pad;
  p.rows1 = 2u * l.ff_pad;
  p.cols0 = plan.width_pad;
  p.activation = plan.activation;
  p.norm = l.norm_mlp;
  p.out_act = out;
  return p;
}

// One token: the stream with its pending output, and the projections that read or feed it.
struct StepBuilder {
  Session *s;
  ResidualStream stream;
  uint64_t launches = 0;

  const ParallelPlan &plan() const { return *s->parallel; }
  float *other() const { return stream.h == s->h_a ? s->h_b : s->h_a; }

  // kSandwichIn, kSandwichGate and kSandwichJoin: the pending output joins the stream on the way.
  cudaError_t behind_norm(uint32_t kind, ParallelProjectionParams p) {
    p.h = stream.h;
    p.pending = stream.pending;
    p.after = stream.after;
    p.h_out = other();
    p.layer_norm = plan().layer_norm;
    p.eps = s->rms_eps;
    p.width = plan().width;
    p.pdl = s->use_pdl ? 1u : 0u;
    p.error_word = s->device_error;
    stream.pending = nullptr;
    if (!plan().f32 && parallel_stream_eligible(kind, p, s->sm_count)) {
      if (p.pending != nullptr && kind != kSandwichJoin) stream.h = p.h_out;
      launches += 1;
      return launch_parallel_projection(s->stream, kind, p, s->sm_count);
    }
    StreamNormParams norm = layer_stream_norm(s, stream.h, p.norm, s->x_scratch);
    norm.pending = p.pending;
    norm.after = p.after;
    norm.first = p.first;
    launches += 2;
    const cudaError_t err = launch_stream_norm(s->stream, norm, plan().f32, 1, p.pdl != 0);
    p.x0 = s->x_scratch;
    return err != cudaSuccess ? err : launch_parallel_projection_plain(s->stream, kParallelIn, p, 1, plan().f32);
  }

  // A sublayer's output projection: pending from here on, with `after` as its norm.
  cudaError_t output(ParallelProjectionParams p, const uint16_t *after) {
    p.pdl = s->use_pdl ? 1u : 0u;
    p.error_word = s->device_error;
    stream.pending = p.out_f32;
    stream.after = after;
    launches += 1;
    if (!plan().f32 && parallel_stream_eligible(kSandwichOut, p, s->sm_count))
      return launch_parallel_projection(s->stream, kSandwichOut, p, s->sm_count);
    return launch_parallel_projection_plain(s->stream, kParallelIn, p, 1, plan().f32);
  }

  cudaError_t state_space(const ParallelLayerPlan &l, const ParallelRun &run) {
    StateSpaceParams p = layer_state_space(s, l, run);
    p.in = s->qkv;
    p.out = s->mixed;
    p.cursor = s->device_cursor;
    p.max_context = s->max_context;
    p.recurrent = s->recurrent;
    launches += 1;
    return launch_state_space_step(s->stream, p);
  }

  cudaError_t state_space_output(const ParallelLayerPlan &l) {
    ParallelProjectionParams p = matrix(l.w_o, plan().width_pad, l.attn_pad, s->o_out);
    p.x_f32 = s->mixed;
    p.norm = l.group_norm;
    p.groups = l.space.norm_groups;
    p.width = l.attn_width;
    p.eps = s->rms_eps;
    if (!plan().f32 && parallel_stream_eligible(kSandwichOut, p, s->sm_count)) return output(p, l.norm_after);
    p.groups = 0;
    p.x0 = s->attn_bf16;
    launches += 1;
    const cudaError_t err = launch_grouped_norm(s->stream, s->mixed, l.attn_pad, l.group_norm, l.attn_width, l.space.norm_groups,
                                                s->rms_eps, s->attn_bf16, l.attn_pad, plan().f32, 1, s->use_pdl);
    return err != cudaSuccess ? err : output(p, l.norm_after);
  }
};

// A block of rows: the stream is ws.h_b, a pending output ws.h_a.
struct BlockBuilder {
  Session *s;
  const ParallelBlock &b;
  ResidualStream stream;
  uint64_t launches = 0;

  const ParallelPlan &plan() const { return *s->parallel; }
  const BlockWorkspace &ws() const { return s->weights->block_ws; }

  // The pending output joins the stream; x = the norm with `weight`, or [stream; first], or nothing.
  cudaError_t norm(const uint16_t *weight, const float *first, void *x) {
    StreamNormParams p = layer_stream_norm(s, stream.h, weight, x);
    p.pending = stream.pending;
    p.after = stream.after;
    p.first = first;
    if (p.pending == nullptr && x == nullptr) return cudaSuccess;
    stream.pending = nullptr;
    launches += 1;
    return launch_stream_norm(b.stream, p, plan().f32, b.rows, s->use_pdl);
  }

  // One matrix (out_f32), or gate/up pairs (out_act), over activations x.
  cudaError_t project(ParallelProjectionParams p, const void *x) {
    launches += 1;
    if (plan().f32) {
      p.x0 = x;
      p.pdl = s->use_pdl ? 1u : 0u;
      return launch_parallel_projection_plain(b.stream, kParallelIn, p, b.rows, true);
    }
    GemmParams g{};
    const bool pairs = p.rows1 != 0;
    g.weight = pairs ? p.w1 : p.w0;
    g.rows = pairs ? p.rows1 : p.rows0;
    g.cols = p.cols0;
    g.x = static_cast<const uint16_t *>(x);
    g.epilogue = pairs ? kEpilogueSwiglu : kEpilogueStore;
    g.activation = p.activation;
    g.row_add = p.row_add;
    g.out_f32 = p.out_f32;
    g.out_bf16 = static_cast<uint16_t *>(p.out_act);
    return parallel_block_gemm(s, b.stream, g, b.rows);
  }

  cudaError_t state_space(const ParallelLayerPlan &l, const ParallelRun &run) {
    StateSpaceParams p = layer_state_space(s, l, run);
    p.in = ws().qkv;
    p.out = ws().mixed;
    p.convolved = ws().convolved;
    p.rows = ws().attn_rows;
    p.row_count = b.rows;
    const bool block = b.one_session && b.rows > 1;
    launches += block ? 3 : 2;
    cudaError_t err = block ? launch_state_space_block(b.stream, p) : launch_state_space_step(b.stream, p);
    if (err == cudaSuccess)
      err = launch_grouped_norm(b.stream, ws().mixed, l.attn_pad, l.group_norm, l.attn_width, l.space.norm_groups, s->rms_eps,
                                ws().attn, l.attn_pad, plan().f32, b.rows, s->use_pdl);
    return err;
  }
};

}  // namespace

cudaError_t enqueue_sandwich_layers(Session *s, uint32_t splits, ResidualStream *stream, uint64_t *launches, StepProfile *prof,
                                    ProfileMark mark) {
  const ParallelPlan &plan = *s->parallel;
  StepBuilder step{s, *stream};
  cudaError_t err = cudaSuccess;
  for (size_t index = 0; err == cudaSuccess && index < plan.runs.size(); ++index) {
    const ParallelRun &run = plan.runs[index];
    const ParallelLayerPlan &l = plan.layers[run.layer];
    if (run.step >= 0 && plan.loop_input) {
      float *joined = step.other();
      ParallelProjectionParams p = matrix(plan.w_join, plan.width_pad, 2u * plan.width_pad, joined);
      p.first = s->first;
      p.row_add = step_vector(plan, run);
      err = step.behind_norm(kSandwichJoin, p);
      step.stream.h = joined;
      mark(s, prof, kBucketQkv);
    } else if (run.step >= 0) {
      // a pass vector alone: the stream changes in place, without a projection to ride on
      StreamNormParams p = layer_stream_norm(s, step.stream.h, nullptr, nullptr);
      p.pending = step.stream.pending;
      p.after = step.stream.after;
      p.step = step_vector(plan, run);
      err = launch_stream_norm(s->stream, p, plan.f32, 1, s->use_pdl);
      step.stream.pending = nullptr;
      step.launches += 1;
    }
    ParallelProjectionParams in = matrix(l.w_in, l.qkv_pad, plan.width_pad, s->qkv);
    in.norm = l.norm;
    if (err == cudaSuccess) err = step.behind_norm(kSandwichIn, in);
    mark(s, prof, kBucketQkv);
    if (err == cudaSuccess)
      err = l.state_space ? step.state_space(l, run) : enqueue_step_attention(s, l, run, splits, &step.launches);
    mark(s, prof, kBucketAttention);
    if (err == cudaSuccess) {
      if (l.state_space) {
        err = step.state_space_output(l);
      } else {
        ParallelProjectionParams out = matrix(l.w_o, plan.width_pad, l.attn_pad, s->o_out);
        out.x0 = s->attn_bf16;
        err = step.output(out, l.norm_after);
      }
    }
    mark(s, prof, kBucketO);
    if (err != cudaSuccess || l.ff_pad == 0) continue;
    err = step.behind_norm(kSandwichGate, gate_up(plan, l, s->ff_bf16));
    mark(s, prof, kBucketGateUp);
    ParallelProjectionParams down = matrix(l.w_down, plan.width_pad, l.ff_pad, s->down);
    down.x0 = s->ff_bf16;
    if (err == cudaSuccess) err = step.output(down, l.norm_mlp_after);
    mark(s, prof, kBucketDown);
  }
  *stream = step.stream;
  if (launches != nullptr) *launches += step.launches;
  return err;
}

cudaError_t enqueue_sandwich_block_layers(Session *s, const ParallelBlock &b, uint64_t *launches) {
  const ParallelPlan &plan = *s->parallel;
  const BlockWorkspace &ws = s->weights->block_ws;
  BlockBuilder block{s, b, ResidualStream{ws.h_b, nullptr, nullptr}};
  auto pending = [&](const uint16_t *after) {
    block.stream.pending = ws.h_a;
    block.stream.after = after;
  };
  cudaError_t err = cudaSuccess;
  for (size_t index = 0; err == cudaSuccess && index < plan.runs.size(); ++index) {
    const ParallelRun &run = plan.runs[index];
    const ParallelLayerPlan &l = plan.layers[run.layer];
    if (run.step >= 0 && plan.loop_input) {
      err = block.norm(nullptr, ws.first, ws.x_bf16);
      ParallelProjectionParams p = matrix(plan.w_join, plan.width_pad, 2u * plan.width_pad, ws.h_b);
      p.row_add = step_vector(plan, run);
      if (err == cudaSuccess) err = block.project(p, ws.x_bf16);
    } else if (run.step >= 0) {
      if (err == cudaSuccess) err = block.norm(nullptr, nullptr, nullptr);
      StreamNormParams p = layer_stream_norm(s, ws.h_b, nullptr, nullptr);
      p.step = step_vector(plan, run);
      if (err == cudaSuccess) err = launch_stream_norm(b.stream, p, plan.f32, b.rows, s->use_pdl);
      block.launches += 1;
    }
    if (err == cudaSuccess) err = block.norm(l.norm, nullptr, ws.x_bf16);
    if (err == cudaSuccess) err = block.project(matrix(l.w_in, l.qkv_pad, plan.width_pad, ws.qkv), ws.x_bf16);
    if (err == cudaSuccess)
      err = l.state_space ? block.state_space(l, run) : enqueue_block_attention(s, b, l, run, &block.launches);
    if (err == cudaSuccess) err = block.project(matrix(l.w_o, plan.width_pad, l.attn_pad, ws.h_a), ws.attn);
    pending(l.norm_after);
    if (l.ff_pad != 0) {
      if (err == cudaSuccess) err = block.norm(l.norm_mlp, nullptr, ws.x_bf16);
      if (err == cudaSuccess) err = block.project(gate_up(plan, l, ws.ff), ws.x_bf16);
      if (err == cudaSuccess) err = block.project(matrix(l.w_down, plan.width_pad, l.ff_pad, ws.h_a), ws.ff);
      pending(l.norm_mlp_after);
    }
    const bool last = index + 1u == plan.runs.size();
    if (err == cudaSuccess && (last || s->capture_stream != nullptr)) err = block.norm(nullptr, nullptr, nullptr);
    if (err == cudaSuccess) err = capture_block_stream(s, b, index);
  }
  if (launches != nullptr) *launches += block.launches;
  return err;
}

}  // namespace nb
