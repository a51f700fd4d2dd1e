// Decoders described layer by layer, every size per layer, a range of layers run several times with the
// same weights (NervaB200ParallelModel).  This file turns the description into a plan (padded weights,
// layer runs, cache and state offsets) and enqueues the layers of parallel blocks,
// x += ls1 * attention(norm(x)) + ls2 * mlp(norm(x)), for the session's two step functions: the decode
// step (session.cu) and the block step (block_step.cu); sandwich blocks are in sandwich_step.cu.  Token
// fetch, embedding, sampler, token ring, graphs, page table and forks are the session's own.
//
// Decode step, per layer run: norm + [Q; K; V] -> attention, with norm + gate/up streaming beside it ->
// [O | down] + residual: four launches.  Block step: norm, one projection for all five input matrices, q/k preparation + cache
// append, attention, O and down with the residual add in their epilogues.
#include <math.h>

#include <algorithm>
#include <vector>

#include "common.cuh"
#include "session.h"

namespace nb {
namespace {

typedef NervaCudaHfDecodeSequenceSession Session;

uint32_t round_up(uint32_t v, uint32_t m) { return (v + m - 1u) / m * m; }

// Angle per position of every rotated pair.  Scaled (YaRN): pairs that turn more than `fast` times over
// the original length keep their frequency, pairs that turn less than `slow` times have it divided by
// `factor`, with a linear ramp over the pair index in between, and cos and sin grow by 0.1 ln(factor) + 1.
void rotary_table(const NervaB200ParallelLayer &l, std::vector<float> *out, float *magnitude) {
  const uint32_t pairs = l.rotary_dims / 2u;
  const double dims = l.rotary_dims;
  const bool scaled = l.yarn_factor != 0.0 && pairs != 0;
  double lo = 0.0, hi = 0.0;
  if (scaled) {
    auto dim_of = [&](double turns) {
      return dims * log(l.yarn_original / (2.0 * M_PI * turns)) / (2.0 * log(l.rotary_base));
    };
    lo = std::max(floor(dim_of(l.yarn_fast)), 0.0);
    hi = std::min(ceil(dim_of(l.yarn_slow)), dims - 1.0);
  }
  out->clear();
  for (uint32_t i = 0; i < pairs; ++i) {
    double f = pow(l.rotary_base, -2.0 * i / dims);
    if (scaled) {
      const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
      f = f / l.yarn_factor * ramp + f * (1.0 - ramp);
    }
    out->push_back(static_cast<float>(f));
  }
  *magnitude = scaled ? static_cast<float>(0.1 * log(l.yarn_factor) + 1.0) : 1.0f;
}

const uint16_t *arena_at(const Session *s, uint64_t offset) {
  return offset == kMissingOffset ? nullptr : s->weights->arena + offset;
}

const uint16_t *step_vector(const ParallelPlan &plan, const ParallelRun &run) {
  return run.step < 0 ? nullptr : plan.loop_vectors + static_cast<uint64_t>(run.step) * plan.width_pad;
}

// The matrices and sizes of a layer's two projection launches; activations and outputs are the caller's.
ParallelProjectionParams layer_in(const ParallelPlan &plan, const ParallelLayerPlan &l, float eps) {
  ParallelProjectionParams p{};
  p.w0 = l.w_in;
  p.rows0 = l.qkv_pad;
  p.cols0 = plan.width_pad;
  p.w1 = l.w_in + static_cast<uint64_t>(l.qkv_pad) * plan.width_pad;
  p.rows1 = 2u * l.ff_pad;
  p.norm = l.norm;
  p.width = plan.width;
  p.eps = eps;
  return p;
}
ParallelProjectionParams layer_out(const ParallelPlan &plan, const ParallelLayerPlan &l) {
  ParallelProjectionParams p{};
  p.w0 = l.w_o;
  p.rows0 = plan.width_pad;
  p.cols0 = l.attn_pad;
  if (l.ff_pad != 0) {
    p.w1 = l.w_down;
    p.rows1 = plan.width_pad;
    p.cols1 = l.ff_pad;
  }
  if (l.layer_scale) {
    p.scale0 = l.ls_attn;
    p.scale1 = l.ls_mlp;
  }
  return p;
}
// The two halves of an output launch, for shapes whose vectors do not fit one block together.
ParallelProjectionParams first_matrix(ParallelProjectionParams p) {
  p.w1 = nullptr;
  p.rows1 = p.cols1 = 0;
  return p;
}
ParallelProjectionParams second_matrix(ParallelProjectionParams p) {
  p.w0 = p.w1;
  p.rows0 = p.rows1;
  p.cols0 = p.cols1;
  p.x0 = p.x1;
  p.scale0 = p.scale1;
  p.step = nullptr;  // added by the first
  return first_matrix(p);
}
WindowAttentionParams layer_attention(const ParallelPlan &plan, const ParallelLayerPlan &l, const ParallelRun &run) {
  WindowAttentionParams p{};
  p.s = l.shape;
  p.qkv_stride = l.qkv_pad;
  p.out_stride = l.attn_pad;
  p.key_offset = run.key_offset;
  p.value_offset = run.value_offset;
  p.f32 = plan.f32 ? 1u : 0u;
  return p;
}

// Rows below which a block's attention is one query per thread block: a tile of the tensor-pipe kernel
// would be mostly empty and walk its keys alone.
constexpr uint32_t kPrefillTileMinRows = 8;

// Checks a layer's attention and fills its part of the plan; why it is refused, or null.
const char *plan_attention(const NervaB200ParallelLayer &in, bool f32, float eps, ParallelPlan *plan, ParallelLayerPlan *out) {
  ParallelLayerPlan &l = *out;
  if (in.heads == 0 || in.kv_heads == 0 || in.heads % in.kv_heads != 0 || in.qk_dim == 0 || in.v_dim == 0 ||
      in.qk_dim > 256u || in.v_dim > 256u)
    return "needs heads divisible by kv_heads and head sizes of 1 to 256";
  if (in.rotary_dims % 2u != 0 || in.rotary_dims > in.qk_dim ||
      (in.rotary_dims != 0 && !(in.rotary_base > 0.0 && in.rotary_base != 1.0)) ||
      (in.yarn_factor != 0.0 && !(in.yarn_factor > 0.0 && in.yarn_original > 0.0 && in.yarn_fast > 0.0 && in.yarn_slow > 0.0)))
    return "rotation";
  if (!(in.score_softcap >= 0.0f)) return "score soft cap";
  WindowAttentionShape &a = l.shape;
  a.heads = in.heads;
  a.kv_heads = in.kv_heads;
  a.qk_dim = in.qk_dim;
  a.v_dim = in.v_dim;
  a.qk_pad = round_up(in.qk_dim, 16);
  a.v_pad = round_up(in.v_dim, 16);
  a.window = in.window;
  a.keep_first = in.window != 0 ? in.keep_first : 0u;
  a.head_gate = in.head_gate != 0 ? 1u : 0u;
  a.softcap = in.score_softcap;
  a.rotary_pairs = in.rotary_dims / 2u;
  a.qk_norm = in.qk_norm;
  a.scale = in.score_scale;
  a.eps = eps;
  rotary_table(in, &l.frequencies, &a.rotary_magnitude);
  if (!window_attention_supported(a, f32)) return "attention shape";
  l.qkv_rows = in.heads * in.qk_dim + in.kv_heads * (in.qk_dim + in.v_dim) + (a.head_gate != 0 ? in.heads : 0u);
  plan->max_heads = std::max(plan->max_heads, in.heads);
  plan->max_v_pad = std::max(plan->max_v_pad, a.v_pad);
  return nullptr;
}

const char *plan_state_space(const NervaB200ParallelLayer &in, float eps, ParallelPlan *plan, ParallelLayerPlan *l) {
  StateSpaceShape &space = l->space;
  space.heads = in.heads;
  space.v_dim = in.v_dim;
  space.state = in.state_size;
  space.groups = in.state_groups;
  space.taps = in.conv_taps;
  space.norm_groups = in.norm_groups;
  space.eps = eps;
  if (!state_space_supported(space))
    return "needs heads divisible by state groups, a state of 1 to 256, 1 to 16 convolution taps and norm groups of equal size";
  l->state_space = true;
  l->qkv_rows = space.in_rows();
  plan->max_conv_width = std::max(plan->max_conv_width, space.conv_width());
  return nullptr;
}

}  // namespace

cudaError_t parallel_block_gemm(NervaCudaHfDecodeSequenceSession *s, cudaStream_t stream, GemmParams g, uint32_t tokens) {
  const BlockWorkspace &ws = s->weights->block_ws;
  g.tokens = tokens;
  g.workspace = ws.gemm_workspace;
  g.error_word = s->device_error;
  g.pdl = s->use_pdl ? 1u : 0u;
  return launch_gemm_tc(stream, g, s->sm_count);
}

StreamNormParams layer_stream_norm(const NervaCudaHfDecodeSequenceSession *s, float *h, const uint16_t *weight, void *x) {
  const ParallelPlan &plan = *s->parallel;
  StreamNormParams p{};
  p.h = h;
  p.norm = weight;
  p.layer_norm = plan.layer_norm;
  p.eps = s->rms_eps;
  p.width = plan.width;
  p.padded = plan.width_pad;
  p.x = x;
  return p;
}

cudaError_t capture_block_stream(NervaCudaHfDecodeSequenceSession *s, const ParallelBlock &b, size_t run) {
  if (s->capture_stream == nullptr || !b.one_session || b.capture_row >= s->capture_rows) return cudaSuccess;
  const ParallelPlan &plan = *s->parallel;
  const uint32_t rows = std::min(b.rows, s->capture_rows - b.capture_row);
  return cudaMemcpy2DAsync(s->capture_stream + (run * s->capture_rows + b.capture_row) * plan.width, plan.width * sizeof(float),
                           s->weights->block_ws.h_b, plan.width_pad * sizeof(float), plan.width * sizeof(float), rows,
                           cudaMemcpyDeviceToHost, b.stream);
}

std::shared_ptr<ParallelPlan> make_parallel_plan(const NervaB200ParallelModel &m, uint32_t width, uint32_t vocab, float eps) {
  auto refuse = [](const char *why) {
    set_last_error(std::string("model not supported: ") + why);
    return std::shared_ptr<ParallelPlan>();
  };
  auto plan = std::make_shared<ParallelPlan>();
  if (m.compute != NERVA_DTYPE_BF16 && m.compute != NERVA_DTYPE_F32) return refuse("compute type");
  plan->f32 = m.compute == NERVA_DTYPE_F32;
  plan->width = width;
  plan->width_pad = round_up(width, 64);
  plan->vocab = vocab;
  plan->embedding_scale = m.embedding_scale;
  plan->logit_scale = m.logit_scale;
  plan->softcap = m.logit_softcap;
  plan->loop_times = m.loop_times;
  if (m.block > NERVA_B200_BLOCK_SANDWICH || m.norm > NERVA_B200_NORM_LAYER || m.activation > NERVA_B200_ACTIVATION_GELU_TANH)
    return refuse("block, norm or activation");
  plan->sandwich = m.block == NERVA_B200_BLOCK_SANDWICH;
  plan->layer_norm = m.norm == NERVA_B200_NORM_LAYER ? 1u : 0u;
  plan->activation = m.activation == NERVA_B200_ACTIVATION_GELU_TANH ? kActivationGeluTanh : kActivationSilu;
  plan->loop_input = m.loop_input != 0 && m.loop_times != 0;
  if (!plan->sandwich && (plan->layer_norm != 0 || plan->loop_input))
    return refuse("layer norms and a loop's input projection come with sandwich blocks");
  if (m.loop_times != 0 && (m.loop_start >= m.loop_stop || m.loop_stop > m.layer_count)) return refuse("loop range");
  for (uint32_t i = 0; i < m.layer_count; ++i) {
    const NervaB200ParallelLayer &in = m.layers[i];
    ParallelLayerPlan l;
    const bool space = in.mixer == NERVA_B200_MIXER_STATE_SPACE;
    if (in.mixer > NERVA_B200_MIXER_STATE_SPACE || (space && !plan->sandwich)) return refuse("mixer");
    if (plan->sandwich && in.layer_scale != 0) return refuse("layer scales come with parallel blocks");
    const char *why = space ? plan_state_space(in, eps, plan.get(), &l) : plan_attention(in, plan->f32, eps, plan.get(), &l);
    if (why != nullptr) return refuse(why);
    l.intermediate = in.intermediate;
    l.ff_pad = round_up(in.intermediate, 64);
    l.qkv_pad = round_up(l.qkv_rows, 64);
    l.attn_width = in.heads * in.v_dim;
    l.attn_pad = round_up(l.attn_width, 64);
    l.layer_scale = in.layer_scale != 0;
    plan->max_qkv_pad = std::max(plan->max_qkv_pad, l.qkv_pad);
    plan->max_attn_pad = std::max(plan->max_attn_pad, l.attn_pad);
    plan->max_ff_pad = std::max(plan->max_ff_pad, l.ff_pad);
    if (space) plan->max_space_pad = std::max(plan->max_space_pad, l.attn_pad);
    plan->layers.push_back(l);
  }
  auto run = [&](uint32_t layer, int32_t step) {
    ParallelRun r;
    r.layer = layer;
    r.step = step;
    plan->runs.push_back(r);
  };
  const uint32_t start = m.loop_times != 0 ? m.loop_start : m.layer_count;
  for (uint32_t i = 0; i < start; ++i) run(i, -1);
  for (uint32_t t = 0; t < m.loop_times; ++t)
    for (uint32_t i = start; i < m.loop_stop; ++i) run(i, i == start ? static_cast<int32_t>(t) : -1);
  for (uint32_t i = m.loop_times != 0 ? m.loop_stop : start; i < m.layer_count; ++i) run(i, -1);
  return plan;
}

void place_parallel_cache(ParallelPlan *plan, uint32_t pages) {
  const uint64_t tokens = static_cast<uint64_t>(pages) * NERVA_KV_CACHE_BLOCK_TOKENS;
  plan->key_elems = plan->value_elems = plan->recurrent_floats = 0;
  for (ParallelRun &r : plan->runs) {
    if (plan->layers[r.layer].state_space) {
      const StateSpaceShape &space = plan->layers[r.layer].space;
      auto place = [&](uint64_t floats) {  // 16-byte pieces
        const uint64_t at = plan->recurrent_floats;
        plan->recurrent_floats += (floats + 3u) / 4u * 4u;
        return at;
      };
      r.state_offset = place(static_cast<uint64_t>(space.heads) * space.state * space.v_dim);
      r.history_offset = place(static_cast<uint64_t>(space.taps) * space.channels());
      continue;
    }
    const WindowAttentionShape &a = plan->layers[r.layer].shape;
    r.key_offset = plan->key_elems;
    r.value_offset = plan->value_elems;
    plan->key_elems += tokens * a.kv_heads * a.qk_pad;
    plan->value_elems += tokens * a.kv_heads * a.v_pad;
  }
}

cudaError_t pack_parallel_weights(Session *s) {
  const ParallelPlan &plan = *s->parallel;
  const uint32_t width = plan.width, pad = plan.width_pad;
  cudaError_t err = cudaSuccess;
  auto clear = [&](void *p, uint64_t bytes) {
    if (err == cudaSuccess && bytes != 0) err = cudaMemsetAsync(p, 0, bytes, s->stream);
  };
  auto pack = [&](uint64_t offset, uint32_t rows, uint32_t cols, uint16_t *dst, uint32_t dst_cols, uint32_t step,
                  uint32_t first) {
    if (err == cudaSuccess && rows != 0)
      err = launch_pack_rows(s->stream, arena_at(s, offset), rows, cols, dst, dst_cols, step, first);
  };
  clear(plan.loop_vectors, static_cast<uint64_t>(std::max(plan.loop_times, 1u)) * pad * 2u);
  pack(s->layout.loop_vectors, plan.loop_times, width, plan.loop_vectors, pad, 1, 0);
  if (plan.loop_input) {
    // [out][stream | embedding], each half padded: as rows of one half, the halves of a matrix row follow each other
    clear(plan.w_join, 2ull * pad * pad * 2u);
    pack(s->layout.loop_input, 2u * width, width, plan.w_join, pad, 1, 0);
  }
  for (size_t i = 0; i < plan.layers.size(); ++i) {
    const ParallelLayerPlan &l = plan.layers[i];
    const LayerLayout &L = s->layout.layers[i];
    const WindowAttentionShape &a = l.shape;
    clear(l.w_in, (l.qkv_pad + 2ull * l.ff_pad) * pad * 2u);
    clear(l.w_o, static_cast<uint64_t>(pad) * l.attn_pad * 2u);
    clear(l.w_down, static_cast<uint64_t>(pad) * std::max(l.ff_pad, 8u) * 2u);
    clear(l.norm, pad * 2u);
    clear(l.ls_attn, pad * 2u);
    clear(l.ls_mlp, pad * 2u);
    if (l.state_space) {
      pack(L.w_space, l.qkv_rows, width, l.w_in, pad, 1, 0);
      clear(l.group_norm, l.attn_pad * 2u);
      pack(L.group_norm, 1, l.attn_width, l.group_norm, l.attn_pad, 1, 0);
    } else {
      const uint32_t q_rows = a.heads * a.qk_dim, k_rows = a.kv_heads * a.qk_dim, v_rows = a.kv_heads * a.v_dim;
      pack(L.w_q, q_rows, width, l.w_in, pad, 1, 0);
      pack(L.w_k, k_rows, width, l.w_in, pad, 1, q_rows);
      pack(L.w_v, v_rows, width, l.w_in, pad, 1, q_rows + k_rows);
      if (a.head_gate != 0) pack(L.w_head_gate, a.heads, width, l.w_in, pad, 1, q_rows + k_rows + v_rows);
    }
    if (plan.sandwich) {
      clear(l.norm_after, pad * 2u);
      clear(l.norm_mlp, pad * 2u);
      clear(l.norm_mlp_after, pad * 2u);
      pack(L.norm_after, 1, width, l.norm_after, pad, 1, 0);
      if (l.intermediate != 0) {
        pack(L.rms_mlp, 1, width, l.norm_mlp, pad, 1, 0);
        pack(L.norm_mlp_after, 1, width, l.norm_mlp_after, pad, 1, 0);
      }
    }
    pack(L.w_o, width, l.attn_width, l.w_o, l.attn_pad, 1, 0);
    pack(L.rms_attn, 1, width, l.norm, pad, 1, 0);
    if (l.intermediate != 0) {
      pack(L.w_gate, l.intermediate, width, l.w_in, pad, 2, l.qkv_pad);
      pack(L.w_up, l.intermediate, width, l.w_in, pad, 2, l.qkv_pad + 1u);
      pack(L.w_down, width, l.intermediate, l.w_down, l.ff_pad, 1, 0);
    }
    if (l.layer_scale) {
      pack(L.ls_attn, 1, width, l.ls_attn, pad, 1, 0);
      if (l.intermediate != 0) pack(L.ls_mlp, 1, width, l.ls_mlp, pad, 1, 0);
    }
    if (err == cudaSuccess && !l.frequencies.empty())
      err = cudaMemcpyAsync(l.frequency, l.frequencies.data(), l.frequencies.size() * sizeof(float),
                            cudaMemcpyHostToDevice, s->stream);
    s->parallel->layers[i].shape.frequency = l.frequency;
  }
  clear(plan.final_norm, pad * 2u);
  clear(plan.head, static_cast<uint64_t>(plan.vocab) * pad * 2u);
  pack(s->layout.final_norm, 1, width, plan.final_norm, pad, 1, 0);
  pack(s->layout.lm_head, plan.vocab, width, plan.head, pad, 1, 0);
  return err;
}

uint32_t parallel_attention_splits(const ParallelPlan &plan, uint32_t target_context) {
  uint32_t most = 1;
  for (const ParallelLayerPlan &l : plan.layers) {
    if (!l.state_space) most = std::max(most, window_attention_splits(target_context, l.shape.window, l.shape.keep_first));
  }
  return most;
}

cudaError_t enqueue_step_attention(Session *s, const ParallelLayerPlan &l, const ParallelRun &run, uint32_t splits,
                                   uint64_t *launches) {
  WindowAttentionParams a = layer_attention(*s->parallel, l, run);
  a.pdl = s->use_pdl ? 1u : 0u;
  a.qkv = s->qkv;
  a.out = s->attn_bf16;
  a.splits = std::min(splits, window_attention_splits(UINT32_MAX / 2u, l.shape.window, l.shape.keep_first));
  a.partial_acc = s->partial_acc;
  a.partial_m = s->partial_m;
  a.partial_l = s->partial_l;
  a.tickets = s->attn_tickets;
  a.cursor = s->device_cursor;
  a.max_context = s->max_context;
  a.page_count = s->kv_pages;
  a.keys = s->kv_keys;
  a.values = s->kv_values;
  a.page_table = s->page_table;
  a.error_word = s->device_error;
  *launches += 1;
  return launch_window_attention(s->stream, a);
}

cudaError_t enqueue_block_attention(Session *s, const ParallelBlock &b, const ParallelLayerPlan &l, const ParallelRun &run,
                                    uint64_t *launches) {
  const ParallelPlan &plan = *s->parallel;
  const BlockWorkspace &ws = s->weights->block_ws;
  WindowAttentionParams a = layer_attention(plan, l, run);
  a.pdl = s->use_pdl ? 1u : 0u;
  a.qkv = ws.qkv;
  a.out = ws.attn;
  a.partial_acc = ws.partial_acc;
  a.partial_m = ws.partial_m;
  a.partial_l = ws.partial_l;
  a.tickets = ws.attn_tickets;
  a.rows = ws.attn_rows;
  a.row_count = b.rows;
  *launches += 2;
  const cudaError_t err = launch_window_publish(b.stream, a);
  if (err != cudaSuccess) return err;
  if (b.one_session && b.rows >= kPrefillTileMinRows && !plan.f32) return launch_window_prefill(b.stream, a);
  a.splits = window_rows_splits(l.shape, b.rows, b.longest, s->sm_count);
  return launch_window_attention(b.stream, a);
}

cudaError_t enqueue_parallel_layers(Session *s, uint32_t splits, ResidualStream *stream, uint64_t *launches, StepProfile *prof,
                                    ProfileMark mark) {
  const ParallelPlan &plan = *s->parallel;
  if (plan.sandwich) return enqueue_sandwich_layers(s, splits, stream, launches, prof, mark);
  const uint32_t pdl = s->use_pdl ? 1u : 0u;
  uint64_t n = 0;
  cudaError_t err = cudaSuccess;
  for (const ParallelRun &run : plan.runs) {
    const ParallelLayerPlan &l = plan.layers[run.layer];
    const uint16_t *step = step_vector(plan, run);
    ParallelProjectionParams in = layer_in(plan, l, s->rms_eps);
    in.pdl = pdl;
    in.error_word = s->device_error;
    in.h = s->h_b;
    in.step = step;
    in.out_f32 = s->qkv;
    in.out_act = s->ff_bf16;
    in.activation = plan.activation;
    ParallelProjectionParams out = layer_out(plan, l);
    out.pdl = pdl;
    out.error_word = s->device_error;
    out.h = out.h_out = s->h_b;
    out.step = step;
    out.x0 = s->attn_bf16;
    out.x1 = s->ff_bf16;
    const bool gate = l.ff_pad != 0;
    const bool streamed = !plan.f32 && parallel_stream_eligible(kParallelIn, in, s->sm_count) &&
                          (!gate || parallel_stream_eligible(kParallelGate, in, s->sm_count)) &&
                          parallel_stream_eligible(kParallelOut, first_matrix(out), s->sm_count) &&
                          (out.rows1 == 0 || parallel_stream_eligible(kParallelOut, second_matrix(out), s->sm_count));
    if (streamed) {
      err = launch_parallel_projection(s->stream, kParallelIn, in, s->sm_count);
      n += 1;
    } else {
      StreamNormParams norm = layer_stream_norm(s, s->h_b, l.norm, s->x_scratch);
      norm.step = step;
      err = launch_stream_norm(s->stream, norm, plan.f32, 1, pdl != 0);
      out.step = nullptr;  // it is part of the stream now
      in.x0 = s->x_scratch;
      if (err == cudaSuccess) err = launch_parallel_projection_plain(s->stream, kParallelIn, in, 1, plan.f32);
      n += 2;
    }
    mark(s, prof, kBucketQkv);
    if (err != cudaSuccess) break;

    err = enqueue_step_attention(s, l, run, splits, &n);
    mark(s, prof, kBucketAttention);
    if (err != cudaSuccess) break;
    if (streamed && gate) {
      err = launch_parallel_projection(s->stream, kParallelGate, in, s->sm_count);
      n += 1;
      mark(s, prof, kBucketGateUp);
      if (err != cudaSuccess) break;
    }

    if (!streamed) {
      err = launch_parallel_projection_plain(s->stream, kParallelOut, out, 1, plan.f32);
      n += 1;
    } else if (parallel_stream_eligible(kParallelOut, out, s->sm_count)) {
      err = launch_parallel_projection(s->stream, kParallelOut, out, s->sm_count);
      n += 1;
    } else {
      // both activation vectors do not fit beside the weight ring: one matrix after the other
      err = launch_parallel_projection(s->stream, kParallelOut, first_matrix(out), s->sm_count);
      if (err == cudaSuccess) err = launch_parallel_projection(s->stream, kParallelOut, second_matrix(out), s->sm_count);
      n += 2;
    }
    mark(s, prof, kBucketDown);
    if (err != cudaSuccess) break;
  }
  if (launches != nullptr) *launches += n;
  return err;
}

cudaError_t enqueue_parallel_head(Session *s, const ResidualStream &stream, uint32_t *partials, uint64_t *launches) {
  const ParallelPlan &plan = *s->parallel;
  const uint32_t kind = plan.sandwich ? kSandwichHead : kParallelHead;
  ParallelProjectionParams p{};
  p.w0 = plan.head;
  p.rows0 = plan.vocab;
  p.cols0 = plan.width_pad;
  p.h = stream.h;
  p.pending = stream.pending;
  p.after = stream.after;
  p.h_out = stream.h == s->h_a ? s->h_b : s->h_a;
  p.layer_norm = plan.layer_norm;
  p.norm = plan.final_norm;
  p.width = plan.width;
  p.eps = s->rms_eps;
  p.out_f32 = s->logits;
  p.scale = plan.logit_scale;
  p.softcap = plan.softcap;
  p.best_value = s->best_value;
  p.best_index = s->best_index;
  p.error_word = s->device_error;
  p.pdl = s->use_pdl ? 1u : 0u;
  if (!plan.f32 && parallel_stream_eligible(kind, p, s->sm_count)) {
    *partials = parallel_stream_blocks(kind, p, s->sm_count);
    if (launches != nullptr) *launches += 1;
    return launch_parallel_projection(s->stream, kind, p, s->sm_count);
  }
  StreamNormParams norm = layer_stream_norm(s, stream.h, plan.final_norm, s->x_scratch);
  norm.pending = stream.pending;
  norm.after = stream.after;
  cudaError_t err = launch_stream_norm(s->stream, norm, plan.f32, 1, p.pdl != 0);
  p.x0 = s->x_scratch;
  if (err == cudaSuccess) err = launch_parallel_projection_plain(s->stream, kParallelHead, p, 1, plan.f32);
  *partials = std::min(kBlockArgmaxChunks, s->sm_count);
  if (err == cudaSuccess)
    err = launch_argmax_partials(s->stream, s->logits, plan.vocab, 1, *partials, s->best_value, s->best_index, p.pdl != 0);
  if (launches != nullptr) *launches += 3;
  return err;
}

cudaError_t enqueue_parallel_block_layers(Session *s, const ParallelBlock &b, uint64_t *launches) {
  const ParallelPlan &plan = *s->parallel;
  if (plan.sandwich) return enqueue_sandwich_block_layers(s, b, launches);
  const BlockWorkspace &ws = s->weights->block_ws;
  const uint32_t pdl = s->use_pdl ? 1u : 0u;
  uint64_t n = 0;
  cudaError_t err = cudaSuccess;
  for (size_t index = 0; err == cudaSuccess && index < plan.runs.size(); ++index) {
    const ParallelRun &run = plan.runs[index];
    const ParallelLayerPlan &l = plan.layers[run.layer];
    StreamNormParams norm = layer_stream_norm(s, ws.h_b, l.norm, ws.x_bf16);
    norm.step = step_vector(plan, run);
    err = launch_stream_norm(b.stream, norm, plan.f32, b.rows, pdl != 0);
    ParallelProjectionParams in = layer_in(plan, l, s->rms_eps);
    if (err == cudaSuccess && plan.f32) {
      in.x0 = ws.x_bf16;
      in.out_f32 = ws.qkv;
      in.out_act = ws.ff;
      in.activation = plan.activation;
      in.pdl = pdl;
      err = launch_parallel_projection_plain(b.stream, kParallelIn, in, b.rows, true);
    } else if (err == cudaSuccess) {
      GemmParams g{};
      g.weight = l.w_in;
      g.rows = l.qkv_pad + 2u * l.ff_pad;
      g.cols = plan.width_pad;
      g.x = ws.x_bf16;
      g.epilogue = l.ff_pad != 0 ? kEpilogueStoreSwiglu : kEpilogueStore;
      g.split_row = l.qkv_pad;
      g.activation = plan.activation;
      g.out_f32 = ws.qkv;
      g.out_bf16 = ws.ff;
      err = parallel_block_gemm(s, b.stream, g, b.rows);
    }
    if (err == cudaSuccess) err = enqueue_block_attention(s, b, l, run, &n);

    ParallelProjectionParams out = layer_out(plan, l);
    if (err == cudaSuccess && plan.f32) {
      out.h = out.h_out = ws.h_b;
      out.x0 = ws.attn;
      out.x1 = ws.ff;
      out.pdl = pdl;
      err = launch_parallel_projection_plain(b.stream, kParallelOut, out, b.rows, true);
      n += 3;
    } else if (err == cudaSuccess) {
      GemmParams g{};
      g.rows = plan.width_pad;
      g.epilogue = kEpilogueStore;
      g.resid_in = g.out_f32 = ws.h_b;
      g.weight = out.w0;
      g.cols = out.cols0;
      g.x = ws.attn;
      g.row_scale = out.scale0;
      err = parallel_block_gemm(s, b.stream, g, b.rows);
      if (err == cudaSuccess && l.ff_pad != 0) {
        g.weight = out.w1;
        g.cols = out.cols1;
        g.x = ws.ff;
        g.row_scale = out.scale1;
        err = parallel_block_gemm(s, b.stream, g, b.rows);
      }
      n += l.ff_pad != 0 ? 4 : 3;
    }
    if (err == cudaSuccess) err = capture_block_stream(s, b, index);
  }
  if (launches != nullptr) *launches += n;
  return err;
}

cudaError_t enqueue_parallel_block_head(Session *s, cudaStream_t stream, uint32_t count, const uint32_t *row_index,
                                        uint64_t *launches) {
  const ParallelPlan &plan = *s->parallel;
  const BlockWorkspace &ws = s->weights->block_ws;
  StreamNormParams norm = layer_stream_norm(s, ws.h_b, plan.final_norm, ws.x_bf16);
  norm.row_index = row_index;
  cudaError_t err = launch_stream_norm(stream, norm, plan.f32, count, s->use_pdl);
  if (err == cudaSuccess && plan.f32) {
    ParallelProjectionParams p{};
    p.w0 = plan.head;
    p.rows0 = plan.vocab;
    p.cols0 = plan.width_pad;
    p.x0 = ws.x_bf16;
    p.out_f32 = ws.logits;
    p.scale = plan.logit_scale;
    p.softcap = plan.softcap;
    p.pdl = s->use_pdl ? 1u : 0u;
    err = launch_parallel_projection_plain(stream, kParallelHead, p, count, true);
  } else if (err == cudaSuccess) {
    GemmParams g{};
    g.weight = plan.head;
    g.rows = plan.vocab;
    g.cols = plan.width_pad;
    g.x = ws.x_bf16;
    g.epilogue = kEpilogueStore;
    g.scale = plan.logit_scale;
    g.softcap = plan.softcap;
    g.out_f32 = ws.logits;
    err = parallel_block_gemm(s, stream, g, count);
  }
  if (launches != nullptr) *launches += 2;
  return err;
}

}  // namespace nb
