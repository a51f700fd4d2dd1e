// Resident decode session: everything a session owns on the host and on the
// device.  Mirrors the role of the reference's
// hf_decode_sequence/session_state.cuh:1-222 (device pointers, cached graphs,
// cursor, token ring) with a different memory plan: two device allocations per
// session (shared weights, private state), each carved by a StaticArena, and
// nothing allocated after create.
#pragma once

#include <cuda_runtime.h>
#include <stdint.h>

#include <memory>
#include <string>
#include <deque>
#include <vector>

#include "../../include/nerva_b200_api.h"
#include "host_memory.h"
#include "kernels.cuh"

namespace nb {

constexpr uint64_t kMissingOffset = UINT64_MAX;

// Offsets (16-bit elements) of one layer's tensors in the upload arena; the
// order is the reference's pack_layer (hf_decode_sequence/weights.cu:487-591).
struct LayerLayout {
  uint64_t rms_attn = kMissingOffset, rms_mlp = kMissingOffset;
  uint64_t w_q = kMissingOffset, w_q_gate = kMissingOffset, q_norm = kMissingOffset;
  uint64_t w_k = kMissingOffset, k_norm = kMissingOffset, w_v = kMissingOffset;
  uint64_t w_o = kMissingOffset;
  uint64_t w_gate = kMissingOffset, w_up = kMissingOffset, w_down = kMissingOffset;
  uint64_t w_router = kMissingOffset, w_expert_gate_up = kMissingOffset;
  uint64_t w_expert_down = kMissingOffset;
  uint64_t w_shared_gate = kMissingOffset, w_shared_up = kMissingOffset;
  uint64_t w_shared_down = kMissingOffset, w_shared_router = kMissingOffset;
  uint64_t q_bias = kMissingOffset, k_bias = kMissingOffset, v_bias = kMissingOffset;
  uint64_t o_bias = kMissingOffset;
  uint32_t mlp_kind = 0, moe_intermediate = 0, shared_intermediate = 0;
  uint32_t num_experts = 0, top_k = 0, norm_topk_prob = 0;
  // DeepSeek multi-head latent attention (attention_kind 2): w_q is the query projection
  // [heads * (nope + rope)][hidden], w_k the latent + rotary-key projection [rank + rope][hidden],
  // k_norm the latent's norm weight [rank], w_v the up-projection [heads * (nope + v)][rank]
  // (per head: nope rows of W_UK, then v rows of W_UV), w_o [hidden][heads * v] — the slots the
  // reference's packer uses for them (hf_decode_sequence/deepseek/weights_pack.inc.cu:156-186).
  uint32_t attention_kind = 0, kv_lora_rank = 0, qk_nope = 0, qk_rope = 0;
  // Sparse-MoE expert matrices: Qwen-style layers hold per expert [gate rows | up rows]
  // (expert_up_offset = moe_intermediate * hidden inside a stride of twice that); DeepSeek layers
  // hold all gate matrices, then all up matrices (weights_pack.inc.cu:303-312).
  uint64_t expert_stride = 0, expert_up_offset = 0;
  // parallel blocks (rms_attn is the layer's one norm): per-channel scales of the two sublayers
  uint64_t ls_attn = kMissingOffset, ls_mlp = kMissingOffset;
  // sandwich blocks: the norms behind the sublayers (rms_attn, rms_mlp are those in front); attention's output
  // gate; a state space's input projection (w_o is its output) and small tensors
  uint64_t norm_after = kMissingOffset, norm_mlp_after = kMissingOffset, w_head_gate = kMissingOffset;
  uint64_t w_space = kMissingOffset, conv = kMissingOffset, conv_bias = kMissingOffset, step_bias = kMissingOffset;
  uint64_t a_log = kMissingOffset, skip = kMissingOffset, group_norm = kMissingOffset;
  // expert parallel: the experts whose matrices this arena holds (all of them otherwise)
  uint32_t expert_base = 0, expert_local = 0;
};

struct ArenaLayout {
  uint64_t embeddings = 0, input = 0, scratch = 0, final_norm = 0, lm_head = 0;
  uint64_t loop_vectors = kMissingOffset;  // [loop_times][hidden]
  uint64_t loop_input = kMissingOffset;    // [hidden][2 hidden]
  uint64_t elements = 0;
  std::vector<LayerLayout> layers;
};

struct ModelDims {
  uint32_t dtype = 0, hidden = 0, heads = 0, kv_heads = 0, head_dim = 0;
  uint32_t intermediate = 0, vocab = 0, layers = 0;
  // vocab = rows of lm_head held here; a tensor-parallel rank holds a shard of the
  // rows starting at vocab_offset, while the embedding table keeps embed_vocab rows.
  uint32_t embed_vocab = 0, vocab_offset = 0;
  // latent attention (every layer, or none): rows of the fused query + latent projection and width
  // of a cache row; zero for ordinary attention
  uint32_t mla_rank = 0, mla_nope = 0, mla_rope = 0;
  // expert parallel (ep_world > 1): this rank's arena holds num_experts / ep_world routed experts per layer
  uint32_t ep_world = 1, ep_rank = 0;
  uint64_t attention_hidden() const { return static_cast<uint64_t>(heads) * head_dim; }
  uint64_t kv_hidden() const { return static_cast<uint64_t>(kv_heads) * head_dim; }
  bool mla() const { return mla_rank != 0; }
  uint64_t mla_q_rows() const { return static_cast<uint64_t>(heads) * (mla_nope + mla_rope); }
  uint64_t mla_width() const { return static_cast<uint64_t>(mla_rank) + mla_rope; }
  // rows of the packed first projection of a layer: [Q; K; V], or [Q; latent + rotary key]
  uint64_t qkv_rows() const { return mla() ? mla_q_rows() + mla_width() : attention_hidden() + 2 * kv_hidden(); }
  // elements of one cached row per array
  uint64_t kv_row() const { return mla() ? mla_width() : kv_hidden(); }
};

bool valid_layer(const NervaCudaHfDecodeChainLayer &layer, bool require_sources);
bool layer_supported(const NervaCudaHfDecodeChainLayer &layer);
ArenaLayout compute_arena_layout(const ModelDims &dims, const NervaCudaHfDecodeChainLayer *layers,
                                 const NervaB200ParallelModel *parallel = nullptr);

// ---- decoders described layer by layer (parallel_step.cu; sandwich blocks: sandwich_step.cu) ----
// One layer: its mixer's shape and the padded copies of its weights the kernels read (every
// dimension a projection sums over, and every output of the residual stream, rounded up to 64 with
// zeros, so that neither TMA nor the norm prologue sees an odd size).
struct ParallelLayerPlan {
  bool state_space = false;
  WindowAttentionShape shape{};               // attention
  StateSpaceShape space{};                    // state space
  uint32_t intermediate = 0, ff_pad = 0;      // 0: no feed-forward
  uint32_t qkv_rows = 0, qkv_pad = 0;         // rows of the mixer's input projection ([Q; K; V; gates]), rounded up
  uint32_t attn_width = 0, attn_pad = 0;      // heads * v_dim
  bool layer_scale = false;
  std::vector<float> frequencies;
  uint16_t *w_in = nullptr;    // [qkv_pad + 2 ff_pad][width_pad]: Q, K, V, then gate/up rows interleaved
  uint16_t *w_o = nullptr;     // [width_pad][attn_pad]
  uint16_t *w_down = nullptr;  // [width_pad][ff_pad]
  uint16_t *norm = nullptr, *ls_attn = nullptr, *ls_mlp = nullptr;  // [width_pad]
  uint16_t *norm_after = nullptr, *norm_mlp = nullptr, *norm_mlp_after = nullptr;  // [width_pad], sandwich blocks
  uint16_t *group_norm = nullptr;             // [attn_pad], state space
  float *frequency = nullptr;
};
// One execution of a layer: a looped layer runs several times, each with its own part of the cache or state.
struct ParallelRun {
  uint32_t layer = 0;
  int32_t step = -1;  // row of the loop vectors added to the stream before this run, -1: none
  uint64_t key_offset = 0, value_offset = 0;  // elements from the start of a session's K / V array
  uint64_t state_offset = 0, history_offset = 0;  // floats from the start of a session's recurrent state
};
struct ParallelPlan {
  bool f32 = false, sandwich = false;
  uint32_t layer_norm = 0, activation = 0;
  uint32_t width = 0, width_pad = 0, vocab = 0, loop_times = 0;
  float embedding_scale = 1.0f, logit_scale = 0.0f, softcap = 0.0f;
  std::vector<ParallelLayerPlan> layers;
  std::vector<ParallelRun> runs;
  uint64_t key_elems = 0, value_elems = 0;    // per session, all runs
  uint64_t recurrent_floats = 0;              // per session, all runs
  uint32_t max_heads = 0, max_qkv_pad = 0, max_attn_pad = 0, max_ff_pad = 0, max_v_pad = 0;  // heads, v_pad: attention
  uint32_t max_space_pad = 0, max_conv_width = 0;  // state-space layers: attn_pad, convolved row
  uint16_t *loop_vectors = nullptr;           // [loop_times][width_pad]
  bool loop_input = false;
  uint16_t *w_join = nullptr;                 // [width_pad][2 width_pad]: stream columns, embedding columns
  uint16_t *final_norm = nullptr, *head = nullptr;  // [width_pad], [vocab][width_pad]
  uint32_t element_bytes() const { return f32 ? 4u : 2u; }
  uint32_t x_width() const { return loop_input ? 2u * width_pad : width_pad; }  // widest normalised activation row
};
// The residual stream of one token between two launches: h, and a sublayer output that has not joined it yet
// (h + norm(pending) is the stream; sandwich blocks only).
struct ResidualStream {
  float *h = nullptr;
  const float *pending = nullptr;
  const uint16_t *after = nullptr;  // the weight of pending's norm
};
// Null (with the reason in last_error) when the description is inconsistent or beyond the kernels.
std::shared_ptr<ParallelPlan> make_parallel_plan(const NervaB200ParallelModel &model, uint32_t width, uint32_t vocab,
                                                 float eps);
// Cache offsets of the runs for a session of `pages` pages.
void place_parallel_cache(ParallelPlan *plan, uint32_t pages);
struct StepProfile;
typedef void (*ProfileMark)(NervaCudaHfDecodeSequenceSession *, StepProfile *, uint32_t bucket);
cudaError_t pack_parallel_weights(NervaCudaHfDecodeSequenceSession *s);
// All layer runs of one decode step (stream: s->h_b in, what the head takes out), and its head; enqueue only.
cudaError_t enqueue_parallel_layers(NervaCudaHfDecodeSequenceSession *s, uint32_t splits, ResidualStream *stream,
                                    uint64_t *launches, StepProfile *prof, ProfileMark mark);
cudaError_t enqueue_parallel_head(NervaCudaHfDecodeSequenceSession *s, const ResidualStream &stream, uint32_t *partials,
                                  uint64_t *launches);
uint32_t parallel_attention_splits(const ParallelPlan &plan, uint32_t target_context);
uint64_t hash_tokens(const uint32_t *tokens, uint32_t count);
uint64_t hash_weight_descriptors(const NervaCudaHfDecodeSequenceWeightBlock *blocks, uint32_t count);
void set_last_error(const std::string &text);

// One token of a block step: where its id comes from and where errors go.
struct BlockTokenRow {
  const uint32_t *prompt;
  const uint32_t *prompt_count;
  const NervaCudaSyntheticTokenSlot *slots;
  uint32_t position, vocab;
  uint32_t *error_word;
};

// Scratch of the block steps (several tokens through every layer together: the packed step of
// batch_advance_one and the chunked prefill of session_start).  One per weight set, allocated at
// create and shared by the forks; a block step runs on one stream at a time.
struct BlockWorkspace {
  void *block = nullptr;
  uint64_t bytes = 0;
  uint32_t max_rows = 0, sample_rows = 0;
  uint16_t *x_bf16 = nullptr;   // [max_rows][x_elems] normalised activations, the B operand of the next GEMM
  float *qkv = nullptr;         // [max_rows][A + 2 KV]
  uint16_t *attn = nullptr;     // [max_rows][A]
  float *h_a = nullptr, *h_b = nullptr;  // [max_rows][hidden] residual stream, ping-pong; sandwich blocks keep
                                         // the stream in h_b and a sublayer's output in h_a
  float *first = nullptr;       // [max_rows][hidden] embedding output, where passes begin with it
  float *mixed = nullptr;       // [max_rows][heads * v_dim] state-space output in front of its norm
  void *convolved = nullptr;    // [max_rows][convolved row] of a state-space layer
  uint16_t *ff = nullptr;       // [max_rows][intermediate]
  float *logits = nullptr;      // [sample_rows][vocab]
  float *partial_acc = nullptr, *partial_m = nullptr, *partial_l = nullptr;  // split attention, per row
  uint32_t *attn_tickets = nullptr;  // [max_rows][kv_heads]
  float *gemm_workspace = nullptr;
  uint32_t *gemm_tickets = nullptr;
  float *best_value = nullptr;  // [sample_rows][kBlockArgmaxChunks]
  uint32_t *best_index = nullptr;
  FusedAttentionRow *attn_rows = nullptr;  // [max_rows] device copies of the row descriptors
  bool paged_rows = false;      // the rows' attention runs on the paged tensor-pipe kernel (attention.cu)
  BlockTokenRow *token_rows = nullptr;
  BlockSampleRow *sample_rows_dev = nullptr;  // [sample_rows] device copies of the sampler's row descriptors
  uint32_t *head_rows = nullptr;  // [sample_rows] rows of the block whose logits are wanted
};
constexpr uint32_t kBlockArgmaxChunks = 64;
constexpr uint32_t kBlockMaxRows = 256;       // one MMA N
constexpr uint32_t kBlockSampleRows = 32;     // sessions per packed decode step (hf_decode_sequence/types.cuh:63)

// Device weights shared between a session and its forks.
struct SharedWeights {
  void *block = nullptr;  // one allocation
  uint64_t block_bytes = 0;
  uint16_t *arena = nullptr;          // upload arena (reference layout)
  uint16_t *qkv_packed = nullptr;     // [layers][(A + 2 KV) x H]
  uint16_t *gate_up_packed = nullptr; // [layers][2 I x H], rows interleaved gate/up
  BlockWorkspace block_ws;            // empty when the model has no block-step path
  ~SharedWeights() {
    if (block != nullptr) cudaFree(block);
    if (block_ws.block != nullptr) cudaFree(block_ws.block);
  }
};

// Event-per-launch-group timing of un-captured steps (the reference's
// detailed_profile path, hf_decode_sequence/session_decode_prefill.inc.cu:374-810).
enum ProfileBucket : uint32_t {
  kBucketEmbed = 0, kBucketQkv, kBucketAttention, kBucketO, kBucketGateUp, kBucketDown,
  kBucketLmHead, kBucketSampling, kBucketCount
};
struct StepProfile {
  std::vector<cudaEvent_t> events;
  std::vector<uint32_t> bucket;  // bucket[i] labels the interval events[i] -> events[i+1]
  uint32_t used = 0;
};

struct GraphEntry {
  uint32_t splits = 0, sample = 0, engine = 0;
  cudaGraph_t graph = nullptr;
  cudaGraphExec_t exec = nullptr;  // null: the step is launched directly (capture was refused)
  uint64_t nodes = 0;
};

struct StepLayerDev;
struct JobDesc;
struct StepKernelParams;
uint32_t step_kernel_smem_bytes(uint32_t x_elems, uint32_t row_elems);
bool step_kernel_supported(uint32_t hidden, uint32_t heads, uint32_t kv_heads, uint32_t head_dim,
                           uint32_t intermediate, uint32_t x_elems, uint32_t row_elems);
cudaError_t configure_step_kernel();
cudaError_t launch_step_kernel(cudaStream_t stream, const StepKernelParams &p, uint32_t blocks);

// ---- block steps (block_step.cu) ----
// True when every layer is dense SwiGLU without biases, the fused attention kernel serves the head
// shape and every projection width is a multiple of 64: the shapes the block kernels run.
bool block_step_supported(const NervaCudaHfDecodeSequenceSession *s);
// Allocates s->weights->block_ws (at create).
cudaError_t allocate_block_workspace(NervaCudaHfDecodeSequenceSession *s);
// One token for each of `count` sessions that share weights, on `stream`: the weights are streamed
// once for the block.  Every session must be idle, positioned at its next token, and its stream
// synchronised.  Enqueues only; the caller copies the token slots back and synchronises.
cudaError_t enqueue_block_decode(NervaCudaHfDecodeSequenceSession *const *sessions, uint32_t count,
                                 cudaStream_t stream, uint64_t *launches);
// Logits wanted from a prefill: places[i] counts from the first position of the call, values go to
// logits[i][vocab] (host).
struct WantedLogits {
  const uint32_t *places = nullptr;
  uint32_t count = 0;
  float *logits = nullptr;
};
// Prompt positions [begin, prompt_count) of one session through every layer in chunks of up to
// kBlockMaxRows tokens, writing the same paged bf16 K/V the decode step reads, then the final
// norm, lm_head and the sampler for the last position.  Leaves the cursor at prompt_count.
cudaError_t enqueue_chunked_prefill(NervaCudaHfDecodeSequenceSession *s, uint32_t begin, uint32_t prompt_count,
                                    const WantedLogits &wanted, uint64_t *launches);
// The layer runs of a decoder described layer by layer over the block's rows (ws.h_b in and out) and the head of
// `count` rows (row_index: device array of block rows, null: the first `count`) into ws.logits.
struct ParallelBlock {
  cudaStream_t stream;
  uint32_t rows, longest;
  bool one_session;            // consecutive positions of one session
  uint32_t capture_row;        // row of the capture buffer the first row of the block goes to
};
cudaError_t enqueue_parallel_block_layers(NervaCudaHfDecodeSequenceSession *s, const ParallelBlock &b, uint64_t *launches);
// Pieces both kinds of block are made of: the norm between two projections, a projection of the block's rows, its attention (ws.qkv -> ws.attn),
// the parameters of a layer run's attention, and the copy of the stream behind a layer run into the session's
// capture buffer.
StreamNormParams layer_stream_norm(const NervaCudaHfDecodeSequenceSession *s, float *h, const uint16_t *weight, void *x);
cudaError_t parallel_block_gemm(NervaCudaHfDecodeSequenceSession *s, cudaStream_t stream, GemmParams g, uint32_t tokens);
cudaError_t enqueue_block_attention(NervaCudaHfDecodeSequenceSession *s, const ParallelBlock &b, const ParallelLayerPlan &l,
                                    const ParallelRun &run, uint64_t *launches);
cudaError_t enqueue_step_attention(NervaCudaHfDecodeSequenceSession *s, const ParallelLayerPlan &l, const ParallelRun &run,
                                   uint32_t splits, uint64_t *launches);
cudaError_t capture_block_stream(NervaCudaHfDecodeSequenceSession *s, const ParallelBlock &b, size_t run);
// Sandwich blocks (sandwich_step.cu).
cudaError_t enqueue_sandwich_layers(NervaCudaHfDecodeSequenceSession *s, uint32_t splits, ResidualStream *stream,
                                    uint64_t *launches, StepProfile *prof, ProfileMark mark);
cudaError_t enqueue_sandwich_block_layers(NervaCudaHfDecodeSequenceSession *s, const ParallelBlock &b, uint64_t *launches);
cudaError_t enqueue_parallel_block_head(NervaCudaHfDecodeSequenceSession *s, cudaStream_t stream, uint32_t count,
                                        const uint32_t *row_index, uint64_t *launches);

}  // namespace nb

// The opaque handle of the C ABI.
struct NervaCudaHfDecodeSequenceSession {
  nb::ModelDims dims;
  uint32_t max_context = 0;
  float rms_eps = 0.0f, rope_theta = 0.0f;
  uint32_t sm_count = 0;
  uint32_t engine = 0;
  uint32_t detailed_profile = 0;
  nb::ArenaLayout layout;
  std::vector<NervaCudaHfDecodeChainLayer> layer_meta;  // scalars only; pointers cleared

  // planned-weight echo
  uint64_t resident_weight_bytes = 0;
  uint32_t planned_weight_blocks = 0, planned_gpu_resident_blocks = 0, planned_gpu_staged_blocks = 0;
  uint64_t planned_weight_bytes = 0, planned_gpu_resident_weight_bytes = 0;
  uint64_t planned_gpu_staged_weight_bytes = 0;
  uint32_t planned_weight_descriptor_count = 0;
  uint64_t planned_weight_descriptor_hash = 0;

  std::shared_ptr<nb::SharedWeights> weights;
  std::shared_ptr<nb::ParallelPlan> parallel;  // decoders described layer by layer only
  float *capture_stream = nullptr;             // host buffer of nerva_b200_session_capture_stream
  uint32_t capture_rows = 0;
  nb::StaticArena weight_arena, state_arena;
  nb::KvPagePool kv_pool;

  // private device state (one allocation)
  void *state_block = nullptr;
  uint64_t state_bytes = 0;
  uint16_t *kv_keys = nullptr, *kv_values = nullptr;  // [layers][pages][16][kv_hidden]
  uint64_t kv_layer_elems = 0;
  // the two arrays as 2-D tensor maps [layers * pages * 16][kv_hidden] (boxes of 64 dims x one page),
  // encoded once when the state is allocated; read by the row form of the paged attention kernel
  nb::TensorMapStorage kv_map_k{}, kv_map_v{};
  bool kv_maps = false;
  uint32_t kv_pages = 0;
  uint32_t *page_table = nullptr;
  float *h_a = nullptr, *h_b = nullptr, *qkv = nullptr, *o_out = nullptr, *down = nullptr;
  // decoders described layer by layer: recurrent state of all layer runs, the token's embedding output, and a
  // state-space layer's output in front of its norm
  float *recurrent = nullptr, *first = nullptr, *mixed = nullptr;
  float *logits = nullptr;
  float *partial_acc = nullptr, *partial_m = nullptr, *partial_l = nullptr;
  uint32_t max_splits = 1;
  uint32_t *attn_tickets = nullptr;  // per-head completion tickets of the fused attention kernel
  bool fused_attention = false;      // head_dim 64/128: one attention launch per layer
  bool use_pdl = true;               // programmatic dependent launch between the step's kernels
                                     // (NERVA_B200_PDL=0 at create turns it off)
  uint16_t *attn_bf16 = nullptr, *ff_bf16 = nullptr, *x_scratch = nullptr;
  float *best_value = nullptr;
  uint32_t *best_index = nullptr;
  // whole-step kernel (engine 1)
  nb::StepLayerDev *step_layers = nullptr;
  nb::JobDesc *step_jobs = nullptr;
  uint32_t *barrier_counter = nullptr;
  unsigned long long *phase_cycles = nullptr;  // per-phase SM cycles of block 0 (tuning aid)
  bool phase_profile = false;                  // NERVA_B200_PHASE_PROFILE=1 at create
  // Tuning aid (NERVA_B200_TIMELINE=1 at create): per launch of a step, %globaltimer
  // stamps of the first and the last block (see kTimelineSlots in kernels.cuh).
  unsigned long long *timeline = nullptr;
  uint32_t timeline_nodes = 0;
  bool timeline_on = false;
  // sparse MoE layers: routing scratch
  bool has_moe = false;
  std::vector<int32_t> dense_ordinal;  // per layer: index of its packed gate/up copy, -1 for sparse layers
  // latent attention scratch
  float *mla_ql = nullptr;             // [heads][rank] absorbed queries
  float *router_logits = nullptr, *route_weights = nullptr, *shared_gate = nullptr, *moe_gate_up = nullptr;
  uint32_t *route_ids = nullptr;
  float *moe_partial = nullptr;        // [17][hidden] per-expert contributions of a sparse MLP (moe.cu)
  uint32_t *moe_ticket = nullptr;      // completion counter of the expert down launch, zero between launches
  // tensor parallel (nerva_b200_session_create_sharded)
  uint32_t tp_world = 1, tp_rank = 0;
  bool tp_two_stage = false;   // two ranks only: use the two-stage gather of the larger worlds
  void *comm_block = nullptr;  // this rank's exchange buffer (own allocation, exported to the peers)
  uint64_t comm_bytes = 0;
  void *comm_peers[nb::kMaxTpWorld] = {};  // every rank's exchange buffer as mapped here
  bool tp_attached = false;
  uint32_t x_elems = 0;
  uint32_t row_elems = 0;  // rows of the largest per-block row range of any projection
  bool step_kernel_ok = false;
  NervaCudaSyntheticTokenSlot *device_slots = nullptr;
  uint32_t *device_cursor = nullptr, *device_error = nullptr, *device_prompt = nullptr;
  uint64_t slots_bytes = 0;

  NervaCudaSyntheticTokenSlot *host_slots = nullptr;  // pinned
  uint32_t *host_error = nullptr;                     // pinned, 1 word

  cudaStream_t stream = nullptr;
  cudaEvent_t ev_start = nullptr, ev_stop = nullptr;
  std::deque<nb::GraphEntry> graphs;  // deque: entries keep their address when more are cached

  // active request
  bool started = false, finished = false;
  uint32_t prompt_count = 0, has_eos = 0, eos_token = 0, seed_token = 0;
  uint32_t observed = 0, cursor = 0;
  bool logits_valid = false;
  // Sampler of the active request: 1 = arg-max, 2 = temperature / top-k / top-p from device_sampler.
  uint32_t sample_kind = 1;
  nb::SamplerParams host_sampler{};
  nb::SamplerParams *device_sampler = nullptr;
  uint64_t hot_path_allocations = 0;
};

// Element offset of layer l's packed gate/up copy (dense layers only; sparse layers have none).
inline uint64_t gate_up_packed_offset(const NervaCudaHfDecodeSequenceSession *s, uint32_t l) {
  return static_cast<uint64_t>(s->dense_ordinal[l]) * 2u * s->dims.intermediate * s->dims.hidden;
}
