// Projections of decoders described layer by layer for one token, and the plain any-shape form of the
// same for a block of tokens.
//
// Parallel blocks (one norm in front of mixer and feed-forward, both results summed into the residual
// stream).
// The streaming form puts two weight matrices into one launch on the row-stream core
// (row_stream.cuh): its ring runs across a job list, so the second matrix's bytes follow the first's
// without a gap.
//   kParallelIn    [Q; K; V] behind the norm prologue
//   kParallelGate  the interleaved gate/up matrix behind the same prologue
//   kParallelOut   O and down, dealt to the blocks by the same row ranges, so the block that owns a
//                  row of the stream has both sums and writes h + scale0 * O + scale1 * down once
//   kParallelHead  the head behind the final norm, logits soft-capped before the arg-max
// In a parallel block the feed-forward does not wait for the attention: kParallelGate streams its
// matrix while the attention of the same layer runs beside it on the same SMs.  For that the two
// kernels around the attention take two ring slots per warp instead of three, which leaves shared
// memory for the attention's blocks (see the launch order in kernels.cuh).
//
// Sandwich blocks (a norm in front of and behind each sublayer): five launches per layer, In, mixer, Out,
// Gate, Out.  What a sublayer returns has to be normalised as a whole before it joins the stream, so
// kSandwichOut stores it plainly and the next prologue adds it: every block computes h + norm(pending) and
// its norm from two vectors that sit in L2, one extra synchronisation, where a launch of its own would cost
// a round trip between two weight streams.
#include "kernels.cuh"
#include "row_stream.cuh"
#include "step_device.cuh"

namespace nb {
namespace {

constexpr uint32_t kNoIndex = 0xffffffffu;
// Ring slots per warp: two where an attention block shares the SM.
constexpr uint32_t slots_of(uint32_t kind) { return kind == kParallelIn || kind == kParallelGate ? 2u : kStreamSlots; }
constexpr bool sandwich_prologue(uint32_t kind) {
  return kind == kSandwichIn || kind == kSandwichGate || kind == kSandwichHead || kind == kSandwichJoin;
}
constexpr bool gate_pairs(uint32_t kind) { return kind == kParallelGate || kind == kSandwichGate; }
constexpr uint32_t kGroupChunk = 128;  // elements a warp normalises together: parts of a grouped norm are multiples of it
constexpr uint32_t kMaxGroupChunks = kNormRegIters * kStreamThreads * 4u / kGroupChunk;
constexpr uint32_t ring_bytes(uint32_t kind) { return kStreamWarps * slots_of(kind) * kChunkBytes; }

__device__ __forceinline__ bool candidate_better(float v, uint32_t i, float best_v, uint32_t best_i) {
  return v > best_v || (v == best_v && i < best_i);
}
__device__ __forceinline__ float soft_cap(float y, float cap) { return cap > 0.0f ? cap * tanhf(y / cap) : y; }
__device__ __forceinline__ float logit(const ParallelProjectionParams &p, float y) {
  return soft_cap(p.scale != 0.0f ? y * p.scale : y, p.softcap);
}

constexpr uint32_t kPlainL2PrefetchBytes = 16384;  // per warp, behind the plain vector copies

struct ParallelShared {
  StreamShared first, second;  // the ring's barriers are first's; each job has its own edge records
  JobDesc jobs[2];
  float scratch[2u * kMomentsScratch];
  float best_v[kStreamWarps];
  uint32_t best_i[kStreamWarps];
};

__host__ __device__ inline uint32_t round128(uint32_t v) { return (v + 127u) & ~127u; }

// The sandwich prologue: x (shared memory) from the residual stream and a pending sublayer output.
template <uint32_t KIND, class Fill>
__device__ __forceinline__ void sandwich_norm(const ParallelProjectionParams &p, uint16_t *x, float *scratch, Fill fill) {
  constexpr bool kJoin = KIND == kSandwichJoin;
  const uint32_t cols = kJoin ? p.cols0 / 2u : p.cols0, vecs = cols / 4u;
  NormWeightRegs weights, after;
  if (!kJoin) norm_weights_preload(weights, p.norm, cols);
  if (p.pending != nullptr) norm_weights_preload(after, p.after, cols);
  pdl_wait();
  NormValueRegs h, y;
  norm_single_load(h, p.h, cols);
  if (p.pending != nullptr) norm_single_load(y, p.pending, cols);
  fill();
  if (p.pending != nullptr) {
    const NormMoments m = norm_moments(y.v, p.width, p.layer_norm, p.eps, scratch);
#pragma unroll
    for (uint32_t k = 0; k < kNormRegIters; ++k) {
      h.v[k].x += (y.v[k].x - m.mean) * m.scale * bf16x2_lo(after.w[k].x);
      h.v[k].y += (y.v[k].y - m.mean) * m.scale * bf16x2_hi(after.w[k].x);
      h.v[k].z += (y.v[k].z - m.mean) * m.scale * bf16x2_lo(after.w[k].y);
      h.v[k].w += (y.v[k].w - m.mean) * m.scale * bf16x2_hi(after.w[k].y);
    }
    if (!kJoin && blockIdx.x == 0) {  // the others only read h: the new stream goes to another buffer
#pragma unroll
      for (uint32_t k = 0; k < kNormRegIters; ++k) {
        const uint32_t i = threadIdx.x + k * blockDim.x;
        if (i < vecs) reinterpret_cast<float4 *>(p.h_out)[i] = h.v[k];
      }
    }
  }
  if (kJoin) {
    NormValueRegs first;
    norm_single_load(first, p.first, cols);
#pragma unroll
    for (uint32_t k = 0; k < kNormRegIters; ++k) {
      const uint32_t i = threadIdx.x + k * blockDim.x;
      if (i < vecs) {
        const float4 a = h.v[k], b = first.v[k];
        reinterpret_cast<uint2 *>(x)[i] = make_uint2(f32_to_bf16_bits(a.x) | static_cast<uint32_t>(f32_to_bf16_bits(a.y)) << 16,
                                                     f32_to_bf16_bits(a.z) | static_cast<uint32_t>(f32_to_bf16_bits(a.w)) << 16);
        reinterpret_cast<uint2 *>(x + cols)[i] =
            make_uint2(f32_to_bf16_bits(b.x) | static_cast<uint32_t>(f32_to_bf16_bits(b.y)) << 16,
                       f32_to_bf16_bits(b.z) | static_cast<uint32_t>(f32_to_bf16_bits(b.w)) << 16);
      }
    }
    return;
  }
  const NormMoments m = norm_moments(h.v, p.width, p.layer_norm, p.eps, scratch + kMomentsScratch);
#pragma unroll
  for (uint32_t k = 0; k < kNormRegIters; ++k) {
    const uint32_t i = threadIdx.x + k * blockDim.x;
    if (i < vecs) reinterpret_cast<uint2 *>(x)[i] = normed_bf16x4(h.v[k], weights.w[k], m);
  }
}

// x (shared memory) = grouped RMS norm of p.x_f32.  A warp's 128 values of one iteration lie in one part.
template <class Fill>
__device__ __forceinline__ void grouped_norm(const ParallelProjectionParams &p, uint16_t *x, float *scratch, Fill fill) {
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5, vecs = p.cols0 / 4u;
  NormWeightRegs weights;
  norm_weights_preload(weights, p.norm, p.cols0);
  pdl_wait();
  NormValueRegs y;
  norm_single_load(y, p.x_f32, p.cols0);
  fill();
  float *chunk_sum = scratch, *group_scale = scratch + kMaxGroupChunks;
#pragma unroll
  for (uint32_t k = 0; k < kNormRegIters; ++k) {
    const float4 v = y.v[k];
    const float square = warp_sum((v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w));
    if (lane == 0) chunk_sum[k * kStreamWarps + warp] = square;
  }
  __syncthreads();
  const uint32_t part = p.width / p.groups, chunks = part / kGroupChunk;
  for (uint32_t g = threadIdx.x; g < p.groups; g += blockDim.x) {
    float total = 0.0f;
    for (uint32_t c = 0; c < chunks; ++c) total += chunk_sum[g * chunks + c];
    group_scale[g] = 1.0f / sqrtf(total / static_cast<float>(part) + p.eps);
  }
  __syncthreads();
#pragma unroll
  for (uint32_t k = 0; k < kNormRegIters; ++k) {
    const uint32_t i = threadIdx.x + k * blockDim.x;
    if (i < vecs) {
      const uint32_t g = 4u * i / part;  // elements behind the last part are zero
      reinterpret_cast<uint2 *>(x)[i] =
          normed_bf16x4(y.v[k], weights.w[k], NormMoments{0.0f, g < p.groups ? group_scale[g] : 0.0f});
    }
  }
}
static_assert(2u * kMaxGroupChunks <= 2u * kMomentsScratch, "a grouped norm's sums and scales fit the scratch");

template <uint32_t KIND>
__global__ void __launch_bounds__(kStreamThreads, 1) parallel_stream_kernel(ParallelProjectionParams p) {
  constexpr uint32_t SLOTS = slots_of(KIND);
  constexpr uint32_t kRing = ring_bytes(KIND);
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t *ring = smem;
  uint16_t *x0 = reinterpret_cast<uint16_t *>(smem + kRing);
  uint16_t *x1 = reinterpret_cast<uint16_t *>(smem + kRing + round128(p.cols0 * 2u));
  const bool second = KIND == kParallelOut && p.rows1 != 0;
  const uint32_t x_bytes = round128(p.cols0 * 2u) + (second ? round128(p.cols1 * 2u) : 0u);
  ParallelShared &sh = *reinterpret_cast<ParallelShared *>(smem + kRing + x_bytes);
  float *total0 = reinterpret_cast<float *>(smem + kRing + x_bytes + round128(sizeof(ParallelShared)));
  constexpr uint32_t unit = gate_pairs(KIND) ? 2u : 1u;
  const uint32_t rows_all = gate_pairs(KIND) ? p.rows1 : p.rows0;

  if (KIND != kParallelIn) pdl_trigger();
  if (threadIdx.x == 0) {
    sh.jobs[0] = JobDesc{gate_pairs(KIND) ? p.w1 : p.w0, rows_all, p.cols0, unit, 0};
    sh.jobs[1] = JobDesc{p.w1, p.rows1, p.cols1, 1, 0};
  }
  __syncthreads();
  RowStream rs;
  stream_init<SLOTS>(rs, ring, sh.first, sh.jobs, second ? 2u : 1u);
  // ahead of a norm prologue one slot is held back: the activation loads would queue behind a whole ring
  stream_fill<SLOTS>(rs, KIND == kParallelOut ? SLOTS : SLOTS - 1u);

  uint32_t begin0, end0, begin1 = 0, end1 = 0;
  block_row_range(rows_all, unit, blockIdx.x, gridDim.x, &begin0, &end0);
  if (second) block_row_range(p.rows1, 1, blockIdx.x, gridDim.x, &begin1, &end1);
  const uint32_t rows0 = end0 - begin0, rows1 = end1 - begin1;
  float *total1 = total0 + rows0;
  for (uint32_t r = threadIdx.x; r < rows0 + rows1; r += blockDim.x) total0[r] = 0.0f;

  float resid_first = 0.0f;
  auto fill = [&]() { stream_fill<SLOTS>(rs); };  // the ring slot held back, behind the activation loads
  if (sandwich_prologue(KIND)) {
    sandwich_norm<KIND>(p, x0, sh.scratch, fill);
  } else if (KIND == kSandwichOut) {
    if (p.groups != 0) {
      grouped_norm(p, x0, sh.scratch, fill);
    } else {
      pdl_wait();
      const uint4 *src0 = reinterpret_cast<const uint4 *>(p.x0);
      for (uint32_t i = threadIdx.x; i < p.cols0 / 8u; i += blockDim.x) reinterpret_cast<uint4 *>(x0)[i] = __ldcg(src0 + i);
      fill();
      stream_prefetch_l2(rs, kPlainL2PrefetchBytes);
    }
  } else if (KIND == kParallelOut) {
    pdl_wait();
    if (threadIdx.x < rows0) resid_first = __ldcg(p.h + begin0 + threadIdx.x);
    const uint4 *src0 = reinterpret_cast<const uint4 *>(p.x0);
    for (uint32_t i = threadIdx.x; i < p.cols0 / 8u; i += blockDim.x) reinterpret_cast<uint4 *>(x0)[i] = __ldcg(src0 + i);
    if (second) {
      const uint4 *src1 = reinterpret_cast<const uint4 *>(p.x1);
      for (uint32_t i = threadIdx.x; i < p.cols1 / 8u; i += blockDim.x) reinterpret_cast<uint4 *>(x1)[i] = __ldcg(src1 + i);
    }
    stream_prefetch_l2(rs, kPlainL2PrefetchBytes);
  } else {
    NormWeightRegs weights, step;
    norm_weights_preload(weights, p.norm, p.cols0);
    if (p.step != nullptr) norm_weights_preload(step, p.step, p.cols0);
    if (KIND != kParallelGate) pdl_wait();
    if (KIND == kParallelIn) pdl_trigger();  // whoever runs after this knows that h is complete
    NormValueRegs values;
    norm_single_load(values, p.h, p.cols0);
    stream_fill<SLOTS>(rs);  // the ring slot held back, now behind the activation loads
    if (p.step != nullptr) {
#pragma unroll
      for (uint32_t k = 0; k < kNormRegIters; ++k) {
        values.v[k].x += bf16x2_lo(step.w[k].x);
        values.v[k].y += bf16x2_hi(step.w[k].x);
        values.v[k].z += bf16x2_lo(step.w[k].y);
        values.v[k].w += bf16x2_hi(step.w[k].y);
      }
    }
    norm_single_finish(x0, values, weights, p.eps, p.cols0, sh.scratch, p.width);
  }
  __syncthreads();

  stream_consume<false, SLOTS>(rs, sh.first, 0, x0, total0, p.error_word);
  if (second) stream_consume<false, SLOTS>(rs, sh.second, 1, x1, total1, p.error_word);
  __syncthreads();

  if (KIND == kParallelIn || KIND == kSandwichIn || KIND == kSandwichOut) {
    for (uint32_t r = threadIdx.x; r < rows0; r += blockDim.x)
      p.out_f32[begin0 + r] = stream_row_total(sh.first, total0, r);
  } else if (KIND == kSandwichJoin) {
    for (uint32_t r = threadIdx.x; r < rows0; r += blockDim.x) {
      const float y = stream_row_total(sh.first, total0, r);
      p.out_f32[begin0 + r] = p.row_add != nullptr ? y + bf16_bits_to_f32(p.row_add[begin0 + r]) : y;
    }
  } else if (gate_pairs(KIND)) {
    uint16_t *act = reinterpret_cast<uint16_t *>(p.out_act);
    for (uint32_t i = threadIdx.x; i < rows0 / 2u; i += blockDim.x) {
      const float gate = stream_row_total(sh.first, total0, 2u * i);
      const float up = stream_row_total(sh.first, total0, 2u * i + 1u);
      act[begin0 / 2u + i] = f32_to_bf16_bits(activate(p.activation, gate) * up);
    }
    if (KIND == kParallelGate) pdl_wait();  // the attention beside this launch: the next launch waits for this one only
  } else if (KIND == kParallelOut) {
    for (uint32_t r = threadIdx.x; r < rows0; r += blockDim.x) {
      const uint32_t row = begin0 + r;
      float resid = r == threadIdx.x ? resid_first : __ldcg(p.h + row);
      if (p.step != nullptr) resid += bf16_bits_to_f32(p.step[row]);
      float y = stream_row_total(sh.first, total0, r);
      if (p.scale0 != nullptr) y *= bf16_bits_to_f32(p.scale0[row]);
      if (second) {
        float z = stream_row_total(sh.second, total1, r);
        if (p.scale1 != nullptr) z *= bf16_bits_to_f32(p.scale1[row]);
        y += z;
      }
      p.h_out[row] = resid + y;
    }
  } else {
    float bv = -INFINITY;
    uint32_t bi = kNoIndex;
    for (uint32_t r = threadIdx.x; r < rows0; r += blockDim.x) {
      const float v = logit(p, stream_row_total(sh.first, total0, r));
      p.out_f32[begin0 + r] = v;
      if (isfinite(v) && candidate_better(v, begin0 + r, bv, bi)) {
        bv = v;
        bi = begin0 + r;
      }
    }
    for (int offset = 16; offset > 0; offset >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, offset);
      const uint32_t oi = __shfl_xor_sync(0xffffffffu, bi, offset);
      if (oi != kNoIndex && candidate_better(ov, oi, bv, bi)) {
        bv = ov;
        bi = oi;
      }
    }
    if ((threadIdx.x & 31u) == 0) {
      sh.best_v[threadIdx.x >> 5] = bv;
      sh.best_i[threadIdx.x >> 5] = bi;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
      bv = -INFINITY;
      bi = kNoIndex;
      for (uint32_t w = 0; w < kStreamWarps; ++w) {
        if (sh.best_i[w] != kNoIndex && candidate_better(sh.best_v[w], sh.best_i[w], bv, bi)) {
          bv = sh.best_v[w];
          bi = sh.best_i[w];
        }
      }
      p.best_value[blockIdx.x] = bv;
      p.best_index[blockIdx.x] = bi;
    }
  }
  stream_drain<SLOTS>(rs);
}

uint32_t stream_blocks(uint32_t kind, const ParallelProjectionParams &p, uint32_t sm_count) {
  // one block per SM; fewer when the matrices are too small to give every warp of every block 4 KiB
  const uint32_t rows = gate_pairs(kind) ? p.rows1 : p.rows0;
  uint64_t bytes = static_cast<uint64_t>(rows) * p.cols0 * 2u;
  if (kind == kParallelOut) bytes += static_cast<uint64_t>(p.rows1) * p.cols1 * 2u;
  uint64_t blocks = bytes / (static_cast<uint64_t>(kStreamWarps) * 4096u);
  const uint32_t units = gate_pairs(kind) ? rows / 2u : rows;
  if (blocks > units) blocks = units;
  if (blocks > sm_count) blocks = sm_count;
  return blocks == 0 ? 1u : static_cast<uint32_t>(blocks);
}

uint32_t stream_smem_bytes(uint32_t kind, const ParallelProjectionParams &p, uint32_t blocks) {
  const bool second = kind == kParallelOut && p.rows1 != 0;
  uint32_t rows = gate_pairs(kind) ? max_rows_per_block(p.rows1, 2, blocks) : max_rows_per_block(p.rows0, 1, blocks);
  if (second) rows += max_rows_per_block(p.rows1, 1, blocks);
  return ring_bytes(kind) + round128(p.cols0 * 2u) + (second ? round128(p.cols1 * 2u) : 0u) +
         round128(sizeof(ParallelShared)) + round128(rows * 4u + 16u);
}

// ---------------------------------------------------------------- plain form ----
// One warp per output row (or gate/up pair) and up to kPlainTokens tokens; lane l takes elements
// 2l, 2l+1 of every 64.  The form every shape and the fp32 sessions run.
constexpr uint32_t kPlainTokens = 4;
constexpr uint32_t kPlainWarps = 8;

__device__ __forceinline__ float2 load_pair(const float *x) { return __ldcg(reinterpret_cast<const float2 *>(x)); }
__device__ __forceinline__ float2 load_pair(const uint16_t *x) {
  const uint32_t w = __ldcg(reinterpret_cast<const uint32_t *>(x));
  return make_float2(bf16x2_lo(w), bf16x2_hi(w));
}
__device__ __forceinline__ void store_act(float *out, float v) { *out = v; }
__device__ __forceinline__ void store_act(uint16_t *out, float v) { *out = f32_to_bf16_bits(v); }

template <class X>
__device__ __forceinline__ void plain_dots(const uint16_t *w, const X *x, uint32_t cols, uint32_t tokens,
                                           float (&acc)[kPlainTokens]) {
#pragma unroll
  for (uint32_t m = 0; m < kPlainTokens; ++m) acc[m] = 0.0f;
  for (uint32_t k = 2u * (threadIdx.x & 31u); k < cols; k += 64u) {
    const uint32_t wk = __ldg(reinterpret_cast<const uint32_t *>(w + k));
#pragma unroll
    for (uint32_t m = 0; m < kPlainTokens; ++m) {
      if (m < tokens) {
        const float2 xk = load_pair(x + static_cast<uint64_t>(m) * cols + k);
        acc[m] = fmaf(bf16x2_lo(wk), xk.x, acc[m]);
        acc[m] = fmaf(bf16x2_hi(wk), xk.y, acc[m]);
      }
    }
  }
#pragma unroll
  for (uint32_t m = 0; m < kPlainTokens; ++m) acc[m] = warp_sum(acc[m]);
}

template <class X, uint32_t KIND>
__global__ void __launch_bounds__(kPlainWarps * 32) parallel_plain_kernel(ParallelProjectionParams p, uint32_t tokens) {
  pdl_trigger();
  pdl_wait();
  const uint32_t lane = threadIdx.x & 31u;
  const uint32_t unit = blockIdx.x * kPlainWarps + (threadIdx.x >> 5);
  const uint32_t m0 = blockIdx.y * kPlainTokens;
  const uint32_t count = tokens - m0 < kPlainTokens ? tokens - m0 : kPlainTokens;
  const X *x0 = reinterpret_cast<const X *>(p.x0) + static_cast<uint64_t>(m0) * p.cols0;
  if (KIND == kParallelIn && unit >= p.rows0) {
    const uint32_t pair = unit - p.rows0;
    if (pair >= p.rows1 / 2u) return;
    float gate[kPlainTokens], up[kPlainTokens];
    plain_dots(p.w1 + static_cast<uint64_t>(2u * pair) * p.cols0, x0, p.cols0, count, gate);
    plain_dots(p.w1 + static_cast<uint64_t>(2u * pair + 1u) * p.cols0, x0, p.cols0, count, up);
    if (lane != 0) return;
    for (uint32_t m = 0; m < count; ++m)
      store_act(reinterpret_cast<X *>(p.out_act) + static_cast<uint64_t>(m0 + m) * (p.rows1 / 2u) + pair,
                activate(p.activation, gate[m]) * up[m]);
    return;
  }
  if (unit >= p.rows0) return;
  float y[kPlainTokens];
  plain_dots(p.w0 + static_cast<uint64_t>(unit) * p.cols0, x0, p.cols0, count, y);
  if (KIND == kParallelOut) {
    float z[kPlainTokens];
    if (p.rows1 != 0)
      plain_dots(p.w1 + static_cast<uint64_t>(unit) * p.cols1,
                 reinterpret_cast<const X *>(p.x1) + static_cast<uint64_t>(m0) * p.cols1, p.cols1, count, z);
    if (lane != 0) return;
    const float s0 = p.scale0 != nullptr ? bf16_bits_to_f32(p.scale0[unit]) : 1.0f;
    const float s1 = p.scale1 != nullptr ? bf16_bits_to_f32(p.scale1[unit]) : 1.0f;
    for (uint32_t m = 0; m < count; ++m) {
      const uint64_t at = static_cast<uint64_t>(m0 + m) * p.rows0 + unit;
      p.h_out[at] = __ldcg(p.h + at) + (p.rows1 != 0 ? y[m] * s0 + z[m] * s1 : y[m] * s0);
    }
    return;
  }
  if (lane != 0) return;
  const float add = KIND == kParallelIn && p.row_add != nullptr ? bf16_bits_to_f32(p.row_add[unit]) : 0.0f;
  for (uint32_t m = 0; m < count; ++m)
    p.out_f32[static_cast<uint64_t>(m0 + m) * p.rows0 + unit] = KIND == kParallelHead ? logit(p, y[m]) : y[m] + add;
}

constexpr uint32_t kNormThreads = 256;

// Four consecutive values of a padded row, those beyond `width` dropped.
__device__ __forceinline__ void only_below(float (&v)[4], uint32_t i, uint32_t width) {
#pragma unroll
  for (uint32_t j = 0; j < 4u; ++j)
    if (i + j >= width) v[j] = 0.0f;
}

// Mean (zero for RMS norms) and scale of a row's norm; any width, the values come from L1 or L2 again.
__device__ __forceinline__ NormMoments row_moments(const float *row, const StreamNormParams &p, float *scratch) {
  NormMoments m{0.0f, 0.0f};
  if (p.layer_norm != 0) {
    float sum = 0.0f;
    for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
      const float4 v = *reinterpret_cast<const float4 *>(row + i);
      sum += (v.x + v.y) + (v.z + v.w);  // zeros beyond the width
    }
    m.mean = block_sum(sum, scratch) / static_cast<float>(p.width);
  }
  float sumsq = 0.0f;
  for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
    const float4 v = *reinterpret_cast<const float4 *>(row + i);
    float d[4] = {v.x - m.mean, v.y - m.mean, v.z - m.mean, v.w - m.mean};
    if (p.layer_norm != 0) only_below(d, i, p.width);
    sumsq += d[0] * d[0] + d[1] * d[1] + d[2] * d[2] + d[3] * d[3];
  }
  m.scale = 1.0f / sqrtf(block_sum(sumsq, scratch) / static_cast<float>(p.width) + p.eps);
  return m;
}

// A row's pending output and norm with every value read once: the sandwich prologue for a block of rows.
template <class X>
__device__ __forceinline__ void norm_in_registers(const StreamNormParams &p, float *row, uint32_t source) {
  __shared__ float scratch[2u * kMomentsScratch];
  const uint32_t vecs = p.padded / 4u;
  NormValueRegs h, y;
  norm_single_load(h, row, p.padded);
  if (p.pending != nullptr) {
    norm_single_load(y, p.pending + static_cast<uint64_t>(source) * p.padded, p.padded);
    const NormMoments m = norm_moments(y.v, p.width, p.layer_norm, p.eps, scratch);
#pragma unroll
    for (uint32_t k = 0; k < kNormRegIters; ++k) {
      const uint32_t i = threadIdx.x + k * kNormThreads;
      if (i < vecs) {
        const uint2 w = reinterpret_cast<const uint2 *>(p.after)[i];
        h.v[k].x += (y.v[k].x - m.mean) * m.scale * bf16x2_lo(w.x);
        h.v[k].y += (y.v[k].y - m.mean) * m.scale * bf16x2_hi(w.x);
        h.v[k].z += (y.v[k].z - m.mean) * m.scale * bf16x2_lo(w.y);
        h.v[k].w += (y.v[k].w - m.mean) * m.scale * bf16x2_hi(w.y);
        reinterpret_cast<float4 *>(row)[i] = h.v[k];
      }
    }
  }
  if (p.x == nullptr) return;
  const NormMoments m = norm_moments(h.v, p.width, p.layer_norm, p.eps, scratch + kMomentsScratch);
  X *out = reinterpret_cast<X *>(p.x) + static_cast<uint64_t>(blockIdx.x) * p.padded;
#pragma unroll
  for (uint32_t k = 0; k < kNormRegIters; ++k) {
    const uint32_t i = threadIdx.x + k * kNormThreads;
    if (i < vecs) {
      const uint2 w = reinterpret_cast<const uint2 *>(p.norm)[i];
      store_act(out + 4u * i, (h.v[k].x - m.mean) * m.scale * bf16x2_lo(w.x));
      store_act(out + 4u * i + 1u, (h.v[k].y - m.mean) * m.scale * bf16x2_hi(w.x));
      store_act(out + 4u * i + 2u, (h.v[k].z - m.mean) * m.scale * bf16x2_lo(w.y));
      store_act(out + 4u * i + 3u, (h.v[k].w - m.mean) * m.scale * bf16x2_hi(w.y));
    }
  }
}

// One block per row.
template <class X>
__global__ void __launch_bounds__(kNormThreads) stream_norm_kernel(StreamNormParams p) {
  __shared__ float scratch[40];
  pdl_trigger();
  pdl_wait();
  const uint32_t source = p.row_index != nullptr ? p.row_index[blockIdx.x] : blockIdx.x;
  float *row = p.h + static_cast<uint64_t>(source) * p.padded;
  if (p.layer_norm != 0 && p.step == nullptr && p.first == nullptr && p.padded <= 4u * kNormRegIters * kNormThreads) {
    norm_in_registers<X>(p, row, source);
    return;
  }
  if (p.step != nullptr) {
    for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
      float4 v = *reinterpret_cast<const float4 *>(row + i);
      const uint2 s = *reinterpret_cast<const uint2 *>(p.step + i);
      v.x += bf16x2_lo(s.x);
      v.y += bf16x2_hi(s.x);
      v.z += bf16x2_lo(s.y);
      v.w += bf16x2_hi(s.y);
      *reinterpret_cast<float4 *>(row + i) = v;  // read back below by the same thread
    }
  }
  if (p.pending != nullptr) {
    const float *y = p.pending + static_cast<uint64_t>(source) * p.padded;
    const NormMoments m = row_moments(y, p, scratch);
    for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
      float4 v = *reinterpret_cast<const float4 *>(row + i);
      const float4 u = *reinterpret_cast<const float4 *>(y + i);
      const uint2 w = *reinterpret_cast<const uint2 *>(p.after + i);
      v.x += (u.x - m.mean) * m.scale * bf16x2_lo(w.x);
      v.y += (u.y - m.mean) * m.scale * bf16x2_hi(w.x);
      v.z += (u.z - m.mean) * m.scale * bf16x2_lo(w.y);
      v.w += (u.w - m.mean) * m.scale * bf16x2_hi(w.y);
      *reinterpret_cast<float4 *>(row + i) = v;
    }
  }
  if (p.x == nullptr) return;
  if (p.first != nullptr) {
    X *out = reinterpret_cast<X *>(p.x) + static_cast<uint64_t>(blockIdx.x) * 2u * p.padded;
    const float *first = p.first + static_cast<uint64_t>(source) * p.padded;
    for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
      const float4 v = *reinterpret_cast<const float4 *>(row + i);
      const float4 f = *reinterpret_cast<const float4 *>(first + i);
      const float a[4] = {v.x, v.y, v.z, v.w}, b[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
      for (uint32_t j = 0; j < 4u; ++j) {
        store_act(out + i + j, a[j]);
        store_act(out + p.padded + i + j, b[j]);
      }
    }
    return;
  }
  X *out = reinterpret_cast<X *>(p.x) + static_cast<uint64_t>(blockIdx.x) * p.padded;
  const NormMoments m = row_moments(row, p, scratch);
  for (uint32_t i = threadIdx.x * 4u; i < p.padded; i += kNormThreads * 4u) {
    const float4 v = *reinterpret_cast<const float4 *>(row + i);
    const uint2 w = *reinterpret_cast<const uint2 *>(p.norm + i);
    store_act(out + i, (v.x - m.mean) * m.scale * bf16x2_lo(w.x));
    store_act(out + i + 1u, (v.y - m.mean) * m.scale * bf16x2_hi(w.x));
    store_act(out + i + 2u, (v.z - m.mean) * m.scale * bf16x2_lo(w.y));
    store_act(out + i + 3u, (v.w - m.mean) * m.scale * bf16x2_hi(w.y));
  }
}

typedef void (*StreamKernel)(ParallelProjectionParams);
StreamKernel stream_kernel(uint32_t kind) {
  switch (kind) {
    case kParallelIn: return parallel_stream_kernel<kParallelIn>;
    case kParallelOut: return parallel_stream_kernel<kParallelOut>;
    case kParallelHead: return parallel_stream_kernel<kParallelHead>;
    case kParallelGate: return parallel_stream_kernel<kParallelGate>;
    case kSandwichIn: return parallel_stream_kernel<kSandwichIn>;
    case kSandwichGate: return parallel_stream_kernel<kSandwichGate>;
    case kSandwichHead: return parallel_stream_kernel<kSandwichHead>;
    case kSandwichOut: return parallel_stream_kernel<kSandwichOut>;
    case kSandwichJoin: return parallel_stream_kernel<kSandwichJoin>;
    default: return nullptr;
  }
}

}  // namespace

cudaError_t configure_parallel_projection() {
  cudaError_t err = cudaSuccess;
  for (uint32_t kind = 0; err == cudaSuccess && kind < kProjectionKinds; ++kind)
    err = cudaFuncSetAttribute(stream_kernel(kind), cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
  return err;
}

bool parallel_stream_eligible(uint32_t kind, const ParallelProjectionParams &p, uint32_t sm_count) {
  auto aligned = [](const void *q) { return reinterpret_cast<uintptr_t>(q) % 16u == 0; };
  auto vector_aligned = [](const void *q) { return reinterpret_cast<uintptr_t>(q) % 8u == 0; };
  constexpr uint32_t kMaxNormCols = 4u * kNormRegIters * kStreamThreads;
  if (kind >= kProjectionKinds || p.cols0 == 0 || p.cols0 % 8u != 0) return false;
  if (gate_pairs(kind) ? p.rows1 == 0 || p.rows1 % 2u != 0 || !aligned(p.w1) : p.rows0 == 0 || !aligned(p.w0))
    return false;
  if (kind == kParallelOut && p.rows1 != 0 && (!aligned(p.w1) || p.cols1 % 8u != 0)) return false;
  if (kind == kParallelOut) {
    if (!aligned(p.x0) || (p.rows1 != 0 && (!aligned(p.x1) || p.rows1 != p.rows0))) return false;
  } else if (kind == kSandwichOut) {
    if (p.groups == 0 ? !aligned(p.x0)
                      : p.width % (p.groups * kGroupChunk) != 0 || p.cols0 > kMaxNormCols || !aligned(p.x_f32) ||
                            !vector_aligned(p.norm))
      return false;
  } else {
    const uint32_t cols = kind == kSandwichJoin ? p.cols0 / 2u : p.cols0;
    if (cols > kMaxNormCols || cols % 8u != 0 || !aligned(p.h) || !vector_aligned(p.norm) || !vector_aligned(p.step))
      return false;
    if (!aligned(p.pending) || !vector_aligned(p.after) || !aligned(p.first) ||
        (p.pending != nullptr && (p.after == nullptr || (kind != kSandwichJoin && (!aligned(p.h_out) || p.h_out == p.h)))))
      return false;
  }
  return stream_smem_bytes(kind, p, stream_blocks(kind, p, sm_count)) <= 227u * 1024u;
}

uint32_t parallel_stream_blocks(uint32_t kind, const ParallelProjectionParams &p, uint32_t sm_count) {
  return stream_blocks(kind, p, sm_count);
}

cudaError_t launch_parallel_projection(cudaStream_t stream, uint32_t kind, const ParallelProjectionParams &p,
                                       uint32_t sm_count) {
  if (!parallel_stream_eligible(kind, p, sm_count)) return cudaErrorInvalidValue;
  const uint32_t blocks = stream_blocks(kind, p, sm_count);
  return launch_with_pdl(stream_kernel(kind), dim3(blocks), dim3(kStreamThreads), stream_smem_bytes(kind, p, blocks), stream,
                         p.pdl != 0, p);
}

cudaError_t launch_parallel_projection_plain(cudaStream_t stream, uint32_t kind, const ParallelProjectionParams &p,
                                             uint32_t tokens, bool f32) {
  const uint32_t units = p.rows0 + (kind == kParallelIn ? p.rows1 / 2u : 0u);
  if (tokens == 0 || kind > kParallelHead || units == 0 || p.cols0 % 64u != 0 || p.cols1 % 64u != 0) return cudaErrorInvalidValue;
  const dim3 grid((units + kPlainWarps - 1u) / kPlainWarps, (tokens + kPlainTokens - 1u) / kPlainTokens);
  void (*kernel)(ParallelProjectionParams, uint32_t);
  if (f32)
    kernel = kind == kParallelIn    ? parallel_plain_kernel<float, kParallelIn>
             : kind == kParallelOut ? parallel_plain_kernel<float, kParallelOut>
                                    : parallel_plain_kernel<float, kParallelHead>;
  else
    kernel = kind == kParallelIn    ? parallel_plain_kernel<uint16_t, kParallelIn>
             : kind == kParallelOut ? parallel_plain_kernel<uint16_t, kParallelOut>
                                    : parallel_plain_kernel<uint16_t, kParallelHead>;
  return launch_with_pdl(kernel, grid, dim3(kPlainWarps * 32), 0, stream, p.pdl != 0, p, tokens);
}

cudaError_t launch_stream_norm(cudaStream_t stream, const StreamNormParams &p, bool f32, uint32_t rows, bool pdl) {
  if (rows == 0 || p.padded % 4u != 0 || (p.row_index != nullptr && (p.step != nullptr || p.pending != nullptr)))
    return cudaErrorInvalidValue;
  return launch_with_pdl(f32 ? stream_norm_kernel<float> : stream_norm_kernel<uint16_t>, dim3(rows), dim3(kNormThreads), 0,
                         stream, pdl, p);
}

}  // namespace nb
