// Selective state-space mixer: causal convolution per channel, then per head a state S [state][v_dim] with
//   S <- exp(-exp(a_log) d) S + d B x^T,   y = S^T C + skip x,   d = softplus(step + bias),
// and y * silu(z).  State, decays and step sizes are fp32 everywhere.
//
//   state_space_step_kernel  one token per row (the lone step, or rows of different sessions).  A block
//                            owns 32 value columns of a head, its share of the state in registers, and
//                            does the convolution of the channels it needs.  State and history are
//                            requested before the dependency wait: the step before this one wrote them.
//   state_space_conv_kernel  convolution and silu of a block of consecutive positions of one session,
//                            heads and groups padded to 16 elements.
//   state_space_rows_kernel  the recurrence over such a block, token by token, state in registers: fp32
//                            sessions and blocks of a few tokens.
//   state_space_scan_kernel  the same on the tensor pipe (mma.sync) in chunks of 64 tokens.  With L the
//                            running sum of -exp(a_log) d inside the chunk,
//                              y_t = exp(L_t) S^T C_t + sum over s <= t of (C_t . B_s) exp(L_t - L_s) d_s x_s
//                              S  <- exp(L_end) S + sum over s of B_s (exp(L_end - L_s) d_s x_s)^T
//                            The state stays in fp32 accumulators from chunk to chunk.  Where an fp32
//                            factor (state, weights, scaled x) meets the convolved bf16 values it enters
//                            as a bf16 rounding plus its remainder.
//   grouped_norm_kernel      RMS norm of a row in equal parts, in front of the output projection.
#include "common.cuh"
#include "kernels.cuh"
#include "mma_bf16.cuh"

namespace nb {
namespace {

constexpr uint32_t kMaxTaps = 16;
constexpr uint32_t kMaxState = 256;
constexpr uint32_t kColumns = 32;  // value columns of a block
constexpr uint32_t kStepThreads = 256;
constexpr uint32_t kStepWarps = kStepThreads / 32;

// ---------------------------------------------------------------- one token per row ----
// A thread holds four neighbouring columns of state rows r, r + 32, ...: eight threads span a block's 32
// columns.  ROWS_PER: rows a thread holds.  VECTOR: v_dim is a multiple of 4, so that the four columns are
// one 16-byte access.
template <uint32_t ROWS_PER, bool VECTOR>
__global__ void __launch_bounds__(kStepThreads) state_space_step_kernel(StateSpaceParams p) {
  constexpr uint32_t kRowStep = kStepThreads / 8u;
  constexpr uint32_t kMaxValues = kColumns + 2u * kRowStep * ROWS_PER;
  constexpr uint32_t kChannels = (kMaxValues + kStepThreads - 1u) / kStepThreads;
  __shared__ __align__(16) float values[kMaxValues];  // x | B | C behind convolution and silu
  __shared__ __align__(16) float part[kStepWarps][kColumns];
  const StateSpaceShape &s = p.s;
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
  const uint32_t tiles = (s.v_dim + kColumns - 1u) / kColumns;
  const uint32_t head = blockIdx.x / tiles, column0 = (blockIdx.x - head * tiles) * kColumns;
  const uint32_t group = head / (s.heads / s.groups);
  const bool several = p.rows != nullptr;
  pdl_trigger();
  uint32_t position, max_context;
  float *recurrent;
  if (several) {
    const FusedAttentionRow &r = p.rows[blockIdx.y];
    position = r.position;
    max_context = r.max_context;
    recurrent = r.recurrent;
  } else {
    position = *p.cursor;  // changes in the last kernel of a step only
    max_context = p.max_context;
    recurrent = p.recurrent;
  }
  if (position >= max_context) {
    pdl_wait();
    return;
  }
  const uint32_t quad = 4u * (threadIdx.x & 7u), row0 = threadIdx.x >> 3;  // columns column0 + quad .. + 3
  float *state = recurrent + p.state_offset + static_cast<uint64_t>(head) * s.state * s.v_dim + column0 + quad;
  float held[ROWS_PER][4];
#pragma unroll
  for (uint32_t i = 0; i < ROWS_PER; ++i) {
    const uint32_t n = row0 + i * kRowStep;
    const float *src = state + static_cast<uint64_t>(n) * s.v_dim;
#pragma unroll
    for (uint32_t j = 0; j < 4u; ++j) held[i][j] = 0.0f;
    if (n < s.state && position != 0) {
      if (VECTOR) {
        if (column0 + quad < s.v_dim) {
          const float4 v = __ldcg(reinterpret_cast<const float4 *>(src));
          held[i][0] = v.x;
          held[i][1] = v.y;
          held[i][2] = v.z;
          held[i][3] = v.w;
        }
      } else {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j)
          if (column0 + quad + j < s.v_dim) held[i][j] = __ldcg(src + j);
      }
    }
  }

  // the convolution of this block's x columns and of its group's B and C
  const uint32_t inner = s.inner(), channels = s.channels(), shared = s.groups * s.state;
  float *history = recurrent + p.history_offset;
  const float *in = p.in + static_cast<uint64_t>(blockIdx.y) * p.in_stride;
  const uint32_t wanted = kColumns + 2u * s.state;
  auto channel_of = [&](uint32_t i) {  // channels: none
    if (i >= wanted) return channels;
    if (i < kColumns) return column0 + i < s.v_dim ? head * s.v_dim + column0 + i : channels;
    const uint32_t n = i - kColumns;
    return n < s.state ? inner + group * s.state + n : inner + shared + group * s.state + (n - s.state);
  };
  const uint32_t column = column0 + lane;
  const bool live = column < s.v_dim;
  float sum[kChannels], newest[kChannels], u[kChannels], step_in = 0.0f, z = 0.0f;
  auto load_inputs = [&]() {
#pragma unroll
    for (uint32_t k = 0; k < kChannels; ++k) {
      const uint32_t ch = channel_of(threadIdx.x + k * kStepThreads);
      u[k] = ch < channels ? __ldcg(in + inner + ch) : 0.0f;
    }
    step_in = __ldcg(in + inner + channels + head);
    if (live && warp == 0) z = __ldcg(in + head * s.v_dim + column);
  };
  // Alone, what the earlier tokens left is summed while the projection still runs.  With many rows most blocks
  // start after it has ended, and all loads travel together.
  if (several) {
    pdl_wait();
    load_inputs();
  }
#pragma unroll
  for (uint32_t k = 0; k < kChannels; ++k) {
    const uint32_t ch = channel_of(threadIdx.x + k * kStepThreads);
    sum[k] = newest[k] = 0.0f;
    if (ch < channels) {
      const uint16_t *w = p.conv + static_cast<uint64_t>(ch) * s.taps;
      sum[k] = bf16_bits_to_f32(p.conv_bias[ch]);
      newest[k] = bf16_bits_to_f32(w[s.taps - 1u]);
#pragma unroll 3
      for (uint32_t back = 1; back < s.taps; ++back) {
        if (back <= position)
          sum[k] = fmaf(bf16_bits_to_f32(w[s.taps - 1u - back]),
                        __ldcg(history + static_cast<uint64_t>((position - back) % s.taps) * channels + ch), sum[k]);
      }
    }
  }
  const float rate = expf(bf16_bits_to_f32(p.a_log[head])), bias = bf16_bits_to_f32(p.step_bias[head]);
  const float skip = bf16_bits_to_f32(p.skip[head]);
  if (!several) {
    pdl_wait();
    load_inputs();
  }

  const bool owns_shared = column0 == 0 && head % (s.heads / s.groups) == 0;
#pragma unroll
  for (uint32_t k = 0; k < kChannels; ++k) {
    const uint32_t i = threadIdx.x + k * kStepThreads, ch = channel_of(i);
    if (i < wanted) values[i] = ch < channels ? silu(fmaf(newest[k], u[k], sum[k])) : 0.0f;
    if (ch < channels && (i < kColumns || owns_shared)) history[static_cast<uint64_t>(position % s.taps) * channels + ch] = u[k];
  }
  const float step = softplus(step_in + bias);
  const float decay = expf(-rate * step);
  __syncthreads();
  const float4 x4 = *reinterpret_cast<const float4 *>(values + quad);
  const float fed[4] = {step * x4.x, step * x4.y, step * x4.z, step * x4.w};
  const float *b = values + kColumns, *c = b + s.state;
  float y[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
  for (uint32_t i = 0; i < ROWS_PER; ++i) {
    const uint32_t n = row0 + i * kRowStep;
    if (n < s.state) {
      const float bn = b[n], cn = c[n];
#pragma unroll
      for (uint32_t j = 0; j < 4u; ++j) {
        held[i][j] = fmaf(decay, held[i][j], fed[j] * bn);
        y[j] = fmaf(held[i][j], cn, y[j]);
      }
      float *dst = state + static_cast<uint64_t>(n) * s.v_dim;
      if (VECTOR) {
        if (column0 + quad < s.v_dim)
          *reinterpret_cast<float4 *>(dst) = make_float4(held[i][0], held[i][1], held[i][2], held[i][3]);
      } else {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j)
          if (column0 + quad + j < s.v_dim) dst[j] = held[i][j];
      }
    }
  }
#pragma unroll
  for (uint32_t j = 0; j < 4u; ++j) {  // the warp's four rows
    y[j] += __shfl_xor_sync(0xffffffffu, y[j], 8);
    y[j] += __shfl_xor_sync(0xffffffffu, y[j], 16);
  }
  if (lane < 8u) *reinterpret_cast<float4 *>(&part[warp][quad]) = make_float4(y[0], y[1], y[2], y[3]);
  __syncthreads();
  if (warp != 0 || !live) return;
  float total = skip * values[lane];
#pragma unroll
  for (uint32_t w = 0; w < kStepWarps; ++w) total += part[w][lane];
  p.out[static_cast<uint64_t>(blockIdx.y) * p.out_stride + head * s.v_dim + column] = total * silu(z);
}

// ---------------------------------------------------------------- a block of one session ----
__device__ __forceinline__ void put(float *dst, float v) { *dst = v; }
__device__ __forceinline__ void put(uint16_t *dst, float v) { *dst = f32_to_bf16_bits(v); }
__device__ __forceinline__ float get(const float *src) { return __ldcg(src); }
__device__ __forceinline__ float get(const uint16_t *src) { return bf16_bits_to_f32(__ldcg(src)); }

constexpr uint32_t kConvThreads = 128, kConvRows = 16;

// Channel of column j of a convolved row; channels(): padding.
__device__ __forceinline__ uint32_t padded_channel(const StateSpaceShape &s, uint32_t j) {
  const uint32_t v_pad = s.v_pad(), n_pad = s.state_pad(), x_width = s.heads * v_pad;
  if (j < x_width) {
    const uint32_t head = j / v_pad, e = j - head * v_pad;
    return e < s.v_dim ? head * s.v_dim + e : s.channels();
  }
  const uint32_t g = (j - x_width) / n_pad, e = (j - x_width) - g * n_pad;  // B groups, then C groups
  return e < s.state ? s.inner() + g * s.state + e : s.channels();
}

// Grid (columns / 128, rows / 16): a thread slides one channel over its rows.  TAPS: of the registers.
template <class T, uint32_t TAPS>
__global__ void __launch_bounds__(kConvThreads) state_space_conv_kernel(StateSpaceParams p) {
  const StateSpaceShape &s = p.s;
  pdl_trigger();
  const uint32_t width = s.conv_width(), j = blockIdx.x * kConvThreads + threadIdx.x;
  const uint32_t row0 = blockIdx.y * kConvRows;
  const uint32_t row_end = row0 + kConvRows < p.row_count ? row0 + kConvRows : p.row_count;
  const FusedAttentionRow &r0 = p.rows[0];
  const uint32_t base = r0.position;
  const bool fits = base + row_end <= r0.max_context;
  const uint32_t channels = s.channels(), ch = j < width ? padded_channel(s, j) : channels;
  float w[TAPS], u[TAPS];  // w[k] meets the input k positions back, u[k] holds it
  float bias = 0.0f;
#pragma unroll
  for (uint32_t k = 0; k < TAPS; ++k) w[k] = u[k] = 0.0f;
  if (ch < channels) {
    bias = bf16_bits_to_f32(p.conv_bias[ch]);
#pragma unroll
    for (uint32_t k = 0; k < TAPS; ++k)
      if (k < s.taps) w[k] = bf16_bits_to_f32(p.conv[static_cast<uint64_t>(ch) * s.taps + s.taps - 1u - k]);
  }
  pdl_wait();
  if (j >= width || !fits) return;
  T *out = reinterpret_cast<T *>(p.convolved) + j;
  if (ch == channels) {
    for (uint32_t r = row0; r < row_end; ++r) put(out + static_cast<uint64_t>(r) * width, 0.0f);
    return;
  }
  const float *in = p.in + s.inner() + ch;
  const float *history = r0.recurrent + p.history_offset + ch;
#pragma unroll
  for (uint32_t k = 1; k < TAPS; ++k) {  // the inputs in front of row0
    if (k < s.taps && base + row0 >= k)
      u[k - 1u] = row0 >= k ? __ldcg(in + static_cast<uint64_t>(row0 - k) * p.in_stride)
                            : __ldcg(history + static_cast<uint64_t>((base + row0 - k) % s.taps) * channels);
  }
  for (uint32_t r = row0; r < row_end; ++r) {
#pragma unroll
    for (uint32_t k = TAPS - 1u; k > 0; --k) u[k] = u[k - 1u];
    u[0] = __ldcg(in + static_cast<uint64_t>(r) * p.in_stride);
    float v = bias;
#pragma unroll
    for (uint32_t k = 0; k < TAPS; ++k) v = fmaf(w[k], u[k], v);
    put(out + static_cast<uint64_t>(r) * width, silu(v));
  }
}

// The last inputs of a block into the convolution's ring: this block's x columns, and B and C of its group
// when it is the group's first.  The convolution of the block is complete.
__device__ __forceinline__ void keep_history(const StateSpaceParams &p, float *recurrent, uint32_t base, uint32_t head,
                                             uint32_t column0) {
  const StateSpaceShape &s = p.s;
  const uint32_t channels = s.channels(), inner = s.inner(), shared = s.groups * s.state;
  const uint32_t per_group = s.heads / s.groups, group = head / per_group;
  const uint32_t wanted = kColumns + (column0 == 0 && head % per_group == 0 ? 2u * s.state : 0u);
  const uint32_t kept = s.taps - 1u < p.row_count ? s.taps - 1u : p.row_count;
  for (uint32_t i = threadIdx.x; i < wanted; i += blockDim.x) {
    uint32_t ch;
    if (i < kColumns) {
      if (column0 + i >= s.v_dim) continue;
      ch = head * s.v_dim + column0 + i;
    } else {
      const uint32_t n = i - kColumns;
      ch = n < s.state ? inner + group * s.state + n : inner + shared + group * s.state + (n - s.state);
    }
    for (uint32_t r = p.row_count - kept; r < p.row_count; ++r)
      recurrent[p.history_offset + static_cast<uint64_t>((base + r) % s.taps) * channels + ch] =
          __ldcg(p.in + static_cast<uint64_t>(r) * p.in_stride + inner + ch);
  }
}

template <class T, uint32_t ROWS_PER>
__global__ void __launch_bounds__(kStepThreads) state_space_rows_kernel(StateSpaceParams p) {
  constexpr uint32_t kWanted = kColumns + 2u * kStepWarps * ROWS_PER;
  constexpr uint32_t kValues = (kWanted + kStepThreads - 1u) / kStepThreads;
  __shared__ float values[2][kWanted];  // x | B | C of a row
  __shared__ float part[2][kStepWarps][kColumns];
  const StateSpaceShape &s = p.s;
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
  const uint32_t tiles = (s.v_dim + kColumns - 1u) / kColumns;
  const uint32_t head = blockIdx.x / tiles, column0 = (blockIdx.x - head * tiles) * kColumns;
  const uint32_t group = head / (s.heads / s.groups);
  pdl_trigger();
  const FusedAttentionRow &r0 = p.rows[0];
  const uint32_t base = r0.position;
  const uint32_t column = column0 + lane;
  const bool live = column < s.v_dim;
  float *state = r0.recurrent + p.state_offset + static_cast<uint64_t>(head) * s.state * s.v_dim + column;
  float held[ROWS_PER];
#pragma unroll
  for (uint32_t i = 0; i < ROWS_PER; ++i) {  // written by an earlier block step
    const uint32_t n = warp + i * kStepWarps;
    held[i] = live && n < s.state && base != 0 ? __ldcg(state + static_cast<uint64_t>(n) * s.v_dim) : 0.0f;
  }
  const float rate = expf(bf16_bits_to_f32(p.a_log[head])), bias = bf16_bits_to_f32(p.step_bias[head]);
  const float skip = bf16_bits_to_f32(p.skip[head]);
  pdl_wait();
  if (base + p.row_count > r0.max_context) return;

  const uint32_t width = s.conv_width(), x_width = s.heads * s.v_pad(), n_pad = s.state_pad();
  const T *convolved = reinterpret_cast<const T *>(p.convolved);
  const uint32_t wanted = kColumns + 2u * s.state;
  float next[kValues], next_step = 0.0f, next_z = 0.0f;
  auto fetch = [&](uint32_t r) {
    const T *row = convolved + static_cast<uint64_t>(r) * width;
    const float *in = p.in + static_cast<uint64_t>(r) * p.in_stride;
#pragma unroll
    for (uint32_t k = 0; k < kValues; ++k) {
      const uint32_t i = threadIdx.x + k * kStepThreads;
      next[k] = 0.0f;
      if (i < kColumns) {
        if (column0 + i < s.v_dim) next[k] = get(row + head * s.v_pad() + column0 + i);
      } else if (i < wanted) {
        const uint32_t n = i - kColumns;
        next[k] = n < s.state ? get(row + x_width + group * n_pad + n)
                              : get(row + x_width + (s.groups + group) * n_pad + (n - s.state));
      }
    }
    next_step = __ldcg(in + s.inner() + s.channels() + head);
    if (warp == 0 && live) next_z = __ldcg(in + head * s.v_dim + column);
  };
  fetch(0);
  for (uint32_t r = 0; r < p.row_count; ++r) {
    const uint32_t stage = r & 1u;
#pragma unroll
    for (uint32_t k = 0; k < kValues; ++k) {
      const uint32_t i = threadIdx.x + k * kStepThreads;
      if (i < wanted) values[stage][i] = next[k];
    }
    const float step = softplus(next_step + bias), z = next_z;
    const float decay = expf(-rate * step);
    __syncthreads();
    if (r + 1u < p.row_count) fetch(r + 1u);
    const float x = values[stage][lane], fed = step * x;
    const float *b = values[stage] + kColumns, *c = b + s.state;
    float y = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < ROWS_PER; ++i) {
      const uint32_t n = warp + i * kStepWarps;
      if (n < s.state) {
        held[i] = fmaf(decay, held[i], fed * b[n]);
        y = fmaf(held[i], c[n], y);
      }
    }
    part[stage][warp][lane] = y;
    __syncthreads();
    if (warp == 0 && live) {
      y = skip * x;
#pragma unroll
      for (uint32_t w = 0; w < kStepWarps; ++w) y += part[stage][w][lane];
      p.out[static_cast<uint64_t>(r) * p.out_stride + head * s.v_dim + column] = y * silu(z);
    }
  }
#pragma unroll
  for (uint32_t i = 0; i < ROWS_PER; ++i) {
    const uint32_t n = warp + i * kStepWarps;
    if (live && n < s.state) state[static_cast<uint64_t>(n) * s.v_dim] = held[i];
  }
  keep_history(p, r0.recurrent, base, head, column0);
}

// ------------------------------------------------------------------ chunks on the tensor pipe ----
constexpr uint32_t kChunk = 64;
constexpr uint32_t kScanThreads = 256;
constexpr uint32_t kScanWarps = kScanThreads / 32u;
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kScanMaxRows = 256;  // rows of a block

__device__ __forceinline__ void cp_async_16(void *dst, const void *src, bool valid) {  // zeros when not valid
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(valid ? 16u : 0u)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

struct ScanLayout {  // bytes; rows are an odd number of 16-byte pieces apart (ldmatrix without bank conflicts)
  uint32_t n_row, x_row, stage, fed, states, total;
  __host__ __device__ explicit ScanLayout(const StateSpaceShape &s) {
    n_row = s.state_pad() * 2u + 16u;
    x_row = kColumns * 2u + 16u;
    stage = kChunk * (2u * n_row + x_row);  // B | C | x
    fed = kChunk * x_row;                   // scaled x, one part
    states = s.state_pad() * x_row;         // state, one part
    total = 2u * stage + 2u * fed + 2u * states;
  }
};

// Grid (value columns / 32, heads).  MT: m-tiles of 16 state rows a warp holds (state <= 128 MT).  Outputs: warps
// 0..3 take 16 columns of the token tiles 0..3, warps 4..7 the other 16 columns of the tiles 3..0, so that the
// two warps of an SM partition share the triangle of earlier tokens evenly.
template <uint32_t MT>
__global__ void __launch_bounds__(kScanThreads) state_space_scan_kernel(StateSpaceParams p) {
  constexpr uint32_t NT = kColumns / 8u, YT = NT / 2u;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float log_decay_all[kScanMaxRows], steps_all[kScanMaxRows], to_end_all[kScanMaxRows];
  const StateSpaceShape &s = p.s;
  const ScanLayout L(s);
  uint8_t *fed_hi = smem + 2u * L.stage, *fed_lo = fed_hi + L.fed;
  uint8_t *state_hi = fed_lo + L.fed, *state_lo = state_hi + L.states;
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3u;
  const uint32_t token_tile = warp < 4u ? warp : kScanWarps - 1u - warp, y_first = warp < 4u ? 0u : kColumns / 2u;
  const uint32_t head = blockIdx.y, column0 = blockIdx.x * kColumns;
  const uint32_t group = head / (s.heads / s.groups);
  const uint32_t n_pad = s.state_pad(), m_tiles = n_pad / 16u;
  pdl_trigger();
  const FusedAttentionRow &r0 = p.rows[0];
  const uint32_t base = r0.position;
  float *state = r0.recurrent + p.state_offset + static_cast<uint64_t>(head) * s.state * s.v_dim + column0;
  // held[m][n]: state rows 16 (warp + 8 m) + g (+ 8), columns 8 n + 2 t (+ 1); written by an earlier block step
  float held[MT][NT][4];
#pragma unroll
  for (uint32_t m = 0; m < MT; ++m) {
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
#pragma unroll
      for (uint32_t j = 0; j < 4u; ++j) {
        const uint32_t row = 16u * (warp + kScanWarps * m) + g + 8u * (j >> 1), col = 8u * n + 2u * t4 + (j & 1u);
        held[m][n][j] = base != 0 && row < s.state && column0 + col < s.v_dim
                            ? __ldcg(state + static_cast<uint64_t>(row) * s.v_dim + col)
                            : 0.0f;
      }
    }
  }
  const float rate = kLog2e * expf(bf16_bits_to_f32(p.a_log[head]));  // decays are powers of two here
  const float bias = bf16_bits_to_f32(p.step_bias[head]), skip = bf16_bits_to_f32(p.skip[head]);
  pdl_wait();
  if (base + p.row_count > r0.max_context) return;

  const uint32_t width = s.conv_width(), x_width = s.heads * s.v_pad();
  const uint16_t *convolved = reinterpret_cast<const uint16_t *>(p.convolved);
  const uint16_t *x_src = convolved + head * s.v_pad() + column0;
  const uint16_t *b_src = convolved + x_width + group * n_pad, *c_src = b_src + s.groups * n_pad;
  const uint32_t n_pieces = n_pad / 8u, x_pieces = kColumns / 8u;
  const uint32_t x_valid = (s.v_pad() - column0 < kColumns ? s.v_pad() - column0 : kColumns) / 8u;  // pieces inside the head
  const uint32_t pieces = 2u * n_pieces + x_pieces;
  auto issue = [&](uint32_t chunk) {  // one commit group per chunk
    uint8_t *b = smem + (chunk & 1u) * L.stage, *c = b + kChunk * L.n_row, *x = c + kChunk * L.n_row;
    const uint32_t first = chunk * kChunk;
    // a lane takes one 16-byte piece of the B, C or x row of every eighth token
    for (uint32_t piece = lane; piece < pieces; piece += 32u) {
      const uint16_t *src = b_src + piece * 8u;
      uint8_t *dst = b + piece * 16u;
      uint32_t dst_step = L.n_row;
      bool used = true;
      if (piece >= 2u * n_pieces) {
        const uint32_t e = piece - 2u * n_pieces;
        used = e < x_valid;
        src = x_src + (used ? e * 8u : 0u);
        dst = x + e * 16u;
        dst_step = L.x_row;
      } else if (piece >= n_pieces) {
        src = c_src + (piece - n_pieces) * 8u;
        dst = c + (piece - n_pieces) * 16u;
      }
#pragma unroll
      for (uint32_t t = warp; t < kChunk; t += kScanWarps) {
        const bool inside = first + t < p.row_count;
        cp_async_16(dst + t * dst_step, src + static_cast<uint64_t>(inside ? first + t : 0u) * width, inside && used);
      }
    }
    cp_async_commit();
  };
  // fragment offsets: A operand rows, B operand rows stored [n][k], B operand stored [k][n], A operand stored [k][m]
  const uint32_t a_row = (lane & 7u) + 8u * ((lane >> 3) & 1u), a_off = (lane >> 4) * 16u;
  const uint32_t nk_row = (lane & 7u) + 8u * (lane >> 4), nk_off = ((lane >> 3) & 1u) * 16u;
  const uint32_t kn_row = a_row, kn_off = a_off;
  const uint32_t km_row = nk_row, km_off = nk_off;

  const uint32_t chunks = (p.row_count + kChunk - 1u) / kChunk;
  issue(0);
  for (uint32_t chunk = warp; chunk < chunks; chunk += kScanWarps) {
    // step sizes and their running sums, a chunk per warp: tokens 2 lane, 2 lane + 1; rows behind the block change nothing
    float d[2], sum[2];
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      const uint32_t r = chunk * kChunk + 2u * lane + i;
      d[i] = r < p.row_count
                 ? softplus(__ldcg(p.in + static_cast<uint64_t>(r) * p.in_stride + s.inner() + s.channels() + head) + bias)
                 : 0.0f;
    }
    sum[0] = d[0];
    sum[1] = d[0] + d[1];
    float through = sum[1], from = sum[1];  // sums up to and from this lane's tokens
#pragma unroll
    for (uint32_t o = 1; o < 32u; o <<= 1) {
      const float left = __shfl_up_sync(0xffffffffu, through, o), right = __shfl_down_sync(0xffffffffu, from, o);
      if (lane >= o) through += left;
      if (lane + o < 32u) from += right;
    }
    float before = __shfl_up_sync(0xffffffffu, through, 1), behind = __shfl_down_sync(0xffffffffu, from, 1);
    if (lane == 0) before = 0.0f;
    if (lane == 31) behind = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      const uint32_t t = chunk * kChunk + 2u * lane + i;
      steps_all[t] = d[i];
      log_decay_all[t] = -rate * (before + sum[i]);
      // not a difference of the running sums: the last token's factor is exactly one
      to_end_all[t] = exp2f(-rate * (i == 0 ? behind + d[1] : behind)) * d[i];
    }
  }
  for (uint32_t chunk = 0; chunk < chunks; ++chunk) {
    const uint32_t first = chunk * kChunk;
    const float *log_decay = log_decay_all + first, *steps = steps_all + first, *to_end = to_end_all + first;
    cp_async_wait<0>();
    __syncthreads();  // this chunk's rows and steps are in place; the other stage is free
    if (chunk + 1u < chunks) issue(chunk + 1u);
    uint8_t *b_sh = smem + (chunk & 1u) * L.stage, *c_sh = b_sh + kChunk * L.n_row, *x_sh = c_sh + kChunk * L.n_row;

    // z of this thread's outputs, on its way while the products run
    float z[2][YT][2];
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      const uint32_t r = first + 16u * token_tile + g + 8u * i;
#pragma unroll
      for (uint32_t n = 0; n < YT; ++n) {
#pragma unroll
        for (uint32_t j = 0; j < 2u; ++j) {
          const uint32_t col = column0 + y_first + 8u * n + 2u * t4 + j;
          z[i][n][j] = r < p.row_count && col < s.v_dim
                           ? __ldcg(p.in + static_cast<uint64_t>(r) * p.in_stride + head * s.v_dim + col)
                           : 0.0f;
        }
      }
    }
    // state at the chunk's start and x scaled for its end, both as two bf16 parts
#pragma unroll
    for (uint32_t m = 0; m < MT; ++m) {
      const uint32_t tile = warp + kScanWarps * m;
      if (tile < m_tiles) {
#pragma unroll
        for (uint32_t n = 0; n < NT; ++n) {
#pragma unroll
          for (uint32_t i = 0; i < 2u; ++i) {
            const uint32_t at = (16u * tile + g + 8u * i) * L.x_row + (8u * n + 2u * t4) * 2u;
            *reinterpret_cast<uint32_t *>(state_hi + at) = pack_bf16_hi(held[m][n][2u * i], held[m][n][2u * i + 1u]);
            *reinterpret_cast<uint32_t *>(state_lo + at) = pack_bf16_lo(held[m][n][2u * i], held[m][n][2u * i + 1u]);
          }
        }
      }
    }
    for (uint32_t i = threadIdx.x; i < kChunk * (kColumns / 2u); i += kScanThreads) {
      const uint32_t t = i / (kColumns / 2u), at = t * L.x_row + (i - t * (kColumns / 2u)) * 4u;
      const uint32_t x = *reinterpret_cast<const uint32_t *>(x_sh + at);
      const float u = bf16x2_lo(x) * to_end[t], v = bf16x2_hi(x) * to_end[t];
      *reinterpret_cast<uint32_t *>(fed_hi + at) = pack_bf16_hi(u, v);
      *reinterpret_cast<uint32_t *>(fed_lo + at) = pack_bf16_lo(u, v);
    }
    __syncthreads();

    // what the state gives: rows 16 token_tile + g (+ 8) of the chunk
    float y[YT][4];
#pragma unroll
    for (uint32_t n = 0; n < YT; ++n) y[n][0] = y[n][1] = y[n][2] = y[n][3] = 0.0f;
    const uint32_t c_addr = smem_addr(c_sh) + (16u * token_tile + a_row) * L.n_row + a_off;
#pragma unroll 4
    for (uint32_t ks = 0; ks < n_pad / 16u; ++ks) {
      uint32_t ca[4], hi[4], lo[4];
      ldmatrix_x4(ca, c_addr + ks * 32u);
      const uint32_t at = (ks * 16u + kn_row) * L.x_row + y_first * 2u + kn_off;
      ldmatrix_x4_trans(hi, smem_addr(state_hi) + at);
      ldmatrix_x4_trans(lo, smem_addr(state_lo) + at);
      mma_bf16(y[0], ca, hi[0], hi[1]);
      mma_bf16(y[1], ca, hi[2], hi[3]);
      mma_bf16(y[0], ca, lo[0], lo[1]);
      mma_bf16(y[1], ca, lo[2], lo[3]);
    }
    const uint32_t row[2] = {16u * token_tile + g, 16u * token_tile + g + 8u};
    const float here[2] = {log_decay[row[0]], log_decay[row[1]]};
    const float from_start[2] = {exp2f(here[0]), exp2f(here[1])};
#pragma unroll
    for (uint32_t n = 0; n < YT; ++n) {
      y[n][0] *= from_start[0];
      y[n][1] *= from_start[0];
      y[n][2] *= from_start[1];
      y[n][3] *= from_start[1];
    }
    // what the chunk's own tokens give: 16 of them at a time, up to the diagonal
    for (uint32_t kb = 0; kb <= token_tile; ++kb) {
      float sc[2][4];
#pragma unroll
      for (uint32_t n = 0; n < 2u; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
      const uint32_t b_addr = smem_addr(b_sh) + (16u * kb + nk_row) * L.n_row + nk_off;
#pragma unroll 4
      for (uint32_t ks = 0; ks < n_pad / 16u; ++ks) {
        uint32_t ca[4], bb[4];
        ldmatrix_x4(ca, c_addr + ks * 32u);
        ldmatrix_x4(bb, b_addr + ks * 32u);
        mma_bf16(sc[0], ca, bb[0], bb[1]);
        mma_bf16(sc[1], ca, bb[2], bb[3]);
      }
#pragma unroll
      for (uint32_t n = 0; n < 2u; ++n) {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j) {
          const uint32_t from = 16u * kb + 8u * n + 2u * t4 + (j & 1u), i = j >> 1;
          sc[n][j] = from <= row[i] ? sc[n][j] * exp2f(here[i] - log_decay[from]) * steps[from] : 0.0f;
        }
      }
      const uint32_t hi[4] = {pack_bf16_hi(sc[0][0], sc[0][1]), pack_bf16_hi(sc[0][2], sc[0][3]),
                              pack_bf16_hi(sc[1][0], sc[1][1]), pack_bf16_hi(sc[1][2], sc[1][3])};
      const uint32_t lo[4] = {pack_bf16_lo(sc[0][0], sc[0][1]), pack_bf16_lo(sc[0][2], sc[0][3]),
                              pack_bf16_lo(sc[1][0], sc[1][1]), pack_bf16_lo(sc[1][2], sc[1][3])};
      uint32_t xb[4];
      ldmatrix_x4_trans(xb, smem_addr(x_sh) + (16u * kb + kn_row) * L.x_row + y_first * 2u + kn_off);
      mma_bf16(y[0], hi, xb[0], xb[1]);
      mma_bf16(y[1], hi, xb[2], xb[3]);
      mma_bf16(y[0], lo, xb[0], xb[1]);
      mma_bf16(y[1], lo, xb[2], xb[3]);
    }
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      const uint32_t r = first + row[i];
      if (r < p.row_count) {
        float *out = p.out + static_cast<uint64_t>(r) * p.out_stride + head * s.v_dim;
#pragma unroll
        for (uint32_t n = 0; n < YT; ++n) {
          const uint32_t x = *reinterpret_cast<const uint32_t *>(x_sh + row[i] * L.x_row + (y_first + 8u * n + 2u * t4) * 2u);
          const uint32_t col = column0 + y_first + 8u * n + 2u * t4;
          if (col < s.v_dim) out[col] = fmaf(skip, bf16x2_lo(x), y[n][2u * i]) * silu(z[i][n][0]);
          if (col + 1u < s.v_dim) out[col + 1u] = fmaf(skip, bf16x2_hi(x), y[n][2u * i + 1u]) * silu(z[i][n][1]);
        }
      }
    }
    // the state at the chunk's end
    const float whole = exp2f(log_decay[kChunk - 1u]);
#pragma unroll
    for (uint32_t m = 0; m < MT; ++m) {
      const uint32_t tile = warp + kScanWarps * m;
      if (tile < m_tiles) {
#pragma unroll
        for (uint32_t n = 0; n < NT; ++n) {
#pragma unroll
          for (uint32_t j = 0; j < 4u; ++j) held[m][n][j] *= whole;
        }
#pragma unroll
        for (uint32_t ks = 0; ks < kChunk / 16u; ++ks) {
          uint32_t ba[4];
          ldmatrix_x4_trans(ba, smem_addr(b_sh) + (ks * 16u + km_row) * L.n_row + tile * 32u + km_off);
#pragma unroll
          for (uint32_t np = 0; np < NT / 2u; ++np) {
            uint32_t hi[4], lo[4];
            const uint32_t at = (ks * 16u + kn_row) * L.x_row + np * 32u + kn_off;
            ldmatrix_x4_trans(hi, smem_addr(fed_hi) + at);
            ldmatrix_x4_trans(lo, smem_addr(fed_lo) + at);
            mma_bf16(held[m][2u * np], ba, hi[0], hi[1]);
            mma_bf16(held[m][2u * np], ba, lo[0], lo[1]);
            mma_bf16(held[m][2u * np + 1u], ba, hi[2], hi[3]);
            mma_bf16(held[m][2u * np + 1u], ba, lo[2], lo[3]);
          }
        }
      }
    }
    __syncthreads();  // state and scaled x may be overwritten
  }
#pragma unroll
  for (uint32_t m = 0; m < MT; ++m) {
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
#pragma unroll
      for (uint32_t j = 0; j < 4u; ++j) {
        const uint32_t row = 16u * (warp + kScanWarps * m) + g + 8u * (j >> 1), col = 8u * n + 2u * t4 + (j & 1u);
        if (row < s.state && column0 + col < s.v_dim) state[static_cast<uint64_t>(row) * s.v_dim + col] = held[m][n][j];
      }
    }
  }
  keep_history(p, r0.recurrent, base, head, column0);
}

// ---------------------------------------------------------------- grouped norm ----
constexpr uint32_t kGroupThreads = 128;

// Grid (groups, rows).
template <class T>
__global__ void __launch_bounds__(kGroupThreads) grouped_norm_kernel(const float *y, uint32_t y_stride, const uint16_t *weight,
                                                                     uint32_t part, float eps, T *x, uint32_t x_stride) {
  __shared__ float scratch[40];
  pdl_trigger();
  pdl_wait();
  const uint32_t begin = blockIdx.x * part;
  const float *src = y + static_cast<uint64_t>(blockIdx.y) * y_stride + begin;
  T *dst = x + static_cast<uint64_t>(blockIdx.y) * x_stride + begin;
  float sumsq = 0.0f;
  for (uint32_t i = threadIdx.x; i < part; i += kGroupThreads) {
    const float v = src[i];
    sumsq = fmaf(v, v, sumsq);
  }
  const float scale = 1.0f / sqrtf(block_sum(sumsq, scratch) / static_cast<float>(part) + eps);
  for (uint32_t i = threadIdx.x; i < part; i += kGroupThreads) put(dst + i, src[i] * scale * bf16_bits_to_f32(weight[begin + i]));
}

uint32_t column_tiles(const StateSpaceShape &s) { return (s.v_dim + kColumns - 1u) / kColumns; }

// Rows from which a block runs in chunks on the tensor pipe.
constexpr uint32_t kScanMinRows = 16;

template <class T>
cudaError_t launch_block(cudaStream_t stream, const StateSpaceParams &p) {
  const StateSpaceShape &s = p.s;
  const dim3 conv_grid((s.conv_width() + kConvThreads - 1u) / kConvThreads, (p.row_count + kConvRows - 1u) / kConvRows);
  cudaError_t err = launch_with_pdl(s.taps <= 4u ? state_space_conv_kernel<T, 4> : state_space_conv_kernel<T, kMaxTaps>,
                                    conv_grid, dim3(kConvThreads), 0, stream, p.pdl != 0, p);
  if (err != cudaSuccess) return err;
  if (sizeof(T) == 2u && p.row_count >= kScanMinRows)
    return launch_with_pdl(s.state <= 128u ? state_space_scan_kernel<1> : state_space_scan_kernel<2>,
                           dim3(column_tiles(s), s.heads), dim3(kScanThreads), ScanLayout(s).total, stream, p.pdl != 0, p);
  return launch_with_pdl(s.state <= 128u ? state_space_rows_kernel<T, 16> : state_space_rows_kernel<T, 32>,
                         dim3(column_tiles(s) * s.heads), dim3(kStepThreads), 0, stream, p.pdl != 0, p);
}

}  // namespace

bool state_space_supported(const StateSpaceShape &s) {
  return s.heads != 0 && s.v_dim != 0 && s.state != 0 && s.state <= kMaxState && s.groups != 0 && s.heads % s.groups == 0 &&
         s.taps != 0 && s.taps <= kMaxTaps && s.norm_groups != 0 && s.inner() % s.norm_groups == 0 && s.heads <= 65535u &&
         s.norm_groups <= 65535u;
}

cudaError_t configure_state_space() {
  cudaError_t err = cudaSuccess;
  for (const void *kernel : {reinterpret_cast<const void *>(state_space_scan_kernel<1>),
                             reinterpret_cast<const void *>(state_space_scan_kernel<2>)})
    if (err == cudaSuccess) err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  return err;
}

cudaError_t launch_state_space_step(cudaStream_t stream, const StateSpaceParams &p) {
  if (!state_space_supported(p.s) || (p.rows != nullptr && (p.row_count == 0 || p.row_count > 65535u)))
    return cudaErrorInvalidValue;
  void (*kernel)(StateSpaceParams);
  if (p.s.v_dim % 4u == 0)
    kernel = p.s.state <= 128u ? state_space_step_kernel<4, true> : state_space_step_kernel<8, true>;
  else
    kernel = p.s.state <= 128u ? state_space_step_kernel<4, false> : state_space_step_kernel<8, false>;
  return launch_with_pdl(kernel, dim3(column_tiles(p.s) * p.s.heads, p.rows != nullptr ? p.row_count : 1u), dim3(kStepThreads), 0, stream,
                         p.pdl != 0, p);
}

cudaError_t launch_state_space_block(cudaStream_t stream, const StateSpaceParams &p) {
  if (!state_space_supported(p.s) || p.rows == nullptr || p.row_count == 0 || p.row_count > kScanMaxRows || p.convolved == nullptr)
    return cudaErrorInvalidValue;
  return p.f32 != 0 ? launch_block<float>(stream, p) : launch_block<uint16_t>(stream, p);
}

cudaError_t launch_grouped_norm(cudaStream_t stream, const float *y, uint32_t y_stride, const uint16_t *weight,
                                uint32_t width, uint32_t groups, float eps, void *x, uint32_t x_stride, bool f32,
                                uint32_t rows, bool pdl) {
  if (rows == 0 || rows > 65535u || groups == 0 || width % groups != 0) return cudaErrorInvalidValue;
  const dim3 grid(groups, rows);
  const uint32_t part = width / groups;
  if (f32)
    return launch_with_pdl(grouped_norm_kernel<float>, grid, dim3(kGroupThreads), 0, stream, pdl, y, y_stride, weight, part,
                           eps, static_cast<float *>(x), x_stride);
  return launch_with_pdl(grouped_norm_kernel<uint16_t>, grid, dim3(kGroupThreads), 0, stream, pdl, y, y_stride, weight, part,
                         eps, static_cast<uint16_t *>(x), x_stride);
}

}  // namespace nb
