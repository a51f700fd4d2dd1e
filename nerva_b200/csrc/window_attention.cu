// Sliding-window grouped-query attention over the paged cache, for heads of any size up to 256 with
// separate query/key and value widths: a rotation of the leading dimensions of a head (its
// frequencies and the factor on cos and sin come as a table, so plain and scaled rotations look
// alike here), then an optional weightless RMS norm of q and k, softmax over the keys in the window.
// Optionally the first positions stay visible behind the window (the kernels then walk the tiles that
// hold them in front of the window's own), scores are soft-capped, and a sigmoid gate per head scales
// the result.
//
//   window_attention_kernel   one query token per row.  The lone decode step (ROWS = false) prepares
//                             q, appends the new K/V row and attends in one launch; block rows of an
//                             fp32 session (ROWS = true) find both done by window_publish_kernel.
//                             Grid (KV head x group of 8 query heads x span, row); the spans divide
//                             the window, not the context.  fp32 arithmetic on the CUDA cores, K/V in
//                             shared memory.
//   window_rows_kernel        the block rows of a bf16 session (packed decode step, short portions) on
//                             the tensor pipe, same grid.
//   window_prefill_kernel     64 (position, head) rows of one KV head against 64-token tiles on the
//                             tensor pipe (mma.sync, bf16), flash-attention style: scores and softmax
//                             stay in registers.  Queries and probabilities are split into a bf16
//                             rounding and its remainder, so a product loses only the rounding of the
//                             cached row.  Only tiles that meet some row's window are loaded.
#include <math.h>

#include "common.cuh"
#include "kernels.cuh"
#include "mma_bf16.cuh"

namespace nb {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kPageTokens = NERVA_KV_CACHE_BLOCK_TOKENS;
constexpr uint32_t kTile = 32;             // tokens of one score tile: one per lane
constexpr uint32_t kWarps = 8;             // of a window_attention_kernel block
constexpr uint32_t kHeadsPerBlock = 8;
constexpr uint32_t kMaxSmem = 227u * 1024u;

template <uint32_t BYTES>
__device__ __forceinline__ void cp_async_zfill(void *dst, const void *src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(valid ? BYTES : 0u)
               : "memory");
}
__device__ __forceinline__ void cp_async_16(void *dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

__device__ __forceinline__ void to_cache(float *dst, float v) { *dst = v; }
__device__ __forceinline__ void to_cache(uint16_t *dst, float v) { *dst = f32_to_bf16_bits(v); }
__device__ __forceinline__ float from_cache(float v) { return v; }
__device__ __forceinline__ float from_cache(uint16_t v) { return bf16_bits_to_f32(v); }
__device__ __forceinline__ float2 cache_pair(const float *p) { return *reinterpret_cast<const float2 *>(p); }
__device__ __forceinline__ float2 cache_pair(const uint16_t *p) {
  const uint32_t w = *reinterpret_cast<const uint32_t *>(p);
  return make_float2(bf16x2_lo(w), bf16x2_hi(w));
}
// q . k over one 16-byte piece of a cached row.
__device__ __forceinline__ float dot_piece(const float *k, const float *q, float acc) {
  const float4 a = *reinterpret_cast<const float4 *>(k), b = *reinterpret_cast<const float4 *>(q);
  acc = fmaf(a.x, b.x, acc);
  acc = fmaf(a.y, b.y, acc);
  acc = fmaf(a.z, b.z, acc);
  return fmaf(a.w, b.w, acc);
}
__device__ __forceinline__ float dot_piece(const uint16_t *k, const float *q, float acc) {
  const uint4 w = *reinterpret_cast<const uint4 *>(k);
  const float4 a = *reinterpret_cast<const float4 *>(q), b = *reinterpret_cast<const float4 *>(q + 4);
  acc = fmaf(bf16x2_lo(w.x), a.x, acc);
  acc = fmaf(bf16x2_hi(w.x), a.y, acc);
  acc = fmaf(bf16x2_lo(w.y), a.z, acc);
  acc = fmaf(bf16x2_hi(w.y), a.w, acc);
  acc = fmaf(bf16x2_lo(w.z), b.x, acc);
  acc = fmaf(bf16x2_hi(w.z), b.y, acc);
  acc = fmaf(bf16x2_lo(w.w), b.z, acc);
  return fmaf(bf16x2_hi(w.w), b.w, acc);
}

// The tiles of `size` tokens a query walks: those that hold kept first positions and lie in front of the
// window, then the window's.
struct TileWalk {
  uint32_t kept, first;  // tiles in front; first tile of the window
  __device__ __forceinline__ TileWalk(uint32_t keep_first, uint32_t lo, uint32_t size) {
    first = lo / size;
    kept = (keep_first + size - 1u) / size;
    if (kept > first) kept = first;
  }
  __device__ __forceinline__ uint32_t count(uint32_t end, uint32_t size) const {  // tiles, for a window that ends at `end`
    return kept + (end + size - 1u) / size - first;
  }
  __device__ __forceinline__ uint32_t tile(uint32_t i) const { return i < kept ? i : first + (i - kept); }
};

// EXTRAS of the kernels below: kept first positions, score cap and output gates.  Without them the code
// is the plain window's.
__host__ __device__ inline bool has_extras(const WindowAttentionShape &s) {
  return s.keep_first != 0 || s.softcap > 0.0f || s.head_gate != 0;
}

// Soft cap of a score that carries a factor log2(e).
__device__ __forceinline__ float cap_score(float score, float cap2) { return cap2 * tanhf(score / cap2); }
// The same through one exponential, absolute error a few 1e-7 of the cap.
__device__ __forceinline__ float cap_score_fast(float score, float cap2, float inv_cap2) {
  const float e = exp2f(score * inv_cap2 * (2.0f * kLog2e));
  return cap2 - __fdividef(2.0f * cap2, e + 1.0f);
}

// Factor of a head's output.
template <bool EXTRAS>
__device__ __forceinline__ float output_gate(const WindowAttentionParams &p, uint32_t row, uint32_t h) {
  const WindowAttentionShape &s = p.s;
  if (!EXTRAS || s.head_gate == 0) return 1.0f;
  const uint32_t at = (s.heads + s.kv_heads) * s.qk_dim + s.kv_heads * s.v_dim + h;
  return sigmoid(__ldcg(p.qkv + static_cast<uint64_t>(row) * p.qkv_stride + at));
}

// (sin, cos) of pair i at a position, with the magnitude of a scaled rotation.
__device__ __forceinline__ float2 rotation(const WindowAttentionShape &s, uint32_t position, uint32_t i) {
  float2 t;
  sincosf(static_cast<float>(position) * s.frequency[i], &t.x, &t.y);
  t.x *= s.rotary_magnitude;
  t.y *= s.rotary_magnitude;
  return t;
}

// One warp: the head in v[0 .. qk_dim) (shared memory) is rotated (turn(i): rotation of pair i) and
// normalised in place.
template <class Turn>
__device__ __forceinline__ void rotate_and_norm(float *v, const WindowAttentionShape &s, Turn turn) {
  const uint32_t lane = threadIdx.x & 31u;
  __syncwarp();
  for (uint32_t i = lane; i < s.rotary_pairs; i += 32u) {
    const float2 t = turn(i);
    const float a = v[i], b = v[i + s.rotary_pairs];
    v[i] = a * t.y - b * t.x;
    v[i + s.rotary_pairs] = b * t.y + a * t.x;
  }
  __syncwarp();
  if (s.qk_norm == 0) return;
  float sumsq = 0.0f;
  for (uint32_t i = lane; i < s.qk_dim; i += 32u) sumsq += v[i] * v[i];
  sumsq = warp_sum(sumsq);
  const float scale = 1.0f / sqrtf(sumsq / static_cast<float>(s.qk_dim) + s.eps);
  for (uint32_t i = lane; i < s.qk_dim; i += 32u) v[i] *= scale;
  __syncwarp();
}

// Cached row (page, slot) of a KV head, in elements of a row of `width` per head.
__device__ __forceinline__ uint64_t cache_row(uint32_t page, uint32_t token, uint32_t kv_heads, uint32_t kvh, uint32_t width) {
  return ((static_cast<uint64_t>(page) * kPageTokens + token % kPageTokens) * kv_heads + kvh) * width;
}

// Grid ((heads + kv_heads) / 8, rows), a warp per head: a query head is prepared in place, a KV head's K
// and V go to the cache.  Without rotation and norm there is nothing to prepare: KV heads only.
constexpr uint32_t kPublishWarps = 8;
__host__ __device__ inline bool queries_prepared(const WindowAttentionShape &s) { return s.rotary_pairs != 0 || s.qk_norm != 0; }
template <class T>
__global__ void __launch_bounds__(kPublishWarps * 32) window_publish_kernel(WindowAttentionParams p) {
  __shared__ float heads[kPublishWarps][256];
  __shared__ float2 turn[128];
  pdl_trigger();
  const WindowAttentionShape &s = p.s;
  const FusedAttentionRow &r = p.rows[blockIdx.y];
  if (r.position >= r.max_context) {
    pdl_wait();
    return;
  }
  for (uint32_t i = threadIdx.x; i < s.rotary_pairs; i += blockDim.x) turn[i] = rotation(s, r.position, i);
  __syncthreads();
  pdl_wait();
  const uint32_t lane = threadIdx.x & 31u;
  const uint32_t unit = (queries_prepared(s) ? 0u : s.heads) + blockIdx.x * kPublishWarps + (threadIdx.x >> 5);
  if (unit >= s.heads + s.kv_heads) return;
  float *head = heads[threadIdx.x >> 5];
  const bool query = unit < s.heads;
  const uint32_t h = query ? unit : unit - s.heads;
  float *row = p.qkv + static_cast<uint64_t>(blockIdx.y) * p.qkv_stride;
  float *src = row + (query ? 0u : s.heads * s.qk_dim) + h * s.qk_dim;
  for (uint32_t i = lane; i < s.qk_dim; i += 32u) head[i] = __ldcg(src + i);
  rotate_and_norm(head, s, [&](uint32_t i) { return turn[i]; });
  if (query) {
    for (uint32_t i = lane; i < s.qk_dim; i += 32u) src[i] = head[i];
    return;
  }
  const uint32_t page = r.page_table[r.position / kPageTokens];
  if (page >= r.page_count) {
    report_error(r.error_word, kErrPageOutOfRange);
    return;
  }
  T *k_out = reinterpret_cast<T *>(r.key_pages) + p.key_offset + cache_row(page, r.position, s.kv_heads, h, s.qk_pad);
  T *v_out = reinterpret_cast<T *>(r.value_pages) + p.value_offset + cache_row(page, r.position, s.kv_heads, h, s.v_pad);
  const float *v_in = row + (s.heads + s.kv_heads) * s.qk_dim + h * s.v_dim;
  for (uint32_t i = lane; i < s.qk_pad; i += 32u) to_cache(k_out + i, i < s.qk_dim ? head[i] : 0.0f);
  for (uint32_t i = lane; i < s.v_pad; i += 32u) to_cache(v_out + i, i < s.v_dim ? __ldcg(v_in + i) : 0.0f);
}

template <class T>
struct DecodeLayout {
  uint32_t k_row, v_row;  // bytes of a staged row; K rows are 16 bytes apart from a multiple of 32 (bank-conflict-free)
  uint32_t stage, total;
  __host__ __device__ DecodeLayout(const WindowAttentionShape &s, uint32_t chunk_tokens) {
    k_row = s.qk_pad * static_cast<uint32_t>(sizeof(T)) + 16u;
    v_row = s.v_pad * static_cast<uint32_t>(sizeof(T));
    stage = chunk_tokens * (k_row + v_row);
    // two stages | q [8][qk_pad] | k_new [qk_pad] | v_new [v_pad] | p [16][32]
    total = 2u * stage + (kHeadsPerBlock * s.qk_pad + s.qk_pad + s.v_pad + 2u * kHeadsPerBlock * kTile) * 4u;
  }
};

// Score tiles per chunk: two, or one where two stages of two tiles do not fit shared memory.
template <class T>
uint32_t chunk_tiles(const WindowAttentionShape &s) {
  return DecodeLayout<T>(s, 2u * kTile).total <= kMaxSmem - 2048u ? 2u : 1u;
}

// After every thread's partials of its block are stored: the block that draws the last ticket of its
// heads merges their spans (one acquire-release atomic between the block's barriers orders the
// partials).  Called by the whole block.
template <class T, uint32_t PAIRS, bool EXTRAS>
__device__ __forceinline__ void merge_spans(const WindowAttentionParams &p, uint32_t row, uint32_t head0, uint32_t hb,
                                            uint32_t *ticket) {
  const WindowAttentionShape &s = p.s;
  const uint32_t lane = threadIdx.x & 31u, warps = blockDim.x >> 5, S = p.splits;
  uint32_t *counter = p.tickets + static_cast<uint64_t>(row) * s.heads + head0;
  __syncthreads();
  if (threadIdx.x == 0) {
    uint32_t drawn;
    asm volatile("atom.acq_rel.gpu.global.add.u32 %0, [%1], 1;" : "=r"(drawn) : "l"(counter) : "memory");
    *ticket = drawn;
  }
  __syncthreads();
  if (*ticket != S - 1u) return;
  for (uint32_t hw = threadIdx.x >> 5; hw < hb; hw += warps) {
    const uint32_t h = head0 + hw;
    const uint64_t slot0 = (static_cast<uint64_t>(row) * s.heads + h) * S;
    // every load of a batch of spans is issued before anything is computed from it; the first batch
    // travels together with the spans' maxima and sums
    constexpr uint32_t kBatch = PAIRS <= 2u ? 16u : 8u;
    float2 v[kBatch][PAIRS];
    auto load = [&](uint32_t first) {
#pragma unroll
      for (uint32_t u = 0; u < kBatch; ++u) {
#pragma unroll
        for (uint32_t j = 0; j < PAIRS; ++j) {
          const uint32_t d = 2u * lane + 64u * j;
          v[u][j] = first + u < S && d < s.v_pad
                        ? __ldcg(reinterpret_cast<const float2 *>(p.partial_acc + (slot0 + first + u) * s.v_pad + d))
                        : make_float2(0.0f, 0.0f);
        }
      }
    };
    float ms = -INFINITY, ls = 0.0f;
    if (lane < S) {
      ms = __ldcg(p.partial_m + slot0 + lane);
      ls = __ldcg(p.partial_l + slot0 + lane);
    }
    load(0);
    const float m = warp_max(ls > 0.0f ? ms : -INFINITY);
    float w = ls > 0.0f ? exp2f(ms - m) : 0.0f;
    w /= warp_sum(ls * w);
    float a[2u * PAIRS];
#pragma unroll
    for (uint32_t i = 0; i < 2u * PAIRS; ++i) a[i] = 0.0f;
    for (uint32_t first = 0; first < S; first += kBatch) {
      if (first != 0) load(first);
#pragma unroll
      for (uint32_t u = 0; u < kBatch; ++u) {
        const float wi = __shfl_sync(0xffffffffu, w, (first + u) & 31u);  // zero beyond the last span
#pragma unroll
        for (uint32_t j = 0; j < PAIRS; ++j) {
          a[2u * j] = fmaf(v[u][j].x, wi, a[2u * j]);
          a[2u * j + 1u] = fmaf(v[u][j].y, wi, a[2u * j + 1u]);
        }
      }
    }
    T *out = reinterpret_cast<T *>(p.out) + static_cast<uint64_t>(row) * p.out_stride + h * s.v_dim;
    const float gate = output_gate<EXTRAS>(p, row, h);
#pragma unroll
    for (uint32_t i = 0; i < 2u * PAIRS; ++i) {
      const uint32_t d = 2u * lane + 64u * (i / 2u) + (i & 1u);
      if (d < s.v_dim) to_cache(out + d, a[i] * gate);
    }
  }
  if (threadIdx.x == 0) *counter = 0;  // ready for the next launch
}

// PAIRS: value pairs (2 lane + 64 j, +1) a lane accumulates; v_pad <= 64 PAIRS.
// A warp has at most two work items: heads x tiles <= 2 kWarps.  Two stages of two 128-dim bf16 tiles take
// 75 KB, which fits beside a weight-streaming block with two ring slots per warp on the same SM.
template <class T, uint32_t PAIRS, bool ROWS, bool EXTRAS>
__global__ void __launch_bounds__(kWarps * 32) window_attention_kernel(WindowAttentionParams p, uint32_t tiles) {
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ uint32_t ticket;
  __shared__ float2 turn[ROWS ? 1 : 128];  // sin and cos of the lone step's rotation
  const WindowAttentionShape &s = p.s;
  const uint32_t chunk_tokens = tiles * kTile;
  const DecodeLayout<T> layout(s, chunk_tokens);
  float *q_sh = reinterpret_cast<float *>(smem + 2u * layout.stage);
  float *k_new = q_sh + kHeadsPerBlock * s.qk_pad;
  float *v_new = k_new + s.qk_pad;
  float *p_sh = v_new + s.v_pad;

  pdl_trigger();
  if (ROWS) pdl_wait();
  const uint32_t row = blockIdx.y;
  uint32_t position, page_count;
  T *keys, *values;
  const uint32_t *table;
  uint32_t *error_word;
  if (ROWS) {
    const FusedAttentionRow &r = p.rows[row];
    position = r.position;
    page_count = r.page_count;
    keys = reinterpret_cast<T *>(r.key_pages) + p.key_offset;
    values = reinterpret_cast<T *>(r.value_pages) + p.value_offset;
    table = r.page_table;
    error_word = r.error_word;
    if (position >= r.max_context) return;
  } else {
    position = *p.cursor;  // changes in the last kernel of a step only
    page_count = p.page_count;
    keys = reinterpret_cast<T *>(p.keys) + p.key_offset;
    values = reinterpret_cast<T *>(p.values) + p.value_offset;
    table = p.page_table;
    error_word = p.error_word;
    if (position >= p.max_context) {
      pdl_wait();
      return;
    }
  }
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
  const uint32_t group = s.heads / s.kv_heads;
  const uint32_t subs = (group + kHeadsPerBlock - 1u) / kHeadsPerBlock;
  const uint32_t S = p.splits;
  const uint32_t unit = blockIdx.x / S, span = blockIdx.x - unit * S;
  const uint32_t kvh = unit / subs, sub = unit - kvh * subs;
  const uint32_t head0 = kvh * group + sub * kHeadsPerBlock;
  const uint32_t left_heads = group - sub * kHeadsPerBlock;
  const uint32_t hb = left_heads < kHeadsPerBlock ? left_heads : kHeadsPerBlock;
  // cached tokens [lo, hist) and those below keep_first are seen; the lone step's own token comes from the projection
  const uint32_t hist = ROWS ? position + 1u : position;
  const uint32_t lo = s.window != 0 && position + 1u > s.window ? position + 1u - s.window : 0u;
  const uint32_t keep_first = EXTRAS ? s.keep_first : 0u;
  const bool capped = EXTRAS && s.softcap > 0.0f;
  const TileWalk walk(keep_first, lo, chunk_tokens);
  const uint32_t chunks = walk.count(hist, chunk_tokens);  // lo <= hist: never negative
  const uint32_t chunk_begin = chunks * span / S, chunk_end = chunks * (span + 1u) / S;  // numbers in the walk
  const bool owns_current = !ROWS && span + 1u == S;

  const uint32_t k_pieces = s.qk_pad * static_cast<uint32_t>(sizeof(T)) / 16u;
  const uint32_t v_pieces = s.v_pad * static_cast<uint32_t>(sizeof(T)) / 16u;
  const uint32_t row_pieces = k_pieces + v_pieces;
  auto issue = [&](uint32_t number, uint32_t stage) {
    const uint32_t chunk = walk.tile(number);
    uint8_t *k_stage = smem + stage * layout.stage;
    uint8_t *v_stage = k_stage + chunk_tokens * layout.k_row;
    const uint32_t first = chunk * chunk_tokens;
    // the chunk's page-table entries, one per lane, handed out by shuffle
    const uint32_t pages = chunk_tokens / kPageTokens;
    uint32_t my_page = 0;
    const uint32_t page_token = first + lane * kPageTokens;
    if (lane < pages && page_token < hist && (page_token + kPageTokens > lo || page_token / kTile * kTile < keep_first)) {
      my_page = table[first / kPageTokens + lane];
      if (my_page >= page_count) {
        report_error(error_word, kErrPageOutOfRange);
        my_page = 0;
      }
    }
    // a warp copies whole tokens; lanes take the 16-byte pieces of the K row, then of the V row
    for (uint32_t t = warp; t < chunk_tokens; t += kWarps) {
      const uint32_t page = __shfl_sync(0xffffffffu, my_page, t / kPageTokens);
      const uint32_t token = first + t;
      // a tile with kept tokens is copied whole: its invisible rows meet probabilities of zero
      if (token >= hist || (token < lo && token / kTile * kTile >= keep_first)) continue;
      const T *k_src = keys + cache_row(page, token, s.kv_heads, kvh, s.qk_pad);
      const T *v_src = values + cache_row(page, token, s.kv_heads, kvh, s.v_pad);
      for (uint32_t c = lane; c < row_pieces; c += 32u) {
        if (c < k_pieces)
          cp_async_16(k_stage + t * layout.k_row + c * 16u, reinterpret_cast<const uint8_t *>(k_src) + c * 16u);
        else
          cp_async_16(v_stage + t * layout.v_row + (c - k_pieces) * 16u,
                      reinterpret_cast<const uint8_t *>(v_src) + (c - k_pieces) * 16u);
      }
    }
    cp_async_commit();
  };
  // cached rows were written by earlier steps: requested before the wait for this step's projection
  if (chunk_begin < chunk_end) issue(chunk_begin, 0);
  if (chunk_begin + 1u < chunk_end) issue(chunk_begin + 1u, 1);
  if (!ROWS) {
    for (uint32_t i = threadIdx.x; i < s.rotary_pairs; i += blockDim.x) turn[i] = rotation(s, position, i);
    __syncthreads();
    pdl_wait();
  }

  const float *qkv = p.qkv + static_cast<uint64_t>(row) * p.qkv_stride;
  const float qscale = s.scale * kLog2e, cap2 = s.softcap * kLog2e;
  for (uint32_t w = warp; w < hb; w += kWarps) {
    float *q = q_sh + w * s.qk_pad;
    const float *src = qkv + (head0 + w) * s.qk_dim;
    for (uint32_t i = lane; i < s.qk_pad; i += 32u) q[i] = i < s.qk_dim ? __ldcg(src + i) : 0.0f;
    if (!ROWS) rotate_and_norm(q, s, [&](uint32_t i) { return turn[i]; });
    __syncwarp();
    for (uint32_t i = lane; i < s.qk_dim; i += 32u) q[i] *= qscale;
  }
  if (owns_current && warp == kWarps - 1u) {  // the warp with the fewest queries
    const float *k_src = qkv + s.heads * s.qk_dim + kvh * s.qk_dim;
    const float *v_src = qkv + (s.heads + s.kv_heads) * s.qk_dim + kvh * s.v_dim;
    for (uint32_t i = lane; i < s.qk_pad; i += 32u) k_new[i] = i < s.qk_dim ? __ldcg(k_src + i) : 0.0f;
    rotate_and_norm(k_new, s, [&](uint32_t i) { return turn[i]; });
    __syncwarp();
    uint32_t page = table[position / kPageTokens];
    if (page >= page_count) {
      report_error(error_word, kErrPageOutOfRange);
      page = 0;
    }
    T *k_out = keys + cache_row(page, position, s.kv_heads, kvh, s.qk_pad);
    T *v_out = values + cache_row(page, position, s.kv_heads, kvh, s.v_pad);
    for (uint32_t i = lane; i < s.qk_pad; i += 32u) {
      T k;
      to_cache(&k, k_new[i]);
      k_new[i] = from_cache(k);
      if (sub == 0) k_out[i] = k;
    }
    for (uint32_t i = lane; i < s.v_pad; i += 32u) {
      T v;
      to_cache(&v, i < s.v_dim ? __ldcg(v_src + i) : 0.0f);
      v_new[i] = from_cache(v);
      if (sub == 0) v_out[i] = v;
    }
  }

  // work items (head, tile of the chunk): item = tile * hb + head; a warp has at most two
  const uint32_t items = hb * tiles;
  float m_run[2], l_run[2], acc[2][2u * PAIRS];
#pragma unroll
  for (uint32_t u = 0; u < 2u; ++u) {
    m_run[u] = -INFINITY;
    l_run[u] = 0.0f;
#pragma unroll
    for (uint32_t i = 0; i < 2u * PAIRS; ++i) acc[u][i] = 0.0f;
  }
  for (uint32_t chunk = chunk_begin; chunk < chunk_end; ++chunk) {
    const uint32_t stage = (chunk - chunk_begin) & 1u;
    if (chunk + 1u < chunk_end) {
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint8_t *k_stage = smem + stage * layout.stage;
    const uint8_t *v_stage = k_stage + chunk_tokens * layout.k_row;
#pragma unroll
    for (uint32_t u = 0; u < 2u; ++u) {
      const uint32_t item = warp + u * kWarps;
      if (item < items) {
        const uint32_t tile = item / hb, head = item - tile * hb;
        const uint32_t first = walk.tile(chunk) * chunk_tokens + tile * kTile;
        // the tile's visible tokens lie in [first + t0, first + t1)
        const bool kept = first < keep_first;
        const uint32_t t0 = lo > first && !kept ? lo - first : 0u;
        const uint32_t end = kept && lo >= first + kTile && keep_first < hist ? keep_first : hist;
        const uint32_t t1 = end > first ? (end - first < kTile ? end - first : kTile) : 0u;
        if (t0 < t1) {
          float score = -INFINITY;
          if (lane >= t0 && lane < t1 && (first + lane >= lo || first + lane < keep_first)) {
            const T *k_row = reinterpret_cast<const T *>(k_stage + (tile * kTile + lane) * layout.k_row);
            const float *q = q_sh + head * s.qk_pad;
            constexpr uint32_t kElems = 16u / sizeof(T);
            float part[2] = {0.0f, 0.0f};
            for (uint32_t c = 0; c < k_pieces; c += 2u) {  // qk_pad is a multiple of 16: an even number of pieces
              part[0] = dot_piece(k_row + c * kElems, q + c * kElems, part[0]);
              part[1] = dot_piece(k_row + (c + 1u) * kElems, q + (c + 1u) * kElems, part[1]);
            }
            score = part[0] + part[1];
            if (capped) score = cap_score(score, cap2);
          }
          const float m_new = fmaxf(m_run[u], warp_max(score));  // some token of the tile is visible: finite
          const float pr = exp2f(score - m_new);
          const float corr = exp2f(m_run[u] - m_new);
          l_run[u] = l_run[u] * corr + warp_sum(pr);
          m_run[u] = m_new;
#pragma unroll
          for (uint32_t i = 0; i < 2u * PAIRS; ++i) acc[u][i] *= corr;
          p_sh[item * kTile + lane] = pr;
          __syncwarp();
#pragma unroll 8
          for (uint32_t t = t0; t < t1; ++t) {
            const float pt = p_sh[item * kTile + t];
            const T *v_row = reinterpret_cast<const T *>(v_stage + (tile * kTile + t) * layout.v_row);
#pragma unroll
            for (uint32_t j = 0; j < PAIRS; ++j) {
              const uint32_t d = 2u * lane + 64u * j;
              if (d < s.v_pad) {
                const float2 v = cache_pair(v_row + d);
                acc[u][2u * j] = fmaf(pt, v.x, acc[u][2u * j]);
                acc[u][2u * j + 1u] = fmaf(pt, v.y, acc[u][2u * j + 1u]);
              }
            }
          }
          __syncwarp();
        }
      }
    }
    __syncthreads();
    if (chunk + 2u < chunk_end) issue(chunk + 2u, stage);
  }
  __syncthreads();  // q, k_new, v_new are visible also when no chunk ran; the stages are idle

  // every item's state through the stage memory, then a warp finishes each head
  float *handoff = reinterpret_cast<float *>(smem);  // [item][32 lanes][2 PAIRS + 2]
  constexpr uint32_t kRec = 2u * PAIRS + 2u;
#pragma unroll
  for (uint32_t u = 0; u < 2u; ++u) {
    const uint32_t item = warp + u * kWarps;
    if (item < items) {
      float *dst = handoff + (item * 32u + lane) * kRec;
#pragma unroll
      for (uint32_t i = 0; i < 2u * PAIRS; ++i) dst[i] = acc[u][i];
      dst[2u * PAIRS] = m_run[u];
      dst[2u * PAIRS + 1u] = l_run[u];
    }
  }
  __syncthreads();
  const uint64_t out_row = static_cast<uint64_t>(row) * p.out_stride;
  for (uint32_t w = warp; w < hb; w += kWarps) {
    const uint32_t h = head0 + w;
    float m = -INFINITY, l = 0.0f, a[2u * PAIRS];
#pragma unroll
    for (uint32_t i = 0; i < 2u * PAIRS; ++i) a[i] = 0.0f;
    auto fold = [&](float m1, float l1, const float *v) {
      const float m2 = fmaxf(m, m1);
      const float c0 = exp2f(m - m2), c1 = exp2f(m1 - m2);
      l = l * c0 + l1 * c1;
#pragma unroll
      for (uint32_t i = 0; i < 2u * PAIRS; ++i) a[i] = a[i] * c0 + v[i] * c1;
      m = m2;
    };
    for (uint32_t tile = 0; tile < tiles; ++tile) {
      const float *src = handoff + ((tile * hb + w) * 32u + lane) * kRec;
      if (src[2u * PAIRS + 1u] > 0.0f) fold(src[2u * PAIRS], src[2u * PAIRS + 1u], src);
    }
    if (owns_current) {
      const float *q = q_sh + w * s.qk_pad;
      float dot = 0.0f;
      for (uint32_t i = lane; i < s.qk_pad; i += 32u) dot = fmaf(q[i], k_new[i], dot);
      dot = warp_sum(dot);
      if (capped) dot = cap_score(dot, cap2);
      float v[2u * PAIRS];
#pragma unroll
      for (uint32_t j = 0; j < PAIRS; ++j) {
        const uint32_t d = 2u * lane + 64u * j;
        v[2u * j] = d < s.v_pad ? v_new[d] : 0.0f;
        v[2u * j + 1u] = d < s.v_pad ? v_new[d + 1u] : 0.0f;
      }
      fold(dot, 1.0f, v);
    }
    if (S == 1u) {
      const float inv = output_gate<EXTRAS>(p, row, h) / l;
#pragma unroll
      for (uint32_t i = 0; i < 2u * PAIRS; ++i) {
        const uint32_t d = 2u * lane + 64u * (i / 2u) + (i & 1u);
        if (d < s.v_dim) to_cache(reinterpret_cast<T *>(p.out) + out_row + h * s.v_dim + d, a[i] * inv);
      }
    } else {
      const uint64_t slot = (static_cast<uint64_t>(row) * s.heads + h) * S + span;
#pragma unroll
      for (uint32_t j = 0; j < PAIRS; ++j) {
        const uint32_t d = 2u * lane + 64u * j;
        if (d < s.v_pad)
          *reinterpret_cast<float2 *>(p.partial_acc + slot * s.v_pad + d) = make_float2(a[2u * j], a[2u * j + 1u]);
      }
      if (lane == 0) {
        p.partial_m[slot] = m;
        p.partial_l[slot] = l;
      }
    }
  }
  if (S == 1u) return;
  merge_spans<T, PAIRS, EXTRAS>(p, row, head0, hb, &ticket);
}

// ------------------------------------------------------- block rows on the tensor pipe ----
// One query token per row, bf16 cache.  A block serves up to eight query heads of one KV head over one
// span of pages; each of its four warps walks its own pages through a private ring of cp.async stages
// (no block barrier in the loop).  The sixteen rows of the MMA hold the heads twice: rows 0..7 the bf16
// roundings of the queries (and of the probabilities), rows 8..15 what the rounding lost; the accumulator
// fragment puts rows r and r + 8 into one thread, which adds them.
constexpr uint32_t kRowWarps = 4;
constexpr uint32_t kRowStages = 3;

struct RowLayout {
  uint32_t k_row, v_row, stage, ring, total;
  __host__ __device__ explicit RowLayout(const WindowAttentionShape &s) {
    k_row = s.qk_pad * 2u + 16u;  // an odd number of 16-byte pieces: ldmatrix without bank conflicts
    v_row = s.v_pad * 2u + 16u;
    stage = kPageTokens * (k_row + v_row);
    ring = kRowStages * stage;
    total = kRowWarps * ring + 16u * k_row;  // rings | q: 8 rows high parts, 8 rows low parts
  }
};

template <uint32_t PAIRS, bool EXTRAS>
__global__ void __launch_bounds__(kRowWarps * 32) window_rows_kernel(WindowAttentionParams p) {
  constexpr uint32_t NT = 8u * PAIRS;  // value n-tiles of 8 dims: v_pad <= 64 PAIRS
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ uint32_t ticket;
  const WindowAttentionShape &s = p.s;
  const RowLayout L(s);
  uint8_t *q_sh = smem + kRowWarps * L.ring;
  pdl_trigger();
  pdl_wait();
  const uint32_t row = blockIdx.y;
  const FusedAttentionRow &r = p.rows[row];
  if (r.position >= r.max_context) return;
  const uint16_t *keys = r.key_pages + p.key_offset, *values = r.value_pages + p.value_offset;
  const uint32_t lane = threadIdx.x & 31u, warp = threadIdx.x >> 5;
  const uint32_t group = s.heads / s.kv_heads;
  const uint32_t subs = (group + kHeadsPerBlock - 1u) / kHeadsPerBlock;
  const uint32_t S = p.splits;
  const uint32_t unit = blockIdx.x / S, span = blockIdx.x - unit * S;
  const uint32_t kvh = unit / subs, sub = unit - kvh * subs;
  const uint32_t head0 = kvh * group + sub * kHeadsPerBlock;
  const uint32_t left_heads = group - sub * kHeadsPerBlock;
  const uint32_t hb = left_heads < kHeadsPerBlock ? left_heads : kHeadsPerBlock;
  const uint32_t hist = r.position + 1u;
  const uint32_t lo = s.window != 0 && hist > s.window ? hist - s.window : 0u;
  const uint32_t keep_first = EXTRAS ? s.keep_first : 0u;
  const bool capped = EXTRAS && s.softcap > 0.0f;
  const TileWalk walk(keep_first, lo, kPageTokens);
  const uint32_t pages = walk.count(hist, kPageTokens);
  const uint32_t page_begin = pages * span / S, page_end = pages * (span + 1u) / S;  // numbers in the walk
  const uint32_t first = page_begin + warp;
  auto visible = [&](uint32_t token) { return token < hist && (token >= lo || token < keep_first); };
  const uint32_t my_pages = first < page_end ? (page_end - first + kRowWarps - 1u) / kRowWarps : 0u;

  uint8_t *ring = smem + warp * L.ring;
  const uint32_t k_pieces = s.qk_pad / 8u, v_pieces = s.v_pad / 8u, row_pieces = k_pieces + v_pieces;
  auto issue = [&](uint32_t i) {  // one commit group per page, also when there is none left
    if (i < my_pages) {
      const uint32_t logical = walk.tile(first + i * kRowWarps);
      uint32_t page = r.page_table[logical];
      if (page >= r.page_count) {
        report_error(r.error_word, kErrPageOutOfRange);
        page = 0;
      }
      uint8_t *k_stage = ring + (i % kRowStages) * L.stage;
      uint8_t *v_stage = k_stage + kPageTokens * L.k_row;
      const uint32_t token0 = logical * kPageTokens;
      // a lane takes one 16-byte piece of the K or V row of all sixteen tokens
      for (uint32_t piece = lane; piece < row_pieces; piece += 32u) {
        const bool is_k = piece < k_pieces;
        const uint16_t *src = is_k ? keys + cache_row(page, 0, s.kv_heads, kvh, s.qk_pad) + piece * 8u
                                   : values + cache_row(page, 0, s.kv_heads, kvh, s.v_pad) + (piece - k_pieces) * 8u;
        const uint32_t src_step = s.kv_heads * (is_k ? s.qk_pad : s.v_pad);
        uint8_t *dst = is_k ? k_stage + piece * 16u : v_stage + (piece - k_pieces) * 16u;
        const uint32_t dst_step = is_k ? L.k_row : L.v_row;
        if (token0 >= lo && token0 + kPageTokens <= hist) {
#pragma unroll
          for (uint32_t t = 0; t < kPageTokens; ++t) cp_async_16(dst + t * dst_step, src + t * src_step);
        } else {  // tokens outside the window are filled with zeros
#pragma unroll
          for (uint32_t t = 0; t < kPageTokens; ++t)
            cp_async_zfill<16>(dst + t * dst_step, src + t * src_step, visible(token0 + t));
        }
      }
    }
    cp_async_commit();
  };
  issue(0);
  issue(1);

  const float qscale = s.scale * kLog2e, cap2 = s.softcap * kLog2e, inv_cap2 = cap2 > 0.0f ? 1.0f / cap2 : 0.0f;
  const float *q_in = p.qkv + static_cast<uint64_t>(row) * p.qkv_stride + head0 * s.qk_dim;
  const uint32_t q_pairs = s.qk_pad / 2u;
  for (uint32_t i = threadIdx.x; i < kHeadsPerBlock * q_pairs; i += blockDim.x) {
    const uint32_t h = i / q_pairs, d = 2u * (i - h * q_pairs);
    const float a = h < hb && d < s.qk_dim ? __ldcg(q_in + h * s.qk_dim + d) * qscale : 0.0f;
    const float b = h < hb && d + 1u < s.qk_dim ? __ldcg(q_in + h * s.qk_dim + d + 1u) * qscale : 0.0f;
    *reinterpret_cast<uint32_t *>(q_sh + h * L.k_row + d * 2u) = pack_bf16_hi(a, b);
    *reinterpret_cast<uint32_t *>(q_sh + (h + 8u) * L.k_row + d * 2u) = pack_bf16_lo(a, b);
  }
  __syncthreads();

  const uint32_t t4 = lane & 3u, g = lane >> 2;
  const uint32_t q_addr = smem_addr(q_sh) + ((lane & 7u) + 8u * ((lane >> 3) & 1u)) * L.k_row + (lane >> 4) * 16u;
  const uint32_t k_off = ((lane & 7u) + 8u * (lane >> 4)) * L.k_row + ((lane >> 3) & 1u) * 16u;
  const uint32_t v_off = ((lane & 7u) + 8u * ((lane >> 3) & 1u)) * L.v_row + (lane >> 4) * 16u;
  float m_run = -INFINITY, l_run = 0.0f;
  float o[NT][4];
#pragma unroll
  for (uint32_t n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
  for (uint32_t i = 0; i < my_pages; ++i) {
    issue(i + 2u);
    cp_async_wait<2>();
    __syncwarp();
    const uint32_t k_base = smem_addr(ring + (i % kRowStages) * L.stage);
    const uint32_t v_base = k_base + kPageTokens * L.k_row;
    const uint32_t token0 = walk.tile(first + i * kRowWarps) * kPageTokens;
    float sc[2][4];
#pragma unroll
    for (uint32_t n = 0; n < 2u; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
#pragma unroll 4
    for (uint32_t ks = 0; ks < s.qk_pad / 16u; ++ks) {
      uint32_t qa[4], kb[4];
      ldmatrix_x4(qa, q_addr + ks * 32u);
      ldmatrix_x4(kb, k_base + k_off + ks * 32u);
      mma_bf16(sc[0], qa, kb[0], kb[1]);
      mma_bf16(sc[1], qa, kb[2], kb[3]);
    }
    // head g's scores of tokens 2t, 2t + 1 and 8 + 2t, 9 + 2t
    float v[4] = {sc[0][0] + sc[0][2], sc[0][1] + sc[0][3], sc[1][0] + sc[1][2], sc[1][1] + sc[1][3]};
#pragma unroll
    for (uint32_t j = 0; j < 4u; ++j) {
      const uint32_t token = token0 + 8u * (j >> 1) + 2u * t4 + (j & 1u);
      if (capped) v[j] = cap_score_fast(v[j], cap2, inv_cap2);
      if (!visible(token)) v[j] = -INFINITY;
    }
    float m_page = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
    m_page = fmaxf(m_page, __shfl_xor_sync(0xffffffffu, m_page, 1));
    m_page = fmaxf(m_page, __shfl_xor_sync(0xffffffffu, m_page, 2));
    const float m_new = fmaxf(m_run, m_page);  // every page of the span has a visible token: finite
    const float corr = exp2f(m_run - m_new);
    m_run = m_new;
#pragma unroll
    for (uint32_t j = 0; j < 4u; ++j) v[j] = exp2f(v[j] - m_new);
    l_run = l_run * corr + ((v[0] + v[1]) + (v[2] + v[3]));  // this thread's share; the quad is summed at the end
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
      o[n][0] *= corr;
      o[n][1] *= corr;
      o[n][2] *= corr;
      o[n][3] *= corr;
    }
    const uint32_t pa[4] = {pack_bf16_hi(v[0], v[1]), pack_bf16_lo(v[0], v[1]), pack_bf16_hi(v[2], v[3]),
                            pack_bf16_lo(v[2], v[3])};
#pragma unroll
    for (uint32_t np = 0; np < NT / 2u; ++np) {
      if (np * 16u < s.v_pad) {
        uint32_t vb[4];
        ldmatrix_x4_trans(vb, v_base + v_off + np * 32u);
        mma_bf16(o[2u * np], pa, vb[0], vb[1]);
        mma_bf16(o[2u * np + 1u], pa, vb[2], vb[3]);
      }
    }
    __syncwarp();  // the stage is free for the copy the next iteration issues
  }
  cp_async_wait<0>();
  l_run += __shfl_xor_sync(0xffffffffu, l_run, 1);
  l_run += __shfl_xor_sync(0xffffffffu, l_run, 2);
  __syncthreads();
  // the warps' states through the ring memory: [warp][head][v_pad | m | l]
  float *merge = reinterpret_cast<float *>(smem);
  const uint32_t rec = s.v_pad + 2u;
  if (g < hb) {
    float *dst = merge + (warp * kHeadsPerBlock + g) * rec;
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
      if (n * 8u < s.v_pad) {
        dst[n * 8u + 2u * t4] = o[n][0] + o[n][2];
        dst[n * 8u + 2u * t4 + 1u] = o[n][1] + o[n][3];
      }
    }
    if (t4 == 0) {
      dst[s.v_pad] = m_run;
      dst[s.v_pad + 1u] = l_run;
    }
  }
  __syncthreads();
  for (uint32_t idx = threadIdx.x; idx < hb * s.v_pad; idx += blockDim.x) {
    const uint32_t h = idx / s.v_pad, d = idx - h * s.v_pad;
    float m = -INFINITY, a = 0.0f, l = 0.0f;
    for (uint32_t w = 0; w < kRowWarps; ++w) m = fmaxf(m, merge[(w * kHeadsPerBlock + h) * rec + s.v_pad]);
    for (uint32_t w = 0; w < kRowWarps; ++w) {
      const float *src = merge + (w * kHeadsPerBlock + h) * rec;
      if (src[s.v_pad + 1u] > 0.0f) {
        const float c = exp2f(src[s.v_pad] - m);
        a = fmaf(src[d], c, a);
        l = fmaf(src[s.v_pad + 1u], c, l);
      }
    }
    if (S == 1u) {
      if (d < s.v_dim)
        reinterpret_cast<uint16_t *>(p.out)[static_cast<uint64_t>(row) * p.out_stride + (head0 + h) * s.v_dim + d] =
            f32_to_bf16_bits(a / l * output_gate<EXTRAS>(p, row, head0 + h));
    } else {
      const uint64_t slot = (static_cast<uint64_t>(row) * s.heads + head0 + h) * S + span;
      p.partial_acc[slot * s.v_pad + d] = a;
      if (d == 0) {
        p.partial_m[slot] = m;
        p.partial_l[slot] = l;
      }
    }
  }
  if (S != 1u) merge_spans<uint16_t, PAIRS, EXTRAS>(p, row, head0, hb, &ticket);
}

uint32_t rows_smem(const WindowAttentionShape &s) {
  const RowLayout L(s);
  const uint32_t merge = kRowWarps * kHeadsPerBlock * (s.v_pad + 2u) * 4u;
  return merge <= kRowWarps * L.ring ? L.total : 0u;
}

// ------------------------------------------------------------------ prefill tile ----
constexpr uint32_t kTileRows = 64;    // (position, head) rows of a block: 16 per warp
constexpr uint32_t kKeyTile = 64;
constexpr uint32_t kPrefillThreads = 128;  // per key group

// GROUPS sets of four warps share the block's queries and take every GROUPS-th key tile each; their
// softmax states are merged at the end.  A chunk of 256 positions gives fewer blocks than SMs at eight KV
// heads, so one set of warps would leave the SM idle while its loads and shuffles are in flight.

struct PrefillLayout {
  uint32_t q_row, k_row, v_row, stage, total;  // bytes; rows are an odd number of 16-byte pieces apart
  __host__ __device__ PrefillLayout(const WindowAttentionShape &s, uint32_t groups) {
    q_row = k_row = s.qk_pad * 2u + 16u;
    v_row = s.v_pad * 2u + 16u;
    stage = kKeyTile * (k_row + v_row);
    total = 2u * kTileRows * q_row + groups * 2u * stage;  // q high and low parts | two K/V stages per group
  }
};

// NT: value n-tiles of 8 dims held in registers (v_pad <= 8 NT).
template <uint32_t NT, uint32_t GROUPS, bool EXTRAS>
__global__ void __launch_bounds__(GROUPS * kPrefillThreads) window_prefill_kernel(WindowAttentionParams p) {
  extern __shared__ __align__(128) uint8_t smem[];
  const WindowAttentionShape &s = p.s;
  const PrefillLayout L(s, GROUPS);
  const uint32_t key_group = GROUPS == 1u ? 0u : threadIdx.x / kPrefillThreads;
  auto group_sync = [&]() {
    asm volatile("bar.sync %0, %1;" ::"r"(1u + key_group), "n"(kPrefillThreads) : "memory");
  };
  uint8_t *q_hi = smem, *q_lo = smem + kTileRows * L.q_row;
  uint8_t *stages = smem + 2u * kTileRows * L.q_row + key_group * 2u * L.stage;
  pdl_trigger();
  pdl_wait();
  const uint32_t tid = threadIdx.x % kPrefillThreads, lane = tid & 31u, warp = tid >> 5;
  const uint32_t group = s.heads / s.kv_heads;
  const uint32_t kvh = blockIdx.y;
  const uint32_t total_rows = p.row_count * group;
  const uint32_t f0 = blockIdx.x * kTileRows;
  const uint32_t f_end = f0 + kTileRows < total_rows ? f0 + kTileRows : total_rows;
  const FusedAttentionRow &r0 = p.rows[0];
  const uint32_t base = r0.position;
  const uint32_t pos_first = base + f0 / group, pos_last = base + (f_end - 1u) / group;
  if (pos_last >= r0.max_context) return;
  const uint16_t *keys = r0.key_pages + p.key_offset, *values = r0.value_pages + p.value_offset;

  const uint32_t kv_lo = s.window != 0 && pos_first + 1u > s.window ? pos_first + 1u - s.window : 0u;
  const uint32_t kv_end = pos_last + 1u;
  const uint32_t keep_first = EXTRAS ? s.keep_first : 0u;
  const bool capped = EXTRAS && s.softcap > 0.0f;
  const TileWalk walk(keep_first, kv_lo, kKeyTile);
  const uint32_t tile_begin = key_group, tile_end = walk.count(kv_end, kKeyTile);  // numbers in the walk
  const uint32_t k_pieces = s.qk_pad / 8u, v_pieces = s.v_pad / 8u, row_pieces = k_pieces + v_pieces;
  auto issue = [&](uint32_t tile) {
    uint8_t *k_stage = stages + ((tile - tile_begin) / GROUPS & 1u) * L.stage;
    uint8_t *v_stage = k_stage + kKeyTile * L.k_row;
    const uint32_t first = walk.tile(tile) * kKeyTile;
    uint32_t my_page = 0;
    if (lane < kKeyTile / kPageTokens && first + lane * kPageTokens < kv_end) {
      my_page = r0.page_table[first / kPageTokens + lane];
      if (my_page >= r0.page_count) {
        report_error(r0.error_word, kErrPageOutOfRange);
        my_page = 0;
      }
    }
    for (uint32_t t = warp; t < kKeyTile; t += kPrefillThreads / 32u) {
      const uint32_t page = __shfl_sync(0xffffffffu, my_page, t / kPageTokens);
      const uint32_t token = first + t;
      const bool valid = token < kv_end;  // rows behind the last query are filled with zeros
      const uint16_t *k_src = keys + (valid ? cache_row(page, token, s.kv_heads, kvh, s.qk_pad) : 0u);
      const uint16_t *v_src = values + (valid ? cache_row(page, token, s.kv_heads, kvh, s.v_pad) : 0u);
      for (uint32_t c = lane; c < row_pieces; c += 32u) {
        if (c < k_pieces)
          cp_async_zfill<16>(k_stage + t * L.k_row + c * 16u, k_src + c * 8u, valid);
        else
          cp_async_zfill<16>(v_stage + t * L.v_row + (c - k_pieces) * 16u, v_src + (c - k_pieces) * 8u, valid);
      }
    }
    cp_async_commit();
  };
  if (tile_begin < tile_end) issue(tile_begin);
  if (tile_begin + GROUPS < tile_end) issue(tile_begin + GROUPS);

  // queries, scaled so that the softmax runs on exp2, as a bf16 rounding and its remainder
  const float qscale = s.scale * kLog2e, cap2 = s.softcap * kLog2e, inv_cap2 = cap2 > 0.0f ? 1.0f / cap2 : 0.0f;
  const uint32_t q_pairs = s.qk_pad / 2u;
  for (uint32_t i = threadIdx.x; i < kTileRows * q_pairs; i += GROUPS * kPrefillThreads) {
    const uint32_t row = i / q_pairs, d = 2u * (i - row * q_pairs);
    const uint32_t f = f0 + row;
    float a = 0.0f, b = 0.0f;
    if (f < f_end) {
      const float *src = p.qkv + static_cast<uint64_t>(f / group) * p.qkv_stride + (kvh * group + f % group) * s.qk_dim;
      if (d < s.qk_dim) a = __ldcg(src + d) * qscale;
      if (d + 1u < s.qk_dim) b = __ldcg(src + d + 1u) * qscale;
    }
    *reinterpret_cast<uint32_t *>(q_hi + row * L.q_row + d * 2u) = pack_bf16_hi(a, b);
    *reinterpret_cast<uint32_t *>(q_lo + row * L.q_row + d * 2u) = pack_bf16_lo(a, b);
  }

  // this thread's two rows: g and g + 8 of the warp's sixteen
  const uint32_t g = lane >> 2, t4 = lane & 3u;
  uint32_t pos[2];
  bool live[2];
#pragma unroll
  for (uint32_t i = 0; i < 2u; ++i) {
    const uint32_t f = f0 + warp * 16u + g + 8u * i;
    live[i] = f < f_end;
    pos[i] = base + (live[i] ? f : f_end - 1u) / group;
  }
  const uint32_t window = s.window != 0 ? s.window : 0xffffffffu;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.0f, 0.0f};
  float o[NT][4];
#pragma unroll
  for (uint32_t n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
  const uint32_t q_row = warp * 16u + (lane & 7u) + 8u * ((lane >> 3) & 1u);  // ldmatrix row of the A fragment
  const uint32_t q_piece = lane >> 4;
  const uint32_t k_row = (lane & 7u) + 8u * (lane >> 4), k_piece = (lane >> 3) & 1u;
  const uint32_t v_row = (lane & 7u) + 8u * ((lane >> 3) & 1u), v_piece = lane >> 4;
  const uint32_t q_hi_addr = smem_addr(q_hi) + q_row * L.q_row + q_piece * 16u;
  const uint32_t q_lo_addr = smem_addr(q_lo) + q_row * L.q_row + q_piece * 16u;

  __syncthreads();  // the queries are in place
  for (uint32_t tile = tile_begin; tile < tile_end; tile += GROUPS) {
    if (tile + GROUPS < tile_end) {
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    group_sync();
    const uint32_t k_base = smem_addr(stages + ((tile - tile_begin) / GROUPS & 1u) * L.stage);
    const uint32_t v_base = k_base + kKeyTile * L.k_row;
    const uint32_t first = walk.tile(tile) * kKeyTile;
    float sc[8][4];
#pragma unroll
    for (uint32_t n = 0; n < 8u; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.0f;
    for (uint32_t ks = 0; ks < s.qk_pad / 16u; ++ks) {
      uint32_t ah[4], al[4];
      ldmatrix_x4(ah, q_hi_addr + ks * 32u);
      ldmatrix_x4(al, q_lo_addr + ks * 32u);
#pragma unroll
      for (uint32_t np = 0; np < 4u; ++np) {
        uint32_t kb[4];
        ldmatrix_x4(kb, k_base + (np * 16u + k_row) * L.k_row + (ks * 2u + k_piece) * 16u);
        mma_bf16(sc[2u * np], ah, kb[0], kb[1]);
        mma_bf16(sc[2u * np], al, kb[0], kb[1]);
        mma_bf16(sc[2u * np + 1u], ah, kb[2], kb[3]);
        mma_bf16(sc[2u * np + 1u], al, kb[2], kb[3]);
      }
    }
    if (capped) {
#pragma unroll
      for (uint32_t n = 0; n < 8u; ++n) {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j) sc[n][j] = cap_score_fast(sc[n][j], cap2, inv_cap2);
      }
    }
    // visible: 0 <= pos - token, and pos - token < window or token < keep_first
    float m_tile[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (uint32_t n = 0; n < 8u; ++n) {
#pragma unroll
      for (uint32_t j = 0; j < 4u; ++j) {
        const uint32_t token = first + n * 8u + 2u * t4 + (j & 1u);
        const uint32_t i = j >> 1;
        if (!(token <= pos[i] && (pos[i] - token < window || token < keep_first))) sc[n][j] = -INFINITY;
        m_tile[i] = fmaxf(m_tile[i], sc[n][j]);
      }
    }
    float corr[2];
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      m_tile[i] = fmaxf(m_tile[i], __shfl_xor_sync(0xffffffffu, m_tile[i], 1));
      m_tile[i] = fmaxf(m_tile[i], __shfl_xor_sync(0xffffffffu, m_tile[i], 2));
      const float m_new = fmaxf(m_run[i], m_tile[i]);
      const float ref = m_new == -INFINITY ? 0.0f : m_new;  // no key of the row seen yet
      corr[i] = exp2f(m_run[i] - ref);
      m_run[i] = m_new;
      float sum = 0.0f;
#pragma unroll
      for (uint32_t n = 0; n < 8u; ++n) {
        sc[n][2u * i] = exp2f(sc[n][2u * i] - ref);
        sc[n][2u * i + 1u] = exp2f(sc[n][2u * i + 1u] - ref);
        sum += sc[n][2u * i] + sc[n][2u * i + 1u];
      }
      l_run[i] = l_run[i] * corr[i] + sum;  // this thread's share; the quad is summed at the end
    }
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
      o[n][0] *= corr[0];
      o[n][1] *= corr[0];
      o[n][2] *= corr[1];
      o[n][3] *= corr[1];
    }
#pragma unroll
    for (uint32_t ts = 0; ts < 4u; ++ts) {  // 16 tokens each
      const float *c0 = sc[2u * ts], *c1 = sc[2u * ts + 1u];
      const uint32_t ph[4] = {pack_bf16_hi(c0[0], c0[1]), pack_bf16_hi(c0[2], c0[3]), pack_bf16_hi(c1[0], c1[1]),
                              pack_bf16_hi(c1[2], c1[3])};
      const uint32_t pl[4] = {pack_bf16_lo(c0[0], c0[1]), pack_bf16_lo(c0[2], c0[3]), pack_bf16_lo(c1[0], c1[1]),
                              pack_bf16_lo(c1[2], c1[3])};
#pragma unroll
      for (uint32_t np = 0; np < NT / 2u; ++np) {
        if (np * 16u < s.v_pad) {
          uint32_t vb[4];
          ldmatrix_x4_trans(vb, v_base + (ts * 16u + v_row) * L.v_row + (np * 2u + v_piece) * 16u);
          mma_bf16(o[2u * np], ph, vb[0], vb[1]);
          mma_bf16(o[2u * np], pl, vb[0], vb[1]);
          mma_bf16(o[2u * np + 1u], ph, vb[2], vb[3]);
          mma_bf16(o[2u * np + 1u], pl, vb[2], vb[3]);
        }
      }
    }
    group_sync();
    if (tile + 2u * GROUPS < tile_end) issue(tile + 2u * GROUPS);
  }
#pragma unroll
  for (uint32_t i = 0; i < 2u; ++i) {
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 1);
    l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], 2);
  }
  if (GROUPS == 2u) {
    // the second group's state goes through the stages (idle now): [thread][4 NT + 4], one column per thread
    float *hand = reinterpret_cast<float *>(smem + 2u * kTileRows * L.q_row) + tid;
    __syncthreads();
    if (key_group == 1u) {
#pragma unroll
      for (uint32_t n = 0; n < NT; ++n) {
        if (n * 8u < s.v_pad) {
#pragma unroll
          for (uint32_t j = 0; j < 4u; ++j) hand[(4u + n * 4u + j) * kPrefillThreads] = o[n][j];
        }
      }
#pragma unroll
      for (uint32_t i = 0; i < 2u; ++i) {
        hand[i * kPrefillThreads] = m_run[i];
        hand[(2u + i) * kPrefillThreads] = l_run[i];
      }
    }
    __syncthreads();
    if (key_group == 1u) return;
    float c0[2], c1[2];
#pragma unroll
    for (uint32_t i = 0; i < 2u; ++i) {
      const float m1 = hand[i * kPrefillThreads], l1 = hand[(2u + i) * kPrefillThreads];
      const float m = fmaxf(m_run[i], m1);  // one of the groups has seen the row's own key: finite
      c0[i] = exp2f(m_run[i] - m);
      c1[i] = exp2f(m1 - m);
      l_run[i] = l_run[i] * c0[i] + l1 * c1[i];
    }
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
      if (n * 8u < s.v_pad) {
#pragma unroll
        for (uint32_t j = 0; j < 4u; ++j)
          o[n][j] = o[n][j] * c0[j >> 1] + hand[(4u + n * 4u + j) * kPrefillThreads] * c1[j >> 1];
      }
    }
  }
#pragma unroll
  for (uint32_t i = 0; i < 2u; ++i) {
    if (!live[i]) continue;
    const uint32_t f = f0 + warp * 16u + g + 8u * i;
    uint16_t *dst = reinterpret_cast<uint16_t *>(p.out) + static_cast<uint64_t>(f / group) * p.out_stride +
                    (kvh * group + f % group) * s.v_dim;
    const float inv = output_gate<EXTRAS>(p, f / group, kvh * group + f % group) / l_run[i];
#pragma unroll
    for (uint32_t n = 0; n < NT; ++n) {
      const uint32_t d = n * 8u + 2u * t4;
      if (d < s.v_dim) dst[d] = f32_to_bf16_bits(o[n][2u * i] * inv);
      if (d + 1u < s.v_dim) dst[d + 1u] = f32_to_bf16_bits(o[n][2u * i + 1u] * inv);
    }
  }
}

// Two key groups where their stages fit and the hand-over fits the stages.
uint32_t prefill_groups(const WindowAttentionShape &s) {
  const PrefillLayout L(s, 2);
  const uint32_t hand = (4u + s.v_pad / 8u * 4u) * kPrefillThreads * 4u;
  return s.v_pad <= 128u && L.total <= kMaxSmem - 2048u && hand <= 4u * L.stage ? 2u : 1u;
}

template <class T, bool ROWS, bool EXTRAS>
void (*decode_kernel(uint32_t v_pad))(WindowAttentionParams, uint32_t) {
  if (v_pad <= 64u) return window_attention_kernel<T, 1, ROWS, EXTRAS>;
  if (v_pad <= 128u) return window_attention_kernel<T, 2, ROWS, EXTRAS>;
  return window_attention_kernel<T, 4, ROWS, EXTRAS>;
}
template <class T, bool ROWS>
void (*decode_kernel(const WindowAttentionShape &s))(WindowAttentionParams, uint32_t) {
  return has_extras(s) ? decode_kernel<T, ROWS, true>(s.v_pad) : decode_kernel<T, ROWS, false>(s.v_pad);
}
template <bool EXTRAS>
void (*rows_kernel(uint32_t v_pad))(WindowAttentionParams) {
  if (v_pad <= 64u) return window_rows_kernel<1, EXTRAS>;
  if (v_pad <= 128u) return window_rows_kernel<2, EXTRAS>;
  return window_rows_kernel<4, EXTRAS>;
}
template <bool EXTRAS>
void (*prefill_kernel(uint32_t v_pad, uint32_t groups))(WindowAttentionParams) {
  if (groups == 2u) return v_pad <= 64u ? window_prefill_kernel<8, 2, EXTRAS> : window_prefill_kernel<16, 2, EXTRAS>;
  if (v_pad <= 64u) return window_prefill_kernel<8, 1, EXTRAS>;
  if (v_pad <= 128u) return window_prefill_kernel<16, 1, EXTRAS>;
  return window_prefill_kernel<32, 1, EXTRAS>;
}

// The hand-off of the items' states reuses the stages; both must fit.
template <class T>
uint32_t decode_smem(const WindowAttentionShape &s, uint32_t tiles) {
  const DecodeLayout<T> layout(s, tiles * kTile);
  const uint32_t pairs = s.v_pad <= 64u ? 1u : (s.v_pad <= 128u ? 2u : 4u);
  const uint32_t handoff = tiles * kHeadsPerBlock * 32u * (2u * pairs + 2u) * 4u;
  // k_new, v_new and q are read after the hand-off is written: it must stay inside the stages
  return handoff <= 2u * layout.stage ? layout.total : 0u;
}

template <class T>
cudaError_t launch_decode(cudaStream_t stream, const WindowAttentionParams &p) {
  constexpr bool kHasRows = sizeof(T) == 4u;  // bf16 rows run on the tensor pipe
  const uint32_t tiles = chunk_tiles<T>(p.s);
  const uint32_t bytes = decode_smem<T>(p.s, tiles);
  if (bytes == 0 || bytes > kMaxSmem - 2048u) return cudaErrorNotSupported;
  const uint32_t group = p.s.heads / p.s.kv_heads;
  const uint32_t subs = (group + kHeadsPerBlock - 1u) / kHeadsPerBlock;
  const bool rows = p.rows != nullptr;
  const dim3 grid(p.s.kv_heads * subs * p.splits, rows ? p.row_count : 1u);
  return launch_with_pdl(rows && kHasRows ? decode_kernel<float, true>(p.s) : decode_kernel<T, false>(p.s), grid,
                         dim3(kWarps * 32), bytes, stream, p.pdl != 0, p,
                         tiles);
}

}  // namespace

bool window_attention_supported(const WindowAttentionShape &s, bool f32) {
  if (s.heads == 0 || s.kv_heads == 0 || s.heads % s.kv_heads != 0 || s.qk_dim == 0 || s.v_dim == 0 || s.qk_pad > 256u ||
      s.v_pad > 256u || s.qk_pad % 16u != 0 || s.v_pad % 16u != 0 || 2u * s.rotary_pairs > s.qk_dim)
    return false;
  const uint32_t lone = f32 ? decode_smem<float>(s, chunk_tiles<float>(s)) : decode_smem<uint16_t>(s, chunk_tiles<uint16_t>(s));
  auto fits = [](uint32_t bytes) { return bytes != 0 && bytes <= kMaxSmem - 2048u; };
  return fits(lone) && (f32 || (fits(rows_smem(s)) && fits(PrefillLayout(s, prefill_groups(s)).total)));
}

// Spans for a step whose context is at most target_context: one 64-token chunk per block up to
// kWindowMaxSplits, in powers of two so that a growing context re-captures the step rarely, but never
// more than a full window (which may begin and end inside a chunk) and the kept first positions need.
uint32_t window_attention_splits(uint32_t target_context, uint32_t window, uint32_t keep_first) {
  constexpr uint32_t kChunk = 2u * kTile;
  const uint32_t chunks = target_context / kChunk + (target_context % kChunk != 0 ? 1u : 0u);
  uint32_t s = 1;
  while (s < chunks && s < kWindowMaxSplits) s <<= 1;
  if (window != 0) {
    const uint32_t most = (window - 1u) / kChunk + 2u + keep_first / kChunk + (keep_first % kChunk != 0 ? 1u : 0u);
    if (s > most) s = most;
  }
  return s;
}

// Spans of a block of rows: two blocks per SM are resident, so the count that minimises waves x pages per
// span, as for the paged kernel of the dense models.
uint32_t window_rows_splits(const WindowAttentionShape &s, uint32_t rows, uint32_t longest_context, uint32_t sm_count) {
  const uint32_t group = s.heads / s.kv_heads;
  uint32_t keys = longest_context;
  const uint64_t seen = static_cast<uint64_t>(s.window) + kPageTokens + (s.keep_first != 0 ? s.keep_first + kPageTokens : 0u);
  if (s.window != 0 && seen < keys) keys = static_cast<uint32_t>(seen);
  const uint32_t splits =
      attention_default_splits(keys, rows, s.kv_heads * ((group + kHeadsPerBlock - 1u) / kHeadsPerBlock), sm_count);
  return splits > kWindowMaxSplits ? kWindowMaxSplits : splits;
}

cudaError_t configure_window_attention() {
  cudaError_t err = cudaSuccess;
  auto set = [&](const void *kernel) {
    if (err == cudaSuccess)
      err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kMaxSmem - 2048u));
  };
  for (uint32_t v : {64u, 128u, 256u}) {
    set(reinterpret_cast<const void *>(decode_kernel<uint16_t, false, false>(v)));
    set(reinterpret_cast<const void *>(decode_kernel<uint16_t, false, true>(v)));
    set(reinterpret_cast<const void *>(decode_kernel<float, false, false>(v)));
    set(reinterpret_cast<const void *>(decode_kernel<float, false, true>(v)));
    set(reinterpret_cast<const void *>(decode_kernel<float, true, false>(v)));
    set(reinterpret_cast<const void *>(decode_kernel<float, true, true>(v)));
    set(reinterpret_cast<const void *>(rows_kernel<false>(v)));
    set(reinterpret_cast<const void *>(rows_kernel<true>(v)));
    for (uint32_t groups : {1u, 2u}) {
      set(reinterpret_cast<const void *>(prefill_kernel<false>(v, groups)));
      set(reinterpret_cast<const void *>(prefill_kernel<true>(v, groups)));
    }
  }
  return err;
}

cudaError_t launch_window_publish(cudaStream_t stream, const WindowAttentionParams &p) {
  if (p.rows == nullptr || p.row_count == 0 || p.row_count > 65535u) return cudaErrorInvalidValue;
  const uint32_t units = p.s.kv_heads + (queries_prepared(p.s) ? p.s.heads : 0u);
  const dim3 grid((units + kPublishWarps - 1u) / kPublishWarps, p.row_count);
  return launch_with_pdl(p.f32 != 0 ? window_publish_kernel<float> : window_publish_kernel<uint16_t>, grid,
                         dim3(kPublishWarps * 32), 0, stream, p.pdl != 0, p);
}

cudaError_t launch_window_attention(cudaStream_t stream, const WindowAttentionParams &p) {
  if (p.splits == 0 || p.splits > kWindowMaxSplits || (p.rows != nullptr && (p.row_count == 0 || p.row_count > 65535u)))
    return cudaErrorInvalidValue;
  if (p.rows != nullptr && p.f32 == 0) {
    const uint32_t subs = (p.s.heads / p.s.kv_heads + kHeadsPerBlock - 1u) / kHeadsPerBlock;
    void (*kernel)(WindowAttentionParams) = has_extras(p.s) ? rows_kernel<true>(p.s.v_pad) : rows_kernel<false>(p.s.v_pad);
    return launch_with_pdl(kernel, dim3(p.s.kv_heads * subs * p.splits, p.row_count), dim3(kRowWarps * 32),
                           rows_smem(p.s), stream, p.pdl != 0, p);
  }
  return p.f32 != 0 ? launch_decode<float>(stream, p) : launch_decode<uint16_t>(stream, p);
}

cudaError_t launch_window_prefill(cudaStream_t stream, const WindowAttentionParams &p) {
  if (p.rows == nullptr || p.row_count == 0 || p.f32 != 0) return cudaErrorInvalidValue;
  const uint32_t rows = p.row_count * (p.s.heads / p.s.kv_heads);
  const dim3 grid((rows + kTileRows - 1u) / kTileRows, p.s.kv_heads);
  const uint32_t groups = prefill_groups(p.s);
  const uint32_t bytes = PrefillLayout(p.s, groups).total;
  void (*kernel)(WindowAttentionParams) =
      has_extras(p.s) ? prefill_kernel<true>(p.s.v_pad, groups) : prefill_kernel<false>(p.s.v_pad, groups);
  return launch_with_pdl(kernel, grid, dim3(groups * kPrefillThreads), bytes, stream, p.pdl != 0, p);
}

}  // namespace nb
