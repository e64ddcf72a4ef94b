// Prompt attention whose heads' weights are mixed before they meet the values, on the 5th-generation tensor cores
// (tcgen05): bfloat16, heads of 128 channels, up to 32 of them.  attention_mixed.cu says what is computed;
// attention_mixed_mma.cu has the same three steps for heads of 64 channels.
//
//   mixed_row_sums_tc   per head and 128 queries: S = Q K^T (128 x 128 accumulators in tensor memory, two of them) and the
//                       log of every row's sum; a row belongs to two threads, half of a tile's keys each
//   mixed_weights_tc    a CTA takes Q queries and ALL heads (Q x heads = 512 columns at 16 and 32 heads), the transposed
//                       scores of 128 keys: accumulator lane = key, column = (head, query).  So a thread has one key's
//                       scores in every head, and the mixture of the heads needs nobody else: it reads a head's columns,
//                       takes the exponentials against the rows' sums, and adds them, times the head's column of the
//                       mixing matrix, into the sums of all result heads (packed 32-bit multiply-adds, every chain
//                       independent of the others).  Neighbouring lanes then exchange values so that a lane stores two
//                       keys' weights of one query at once.
//   mixed_values_tc     per head and 128 queries: mixed weights (bf16, keys contiguous) times values, the accumulator in
//                       tensor memory over all keys
// The mixed weights lie in memory as [tile of 128 queries][head][query][key], keys counted from the multiple of 128 at or
// below the first one that the tile's first query sees; places that a query does not see hold zeros.  Tiles are copied with
// cp.async into the 128-byte swizzle that the products' descriptors describe, since their rows are scattered over pages.
// Every wait is bounded in time; where one runs out g_mixed_error is set, nobody waits any more, and the CTA still frees
// its tensor memory and returns.
#include <algorithm>
#include "tcgen05.cuh"

using namespace mir;
using namespace mir::tc;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int kDim = 128;
constexpr int kTile = 128;                          // queries per tile, keys per tile
constexpr int kHalf = kTile * 128;                  // bytes of a 128-row x 64-element half of an operand
constexpr int kOperand = 2 * kHalf;                 // 32 KB
constexpr float kLog2e = 1.4426950408889634f;

__device__ int g_mixed_error = 0;

__device__ __forceinline__ float fast_exp2(float x) {            // the hardware's approximation (2 ulp)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack_bf16(float low, float high) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(low, high);
  return *reinterpret_cast<const uint32_t*>(&v);
}
typedef unsigned long long pair32;                               // two 32-bit numbers, multiplied and added at once
__device__ __forceinline__ pair32 make_pair(float a, float b) {
  pair32 p;
  asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(a), "f"(b));
  return p;
}
__device__ __forceinline__ void split_pair(pair32 p, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(p));
}
__device__ __forceinline__ pair32 fma_pair(pair32 a, pair32 b, pair32 c) {
  pair32 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// what this thread wrote into shared memory becomes visible to the tensor cores (a barrier must follow)
__device__ __forceinline__ void fence_for_tensor_cores() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

__device__ __forceinline__ int first_visible(int position, int window, int chunk) {
  int first = 0;
  if (window > 0) first = max(first, position + 1 - window);
  if (chunk > 0) first = max(first, position - position % chunk);
  return first;
}

// A tile of 128 consecutive tokens of one request row.
struct QueryTile {
  int row, token0, here, position0, key_begin, key_end;          // key_begin is a multiple of 128
};
__device__ __forceinline__ QueryTile query_tile(int row, int tile, int begin, int count, int context, int window, int chunk) {
  QueryTile w;
  w.row = row;
  w.token0 = begin + tile * kTile;
  w.here = min(kTile, count - tile * kTile);
  w.position0 = context - count + tile * kTile;
  w.key_begin = first_visible(w.position0, window, chunk) / kTile * kTile;
  w.key_end = w.position0 + w.here;
  return w;
}
__device__ __forceinline__ bool find_tile(int index, const int* query_starts, const int* context_lens, int rows, int window,
                                          int chunk, QueryTile& w) {
  for (int r = 0; r < rows; ++r) {
    const int begin = query_starts[r], count = query_starts[r + 1] - begin;
    const int tiles = (count + kTile - 1) / kTile;
    if (index < tiles) {
      w = query_tile(r, index, begin, count, context_lens[r], window, chunk);
      return true;
    }
    index -= tiles;
  }
  return false;
}

// ROWS rows of 128 elements (key or value rows of one kv head, from the pages) into two swizzled halves at `dst`, by
// WARPS warps: a warp copies whole rows, sixteen lanes a row, two rows at a time.  Which cache rows its 2 * COPIES rows are
// is looked up once, a lane a row, and kept by the caller (the tile's other kv heads lie beside them): -1 for rows at `limit`
// and beyond and rows whose page was given back, which become zeros.
template <int ROWS, int WARPS>
__device__ __forceinline__ int cache_row(const int* __restrict__ table, int page_size, int key0, int limit, int warp, int lane) {
  constexpr int COPIES = ROWS / (2 * WARPS);
  static_assert(ROWS % (2 * WARPS) == 0 && 2 * COPIES <= 32, "a warp looks up its rows at once");
  const int key = key0 + (lane >> 1) * (2 * WARPS) + warp * 2 + (lane & 1);
  if (lane >= 2 * COPIES || key >= limit) return -1;
  const int block = key / page_size, page = table[block];
  return page < 0 ? -1 : page * page_size + (key - block * page_size);
}
template <int ROWS, int WARPS>
__device__ __forceinline__ void load_rows(uint32_t dst, const bf16* __restrict__ pages, int kv_heads, int kv_head, int mine,
                                          int warp, int lane) {
  constexpr int COPIES = ROWS / (2 * WARPS);
  const int piece = lane & 15, second = lane >> 4;
  const bf16* const from = pages + (size_t)kv_head * kDim + piece * 8;
  const size_t row_stride = (size_t)kv_heads * kDim;
#pragma unroll
  for (int i = 0; i < COPIES; ++i) {
    const int r = i * (2 * WARPS) + warp * 2 + second;
    const int row = __shfl_sync(0xffffffffu, mine, i * 2 + second);
    copy16(dst + (piece >> 3) * (ROWS * 128) + r * 128 + (((piece & 7) ^ (r & 7)) << 4),
           row >= 0 ? from + row * row_stride : pages, row >= 0);
  }
}

// Tensor memory for the CTA (by warp 0), and one barrier per entry of `count`.
__device__ __forceinline__ uint32_t allocate(uint32_t* place, uint32_t columns, uint64_t* barriers, int count) {
  if (threadIdx.x < 32) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(place)), "r"(columns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < count; ++i) barrier_init(smem_u32(barriers + i), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  tensor_fence_before_sync();
  __syncthreads();
  tensor_fence_after_sync();
  return *place;
}
__device__ __forceinline__ void release(uint32_t tmem, uint32_t columns) {
  tensor_fence_before_sync();
  __syncthreads();
  tensor_fence_after_sync();
  if (threadIdx.x < 32)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(columns) : "memory");
}
// Waits while `alive`; a wait that runs out says so and ends all waiting of this thread.
__device__ __forceinline__ void wait_alive(uint32_t barrier, uint32_t parity, bool& alive, int role) {
  if (alive && !wait_barrier(barrier, parity)) {
    g_mixed_error = role;
    alive = false;
  }
}

// ---------------------------------------------------------------------------------------------- row sums
// grid (heads, tiles of 128 queries), 256 threads.  log_sums [heads, tokens]: log2 of the sum over a query's visible keys
// of 2^(score log2 e).
__global__ void __launch_bounds__(256)
mixed_row_sums_tc_kernel(const bf16* __restrict__ q, long long q_stride, const bf16* __restrict__ k_pages,
                         const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                         const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, float scale2,
                         int window, int chunk, float* __restrict__ log_sums, int tokens) {
  extern __shared__ unsigned char dynamic[];
  __shared__ uint32_t tmem_place;
  __shared__ __align__(8) uint64_t barriers[2];
  __shared__ float tops[2][kTile], sums[2][kTile];
  QueryTile w;
  // (late tiles of a request see the most keys: they come first)
  if (!find_tile(gridDim.y - 1 - blockIdx.y, query_starts, context_lens, rows, window, chunk, w)) return;
  const uint32_t base = (smem_u32(dynamic) + 1023u) & ~1023u;
  const uint32_t q_at = base, k_at = base + kOperand;
  const int head = blockIdx.x, kv_head = head / (heads / kv_heads);
  const int* table = block_table + (size_t)w.row * table_width;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int tiles = (w.key_end - w.key_begin + kTile - 1) / kTile;
  const uint32_t tmem = allocate(&tmem_place, 256, barriers, 2);

  auto fetch = [&](int t) {
    if (t < tiles)
      load_rows<kTile, 8>(k_at + (t & 1) * kOperand, k_pages, kv_heads, kv_head,
                          cache_row<kTile, 8>(table, page_size, w.key_begin + t * kTile, w.key_end, warp, lane), warp, lane);
    copy_commit();
  };
  for (int i = threadIdx.x; i < kTile * 16; i += 256) {
    const int r = i / 16, piece = i % 16;
    const bool there = r < w.here;
    copy16(q_at + (piece >> 3) * kHalf + r * 128 + (((piece & 7) ^ (r & 7)) << 4),
           there ? q + (size_t)(w.token0 + r) * q_stride + (size_t)head * kDim + piece * 8 : q, there);
  }
  fetch(0);
  fetch(1);

  const int my_row = (warp & 3) * 32 + lane, half = warp >> 2;
  const int position = my_row < w.here ? w.position0 + my_row : -1;
  const int first = my_row < w.here ? first_visible(position, window, chunk) : 0;
  float top = -INFINITY, sum = 0.0f;
  auto process = [&](int t) {
    const int key0 = w.key_begin + t * kTile + half * 64;
    const bool whole = __all_sync(0xffffffffu, key0 >= first && key0 + 63 <= position);
#pragma unroll
    for (int part = 0; part < 2; ++part) {
      float s[32];
      tmem_load_32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (t & 1) * kTile + half * 64 + part * 32, s);
      if (!whole) {
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const int key = key0 + part * 32 + c;
          s[c] = key >= first && key <= position ? s[c] : -INFINITY;
        }
      }
      float most[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int c = 4; c < 32; ++c) most[c & 3] = fmaxf(most[c & 3], s[c]);
      const float next = fmaxf(top, fmaxf(fmaxf(most[0], most[1]), fmaxf(most[2], most[3])) * scale2);
      const float shift = next == -INFINITY ? 0.0f : next;        // (a row that has seen nothing yet: every term is 0)
      float more[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int c = 0; c < 32; ++c) more[c & 3] += fast_exp2(fmaf(s[c], scale2, -shift));
      sum = sum * fast_exp2(top - shift) + ((more[0] + more[1]) + (more[2] + more[3]));
      top = next;
    }
  };
  bool alive = true;
  constexpr uint32_t idesc = instruction_descriptor(kTile, kTile);
  for (int t = 0; t < tiles; ++t) {
    copy_wait<1>();
    fence_for_tensor_cores();
    tensor_fence_before_sync();                                  // (the scores two tiles back have been read)
    __syncthreads();
    if (warp == 0) {
      tensor_fence_after_sync();
      const uint32_t elected = elect_one();
      const uint32_t a = operand_low(q_at), b = operand_low(k_at + (t & 1) * kOperand);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const uint32_t step = (k >> 2) * (kHalf >> 4) + (k & 3) * 2;
        mma_bf16_ss_halves(tmem + (t & 1) * kTile, a + step, b + step, idesc, (uint32_t)(k > 0), elected);
      }
      mma_commit_elected(smem_u32(barriers + (t & 1)), elected);
    }
    if (t > 0) process(t - 1);
    wait_alive(smem_u32(barriers + (t & 1)), (t >> 1) & 1, alive, 1);
    tensor_fence_after_sync();
    fetch(t + 2);
  }
  process(tiles - 1);
  tops[half][my_row] = top;
  sums[half][my_row] = sum;
  copy_wait<0>();
  release(tmem, 256);                                            // (a barrier among other things)
  if (half == 0 && my_row < w.here) {
    const float other = tops[1][my_row], all = fmaxf(top, other);
    const float total = sum * fast_exp2(top - all) + sums[1][my_row] * fast_exp2(other - all);
    log_sums[(size_t)head * tokens + w.token0 + my_row] = all + log2f(total);
  }
}

// ---------------------------------------------------------------------------------------------- mixed weights
template <int COLUMNS>
__device__ __forceinline__ void tmem_request(uint32_t address, uint32_t (&r)[COLUMNS]) {
  static_assert(COLUMNS == 4 || COLUMNS == 8, "columns of one request");
  if constexpr (COLUMNS == 4)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(address) : "memory");
  else
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(address) : "memory");
}
// Waits for this thread's requests; the registers are operands so that nothing that uses them can be moved ahead of it.
__device__ __forceinline__ void tmem_request_wait(uint32_t (&r)[4]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;" : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]) : : "memory");
}
__device__ __forceinline__ void tmem_request_wait(uint32_t (&r)[8]) {
  asm volatile("tcgen05.wait::ld.sync.aligned;"
               : "+r"(r[0]), "+r"(r[1]), "+r"(r[2]), "+r"(r[3]), "+r"(r[4]), "+r"(r[5]), "+r"(r[6]), "+r"(r[7]) : : "memory");
}

__host__ __device__ constexpr int queries_for(int padded_heads) { return padded_heads == 32 ? 16 : 32; }
constexpr int kMixers = 256, kLoaders = 128;
constexpr int kMixerRegisters = 216, kLoaderRegisters = 72;      // together what 384 threads are launched with (168 each)
// The mixing matrix comes as a launch parameter: every thread uses the same number at the same time, and a parameter's
// reach the multiply-adds through the constant cache; the same numbers from shared memory cost 512 bytes of register
// writes per 16 of them and warp, which bound the kernel.
struct MixMatrix { float of[32 * 32]; };                         // [head][result head], rows of 8, 16 or 32

// Barriers of the mixing kernel: a stage's keys are there, its products are over, all scores of a tile are there.
enum { KEYS_FULL = 0, KEYS_FREE = 2, SCORES_FULL = 4, WEIGHTS_BARRIERS = 5 };

// What a CTA works on: Q queries and a segment of their tile's keys.  The items of a launch are counted from its last tile of
// queries backwards (late tiles of a request see the most keys: they come first), a tile's segments one after the other and
// within a segment its groups of Q queries; only items that exist are counted, so that a CTA which takes every n-th gets its
// share.
struct MixItem {
  QueryTile w;
  int sub, here, position0, token0, segment_begin, segment_end, seen_begin, seen_end;
  // the walk over the tiles: tile `tile` of row `row` is the batch's tile `index`, has `subs` groups of queries and `items`
  // items, and `passed` items lie behind it
  int row, tile, index, subs, items, passed;
};
__device__ __forceinline__ void start_mix_items(const int* query_starts, int rows, MixItem& m) {
  m.row = rows;
  m.tile = m.index = m.items = m.passed = 0;
  for (int r = 0; r < rows; ++r) m.index += (query_starts[r + 1] - query_starts[r] + kTile - 1) / kTile;
}
// Item `rank` of the launch (ranks ascend from call to call); false when there are no more.
template <int Q>
__device__ __forceinline__ bool mix_item(int rank, int first_tile, int slab_tiles, const int* query_starts,
                                         const int* context_lens, int window, int chunk, int segment_tiles, int key_columns,
                                         MixItem& m) {
  int tiles = 0;
  while (rank >= m.passed + m.items) {
    m.passed += m.items;
    m.items = 0;
    while (m.tile == 0) {
      if (m.row == 0) return false;
      --m.row;
      m.tile = (query_starts[m.row + 1] - query_starts[m.row] + kTile - 1) / kTile;
    }
    --m.tile;
    --m.index;
    if (m.index < first_tile) return false;
    if (m.index >= first_tile + slab_tiles) continue;
    const int begin = query_starts[m.row];
    m.w = query_tile(m.row, m.tile, begin, query_starts[m.row + 1] - begin, context_lens[m.row], window, chunk);
    tiles = min((m.w.key_end - m.w.key_begin + kTile - 1) / kTile, key_columns / kTile);
    m.subs = (m.w.here + Q - 1) / Q;
    m.items = m.subs * ((tiles + segment_tiles - 1) / segment_tiles);
  }
  tiles = min((m.w.key_end - m.w.key_begin + kTile - 1) / kTile, key_columns / kTile);
  const int local = rank - m.passed;
  m.sub = local % m.subs;
  m.here = min(Q, m.w.here - m.sub * Q);
  m.segment_begin = local / m.subs * segment_tiles;
  m.segment_end = min(m.segment_begin + segment_tiles, tiles);
  m.token0 = m.w.token0 + m.sub * Q;
  m.position0 = m.w.position0 + m.sub * Q;
  // the key tiles that one of these queries sees; the others of the segment are zeros
  m.seen_begin = max(m.segment_begin, (first_visible(m.position0, window, chunk) - m.w.key_begin) / kTile);
  m.seen_end = min(m.segment_end, (m.position0 + m.here - m.w.key_begin + kTile - 1) / kTile);
  return true;
}

// One CTA per SM goes over the items (a unit of Q queries, a segment of the keys), kMixers + kLoaders threads.  Mixer: key =
// its lane of the accumulators (four warps), half of the queries (two sets of four warps); the first of their warps
// issues the products as keys arrive.  Loaders: the key tiles of one kv head after the other, two stages ahead.  Stages and
// barrier phases run on across the items.
template <int HEADS>
__global__ void __launch_bounds__(kMixers + kLoaders, 1)
mixed_weights_tc_kernel(const bf16* __restrict__ q, long long q_stride, const bf16* __restrict__ k_pages,
                        const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                        const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, float scale2,
                        int window, int chunk, const __grid_constant__ MixMatrix mix,
                        const float* __restrict__ log_sums, int tokens, int first_tile, int slab_tiles,
                        int segment_tiles, int key_columns, bf16* __restrict__ mixed) {
  constexpr int Q = queries_for(HEADS), SET = Q / (kMixers / 128);
  constexpr int QB = HEADS == 32 ? 4 : 8;                        // queries a thread mixes at a time
  constexpr int GB = HEADS == 32 ? 4 : 2;                                          // heads whose scores it asks for at a time
  constexpr uint32_t COLUMNS = HEADS * Q;
  extern __shared__ unsigned char dynamic[];
  __shared__ uint32_t tmem_place;
  __shared__ __align__(8) uint64_t barriers[WEIGHTS_BARRIERS];
  __shared__ __align__(16) float sums_s[HEADS * Q];              // [head][query]
  const uint32_t base = (smem_u32(dynamic) + 1023u) & ~1023u;
  const uint32_t q_half = (uint32_t)(Q * heads) * 128u;          // bytes of a 64-element half of all the queries' rows
  const uint32_t k_at = base, q_at = base + 2 * kOperand;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int per_group = heads / kv_heads;
  const uint32_t bar = smem_u32(barriers);
  if (threadIdx.x == 0)
    for (int i = 0; i < WEIGHTS_BARRIERS; ++i) barrier_init(bar + i * 8, i < KEYS_FREE ? kLoaders : 1);
  const uint32_t tmem = allocate(&tmem_place, COLUMNS, nullptr, 0);
  bool alive = true;
  int step = 0;                                                  // key tiles (of one kv head) so far, over all items
  MixItem m;
  start_mix_items(query_starts, rows, m);

  if (threadIdx.x >= kMixers) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kLoaderRegisters));
    const int loader = warp - kMixers / 32;
    for (int rank = blockIdx.x; mix_item<Q>(rank, first_tile, slab_tiles, query_starts, context_lens, window, chunk,
                                            segment_tiles, key_columns, m); rank += gridDim.x) {
      const int* table = block_table + (size_t)m.w.row * table_width;
      for (int kt = m.seen_begin; kt < m.seen_end; ++kt) {
        const int mine = cache_row<kTile, kLoaders / 32>(table, page_size, m.w.key_begin + kt * kTile, m.w.key_end, loader, lane);
        for (int kv_head = 0; kv_head < kv_heads; ++kv_head, ++step) {
          const int stage = step & 1;
          if (step >= 2) wait_alive(bar + (KEYS_FREE + stage) * 8, ((step >> 1) - 1) & 1, alive, 2);
          __syncwarp();
          load_rows<kTile, kLoaders / 32>(k_at + stage * kOperand, k_pages, kv_heads, kv_head, mine, loader, lane);
          copy_commit();
          if (step > 0) {                                        // the stage before: it has landed, and the tensor cores may see it
            copy_wait<1>();
            fence_for_tensor_cores();
            barrier_arrive(bar + (KEYS_FULL + (stage ^ 1)) * 8);
          }
        }
      }
    }
    if (step > 0) {
      copy_wait<0>();
      fence_for_tensor_cores();
      barrier_arrive(bar + (KEYS_FULL + ((step - 1) & 1)) * 8);
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kMixerRegisters));
    const int quarter = (warp & 3) * 32, set = warp >> 2;
    const uint32_t lane_at = tmem + ((uint32_t)quarter << 16);
    const size_t head_stride = (size_t)kTile * key_columns;
    int tile_count = 0;                                          // tiles of keys so far, over all items
    for (int rank = blockIdx.x; mix_item<Q>(rank, first_tile, slab_tiles, query_starts, context_lens, window, chunk,
                                            segment_tiles, key_columns, m); rank += gridDim.x) {
      bf16* const result = mixed + ((size_t)(m.index - first_tile) * heads * kTile + m.sub * Q) * key_columns;
      for (int kt = m.segment_begin; kt < m.segment_end; ++kt) {
        if (kt >= m.seen_begin && kt < m.seen_end) continue;
        for (int i = threadIdx.x; i < heads * m.here * 16; i += kMixers) {
          const int row = i / 16, h = row / m.here, query = row - h * m.here;
          *reinterpret_cast<uint4*>(result + h * head_stride + (size_t)query * key_columns + kt * kTile + i % 16 * 8) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
      if (m.seen_begin >= m.seen_end) continue;
      asm volatile("bar.sync 1, %0;" ::"n"(kMixers) : "memory");    // (the last item's sums and queries are used no more)
      // row head * Q + query of the second operand
      for (int i = threadIdx.x; i < heads * Q * 16; i += kMixers) {
        const int row = i / 16, piece = i % 16, query = row % Q;
        const bool there = query < m.here;
        copy16(q_at + (piece >> 3) * q_half + row * 128 + (((piece & 7) ^ (row & 7)) << 4),
               there ? q + (size_t)(m.token0 + query) * q_stride + (size_t)(row / Q) * kDim + piece * 8 : q, there);
      }
      copy_commit();
      for (int i = threadIdx.x; i < HEADS * Q; i += kMixers) {
        const int g = i / Q, query = i % Q;
        sums_s[i] = g < heads && query < m.here ? log_sums[(size_t)g * tokens + m.token0 + query] : 0.0f;
      }
      copy_wait<0>();
      fence_for_tensor_cores();
      for (int kt = m.seen_begin; kt < m.seen_end; ++kt, ++tile_count) {
        tensor_fence_before_sync();                              // (the last tile's scores have been read)
        asm volatile("bar.sync 1, %0;" ::"n"(kMixers) : "memory");
        if (warp == 0) {
          tensor_fence_after_sync();
          const uint32_t elected = elect_one();
          for (int group = 0; group < kv_heads; ++group, ++step) {
            const int stage = step & 1;
            wait_alive(bar + (KEYS_FULL + stage) * 8, (step >> 1) & 1, alive, 2);
            __syncwarp();
            tensor_fence_after_sync();
            const uint32_t a = operand_low(k_at + stage * kOperand);
            for (int n0 = 0; n0 < per_group * Q; n0 += 256) {
              const uint32_t idesc = instruction_descriptor(kTile, min(256, per_group * Q - n0));
              const uint32_t b = operand_low(q_at + (uint32_t)(group * per_group * Q + n0) * 128u);
#pragma unroll
              for (int k = 0; k < 8; ++k)
                mma_bf16_ss_halves(tmem + group * per_group * Q + n0, a + (k >> 2) * (kHalf >> 4) + (k & 3) * 2,
                                   b + (k >> 2) * (q_half >> 4) + (k & 3) * 2, idesc, (uint32_t)(k > 0), elected);
            }
            mma_commit_elected(bar + (KEYS_FREE + stage) * 8, elected);
          }
          mma_commit_elected(bar + SCORES_FULL * 8, elected);
        }
        wait_alive(bar + SCORES_FULL * 8, tile_count & 1, alive, 2);
        __syncwarp();
        tensor_fence_after_sync();
        const int key = m.w.key_begin + kt * kTile + quarter + lane;
#pragma unroll 1
        for (int q0 = set * SET; q0 < (set + 1) * SET; q0 += QB) {
          bool seen[QB];
#pragma unroll
          for (int i = 0; i < QB; ++i) {
            const int position = m.position0 + q0 + i;
            seen[i] = q0 + i < m.here && key <= position && key >= first_visible(position, window, chunk);
          }
          pair32 acc[QB][HEADS / 2];
#pragma unroll
          for (int i = 0; i < QB; ++i)
#pragma unroll
            for (int h = 0; h < HEADS / 2; ++h) acc[i][h] = 0ull;
          auto request = [&](int g, uint32_t (&scores)[GB][QB]) {  // (columns behind the last head: read, and not used)
#pragma unroll
            for (int e = 0; e < GB; ++e) tmem_request<QB>(lane_at + (g + e) * Q + q0, scores[e]);
          };
          auto add_heads = [&](int g, uint32_t (&scores)[GB][QB]) {
#pragma unroll
            for (int e = 0; e < GB; ++e)
#pragma unroll
              for (int i = 0; i < QB; ++i) {
                const float v = fast_exp2(fmaf(__uint_as_float(scores[e][i]), scale2, -sums_s[(g + e) * Q + q0 + i]));
                scores[e][i] = seen[i] && g + e < heads ? __float_as_uint(v) : 0u;
              }
#pragma unroll
            for (int e = 0; e < GB; ++e) {
              pair32 weight[QB];
#pragma unroll
              for (int i = 0; i < QB; ++i) weight[i] = make_pair(__uint_as_float(scores[e][i]), __uint_as_float(scores[e][i]));
#pragma unroll
              for (int h = 0; h < HEADS / 2; ++h) {
                const pair32 both = make_pair(mix.of[(g + e) * HEADS + 2 * h], mix.of[(g + e) * HEADS + 2 * h + 1]);
#pragma unroll
                for (int i = 0; i < QB; ++i) acc[i][h] = fma_pair(both, weight[i], acc[i][h]);
              }
            }
          };
          auto arrived = [&](uint32_t (&scores)[GB][QB]) {
#pragma unroll
            for (int e = 0; e < GB; ++e) tmem_request_wait(scores[e]);
          };
          // some heads' scores are on their way while the heads before are added
          uint32_t front[GB][QB], back[GB][QB];
          request(0, front);
          arrived(front);
#pragma unroll 1
          for (int g = 0; g < heads; g += 2 * GB) {
            request(g + GB, back);
            add_heads(g, front);
            arrived(back);
            if (g + 2 * GB < heads) request(g + 2 * GB, front);
            add_heads(g + GB, back);
            if (g + 2 * GB < heads) arrived(front);
          }
          // neighbouring lanes hold neighbouring keys: the even one stores both keys of a query, the odd one of the next query
          const bool even = (lane & 1) == 0;
#pragma unroll
          for (int i = 0; i < QB; i += 2) {
            const int query = q0 + i + (even ? 0 : 1);
            bf16* to = result + (size_t)query * key_columns + kt * kTile + quarter + (lane & ~1);
            const bool there = query < m.here;
#pragma unroll
            for (int h = 0; h < HEADS / 2; ++h) {
              float a0, a1, b0, b1;
              split_pair(acc[i][h], a0, a1);
              split_pair(acc[i + 1][h], b0, b1);
              const float other0 = __shfl_xor_sync(0xffffffffu, even ? b0 : a0, 1);
              const float other1 = __shfl_xor_sync(0xffffffffu, even ? b1 : a1, 1);
              if (there && 2 * h < heads)
                *reinterpret_cast<uint32_t*>(to + (2 * h) * head_stride) = even ? pack_bf16(a0, other0) : pack_bf16(other0, b0);
              if (there && 2 * h + 1 < heads)
                *reinterpret_cast<uint32_t*>(to + (2 * h + 1) * head_stride) = even ? pack_bf16(a1, other1) : pack_bf16(other1, b1);
            }
          }
        }
      }
    }
  }
  __syncwarp();
  release(tmem, COLUMNS);
}

// ---------------------------------------------------------------------------------------------- values
constexpr int kSlab = 64;                           // keys per step
constexpr int kSlabStages = 3;
constexpr int kSlabWeights = kTile * 128, kSlabValues = 2 * kSlab * 128;      // bytes of its two operands

// grid (heads, tiles of 128 queries), 256 threads.
__global__ void __launch_bounds__(256)
mixed_values_tc_kernel(const bf16* __restrict__ mixed, bf16* __restrict__ out, const bf16* __restrict__ v_pages,
                       const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                       const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, int window,
                       int chunk, int first_tile, int key_columns) {
  extern __shared__ unsigned char dynamic[];
  __shared__ uint32_t tmem_place;
  __shared__ __align__(8) uint64_t barriers[kSlabStages];
  QueryTile w;
  const int local_tile = gridDim.y - 1 - blockIdx.y;             // (late tiles of a request see the most keys: they come first)
  if (!find_tile(first_tile + local_tile, query_starts, context_lens, rows, window, chunk, w)) return;
  const uint32_t base = (smem_u32(dynamic) + 1023u) & ~1023u;
  const int head = blockIdx.x, kv_head = head / (heads / kv_heads);
  const int* table = block_table + (size_t)w.row * table_width;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int slabs = min((w.key_end - w.key_begin + kSlab - 1) / kSlab, key_columns / kSlab);
  const bf16* const weights = mixed + ((size_t)local_tile * heads + head) * kTile * key_columns;
  const uint32_t tmem = allocate(&tmem_place, 128, barriers, kSlabStages);

  auto fetch = [&](int s) {
    if (s < slabs) {
      const uint32_t a = base + (s % kSlabStages) * (kSlabWeights + kSlabValues), v = a + kSlabWeights;
#pragma unroll
      for (int i = 0; i < kTile * 8; i += 256) {
        const int r = (i + threadIdx.x) / 8, piece = threadIdx.x % 8;
        const bool there = r < w.here;
        copy16(a + r * 128 + ((piece ^ (r & 7)) << 4), there ? weights + (size_t)r * key_columns + s * kSlab + piece * 8 : weights, there);
      }
      load_rows<kSlab, 8>(v, v_pages, kv_heads, kv_head,
                          cache_row<kSlab, 8>(table, page_size, w.key_begin + s * kSlab, w.key_end, warp, lane), warp, lane);
    }
    copy_commit();
  };
  fetch(0);
  fetch(1);
  bool alive = true;
  constexpr uint32_t idesc = instruction_descriptor(kTile, kDim, true);
  for (int s = 0; s < slabs; ++s) {
    const int stage = s % kSlabStages;
    copy_wait<1>();
    fence_for_tensor_cores();
    __syncthreads();
    if (warp == 0) {
      tensor_fence_after_sync();
      const uint32_t elected = elect_one();
      const uint32_t at = base + stage * (kSlabWeights + kSlabValues);
      const uint32_t a = operand_low(at), b = operand_low_mn_major(at + kSlabWeights, kSlab * 128);
#pragma unroll
      for (int k = 0; k < kSlab / 16; ++k)
        mma_bf16_ss_halves(tmem, a + k * 2, b + k * 128, idesc, (uint32_t)(s > 0 || k > 0), elected);
      mma_commit_elected(smem_u32(barriers + stage), elected);
    }
    if (s > 0) wait_alive(smem_u32(barriers + (s - 1) % kSlabStages), ((s - 1) / kSlabStages) & 1, alive, 3);
    fetch(s + 2);                                                // (into the stage of the slab before this one)
  }
  wait_alive(smem_u32(barriers + (slabs - 1) % kSlabStages), ((slabs - 1) / kSlabStages) & 1, alive, 3);
  tensor_fence_after_sync();
  const int row = (warp & 3) * 32 + lane, column = (warp >> 2) * 64;
  bf16* to = out + ((size_t)(w.token0 + row) * heads + head) * kDim + column;
#pragma unroll
  for (int part = 0; part < 2; ++part) {
    float o[32];
    tmem_load_32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + column + part * 32, o);
    if (row < w.here) {
#pragma unroll
      for (int c = 0; c < 32; c += 8)
        *reinterpret_cast<uint4*>(to + part * 32 + c) = make_uint4(pack_bf16(o[c], o[c + 1]), pack_bf16(o[c + 2], o[c + 3]),
                                                                   pack_bf16(o[c + 4], o[c + 5]), pack_bf16(o[c + 6], o[c + 7]));
    }
  }
  copy_wait<0>();
  release(tmem, 128);
}

int reserve(const void* kernel, size_t smem, const char* what) {
  const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (err == cudaSuccess) return MIR_OK;
  mir_set_error("%s: cannot reserve %zu bytes of shared memory: %s", what, smem, cudaGetErrorString(err));
  return MIR_CUDA_ERROR;
}

}  // namespace

// 0, or which kernel gave up a bounded wait (1 row sums, 2 weights, 3 values).  Synchronises the device.
MIR_EXPORT int mir_mixed_attention_tc_error() {
  int value = -1;
  if (cudaMemcpyFromSymbol(&value, g_mixed_error, sizeof(int)) != cudaSuccess) return -1;
  return value;
}

MIR_EXPORT int mir_mixed_prefill_tc_takes(int heads, int dim, int value_dim) {
  return heads > 0 && heads <= 32 && dim == kDim && value_dim == kDim;
}

// Portions: row r brings the tokens query_starts[r] .. query_starts[r + 1] of qkv and out and has context_lens[r] keys after
// the step.  tiles: at least the number of tiles of 128 tokens over all rows; the mixed weights of slab_tiles of them at a
// time pass through `mixed` (slab_tiles * heads * 128 * key_columns * 2 bytes), key_columns a multiple of 128: enough for the
// keys from the multiple of 128 below the first one a tile sees to its last query.  scale is above zero.  mix is in host
// memory.
MIR_EXPORT int mir_mixed_prefill_attention_tc_bf16(const void* q, long long q_stride, void* out, const void* k_pages,
                                                   const void* v_pages, const int* block_table, int table_width,
                                                   const int* query_starts, const int* context_lens, int rows, int tokens,
                                                   int page_size, int heads, int kv_heads, int dim, int value_dim, float scale,
                                                   const float* mix, int window, int chunk, int tiles, int slab_tiles,
                                                   int key_columns, int segment_tiles, float* log_sums, void* mixed,
                                                   cudaStream_t stream) {
  if (rows == 0 || tokens == 0 || tiles == 0) return MIR_OK;
  if (!mir_mixed_prefill_tc_takes(heads, dim, value_dim) || kv_heads <= 0 || heads % kv_heads || page_size <= 0 ||
      table_width <= 0 || window < 0 || chunk < 0 || rows < 0 || tiles < 0 || tiles > 8191 || slab_tiles <= 0 ||
      key_columns <= 0 || key_columns % kTile || segment_tiles <= 0 || !(scale > 0.0f) || q_stride % 8 || (uintptr_t)q % 16 ||
      (uintptr_t)out % 16 || (uintptr_t)k_pages % 16 || (uintptr_t)v_pages % 16 || (uintptr_t)mixed % 16) {
    mir_set_error("mixed_prefill_attention_tc: sizes or alignment the kernels do not take (heads %d over %d, widths %d and "
                  "%d, tiles %d, scale %g)", heads, kv_heads, dim, value_dim, tiles, scale);
    return MIR_BAD_ARGUMENT;
  }
  const float scale2 = scale * kLog2e;
  const bf16 *qb = (const bf16*)q, *kb = (const bf16*)k_pages, *vb = (const bf16*)v_pages;
  int status;
  const size_t sums_smem = 3 * kOperand + 1024;
  if ((status = reserve((const void*)mixed_row_sums_tc_kernel, sums_smem, "mixed_row_sums_tc")) != MIR_OK) return status;
  mixed_row_sums_tc_kernel<<<dim3(heads, tiles), 256, sums_smem, stream>>>(
      qb, q_stride, kb, block_table, table_width, query_starts, context_lens, rows, page_size, heads, kv_heads, scale2, window,
      chunk, log_sums, tokens);
  if ((status = mir_check_launch("mixed_row_sums_tc")) != MIR_OK) return status;
  const int segments = (key_columns / kTile + segment_tiles - 1) / segment_tiles;
  const size_t values_smem = kSlabStages * (kSlabWeights + kSlabValues) + 1024;
  if ((status = reserve((const void*)mixed_values_tc_kernel, values_smem, "mixed_values_tc")) != MIR_OK) return status;
  for (int from = 0; from < tiles; from += slab_tiles) {
    const int here = std::min(slab_tiles, tiles - from);
#define MIR_WEIGHTS(H)                                                                                                   \
  do {                                                                                                                   \
    MixMatrix matrix = {};                                                                                              \
    for (int g = 0; g < heads; ++g)                                                                                     \
      for (int h = 0; h < heads; ++h) matrix.of[g * H + h] = mix[h * heads + g];                                        \
    const size_t smem = 2 * kOperand + (size_t)queries_for(H) * heads * 256 + 1024;                                      \
    if ((status = reserve((const void*)mixed_weights_tc_kernel<H>, smem, "mixed_weights_tc")) != MIR_OK) return status;  \
    mixed_weights_tc_kernel<H><<<dim3(std::min(mir_sm_count(), here * segments * (kTile / queries_for(H)))), kMixers + kLoaders, smem, stream>>>( \
        qb, q_stride, kb, block_table, table_width, query_starts, context_lens, rows, page_size, heads, kv_heads, scale2, \
        window, chunk, matrix, log_sums, tokens, from, here, segment_tiles,                  \
        key_columns, (bf16*)mixed);                           \
  } while (0)
    if (heads <= 8) MIR_WEIGHTS(8);
    else if (heads <= 16) MIR_WEIGHTS(16);
    else MIR_WEIGHTS(32);
#undef MIR_WEIGHTS
    if ((status = mir_check_launch("mixed_weights_tc")) != MIR_OK) return status;
    mixed_values_tc_kernel<<<dim3(heads, here), 256, values_smem, stream>>>(
        (const bf16*)mixed, (bf16*)out, vb, block_table, table_width, query_starts, context_lens, rows, page_size, heads,
        kv_heads, window, chunk, from, key_columns);
    if ((status = mir_check_launch("mixed_values_tc")) != MIR_OK) return status;
  }
  return MIR_OK;
}
