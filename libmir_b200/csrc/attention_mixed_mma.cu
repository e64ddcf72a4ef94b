// bfloat16 attention whose heads' weights are mixed before they meet the values (attention_mixed.cu says what is computed;
// it is the reference kernel for every other size and type).  A key's mixed weight in one head needs its normalised
// weight in every head, so the softmax comes first; and every output head needs every key's mixed weights, which is more
// than one SM can hold for all heads, so the mixed weights pass through memory, in the order the products read them.
//
// Portions of prompts (tensor cores, mma.sync m16n8k16, head widths 64 and 128, up to 32 heads), three kernels:
//   mixed_row_sums     the log of each (head, query)'s sum over its visible keys: Q K^T and a running softmax, no values
//   mixed_weights      16 queries and 64 keys at a time, a warp takes 8 keys: Q K^T of ALL heads, whose accumulators hold
//                      the same (query, key) places in the same thread, so that the mixture is arithmetic in registers
//                      (packed 32-bit multiply-adds); the mixed weights leave as bfloat16 in the order in which
//                      the next kernel's threads want them as the first operand of their products
//   mixed_values       64 queries of one head: mixed weights times values
// Key tiles start at multiples of 64 positions, so all three see the same tiles whatever the run or window.
//
// Single tokens (any head counts, widths that are multiples of 8 up to 256), two kernels, keys in parts of 64:
//   mixed_decode_scores   the scores of one part and kv head, and the part's maximum and sum per head
//   mixed_decode_values   every head's weights from its parts' sums, their mixture for this kv head's query heads, and the
//                         part's share of the result; whoever finishes a kv head's last part adds the parts' shares (they
//                         are normalised already)
// Scores, softmax, mixture and sums are 32-bit.  A part or tile starts at a place that depends on the query's position
// alone, and parts are added in ascending order.
#include <algorithm>
#include <cfloat>
#include "common.cuh"

using namespace mir;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int kKeys = 64;                           // keys per tile, and per part of a single token's keys
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy16(void* dst, const void* src, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float low, float high) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(low, high);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float exp2_fast(float x) {             // the hardware's approximation (2 ulp)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two 32-bit numbers side by side, and a multiply-add on both at once
typedef unsigned long long pair32;
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

// The first key that the query at `position` sees.
__device__ __forceinline__ int first_visible(int position, int window, int chunk) {
  int first = 0;
  if (window > 0) first = max(first, position + 1 - window);
  if (chunk > 0) first = max(first, position - position % chunk);
  return first;
}

// Which request row and which of its tiles of 64 tokens the `index`-th tile of the batch is; false behind the last one.
__device__ __forceinline__ bool find_tile(int index, const int* query_starts, int rows, int& row, int& tile) {
  for (int r = 0; r < rows; ++r) {
    const int tiles = (query_starts[r + 1] - query_starts[r] + 63) / 64;
    if (index < tiles) { row = r; tile = index; return true; }
    index -= tiles;
  }
  return false;
}

// Rows key0 .. key0 + 63 of one kv head from the pages into shared rows of W + 8 elements; rows at `limit` and beyond, and
// rows whose page was given back, are zeros.
template <int W, int THREADS>
__device__ __forceinline__ void load_rows(bf16* dst, const bf16* __restrict__ pages, const int* __restrict__ table,
                                          int page_size, int kv_heads, int kv_head, int key0, int limit) {
  constexpr int PIECES = W / 8, ROWS = THREADS / PIECES;
  const int sub = threadIdx.x / PIECES, piece = threadIdx.x % PIECES;
#pragma unroll
  for (int i = 0; i < kKeys; i += ROWS) {
    const int key = key0 + i + sub;
    const int page = key < limit ? table[key / page_size] : -1;
    const bf16* from = page >= 0 ? pages + (((size_t)page * page_size + key % page_size) * kv_heads + kv_head) * W + piece * 8 : pages;
    copy16(dst + (size_t)(i + sub) * (W + 8) + piece * 8, from, page >= 0);
  }
}

// ---------------------------------------------------------------------------------------------- prompts: row sums
// grid (heads, tiles of 64 queries), 128 threads.  log_sums [heads, tokens]: log2 of the sum over a query's visible keys of
// 2^(score log2 e), -inf where nothing is seen.
template <int D>
__global__ void __launch_bounds__(128)
mixed_row_sums_kernel(const bf16* __restrict__ q, long long q_stride, const bf16* __restrict__ k_pages,
                      const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                      const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, float scale2,
                      int window, int chunk, float* __restrict__ log_sums, int tokens) {
  extern __shared__ __align__(16) unsigned char shared[];
  constexpr int LD = D + 8;
  bf16* const q_s = reinterpret_cast<bf16*>(shared);
  bf16* const k_s = q_s + 64 * LD;
  int row, tile;
  if (!find_tile(blockIdx.y, query_starts, rows, row, tile)) return;
  const int head = blockIdx.x, kv_head = head / (heads / kv_heads);
  const int begin = query_starts[row], count = query_starts[row + 1] - begin;
  const int t0 = tile * 64, here = min(64, count - t0);
  const int p0 = context_lens[row] - count + t0;                 // position of the tile's first query
  const int* table = block_table + (size_t)row * table_width;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int key_begin = first_visible(p0, window, chunk) / kKeys * kKeys, key_end = p0 + here;

  for (int i = threadIdx.x; i < 64 * (D / 8); i += 128) {
    const int r = i / (D / 8), piece = i % (D / 8);
    const bool there = r < here;
    copy16(q_s + r * LD + piece * 8, there ? q + (size_t)(begin + t0 + r) * q_stride + (size_t)head * D + piece * 8 : q, there);
  }
  load_rows<D, 128>(k_s, k_pages, table, page_size, kv_heads, kv_head, key_begin, key_end);
  copy_commit();
  copy_wait<0>();
  __syncthreads();
  uint32_t a[D / 16][4];
#pragma unroll
  for (int k = 0; k < D / 16; ++k) ldmatrix_x4(a[k], q_s + (warp * 16 + (lane & 15)) * LD + k * 16 + (lane >> 4) * 8);
  int position[2], first[2];
  float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = warp * 16 + (lane >> 2) + 8 * e;
    position[e] = r < here ? p0 + r : -1;
    first[e] = r < here ? first_visible(p0 + r, window, chunk) : 0;
  }
  int buffer = 0;
  for (int key0 = key_begin; key0 < key_end; key0 += kKeys, buffer ^= 1) {
    if (key0 != key_begin) { copy_wait<0>(); __syncthreads(); }
    if (key0 + kKeys < key_end) {
      load_rows<D, 128>(k_s + (buffer ^ 1) * 64 * LD, k_pages, table, page_size, kv_heads, kv_head, key0 + kKeys, key_end);
      copy_commit();
    }
    const bf16* tile_s = k_s + buffer * 64 * LD;
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[nt][e] = 0.0f;
#pragma unroll
    for (int k = 0; k < D / 16; ++k) {
#pragma unroll
      for (int nt = 0; nt < 8; nt += 2) {
        uint32_t b[4];
        ldmatrix_x4(b, tile_s + (nt * 8 + (lane & 7) + ((lane >> 4) & 1) * 8) * LD + k * 16 + ((lane >> 3) & 1) * 8);
        mma(s[nt], a[k], b[0], b[1]);
        mma(s[nt + 1], a[k], b[2], b[3]);
      }
    }
    float tile_top[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = key0 + nt * 8 + (lane & 3) * 2 + (e & 1), r = e >> 1;
        s[nt][e] = key <= position[r] && key >= first[r] ? s[nt][e] * scale2 : -INFINITY;
        tile_top[r] = fmaxf(tile_top[r], s[nt][e]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      tile_top[r] = fmaxf(tile_top[r], __shfl_xor_sync(0xffffffffu, tile_top[r], 1));
      tile_top[r] = fmaxf(tile_top[r], __shfl_xor_sync(0xffffffffu, tile_top[r], 2));
      const float next = fmaxf(top[r], tile_top[r]);
      if (next == -INFINITY) continue;
      float more = 0.0f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) more += exp2_fast(s[nt][2 * r] - next) + exp2_fast(s[nt][2 * r + 1] - next);
      sum[r] = sum[r] * exp2_fast(top[r] - next) + more;
      top[r] = next;
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
    const int local = warp * 16 + (lane >> 2) + 8 * r;
    if ((lane & 3) == 0 && local < here)
      log_sums[(size_t)head * tokens + begin + t0 + local] = top[r] + log2f(sum[r]);
  }
}

// ---------------------------------------------------------------------------------------------- prompts: mixed weights
// grid (segments of the keys, 4 x tiles of 64 queries), 256 threads: 16 queries, all heads, `segment_tiles` tiles of keys.
// mixed: per (tile of 16 queries, head, block of 8 keys) 32 lanes x 8 bytes; lane l holds the queries l / 4 and l / 4 + 8 at
// the keys 2 (l % 4) and the next one.
constexpr int kStages = 3;

template <int D, int HEADS>
__global__ void __launch_bounds__(256, 1)
mixed_weights_kernel(const bf16* __restrict__ q, long long q_stride, const bf16* __restrict__ k_pages,
                     const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                     const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, float scale2,
                     int window, int chunk, const float* __restrict__ mix, const float* __restrict__ log_sums, int tokens,
                     int first_tile, int segment_tiles, int key_blocks, uint2* __restrict__ mixed) {
  extern __shared__ __align__(16) unsigned char shared[];
  constexpr int LD = D + 8;
  const int q_ld = heads * D + 8;
  pair32* const mix_s = reinterpret_cast<pair32*>(shared);                           // [HEADS][HEADS], both halves equal
  float* const sums_s = reinterpret_cast<float*>(mix_s + HEADS * HEADS);             // [HEADS][16]
  bf16* const k_s = reinterpret_cast<bf16*>(sums_s + HEADS * 16);
  bf16* const q_s = k_s + kStages * kKeys * LD;
  int row, tile;
  if (!find_tile(first_tile + blockIdx.y / 4, query_starts, rows, row, tile)) return;
  const int begin = query_starts[row], count = query_starts[row + 1] - begin;
  const int t0 = tile * 64 + (blockIdx.y & 3) * 16;
  if (t0 >= count) return;
  const int here = min(16, count - t0);
  const int p0 = context_lens[row] - count + t0;
  const int key_begin = first_visible(p0, window, chunk) / kKeys * kKeys, key_end = p0 + here;
  const int tiles = (key_end - key_begin + kKeys - 1) / kKeys;
  const int from_tile = blockIdx.x * segment_tiles;
  const int to_tile = min(min(from_tile + segment_tiles, tiles), key_blocks / 8);
  if (from_tile >= to_tile) return;
  const int* table = block_table + (size_t)row * table_width;
  const int thread = threadIdx.x, lane = thread & 31, warp = thread >> 5;
  const int per_group = heads / kv_heads;

  // the sequence of key tiles this CTA goes through: for every tile of keys, every kv head
  const int steps = (to_tile - from_tile) * kv_heads;
  auto fetch = [&](int step) {
    if (step < steps) {
      const int key0 = key_begin + (from_tile + step / kv_heads) * kKeys;
      load_rows<D, 256>(k_s + (step % kStages) * kKeys * LD, k_pages, table, page_size, kv_heads, step % kv_heads, key0, key_end);
    }
    copy_commit();                                               // (an empty group where there is nothing left to fetch)
  };
  for (int i = thread; i < 16 * heads * (D / 8); i += 256) {
    const int r = i / (heads * (D / 8)), piece = i - r * (heads * (D / 8));
    const bool there = r < here;
    copy16(q_s + (size_t)r * q_ld + piece * 8, there ? q + (size_t)(begin + t0 + r) * q_stride + piece * 8 : q, there);
  }
  fetch(0);
  fetch(1);
  for (int i = thread; i < HEADS * HEADS; i += 256) {
    const int h = i / HEADS, g = i % HEADS;
    const float m = h < heads && g < heads ? mix[h * heads + g] : 0.0f;
    mix_s[i] = make_pair(m, m);
  }
  for (int i = thread; i < HEADS * 16; i += 256) {
    const int g = i / 16, r = i % 16;
    sums_s[i] = g < heads && r < here ? log_sums[(size_t)g * tokens + begin + t0 + r] : 0.0f;
  }
  int position[2], first[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = (lane >> 2) + 8 * e;
    position[e] = r < here ? p0 + r : -1;
    first[e] = r < here ? first_visible(p0 + r, window, chunk) : 0;
  }
  const bf16* const a_at = q_s + (size_t)(lane & 15) * q_ld + (lane >> 4) * 8;
  uint2* const tile_out = mixed + (size_t)blockIdx.y * heads * key_blocks * 32 + lane;
  int step = 0;
  for (int kt = from_tile; kt < to_tile; ++kt) {
    const int key0 = key_begin + kt * kKeys + warp * 8;
    bool seen[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = key0 + (lane & 3) * 2 + (e & 1);
      seen[e] = key <= position[e >> 1] && key >= first[e >> 1];
    }
    pair32 weights[HEADS][2];
    uint32_t b[D / 32][4];
    int used = per_group;
#pragma unroll
    for (int g = 0; g < HEADS; ++g) {
      weights[g][0] = 0ull;
      weights[g][1] = 0ull;
      if (g < heads) {
        if (used == per_group) {                                 // the next kv head's keys
          copy_wait<1>();
          __syncthreads();
          fetch(step + 2);
          const bf16* tile_s = k_s + (step % kStages) * kKeys * LD + (warp * 8 + (lane & 7)) * LD + (lane >> 3) * 8;
#pragma unroll
          for (int k = 0; k < D / 32; ++k) ldmatrix_x4(b[k], tile_s + k * 32);
          ++step;
          used = 0;
        }
        ++used;
        float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int k = 0; k < D / 32; ++k) {
          uint32_t a[4];
          ldmatrix_x4(a, a_at + g * D + k * 32);
          mma(s, a, b[k][0], b[k][1]);
          ldmatrix_x4(a, a_at + g * D + k * 32 + 16);
          mma(s, a, b[k][2], b[k][3]);
        }
        const float low = sums_s[g * 16 + (lane >> 2)], high = sums_s[g * 16 + (lane >> 2) + 8];
        const float w0 = seen[0] ? exp2_fast(fmaf(s[0], scale2, -low)) : 0.0f;
        const float w1 = seen[1] ? exp2_fast(fmaf(s[1], scale2, -low)) : 0.0f;
        const float w2 = seen[2] ? exp2_fast(fmaf(s[2], scale2, -high)) : 0.0f;
        const float w3 = seen[3] ? exp2_fast(fmaf(s[3], scale2, -high)) : 0.0f;
        weights[g][0] = make_pair(w0, w1);
        weights[g][1] = make_pair(w2, w3);
      }
    }
    const size_t block = (size_t)(kt * 8 + warp);
#pragma unroll 2
    for (int h = 0; h < heads; ++h) {
      pair32 upper = 0ull, lower = 0ull;
      const ulonglong2* m = reinterpret_cast<const ulonglong2*>(mix_s + h * HEADS);
#pragma unroll
      for (int g = 0; g < HEADS; g += 2) {
        const ulonglong2 both = m[g / 2];
        upper = fma_pair(both.x, weights[g][0], upper);
        lower = fma_pair(both.x, weights[g][1], lower);
        upper = fma_pair(both.y, weights[g + 1][0], upper);
        lower = fma_pair(both.y, weights[g + 1][1], lower);
      }
      float u0, u1, l0, l1;
      split_pair(upper, u0, u1);
      split_pair(lower, l0, l1);
      tile_out[((size_t)h * key_blocks + block) * 32] = make_uint2(pack_bf16(u0, u1), pack_bf16(l0, l1));
    }
  }
  copy_wait<0>();
}

// ---------------------------------------------------------------------------------------------- prompts: values
// grid (heads, tiles of 64 queries), 128 threads; a warp takes 16 queries and the whole value width.
template <int W>
__global__ void __launch_bounds__(128)
mixed_values_kernel(const uint2* __restrict__ mixed, bf16* __restrict__ out, const bf16* __restrict__ v_pages,
                    const int* __restrict__ block_table, int table_width, const int* __restrict__ query_starts,
                    const int* __restrict__ context_lens, int rows, int page_size, int heads, int kv_heads, int window,
                    int chunk, int first_tile, int key_blocks) {
  extern __shared__ __align__(16) unsigned char shared[];
  constexpr int LD = W + 8;
  bf16* const v_s = reinterpret_cast<bf16*>(shared);
  int row, tile;
  if (!find_tile(first_tile + blockIdx.y, query_starts, rows, row, tile)) return;
  const int head = blockIdx.x, kv_head = head / (heads / kv_heads);
  const int begin = query_starts[row], count = query_starts[row + 1] - begin;
  const int t0 = tile * 64, here = min(64, count - t0);
  const int p0 = context_lens[row] - count + t0;
  const int* table = block_table + (size_t)row * table_width;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int key_begin = first_visible(p0, window, chunk) / kKeys * kKeys, key_end = p0 + here;
  // this warp's own queries and keys
  const int mine = min(16, here - warp * 16);
  const int my_begin = mine > 0 ? first_visible(p0 + warp * 16, window, chunk) / kKeys * kKeys : 0;
  const int my_end = mine > 0 ? min(p0 + warp * 16 + mine, my_begin + key_blocks * 8) : 0;
  const uint2* weights = mixed + ((size_t)(blockIdx.y * 4 + warp) * heads + head) * key_blocks * 32 + lane;

  float o[W / 8][4];
#pragma unroll
  for (int nt = 0; nt < W / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[nt][e] = 0.0f;
  load_rows<W, 128>(v_s, v_pages, table, page_size, kv_heads, kv_head, key_begin, key_end);
  copy_commit();
  int buffer = 0;
  for (int key0 = key_begin; key0 < key_end; key0 += kKeys, buffer ^= 1) {
    const bool concerned = key0 >= my_begin && key0 < my_end;
    uint2 low[4], high[4];
    if (concerned) {
      const uint2* from = weights + (size_t)((key0 - my_begin) / 8) * 32;
#pragma unroll
      for (int k = 0; k < 4; ++k) { low[k] = from[2 * k * 32]; high[k] = from[(2 * k + 1) * 32]; }
    }
    copy_wait<0>();
    __syncthreads();
    if (key0 + kKeys < key_end) {
      load_rows<W, 128>(v_s + (buffer ^ 1) * kKeys * LD, v_pages, table, page_size, kv_heads, kv_head, key0 + kKeys, key_end);
      copy_commit();
    }
    if (!concerned) continue;
    const bf16* tile_s = v_s + buffer * kKeys * LD + ((lane & 7) + ((lane >> 3) & 1) * 8) * LD + ((lane >> 4) & 1) * 8;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const uint32_t a[4] = {low[k].x, low[k].y, high[k].x, high[k].y};
#pragma unroll
      for (int nt = 0; nt < W / 8; nt += 2) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, tile_s + k * 16 * LD + nt * 8);
        mma(o[nt], a, b[0], b[1]);
        mma(o[nt + 1], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int local = warp * 16 + (lane >> 2) + 8 * r;
    if (local >= here) continue;
    bf16* to = out + ((size_t)(begin + t0 + local) * heads + head) * W + (lane & 3) * 2;
#pragma unroll
    for (int nt = 0; nt < W / 8; ++nt)
      *reinterpret_cast<uint32_t*>(to + nt * 8) = pack_bf16(o[nt][2 * r], o[nt][2 * r + 1]);
  }
}

// ---------------------------------------------------------------------------------------------- single tokens
// grid (parts of 64 keys, rows, kv heads x blocks of R query heads), 128 threads.  LANES lanes read a key's row, 16 bytes
// each.  scores [rows, heads, parts * 64] in units of log2 e; stats [rows, heads, parts, 2]: a part's maximum and its sum
// of 2^(score - maximum).
template <int R, int LANES>
__global__ void __launch_bounds__(128)
mixed_decode_scores_kernel(const bf16* __restrict__ q, long long q_stride, const bf16* __restrict__ k_pages,
                           const int* __restrict__ block_table, int table_width, const int* __restrict__ positions,
                           int page_size, int heads, int kv_heads, int dim, float scale2, int window, int chunk, int parts,
                           float* __restrict__ scores, float2* __restrict__ stats, int* __restrict__ arrived) {
  constexpr int PASSES = kKeys * LANES / 128, SUBS = 32 / LANES;
  __shared__ float s_s[R][kKeys];
  grid_launch_dependents();
  grid_dependency_wait();
  const int part = blockIdx.x, row = blockIdx.y;
  const int position = positions[row];
  if (position < 0) return;
  const int first = first_visible(position, window, chunk);
  const int key0 = first + part * kKeys;
  if (key0 > position) return;
  const int count = min(kKeys, position + 1 - key0);
  const int per_group = heads / kv_heads, blocks = (per_group + R - 1) / R;
  const int kv_head = blockIdx.z / blocks, head0 = kv_head * per_group + (blockIdx.z % blocks) * R;
  const int mine = min(R, (kv_head + 1) * per_group - head0);
  if (part == 0 && threadIdx.x == 0) arrived[(size_t)row * gridDim.z + blockIdx.z] = 0;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int piece = lane % LANES, sub = lane / LANES;
  const bool reads = piece * 8 < dim;
  const int* table = block_table + (size_t)row * table_width;
  uint4 raw[PASSES];
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int j = (p * 4 + warp) * SUBS + sub, key = key0 + j;
    raw[p] = make_uint4(0u, 0u, 0u, 0u);
    if (reads && j < count)
      raw[p] = *reinterpret_cast<const uint4*>(
          k_pages + (((size_t)table[key / page_size] * page_size + key % page_size) * kv_heads + kv_head) * dim + piece * 8);
  }
  float query[R][8];
#pragma unroll
  for (int r = 0; r < R; ++r) {
#pragma unroll
    for (int i = 0; i < 8; ++i) query[r][i] = 0.0f;
    if (reads && r < mine) load8(q + (size_t)row * q_stride + (size_t)(head0 + r) * dim + piece * 8, query[r]);
  }
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw[p]);
    float k8[8];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      k8[2 * i] = f.x;
      k8[2 * i + 1] = f.y;
    }
    const int j = (p * 4 + warp) * SUBS + sub;
    // R sums over LANES lanes: in each step a lane hands half of its heads over, as long as it has more than one
    float dot[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      dot[r] = 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) dot[r] = fmaf(query[r][i], k8[i], dot[r]);
    }
    int head = 0;
#pragma unroll
    for (int o = LANES / 2, held = R; o > 0; o >>= 1) {
      const bool upper = (piece & o) != 0;
      if (held > 1) {
        held /= 2;
        head += upper ? held : 0;
#pragma unroll
        for (int r = 0; r < R / 2; ++r) {
          if (r < held) {
            const float other = __shfl_xor_sync(0xffffffffu, upper ? dot[r] : dot[r + held], o);
            dot[r] = (upper ? dot[r + held] : dot[r]) + other;
          }
        }
      } else {
        dot[0] += __shfl_xor_sync(0xffffffffu, dot[0], o);
      }
    }
    if (piece % (LANES / R) == 0) s_s[head][j] = dot[0] * scale2;
  }
  __syncthreads();
  for (int r = warp; r < mine; r += 4) {
    const float a = lane < count ? s_s[r][lane] : -INFINITY, b = lane + 32 < count ? s_s[r][lane + 32] : -INFINITY;
    const float top = warp_max(fmaxf(a, b));
    const float sum = warp_sum(exp2f(a - top) + exp2f(b - top));
    const size_t at = (size_t)row * heads + head0 + r;
    float* to = scores + at * parts * kKeys + part * kKeys;
    to[lane] = a;
    to[lane + 32] = b;
    if (lane == 0) stats[at * parts + part] = make_float2(top, sum);
  }
}

// The same grid.  dynamic shared memory (floats): log_sums [heads] | weights [heads * 64] | mixed [R * 64] | sums [4 * R *
// value_dim].  partial [rows, parts, heads, value_dim] 32-bit; arrived [rows, gridDim.z]: parts that are done, set to zero by
// the kernel before.
template <int R, int LANES>
__global__ void __launch_bounds__(128)
mixed_decode_values_kernel(const bf16* __restrict__ v_pages, const int* __restrict__ block_table, int table_width,
                           const int* __restrict__ positions, int page_size, int heads, int kv_heads, int value_dim,
                           int window, int chunk, int parts, const float* __restrict__ mix, const float* __restrict__ scores,
                           const float2* __restrict__ stats, float* __restrict__ partial, int* __restrict__ arrived,
                           bf16* __restrict__ out) {
  constexpr int PASSES = kKeys * LANES / 128, SUBS = 32 / LANES;
  extern __shared__ __align__(16) float shared_f[];
  float* const log_sums = shared_f;
  float* const weights = log_sums + (heads + 3) / 4 * 4;
  float* const mixed = weights + heads * kKeys;
  float* const sums = mixed + R * kKeys;
  grid_launch_dependents();
  grid_dependency_wait();
  const int part = blockIdx.x, row = blockIdx.y;
  const int position = positions[row];
  if (position < 0) return;
  const int first = first_visible(position, window, chunk);
  const int key0 = first + part * kKeys;
  if (key0 > position) return;
  const int count = min(kKeys, position + 1 - key0);
  const int filled = min(parts, (position - first) / kKeys + 1);  // parts that hold any key
  const int per_group = heads / kv_heads, blocks = (per_group + R - 1) / R;
  const int kv_head = blockIdx.z / blocks, head0 = kv_head * per_group + (blockIdx.z % blocks) * R;
  const int mine = min(R, (kv_head + 1) * per_group - head0);
  const int thread = threadIdx.x, lane = thread & 31, warp = thread >> 5;
  const int piece = lane % LANES, sub = lane / LANES;
  const bool reads = piece * 8 < value_dim;
  const int* table = block_table + (size_t)row * table_width;
  uint4 raw[PASSES];
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int j = (p * 4 + warp) * SUBS + sub, key = key0 + j;
    raw[p] = make_uint4(0u, 0u, 0u, 0u);
    if (reads && j < count)
      raw[p] = *reinterpret_cast<const uint4*>(
          v_pages + (((size_t)table[key / page_size] * page_size + key % page_size) * kv_heads + kv_head) * value_dim + piece * 8);
  }
  // four threads go over a head's parts, then put their sums together
  for (int base = 0; base < heads; base += 32) {
    const int g = base + thread / 4;
    const float2* mine_stats = stats + ((size_t)row * heads + min(g, heads - 1)) * parts;
    float top = -INFINITY, sum = 0.0f;
#pragma unroll 4
    for (int p = thread & 3; p < filled; p += 4) {
      const float2 one = mine_stats[p];
      const float next = fmaxf(top, one.x);
      sum = fmaf(one.y, exp2f(one.x - next), sum * exp2f(top - next));
      top = next;
    }
    float all = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
    all = fmaxf(all, __shfl_xor_sync(0xffffffffu, all, 2));
    sum = top == -INFINITY ? 0.0f : sum * exp2f(top - all);
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if ((thread & 3) == 0 && g < heads) log_sums[g] = all + log2f(sum);
  }
  __syncthreads();
  // (behind `count` the scores are -inf)
  const float* part_scores = scores + (size_t)row * heads * parts * kKeys + part * kKeys;
#pragma unroll 4
  for (int i = thread; i < heads * (kKeys / 4); i += 128) {
    const int g = i / (kKeys / 4), j = i % (kKeys / 4) * 4;
    const float4 four = *reinterpret_cast<const float4*>(part_scores + (size_t)g * parts * kKeys + j);
    const float log_sum = log_sums[g];
    *reinterpret_cast<float4*>(weights + g * kKeys + j) =
        make_float4(exp2f(four.x - log_sum), exp2f(four.y - log_sum), exp2f(four.z - log_sum), exp2f(four.w - log_sum));
  }
  __syncthreads();
  for (int i = thread; i < R * (kKeys / 4); i += 128) {
    const int r = i / (kKeys / 4), j = i % (kKeys / 4) * 4;
    float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (r < mine) {
      const float* factors = mix + (size_t)(head0 + r) * heads;
#pragma unroll 8
      for (int g = 0; g < heads; ++g) {
        const float m = __ldg(factors + g);
        const float4 w = *reinterpret_cast<const float4*>(weights + g * kKeys + j);
        sum.x = fmaf(m, w.x, sum.x);
        sum.y = fmaf(m, w.y, sum.y);
        sum.z = fmaf(m, w.z, sum.z);
        sum.w = fmaf(m, w.w, sum.w);
      }
    }
    *reinterpret_cast<float4*>(mixed + r * kKeys + j) = sum;
  }
  __syncthreads();
  float acc[R][8];
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[r][i] = 0.0f;
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int j = (p * 4 + warp) * SUBS + sub;
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw[p]);
    float v8[8];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v8[2 * i] = f.x;
      v8[2 * i + 1] = f.y;
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float w = mixed[r * kKeys + j];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[r][i] = fmaf(w, v8[i], acc[r][i]);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r)
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int o = LANES; o < 32; o <<= 1) acc[r][i] += __shfl_xor_sync(0xffffffffu, acc[r][i], o);
  if (sub == 0 && reads) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      float* to = sums + (size_t)(warp * R + r) * value_dim + piece * 8;
      *reinterpret_cast<float4*>(to) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
      *reinterpret_cast<float4*>(to + 4) = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
    }
  }
  __syncthreads();
  // this part's share; the CTA that brings the last one of a row's parts adds them, in ascending order
  const size_t stride = (size_t)heads * value_dim;
  float* const shares = partial + ((size_t)row * parts * heads + head0) * value_dim;
  __shared__ int last;
  for (int i = thread; i < mine * value_dim; i += 128) {
    const int quarter = R * value_dim;
    shares[part * stride + i] = (sums[i] + sums[quarter + i]) + (sums[2 * quarter + i] + sums[3 * quarter + i]);
  }
  __threadfence();
  __syncthreads();
  if (thread == 0) last = atomicAdd(arrived + (size_t)row * gridDim.z + blockIdx.z, 1) == filled - 1;
  __syncthreads();
  if (!last) return;
  __threadfence();
  for (int c = thread * 4; c < mine * value_dim; c += 512) {
    float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
    for (int p = 0; p < filled; ++p) {
      const float4 share = __ldcg(reinterpret_cast<const float4*>(shares + p * stride + c));
      sum.x += share.x; sum.y += share.y; sum.z += share.z; sum.w += share.w;
    }
    *reinterpret_cast<uint2*>(out + ((size_t)row * heads + head0) * value_dim + c) =
        make_uint2(pack_bf16(sum.x, sum.y), pack_bf16(sum.z, sum.w));
  }
}

template <typename Kernel>
int reserve(Kernel kernel, size_t smem, const char* what) {
  if (smem <= 48 * 1024) return MIR_OK;
  const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (err == cudaSuccess) return MIR_OK;
  mir_set_error("%s: cannot reserve %zu bytes of shared memory: %s", what, smem, cudaGetErrorString(err));
  return MIR_CUDA_ERROR;
}

size_t weights_shared(int dim, int heads, int padded_heads) {
  return (size_t)padded_heads * padded_heads * 8 + (size_t)padded_heads * 16 * 4 + (size_t)kStages * kKeys * (dim + 8) * 2 +
         (size_t)16 * (heads * dim + 8) * 2;
}

int padded_heads(int heads) { return heads <= 8 ? 8 : (heads <= 16 ? 16 : 32); }

}  // namespace

MIR_EXPORT int mir_mixed_prefill_takes(int heads, int dim, int value_dim) {
  return heads > 0 && heads <= 32 && (dim == 64 || dim == 128) && (value_dim == 64 || value_dim == 128) &&
         weights_shared(dim, heads, padded_heads(heads)) <= 227 * 1024;
}

// Portions: row r brings the tokens query_starts[r] .. query_starts[r + 1] of qkv and out and has context_lens[r] keys after
// the step.  tiles: at least the number of tiles of 64 tokens over all rows; the mixed weights of slab_tiles of them at a
// time pass through `mixed` (slab_tiles * 4 * heads * key_blocks * 256 bytes), key_blocks blocks of 8 keys per tile of 16
// queries: enough for the keys from the multiple of 64 below the first visible one to the last query.
MIR_EXPORT int mir_mixed_prefill_attention_bf16(const void* q, long long q_stride, void* out, const void* k_pages,
                                                const void* v_pages, const int* block_table, int table_width,
                                                const int* query_starts, const int* context_lens, int rows, int tokens,
                                                int page_size, int heads, int kv_heads, int dim, int value_dim, float scale,
                                                const float* mix, int window, int chunk, int tiles, int slab_tiles,
                                                int key_blocks, int segment_tiles, float* log_sums, void* mixed,
                                                cudaStream_t stream) {
  if (rows == 0 || tokens == 0 || tiles == 0) return MIR_OK;
  if (!mir_mixed_prefill_takes(heads, dim, value_dim) || kv_heads <= 0 || heads % kv_heads || page_size <= 0 ||
      table_width <= 0 || window < 0 || chunk < 0 || rows < 0 || tiles < 0 || tiles > 16383 || slab_tiles <= 0 ||
      key_blocks <= 0 || key_blocks % 8 || segment_tiles <= 0 || q_stride % 8 || (uintptr_t)q % 16 || (uintptr_t)out % 4 ||
      (uintptr_t)k_pages % 16 || (uintptr_t)v_pages % 16 || (uintptr_t)mixed % 8) {
    mir_set_error("mixed_prefill_attention: sizes or alignment the kernels do not take (heads %d over %d, widths %d and %d, "
                  "tiles %d)", heads, kv_heads, dim, value_dim, tiles);
    return MIR_BAD_ARGUMENT;
  }
  const float scale2 = scale * kLog2e;
  const bf16 *qb = (const bf16*)q, *kb = (const bf16*)k_pages, *vb = (const bf16*)v_pages;
  int status;
#define MIR_SUMS(D)                                                                                                     \
  do {                                                                                                                  \
    const size_t smem = (size_t)3 * 64 * (D + 8) * 2;                                                                   \
    if ((status = reserve(mixed_row_sums_kernel<D>, smem, "mixed_row_sums")) != MIR_OK) return status;                  \
    mixed_row_sums_kernel<D><<<dim3(heads, tiles), 128, smem, stream>>>(                                                \
        qb, q_stride, kb, block_table, table_width, query_starts, context_lens, rows, page_size, heads, kv_heads, scale2, \
        window, chunk, log_sums, tokens);                                                                               \
  } while (0)
  if (dim == 64) MIR_SUMS(64);
  else MIR_SUMS(128);
#undef MIR_SUMS
  if ((status = mir_check_launch("mixed_row_sums")) != MIR_OK) return status;
  const int segments = (key_blocks / 8 + segment_tiles - 1) / segment_tiles;
  for (int from = 0; from < tiles; from += slab_tiles) {
    const int here = std::min(slab_tiles, tiles - from);
#define MIR_WEIGHTS(D, H)                                                                                               \
  do {                                                                                                                  \
    const size_t smem = weights_shared(D, heads, H);                                                                    \
    if ((status = reserve(mixed_weights_kernel<D, H>, smem, "mixed_weights")) != MIR_OK) return status;                 \
    mixed_weights_kernel<D, H><<<dim3(segments, here * 4), 256, smem, stream>>>(                                        \
        qb, q_stride, kb, block_table, table_width, query_starts, context_lens, rows, page_size, heads, kv_heads, scale2, \
        window, chunk, mix, log_sums, tokens, from, segment_tiles, key_blocks, (uint2*)mixed);                          \
  } while (0)
#define MIR_WEIGHTS_FOR(D)                    \
  if (heads <= 8) MIR_WEIGHTS(D, 8);          \
  else if (heads <= 16) MIR_WEIGHTS(D, 16);   \
  else MIR_WEIGHTS(D, 32)
    if (dim == 64) { MIR_WEIGHTS_FOR(64); }
    else { MIR_WEIGHTS_FOR(128); }
#undef MIR_WEIGHTS_FOR
#undef MIR_WEIGHTS
    if ((status = mir_check_launch("mixed_weights")) != MIR_OK) return status;
#define MIR_VALUES(W)                                                                                                   \
  do {                                                                                                                  \
    const size_t smem = (size_t)2 * kKeys * (W + 8) * 2;                                                                \
    if ((status = reserve(mixed_values_kernel<W>, smem, "mixed_values")) != MIR_OK) return status;                      \
    mixed_values_kernel<W><<<dim3(heads, here), 128, smem, stream>>>(                                                   \
        (const uint2*)mixed, (bf16*)out, vb, block_table, table_width, query_starts, context_lens, rows, page_size, heads, \
        kv_heads, window, chunk, from, key_blocks);                                                                     \
  } while (0)
    if (value_dim == 64) MIR_VALUES(64);
    else MIR_VALUES(128);
#undef MIR_VALUES
    if ((status = mir_check_launch("mixed_values")) != MIR_OK) return status;
  }
  return MIR_OK;
}

MIR_EXPORT int mir_mixed_decode_takes(int heads, int kv_heads, int dim, int value_dim) {
  return heads > 0 && heads <= 256 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && dim % 8 == 0 && dim <= 256 &&
         value_dim > 0 && value_dim % 8 == 0 && value_dim <= 256;
}

// Single tokens: row r's query is row r of q.  parts: at least the parts of 64 keys that any row sees; scores [rows, heads,
// parts * 64], stats [rows, heads, parts, 2] and partial [rows, parts, heads, value_dim] are 32-bit scratch, arrived [rows,
// heads] integers.
MIR_EXPORT int mir_mixed_decode_attention_bf16(const void* q, long long q_stride, void* out, const void* k_pages,
                                               const void* v_pages, const int* block_table, int table_width,
                                               const int* positions, int rows, int page_size, int heads, int kv_heads,
                                               int dim, int value_dim, float scale, const float* mix, int window, int chunk,
                                               int parts, float* scores, float* stats, float* partial, int* arrived,
                                               cudaStream_t stream) {
  if (rows == 0) return MIR_OK;
  if (!mir_mixed_decode_takes(heads, kv_heads, dim, value_dim) || page_size <= 0 || table_width <= 0 || window < 0 ||
      chunk < 0 || rows < 0 || rows > 65535 || parts <= 0 || q_stride % 8 || (uintptr_t)q % 16 || (uintptr_t)out % 8 ||
      (uintptr_t)k_pages % 16 || (uintptr_t)v_pages % 16 || (uintptr_t)partial % 16 || (uintptr_t)scores % 16) {
    mir_set_error("mixed_decode_attention: sizes or alignment the kernels do not take (heads %d over %d, widths %d and %d, "
                  "parts %d)", heads, kv_heads, dim, value_dim, parts);
    return MIR_BAD_ARGUMENT;
  }
  const int per_group = heads / kv_heads;
  const int block = per_group == 1 ? 1 : (per_group == 2 ? 2 : (per_group <= 4 ? 4 : 8));
  const dim3 grid(parts, rows, kv_heads * ((per_group + block - 1) / block));
  const float scale2 = scale * kLog2e;
  int status;
#define MIR_BY_LANES(CALL, width) \
  if (width <= 64) CALL(8);       \
  else if (width <= 128) CALL(16); \
  else CALL(32)
#define MIR_BY_BLOCK(CALL)       \
  switch (block) {               \
    case 1: CALL(1); break;      \
    case 2: CALL(2); break;      \
    case 4: CALL(4); break;      \
    default: CALL(8); break;     \
  }
#define MIR_SCORES_LANES(L)                                                                                              \
  status = mir_launch("mixed_decode_scores", mixed_decode_scores_kernel<kBlock, L>, grid, dim3(128), 0, stream, 0,      \
                      (const bf16*)q, q_stride, (const bf16*)k_pages, block_table, table_width, positions, page_size, heads, \
                      kv_heads, dim, scale2, window, chunk, parts, scores, (float2*)stats, arrived)
#define MIR_SCORES(R)                       \
  do {                                      \
    constexpr int kBlock = R;               \
    MIR_BY_LANES(MIR_SCORES_LANES, dim);    \
  } while (0)
  MIR_BY_BLOCK(MIR_SCORES)
  if (status != MIR_OK) return status;
  const size_t smem = ((size_t)(heads + 3) / 4 * 4 + (size_t)heads * kKeys + (size_t)block * kKeys + (size_t)4 * block * value_dim) * 4;
#define MIR_VALUES_LANES(L)                                                                                              \
  do {                                                                                                                   \
    status = reserve(mixed_decode_values_kernel<kBlock, L>, smem, "mixed_decode_values");                               \
    if (status == MIR_OK)                                                                                                \
      status = mir_launch("mixed_decode_values", mixed_decode_values_kernel<kBlock, L>, grid, dim3(128), smem, stream, 0, \
                          (const bf16*)v_pages, block_table, table_width, positions, page_size, heads, kv_heads,        \
                          value_dim, window, chunk, parts, mix, (const float*)scores, (const float2*)stats, partial,    \
                          arrived, (bf16*)out);                                                                         \
  } while (0)
#define MIR_VALUES(R)                          \
  do {                                         \
    constexpr int kBlock = R;                  \
    MIR_BY_LANES(MIR_VALUES_LANES, value_dim); \
  } while (0)
  MIR_BY_BLOCK(MIR_VALUES)
#undef MIR_VALUES
#undef MIR_VALUES_LANES
#undef MIR_SCORES
#undef MIR_SCORES_LANES
#undef MIR_BY_BLOCK
#undef MIR_BY_LANES
  return status;
}
