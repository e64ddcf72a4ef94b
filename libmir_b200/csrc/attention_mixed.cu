// Paged softmax attention whose heads' weights are mixed before they meet the values ("talking heads" behind the softmax):
//     p_g(i, j) = softmax_j(scale q_g(i) . k(j))      out_h(i) = sum_j (sum_g M[h, g] p_g(i, j)) v(j)
// with k, v of the kv head that serves g and h.  Key j is visible to the query at position i iff j <= i and (window == 0 or
// j > i - window) and (chunk == 0 or j / chunk == i / chunk).
//
// This is the reference kernel: portions and decoded tokens, any head counts and widths, float or bf16 storage, one CTA
// per token.  A key's mixed weight in one head needs its weight in every head, so the CTA first finds each head's maximum
// and sum over all visible keys, then walks over the keys again, 32 at a time: weights of all heads, their mixture, and
// the sums over the values, all 32-bit.  Keys are taken in runs of 32 from the first visible one, so a position's result
// is bit-identical however the step was cut.
#include <cfloat>
#include "common.cuh"

using namespace mir;

namespace {

constexpr int kWarps = 8;
constexpr int kKeys = 32;

template <typename T>
__device__ __forceinline__ float dot_row(const float* q, const T* k, int dim) {
  float dot = 0.0f;
  if (dim % 8 == 0) {                                            // (then every key row starts on a 16-byte boundary)
    for (int d = 0; d < dim; d += 8) {
      float k8[8];
      load8(k + d, k8);
#pragma unroll
      for (int i = 0; i < 8; ++i) dot = fmaf(q[d + i], k8[i], dot);
    }
  } else {
    for (int d = 0; d < dim; ++d) dot = fmaf(q[d], to_float(k[d]), dot);
  }
  return dot;
}

// dynamic shared memory (floats): q [heads * dim] | acc [heads * value_dim] | maximum [heads] | 1 / sum [heads] |
// weights [heads * kKeys] | mixed [heads * kKeys]
template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
paged_attention_mixed_kernel(const T* __restrict__ q, long long q_stride, T* __restrict__ out, const T* __restrict__ k_pages,
                             const T* __restrict__ v_pages, const int* __restrict__ block_table, int table_width,
                             const int* __restrict__ row_of_token, const int* __restrict__ positions, int page_size,
                             int heads, int kv_heads, int dim, int value_dim, float scale, const float* __restrict__ mix,
                             int window, int chunk) {
  extern __shared__ __align__(16) float shared[];
  __shared__ size_t key_row[kKeys];
  float* const q_s = shared;
  float* const acc = q_s + heads * dim;
  float* const top = acc + heads * value_dim;
  float* const inverse = top + heads;
  float* const weights = inverse + heads;
  float* const mixed = weights + heads * kKeys;
  const int token = blockIdx.x, thread = threadIdx.x, lane = thread & 31, warp = thread >> 5;
  const int position = positions[token];
  if (position < 0) return;                                      // a padding row of a captured batch
  const int per_group = heads / kv_heads;
  const int* table = block_table + (size_t)row_of_token[token] * table_width;
  int first_key = (window > 0 && position + 1 > window) ? position + 1 - window : 0;
  if (chunk > 0) first_key = max(first_key, position - position % chunk);
  for (int i = thread; i < heads * dim; i += blockDim.x) q_s[i] = to_float(q[(size_t)token * q_stride + i]);
  for (int i = thread; i < heads * value_dim; i += blockDim.x) acc[i] = 0.0f;
  __syncthreads();
  auto row_of_key = [&](int key) { return (size_t)table[key / page_size] * page_size + key % page_size; };
  auto score = [&](int head, int key) {
    return dot_row(q_s + head * dim, k_pages + (row_of_key(key) * kv_heads + head / per_group) * dim, dim) * scale;
  };
  for (int head = warp; head < heads; head += kWarps) {
    float running_max = -FLT_MAX, sum = 0.0f;
    for (int base = first_key; base <= position; base += kKeys) {
      const bool valid = base + lane <= position;
      const float value = valid ? score(head, base + lane) : -FLT_MAX;
      const float next = fmaxf(running_max, warp_max(value));
      sum = sum * expf(running_max - next) + warp_sum(valid ? expf(value - next) : 0.0f);
      running_max = next;
    }
    if (lane == 0) { top[head] = running_max; inverse[head] = 1.0f / sum; }
  }
  __syncthreads();
  for (int base = first_key; base <= position; base += kKeys) {
    const int count = min(kKeys, position - base + 1);
    if (thread < count) key_row[thread] = row_of_key(base + thread);
    for (int head = warp; head < heads; head += kWarps)
      weights[head * kKeys + lane] = lane < count ? expf(score(head, base + lane) - top[head]) * inverse[head] : 0.0f;
    __syncthreads();
    for (int i = thread; i < heads * kKeys; i += blockDim.x) {
      const int head = i / kKeys, j = i % kKeys;
      float sum = 0.0f;
      for (int g = 0; g < heads; ++g) sum = fmaf(mix[head * heads + g], weights[g * kKeys + j], sum);
      mixed[i] = sum;
    }
    __syncthreads();
    for (int i = thread; i < heads * value_dim; i += blockDim.x) {
      const int head = i / value_dim, d = i - head * value_dim;
      const T* values = v_pages + (size_t)(head / per_group) * value_dim + d;
      float sum = acc[i];
      for (int j = 0; j < count; ++j)
        sum = fmaf(mixed[head * kKeys + j], to_float(values[key_row[j] * kv_heads * value_dim]), sum);
      acc[i] = sum;
    }
    __syncthreads();
  }
  for (int i = thread; i < heads * value_dim; i += blockDim.x)
    out[(size_t)token * heads * value_dim + i] = from_float<T>(acc[i]);
}

template <typename T>
int launch(const void* q, long long q_stride, void* out, const void* k_pages, const void* v_pages, const int* block_table,
           int table_width, const int* row_of_token, const int* positions, int tokens, int page_size, int heads,
           int kv_heads, int dim, int value_dim, float scale, const float* mix, int window, int chunk, cudaStream_t stream) {
  const size_t smem = ((size_t)heads * (dim + value_dim + 2 + 2 * kKeys)) * sizeof(float);
  if (smem > 224 * 1024) {
    mir_set_error("paged_attention_mixed: %d heads of %d and %d channels do not fit into shared memory", heads, dim, value_dim);
    return MIR_BAD_ARGUMENT;
  }
  if (smem > 40 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(paged_attention_mixed_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                 (int)smem);
    if (err != cudaSuccess) {
      mir_set_error("paged_attention_mixed: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(err));
      return MIR_CUDA_ERROR;
    }
  }
  paged_attention_mixed_kernel<T><<<dim3(tokens), dim3(kWarps * 32), smem, stream>>>(
      (const T*)q, q_stride, (T*)out, (const T*)k_pages, (const T*)v_pages, block_table, table_width, row_of_token, positions,
      page_size, heads, kv_heads, dim, value_dim, scale, mix, window, chunk);
  return mir_check_launch("paged_attention_mixed");
}

}  // namespace

// q: first query element of token 0, row stride q_stride in elements; mix [heads, heads] 32-bit, indexed [result head,
// head]; window, chunk: 0 for none; out [tokens, heads * value_dim] contiguous.
MIR_EXPORT int mir_paged_attention_mixed(int bf16, const void* q, long long q_stride, void* out, const void* k_pages,
                                         const void* v_pages, const int* block_table, int table_width,
                                         const int* row_of_token, const int* positions, int tokens, int page_size, int heads,
                                         int kv_heads, int dim, int value_dim, float scale, const float* mix, int window,
                                         int chunk, cudaStream_t stream) {
  if (tokens == 0) return MIR_OK;
  if (tokens < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || value_dim <= 0 || page_size <= 0 ||
      table_width <= 0 || window < 0 || chunk < 0 || mix == nullptr) {
    mir_set_error("paged_attention_mixed: bad sizes (tokens %d, heads %d, kv heads %d, dim %d, value dim %d)", tokens, heads,
                  kv_heads, dim, value_dim);
    return MIR_BAD_ARGUMENT;
  }
  if (bf16)
    return launch<__nv_bfloat16>(q, q_stride, out, k_pages, v_pages, block_table, table_width, row_of_token, positions, tokens,
                                 page_size, heads, kv_heads, dim, value_dim, scale, mix, window, chunk, stream);
  return launch<float>(q, q_stride, out, k_pages, v_pages, block_table, table_width, row_of_token, positions, tokens, page_size,
                       heads, kv_heads, dim, value_dim, scale, mix, window, chunk, stream);
}
