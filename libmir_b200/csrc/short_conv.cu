// Short causal convolution per channel with an optional bias, then silu:
//     y[t, c] = silu(sum_j w[c, j] x[t - (taps - 1) + j, c] + bias[c])
// over a request's own tokens, with the taps - 1 inputs before the portion taken from the request's state (zeros at its
// start); then the state moves on to the portion's last inputs.  Sums are 32-bit, taps in ascending order.
//
//   short_conv_silu       one thread per token and channel, any number of taps, any alignment
//   short_conv_silu_wide  up to 4 taps: a thread takes 16 bytes of neighbouring channels and a run of tokens and keeps
//                         the last inputs in registers, so an input is read once per run; a request that brings one token
//                         has its state moved on by the thread that reads it
//   short_conv_tail       the state of every other request
#include "short_conv.cuh"

using namespace mir;

namespace {

__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// grid (tokens, ceil(channels / 256)).  x: the packed projection rows, channel c of token t at x[t * ldx + c].
template <typename T, typename TO>
__global__ void short_conv_silu_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w,
                                       const float* __restrict__ bias, const float* __restrict__ tail,
                                       const int* __restrict__ row_of_token, const int* __restrict__ query_starts,
                                       const int* __restrict__ state_slots, const int* __restrict__ positions,
                                       TO* __restrict__ out, int channels, int taps) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int token = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels || positions[token] < 0) return;
  const int row = row_of_token[token];
  const int start = query_starts[row];
  const int local = token - start;
  const float* old = tail + (size_t)state_slots[row] * (taps - 1) * channels;
  float acc = 0.0f;
  for (int j = 0; j < taps; ++j) {
    const int src = local - (taps - 1) + j;
    const float value = src >= 0 ? to_float(x[(size_t)(start + src) * ldx + c]) : old[(size_t)(taps - 1 + src) * channels + c];
    acc = fmaf(to_float(w[(size_t)c * taps + j]), value, acc);
  }
  if (bias != nullptr) acc += bias[c];
  out[(size_t)token * channels + c] = from_float<TO>(silu(acc));
}

template <typename T> struct Piece { static constexpr int kCount = 16 / sizeof(T); };

__device__ __forceinline__ void load_piece(const __nv_bfloat16* p, float (&v)[8]) { load8(p, v); }
__device__ __forceinline__ void load_piece(const float* p, float (&v)[4]) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <int V>
__device__ __forceinline__ void store_piece(float* p, const float (&v)[V]) {
#pragma unroll
  for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
}
template <int V>
__device__ __forceinline__ void store_piece(__nv_bfloat16* p, const float (&v)[V]) {
  alignas(16) __nv_bfloat162 packed[V / 2];
#pragma unroll
  for (int i = 0; i < V / 2; ++i) packed[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  if constexpr (V == 8) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(packed);
  else *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(packed);
}
template <int V>
__device__ __forceinline__ void load_floats(const float* p, float (&v)[V]) {
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    const float4 a = *reinterpret_cast<const float4*>(p + i);
    v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
  }
}

// grid (ceil(tokens / RUN), ceil(pieces / blockDim.x)); every pointer and stride of x, out, tail and bias on 16 bytes.
template <typename T, typename TO, int TAPS, int RUN>
__global__ void __launch_bounds__(128)
short_conv_silu_wide_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, const float* __restrict__ bias,
                            float* __restrict__ tail, const int* __restrict__ row_of_token,
                            const int* __restrict__ query_starts, const int* __restrict__ state_slots,
                            const int* __restrict__ positions, TO* __restrict__ out, int tokens, int channels) {
  constexpr int V = Piece<T>::kCount;
  grid_launch_dependents();
  grid_dependency_wait();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= channels) return;
  const int first = blockIdx.x * RUN, count = min(RUN, tokens - first);
  uint4 raw[RUN];                                   // all inputs of the run at once: one trip to memory
#pragma unroll
  for (int i = 0; i < RUN; ++i)
    raw[i] = i < count ? *reinterpret_cast<const uint4*>(x + (size_t)(first + i) * ldx + c) : make_uint4(0u, 0u, 0u, 0u);
  float taps[V][TAPS], shift[V];
#pragma unroll
  for (int v = 0; v < V; ++v)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) taps[v][j] = to_float(w[(size_t)(c + v) * TAPS + j]);
#pragma unroll
  for (int v = 0; v < V; ++v) shift[v] = 0.0f;
  if (bias != nullptr) load_floats<V>(bias + c, shift);
  float past[TAPS][V];                              // past[j]: the input TAPS - 1 - j tokens back; the last is the token's own
  int row = -1;
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    if (i >= count) break;
    const int token = first + i;
    if (positions[token] < 0) { row = -1; continue; }            // a padding row of a captured batch
    const int mine = row_of_token[token];
    if (mine == row) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
        for (int v = 0; v < V; ++v) past[j][v] = past[j + 1][v];
    } else {                                        // the run starts here, or another request does
      row = mine;
      const int start = query_starts[row];
      const float* old = tail + (size_t)state_slots[row] * (TAPS - 1) * channels + c;
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) {
        const int src = token - start - (TAPS - 1) + j;
        if (src >= 0) load_piece(x + (size_t)(start + src) * ldx + c, past[j]);
        else load_floats<V>(old + (size_t)(TAPS - 1 + src) * channels, past[j]);
      }
    }
    load_piece(reinterpret_cast<const T*>(&raw[i]), past[TAPS - 1]);
    float result[V];
#pragma unroll
    for (int v = 0; v < V; ++v) {
      float acc = 0.0f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(taps[v][j], past[j][v], acc);
      result[v] = silu(acc + shift[v]);
    }
    store_piece<V>(out + (size_t)token * channels + c, result);
    if (TAPS > 1 && query_starts[row + 1] - query_starts[row] == 1) {
      float* kept = tail + (size_t)state_slots[row] * (TAPS - 1) * channels + c;
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) store_piece<V>(kept + (size_t)j * channels, past[j + 1]);
    }
  }
}

template <typename T, typename TO>
int launch(const T* x, long long ldx, const T* w, const float* bias, float* tail, const int* row_of_token,
           const int* query_starts, const int* state_slots, const int* positions, TO* out, int tokens, int rows,
           int channels, int taps, int single_tokens_only, cudaStream_t stream) {
  constexpr int V = Piece<T>::kCount;
  const bool aligned = channels % V == 0 && channels % 4 == 0 && ldx % V == 0 && (uintptr_t)x % 16 == 0 &&
                       (uintptr_t)out % 16 == 0 && (uintptr_t)tail % 16 == 0 && (uintptr_t)bias % 16 == 0;
  const int threads = channels >= 256 ? 256 : ((channels + 31) / 32) * 32;
  int status, skip_single = 0;
  if (aligned && taps <= 4) {
    const int run = tokens >= 512 ? 8 : 1;
    const int pieces = channels / V;
    const int wide_threads = pieces >= 128 ? 128 : ((pieces + 31) / 32) * 32;
    const dim3 grid((tokens + run - 1) / run, (pieces + wide_threads - 1) / wide_threads);
#define MIR_CONV_RUN(N, R)                                                                                              \
  mir_launch("short_conv_silu_wide", short_conv_silu_wide_kernel<T, TO, N, R>, grid, dim3(wide_threads), 0, stream, 0, x, ldx, \
             w, bias, tail, row_of_token, query_starts, state_slots, positions, out, tokens, channels)
#define MIR_CONV(N) status = run == 8 ? MIR_CONV_RUN(N, 8) : MIR_CONV_RUN(N, 1)
    switch (taps) {
      case 1: MIR_CONV(1); break;
      case 2: MIR_CONV(2); break;
      case 3: MIR_CONV(3); break;
      default: MIR_CONV(4); break;
    }
#undef MIR_CONV
#undef MIR_CONV_RUN
    if (single_tokens_only) return status;
    skip_single = 1;
  } else {
    status = mir_launch("short_conv_silu", short_conv_silu_kernel<T, TO>, dim3(tokens, (channels + threads - 1) / threads),
                        dim3(threads), 0, stream, 0, x, ldx, w, bias, (const float*)tail, row_of_token, query_starts,
                        state_slots, positions, out, channels, taps);
  }
  if (status != MIR_OK || taps == 1) return status;
  return mir_launch("short_conv_tail", short_conv_tail_kernel<T>, dim3(rows, (channels + threads - 1) / threads), dim3(threads),
                    0, stream, 0, x, ldx, tail, query_starts, state_slots, positions, channels, taps, skip_single);
}

}  // namespace

// x [tokens, channels] with row stride ldx and w [channels, taps] in one type (bf16 or 32-bit); bias [channels] 32-bit or
// null; tail [slots, taps - 1, channels] 32-bit, read and moved on; out [tokens, channels] contiguous, in x's type or
// (out_f32) 32-bit.  single_tokens_only: every request brings one token.
MIR_EXPORT int mir_short_conv_silu(int bf16, int out_f32, const void* x, long long ldx, const void* w, const float* bias,
                                   float* tail, const int* row_of_token, const int* query_starts, const int* state_slots,
                                   const int* positions, void* out, int tokens, int rows, int channels, int taps,
                                   int single_tokens_only, cudaStream_t stream) {
  if (tokens == 0 || rows == 0) return MIR_OK;
  if (tokens < 0 || rows < 0 || channels <= 0 || taps < 1 || taps > kMaxTaps) {
    mir_set_error("short_conv_silu: bad sizes (tokens %d, rows %d, channels %d, taps %d; at most %d taps)", tokens, rows,
                  channels, taps, kMaxTaps);
    return MIR_BAD_ARGUMENT;
  }
  if (bf16 && out_f32)
    return launch<__nv_bfloat16, float>((const __nv_bfloat16*)x, ldx, (const __nv_bfloat16*)w, bias, tail, row_of_token,
                                        query_starts, state_slots, positions, (float*)out, tokens, rows, channels, taps,
                                        single_tokens_only, stream);
  if (bf16)
    return launch<__nv_bfloat16, __nv_bfloat16>((const __nv_bfloat16*)x, ldx, (const __nv_bfloat16*)w, bias, tail,
                                                row_of_token, query_starts, state_slots, positions, (__nv_bfloat16*)out,
                                                tokens, rows, channels, taps, single_tokens_only, stream);
  return launch<float, float>((const float*)x, ldx, (const float*)w, bias, tail, row_of_token, query_starts, state_slots,
                              positions, (float*)out, tokens, rows, channels, taps, single_tokens_only, stream);
}
