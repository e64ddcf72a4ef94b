// The selective scan (Mamba): a diagonal recurrence per channel c with N numbers of state, whose step size dt, input
// vector B and read-out vector C are functions of the token:
//     dt = softplus(raw + bias);  S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x_c B_n;  y_c = sum_n S[c, n] C_n + D_c x_c
// and what leaves the kernel is y * silu(z).  The state is 32-bit, [slot][channel][n], read at the start of a request's
// portion and written at its end; softplus, exponentials, state and sums are 32-bit whatever the activations' type T.
//
// A CTA takes 32 channels of one request and walks over the request's tokens of this step.  Four lanes share a channel
// and hold its state in registers, PER numbers each.  The chain from token to token is one fused multiply-add per state
// number; exponentials and products hang off it.  The read-outs of four tokens are reduced over the four lanes together,
// in three shuffles, which leaves each lane one token's sum.  The order of a sum depends on N alone, never on how a prompt
// was cut or what else is in the batch, and both kernels below do the same arithmetic in the same order.
//
//   selective_scan         portions: four warps walk, eight others work for them.  While the walkers go through one chunk
//                          of tokens, the others turn the next chunk's step sizes (and their products with x), B and C
//                          into 32-bit numbers in shared memory, fetch the raw inputs of the chunk behind it, and finish
//                          the chunk before (the term with D, the gate, the result's rows); one barrier per chunk.
//   selective_scan_single  a step of single tokens: four warps, nothing staged ahead.
#include "common.cuh"

using namespace mir;

namespace {

constexpr int kWalkers = 128;                       // threads that hold the state
constexpr int kHelpers = 256;                       // threads that prepare and finish for them (portions)
constexpr int kLanes = 4;                           // lanes that share a channel
constexpr int kChannels = kWalkers / kLanes;        // channels a CTA takes
constexpr int kMaxChunk = 32;
constexpr int kSumRow = 40;                         // floats between two tokens' sums (lanes of a warp on 32 banks)

// log(1 + e^z) = max(z, 0) + log(1 + e) with e = e^-|z| in (0, 1], and log(1 + e) = 2 artanh(s), s = e / (2 + e) <= 1/3, by
// the series 2 (s + s^3/3 + s^5/5 + ...): what is left out behind s^15 is below 2e-9 of the result.
__device__ __forceinline__ float softplus(float z) {
  const float e = expf(-fabsf(z));
  const float s = __fdividef(e, 2.0f + e), q = s * s;
  float sum = 1.0f / 15.0f;
  sum = fmaf(sum, q, 1.0f / 13.0f);
  sum = fmaf(sum, q, 1.0f / 11.0f);
  sum = fmaf(sum, q, 1.0f / 9.0f);
  sum = fmaf(sum, q, 1.0f / 7.0f);
  sum = fmaf(sum, q, 1.0f / 5.0f);
  sum = fmaf(sum, q, 1.0f / 3.0f);
  sum = fmaf(sum, q, 1.0f);
  return fmaxf(z, 0.0f) + 2.0f * s * sum;
}
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
// 2^v for v <= 0: the hardware's approximation (2 ulp), results below the smallest normal number are zero.
__device__ __forceinline__ float exp2_below_one(float v) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(v));
  return y;
}
// Two 32-bit numbers side by side: one instruction multiplies (and adds) both.
typedef unsigned long long pair32;
__device__ __forceinline__ pair32 make_pair(float a, float b) {
  pair32 p;
  asm("mov.b64 %0, {%1, %2};" : "=l"(p) : "f"(a), "f"(b));
  return p;
}
__device__ __forceinline__ void split_pair(pair32 p, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(p));
}
__device__ __forceinline__ pair32 mul_pair(pair32 a, pair32 b) {
  pair32 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ pair32 fma_pair(pair32 a, pair32 b, pair32 c) {
  pair32 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  const unsigned target = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(target), "l"(src) : "memory");
}

// What a lane knows of its channel: PER numbers of state and their rates, in pairs.  An odd number (one) is a pair whose
// second half stays zero.  numbers: how many of them there are (PER, less at the end of a channel, none without one);
// wide: all of them, on 16-byte boundaries.
template <int PER>
struct Channel {
  static constexpr int PAIRS = (PER + 1) / 2;
  pair32 s[PAIRS], rate[PAIRS];
  __device__ __forceinline__ static void load(pair32 (&v)[PAIRS], const float* from, int numbers, bool wide) {
    if (PER % 4 == 0 && wide) {
#pragma unroll
      for (int i = 0; i + 1 < PAIRS; i += 2) {
        const float4 a = *reinterpret_cast<const float4*>(from + 2 * i);
        v[i] = make_pair(a.x, a.y);
        v[i + 1] = make_pair(a.z, a.w);
      }
      return;
    }
#pragma unroll
    for (int i = 0; i < PAIRS; ++i)
      v[i] = make_pair(2 * i < numbers ? from[2 * i] : 0.0f, 2 * i + 1 < numbers ? from[2 * i + 1] : 0.0f);
  }
  __device__ __forceinline__ void store(float* to, int numbers, bool wide) const {
    if (PER % 4 == 0 && wide) {
#pragma unroll
      for (int i = 0; i + 1 < PAIRS; i += 2) {
        float4 a;
        split_pair(s[i], a.x, a.y);
        split_pair(s[i + 1], a.z, a.w);
        *reinterpret_cast<float4*>(to + 2 * i) = a;
      }
      return;
    }
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      float a, b;
      split_pair(s[i], a, b);
      if (2 * i < numbers) to[2 * i] = a;
      if (2 * i + 1 < numbers) to[2 * i + 1] = b;
    }
  }
  // One token: the state moves on; returns this lane's share of the read-out.
  __device__ __forceinline__ float advance(float step, float step_x, const pair32 (&b)[PAIRS], const pair32 (&c)[PAIRS]) {
    const pair32 steps = make_pair(step, step), inputs = make_pair(step_x, step_x);
    pair32 sum = 0ull;
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      float low, high;
      split_pair(mul_pair(steps, rate[i]), low, high);
      s[i] = fma_pair(make_pair(exp2_below_one(low), exp2_below_one(high)), s[i], mul_pair(inputs, b[i]));
      sum = fma_pair(s[i], c[i], sum);
    }
    float even, odd;
    split_pair(sum, even, odd);
    return even + odd;
  }
};

// ---------------------------------------------------------------------------------------------- portions
// Shared memory of chunks of `chunk` tokens, in bytes from the start; every part starts on 16 bytes and is there twice.
template <typename T>
struct Layout {
  int du, b, c, raw_b, raw_c, sums, total;
  __host__ __device__ Layout(int chunk, int columns, int padded) {
    du = 0;                                         // [2][chunk][kChannels] (step, step * x)
    b = du + 2 * chunk * kChannels * 8;             // [2][chunk][padded] 32-bit
    c = b + 2 * chunk * padded * 4;
    raw_b = c + 2 * chunk * padded * 4;             // [2][chunk][columns] as they come
    raw_c = raw_b + 2 * chunk * columns * (int)sizeof(T);
    sums = raw_c + 2 * chunk * columns * (int)sizeof(T);        // [2][chunk][kSumRow]
    total = sums + 2 * chunk * kSumRow * 4;
  }
};

template <int PER>
struct Operands {
  static constexpr int PAIRS = (PER + 1) / 2;
  float2 du;
  pair32 b[PAIRS], c[PAIRS];
  __device__ __forceinline__ static void load_pairs(const float* p, pair32 (&v)[PAIRS]) {
    if constexpr (PER % 4 == 0) {
#pragma unroll
      for (int i = 0; i < PAIRS; i += 2) {
        const ulonglong2 both = *reinterpret_cast<const ulonglong2*>(p + 2 * i);
        v[i] = both.x;
        v[i + 1] = both.y;
      }
    } else if constexpr (PER % 2 == 0) {
#pragma unroll
      for (int i = 0; i < PAIRS; ++i) v[i] = *reinterpret_cast<const pair32*>(p + 2 * i);
    } else {
      v[0] = make_pair(p[0], 0.0f);
    }
  }
  __device__ __forceinline__ void load(const float2* du_at, const float* b_at, const float* c_at) {
    du = *du_at;
    load_pairs(b_at, b);
    load_pairs(c_at, c);
  }
};

// grid (rows, ceil(channels / kChannels)), kWalkers + kHelpers threads.
//   x, z    element (t, c) at x[t * ldx + c], z[t * ldz + c];  raw_step: (t, c) at raw_step[t * channels + c], 32-bit
//   b, c    element (t, n) at b[t * ldb + n], c[t * ldb + n]; rows readable up to `columns`, a multiple of 8
//   rates   [channels, n]: A log2(e);  skip: D;  state [slots, channels, n];  out [tokens, channels]
template <typename T, int PER>
__global__ void __launch_bounds__(kWalkers + kHelpers)
selective_scan_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ raw_step,
                      const float* __restrict__ step_bias, const T* __restrict__ b, const T* __restrict__ c, long long ldb,
                      const T* __restrict__ z, long long ldz, const float* __restrict__ rates,
                      const float* __restrict__ skip, float* __restrict__ state, const int* __restrict__ query_starts,
                      const int* __restrict__ state_slots, const int* __restrict__ positions, T* __restrict__ out,
                      int channels, int n, int columns, int chunk) {
  static_assert(PER == 1 || PER % 2 == 0, "numbers a lane holds come in pairs");
  extern __shared__ __align__(16) unsigned char shared[];
  constexpr int PADDED = kLanes * PER;
  constexpr int V = 16 / sizeof(T);                 // elements in 16 bytes
  constexpr int STRIDE = kHelpers / kChannels;
  constexpr int TOKENS = kMaxChunk / STRIDE;        // of a chunk, for a helper
  const Layout<T> at(chunk, columns, PADDED);
  float2* const du_s = reinterpret_cast<float2*>(shared + at.du);
  float* const b_s = reinterpret_cast<float*>(shared + at.b);
  float* const c_s = reinterpret_cast<float*>(shared + at.c);
  T* const raw_b = reinterpret_cast<T*>(shared + at.raw_b);
  T* const raw_c = reinterpret_cast<T*>(shared + at.raw_c);
  float* const sums = reinterpret_cast<float*>(shared + at.sums);
  const int first_channel = blockIdx.y * kChannels;
  grid_launch_dependents();
  grid_dependency_wait();
  const int row = blockIdx.x;
  const int start = query_starts[row], end = query_starts[row + 1];
  if (end <= start || positions[start] < 0) return;              // the whole CTA: an empty or padding row
  const int chunks = (end - start + chunk - 1) / chunk;

  if (threadIdx.x < kWalkers) {
    const int l = threadIdx.x % kLanes, mine = threadIdx.x / kLanes;
    const int channel = first_channel + mine;
    const int numbers = channel < channels ? min(PER, n - l * PER) : 0;
    const bool wide = numbers == PER && n % 4 == 0;
    const size_t own = (size_t)(channel < channels ? channel : 0) * n + l * PER;
    float* const own_state = state + (size_t)state_slots[row] * channels * n + own;
    Channel<PER> held;
    held.load(held.s, own_state, numbers, wide);
    held.load(held.rate, rates + own, numbers, wide);
    for (int phase = 0; phase < chunks + 2; ++phase) {
      if (phase >= 1 && phase <= chunks) {
        const int which = (phase - 1) & 1;
        const int count = min(chunk, end - start - (phase - 1) * chunk);
        const float2* du_at = du_s + which * chunk * kChannels + mine;
        const float* b_at = b_s + which * chunk * PADDED + l * PER;
        const float* c_at = c_s + which * chunk * PADDED + l * PER;
        float* sum_at = sums + which * chunk * kSumRow + l * kSumRow + mine;
        auto reduce = [&](const float (&y)[4], int t) {          // four tokens over four lanes: lane l is left with t + l
          const bool low = (l & 1) == 0, front = (l & 2) == 0;
          float first = low ? y[0] : y[1], second = low ? y[2] : y[3];
          first += __shfl_xor_sync(0xffffffffu, low ? y[1] : y[0], 1);
          second += __shfl_xor_sync(0xffffffffu, low ? y[3] : y[2], 1);
          float sum = front ? first : second;
          sum += __shfl_xor_sync(0xffffffffu, front ? second : first, 2);
          sum_at[t * kSumRow] = sum;                             // (behind the last token: a place nobody reads)
        };
        int t = 0;
        if constexpr (PER <= 8) {                                // the next four tokens' operands are on their way
          Operands<PER> next[4];
          if (count >= 4) {
#pragma unroll
            for (int i = 0; i < 4; ++i) next[i].load(du_at + i * kChannels, b_at + i * PADDED, c_at + i * PADDED);
          }
          for (; t + 4 <= count; t += 4) {
            float y[4];
            const bool more = t + 8 <= count;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              y[i] = held.advance(next[i].du.x, next[i].du.y, next[i].b, next[i].c);
              if (more) next[i].load(du_at + (t + 4 + i) * kChannels, b_at + (t + 4 + i) * PADDED, c_at + (t + 4 + i) * PADDED);
            }
            reduce(y, t);
          }
        } else {
          for (; t + 4 <= count; t += 4) {
            float y[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              Operands<PER> now;
              now.load(du_at + (t + i) * kChannels, b_at + (t + i) * PADDED, c_at + (t + i) * PADDED);
              y[i] = held.advance(now.du.x, now.du.y, now.b, now.c);
            }
            reduce(y, t);
          }
        }
        if (t < count) {
          float y[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
          for (int i = 0; i < 3; ++i) {
            if (t + i < count) {
              Operands<PER> now;
              now.load(du_at + (t + i) * kChannels, b_at + (t + i) * PADDED, c_at + (t + i) * PADDED);
              y[i] = held.advance(now.du.x, now.du.y, now.b, now.c);
            }
          }
          reduce(y, t);
        }
      }
      __syncthreads();
    }
    held.store(own_state, numbers, wide);
    return;
  }

  // helpers: a thread always works for the same channel
  const int thread = threadIdx.x - kWalkers;
  const int mine = thread % kChannels, first_token = thread / kChannels;
  const int channel = first_channel + mine;
  const bool active = channel < channels;
  const float bias = active ? step_bias[channel] : 0.0f, skip_factor = active ? skip[channel] : 0.0f;
  // raw inputs of the next chunk; x of the chunk that is staged now, walked through, and finished
  float next_step[TOKENS], next_x[TOKENS], staged_x[TOKENS], walked_x[TOKENS], finished_x[TOKENS];
#pragma unroll
  for (int k = 0; k < TOKENS; ++k) staged_x[k] = walked_x[k] = 0.0f;
  auto fetch = [&](int number) {
    const int from = start + number * chunk, count = min(chunk, end - from);
#pragma unroll
    for (int k = 0; k < TOKENS; ++k) {
      const int t = first_token + k * STRIDE;
      const bool there = active && t < count;
      next_step[k] = there ? raw_step[(size_t)(from + t) * channels + channel] : 0.0f;
      next_x[k] = there ? to_float(x[(size_t)(from + t) * ldx + channel]) : 0.0f;
    }
    const int pieces = columns / V, which = number & 1;
    for (int i = thread; i < count * pieces; i += kHelpers) {
      const int t = i / pieces, p = i - t * pieces;
      copy16(raw_b + (size_t)(which * chunk + t) * columns + p * V, b + (size_t)(from + t) * ldb + p * V);
      copy16(raw_c + (size_t)(which * chunk + t) * columns + p * V, c + (size_t)(from + t) * ldb + p * V);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // (B and C of the first chunk are copied by all helpers before any of them reads: a barrier among the helpers)
  fetch(0);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  asm volatile("bar.sync 1, %0;" ::"n"(kHelpers) : "memory");
  for (int phase = 0; phase < chunks + 2; ++phase) {
    const int finished = phase - 2;
    float gates[TOKENS], steps[TOKENS];
#pragma unroll
    for (int k = 0; k < TOKENS; ++k) {
      finished_x[k] = walked_x[k];
      walked_x[k] = staged_x[k];
      staged_x[k] = next_x[k];
      steps[k] = next_step[k];
    }
    if (phase + 1 < chunks) fetch(phase + 1);                    // (memory is asked first, what it brings is used last)
    if (finished >= 0) {
      const int from = start + finished * chunk, count = min(chunk, end - from);
#pragma unroll
      for (int k = 0; k < TOKENS; ++k) {
        const int t = first_token + k * STRIDE;
        gates[k] = active && t < count ? to_float(z[(size_t)(from + t) * ldz + channel]) : 0.0f;
      }
    }
    if (phase < chunks) {
      const int which = phase & 1, count = min(chunk, end - start - phase * chunk);
#pragma unroll
      for (int k = 0; k < TOKENS; ++k) {
        const int t = first_token + k * STRIDE;
        const float step = softplus(steps[k] + bias);
        if (t < count) du_s[(which * chunk + t) * kChannels + mine] = make_float2(step, step * staged_x[k]);
      }
      for (int i = thread; i < count * PADDED; i += kHelpers) {
        const int t = i / PADDED, k = i % PADDED;
        b_s[which * chunk * PADDED + i] = k < n ? to_float(raw_b[(size_t)(which * chunk + t) * columns + k]) : 0.0f;
        c_s[which * chunk * PADDED + i] = k < n ? to_float(raw_c[(size_t)(which * chunk + t) * columns + k]) : 0.0f;
      }
    }
    if (finished >= 0) {
      const int which = finished & 1, from = start + finished * chunk, count = min(chunk, end - from);
#pragma unroll
      for (int k = 0; k < TOKENS; ++k) {
        const int t = first_token + k * STRIDE;
        if (active && t < count) {
          const float value = fmaf(skip_factor, finished_x[k], sums[(which * chunk + t) * kSumRow + mine]);
          out[(size_t)(from + t) * channels + channel] = from_float<T>(value * silu(gates[k]));
        }
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");         // (the next chunk's B and C are here behind the barrier)
    __syncthreads();
  }
}

// ---------------------------------------------------------------------------------------------- single tokens
// The same grid, kWalkers threads: request row r brings token query_starts[r].
template <typename T, int PER>
__global__ void __launch_bounds__(kWalkers)
selective_scan_single_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ raw_step,
                             const float* __restrict__ step_bias, const T* __restrict__ b, const T* __restrict__ c,
                             long long ldb, const T* __restrict__ z, long long ldz, const float* __restrict__ rates,
                             const float* __restrict__ skip, float* __restrict__ state, const int* __restrict__ query_starts,
                             const int* __restrict__ state_slots, const int* __restrict__ positions, T* __restrict__ out,
                             int channels, int n) {
  constexpr int PAIRS = Channel<PER>::PAIRS;
  grid_launch_dependents();
  const int l = threadIdx.x % kLanes;
  const int channel = blockIdx.y * kChannels + threadIdx.x / kLanes;
  const bool active = channel < channels;
  const int numbers = active ? min(PER, n - l * PER) : 0;
  const bool wide = numbers == PER && n % 4 == 0;
  const size_t own = (size_t)(active ? channel : 0) * n + l * PER;
  Channel<PER> held;
  held.load(held.rate, rates + own, numbers, wide);
  const float bias = active ? step_bias[channel] : 0.0f, skip_factor = active ? skip[channel] : 0.0f;
  grid_dependency_wait();
  const int token = query_starts[blockIdx.x];
  if (query_starts[blockIdx.x + 1] <= token || positions[token] < 0) return;    // the whole CTA: an empty or padding row
  float* const own_state = state + (size_t)state_slots[blockIdx.x] * channels * n + own;
  held.load(held.s, own_state, numbers, wide);
  const float input = active ? to_float(x[(size_t)token * ldx + channel]) : 0.0f;
  const float gate = active ? to_float(z[(size_t)token * ldz + channel]) : 0.0f;
  const float step = softplus((active ? raw_step[(size_t)token * channels + channel] : 0.0f) + bias);
  pair32 bb[PAIRS], cc[PAIRS];
  const T* b_at = b + (size_t)token * ldb + l * PER;
  const T* c_at = c + (size_t)token * ldb + l * PER;
#pragma unroll
  for (int i = 0; i < PAIRS; ++i) {
    bb[i] = make_pair(2 * i < numbers ? to_float(b_at[2 * i]) : 0.0f, 2 * i + 1 < numbers ? to_float(b_at[2 * i + 1]) : 0.0f);
    cc[i] = make_pair(2 * i < numbers ? to_float(c_at[2 * i]) : 0.0f, 2 * i + 1 < numbers ? to_float(c_at[2 * i + 1]) : 0.0f);
  }
  float sum = held.advance(step, step * input, bb, cc);
  sum += __shfl_xor_sync(0xffffffffu, sum, 1);
  sum += __shfl_xor_sync(0xffffffffu, sum, 2);
  held.store(own_state, numbers, wide);
  if (active && l == 0) out[(size_t)token * channels + channel] = from_float<T>(fmaf(skip_factor, input, sum) * silu(gate));
}

template <typename T, int PER>
int launch(const void* x, long long ldx, const float* raw_step, const float* step_bias, const void* b, const void* c,
           long long ldb, const void* z, long long ldz, const float* rates, const float* skip, float* state,
           const int* query_starts, const int* state_slots, const int* positions, void* out, int tokens, int rows,
           int channels, int n, int columns, cudaStream_t stream) {
  const dim3 grid(rows, (channels + kChannels - 1) / kChannels);
  if (tokens == rows)                                            // a step of single tokens: every row brings one
    return mir_launch("selective_scan", selective_scan_single_kernel<T, PER>, grid, dim3(kWalkers), 0, stream, 0, (const T*)x,
                      ldx, raw_step, step_bias, (const T*)b, (const T*)c, ldb, (const T*)z, ldz, rates, skip, state,
                      query_starts, state_slots, positions, (T*)out, channels, n);
  int chunk = kMaxChunk;
  while (chunk > 4 && Layout<T>(chunk, columns, kLanes * PER).total > 96 * 1024) chunk /= 2;
  const int smem = Layout<T>(chunk, columns, kLanes * PER).total;
  if (smem > 48 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(selective_scan_kernel<T, PER>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (err != cudaSuccess) {
      mir_set_error("selective_scan: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(err));
      return MIR_CUDA_ERROR;
    }
  }
  return mir_launch("selective_scan", selective_scan_kernel<T, PER>, grid, dim3(kWalkers + kHelpers), smem, stream, 0,
                    (const T*)x, ldx, raw_step, step_bias, (const T*)b, (const T*)c, ldb, (const T*)z, ldz, rates, skip, state,
                    query_starts, state_slots, positions, (T*)out, channels, n, columns, chunk);
}

template <typename T>
int dispatch(const void* x, long long ldx, const float* raw_step, const float* step_bias, const void* b, const void* c,
             long long ldb, const void* z, long long ldz, const float* rates, const float* skip, float* state,
             const int* query_starts, const int* state_slots, const int* positions, void* out, int tokens, int rows,
             int channels, int n, int columns, cudaStream_t stream) {
#define MIR_SCAN(P)                                                                                                   \
  if (n <= kLanes * P)                                                                                                \
    return launch<T, P>(x, ldx, raw_step, step_bias, b, c, ldb, z, ldz, rates, skip, state, query_starts, state_slots, \
                        positions, out, tokens, rows, channels, n, columns, stream)
  MIR_SCAN(1);
  MIR_SCAN(2);
  MIR_SCAN(4);
  MIR_SCAN(6);
  MIR_SCAN(8);
  MIR_SCAN(16);
  MIR_SCAN(32);
  MIR_SCAN(64);
#undef MIR_SCAN
  mir_set_error("selective_scan: %d state numbers a channel are more than 256", n);
  return MIR_BAD_ARGUMENT;
}

}  // namespace

// x, z, b, c in the activations' type with row strides ldx, ldz, ldb (rows and pointers on 16 bytes; b and c readable up
// to `columns`); raw_step [tokens, channels] 32-bit; step_bias, skip [channels], rates [channels, n] 32-bit; state [slots,
// channels, n] 32-bit; out [tokens, channels] in the activations' type.  channels and columns are multiples of 8.
MIR_EXPORT int mir_selective_scan(int bf16, const void* x, long long ldx, const float* raw_step, const float* step_bias,
                                  const void* b, const void* c, long long ldb, const void* z, long long ldz,
                                  const float* rates, const float* skip, float* state, const int* query_starts,
                                  const int* state_slots, const int* positions, void* out, int tokens, int rows,
                                  int channels, int n, int columns, cudaStream_t stream) {
  if (tokens == 0 || rows == 0) return MIR_OK;
  const long long piece = bf16 ? 8 : 4;
  if (tokens < 0 || rows < 0 || channels <= 0 || channels % 8 || n <= 0 || columns < n || columns % 8 || ldx % piece ||
      ldz % piece || ldb % piece || (uintptr_t)x % 16 || (uintptr_t)z % 16 || (uintptr_t)b % 16 || (uintptr_t)c % 16 ||
      (uintptr_t)raw_step % 16 || (uintptr_t)out % 16 || (uintptr_t)state % 16 || (channels + kChannels - 1) / kChannels > 65535) {
    mir_set_error("selective_scan: sizes or alignment the kernel does not take (tokens %d, rows %d, channels %d, state %d of "
                  "%d columns)", tokens, rows, channels, n, columns);
    return MIR_BAD_ARGUMENT;
  }
  if (bf16)
    return dispatch<__nv_bfloat16>(x, ldx, raw_step, step_bias, b, c, ldb, z, ldz, rates, skip, state, query_starts,
                                   state_slots, positions, out, tokens, rows, channels, n, columns, stream);
  return dispatch<float>(x, ldx, raw_step, step_bias, b, c, ldb, z, ldz, rates, skip, state, query_starts, state_slots,
                         positions, out, tokens, rows, channels, n, columns, stream);
}
