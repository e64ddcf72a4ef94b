// The selective scan (Mamba): a diagonal recurrence per channel c with N numbers of state, whose step size dt, input
// vector B and read-out vector C are functions of the token:
//     dt = softplus(raw + bias);  S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x_c B_n;  y_c = sum_n S[c, n] C_n + D_c x_c
// and what leaves the kernel is y * silu(z).  The state is 32-bit, [slot][channel][n], read at the start of a request's
// portion and written at its end; softplus, exponentials, state and sums are 32-bit whatever the activations' type T.
//
// A CTA takes 32 channels of one request and walks over the request's tokens of this step.  Four lanes share a channel
// and hold its state in registers, PER numbers each.  Tokens come in chunks: the raw inputs of the next chunk are copied
// asynchronously into one of two buffers while the current one is worked on; each chunk's step sizes (and their products
// with x), B and C are first turned into 32-bit numbers in shared memory, once per CTA.  The chain from token to token is
// one fused multiply-add per state number; exponentials and products hang off it.  The read-outs of four tokens are
// reduced over the four lanes together, in three shuffles, which leaves each lane one token's sum: it adds the term with
// D, applies the gate and puts the result where z was, and whole rows leave in 16-byte pieces.  The order of a sum depends
// on N alone, never on how a prompt was cut or what else is in the batch.
#include "common.cuh"

using namespace mir;

namespace {

constexpr int kThreads = 128;
constexpr int kLanes = 4;                           // lanes that share a channel
constexpr int kChannels = kThreads / kLanes;        // channels a CTA takes

__device__ __forceinline__ float softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
// 2^v for v <= 0: the hardware's approximation (2 ulp), results below the smallest normal number are zero.
__device__ __forceinline__ float exp2_below_one(float v) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(v));
  return y;
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
  const unsigned target = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(target), "l"(src) : "memory");
}

// Shared memory of a chunk of `chunk` tokens, in bytes from the start; every part starts on 16 bytes.
template <typename T>
struct Layout {
  int dt, x, z, b, c, raw;                          // offsets in a raw buffer, and its size
  int du, bf, cf, total;                            // the 32-bit parts behind the two raw buffers
  __host__ __device__ Layout(int chunk, int columns, int padded) {
    dt = 0;
    x = dt + chunk * kChannels * 4;
    z = x + chunk * kChannels * (int)sizeof(T);
    b = z + chunk * kChannels * (int)sizeof(T);
    c = b + chunk * columns * (int)sizeof(T);
    raw = c + chunk * columns * (int)sizeof(T);
    du = 2 * raw;
    bf = du + chunk * kChannels * 8;
    cf = bf + chunk * padded * 4;
    total = cf + chunk * padded * 4;
  }
};

template <int PER>
__device__ __forceinline__ void load_row(const float* p, float (&v)[PER]) {
  if constexpr (PER % 4 == 0) {
#pragma unroll
    for (int i = 0; i < PER; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(p + i);
      v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
    }
  } else if constexpr (PER % 2 == 0) {
#pragma unroll
    for (int i = 0; i < PER; i += 2) {
      const float2 a = *reinterpret_cast<const float2*>(p + i);
      v[i] = a.x; v[i + 1] = a.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < PER; ++i) v[i] = p[i];
  }
}

// grid (rows, ceil(channels / kChannels)), kThreads threads.
//   x, z    element (t, c) at x[t * ldx + c], z[t * ldz + c];  raw: (t, c) at raw[t * channels + c], 32-bit
//   b, c    element (t, n) at b[t * ldb + n], c[t * ldb + n]; rows readable up to `columns`, a multiple of 8
//   rates   [channels, n]: A log2(e);  skip: D;  state [slots, channels, n];  out [tokens, channels]
template <typename T, int PER>
__global__ void __launch_bounds__(kThreads)
selective_scan_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ raw_step,
                      const float* __restrict__ step_bias, const T* __restrict__ b, const T* __restrict__ c, long long ldb,
                      const T* __restrict__ z, long long ldz, const float* __restrict__ rates,
                      const float* __restrict__ skip, float* __restrict__ state, const int* __restrict__ query_starts,
                      const int* __restrict__ state_slots, const int* __restrict__ positions, T* __restrict__ out,
                      int channels, int n, int columns, int chunk) {
  extern __shared__ __align__(16) unsigned char shared[];
  constexpr int PADDED = kLanes * PER;
  constexpr int V = 16 / sizeof(T);                 // elements in 16 bytes
  const Layout<T> at(chunk, columns, PADDED);
  float2* const du = reinterpret_cast<float2*>(shared + at.du);
  float* const bf = reinterpret_cast<float*>(shared + at.bf);
  float* const cf = reinterpret_cast<float*>(shared + at.cf);
  const int thread = threadIdx.x, l = thread % kLanes, mine = thread / kLanes;
  const int first_channel = blockIdx.y * kChannels;
  const int channel = first_channel + mine;
  const bool active = channel < channels;
  const int here = min(kChannels, channels - first_channel);     // (a multiple of 8)

  float rate[PER], s[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e)
    rate[e] = (active && l * PER + e < n) ? rates[(size_t)channel * n + l * PER + e] : 0.0f;
  const float skip_factor = active ? skip[channel] : 0.0f;
  grid_launch_dependents();
  grid_dependency_wait();
  const int row = blockIdx.x;
  const int start = query_starts[row], end = query_starts[row + 1];
  if (end <= start || positions[start] < 0) return;              // the whole CTA: an empty or padding row
  float* const own_state = state + ((size_t)state_slots[row] * channels + (active ? channel : 0)) * n + l * PER;
  const bool whole = n == PADDED;                                // (then a lane's numbers start on PER * 4 bytes)
  if (whole && active) load_row<PER>(own_state, s);
  else {
#pragma unroll
    for (int e = 0; e < PER; ++e) s[e] = (active && l * PER + e < n) ? own_state[e] : 0.0f;
  }

  auto fetch = [&](int from, unsigned char* buffer) {
    const int count = min(chunk, end - from);
    const int step_pieces = here / 4, wide_pieces = here / V, state_pieces = columns / V;
    const int per_token = step_pieces + 2 * wide_pieces + 2 * state_pieces;
    // a warp takes a token at a time: its lanes walk over the token's pieces
    for (int t = thread >> 5; t < count; t += kThreads / 32) {
      for (int p = thread & 31; p < per_token; p += 32) {
        int i = p;
        if (i < step_pieces) {
          copy16(buffer + at.dt + (t * kChannels + i * 4) * 4, raw_step + (size_t)(from + t) * channels + first_channel + i * 4);
          continue;
        }
        i -= step_pieces;
        if (i < wide_pieces) {
          copy16(buffer + at.x + (t * kChannels + i * V) * (int)sizeof(T), x + (size_t)(from + t) * ldx + first_channel + i * V);
          continue;
        }
        i -= wide_pieces;
        if (i < wide_pieces) {
          copy16(buffer + at.z + (t * kChannels + i * V) * (int)sizeof(T), z + (size_t)(from + t) * ldz + first_channel + i * V);
          continue;
        }
        i -= wide_pieces;
        if (i < state_pieces) {
          copy16(buffer + at.b + (t * columns + i * V) * (int)sizeof(T), b + (size_t)(from + t) * ldb + i * V);
          continue;
        }
        i -= state_pieces;
        copy16(buffer + at.c + (t * columns + i * V) * (int)sizeof(T), c + (size_t)(from + t) * ldb + i * V);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  fetch(start, shared);
  // what the lane turns into 32-bit numbers of a chunk: always the same channel (thread % kChannels)
  const int staged_channel = thread % kChannels;
  const float bias = first_channel + staged_channel < channels ? step_bias[first_channel + staged_channel] : 0.0f;
  int buffer = 0;
  for (int from = start; from < end; from += chunk, buffer ^= 1) {
    const int count = min(chunk, end - from);
    unsigned char* const in = shared + buffer * at.raw;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                             // this chunk is here; the other buffer has been read
    if (from + chunk < end) fetch(from + chunk, shared + (buffer ^ 1) * at.raw);
    const T* const xs = reinterpret_cast<const T*>(in + at.x);
    T* const zs = reinterpret_cast<T*>(in + at.z);
    if (staged_channel < here) {
      const float* steps = reinterpret_cast<const float*>(in + at.dt);
      for (int t = thread / kChannels; t < count; t += kThreads / kChannels) {
        const float step = softplus(steps[t * kChannels + staged_channel] + bias);
        du[t * kChannels + staged_channel] = make_float2(step, step * to_float(xs[t * kChannels + staged_channel]));
      }
    }
    const T* const bs = reinterpret_cast<const T*>(in + at.b);
    const T* const cs = reinterpret_cast<const T*>(in + at.c);
    for (int i = thread; i < count * PADDED; i += kThreads) {
      const int t = i / PADDED, k = i - t * PADDED;
      bf[i] = k < n ? to_float(bs[t * columns + k]) : 0.0f;
      cf[i] = k < n ? to_float(cs[t * columns + k]) : 0.0f;
    }
    __syncthreads();
    const float* b_at = bf + l * PER;
    const float* c_at = cf + l * PER;
    const float2* du_at = du + mine;
    auto advance = [&](int t) {
      const float2 step = du_at[t * kChannels];
      float bb[PER], cc[PER];
      load_row<PER>(b_at + t * PADDED, bb);
      load_row<PER>(c_at + t * PADDED, cc);
      float even = 0.0f, odd = 0.0f;
#pragma unroll
      for (int e = 0; e < PER; ++e) {
        s[e] = fmaf(exp2_below_one(step.x * rate[e]), s[e], step.y * bb[e]);
        if (e & 1) odd = fmaf(s[e], cc[e], odd);
        else even = fmaf(s[e], cc[e], even);
      }
      return even + odd;
    };
    for (int t = 0; t < count; t += 4) {
      float y[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (t + 4 <= count) {
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = advance(t + i);
      } else {
#pragma unroll
        for (int i = 0; i < 3; ++i)
          if (t + i < count) y[i] = advance(t + i);
      }
      // four tokens over four lanes: lane l is left with token t + l
      const bool low = (l & 1) == 0, front = (l & 2) == 0;
      float first = low ? y[0] : y[1], second = low ? y[2] : y[3];
      first += __shfl_xor_sync(0xffffffffu, low ? y[1] : y[0], 1);
      second += __shfl_xor_sync(0xffffffffu, low ? y[3] : y[2], 1);
      float sum = front ? first : second;
      sum += __shfl_xor_sync(0xffffffffu, front ? second : first, 2);
      const int token = t + l;
      if (token < count && active) {
        const int place = token * kChannels + mine;
        const float value = fmaf(skip_factor, to_float(xs[place]), sum);
        zs[place] = from_float<T>(value * silu(to_float(zs[place])));
      }
    }
    __syncthreads();
    const int wide_pieces = here / V;
    for (int i = thread; i < count * (kChannels / V); i += kThreads) {
      const int t = i / (kChannels / V), p = i % (kChannels / V);
      if (p < wide_pieces)
        *reinterpret_cast<uint4*>(out + (size_t)(from + t) * channels + first_channel + p * V) =
            *reinterpret_cast<const uint4*>(zs + t * kChannels + p * V);
    }
  }
  if (!active) return;
#pragma unroll
  for (int e = 0; e < PER; ++e)
    if (l * PER + e < n) own_state[e] = s[e];
}

template <typename T, int PER>
int launch(const void* x, long long ldx, const float* raw_step, const float* step_bias, const void* b, const void* c,
           long long ldb, const void* z, long long ldz, const float* rates, const float* skip, float* state,
           const int* query_starts, const int* state_slots, const int* positions, void* out, int tokens, int rows,
           int channels, int n, int columns, cudaStream_t stream) {
  int chunk = tokens == rows ? 4 : 32;                           // (a step of single tokens stages one)
  while (chunk > 4 && Layout<T>(chunk, columns, kLanes * PER).total > 96 * 1024) chunk /= 2;
  const int smem = Layout<T>(chunk, columns, kLanes * PER).total;
  if (smem > 48 * 1024) {
    const cudaError_t err = cudaFuncSetAttribute(selective_scan_kernel<T, PER>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (err != cudaSuccess) {
      mir_set_error("selective_scan: cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(err));
      return MIR_CUDA_ERROR;
    }
  }
  return mir_launch("selective_scan", selective_scan_kernel<T, PER>, dim3(rows, (channels + kChannels - 1) / kChannels),
                    dim3(kThreads), smem, stream, 0, (const T*)x, ldx, raw_step, step_bias, (const T*)b, (const T*)c, ldb,
                    (const T*)z, ldz, rates, skip, state, query_starts, state_slots, positions, (T*)out, channels, n,
                    columns, chunk);
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
