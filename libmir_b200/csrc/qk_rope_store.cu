// Per-head q/k RMSNorm, rotary position encoding and the write of K and V into cache pages, in one
// kernel over the packed [T, (Hq + Hkv) D + Hkv Dv] output of the QKV projection (Dv = D unless the values have a
// width of their own).
//
// Replaces libmir's qkv_postprocess_bf16.cu:71-183 and kv_cache_bf16.cu:74-97 (two launches and a
// round trip of k and v through memory).  Differences on purpose: the normalised value is not
// rounded to bf16 before the rotation, and the angle table is passed in (so that llama3 scaling,
// which libmir's CUDA loader ignores, is the same code path as the plain table).
//
// q is rotated in place; k (rotated) and v go straight to
//   pages[(slot_mapping[t]) * Hkv + h][:]  with slot = page * page_size + position % page_size,
// and a negative slot means "do not write" (a padded row of a captured decode batch).
// write_kv: 0 only the queries are treated (a reader of another entry's cache), 1 keys and values go to their
// pages, 2 keys are normed and rotated in place like the queries and nothing goes to the pages (a position
// encoding of another kind works on them next; a second call with 1 and neither norm nor rotation then stores).
// interleaved: dims 2i and 2i + 1 of the first rotary_dim dims form pair i, instead of dims i and i + rotary_dim / 2.
// row_stride: elements from one token's row to the next where the row holds more than q, k and v (a gate's
// projection behind them), 0 = packed.  queries_only: the rows hold the query heads alone (a mixer that attends over
// another entry's keys and values).
// QkForms, further forms: magnitude multiplies cos and sin; temperature: a query at position p is multiplied by
// 1 + coef ln(floor((p + 1) / every) + 1), in 32-bit, before it is stored; values_from_keys: the row holds no values, a
// token's value is the key's raw projection, which goes to the value pages as it is.
#include "common.cuh"
#include "trace.cuh"

using namespace mir;

struct QkForms {
  float magnitude = 1.0f;
  float temperature_coef = 0.0f, temperature_every = 0.0f;      // every 0: no temperature
  int values_from_keys = 0;
};

__device__ __forceinline__ float query_temperature(const QkForms& forms, int position) {
  if (forms.temperature_every <= 0.0f) return 1.0f;
  return 1.0f + forms.temperature_coef * logf(floorf(__fdiv_rn((float)(position + 1), forms.temperature_every)) + 1.0f);
}

// Two consecutive elements as floats, and back.
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// One CTA per (token, slice of the token's heads): the token's cosines and sines are computed once into shared
// memory, then each warp takes heads (query, key or value) of the slice.  PAIRED: head_dim is even and
// rotary_dim a multiple of 4, so every lane works on two neighbouring elements (4- or 8-byte accesses).
template <typename T, bool PAIRED>
__global__ void qk_rope_store_kernel(T* __restrict__ qkv, const int* __restrict__ positions,
                                     const int* __restrict__ slot_mapping, const float* __restrict__ inv_freq,
                                     const float* __restrict__ q_norm, const float* __restrict__ k_norm,
                                     T* __restrict__ k_pages, T* __restrict__ v_pages, int heads, int kv_heads,
                                     int head_dim, int value_dim, int rotary_dim, float eps, int write_kv,
                                     int units_per_cta, int interleaved, long long row_stride, int queries_only, QkForms forms) {
  extern __shared__ float angles[];                 // [half] cosines then [half] sines of this token
  grid_launch_dependents();
  grid_dependency_wait();
  const int token = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int units = queries_only ? heads : heads + (forms.values_from_keys ? 1 : 2) * kv_heads;
  const size_t row_width = row_stride > 0 ? (size_t)row_stride
                                          : (size_t)(heads + kv_heads) * head_dim +
                                                (forms.values_from_keys ? 0 : (size_t)kv_heads * value_dim);
  T* row = qkv + (size_t)token * row_width;
  const float position = (float)positions[token];
  const int slot = slot_mapping ? slot_mapping[token] : -1;
  const int half = rotary_dim / 2;
  for (int pair = threadIdx.x; pair < half; pair += blockDim.x) {
    float sine, cosine;
    sincosf(position * inv_freq[pair], &sine, &cosine);
    angles[pair] = cosine * forms.magnitude;
    angles[half + pair] = sine * forms.magnitude;
  }
  const float temperature = query_temperature(forms, positions[token]);
  __syncthreads();
  const int unit_begin = blockIdx.y * units_per_cta, unit_end = min(units, unit_begin + units_per_cta);

  for (int unit = unit_begin + warp; unit < unit_end; unit += warps) {
    T* src = row + (size_t)unit * head_dim;
    if (unit >= heads + kv_heads) {                 // a value head: copy to its page
      if (write_kv != 1 || slot < 0) continue;
      const int value_head = unit - heads - kv_heads;
      src = row + (size_t)(heads + kv_heads) * head_dim + (size_t)value_head * value_dim;
      T* dst = v_pages + ((size_t)slot * kv_heads + value_head) * value_dim;
      if ((value_dim * sizeof(T)) % 16 == 0 && ((uintptr_t)src & 15) == 0 && ((uintptr_t)dst & 15) == 0) {
        const int chunks = value_dim * (int)sizeof(T) / 16;
        for (int c = lane; c < chunks; c += 32) reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(src)[c];
      } else {
        for (int d = lane; d < value_dim; d += 32) dst[d] = src[d];
      }
      continue;
    }
    const bool is_query = unit < heads;
    const bool key_in_place = write_kv == 2;        // normed and rotated keys stay in the packed row
    if (!is_query && !key_in_place && (!write_kv || slot < 0)) continue;
    const float* norm = is_query ? q_norm : k_norm;
    float inverse = 1.0f;
    if (forms.values_from_keys && !is_query && write_kv == 1) {        // the value: the key as it was projected
      T* value = v_pages + ((size_t)slot * kv_heads + (unit - heads)) * head_dim;
      for (int d = lane; d < head_dim; d += 32) value[d] = src[d];
    }
    if (norm) {
      float sum = 0.0f;
      if (PAIRED) {
        for (int d = 2 * lane; d < head_dim; d += 64) {
          const float2 v = load2(src + d);
          sum = fmaf(v.x, v.x, fmaf(v.y, v.y, sum));
        }
      } else {
        for (int d = lane; d < head_dim; d += 32) {
          const float v = to_float(src[d]);
          sum = fmaf(v, v, sum);
        }
      }
      sum = warp_sum(sum);
      inverse = rsqrtf(sum / (float)head_dim + eps);
    }
    const float lift = is_query ? temperature : 1.0f;
    T* dst = (is_query || key_in_place) ? src : k_pages + ((size_t)slot * kv_heads + (unit - heads)) * head_dim;
    if (interleaved) {
      // pair i is (2 i, 2 i + 1): a lane takes whole pairs, so the two layouts of the loop below do not apply
      for (int pair = lane; pair < half; pair += 32) {
        float first, second;
        if (PAIRED) { const float2 v = load2(src + 2 * pair); first = v.x; second = v.y; }
        else { first = to_float(src[2 * pair]); second = to_float(src[2 * pair + 1]); }
        if (norm) {
          first = first * inverse * norm[2 * pair];
          second = second * inverse * norm[2 * pair + 1];
        }
        const float cosine = angles[pair], sine = angles[half + pair];
        first *= lift; second *= lift;
        const float a = first * cosine - second * sine, b = second * cosine + first * sine;
        if (PAIRED) store2(dst + 2 * pair, a, b);
        else { dst[2 * pair] = from_float<T>(a); dst[2 * pair + 1] = from_float<T>(b); }
      }
      for (int d = rotary_dim + lane; d < head_dim; d += 32) {
        float v = to_float(src[d]);
        if (norm) v = v * inverse * norm[d];
        dst[d] = from_float<T>(v * lift);
      }
    } else if (PAIRED) {
      for (int pair = 2 * lane; pair < half; pair += 64) {
        float2 first = load2(src + pair), second = load2(src + pair + half);
        if (norm) {
          first.x *= inverse * norm[pair]; first.y *= inverse * norm[pair + 1];
          second.x *= inverse * norm[pair + half]; second.y *= inverse * norm[pair + half + 1];
        }
        first.x *= lift; first.y *= lift; second.x *= lift; second.y *= lift;
        const float c0 = angles[pair], c1 = angles[pair + 1], s0 = angles[half + pair], s1 = angles[half + pair + 1];
        store2(dst + pair, first.x * c0 - second.x * s0, first.y * c1 - second.y * s1);
        store2(dst + pair + half, first.x * s0 + second.x * c0, first.y * s1 + second.y * c1);
      }
      for (int d = rotary_dim + 2 * lane; d < head_dim; d += 64) {
        float2 v = load2(src + d);
        if (norm) { v.x *= inverse * norm[d]; v.y *= inverse * norm[d + 1]; }
        store2(dst + d, v.x * lift, v.y * lift);
      }
    } else {
      for (int pair = lane; pair < half; pair += 32) {
        float first = to_float(src[pair]);
        float second = to_float(src[pair + half]);
        if (norm) {
          first = first * inverse * norm[pair];
          second = second * inverse * norm[pair + half];
        }
        first *= lift; second *= lift;
        const float cosine = angles[pair], sine = angles[half + pair];
        dst[pair] = from_float<T>(first * cosine - second * sine);
        dst[pair + half] = from_float<T>(first * sine + second * cosine);
      }
      for (int d = rotary_dim + lane; d < head_dim; d += 32) {
        float v = to_float(src[d]);
        if (norm) v = v * inverse * norm[d];
        dst[d] = from_float<T>(v * lift);
      }
    }
  }
}

// time stamps (trace.cuh) of the first and the last CTA of the kernel below: 0 start, 1 the projection is over,
// 2 end; tag 100 / 101
MIR_TRACE_DEFINE(rope)

// bf16, half a head a multiple of 8 elements: L = half / 8 lanes take one head, each with two 16-byte pieces (elements
// 8 l .. 8 l + 7 and those half a head further), so a warp works on 32 / L heads at once and every access is 16 bytes
// wide.  Half-split pairs (the whole head rotated, rotary_dim == head_dim): a lane's two pieces are each other's
// partners.  INTERLEAVED pairs (2 i, 2 i + 1) of the first rotary_dim channels: both of a pair lie in one piece.
// row_width: elements from one token's row to the next (what lies behind q, k and v is left alone); queries_only:
// the rows hold no keys and values.  value_columns > 0: value heads have a width of their own; all of a token's values
// (that many columns, a multiple of 8) are copied to their place in the pages as one run by the token's last CTA.
template <int L, bool INTERLEAVED>
__global__ void qk_rope_store_wide_kernel(__nv_bfloat16* __restrict__ qkv, const int* __restrict__ positions,
                                          const int* __restrict__ slot_mapping, const float* __restrict__ inv_freq,
                                          const float* __restrict__ q_norm, const float* __restrict__ k_norm,
                                          __nv_bfloat16* __restrict__ k_pages, __nv_bfloat16* __restrict__ v_pages,
                                          int heads, int kv_heads, float eps, int write_kv, int units_per_cta,
                                          int rotary_dim, long long row_width, int queries_only, QkForms forms,
                                          int value_columns) {
  constexpr int HALF = 8 * L, DIM = 2 * HALF, GROUPS = 32 / L;
  const int pairs = rotary_dim / 2;                  // HALF for half-split pairs
  __shared__ float angles[DIM];                      // [pairs] cosines then [pairs] sines of this token
  grid_launch_dependents();
  MIR_TRACE_BEGIN(rope, (blockIdx.x == 0 && blockIdx.y == 0) || (blockIdx.x == gridDim.x - 1 && blockIdx.y == gridDim.y - 1),
                  100 + (blockIdx.x == 0 && blockIdx.y == 0 ? 0 : 1))
  if (threadIdx.x == 0) MIR_TRACE_POINT(rope, 0);
  const int token = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int group = lane / L, l = lane % L;
  const int units = queries_only ? heads : heads + (forms.values_from_keys || value_columns > 0 ? 1 : 2) * kv_heads;
  __nv_bfloat16* row = qkv + (size_t)token * (size_t)row_width;
  const float position = (float)positions[token];
  const int slot = slot_mapping ? slot_mapping[token] : -1;
  // positions and slots are older than the kernel before this one (the projection): the angles are computed
  // while it may still be running, then this kernel waits for its rows
  for (int pair = threadIdx.x; pair < pairs; pair += blockDim.x) {
    float sine, cosine;
    sincosf(position * inv_freq[pair], &sine, &cosine);
    angles[pair] = cosine * forms.magnitude;
    angles[pairs + pair] = sine * forms.magnitude;
  }
  const float temperature = query_temperature(forms, positions[token]);
  grid_dependency_wait();
  __syncthreads();
  if (threadIdx.x == 0) MIR_TRACE_POINT(rope, 1);
  const int unit_begin = blockIdx.y * units_per_cta, unit_end = min(units, unit_begin + units_per_cta);
  if (value_columns > 0 && write_kv == 1 && slot >= 0 && blockIdx.y == gridDim.y - 1) {
    const uint4* from = reinterpret_cast<const uint4*>(row + (size_t)(heads + kv_heads) * DIM);
    uint4* to = reinterpret_cast<uint4*>(v_pages + (size_t)slot * value_columns);
    for (int c = threadIdx.x; c < value_columns / 8; c += blockDim.x) to[c] = from[c];
  }
  for (int base = unit_begin + warp * GROUPS; base < unit_end; base += warps * GROUPS) {
    const int unit = base + group;
    const bool active = unit < unit_end;
    const bool is_query = unit < heads, is_value = unit >= heads + kv_heads;
    const __nv_bfloat16* src = row + (size_t)unit * DIM;
    uint4 a = make_uint4(0u, 0u, 0u, 0u), b = a;
    if (active) {
      a = *reinterpret_cast<const uint4*>(src + 8 * l);
      b = *reinterpret_cast<const uint4*>(src + HALF + 8 * l);
    }
    const bool in_place = is_query || (write_kv == 2 && !is_value);
    const bool writes = active && (in_place || (write_kv == 1 && slot >= 0));
    __nv_bfloat16* dst = nullptr;
    if (writes)
      dst = in_place ? row + (size_t)unit * DIM
                     : (is_value ? v_pages + ((size_t)slot * kv_heads + (unit - heads - kv_heads)) * DIM
                                 : k_pages + ((size_t)slot * kv_heads + (unit - heads)) * DIM);
    if (forms.values_from_keys && writes && !is_query && write_kv == 1) {      // the value: the key as it was projected
      __nv_bfloat16* value = v_pages + ((size_t)slot * kv_heads + (unit - heads)) * DIM;
      *reinterpret_cast<uint4*>(value + 8 * l) = a;
      *reinterpret_cast<uint4*>(value + HALF + 8 * l) = b;
    }
    float fa[8], fb[8];
    {
      const __nv_bfloat162* ha = reinterpret_cast<const __nv_bfloat162*>(&a);
      const __nv_bfloat162* hb = reinterpret_cast<const __nv_bfloat162*>(&b);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 x = __bfloat1622float2(ha[i]), y = __bfloat1622float2(hb[i]);
        fa[2 * i] = x.x; fa[2 * i + 1] = x.y; fb[2 * i] = y.x; fb[2 * i + 1] = y.y;
      }
    }
    const float* norm = (!active || is_value) ? nullptr : (is_query ? q_norm : k_norm);
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) sum = fmaf(fa[i], fa[i], fmaf(fb[i], fb[i], sum));
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);   // every lane takes part
    if (norm) {
      const float inverse = rsqrtf(sum / (float)DIM + eps);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        fa[i] *= inverse * norm[8 * l + i];
        fb[i] *= inverse * norm[HALF + 8 * l + i];
      }
    }
    if (!writes) continue;
    if (!is_value) {
      if (is_query && forms.temperature_every > 0.0f) {
#pragma unroll
        for (int i = 0; i < 8; ++i) { fa[i] *= temperature; fb[i] *= temperature; }
      }
      if (INTERLEAVED) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int low = 4 * l + j, high = HALF / 2 + 4 * l + j;      // the pairs of this lane's two pieces
          if (low < pairs) {
            const float cosine = angles[low], sine = angles[pairs + low];
            const float first = fa[2 * j], second = fa[2 * j + 1];
            fa[2 * j] = first * cosine - second * sine;
            fa[2 * j + 1] = second * cosine + first * sine;
          }
          if (high < pairs) {
            const float cosine = angles[high], sine = angles[pairs + high];
            const float first = fb[2 * j], second = fb[2 * j + 1];
            fb[2 * j] = first * cosine - second * sine;
            fb[2 * j + 1] = second * cosine + first * sine;
          }
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float cosine = angles[8 * l + i], sine = angles[HALF + 8 * l + i];
          const float first = fa[i], second = fb[i];
          fa[i] = first * cosine - second * sine;
          fb[i] = first * sine + second * cosine;
        }
      }
      __nv_bfloat162* ha = reinterpret_cast<__nv_bfloat162*>(&a);
      __nv_bfloat162* hb = reinterpret_cast<__nv_bfloat162*>(&b);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        ha[i] = __floats2bfloat162_rn(fa[2 * i], fa[2 * i + 1]);
        hb[i] = __floats2bfloat162_rn(fb[2 * i], fb[2 * i + 1]);
      }
    }
    *reinterpret_cast<uint4*>(dst + 8 * l) = a;                // a value head is copied as it is
    *reinterpret_cast<uint4*>(dst + HALF + 8 * l) = b;
  }
  if (threadIdx.x == 0) MIR_TRACE_POINT(rope, 2);
}

template <int L>
int launch_rope_wide(__nv_bfloat16* qkv, const int* positions, const int* slot_mapping, const float* inv_freq,
                     const float* q_norm, const float* k_norm, __nv_bfloat16* k_pages, __nv_bfloat16* v_pages, int tokens,
                     int heads, int kv_heads, float eps, int write_kv, cudaStream_t stream, int interleaved = 0,
                     int rotary_dim = 16 * L, long long row_width = 0, int queries_only = 0, QkForms forms = {},
                     int value_columns = 0) {
  const int units = queries_only ? heads : heads + (forms.values_from_keys || value_columns > 0 ? 1 : 2) * kv_heads;
  if (row_width == 0) row_width = (long long)units * 16 * L + value_columns;
  const bool many = tokens >= 256;                     // one CTA of 8 warps per token, else CTAs of 4 warps
  const int threads = many ? 256 : 128;
  const int units_per_cta = many ? units : 4 * (32 / L);
  const dim3 grid(tokens, (units + units_per_cta - 1) / units_per_cta);
  if (interleaved)
    return mir_launch_with(mir_pdl_for_streaming(), "qk_rope_store", qk_rope_store_wide_kernel<L, true>, grid, dim3(threads),
                           0, stream, 0, qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, heads,
                           kv_heads, eps, write_kv, units_per_cta, rotary_dim, row_width, queries_only, forms, value_columns);
  return mir_launch_with(mir_pdl_for_streaming(), "qk_rope_store", qk_rope_store_wide_kernel<L, false>, grid, dim3(threads),
                         0, stream, 0, qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, heads,
                         kv_heads, eps, write_kv, units_per_cta, rotary_dim, row_width, queries_only, forms, value_columns);
}

template <typename T>
int launch_rope(T* qkv, const int* positions, const int* slot_mapping, const float* inv_freq, const float* q_norm,
                const float* k_norm, T* k_pages, T* v_pages, int tokens, int heads, int kv_heads, int head_dim,
                int value_dim, int rotary_dim, float eps, int write_kv, int interleaved, long long row_stride,
                int queries_only, QkForms forms, cudaStream_t stream) {
  // few tokens: 4 warps per CTA and enough CTAs per token to give every head a warp; many tokens: one CTA of 8
  // warps per token, so that the token's angles are computed once
  const int units = queries_only ? heads : heads + (forms.values_from_keys ? 1 : 2) * kv_heads;
  const bool many = tokens >= 256;
  const int threads = many ? 256 : 128;
  const int units_per_cta = many ? units : 4;
  const dim3 grid(tokens, (units + units_per_cta - 1) / units_per_cta);
  const size_t smem = (size_t)rotary_dim * sizeof(float);
  // (every head of a row, and every page row, then starts on an even element)
  const bool paired = (head_dim % 2 == 0) && (value_dim % 2 == 0) && (rotary_dim % (interleaved ? 2 : 4) == 0) &&
                      (row_stride % 2 == 0) && ((uintptr_t)qkv % (2 * sizeof(T)) == 0) &&
                      ((uintptr_t)k_pages % (2 * sizeof(T)) == 0);
  if (paired)
    return mir_launch("qk_rope_store", qk_rope_store_kernel<T, true>, grid, dim3(threads), smem, stream, 0, qkv, positions,
                      slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, heads, kv_heads, head_dim, value_dim,
                      rotary_dim, eps, write_kv, units_per_cta, interleaved, row_stride, queries_only, forms);
  return mir_launch("qk_rope_store", qk_rope_store_kernel<T, false>, grid, dim3(threads), smem, stream, 0, qkv, positions,
                    slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, heads, kv_heads, head_dim, value_dim,
                    rotary_dim, eps, write_kv, units_per_cta, interleaved, row_stride, queries_only, forms);
}

static int qk_rope_store_with(int bf16, void* qkv, const int* positions, const int* slot_mapping,
                                 const float* inv_freq, const float* q_norm, const float* k_norm, void* k_pages,
                                 void* v_pages, int tokens, int heads, int kv_heads, int head_dim, int value_dim,
                                 int rotary_dim, float eps, int write_kv, int interleaved, long long row_stride,
                                 int queries_only, const QkForms& forms, cudaStream_t stream) {
  if (tokens == 0) return MIR_OK;
  if (tokens < 0 || heads <= 0 || kv_heads <= 0 || head_dim <= 0 || value_dim <= 0 || rotary_dim < 0 || rotary_dim > head_dim ||
      (rotary_dim & 1)) {
    mir_set_error("qk_rope_store: bad sizes (heads %d, kv heads %d, head_dim %d, rotary_dim %d)", heads, kv_heads,
                  head_dim, rotary_dim);
    return MIR_BAD_ARGUMENT;
  }
  if (rotary_dim > 8192) { mir_set_error("qk_rope_store: rotary_dim %d is too large", rotary_dim); return MIR_BAD_ARGUMENT; }
  if (forms.values_from_keys && (value_dim != head_dim || queries_only || write_kv == 2)) {
    mir_set_error("qk_rope_store: values that are the keys have the keys' width and go to the pages with them");
    return MIR_BAD_ARGUMENT;
  }
  const long long packed_width = (long long)(heads + kv_heads) * head_dim +
                                 (forms.values_from_keys ? 0 : (long long)kv_heads * value_dim);
  if (row_stride < 0 || (row_stride > 0 && row_stride < (queries_only ? (long long)heads * head_dim : packed_width)) ||
      (queries_only && (write_kv != 0 || row_stride == 0))) {
    mir_set_error("qk_rope_store: a row stride of %lld does not hold the row, or rows of queries alone were asked to "
                  "write keys", row_stride);
    return MIR_BAD_ARGUMENT;
  }
  if (row_stride == packed_width && !queries_only) row_stride = 0;
  // (without a rotation the pairs' layout does not matter: the interleaved form takes any row stride)
  const bool wide_rotation = interleaved || rotary_dim == 0 ? true : (rotary_dim == head_dim && row_stride == 0);
  const int value_columns = value_dim != head_dim && !queries_only ? kv_heads * value_dim : 0;
  const int wide_interleaved = interleaved || rotary_dim == 0;
  if (bf16 && wide_rotation && row_stride % 8 == 0 && value_columns % 8 == 0 && head_dim % 16 == 0 &&
      ((uintptr_t)qkv & 15) == 0 && ((uintptr_t)k_pages & 15) == 0 && ((uintptr_t)v_pages & 15) == 0) {
    __nv_bfloat16* q = (__nv_bfloat16*)qkv;
    __nv_bfloat16* kp = (__nv_bfloat16*)k_pages;
    __nv_bfloat16* vp = (__nv_bfloat16*)v_pages;
    switch (head_dim / 16) {                             // lanes per head
      case 1: return launch_rope_wide<1>(q, positions, slot_mapping, inv_freq, q_norm, k_norm, kp, vp, tokens, heads, kv_heads, eps, write_kv, stream, wide_interleaved, rotary_dim, row_stride, queries_only, forms, value_columns);
      case 2: return launch_rope_wide<2>(q, positions, slot_mapping, inv_freq, q_norm, k_norm, kp, vp, tokens, heads, kv_heads, eps, write_kv, stream, wide_interleaved, rotary_dim, row_stride, queries_only, forms, value_columns);
      case 4: return launch_rope_wide<4>(q, positions, slot_mapping, inv_freq, q_norm, k_norm, kp, vp, tokens, heads, kv_heads, eps, write_kv, stream, wide_interleaved, rotary_dim, row_stride, queries_only, forms, value_columns);
      case 8: return launch_rope_wide<8>(q, positions, slot_mapping, inv_freq, q_norm, k_norm, kp, vp, tokens, heads, kv_heads, eps, write_kv, stream, wide_interleaved, rotary_dim, row_stride, queries_only, forms, value_columns);
      case 16: return launch_rope_wide<16>(q, positions, slot_mapping, inv_freq, q_norm, k_norm, kp, vp, tokens, heads, kv_heads, eps, write_kv, stream, wide_interleaved, rotary_dim, row_stride, queries_only, forms, value_columns);
      default: break;                                    // other head sizes: the kernel below
    }
  }
  if (bf16)
    return launch_rope((__nv_bfloat16*)qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, (__nv_bfloat16*)k_pages,
                       (__nv_bfloat16*)v_pages, tokens, heads, kv_heads, head_dim, value_dim, rotary_dim, eps, write_kv,
                       interleaved, row_stride, queries_only, forms, stream);
  return launch_rope((float*)qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, (float*)k_pages, (float*)v_pages,
                     tokens, heads, kv_heads, head_dim, value_dim, rotary_dim, eps, write_kv, interleaved, row_stride,
                     queries_only, forms, stream);
}

MIR_EXPORT int mir_qk_rope_store(int bf16, void* qkv, const int* positions, const int* slot_mapping,
                                 const float* inv_freq, const float* q_norm, const float* k_norm, void* k_pages,
                                 void* v_pages, int tokens, int heads, int kv_heads, int head_dim, int value_dim,
                                 int rotary_dim, float eps, int write_kv, int interleaved, long long row_stride,
                                 int queries_only, cudaStream_t stream) {
  return qk_rope_store_with(bf16, qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, tokens, heads,
                            kv_heads, head_dim, value_dim, rotary_dim, eps, write_kv, interleaved, row_stride,
                            queries_only, QkForms{}, stream);
}

// The same with the further forms (QkForms).
MIR_EXPORT int mir_qk_rope_store_forms(int bf16, void* qkv, const int* positions, const int* slot_mapping,
                                       const float* inv_freq, const float* q_norm, const float* k_norm, void* k_pages,
                                       void* v_pages, int tokens, int heads, int kv_heads, int head_dim, int value_dim,
                                       int rotary_dim, float eps, int write_kv, int interleaved, long long row_stride,
                                       int queries_only, float magnitude, float temperature_coef,
                                       float temperature_every, int values_from_keys, cudaStream_t stream) {
  if (!(magnitude > 0.0f) || !(temperature_every >= 0.0f)) {
    mir_set_error("qk_rope_store: the magnitude must be above zero and the temperature's step not below it");
    return MIR_BAD_ARGUMENT;
  }
  const QkForms forms{magnitude, temperature_coef, temperature_every, values_from_keys};
  return qk_rope_store_with(bf16, qkv, positions, slot_mapping, inv_freq, q_norm, k_norm, k_pages, v_pages, tokens, heads,
                            kv_heads, head_dim, value_dim, rotary_dim, eps, write_kv, interleaved, row_stride,
                            queries_only, forms, stream);
}
