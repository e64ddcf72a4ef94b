// The state of a short causal convolution: a request's last taps - 1 inputs, [slot][tap][channel] 32-bit.
#pragma once
#include "common.cuh"

namespace mir {

constexpr int kMaxTaps = 16;

// grid (rows, ceil(channels / 256)); skip_single: requests that bring one token were moved on by their convolution.
// the last taps-1 inputs of the request, old ones where the portion is shorter.
template <typename T>
__global__ void short_conv_tail_kernel(const T* __restrict__ x, long long ldx, float* __restrict__ tail,
                                       const int* __restrict__ query_starts, const int* __restrict__ state_slots,
                                       const int* __restrict__ positions, int channels, int taps, int skip_single) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int row = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  const int start = query_starts[row], count = query_starts[row + 1] - start;
  if (c >= channels || count <= 0 || positions[start] < 0 || (skip_single && count == 1)) return;
  float* mine = tail + (size_t)state_slots[row] * (taps - 1) * channels;
  float keep[kMaxTaps];
  for (int j = 0; j < taps - 1; ++j) {
    const int src = count - (taps - 1) + j;
    keep[j] = src >= 0 ? to_float(x[(size_t)(start + src) * ldx + c]) : mine[(size_t)(taps - 1 + src) * channels + c];
  }
  for (int j = 0; j < taps - 1; ++j) mine[(size_t)j * channels + c] = keep[j];
}

}  // namespace mir
