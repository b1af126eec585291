// What a short causal convolution over time leaves behind: a request's last taps - 1 inputs.
#pragma once
#include "common.cuh"

// x [T, ld] (the first `channels` columns); a slot's state at state + slot * state_stride:
// [channels, taps - 1], oldest first.  Runs after everything that still reads the old inputs.
template <typename T>
__global__ void causal_conv_state_kernel(float* __restrict__ state, long state_stride,
                                         const T* __restrict__ x, int ld,
                                         const int* __restrict__ cu_tokens,
                                         const int* __restrict__ slots, int n_seqs, int channels,
                                         int taps) {
  pdl_launch_dependents();
  pdl_wait();
  const int keep = taps - 1;
  const size_t total = (size_t)n_seqs * channels;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const int s = (int)(idx / channels), c = (int)(idx - (size_t)s * channels);
    const int t0 = cu_tokens[s], n = cu_tokens[s + 1] - t0;
    float* st = state + (size_t)slots[s] * state_stride + (size_t)c * keep;
    // ascending j reads old entries at j + n >= j only: in place is safe
    for (int j = 0; j < keep; ++j) {
      const int src = n - keep + j;
      st[j] = src >= 0 ? to_float(x[(size_t)(t0 + src) * ld + c]) : st[j + n];
    }
  }
}
