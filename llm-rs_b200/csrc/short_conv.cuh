// Short causal convolutions over time, one filter per channel, in front of recurrent mixers: y_t = bias + sum_j
// taps[K - 1 - j] x_(t - j), zeros before a sequence's start. The last K - 1 rows that entered are per-request state
// (float32 [slots, K - 1, C], oldest row first), so a sequence may be cut anywhere.
#pragma once
#include "common.cuh"

__device__ __forceinline__ float rec_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float rec_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float rec_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// Channel c of token t, which is its request's token number `off` of the step; `taps` is the channel's filter [K],
// `tail` the request's kept rows [K - 1, C].
template <typename TA>
__device__ __forceinline__ float short_conv_at(const TA* __restrict__ x, long long stride, int t, int off, int c,
                                               const float* __restrict__ taps, int K, const float* __restrict__ tail,
                                               int C, float bias) {
  float acc = bias;
  for (int j = 0; j < K; ++j) {      // lag j: the input of j tokens ago
    const int o = off - j;
    const float in = o >= 0 ? to_float(x[(size_t)(t - j) * stride + c]) : tail[(size_t)(K - 1 + o) * C + c];
    acc = fmaf(taps[K - 1 - j], in, acc);
  }
  return acc;
}

// A block per request, after the kernel that reads the old rows: the request's last K - 1 inputs become its state (with
// `in_bias`, a number per channel that is part of every input, added).
template <typename TA>
static __global__ void short_conv_state_kernel(const TA* __restrict__ x, long long stride, float* __restrict__ conv_state,
                                               const int* __restrict__ q_start, const int* __restrict__ n_new,
                                               const int* __restrict__ slot_ids, int C, int K,
                                               const float* __restrict__ in_bias) {
  const int req = blockIdx.x, n = n_new[req], t0 = q_start[req];
  float* tail = conv_state + (size_t)slot_ids[req] * (K - 1) * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
    for (int j = 0; j < K - 1; ++j) {      // ascending: an old row is read before the place it moves from is overwritten
      const int o = n - (K - 1) + j;
      tail[(size_t)j * C + c] = o >= 0 ? to_float(x[(size_t)(t0 + o) * stride + c]) + (in_bias ? in_bias[c] : 0.f)
                                       : tail[(size_t)(j + n) * C + c];
    }
}

template <typename TA>
static int launch_short_conv_state(const TA* x, long long stride, float* conv_state, const int* q_start,
                                   const int* n_new, const int* slot_ids, int n_requests, int C, int K,
                                   cudaStream_t stream, const float* in_bias = nullptr) {
  if (K <= 1) return 0;
  const int slices = (C + 255) / 256;      // a request's channels over several blocks: a thread walks a channel's K - 1 rows
  short_conv_state_kernel<TA><<<dim3(n_requests, slices), 256, 0, stream>>>(x, stride, conv_state, q_start, n_new,
                                                                            slot_ids, C, K, in_bias);
  return llmrs_launch_status("short convolution (state)");
}
