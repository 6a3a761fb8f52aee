// A gated linear recurrence per channel (real-gated linear recurrent unit, RG-LRU) and the stand-alone short convolution
// in front of it.
//
//   u_t = conv_bias + sum_j taps[K - 1 - j] (x_(t-j) + x_bias),  x before the sequence's start counts as zero with no bias
//   r, i = sigmoid of two block-diagonal products of u (their biases added): gemm_grouped.cu's gates epilogue, which
//          leaves per token and channel the pair  a = exp(rate * r),  b = sqrt(1 - a^2) * i * u      (float32)
//   S_t = a_t S_(t-1) + b_t,      out_t = S_t * gelu_tanh(y_t + y_bias)
//
// The state (float32 [slots, W]) and the last K - 1 convolution inputs (float32 [slots, K - 1, W]) are per request.
//
//   scan  the recurrence is an associative composition of affine maps, so a block takes 16 channels of a request and 64 (or
//         32, in steps of short portions) runs of up to 8 tokens side by side: every thread composes its run's maps from registers, a warp per channel
//         composes the runs and turns them into start states, and every thread walks its run again. 512 (256) tokens a
//         turn, the state carried from turn to turn.
//   step  one token per request (decoding): products, gates, recurrence and output in one kernel.
// Everything but x, u, y and the output (activation type) is float32.
#include "common.cuh"
#include "short_conv.cuh"

using bf16 = __nv_bfloat16;

// gelu_tanh(z) = z (1 + tanh(x)) / 2 with x = sqrt(2 / pi) (z + 0.044715 z^3), that is z * sigmoid(2 x). For bfloat16
// activations the exponential and the division are the hardware's (a few units in the last place of float32).
template <typename T>
__device__ __forceinline__ float gelu_tanh(float z) {
  const float x2 = 1.5957691216057308f * fmaf(0.044715f * z * z, z, z);
  return sizeof(T) == 4 ? z / (1.0f + expf(-x2)) : __fdividef(z, 1.0f + __expf(fminf(-x2, 80.0f)));
}

// V neighbouring elements, V * sizeof(T) a multiple of 16 bytes or V == 1.
template <typename T, int V>
__device__ __forceinline__ void load_v(const T* p, float* out) {
  if (V == 1) {
    out[0] = to_float(p[0]);
  } else if (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
      out[i] = a.x; out[i + 1] = a.y; out[i + 2] = a.z; out[i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; i += 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p) + i);
      const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(h[e]);
        out[i + 2 * e] = f.x;
        out[i + 2 * e + 1] = f.y;
      }
    }
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_v(T* p, const float* v) {
  if (V == 1) {
    p[0] = from_float<T>(v[0]);
  } else if (sizeof(T) == 4) {
#pragma unroll
    for (int i = 0; i < V; i += 4)
      *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; i += 8) {
      uint4 raw;
      __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(v[i + 2 * e], v[i + 2 * e + 1]);
      *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p) + i) = raw;
    }
  }
}

// ---------------------------------------------------------------------------------
// The short convolution by itself. A thread: V channels of one token. `taps` is [K, W] (oldest lag first). With `single`
// (every request of the step brings one token) a thread is the only one that touches its channels of its request's kept
// rows and moves them on itself; otherwise a kernel after this one does.
// ---------------------------------------------------------------------------------
template <typename T, int V>
__global__ void short_conv_kernel(const T* __restrict__ x, long long stride, const float* __restrict__ x_bias,
                                  const float* __restrict__ taps, const float* __restrict__ bias,
                                  float* __restrict__ conv_state, const int* __restrict__ token_req,
                                  const int* __restrict__ q_start, const int* __restrict__ slot_ids, T* __restrict__ u,
                                  int W, int K, int single) {
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V, t = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  if (c >= W) return;
  const int req = token_req[t], off = t - q_start[req];
  float* tail = conv_state + (size_t)slot_ids[req] * (K - 1) * W + c;
  float acc[V], in[V], xb[V], own[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    acc[e] = bias ? bias[c + e] : 0.f;
    xb[e] = x_bias ? x_bias[c + e] : 0.f;
    own[e] = 0.f;
  }
  for (int j = 0; j < K; ++j) {      // lag j: the input of j tokens ago
    const int o = off - j;
    if (o >= 0) {
      load_v<T, V>(x + (size_t)(t - j) * stride + c, in);
#pragma unroll
      for (int e = 0; e < V; ++e) in[e] += xb[e];
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) in[e] = tail[(size_t)(K - 1 + o) * W + e];
    }
    const float* w = taps + (size_t)(K - 1 - j) * W + c;
#pragma unroll
    for (int e = 0; e < V; ++e) {
      if (j == 0) own[e] = in[e];
      acc[e] = fmaf(w[e], in[e], acc[e]);
    }
  }
  store_v<T, V>(u + (size_t)t * W + c, acc);
  if (single && K > 1) {
    for (int r = 0; r + 1 < K - 1; ++r)
#pragma unroll
      for (int e = 0; e < V; ++e) tail[(size_t)r * W + e] = tail[(size_t)(r + 1) * W + e];
#pragma unroll
    for (int e = 0; e < V; ++e) tail[(size_t)(K - 2) * W + e] = own[e];
  }
}

// The same with one token per request and a filter of at most four taps: the kept rows are asked for together.
template <typename T, int V, int K>
__global__ void short_conv_step_kernel(const T* __restrict__ x, long long stride, const float* __restrict__ x_bias,
                                       const float* __restrict__ taps, const float* __restrict__ bias,
                                       float* __restrict__ conv_state, const int* __restrict__ slot_ids,
                                       T* __restrict__ u, int W) {
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V, t = blockIdx.x;
  const bool live = c < W;
  float w[K][V], xb[V], acc[V], in[K][V];      // in[j]: the input of j tokens ago
#pragma unroll
  for (int e = 0; e < V; ++e) {
    xb[e] = live && x_bias ? x_bias[c + e] : 0.f;
    acc[e] = live && bias ? bias[c + e] : 0.f;
#pragma unroll
    for (int j = 0; j < K; ++j) w[j][e] = live ? taps[(size_t)(K - 1 - j) * W + c + e] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  if (!live) return;
  float* tail = conv_state + (size_t)slot_ids[t] * (K - 1) * W + c;
  load_v<T, V>(x + (size_t)t * stride + c, in[0]);
#pragma unroll
  for (int j = 1; j < K; ++j) load_v<float, V>(tail + (size_t)(K - 1 - j) * W, in[j]);
#pragma unroll
  for (int e = 0; e < V; ++e) in[0][e] += xb[e];
#pragma unroll
  for (int j = 0; j < K; ++j)
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = fmaf(w[j][e], in[j][e], acc[e]);
  store_v<T, V>(u + (size_t)t * W + c, acc);
#pragma unroll
  for (int j = 0; j < K - 1; ++j) store_v<float, V>(tail + (size_t)(K - 2 - j) * W, in[j]);
}

// Prompts: a thread takes V channels of SC_TOK tokens in a row (of the step, whatever requests they belong to) and keeps
// the last K inputs in registers: every row is read once. All of its rows are asked for before the first is used.
constexpr int SC_TOK = 8;

template <typename T, int V, int K>
__global__ void __launch_bounds__(128)
short_conv_rows_kernel(const T* __restrict__ x, long long stride, const float* __restrict__ x_bias,
                       const float* __restrict__ taps, const float* __restrict__ bias,
                       const float* __restrict__ conv_state, const int* __restrict__ token_req,
                       const int* __restrict__ q_start, const int* __restrict__ slot_ids, T* __restrict__ u, int W,
                       int n_tokens) {
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V, t0 = blockIdx.x * SC_TOK;
  if (c >= W) return;
  const int nt = min(SC_TOK, n_tokens - t0);
  uint4 raw[SC_TOK];
#pragma unroll
  for (int i = 0; i < SC_TOK; ++i)
    if (i < nt) raw[i] = *reinterpret_cast<const uint4*>(x + (size_t)(t0 + i) * stride + c);
  float w[K][V], xb[V], b0[V], win[K][V];      // win[j]: the input of j tokens ago
#pragma unroll
  for (int e = 0; e < V; ++e) {
    xb[e] = x_bias ? x_bias[c + e] : 0.f;
    b0[e] = bias ? bias[c + e] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < K; ++j)
#pragma unroll
    for (int e = 0; e < V; ++e) {
      w[j][e] = taps[(size_t)(K - 1 - j) * W + c + e];
      win[j][e] = 0.f;
    }
#pragma unroll
  for (int i = 0; i < SC_TOK; ++i) {
    if (i >= nt) break;
    const int t = t0 + i, req = token_req[t], off = t - q_start[req];
    if (i == 0 || off == 0) {      // the inputs before this token: earlier rows of the request, or its kept rows
      const float* tail = conv_state + (size_t)slot_ids[req] * (K - 1) * W + c;
#pragma unroll
      for (int j = 1; j < K; ++j) {
        const int o = off - j;
        if (o >= 0) {
          load_v<T, V>(x + (size_t)(t - j) * stride + c, win[j]);
#pragma unroll
          for (int e = 0; e < V; ++e) win[j][e] += xb[e];
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) win[j][e] = tail[(size_t)(K - 1 + o) * W + e];
        }
      }
    } else {
#pragma unroll
      for (int j = K - 1; j > 0; --j)
#pragma unroll
        for (int e = 0; e < V; ++e) win[j][e] = win[j - 1][e];
    }
    load_v<T, V>(reinterpret_cast<const T*>(&raw[i]), win[0]);
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      win[0][e] += xb[e];
      acc[e] = b0[e];
    }
#pragma unroll
    for (int j = 0; j < K; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = fmaf(w[j][e], win[j][e], acc[e]);
    store_v<T, V>(u + (size_t)t * W + c, acc);
  }
}

template <typename T>
static int launch_short_conv(const void* x, long long stride, const float* x_bias, const float* taps, const float* bias,
                             float* conv_state, const int* token_req, const int* q_start, const int* n_new,
                             const int* slot_ids, void* u, int n_tokens, int n_requests, int W, int K, int single,
                             cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = W % V == 0 && stride % V == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)u & 15) == 0;
  const int per = vec ? W / V : W, threads = per >= 128 ? 128 : ((per + 31) / 32) * 32;
  const unsigned slices = (per + threads - 1) / threads;
  const dim3 grid(n_tokens, slices), tiles((n_tokens + SC_TOK - 1) / SC_TOK, slices);
#define LLMRS_SC_ROWS(KK)                                                                                        \
  short_conv_rows_kernel<T, V, KK><<<tiles, threads, 0, stream>>>((const T*)x, stride, x_bias, taps, bias,       \
                                                                  conv_state, token_req, q_start, slot_ids, (T*)u, W, \
                                                                  n_tokens)
  if (vec && !single && K <= 4) {
    if (K == 1) LLMRS_SC_ROWS(1);
    else if (K == 2) LLMRS_SC_ROWS(2);
    else if (K == 3) LLMRS_SC_ROWS(3);
    else LLMRS_SC_ROWS(4);
  } else if (vec && K >= 2 && K <= 4) {
#define LLMRS_SC_STEP(KK)                                                                                              \
  llmrs_launch(short_conv_step_kernel<T, V, KK>, grid, dim3(threads), 0, stream, true, (const T*)x, stride, x_bias, taps, \
               bias, conv_state, slot_ids, (T*)u, W)
    if (K == 2) LLMRS_SC_STEP(2);
    else if (K == 3) LLMRS_SC_STEP(3);
    else LLMRS_SC_STEP(4);
#undef LLMRS_SC_STEP
  } else if (vec) {
    llmrs_launch(short_conv_kernel<T, V>, grid, dim3(threads), 0, stream, true, (const T*)x, stride, x_bias, taps, bias,
                 conv_state, token_req, q_start, slot_ids, (T*)u, W, K, single);
  } else {
    llmrs_launch(short_conv_kernel<T, 1>, grid, dim3(threads), 0, stream, true, (const T*)x, stride, x_bias, taps, bias,
                 conv_state, token_req, q_start, slot_ids, (T*)u, W, K, single);
  }
#undef LLMRS_SC_ROWS
  const int rc = llmrs_launch_status("short_conv");
  if (rc || single) return rc;
  return launch_short_conv_state<T>((const T*)x, stride, conv_state, q_start, n_new, slot_ids, n_requests, W, K, stream,
                                    x_bias);
}

// x: [n_tokens, W] with rows `stride` apart; u: [n_tokens, W] dense. `single`: every request brings exactly one token.
LLMRS_API int llmrs_short_conv(const void* x, long long stride, int dtype, const float* x_bias, const float* taps,
                               const float* bias, float* conv_state, const int* token_req, const int* q_start,
                               const int* n_new, const int* slot_ids, void* u, int n_tokens, int n_requests, int W, int K,
                               int single, cudaStream_t stream) {
  LLMRS_REQUIRE(n_tokens >= 0 && n_requests >= 0 && W > 0 && K > 0, "short_conv: bad sizes");
  LLMRS_REQUIRE(!single || n_tokens == n_requests, "short_conv: %d tokens of %d requests are not one each", n_tokens,
                n_requests);
  if (n_tokens == 0) return 0;
  if (dtype == LLMRS_F32)
    return launch_short_conv<float>(x, stride, x_bias, taps, bias, conv_state, token_req, q_start, n_new, slot_ids, u,
                                    n_tokens, n_requests, W, K, single, stream);
  if (dtype == LLMRS_BF16)
    return launch_short_conv<bf16>(x, stride, x_bias, taps, bias, conv_state, token_req, q_start, n_new, slot_ids, u,
                                   n_tokens, n_requests, W, K, single, stream);
  return llmrs_fail("short_conv: unknown dtype %d", dtype);
}

// ---------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------
constexpr int RS_CH = 16, RS_LEN = 8;

template <typename T, int RS_RUNS>
__global__ void __launch_bounds__(RS_CH * RS_RUNS)
rglru_scan_kernel(const float2* __restrict__ ab, const T* __restrict__ y, long long y_stride,
                  const float* __restrict__ y_bias, float* __restrict__ state, const int* __restrict__ q_start,
                  const int* __restrict__ n_new, const int* __restrict__ slot_ids, T* __restrict__ out,
                  long long out_stride, int W) {
  __shared__ float2 run[RS_CH][RS_RUNS + 1];      // a run's composed map; then, in x, the state it starts from
  __shared__ float carry[RS_CH];
  const int req = blockIdx.y, n = n_new[req], t0 = q_start[req];
  const int tid = threadIdx.x, ch = tid % RS_CH, r = tid / RS_CH, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x * RS_CH + ch;
  const bool cin = c < W;
  float* st = state + (size_t)slot_ids[req] * W + c;
  if (r == 0) carry[ch] = cin ? *st : 0.f;
  const float yb = cin && y_bias ? y_bias[c] : 0.f;
  float2 v[RS_LEN];
  float yv[RS_LEN];
  int first = 0, len = 0;
  auto fetch = [&](int base) {
    const int per = min(RS_LEN, (n - base + RS_RUNS - 1) / RS_RUNS);      // short portions: shorter runs
    first = base + r * per;
    len = cin ? max(0, min(per, n - first)) : 0;
    const float2* src = ab + (size_t)(t0 + first) * W + c;
    const T* ys = y + (size_t)(t0 + first) * y_stride + c;
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) v[l] = l < len ? src[(size_t)l * W] : make_float2(1.f, 0.f);
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) yv[l] = l < len ? to_float(ys[(size_t)l * y_stride]) : 0.f;
  };
  fetch(0);
  for (int base = 0; base < n; base += RS_RUNS * RS_LEN) {
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) {
      A *= v[l].x;
      B = fmaf(v[l].x, B, v[l].y);
    }
    run[ch][r] = make_float2(A, B);
    __syncthreads();
    if (warp < RS_CH) {
      // Lane l holds runs 2 l and 2 l + 1 of channel `warp` (with 32 runs: run l); an inclusive scan over the lanes.
      constexpr int PER = RS_RUNS / 32;
      const float2 p0 = run[warp][PER * lane], p1 = PER == 2 ? run[warp][PER * lane + PER - 1] : make_float2(1.f, 0.f);
      float a = p1.x * p0.x, b = fmaf(p1.x, p0.y, p1.y);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float ea = __shfl_up_sync(0xffffffffu, a, o), eb = __shfl_up_sync(0xffffffffu, b, o);
        if (lane >= o) {
          b = fmaf(a, eb, b);
          a *= ea;
        }
      }
      const float s0 = carry[warp];
      float xa = __shfl_up_sync(0xffffffffu, a, 1), xb = __shfl_up_sync(0xffffffffu, b, 1);
      if (lane == 0) { xa = 1.f; xb = 0.f; }
      const float first_state = fmaf(xa, s0, xb);
      run[warp][PER * lane].x = first_state;
      if (PER == 2) run[warp][PER * lane + PER - 1].x = fmaf(p0.x, first_state, p0.y);
      __syncwarp();
      if (lane == 31) carry[warp] = fmaf(a, s0, b);
    }
    __syncthreads();
    float S = run[ch][r].x;
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) {
      S = fmaf(v[l].x, S, v[l].y);
      v[l].y = S;
    }
    __syncthreads();      // the runs' start states are read before the next turn overwrites them
    // The turn's outputs are made under the loads of the next turn's rows.
    float o[RS_LEN];
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) o[l] = v[l].y * gelu_tanh<T>(yv[l] + yb);
    const int n_out = len;
    T* dst = out + (size_t)(t0 + first) * out_stride + c;
    if (base + RS_RUNS * RS_LEN < n) fetch(base + RS_RUNS * RS_LEN);
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l)
      if (l < n_out) dst[(size_t)l * out_stride] = from_float<T>(o[l]);
  }
  if (r == 0 && cin && n > 0) *st = carry[ch];
}

// ab: [n_tokens, W] pairs (a, b) as the gates epilogue leaves them; y: [n_tokens, W] with rows y_stride apart; out likewise.
LLMRS_API int llmrs_rglru_scan(const float* ab, const void* y, long long y_stride, int dtype, const float* y_bias,
                               float* state, const int* q_start, const int* n_new, const int* slot_ids, void* out,
                               long long out_stride, int n_tokens, int n_requests, int W, cudaStream_t stream) {
  LLMRS_REQUIRE(n_tokens >= 0 && n_requests >= 0 && n_requests <= 65535 && W > 0, "rglru_scan: bad sizes");
  LLMRS_REQUIRE(((uintptr_t)ab & 7) == 0, "rglru_scan: the pairs must be 8-byte aligned");
  if (n_tokens == 0) return 0;
  dim3 grid((W + RS_CH - 1) / RS_CH, n_requests);
  // Portions of 256 tokens on average or fewer: half the runs, so that two blocks share an SM.
  const bool small = n_tokens <= 256LL * n_requests;
#define LLMRS_RS_LAUNCH(T, RUNS)                                                                                       \
  rglru_scan_kernel<T, RUNS><<<grid, RS_CH * RUNS, 0, stream>>>((const float2*)ab, (const T*)y, y_stride, y_bias, state, \
                                                                q_start, n_new, slot_ids, (T*)out, out_stride, W)
  if (dtype == LLMRS_F32) {
    if (small) LLMRS_RS_LAUNCH(float, 32); else LLMRS_RS_LAUNCH(float, 64);
  } else if (dtype == LLMRS_BF16) {
    if (small) LLMRS_RS_LAUNCH(bf16, 32); else LLMRS_RS_LAUNCH(bf16, 64);
  } else
#undef LLMRS_RS_LAUNCH
    return llmrs_fail("rglru_scan: unknown dtype %d", dtype);
  return llmrs_launch_status("rglru_scan");
}

// ---------------------------------------------------------------------------------
// step: one token per request. A block takes 32 output channels (a lane each) of a diagonal block for eight requests; its
// warps share the inputs, and what they summed meets in shared memory, where a warp per request finishes. `w` holds the
// two matrices side by side, [blocks][input][output][r, i], so that a lane's pair is one load and neighbours' are adjacent.
// ---------------------------------------------------------------------------------
constexpr int RT_TOK = 8, RT_AHEAD = 16;      // requests of a block; inputs per warp whose weights are asked for at once

template <typename TW> __device__ __forceinline__ float2 load2(const TW* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

template <typename T, typename TW, int NW>
__global__ void __launch_bounds__(32 * NW)
rglru_step_kernel(const T* __restrict__ u, const TW* __restrict__ w, const float* __restrict__ r_bias,
                  const float* __restrict__ i_bias, const float* __restrict__ rate, const T* __restrict__ y,
                  long long y_stride, const float* __restrict__ y_bias, float* __restrict__ state,
                  const int* __restrict__ slot_ids, T* __restrict__ out, long long out_stride, int n_requests, int blocks,
                  int bn) {
  extern __shared__ __align__(16) float rt_smem[];
  float* us = rt_smem;                                                  // [bn][RT_TOK]
  float2* part = reinterpret_cast<float2*>(us + (size_t)bn * RT_TOK);   // [NW][RT_TOK][32]
  const int W = blocks * bn, tiles = (bn + 31) / 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = blockIdx.x / tiles, c = (blockIdx.x % tiles) * 32 + lane, cc = blk * bn + c;
  const bool live = c < bn;
  const int r0 = blockIdx.y * RT_TOK;
  const int span = (bn + NW - 1) / NW, k_lo = warp * span, k_hi = min(bn, k_lo + span);
  const TW* wp = w + ((size_t)blk * bn * bn + (live ? c : 0)) * 2;
  // What no kernel of the step writes is read before the wait on the kernel before this one.
  float2 ahead[RT_AHEAD];
#pragma unroll
  for (int j = 0; j < RT_AHEAD; ++j)
    ahead[j] = live && k_lo + j < k_hi ? load2<TW>(wp + (size_t)(k_lo + j) * bn * 2) : make_float2(0.f, 0.f);
  const bool own = live && warp < RT_TOK && r0 + warp < n_requests;      // warp q finishes request q
  const float rb = own ? r_bias[cc] : 0.f, ib = own ? i_bias[cc] : 0.f, rt = own ? rate[cc] : 0.f;
  const float yb = own && y_bias ? y_bias[cc] : 0.f;
  pdl_launch_dependents();
  pdl_wait();
  // Every request brings one token: its row is the request's number.
  float* st = own ? state + (size_t)slot_ids[r0 + warp] * W + cc : nullptr;
  const float y_own = own ? to_float(y[(size_t)(r0 + warp) * y_stride + cc]) : 0.f;
  for (int k = warp; k < RT_TOK; k += NW) {
    const bool in = r0 + k < n_requests;
    const T* row = u + (size_t)(r0 + k) * W + (size_t)blk * bn;
    for (int e = lane; e < bn; e += 32) us[e * RT_TOK + k] = in ? to_float(row[e]) : 0.f;
  }
  const float s_own = own ? *st : 0.f;
  __syncthreads();
  float vr[RT_TOK], vi[RT_TOK];
#pragma unroll
  for (int k = 0; k < RT_TOK; ++k) vr[k] = vi[k] = 0.f;
  auto add = [&](float2 a, int k_in) {
    const float4 x0 = *reinterpret_cast<const float4*>(us + k_in * RT_TOK);
    const float4 x1 = *reinterpret_cast<const float4*>(us + k_in * RT_TOK + 4);
    const float x[RT_TOK] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
    for (int k = 0; k < RT_TOK; ++k) {
      vr[k] = fmaf(a.x, x[k], vr[k]);
      vi[k] = fmaf(a.y, x[k], vi[k]);
    }
  };
#pragma unroll
  for (int j = 0; j < RT_AHEAD; ++j)
    if (k_lo + j < k_hi) add(ahead[j], k_lo + j);
#pragma unroll 4
  for (int k_in = k_lo + RT_AHEAD; k_in < k_hi; ++k_in) add(load2<TW>(wp + (size_t)k_in * bn * 2), k_in);
#pragma unroll
  for (int k = 0; k < RT_TOK; ++k) part[(warp * RT_TOK + k) * 32 + lane] = make_float2(vr[k], vi[k]);
  __syncthreads();
  if (own) {
    float zr = rb, zi = ib;
#pragma unroll
    for (int q = 0; q < NW; ++q) {
      const float2 p = part[(q * RT_TOK + warp) * 32 + lane];
      zr += p.x;
      zi += p.y;
    }
    const float rg = 1.0f / (1.0f + expf(-zr)), ig = 1.0f / (1.0f + expf(-zi));
    const float log_a = rt * rg;
    const float S = fmaf(expf(log_a), s_own, sqrtf(-expm1f(2.0f * log_a)) * ig * us[c * RT_TOK + warp]);
    *st = S;
    out[(size_t)(r0 + warp) * out_stride + cc] = from_float<T>(S * gelu_tanh<T>(y_own + yb));
  }
}

// u: [n_requests, W] dense, one row per token of the step; w: [blocks, bn (input), bn (output), 2]; rate: [W], negative.
LLMRS_API int llmrs_rglru_step(const void* u, int dtype, const void* w, int w_dtype, const float* r_bias,
                               const float* i_bias, const float* rate, const void* y, long long y_stride,
                               const float* y_bias, float* state, const int* slot_ids, void* out, long long out_stride,
                               int n_requests, int blocks, int bn, cudaStream_t stream) {
  LLMRS_REQUIRE(n_requests >= 0 && n_requests <= RT_TOK * 65535 && blocks > 0 && bn > 0 && bn <= 1024,
                "rglru_step: bad sizes");
  LLMRS_REQUIRE(((uintptr_t)w & 7) == 0, "rglru_step: the weights must be 8-byte aligned");
  if (n_requests == 0) return 0;
  dim3 grid(blocks * ((bn + 31) / 32), (n_requests + RT_TOK - 1) / RT_TOK);
  const bool wide = bn > 8 * RT_AHEAD;      // sixteen warps then, so that a warp's weights are asked for at once up to 256
  const size_t smem = (size_t)RT_TOK * bn * sizeof(float) + (size_t)(wide ? 16 : 8) * RT_TOK * 32 * sizeof(float2);
#define LLMRS_RT_LAUNCH(T, TW, NW)                                                                                      \
  do {                                                                                                                  \
    static bool configured = false;                                                                                     \
    if (!configured) {                                                                                                  \
      const cudaError_t e = cudaFuncSetAttribute(rglru_step_kernel<T, TW, NW>,                                          \
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, 72 * 1024);               \
      if (e != cudaSuccess) return llmrs_fail("rglru_step: shared memory: %s", cudaGetErrorString(e));                  \
      configured = true;                                                                                                \
    }                                                                                                                   \
    llmrs_launch(rglru_step_kernel<T, TW, NW>, grid, dim3(32 * NW), smem, stream, true, (const T*)u, (const TW*)w, r_bias, \
                 i_bias, rate, (const T*)y, y_stride, y_bias, state, slot_ids, (T*)out, out_stride, n_requests, blocks, bn); \
  } while (0)
  if (dtype == LLMRS_F32 && w_dtype == LLMRS_F32) {
    if (wide) LLMRS_RT_LAUNCH(float, float, 16); else LLMRS_RT_LAUNCH(float, float, 8);
  } else if (dtype == LLMRS_BF16 && w_dtype == LLMRS_BF16) {
    if (wide) LLMRS_RT_LAUNCH(bf16, bf16, 16); else LLMRS_RT_LAUNCH(bf16, bf16, 8);
  } else if (dtype == LLMRS_BF16 && w_dtype == LLMRS_F32) {
    if (wide) LLMRS_RT_LAUNCH(bf16, float, 16); else LLMRS_RT_LAUNCH(bf16, float, 8);
  } else {
    return llmrs_fail("rglru_step: types %d / %d", dtype, w_dtype);
  }
#undef LLMRS_RT_LAUNCH
  return llmrs_launch_status("rglru_step");
}
