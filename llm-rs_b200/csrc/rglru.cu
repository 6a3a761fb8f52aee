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
//   scan  the recurrence is an associative composition of affine maps, so a block takes 16 channels of a request and 64
//         runs of up to 8 tokens side by side: every thread composes its run's maps from registers, a warp per channel
//         composes the runs and turns them into start states, and every thread walks its run again. 512 tokens a turn,
//         the state carried from turn to turn.
//   step  one token per request (decoding): products, gates, recurrence and output in one kernel: a warp takes one output
//         channel of one diagonal block at a time for eight requests, its lanes split the block's inputs.
// Everything but x, u, y and the output (activation type) is float32.
#include "common.cuh"
#include "short_conv.cuh"

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z)));
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

template <typename T>
static int launch_short_conv(const void* x, long long stride, const float* x_bias, const float* taps, const float* bias,
                             float* conv_state, const int* token_req, const int* q_start, const int* n_new,
                             const int* slot_ids, void* u, int n_tokens, int n_requests, int W, int K, int single,
                             cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = W % V == 0 && stride % V == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)u & 15) == 0;
  const int per = vec ? W / V : W, threads = per >= 128 ? 128 : ((per + 31) / 32) * 32;
  dim3 grid(n_tokens, (per + threads - 1) / threads);
  if (vec)
    short_conv_kernel<T, V><<<grid, threads, 0, stream>>>((const T*)x, stride, x_bias, taps, bias, conv_state, token_req,
                                                          q_start, slot_ids, (T*)u, W, K, single);
  else
    short_conv_kernel<T, 1><<<grid, threads, 0, stream>>>((const T*)x, stride, x_bias, taps, bias, conv_state, token_req,
                                                          q_start, slot_ids, (T*)u, W, K, single);
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
constexpr int RS_CH = 16, RS_RUNS = 64, RS_LEN = 8, RS_THREADS = RS_CH * RS_RUNS;

template <typename T>
__global__ void __launch_bounds__(RS_THREADS)
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
  for (int base = 0; base < n; base += RS_RUNS * RS_LEN) {
    const int per = min(RS_LEN, (n - base + RS_RUNS - 1) / RS_RUNS);      // short portions: shorter runs
    const int first = base + r * per;
    const int len = cin ? max(0, min(per, n - first)) : 0;
    float2 v[RS_LEN];
    float yv[RS_LEN];
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) v[l] = l < len ? ab[(size_t)(t0 + first + l) * W + c] : make_float2(1.f, 0.f);
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) yv[l] = l < len ? to_float(y[(size_t)(t0 + first + l) * y_stride + c]) : 0.f;
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) {
      A *= v[l].x;
      B = fmaf(v[l].x, B, v[l].y);
    }
    run[ch][r] = make_float2(A, B);
    __syncthreads();
    if (warp < RS_CH) {
      // Lane l holds runs 2 l and 2 l + 1 of channel `warp`; an inclusive scan of the pairs' maps over the lanes.
      const float2 p0 = run[warp][2 * lane], p1 = run[warp][2 * lane + 1];
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
      run[warp][2 * lane].x = first_state;
      run[warp][2 * lane + 1].x = fmaf(p0.x, first_state, p0.y);
      __syncwarp();
      if (lane == 31) carry[warp] = fmaf(a, s0, b);
    }
    __syncthreads();
    float S = run[ch][r].x;
#pragma unroll
    for (int l = 0; l < RS_LEN; ++l) {
      S = fmaf(v[l].x, S, v[l].y);
      if (l < len) out[(size_t)(t0 + first + l) * out_stride + c] = from_float<T>(S * gelu_tanh(yv[l] + yb));
    }
    __syncthreads();      // the runs' start states are read before the next turn overwrites them
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
  if (dtype == LLMRS_F32)
    rglru_scan_kernel<float><<<grid, RS_THREADS, 0, stream>>>((const float2*)ab, (const float*)y, y_stride, y_bias, state,
                                                              q_start, n_new, slot_ids, (float*)out, out_stride, W);
  else if (dtype == LLMRS_BF16)
    rglru_scan_kernel<bf16><<<grid, RS_THREADS, 0, stream>>>((const float2*)ab, (const bf16*)y, y_stride, y_bias, state,
                                                             q_start, n_new, slot_ids, (bf16*)out, out_stride, W);
  else
    return llmrs_fail("rglru_scan: unknown dtype %d", dtype);
  return llmrs_launch_status("rglru_scan");
}

// ---------------------------------------------------------------------------------
// step: one token per request
// ---------------------------------------------------------------------------------
constexpr int RT_TOK = 8, RT_WARPS = 4, RT_CH = 16;      // requests, warps and output channels of a block

template <typename TW> __device__ __forceinline__ float2 load2(const TW* p);
template <> __device__ __forceinline__ float2 load2<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 load2<bf16>(const bf16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

// PAIR: a diagonal block has an even number of inputs, which the lanes take two at a time.
template <typename T, typename TW, bool PAIR>
__global__ void __launch_bounds__(32 * RT_WARPS)
rglru_step_kernel(const T* __restrict__ u, const TW* __restrict__ wr, const TW* __restrict__ wi,
                  const float* __restrict__ r_bias, const float* __restrict__ i_bias, const float* __restrict__ rate,
                  const T* __restrict__ y, long long y_stride, const float* __restrict__ y_bias,
                  float* __restrict__ state, const int* __restrict__ q_start, const int* __restrict__ slot_ids,
                  T* __restrict__ out, long long out_stride, int n_requests, int blocks, int bn) {
  extern __shared__ __align__(16) float us[];      // [RT_TOK][bn]
  const int W = blocks * bn, tiles = (bn + RT_CH - 1) / RT_CH;
  const int blk = blockIdx.x / tiles, c_lo = (blockIdx.x % tiles) * RT_CH, c_hi = min(bn, c_lo + RT_CH);
  const int r0 = blockIdx.y * RT_TOK, nt = min(RT_TOK, n_requests - r0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < RT_TOK * bn; i += blockDim.x) {
    const int k = i / bn, e = i - k * bn;
    us[i] = k < nt ? to_float(u[(size_t)q_start[r0 + k] * W + (size_t)blk * bn + e]) : 0.f;
  }
  __syncthreads();
  for (int c = c_lo + warp; c < c_hi; c += RT_WARPS) {
    const TW* pr = wr + ((size_t)blk * bn + c) * bn;
    const TW* pi = wi + ((size_t)blk * bn + c) * bn;
    float v[2 * RT_TOK];      // [request][r, i]
#pragma unroll
    for (int k = 0; k < 2 * RT_TOK; ++k) v[k] = 0.f;
    if (PAIR) {
#pragma unroll 4
      for (int e = 2 * lane; e < bn; e += 64) {
        const float2 a = load2<TW>(pr + e), b = load2<TW>(pi + e);
#pragma unroll
        for (int k = 0; k < RT_TOK; ++k) {
          const float2 x = *reinterpret_cast<const float2*>(us + k * bn + e);
          v[2 * k] = fmaf(a.y, x.y, fmaf(a.x, x.x, v[2 * k]));
          v[2 * k + 1] = fmaf(b.y, x.y, fmaf(b.x, x.x, v[2 * k + 1]));
        }
      }
    } else {
      for (int e = lane; e < bn; e += 32) {
        const float a = to_float(pr[e]), b = to_float(pi[e]);
#pragma unroll
        for (int k = 0; k < RT_TOK; ++k) {
          v[2 * k] = fmaf(a, us[k * bn + e], v[2 * k]);
          v[2 * k + 1] = fmaf(b, us[k * bn + e], v[2 * k + 1]);
        }
      }
    }
    // Sixteen sums over the warp in sixteen shuffles: at every distance a lane keeps half of its numbers. In the end
    // lane l holds number l / 2: request l / 4, r or i by bit 1.
#pragma unroll
    for (int o = 16, m = RT_TOK; m >= 1; o >>= 1, m >>= 1) {
#pragma unroll
      for (int k = 0; k < m; ++k) {
        const bool upper = lane & o;
        const float give = upper ? v[k] : v[k + m], keep = upper ? v[k + m] : v[k];
        v[k] = keep + __shfl_xor_sync(0xffffffffu, give, o);
      }
    }
    const float sum = v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
    const float sum_i = __shfl_down_sync(0xffffffffu, sum, 2);
    const int k = lane >> 2;
    if ((lane & 3) == 0 && k < nt) {
      const int req = r0 + k, t = q_start[req], cc = blk * bn + c;
      const float rg = 1.0f / (1.0f + expf(-(sum + r_bias[cc]))), ig = 1.0f / (1.0f + expf(-(sum_i + i_bias[cc])));
      const float log_a = rate[cc] * rg;
      float* st = state + (size_t)slot_ids[req] * W + cc;
      const float S = fmaf(expf(log_a), *st, sqrtf(-expm1f(2.0f * log_a)) * ig * us[k * bn + c]);
      *st = S;
      const float yv = to_float(y[(size_t)t * y_stride + cc]) + (y_bias ? y_bias[cc] : 0.f);
      out[(size_t)t * out_stride + cc] = from_float<T>(S * gelu_tanh(yv));
    }
  }
}

// u: [n_requests, W] dense, one row per token of the step; wr, wi: [blocks, bn, bn]; rate: [W], negative.
LLMRS_API int llmrs_rglru_step(const void* u, int dtype, const void* wr, const void* wi, int w_dtype, const float* r_bias,
                               const float* i_bias, const float* rate, const void* y, long long y_stride,
                               const float* y_bias, float* state, const int* q_start, const int* slot_ids, void* out,
                               long long out_stride, int n_requests, int blocks, int bn, cudaStream_t stream) {
  LLMRS_REQUIRE(n_requests >= 0 && n_requests <= 8 * 65535 && blocks > 0 && bn > 0 && bn <= 1024, "rglru_step: bad sizes");
  if (n_requests == 0) return 0;
  dim3 grid(blocks * ((bn + RT_CH - 1) / RT_CH), (n_requests + RT_TOK - 1) / RT_TOK);
  const size_t smem = (size_t)RT_TOK * bn * sizeof(float);
  const bool pair = bn % 2 == 0 && ((uintptr_t)wr & 7) == 0 && ((uintptr_t)wi & 7) == 0;
#define LLMRS_RT_LAUNCH(T, TW, P)                                                                                     \
  rglru_step_kernel<T, TW, P><<<grid, 32 * RT_WARPS, smem, stream>>>(                                                 \
      (const T*)u, (const TW*)wr, (const TW*)wi, r_bias, i_bias, rate, (const T*)y, y_stride, y_bias, state, q_start, \
      slot_ids, (T*)out, out_stride, n_requests, blocks, bn)
  if (dtype == LLMRS_F32 && w_dtype == LLMRS_F32) {
    if (pair) LLMRS_RT_LAUNCH(float, float, true); else LLMRS_RT_LAUNCH(float, float, false);
  } else if (dtype == LLMRS_BF16 && w_dtype == LLMRS_BF16) {
    if (pair) LLMRS_RT_LAUNCH(bf16, bf16, true); else LLMRS_RT_LAUNCH(bf16, bf16, false);
  } else if (dtype == LLMRS_BF16 && w_dtype == LLMRS_F32) {
    if (pair) LLMRS_RT_LAUNCH(bf16, float, true); else LLMRS_RT_LAUNCH(bf16, float, false);
  } else {
    return llmrs_fail("rglru_step: types %d / %d", dtype, w_dtype);
  }
#undef LLMRS_RT_LAUNCH
  return llmrs_launch_status("rglru_step");
}
