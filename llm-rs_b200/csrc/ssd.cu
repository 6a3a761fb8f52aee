// State-space duality (Mamba-2): the parts around the recurrence, which is the linear recurrence on float32 planes of
// linear_recurrence.cu with keys B, queries C (shared by groups of heads), values x, a decay per (token, head), the step
// size as the value's gain and a skip D:
//
//   S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T,     y_t = S_t^T C_t + D_h x_t,     dt = softplus(raw + dt_bias_h)
//
//   prepare   a block per token: x | B | C through a short causal convolution per channel with a bias, and SiLU; the
//             step size and the decay; all as float32 planes. Then the convolution's last inputs become its state.
//   output    a block per token: y * SiLU(z), each of `parts` equal pieces divided by its own root mean square, times a
//             weight and a fixed scale, rounded once to the activation type.
#include "common.cuh"
#include "short_conv.cuh"

template <typename TA>
__global__ void ssd_prepare_kernel(const TA* __restrict__ xbc, long long stride, const TA* __restrict__ dt_raw,
                                   long long dt_stride, const float* __restrict__ taps, const float* __restrict__ bias,
                                   const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                                   const float* __restrict__ conv_state, const int* __restrict__ token_req,
                                   const int* __restrict__ q_start, const int* __restrict__ slot_ids,
                                   float* __restrict__ X, float* __restrict__ B, float* __restrict__ Cq,
                                   float* __restrict__ decay, float* __restrict__ step, int inner, int wk, int H, int K) {
  const int t = blockIdx.x, req = token_req[t], off = t - q_start[req], C = inner + 2 * wk;
  const float* tail = conv_state + (size_t)slot_ids[req] * (K - 1) * C;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
    const float v = rec_silu(short_conv_at(xbc, stride, t, off, c, taps + (size_t)c * K, K, tail, C, bias[c]));
    if (c < inner) X[(size_t)t * inner + c] = v;
    else if (c < inner + wk) B[(size_t)t * wk + c - inner] = v;
    else Cq[(size_t)t * wk + c - inner - wk] = v;
  }
  if (blockIdx.y != 0) return;
  for (int h = threadIdx.x; h < H; h += blockDim.x) {
    const float dt = rec_softplus(to_float(dt_raw[(size_t)t * dt_stride + h]) + dt_bias[h]);
    step[(size_t)t * H + h] = dt;
    decay[(size_t)t * H + h] = expf(-expf(a_log[h]) * dt);
  }
}

// xbc: [tokens, inner + 2 * groups * state] of `dtype`, rows `stride` apart; dt_raw: [tokens, H] likewise; taps: float32
// [channels, K], bias [channels]; conv_state: float32 [slots, K - 1, channels]; X [tokens, inner], B and Cq [tokens,
// groups * state], decay and step [tokens, H]: float32.
LLMRS_API int llmrs_ssd_prepare(const void* xbc, long long stride, const void* dt_raw, long long dt_stride, int dtype,
                                const float* taps, const float* bias, const float* dt_bias, const float* a_log,
                                float* conv_state, const int* token_req, const int* q_start, const int* n_new,
                                const int* slot_ids, float* X, float* B, float* Cq, float* decay, float* step,
                                int n_tokens, int n_requests, int inner, int groups, int state, int H, int K,
                                cudaStream_t stream) {
  LLMRS_REQUIRE(n_tokens >= 0 && n_requests >= 0 && inner > 0 && groups > 0 && state > 0 && H > 0 && K >= 1,
                "ssd_prepare: bad sizes");
  if (n_tokens == 0 || n_requests == 0) return 0;
  const int wk = groups * state, C = inner + 2 * wk, slices = C > 2048 && n_tokens < 148 ? (C + 2047) / 2048 : 1;
#define LLMRS_SSD_PREPARE(T)                                                                                        \
  do {                                                                                                              \
    ssd_prepare_kernel<T><<<dim3(n_tokens, slices), 256, 0, stream>>>(                                              \
        (const T*)xbc, stride, (const T*)dt_raw, dt_stride, taps, bias, dt_bias, a_log, conv_state, token_req,      \
        q_start, slot_ids, X, B, Cq, decay, step, inner, wk, H, K);                                                 \
    int rc = llmrs_launch_status("ssd_prepare");                                                                    \
    if (rc != 0) return rc;                                                                                         \
    return launch_short_conv_state((const T*)xbc, stride, conv_state, q_start, n_new, slot_ids, n_requests, C, K, stream); \
  } while (0)
  if (dtype == LLMRS_F32) LLMRS_SSD_PREPARE(float);
  if (dtype == LLMRS_BF16) LLMRS_SSD_PREPARE(__nv_bfloat16);
#undef LLMRS_SSD_PREPARE
  return llmrs_fail("ssd_prepare: unknown dtype %d", dtype);
}

template <typename TA>
__global__ void ssd_output_kernel(const float* __restrict__ y, const TA* __restrict__ z, long long z_stride,
                                  const float* __restrict__ norm_w, TA* __restrict__ out, long long out_stride, int inner,
                                  int parts, float eps, float out_scale) {
  extern __shared__ float sh[];      // [inner] the gated row, [parts] 1 / root mean square
  float* row = sh;
  float* inv = sh + inner;
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5, w = inner / parts;
  for (int c = threadIdx.x; c < inner; c += blockDim.x)
    row[c] = y[(size_t)t * inner + c] * rec_silu(to_float(z[(size_t)t * z_stride + c]));
  __syncthreads();
  if (parts >= n_warps) {      // a warp per part
    for (int p = warp; p < parts; p += n_warps) {
      float ss = 0.f;
      for (int i = lane; i < w; i += 32) ss = fmaf(row[p * w + i], row[p * w + i], ss);
      ss = warp_sum(ss);
      if (lane == 0) inv[p] = 1.0f / sqrtf(ss / (float)w + eps);
    }
  } else {                     // few wide parts: the whole block on each
    __shared__ float red[33];
    for (int p = 0; p < parts; ++p) {
      float ss = 0.f;
      for (int i = threadIdx.x; i < w; i += blockDim.x) ss = fmaf(row[p * w + i], row[p * w + i], ss);
      ss = block_sum(ss, red);
      if (threadIdx.x == 0) inv[p] = 1.0f / sqrtf(ss / (float)w + eps);
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < inner; c += blockDim.x)
    out[(size_t)t * out_stride + c] = from_float<TA>(row[c] * inv[c / w] * norm_w[c] * out_scale);
}

// y: float32 [tokens, inner]; z: [tokens, inner] of `dtype` rows `z_stride` apart; out likewise; norm_w: float32 [inner].
LLMRS_API int llmrs_ssd_output(const float* y, const void* z, long long z_stride, int dtype, const float* norm_w, void* out,
                               long long out_stride, int n_tokens, int inner, int parts, float eps, float out_scale,
                               cudaStream_t stream) {
  LLMRS_REQUIRE(n_tokens >= 0 && inner > 0 && parts > 0 && inner % parts == 0,
                "ssd_output: %d channels in %d parts", inner, parts);
  if (n_tokens == 0) return 0;
  const size_t smem = (size_t)(inner + parts) * sizeof(float);
  LLMRS_REQUIRE(smem <= 160 * 1024, "ssd_output: rows of %d channels are too wide", inner);
  const int threads = inner >= 2048 ? 512 : (inner >= 512 ? 256 : 128);
#define LLMRS_SSD_OUTPUT(T)                                                                                            \
  do {                                                                                                                 \
    static size_t configured = 48 * 1024;                                                                              \
    if (smem > configured) {                                                                                           \
      cudaError_t e = cudaFuncSetAttribute(ssd_output_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (e != cudaSuccess) return llmrs_fail("ssd_output: shared memory %zu: %s", smem, cudaGetErrorString(e));       \
      configured = smem;                                                                                               \
    }                                                                                                                  \
    ssd_output_kernel<T><<<n_tokens, threads, smem, stream>>>(y, (const T*)z, z_stride, norm_w, (T*)out, out_stride,   \
                                                              inner, parts, eps, out_scale);                           \
  } while (0)
  if (dtype == LLMRS_F32) LLMRS_SSD_OUTPUT(float);
  else if (dtype == LLMRS_BF16) LLMRS_SSD_OUTPUT(__nv_bfloat16);
  else return llmrs_fail("ssd_output: unknown dtype %d", dtype);
#undef LLMRS_SSD_OUTPUT
  return llmrs_launch_status("ssd_output");
}
