// Helpers of the layered-decoder kernels: typed loads and stores of activations (fp32 or bf16), block reductions,
// the two norms' statistics, sigmoid and log-sigmoid.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>

#include "nb_host.h"
#include "nb_launch.cuh"
#include "../../include/nativebit_b200_layered.h"

namespace nb {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// The two bf16 halves of a 32-bit word as floats (element 0 in the low half).
__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
// log(sigmoid(z)) without overflow on either side
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// Gated pair behind a product: silu(g) * u, or the clamped form.
__device__ __forceinline__ float glu_f(int act, float alpha, float limit, float g, float u) {
  if (act == NB_ACT_CLAMPED_GLU_PAIRS) {
    g = fminf(g, limit);
    return g * sigmoid_f(alpha * g) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
  }
  return silu_f(g) * u;
}

// Sum over the block; `red` has one float per warp and is used by this call only (no barrier protects it afterwards).
template <int kWarps> __device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kWarps; ++i) t += red[i];
  return t;
}

// Mean to take off and factor of a row whose elements each thread visits through `each(f)`: f(value).
// red: 2 * kWarps floats.
template <int kWarps, typename Each>
__device__ __forceinline__ void norm_stats(int kind, int C, float eps, float* red, Each each, float& mean, float& inv) {
  mean = 0.f;
  if (kind == NB_NORM_LAYER) {
    float s = 0.f;
    each([&](float v) { s += v; });
    mean = block_sum<kWarps>(s, red) / (float)C;
  }
  float q = 0.f;
  const float m = mean;
  each([&](float v) { const float d = v - m; q += d * d; });
  inv = 1.0f / sqrtf(block_sum<kWarps>(q, red + kWarps) / (float)C + eps);
}

}  // namespace nb
