// Element types and scalar functions shared by the sequence-mixer kernels.  A kernel is templated
// on the activation / weight element T: bfloat16 (the serving form, fp32 accumulation) or float
// (every operation in fp32).  Everything else -- residual, norms, gates, states -- is fp32 in both.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace llmopt {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float as_float(float v) { return v; }
__device__ __forceinline__ float as_float(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_float<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f32(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float gelu_erf_f32(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }
__device__ __forceinline__ float gelu_tanh_f32(float z) {
  return 0.5f * z * (1.0f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
}

// Sum over a block of `threads` (a multiple of 32, at most 1024); `scratch` holds one float per warp.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const uint32_t warps = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();  // the previous use of the scratch is over
  if ((threadIdx.x & 31u) == 0u) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.0f;
  for (uint32_t w = 0; w < warps; ++w) v += scratch[w];
  return v;
}

}  // namespace llmopt
