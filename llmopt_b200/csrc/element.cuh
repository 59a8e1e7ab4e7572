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

// tanh from its definition, 1 - 2 / (e^2u + 1), and near zero, where that cancels, from its Taylor series
// (next term 17 u^7 / 315): absolute error about 1e-7, relative about 1e-6.
__device__ __forceinline__ float tanh_f32(float u) {
  const float far = 1.0f - __fdividef(2.0f, __expf(2.0f * u) + 1.0f);
  const float square = u * u;
  const float near = u * fmaf(square, fmaf(square, 0.13333333f, -0.33333333f), 1.0f);
  return fabsf(u) < 0.1f ? near : far;
}

// "Dynamic tanh" in the place of a norm: tanh(alpha x) w + b per column; `norm` holds w [width], b [width], alpha.
struct TanhNorm {
  const float* w;
  const float* b;
  float alpha;
  __device__ __forceinline__ TanhNorm(const float* norm, uint32_t width)
      : w(norm), b(norm + width), alpha(__ldg(norm + 2 * (size_t)width)) {}
  __device__ __forceinline__ float operator()(float x, uint32_t column) const {
    return fmaf(tanh_f32(alpha * x), __ldg(w + column), __ldg(b + column));
  }
  __device__ __forceinline__ float4 four(const float4& x, uint32_t column) const {  // column, width: multiples of four
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w + column)), bv = __ldg(reinterpret_cast<const float4*>(b + column));
    return make_float4(fmaf(tanh_f32(alpha * x.x), wv.x, bv.x), fmaf(tanh_f32(alpha * x.y), wv.y, bv.y),
                       fmaf(tanh_f32(alpha * x.z), wv.z, bv.z), fmaf(tanh_f32(alpha * x.w), wv.w, bv.w));
  }
  // (w + b) - 2 w / (e^(2 alpha x) + 1) in a few instructions: the absolute error is that of fp32 at |w| + |b|, but a small
  // tanh keeps fewer of its own digits.
  __device__ __forceinline__ float4 four_short(const float4& x, uint32_t column) const {
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w + column)), bv = __ldg(reinterpret_cast<const float4*>(b + column));
    const float rate = alpha * 2.8853900817779268f;  // 2 log2 e
    auto one = [&](float v, float weight, float bias) {
      float power;
      asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(power) : "f"(rate * v));
      return fmaf(-2.0f * weight, __fdividef(1.0f, power + 1.0f), weight + bias);
    };
    return make_float4(one(x.x, wv.x, bv.x), one(x.y, wv.y, bv.y), one(x.z, wv.z, bv.z), one(x.w, wv.w, bv.w));
  }
};

// Four values to consecutive elements (16- or 8-byte aligned).
__device__ __forceinline__ void store_four(float* target, const float4& v) { *reinterpret_cast<float4*>(target) = v; }
__device__ __forceinline__ void store_four(bf16* target, const float4& v) {
  const __nv_bfloat162 low = __floats2bfloat162_rn(v.x, v.y), high = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(target) =
      make_uint2(*reinterpret_cast<const uint32_t*>(&low), *reinterpret_cast<const uint32_t*>(&high));
}

// Larger values first, then smaller columns, as one unsigned integer.
__device__ __forceinline__ unsigned long long ranked(float value, uint32_t column) {
  uint32_t bits = __float_as_uint(value + 0.0f);  // both zeros are equal
  bits = (bits & 0x80000000u) ? ~bits : bits | 0x80000000u;
  return ((unsigned long long)bits << 32) | (0xffffffffu - column);
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
