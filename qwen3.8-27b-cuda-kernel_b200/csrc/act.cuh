// Activation precision of the dense-weight kernels: every kernel is written once over T = __nv_bfloat16 or float.
#pragma once

#include "common.cuh"

namespace q38 {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// 0.5 x (1 + tanh(sqrt(2 / pi) (x + 0.044715 x^3)))
__device__ __forceinline__ float gelu_tanh_f(float x) {
  const float u = 0.7978845608028654f * (x + 0.044715f * x * x * x);
  return 0.5f * x * (1.0f + tanhf(u));
}
// alpha_p z^2 + z / 2 above zero, alpha_n (e^z - 1 - z) + z / 2 below
__device__ __forceinline__ float xielu_f(float z, float alpha_p, float alpha_n) {
  return (z > 0.0f ? alpha_p * z * z : alpha_n * (expm1f(z) - z)) + 0.5f * z;
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// The A fragments of two k16 steps of mma.m16n8k16 from 16 contiguous bytes of rows g and g + 8. An MMA takes its four A
// registers as one aligned group, and the compiler would regroup the loaded registers anew for every MMA that uses the
// fragment; the OR with a zero it cannot see (blocks here have one layer in z) makes the group a value of its own.
struct AFragPair {
  uint32_t f0[4], f1[4];
};
__device__ __forceinline__ uint32_t pinned(uint32_t x) { return x | (blockDim.z - 1u); }
__device__ __forceinline__ AFragPair a_fragments(const uint4& r0, const uint4& r8) {
  return {{pinned(r0.x), pinned(r8.x), pinned(r0.y), pinned(r8.y)}, {pinned(r0.z), pinned(r8.z), pinned(r0.w), pinned(r8.w)}};
}
// ... against 16 contiguous bytes of a row of B
__device__ __forceinline__ void mma_pair(float (&d)[4], const AFragPair& a, const uint4& b) {
  mma_bf16_16816(d, a.f0, b.x, b.y);
  mma_bf16_16816(d, a.f1, b.z, b.w);
}

// Sum over the CTA's threads (a multiple of 32, at most 1024); every thread gets the result. `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  v = warp_sum(v);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < warps ? red[lane] : 0.0f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  const float r = red[32];
  __syncthreads();
  return r;
}

}  // namespace q38
