// Element-type helpers of the kernels that exist for bf16 and for fp32 activations (E = __nv_bfloat16 or float):
// four consecutive elements at a time, fp32 values in registers either way.
#pragma once
#include "common.cuh"

namespace b200 {

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ float load1(const float* p) { return *p; }
__device__ __forceinline__ float load1(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void store1(float* p, float v) { *p = v; }
__device__ __forceinline__ void store1(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Logistic function in fp32: exact library exponential and division for fp32 activations, the hardware exponential and
// reciprocal (a few fp32 ulp) next to bf16 ones.
template <typename E>
__device__ __forceinline__ float sigmoid_f(float x);
template <>
__device__ __forceinline__ float sigmoid_f<float>(float x) { return 1.0f / (1.0f + expf(-x)); }
template <>
__device__ __forceinline__ float sigmoid_f<__nv_bfloat16>(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
template <typename E>
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f<E>(x); }

// Sum over the block of N values at once; `red` holds N * 32 floats.  Every thread gets the sums.
template <int N>
__device__ __forceinline__ void block_sum(float (&v)[N], float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(v[i]);
  if (warps == 1) return;
  if (lane == 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) red[i * 32 + warp] = v[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = warp_sum(lane < warps ? red[i * 32 + lane] : 0.f);
}

}  // namespace b200
