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

// eight at a time (16 bytes of bf16, 32 of fp32)
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = load4(p), b = load4(p + 4);
  f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = b.x, f[5] = b.y, f[6] = b.z, f[7] = b.w;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  f[0] = bf16_lo(v.x), f[1] = bf16_hi(v.x), f[2] = bf16_lo(v.y), f[3] = bf16_hi(v.y);
  f[4] = bf16_lo(v.z), f[5] = bf16_hi(v.z), f[6] = bf16_lo(v.w), f[7] = bf16_hi(v.w);
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  store4(p, make_float4(f[0], f[1], f[2], f[3]));
  store4(p + 4, make_float4(f[4], f[5], f[6], f[7]));
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}

// 8 raw elements as they come
template <typename E>
struct Raw8 {
  uint4 v[sizeof(E) / 2];
  __device__ __forceinline__ void load(const E* p) {
#pragma unroll
    for (int i = 0; i < static_cast<int>(sizeof(E) / 2); ++i) v[i] = reinterpret_cast<const uint4*>(p)[i];
  }
  __device__ __forceinline__ void get(float (&f)[8]) const { load8(reinterpret_cast<const E*>(&v[0]), f); }
};

__device__ __forceinline__ float rcp_fast(float x) {  // 1 / x, one hardware instruction (about an ulp; 1 / inf = 0)
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// packed fp32 pairs
struct F2 {
  uint64_t v;
};
__device__ __forceinline__ F2 f2(float lo, float hi) {
  F2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r.v) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unf2(F2 a) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(a.v));
  return r;
}
__device__ __forceinline__ F2 mul2(F2 a, F2 b) {
  F2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) {
  F2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return r;
}
__device__ __forceinline__ F2 add2(F2 a, F2 b) {
  F2 r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
  return r;
}

// Logistic function in fp32: exact library exponential and division for fp32 activations, the hardware exponential and
// reciprocal (a few fp32 ulp) next to bf16 ones.
template <typename E>
__device__ __forceinline__ float sigmoid_f(float x);
template <>
__device__ __forceinline__ float sigmoid_f<float>(float x) { return 1.0f / (1.0f + expf(-x)); }
template <>
__device__ __forceinline__ float sigmoid_f<__nv_bfloat16>(float x) { return rcp_fast(1.0f + ex2_fast(-1.4426950408889634f * x)); }
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
