// Scalar and 4-wide loads / stores of bf16 or fp32 tensors as fp32 values, for kernels that are templates over the
// model's dtype and compute in fp32 either way.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace b200 {

__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ float ld1(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<uint32_t*>(&a);
  raw.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the block; every thread gets it. `red`: 33 floats of shared memory. Two barriers.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];
  return t;
}

// 2^x and 1/x by the hardware approximations, denormals flushed (no range-scaling instructions around them)
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float exp_fast(float x) { return ex2_fast(x * 1.4426950408889634f); }

// tanh for results in the given dtype: fp32 gets the library function; for bf16 results 1 - 2 / (1 + e^2x), whose absolute
// error (about 1e-7 of the range) is far below the result's rounding.
__device__ __forceinline__ float tanh_as(float x, const float*) { return tanhf(x); }
__device__ __forceinline__ float tanh_as(float x, const __nv_bfloat16*) {
  return 1.f - 2.f * rcp_fast(1.f + exp_fast(2.f * x));
}

__device__ __forceinline__ float sigmoid_as(float x, const float*) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_as(float x, const __nv_bfloat16*) { return rcp_fast(1.f + exp_fast(-x)); }

// Gated activation g' * sigmoid(alpha * g') * (u' + beta) with g' = min(g, limit) and u' clamped to [-limit, limit]
// (limit: infinity for none). SwiGLU is alpha 1, beta 0. The pointer names the result's dtype.
struct GluParams {
  float limit, alpha, beta;
};
template <class T>
__device__ __forceinline__ float glu_act(float g, float u, GluParams p, const T*) {
  g = fminf(g, p.limit);
  u = fminf(fmaxf(u, -p.limit), p.limit);
  return g * sigmoid_as(p.alpha * g, static_cast<const T*>(nullptr)) * (u + p.beta);
}
__device__ __forceinline__ float glu_act(float g, float u, GluParams p, const __nv_bfloat162*) {
  return glu_act(g, u, p, static_cast<const __nv_bfloat16*>(nullptr));
}

}  // namespace b200
