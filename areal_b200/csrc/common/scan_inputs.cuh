// Inputs of the gated linear recurrences (gated_scan.cu): how the projection row of a token becomes q, f, k and v.
#pragma once
#include "io.cuh"

namespace b200 {

struct ScanArgs {
  const void* x;       // [T, row] projections, pitch ldx
  long long ldx;
  const void* bias;    // mode 0: [H * D] gate bias (model dtype)
  const void* lower;   // mode 0: [H * D] lower bound of the gate (model dtype)
  const float* decay;  // mode 1: [H]
  const int* cu;       // prefill: [n_seq + 1]
  const int* slots;    // [n_seq] state slot of every sequence (negative: keep nothing)
  float* state;        // [n_slots, H, D, Dv]
  float* o;            // [T, H, Dv] fp32
  int H, D, Dv, mode;
};

// x sigmoid(x): bf16 models take the hardware exponential and reciprocal (a few ulp; -0 where exp(-x) overflows), 32-bit
// models the library's.
__device__ __forceinline__ float silu_fast(float x) { return x * rcp_fast(1.f + exp_fast(-x)); }
__device__ __forceinline__ float silu_as(float x, const __nv_bfloat16*) { return silu_fast(x); }
__device__ __forceinline__ float silu_as(float x, const float*) { return x / (1.f + expf(-x)); }
// sigmoid(|z|) and sigmoid(-|z|)
__device__ __forceinline__ float2 sigmoid_pair(float z, const __nv_bfloat16*) {
  const float e = exp_fast(-fabsf(z)), big = rcp_fast(1.f + e);
  return make_float2(big, e * big);
}
__device__ __forceinline__ float2 sigmoid_pair(float z, const float*) {
  const float e = expf(-fabsf(z));
  return make_float2(1.f / (1.f + e), e / (1.f + e));
}

// q, f and k of one channel from the two projections u0, u1 (mode 0: with the channel's gate bias and lower bound;
// mode 1: with the head's decay).
template <class T>
__device__ __forceinline__ void scan_activate(const T* tag, int mode, float u0, float u1, float bias, float low,
                                              float decay, float& q, float& f, float& k) {
  q = silu_as(u0, tag);
  if (mode == 0) {
    const float z = u1 + bias;
    const float2 s = sigmoid_pair(z, tag);
    // the smaller of f and 1 - f comes from the small sigmoid and the other by subtraction where needed: gates that
    // are nearly open keep their distance from 1 to full precision over long products
    if (z >= 0.f) {
      k = (1.f - low) * s.y;
      f = 1.f - k;
    } else {
      k = (1.f - low) * s.x;
      f = fmaf(1.f - low, s.y, low);
    }
  } else {
    k = silu_as(u1, tag);
    f = decay;
  }
}
template <class T>
__device__ __forceinline__ void scan_channel(const ScanArgs& a, const T* row, int h, int d, float& q, float& f,
                                             float& k) {
  const int hd = h * a.D + d;
  const bool gated = a.mode == 0;
  scan_activate(row, a.mode, ld1(row + hd), ld1(row + a.H * a.D + hd), gated ? ld1(static_cast<const T*>(a.bias) + hd) : 0.f,
                gated ? ld1(static_cast<const T*>(a.lower) + hd) : 0.f, gated ? 0.f : a.decay[h], q, f, k);
}
// The value of a bf16 model is a bf16 number in both modes (the activated projection is rounded), so it enters tensor
// core products exactly.
__device__ __forceinline__ float round_as(float v, const float*) { return v; }
__device__ __forceinline__ float round_as(float v, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16(v)); }
template <class T>
__device__ __forceinline__ float scan_value(const ScanArgs& a, const T* row, int h, int j) {
  const float v = ld1(row + 2 * a.H * a.D + h * a.Dv + j);
  return a.mode == 0 ? v : round_as(silu_as(v, row), row);
}

}  // namespace b200
