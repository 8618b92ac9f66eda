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

// x sigmoid(x) with the hardware exponential and reciprocal (a few ulp; -0 where exp(-x) overflows)
__device__ __forceinline__ float silu_fast(float x) { return x * rcp_fast(1.f + exp_fast(-x)); }

// q, f and k of one channel from the two projections u0, u1 (mode 0: with the channel's gate bias and lower bound;
// mode 1: with the head's decay).
__device__ __forceinline__ void scan_activate(int mode, float u0, float u1, float bias, float low, float decay, float& q,
                                              float& f, float& k) {
  q = silu_fast(u0);
  if (mode == 0) {
    const float z = u1 + bias, e = exp_fast(-fabsf(z));
    const float big = rcp_fast(1.f + e), small = e * big;  // sigmoid(|z|), sigmoid(-|z|)
    // the smaller of f and 1 - f comes from the small sigmoid and the other by subtraction where needed: gates that
    // are nearly open keep their distance from 1 to full precision over long products
    if (z >= 0.f) {
      k = (1.f - low) * small;
      f = 1.f - k;
    } else {
      k = (1.f - low) * big;
      f = fmaf(1.f - low, small, low);
    }
  } else {
    k = silu_fast(u1);
    f = decay;
  }
}
template <class T>
__device__ __forceinline__ void scan_channel(const ScanArgs& a, const T* row, int h, int d, float& q, float& f,
                                             float& k) {
  const int hd = h * a.D + d;
  const bool gated = a.mode == 0;
  scan_activate(a.mode, ld1(row + hd), ld1(row + a.H * a.D + hd), gated ? ld1(static_cast<const T*>(a.bias) + hd) : 0.f,
                gated ? ld1(static_cast<const T*>(a.lower) + hd) : 0.f, gated ? 0.f : a.decay[h], q, f, k);
}
// The value of a bf16 model is a bf16 number in both modes (the activated projection is rounded), so it enters tensor
// core products exactly.
__device__ __forceinline__ float round_as(float v, const float*) { return v; }
__device__ __forceinline__ float round_as(float v, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16(v)); }
template <class T>
__device__ __forceinline__ float scan_value(const ScanArgs& a, const T* row, int h, int j) {
  const float v = ld1(row + 2 * a.H * a.D + h * a.Dv + j);
  return a.mode == 0 ? v : round_as(silu_fast(v), row);
}

}  // namespace b200
