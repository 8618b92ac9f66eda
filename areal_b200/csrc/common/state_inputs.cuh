// Inputs of the recurrences with one matrix state and one decay per head (matrix_state.cu, matrix_state_chunk.cu).
#pragma once
#include "io.cuh"

namespace b200 {

struct StateArgs {
  const void* qkv;       // [T][ldq]: q, k (G * D each) | v (H * Dv)
  long long ldq;
  const void *g0, *g1;   // [T][ldx], one number per head: b and a of the delta rule, i and f of mLSTM
  long long ldx;
  const void *p0, *p1;   // [H]: A_log and dt_bias, or the biases of i and f
  float cap;             // mLSTM: the cap of i and f
  int delta;
  int H, G, D, Dv;
};

__device__ __forceinline__ float softplusf(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// Of one token and head: the logarithm of the decay, and the write strength (delta rule) or the log input gate (mLSTM).
template <class T>
__device__ __forceinline__ void head_gates(const StateArgs& a, long long row, int h, float& log_decay, float& write) {
  const float x0 = ld1(static_cast<const T*>(a.g0) + row * a.ldx + h), x1 = ld1(static_cast<const T*>(a.g1) + row * a.ldx + h);
  const float p0 = ld1(static_cast<const T*>(a.p0) + h), p1 = ld1(static_cast<const T*>(a.p1) + h);
  if (a.delta) {
    write = 1.f / (1.f + expf(-x0));
    log_decay = -expf(p0) * softplusf(x1 + p1);
  } else {
    write = a.cap * tanhf((x0 + p0) / a.cap);
    log_decay = -softplusf(-a.cap * tanhf((x1 + p1) / a.cap));
  }
}

// What the output gate multiplies by: silu (delta rule) or sigmoid (mLSTM).
template <class T>
__device__ __forceinline__ float out_gate(float x, int delta, const T* tag) {
  return sigmoid_as(x, tag) * (delta ? x : 1.f);
}

}  // namespace b200
