// Short causal convolutions over time, one filter per channel, of packed sequences:
//
//   y_t = act(sum_j w[c][j] x_(t - taps + 1 + j)) (+ x_t),  x_s = 0 for s < 0
//
// and the rings that later steps go on from: ring [slots][taps][C] holds the input of position p in row p % taps. A
// thread walks 16 tokens of a few channels with the last inputs in registers.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/scan_inputs.cuh"

namespace b200 {

constexpr int kCvTokens = 16, kCvAhead = 4;

struct ConvArgs {
  const void* x;      // [T][ldx]
  long long ldx;
  const void* w;      // [C, taps]
  const int* pos;     // [T] position in the token's sequence
  void* y;            // [T, C]
  const int *cu, *slots;
  void* ring;         // null: nothing is kept
  int n_seq, T, C, taps, silu, add;
};

template <class T, int V>
__device__ __forceinline__ void ldn(const T* p, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = ld1(p);
  } else {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 a = ld4(p + i);
      f[i] = a.x; f[i + 1] = a.y; f[i + 2] = a.z; f[i + 3] = a.w;
    }
  }
}
__device__ __forceinline__ void ldn(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 b = __bfloat1622float2(h[j]);
    f[2 * j] = b.x;
    f[2 * j + 1] = b.y;
  }
}
template <class T, int V>
__device__ __forceinline__ void stn(T* p, const float (&f)[V]) {
  if constexpr (V == 8) {
    uint4 out;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
    *reinterpret_cast<uint4*>(p) = out;
  } else if constexpr (V == 4) {
    st4(p, make_float4(f[0], f[1], f[2], f[3]));
  } else {
    st1(p, f[0]);
  }
}

// TAPS 0: any number of taps, inputs read once per tap
template <class T, int V, int TAPS>
__global__ void __launch_bounds__(256) short_conv_kernel(ConvArgs a) {
  const int nv = a.C / V, taps = TAPS ? TAPS : a.taps;
  const long long chunks = (a.T + kCvTokens - 1) / kCvTokens;
  const long long u = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  const int c = static_cast<int>(u % nv) * V;
  const long long unit = u / nv;
  const T* x = static_cast<const T*>(a.x) + c;
  if (unit >= chunks) {  // the last inputs of every sequence
    const long long s = unit - chunks;
    if (!a.ring || s >= static_cast<long long>(a.n_seq) * taps) return;
    const int seq = static_cast<int>(s / taps), back = static_cast<int>(s % taps) + 1;
    const int slot = a.slots[seq], t0 = a.cu[seq], t = a.cu[seq + 1] - back;
    if (slot < 0 || t < t0) return;
    float f[V];
    ldn(x + t * a.ldx, f);
    stn(static_cast<T*>(a.ring) + (static_cast<long long>(slot) * taps + (t - t0) % taps) * a.C + c, f);
    return;
  }
  const int first = static_cast<int>(unit) * kCvTokens, last = min(a.T, first + kCvTokens);
  const T* w = static_cast<const T*>(a.w) + static_cast<long long>(c) * taps;
  T* y = static_cast<T*>(a.y) + c;
  auto finish = [&](int t, float (&acc)[V], const float (&cur)[V]) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      if (a.silu) acc[e] = silu_as(acc[e], y);
      if (a.add) acc[e] += cur[e];
    }
    stn(y + static_cast<long long>(t) * a.C, acc);
  };
  if constexpr (TAPS > 0) {
    float wt[TAPS * V];  // channel-major, as stored
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      float f[V];
      ldn(w + i * V, f);
#pragma unroll
      for (int e = 0; e < V; ++e) wt[i * V + e] = f[e];
    }
    float win[TAPS][V];  // win[j]: j tokens back
    const int p0 = a.pos[first];
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
#pragma unroll
      for (int e = 0; e < V; ++e) win[j - 1][e] = 0.f;
      if (j <= p0) ldn(x + (first - j) * a.ldx, win[j - 1]);
    }
    for (int tb = first; tb < last; tb += kCvAhead) {  // the loads of a few tokens go out together
      float in[kCvAhead][V];
      bool start[kCvAhead];
#pragma unroll
      for (int i = 0; i < kCvAhead; ++i) {
        const int t = min(tb + i, last - 1);
        ldn(x + t * a.ldx, in[i]);
        start[i] = a.pos[t] == 0;
      }
#pragma unroll
      for (int i = 0; i < kCvAhead; ++i) {
        if (tb + i >= last) break;
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
          for (int e = 0; e < V; ++e) win[j][e] = start[i] ? 0.f : win[j - 1][e];
#pragma unroll
        for (int e = 0; e < V; ++e) win[0][e] = in[i][e];
        float acc[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
          acc[e] = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc[e] = fmaf(win[j][e], wt[e * TAPS + TAPS - 1 - j], acc[e]);
        }
        finish(tb + i, acc, win[0]);
      }
    }
  } else {
    for (int t = first; t < last; ++t) {
      const int n = min(taps, a.pos[t] + 1);
      float acc[V], cur[V], f[V];
      ldn(x + t * a.ldx, cur);
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = cur[e] * ld1(w + e * taps + taps - 1);
      for (int j = 1; j < n; ++j) {
        ldn(x + (t - j) * a.ldx, f);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(f[e], ld1(w + e * taps + taps - 1 - j), acc[e]);
      }
      finish(t, acc, cur);
    }
  }
}

template <class T, int V>
static int launch_short_conv(const ConvArgs& a, cudaStream_t stream) {
  const long long units = (static_cast<long long>((a.T + kCvTokens - 1) / kCvTokens) + (a.ring ? static_cast<long long>(a.n_seq) * a.taps : 0)) *
                          (a.C / V);
  const long long grid = (units + 255) / 256;
  if (grid > 0x7fffffffLL) return -101;
#define B200_CV(K_) short_conv_kernel<T, V, K_><<<static_cast<unsigned>(grid), 256, 0, stream>>>(a)
  switch (a.taps) {
    case 1: B200_CV(1); break;
    case 2: B200_CV(2); break;
    case 3: B200_CV(3); break;
    case 4: B200_CV(4); break;
    default: B200_CV(0); break;
  }
#undef B200_CV
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace b200

extern "C" {

// x [T][ldx], w [C, taps], y [T, C] and ring [slots][taps][C] of the model's dtype (fp32: 1 for fp32, 0 for bf16); ring null:
// nothing is kept. y must not be x.
int b200_short_conv(const void* x, long long ldx, const void* w, const int* pos, void* y, const int* cu, const int* slots,
                    void* ring, int n_seq, int T, int C, int taps, int silu, int add, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || C <= 0) return 0;
  if (taps < 1) return -100;
  const ConvArgs a{x, ldx, w, pos, y, cu, slots, ring, n_seq, T, C, taps, silu, add};
  const int v = fp32 ? 4 : 8;
  auto aligned = [](const void* p) { return !(reinterpret_cast<uintptr_t>(p) & 15); };
  const bool wide = C % v == 0 && ldx % v == 0 && aligned(x) && aligned(w) && aligned(y) && aligned(ring);
  if (fp32) return wide ? launch_short_conv<float, 4>(a, stream) : launch_short_conv<float, 1>(a, stream);
  return wide ? launch_short_conv<__nv_bfloat16, 8>(a, stream) : launch_short_conv<__nv_bfloat16, 1>(a, stream);
}

}  // extern "C"
