// Row kernel of decoders with an fp32 residual stream, shared by the norm families (residual_norm.cu: layer norms on both
// sides of a sublayer; residual_rms.cu: RMS norms on its result):
//
//   res += POST(delta);   y = PRE(res)           (an embedding: res = delta, no POST)
//
// A sublayer's result `delta` is read from where the sublayer left it (the Src types), so that no kernel stands between
// the sublayer's last product and the next sublayer's input:
//   * rows of bf16 or fp32 numbers;
//   * the fp32 K-slices of a split-K projection (decode-sized products), summed here and never rounded;
//   * the rows of a token's chosen experts, weighted here, plus what every token adds to them.
// Everything computed here is fp32; weights and y have the model's dtype. One block per row; a row stays in registers
// between the passes.
#pragma once
#include "host_utils.h"
#include "io.cuh"

#include <type_traits>

namespace b200 {

template <class T>
__device__ __forceinline__ float4 ldv(const T* p, int v) {
  return v == 4 ? ld4(p) : make_float4(ld1(p), 0.f, 0.f, 0.f);
}

template <class T>
struct EmbedSrc {  // ids outside [0, vocab) give a zero row (as the plain embedding kernel does)
  const int* ids;
  const T* table;
  long long vocab;
  int W;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    const long long id = ids[row];
    return id >= 0 && id < vocab ? ldv(table + id * W + c, V) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
};

template <class T>
struct ScaledEmbedSrc {  // scale * table[id], plus the position's row of a second table (null: none; outside it: zero)
  EmbedSrc<T> e;
  float scale;
  const int* pos;
  const T* pos_table;
  long long positions;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    float4 a = e.template load<V>(row, c);
    a = make_float4(a.x * scale, a.y * scale, a.z * scale, a.w * scale);
    if (pos_table) {
      const long long p = pos[row];
      if (p >= 0 && p < positions) {
        const float4 b = ldv(pos_table + p * e.W + c, V);
        a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
      }
    }
    return a;
  }
};

template <class D>
struct RowSrc {
  const D* x;
  long long ld;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    return ldv(x + row * ld + c, V);
  }
};

struct SliceSrc {
  const float* ws;
  long long stride;
  int S, W;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < S; ++s) {
      const float4 v = ldv(ws + s * stride + row * W + c, V);
      a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
    }
    return a;
  }
};

template <class T>
struct ExpertSrc {
  const T* y;        // rows of the experts' results
  const int* dest;   // [rows, k] row of every choice
  const float* w;    // [rows, k]; null: every choice counts once
  int k, W;
  const T* add;      // null, or [rows][ld_add]: added to the sum of the choices
  long long ld_add;
  SliceSrc slices;   // S > 0: the same as the slices of a split product
  const float* add_gate;  // null, or [rows]: what is added is multiplied by the sigmoid of the row's number
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    float4 a = slices.template load<V>(row, c);
    if (add) a = ldv(add + row * ld_add + c, V);
    if (add_gate) {
      const float s = 1.f / (1.f + expf(-__ldg(add_gate + row)));
      a = make_float4(a.x * s, a.y * s, a.z * s, a.w * s);
    }
#pragma unroll 4
    for (int j = 0; j < k; ++j) {
      const float s = w ? __ldg(w + row * k + j) : 1.f;
      const float4 v = ldv(y + static_cast<long long>(__ldg(dest + row * k + j)) * W + c, V);
      a.x = fmaf(s, v.x, a.x); a.y = fmaf(s, v.y, a.y); a.z = fmaf(s, v.z, a.z); a.w = fmaf(s, v.w, a.w);
    }
    return a;
  }
};

// Sum over the block through `red` (32 floats that no other call of the row uses). One barrier.
__device__ __forceinline__ float row_sum(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  v = warp_sum(v);
  if (nw == 1) return v;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];
  return t;
}

enum : int { kNoNorm = 0, kLayerNorm = 1, kRmsNorm = 2 };

struct RowNorms {
  const void *pw, *pb;  // POST's weight and (layer norm) bias
  const void *w, *b;    // PRE's
  float eps, out_scale; // out_scale multiplies the result of an RMS norm in PRE
};

// V: columns per vector; NV: vectors per thread; POST, PRE: kinds of norm (kNoNorm in POST: an embedding)
template <class T, class Src, int V, int NV, int POST, int PRE>
__global__ void __launch_bounds__(NV >= 4 ? 512 : 1024) residual_norm_kernel(Src src, RowNorms nn, float* __restrict__ res,
                                                                             T* __restrict__ y, int W) {
  const T *pw = static_cast<const T*>(nn.pw), *pb = static_cast<const T*>(nn.pb);
  const T *w = static_cast<const T*>(nn.w), *b = static_cast<const T*>(nn.b);
  const float eps = nn.eps;
  __shared__ float red[4][32];
  const long long row = blockIdx.x;
  float* rrow = res + row * W;
  float4 h[NV];
  int stage = 0;
  auto col = [&](int i) { return (i * static_cast<int>(blockDim.x) + static_cast<int>(threadIdx.x)) * V; };
  // (x - mean) / sqrt(var + eps), an RMS norm with the mean left at 0: returns the mean and the factor
  auto moments = [&](auto kind, float& mean, float& k) {
    mean = 0.f;
    if constexpr (kind.value == kLayerNorm) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) s += V == 4 ? (h[i].x + h[i].y) + (h[i].z + h[i].w) : h[i].x;  // zeros past the end
      mean = row_sum(s, red[stage++]) / W;
    }
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) {
        const float a = h[i].x - mean, c = h[i].y - mean, d = h[i].z - mean, e = h[i].w - mean;
        s += V == 4 ? (a * a + c * c) + (d * d + e * e) : a * a;
      }
    k = 1.f / sqrtf(row_sum(s, red[stage++]) / W + eps);
  };
  auto affine = [&](auto kind, float4 v, float mean, float k, const T* wp, const T* bp, int c) {
    const float4 ww = ldv(wp + c, V);
    if constexpr (kind.value == kLayerNorm) {
      const float4 bb = ldv(bp + c, V);
      return make_float4(fmaf((v.x - mean) * k, ww.x, bb.x), fmaf((v.y - mean) * k, ww.y, bb.y),
                         fmaf((v.z - mean) * k, ww.z, bb.z), fmaf((v.w - mean) * k, ww.w, bb.w));
    }
    return make_float4(v.x * k * ww.x, v.y * k * ww.y, v.z * k * ww.z, v.w * k * ww.w);
  };
#pragma unroll
  for (int i = 0; i < NV; ++i)
    h[i] = col(i) < W ? src.template load<V>(row, col(i)) : make_float4(0.f, 0.f, 0.f, 0.f);
  float mean, k;
  if constexpr (POST != kNoNorm) {
    constexpr std::integral_constant<int, POST> kind;
    float4 r[NV];  // the residual is on its way while the statistics are taken
#pragma unroll
    for (int i = 0; i < NV; ++i) r[i] = col(i) < W ? ldv(rrow + col(i), V) : make_float4(0.f, 0.f, 0.f, 0.f);
    moments(kind, mean, k);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) {
        const float4 d = affine(kind, h[i], mean, k, pw, pb, col(i));
        h[i] = make_float4(r[i].x + d.x, r[i].y + d.y, r[i].z + d.z, r[i].w + d.w);
      }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      if (V == 4) st4(rrow + col(i), h[i]);
      else rrow[col(i)] = h[i].x;
    }
  if constexpr (PRE != kNoNorm) {
    constexpr std::integral_constant<int, PRE> kind;
    moments(kind, mean, k);
    if (PRE == kRmsNorm) k *= nn.out_scale;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) h[i] = affine(kind, h[i], mean, k, w, b, col(i));
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      if (V == 4) st4(y + row * W + col(i), h[i]);
      else st1(y + row * W + col(i), h[i].x);
    }
}

template <class T, int POST, int PRE, class Src>
static int launch_residual_norm(const Src& src, const RowNorms& norms, float* res, void* y, long long rows, int W, bool v4,
                                cudaStream_t stream) {
  v4 = v4 && W % 4 == 0;
  const int vecs = v4 ? W / 4 : W;
  // many rows: four vectors per thread keep the barriers cheap; few rows: spread a row over more threads
  int nv = rows >= 4LL * sm_count() ? 4 : 1;
  if (nv == 4 && vecs <= 64) nv = 2;
  while (nv < 8 && (vecs + nv - 1) / nv > (nv >= 4 ? 512 : 1024)) nv <<= 1;
  const int block = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  if (block > (nv >= 4 ? 512 : 1024)) return -100;
  const unsigned grid = static_cast<unsigned>(rows);
#define B200_RL(V_, N_) \
  residual_norm_kernel<T, Src, V_, N_, POST, PRE><<<grid, block, 0, stream>>>(src, norms, res, (T*)y, W)
#define B200_RLN(V_)                                                                                                  \
  if (nv == 1) B200_RL(V_, 1); else if (nv == 2) B200_RL(V_, 2); else if (nv == 4) B200_RL(V_, 4); else B200_RL(V_, 8);
  if (v4) { B200_RLN(4) } else { B200_RLN(1) }
#undef B200_RLN
#undef B200_RL
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace b200
