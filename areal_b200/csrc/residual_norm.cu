// Row kernels of decoders with an fp32 residual stream and layer norms on both sides of a sublayer:
//
//   embed_ln      res = table[id];                            y = LN(res; w, b)
//   residual_ln   res += LN(delta; post_w, post_b);           y = LN(res; w, b)
//
// LN(x) = (x - mean) / sqrt(variance + eps) * w + b with the mean of the squared deviations as variance. A sublayer's
// result `delta` is read from where the sublayer left it, so that no kernel stands between the sublayer's last product and
// the next sublayer's input:
//   * rows of bf16 or fp32 numbers;
//   * the fp32 K-slices of a split-K projection (decode-sized products), summed here and never rounded;
//   * the rows of a token's chosen experts, weighted here.
// Everything computed here is fp32; weights and y have the model's dtype. One block per row; a row stays in registers
// between the passes (mean, deviations, mean, deviations, output).
#include "common/host_utils.h"
#include "common/io.cuh"

extern "C" int b200_gemm_bf16_splitk_partials(const void* A, const void* B, float* workspace, int M, int N, int K,
                                              long long lda, long long ldb, int splits, int* S_out,
                                              long long* stride_out, cudaStream_t stream);

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
  static constexpr bool kPost = false;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    const long long id = ids[row];
    return id >= 0 && id < vocab ? ldv(table + id * W + c, V) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
};

template <class D>
struct RowSrc {
  const D* x;
  long long ld;
  static constexpr bool kPost = true;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    return ldv(x + row * ld + c, V);
  }
};

struct SliceSrc {
  const float* ws;
  long long stride;
  int S, W;
  static constexpr bool kPost = true;
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
  const float* w;    // [rows, k]
  int k, W;
  static constexpr bool kPost = true;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int j = 0; j < k; ++j) {
      const float s = __ldg(w + row * k + j);
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

// V: columns per vector; NV: vectors per thread
template <class T, class Src, int V, int NV>
__global__ void __launch_bounds__(NV >= 4 ? 512 : 1024) residual_ln_kernel(Src src, const T* __restrict__ pw, const T* __restrict__ pb,
                                                           float* __restrict__ res, const T* __restrict__ w,
                                                           const T* __restrict__ b, T* __restrict__ y, int W, float eps) {
  __shared__ float red[4][32];
  const long long row = blockIdx.x;
  float* rrow = res + row * W;
  float4 h[NV];
  int stage = 0;
  auto col = [&](int i) { return (i * static_cast<int>(blockDim.x) + static_cast<int>(threadIdx.x)) * V; };
  // (x - mean) / sqrt(var + eps): returns the mean and the factor
  auto moments = [&](float& mean, float& k) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += V == 4 ? (h[i].x + h[i].y) + (h[i].z + h[i].w) : h[i].x;  // zeros past the end
    mean = row_sum(s, red[stage++]) / W;
    s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) {
        const float a = h[i].x - mean, c = h[i].y - mean, d = h[i].z - mean, e = h[i].w - mean;
        s += V == 4 ? (a * a + c * c) + (d * d + e * e) : a * a;
      }
    k = 1.f / sqrtf(row_sum(s, red[stage++]) / W + eps);
  };
  auto affine = [&](float4 v, float mean, float k, float4 ww, float4 bb) {
    return make_float4(fmaf((v.x - mean) * k, ww.x, bb.x), fmaf((v.y - mean) * k, ww.y, bb.y),
                       fmaf((v.z - mean) * k, ww.z, bb.z), fmaf((v.w - mean) * k, ww.w, bb.w));
  };
#pragma unroll
  for (int i = 0; i < NV; ++i)
    h[i] = col(i) < W ? src.template load<V>(row, col(i)) : make_float4(0.f, 0.f, 0.f, 0.f);
  float mean, k;
  if constexpr (Src::kPost) {
    float4 r[NV];  // the residual is on its way while the statistics are taken
#pragma unroll
    for (int i = 0; i < NV; ++i) r[i] = col(i) < W ? ldv(rrow + col(i), V) : make_float4(0.f, 0.f, 0.f, 0.f);
    moments(mean, k);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) {
        const float4 d = affine(h[i], mean, k, ldv(pw + col(i), V), ldv(pb + col(i), V));
        h[i] = make_float4(r[i].x + d.x, r[i].y + d.y, r[i].z + d.z, r[i].w + d.w);
      }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      if (V == 4) st4(rrow + col(i), h[i]);
      else rrow[col(i)] = h[i].x;
    }
  moments(mean, k);
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      const float4 o = affine(h[i], mean, k, ldv(w + col(i), V), ldv(b + col(i), V));
      if (V == 4) st4(y + row * W + col(i), o);
      else st1(y + row * W + col(i), o.x);
    }
}

template <class T, class Src>
static int launch_residual_ln(const Src& src, const void* pw, const void* pb, float* res, const void* w, const void* b,
                              void* y, long long rows, int W, bool v4, float eps, cudaStream_t stream) {
  v4 = v4 && W % 4 == 0;
  const int vecs = v4 ? W / 4 : W;
  // many rows: four vectors per thread keep the barriers cheap; few rows: spread a row over more threads
  int nv = rows >= 4LL * sm_count() ? 4 : 1;
  if (nv == 4 && vecs <= 64) nv = 2;
  while (nv < 8 && (vecs + nv - 1) / nv > (nv >= 4 ? 512 : 1024)) nv <<= 1;
  const int block = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  if (block > (nv >= 4 ? 512 : 1024)) return -100;
  const unsigned grid = static_cast<unsigned>(rows);
#define B200_RL(V_, N_)                                                                                               \
  residual_ln_kernel<T, Src, V_, N_><<<grid, block, 0, stream>>>(src, (const T*)pw, (const T*)pb, res, (const T*)w,   \
                                                                 (const T*)b, (T*)y, W, eps)
#define B200_RLN(V_)                                                                                                  \
  if (nv == 1) B200_RL(V_, 1); else if (nv == 2) B200_RL(V_, 2); else if (nv == 4) B200_RL(V_, 4); else B200_RL(V_, 8);
  if (v4) { B200_RLN(4) } else { B200_RLN(1) }
#undef B200_RLN
#undef B200_RL
  B200_CHECK(cudaGetLastError());
  return 0;
}

// Activations in place of or behind a projection for dtypes and sizes without a fused form
template <class T>
__global__ void relu2_kernel(T* __restrict__ x, long long n) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const float v = fmaxf(ld1(x + i), 0.f);
    st1(x + i, v * v);
  }
}

__global__ void softcap_kernel(float* __restrict__ x, long long n, float cap) {
  const float inv = 1.f / cap;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x)
    x[i] = cap * tanhf(x[i] * inv);
}

static unsigned flat_grid(long long n) {
  long long g = (n + 255) / 256;
  const long long cap = static_cast<long long>(sm_count()) * 16;
  return static_cast<unsigned>(g < cap ? g : cap);
}

}  // namespace b200

extern "C" {

// fp32: 1 when weights and y are fp32, 0 for bf16. res [rows, W] is fp32.
int b200_embed_ln(const int* ids, const void* table, long long vocab, float* res, const void* w, const void* b, void* y,
                  long long rows, int W, float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (fp32)
    return launch_residual_ln<float>(EmbedSrc<float>{ids, (const float*)table, vocab, W}, nullptr, nullptr, res, w, b, y,
                                     rows, W, true, eps, stream);
  using bf = __nv_bfloat16;
  return launch_residual_ln<bf>(EmbedSrc<bf>{ids, (const bf*)table, vocab, W}, nullptr, nullptr, res, w, b, y, rows, W,
                                true, eps, stream);
}

// delta [rows][ld], bf16 or fp32 (delta_fp32; an fp32 model takes fp32 only). res is updated in place.
int b200_residual_ln(const void* delta, int delta_fp32, long long ld, const void* pw, const void* pb, float* res,
                     const void* w, const void* b, void* y, long long rows, int W, float eps, int fp32,
                     cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (fp32 && !delta_fp32) return -100;
  using bf = __nv_bfloat16;
  const bool v4 = ld % 4 == 0;
  if (fp32)
    return launch_residual_ln<float>(RowSrc<float>{(const float*)delta, ld}, pw, pb, res, w, b, y, rows, W, v4, eps, stream);
  if (delta_fp32)
    return launch_residual_ln<bf>(RowSrc<float>{(const float*)delta, ld}, pw, pb, res, w, b, y, rows, W, v4, eps, stream);
  return launch_residual_ln<bf>(RowSrc<bf>{(const bf*)delta, ld}, pw, pb, res, w, b, y, rows, W, v4, eps, stream);
}

// delta = A [M, K] . B [W, K]^T by split-K into `workspace` (fp32 [splits * ceil(M/128)*128 * W]), all else bf16.
int b200_splitk_residual_ln(const void* A, const void* B, float* workspace, int M, int W, int K, long long lda,
                            long long ldb, int splits, const void* pw, const void* pb, float* res, const void* w,
                            const void* b, void* y, float eps, cudaStream_t stream) {
  using namespace b200;
  if (M <= 0 || W <= 0 || K <= 0) return 0;
  int S = 0;
  long long stride = 0;
  const int rc = b200_gemm_bf16_splitk_partials(A, B, workspace, M, W, K, lda, ldb, splits, &S, &stride, stream);
  if (rc) return rc;
  return launch_residual_ln<__nv_bfloat16>(SliceSrc{workspace, stride, S, W}, pw, pb, res, w, b, y, M, W, true, eps, stream);
}

// delta[t] = sum_j wts[t, j] * rows[dest[t, j]]; rows are [.., W] of the model's dtype.
int b200_experts_residual_ln(const void* rows_y, const int* dest, const float* wts, int k, const void* pw,
                             const void* pb, float* res, const void* w, const void* b, void* y, long long rows, int W,
                             float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (fp32)
    return launch_residual_ln<float>(ExpertSrc<float>{(const float*)rows_y, dest, wts, k, W}, pw, pb, res, w, b, y, rows, W,
                                     true, eps, stream);
  using bf = __nv_bfloat16;
  return launch_residual_ln<bf>(ExpertSrc<bf>{(const bf*)rows_y, dest, wts, k, W}, pw, pb, res, w, b, y, rows, W, true, eps,
                                stream);
}

// x <- max(x, 0)^2
int b200_relu2(void* x, long long n, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (n <= 0) return 0;
  if (fp32) relu2_kernel<<<flat_grid(n), 256, 0, stream>>>((float*)x, n);
  else relu2_kernel<<<flat_grid(n), 256, 0, stream>>>((__nv_bfloat16*)x, n);
  B200_CHECK(cudaGetLastError());
  return 0;
}

// x <- cap * tanh(x / cap), fp32
int b200_softcap(float* x, long long n, float cap, cudaStream_t stream) {
  using namespace b200;
  if (n <= 0) return 0;
  softcap_kernel<<<flat_grid(n), 256, 0, stream>>>(x, n, cap);
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // extern "C"
