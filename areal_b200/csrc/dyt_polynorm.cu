// Row-wise kernels of decoders with an fp32 residual stream, Dynamic Tanh norms and PolyNorm activations:
//
//   embed_dyt     res = table[id];                 y = tanh(alpha * res) * w + b
//   residual_dyt  res += scale * delta;            y = tanh(alpha * res) * w + b
//   polynorm      y = a N(z) + b N(z^2) + c N(z^3) + e,   N(u) = u / sqrt(mean(u^2) + eps)
//   group_rms     y = N(o per group of columns) * w (* sigmoid(gate), or gate * sigmoid(gate))
//
// Dynamic Tanh: Zhu, Chen, He, LeCun, Liu, "Transformers without Normalization". The residual stream and everything
// computed here is fp32; inputs, weights and y have the model's dtype (bf16 or fp32). Dynamic Tanh needs no row
// statistics, so these two kernels are element-wise and the projection in front of them can carry them in its
// epilogue (gemm_bf16.cu, DytEpi).
#include "common/host_utils.h"
#include "common/io.cuh"

namespace b200 {

template <class T, class D, int V>
__global__ void residual_dyt_kernel(const D* __restrict__ delta, long long ld_delta, const T* __restrict__ scale,
                                    float* __restrict__ res, const T* __restrict__ alpha, const T* __restrict__ w,
                                    const T* __restrict__ b, T* __restrict__ y, long long rows, int W) {
  const float al = ld1(alpha);
  const int nv = W / V;
  const long long total = rows * nv;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / nv;
    const int c = static_cast<int>(i % nv) * V;
    float* rp = res + r * W + c;
    if (V == 4) {
      const float4 d = ld4(delta + r * ld_delta + c), s = ld4(scale + c), ww = ld4(w + c), bb = ld4(b + c);
      float4 h = ld4(rp);
      h.x = fmaf(s.x, d.x, h.x); h.y = fmaf(s.y, d.y, h.y); h.z = fmaf(s.z, d.z, h.z); h.w = fmaf(s.w, d.w, h.w);
      st4(rp, h);
      st4(y + r * W + c, make_float4(fmaf(tanh_as(al * h.x, y), ww.x, bb.x), fmaf(tanh_as(al * h.y, y), ww.y, bb.y),
                                     fmaf(tanh_as(al * h.z, y), ww.z, bb.z), fmaf(tanh_as(al * h.w, y), ww.w, bb.w)));
    } else {
      const float h = fmaf(ld1(scale + c), ld1(delta + r * ld_delta + c), *rp);
      *rp = h;
      st1(y + r * W + c, fmaf(tanh_as(al * h, y), ld1(w + c), ld1(b + c)));
    }
  }
}

// ids outside [0, vocab) give a zero row (as the plain embedding kernel does)
template <class T, int V>
__global__ void embed_dyt_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long vocab,
                                 float* __restrict__ res, const T* __restrict__ alpha, const T* __restrict__ w,
                                 const T* __restrict__ b, T* __restrict__ y, long long rows, int W) {
  const float al = ld1(alpha);
  const int nv = W / V;
  const long long total = rows * nv;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / nv;
    const int c = static_cast<int>(i % nv) * V;
    const long long id = ids[r];
    const bool in = id >= 0 && id < vocab;
    if (V == 4) {
      const float4 h = in ? ld4(table + id * W + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 ww = ld4(w + c), bb = ld4(b + c);
      st4(res + r * W + c, h);
      st4(y + r * W + c, make_float4(fmaf(tanh_as(al * h.x, y), ww.x, bb.x), fmaf(tanh_as(al * h.y, y), ww.y, bb.y),
                                     fmaf(tanh_as(al * h.z, y), ww.z, bb.z), fmaf(tanh_as(al * h.w, y), ww.w, bb.w)));
    } else {
      const float h = in ? ld1(table + id * W + c) : 0.f;
      res[r * W + c] = h;
      st1(y + r * W + c, fmaf(tanh_as(al * h, y), ld1(w + c), ld1(b + c)));
    }
  }
}

// One block per row. Up to kPnKeep vectors per thread stay in registers between the two passes; what does not fit is read
// again (from L1 / L2).
constexpr int kPnKeep = 4;
template <class T, int V>
__global__ void polynorm_kernel(const T* __restrict__ z, long long ldz, const T* __restrict__ coef, T* __restrict__ y,
                                int F, float eps) {
  __shared__ float red[3][33];
  const long long row = blockIdx.x;
  const T* zr = z + row * ldz;
  T* yr = y + row * F;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto acc = [&](float u) {
    const float u2 = u * u, u3 = u2 * u;
    s1 += u2;
    s2 = fmaf(u2, u2, s2);
    s3 = fmaf(u3, u3, s3);
  };
  auto load = [&](int c) { return V == 4 ? ld4(zr + c) : make_float4(ld1(zr + c), 0.f, 0.f, 0.f); };
  const int step = blockDim.x * V;
  float4 keep[kPnKeep];
#pragma unroll
  for (int i = 0; i < kPnKeep; ++i) {
    const int c = threadIdx.x * V + i * step;
    keep[i] = c < F ? load(c) : make_float4(0.f, 0.f, 0.f, 0.f);
    acc(keep[i].x); acc(keep[i].y); acc(keep[i].z); acc(keep[i].w);
  }
  for (int c = threadIdx.x * V + kPnKeep * step; c < F; c += step) {
    const float4 v = load(c);
    acc(v.x); acc(v.y); acc(v.z); acc(v.w);
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  s1 = warp_sum(s1); s2 = warp_sum(s2); s3 = warp_sum(s3);
  if (lane == 0) { red[0][warp] = s1; red[1][warp] = s2; red[2][warp] = s3; }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
  for (int i = 0; i < nw; ++i) { s1 += red[0][i]; s2 += red[1][i]; s3 += red[2][i]; }
  const float k1 = ld1(coef) / sqrtf(s1 / F + eps), k2 = ld1(coef + 1) / sqrtf(s2 / F + eps),
              k3 = ld1(coef + 2) / sqrtf(s3 / F + eps), e = ld1(coef + 3);
  auto out = [&](float u) { return fmaf(fmaf(fmaf(k3, u, k2), u, k1), u, e); };
  auto store = [&](int c, float4 v) {
    if (V == 4) st4(yr + c, make_float4(out(v.x), out(v.y), out(v.z), out(v.w)));
    else st1(yr + c, out(v.x));
  };
#pragma unroll
  for (int i = 0; i < kPnKeep; ++i) {
    const int c = threadIdx.x * V + i * step;
    if (c < F) store(c, keep[i]);
  }
  for (int c = threadIdx.x * V + kPnKeep * step; c < F; c += step) store(c, load(c));
}

// o [rows, groups * n] fp32. One warp per (row, group) when a group is narrow, one block per (row, group) else.
// w: [n] shared by the groups (w_per_group 0) or [groups * n]. gate: null or [rows, groups * n] with pitch ld_gate; silu: the
// result is multiplied by gate * sigmoid(gate) instead of sigmoid(gate).
template <class T, bool WARP, int V>
__global__ void group_rms_kernel(const float* __restrict__ o, const T* __restrict__ w, int w_per_group,
                                 const T* __restrict__ gate, long long ld_gate, int silu, T* __restrict__ y,
                                 long long rows, int groups, int n, float eps) {
  auto act = [&](float u) { return sigmoid_as(u, y) * (silu ? u : 1.f); };
  __shared__ float red[33];
  const int nthr = WARP ? 32 : blockDim.x, tid = WARP ? (threadIdx.x & 31) : threadIdx.x;
  const long long unit = WARP ? static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5)
                              : static_cast<long long>(blockIdx.x);
  if (unit >= rows * groups) return;  // whole warps (or no thread) leave
  const long long r = unit / groups;
  const int g = static_cast<int>(unit % groups);
  const float* ob = o + r * groups * n + static_cast<long long>(g) * n;
  T* yb = y + r * groups * n + static_cast<long long>(g) * n;
  const T* wb = w + (w_per_group ? g * n : 0);
  const T* gb = gate ? gate + r * ld_gate + static_cast<long long>(g) * n : nullptr;
  float s = 0.f;
  for (int c = tid * V; c < n; c += nthr * V) {
    if (V == 4) {
      const float4 v = ld4(ob + c);
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    } else {
      s = fmaf(ob[c], ob[c], s);
    }
  }
  s = WARP ? warp_sum(s) : block_sum(s, red);
  const float k = 1.f / sqrtf(s / n + eps);
  for (int c = tid * V; c < n; c += nthr * V) {
    if (V == 4) {
      float4 v = ld4(ob + c);
      const float4 ww = ld4(wb + c);
      v.x *= k * ww.x; v.y *= k * ww.y; v.z *= k * ww.z; v.w *= k * ww.w;
      if (gb) {
        const float4 u = ld4(gb + c);
        v.x *= act(u.x); v.y *= act(u.y); v.z *= act(u.z); v.w *= act(u.w);
      }
      st4(yb + c, v);
    } else {
      float v = ob[c] * k * ld1(wb + c);
      if (gb) v *= act(ld1(gb + c));
      st1(yb + c, v);
    }
  }
}

static unsigned grid_for(long long total, int block, int per_sm) {
  long long g = (total + block - 1) / block;
  const long long cap = static_cast<long long>(sm_count()) * per_sm;
  if (g > cap) g = cap;
  return static_cast<unsigned>(g < 1 ? 1 : g);
}

template <class T>
static int residual_dyt(const void* delta, int delta_fp32, long long ld_delta, const void* scale, float* res,
                        const void* alpha, const void* w, const void* b, void* y, long long rows, int W,
                        cudaStream_t s) {
  const bool v4 = (W % 4 == 0) && (ld_delta % 4 == 0);
  const long long total = rows * (v4 ? W / 4 : W);
  const unsigned grid = grid_for(total, 256, 16);
#define B200_RD(D_, V_)                                                                                             \
  residual_dyt_kernel<T, D_, V_><<<grid, 256, 0, s>>>((const D_*)delta, ld_delta, (const T*)scale, res,             \
                                                      (const T*)alpha, (const T*)w, (const T*)b, (T*)y, rows, W)
  if (delta_fp32) { if (v4) B200_RD(float, 4); else B200_RD(float, 1); }
  else { if (v4) B200_RD(__nv_bfloat16, 4); else B200_RD(__nv_bfloat16, 1); }
#undef B200_RD
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace b200

extern "C" {

// fp32: 1 when weights and y are fp32, 0 for bf16. res [rows, W] fp32 is updated in place.
int b200_residual_dyt(const void* delta, int delta_fp32, long long ld_delta, const void* scale, float* res,
                      const void* alpha, const void* w, const void* b, void* y, long long rows, int W, int fp32,
                      cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  return fp32 ? residual_dyt<float>(delta, delta_fp32, ld_delta, scale, res, alpha, w, b, y, rows, W, stream)
              : residual_dyt<__nv_bfloat16>(delta, delta_fp32, ld_delta, scale, res, alpha, w, b, y, rows, W, stream);
}

int b200_embed_dyt(const int* ids, const void* table, long long vocab, float* res, const void* alpha, const void* w,
                   const void* b, void* y, long long rows, int W, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  const bool v4 = W % 4 == 0;
  const unsigned grid = grid_for(rows * (v4 ? W / 4 : W), 256, 16);
#define B200_ED(T_, V_)                                                                                             \
  embed_dyt_kernel<T_, V_><<<grid, 256, 0, stream>>>(ids, (const T_*)table, vocab, res, (const T_*)alpha,           \
                                                     (const T_*)w, (const T_*)b, (T_*)y, rows, W)
  if (fp32) { if (v4) B200_ED(float, 4); else B200_ED(float, 1); }
  else { if (v4) B200_ED(__nv_bfloat16, 4); else B200_ED(__nv_bfloat16, 1); }
#undef B200_ED
  B200_CHECK(cudaGetLastError());
  return 0;
}

int b200_polynorm(const void* z, long long ldz, const void* coef, void* y, long long rows, int F, float eps, int fp32,
                  cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || F <= 0) return 0;
  const bool v4 = (F % 4 == 0) && (ldz % 4 == 0);
  // three or four vectors per thread when there are rows enough to fill the GPU, one otherwise
  const int vecs = v4 ? F / 4 : F, per = rows >= 4LL * sm_count() ? 3 : 1;
  int block = ((vecs + per - 1) / per + 31) / 32 * 32;
  if (block > 1024) block = 1024;
  using bf = __nv_bfloat16;
  const unsigned grid = static_cast<unsigned>(rows);
  if (fp32) {
    if (v4) polynorm_kernel<float, 4><<<grid, block, 0, stream>>>((const float*)z, ldz, (const float*)coef, (float*)y, F, eps);
    else polynorm_kernel<float, 1><<<grid, block, 0, stream>>>((const float*)z, ldz, (const float*)coef, (float*)y, F, eps);
  } else {
    if (v4) polynorm_kernel<bf, 4><<<grid, block, 0, stream>>>((const bf*)z, ldz, (const bf*)coef, (bf*)y, F, eps);
    else polynorm_kernel<bf, 1><<<grid, block, 0, stream>>>((const bf*)z, ldz, (const bf*)coef, (bf*)y, F, eps);
  }
  B200_CHECK(cudaGetLastError());
  return 0;
}

int b200_group_rms(const float* o, const void* w, int w_per_group, const void* gate, long long ld_gate, int silu, void* y,
                   long long rows, int groups, int n, float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || groups <= 0 || n <= 0) return 0;
  using bf = __nv_bfloat16;
  const bool warp = n <= 512;
  const bool v4 = n % 4 == 0 && (!gate || (ld_gate % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (fp32 ? 16 : 8) == 0));
  int block = 256;
  if (!warp) while (block < 1024 && block * 8 < n) block <<= 1;
  const long long units = rows * groups;
  const unsigned grid = static_cast<unsigned>(warp ? (units + 7) / 8 : units);
#define B200_GR(T_, W_, V_)                                                                                         \
  group_rms_kernel<T_, W_, V_><<<grid, block, 0, stream>>>(o, (const T_*)w, w_per_group, (const T_*)gate, ld_gate,  \
                                                           silu, (T_*)y, rows, groups, n, eps)
#define B200_GRV(T_)                                                                                                \
  if (warp) { if (v4) B200_GR(T_, true, 4); else B200_GR(T_, true, 1); }                                            \
  else { if (v4) B200_GR(T_, false, 4); else B200_GR(T_, false, 1); }
  if (fp32) { B200_GRV(float) } else { B200_GRV(bf) }
#undef B200_GRV
#undef B200_GR
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // extern "C"
