// Row-wise kernels of decoders with an fp32 residual stream, Dynamic Tanh norms and PolyNorm activations:
//
//   embed_dyt     res = table[id];                 y = tanh(alpha * res) * w + b
//   residual_dyt  res += scale * delta;            y = tanh(alpha * res) * w + b
//   polynorm      y = a N(z) + b N(z^2) + c N(z^3) + e,   N(u) = u / sqrt(mean(u^2) + eps)
//   group_rms     y = N(o per group of columns) * w (* sigmoid(gate))
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
      st4(y + r * W + c, make_float4(fmaf(tanhf(al * h.x), ww.x, bb.x), fmaf(tanhf(al * h.y), ww.y, bb.y),
                                     fmaf(tanhf(al * h.z), ww.z, bb.z), fmaf(tanhf(al * h.w), ww.w, bb.w)));
    } else {
      const float h = fmaf(ld1(scale + c), ld1(delta + r * ld_delta + c), *rp);
      *rp = h;
      st1(y + r * W + c, fmaf(tanhf(al * h), ld1(w + c), ld1(b + c)));
    }
  }
}

// ids outside [0, vocab) give a zero row (as the plain embedding kernel does)
template <class T>
__global__ void embed_dyt_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long vocab,
                                 float* __restrict__ res, const T* __restrict__ alpha, const T* __restrict__ w,
                                 const T* __restrict__ b, T* __restrict__ y, long long rows, int W) {
  const float al = ld1(alpha);
  const long long total = rows * W;
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long r = i / W;
    const int c = static_cast<int>(i % W);
    const long long id = ids[r];
    const float h = (id >= 0 && id < vocab) ? ld1(table + id * W + c) : 0.f;
    res[i] = h;
    st1(y + i, fmaf(tanhf(al * h), ld1(w + c), ld1(b + c)));
  }
}

// One block per row; the row is read twice, the second time from L1 / L2.
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
  for (int c = threadIdx.x * V; c < F; c += blockDim.x * V) {
    if (V == 4) {
      const float4 v = ld4(zr + c);
      acc(v.x); acc(v.y); acc(v.z); acc(v.w);
    } else {
      acc(ld1(zr + c));
    }
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
  for (int c = threadIdx.x * V; c < F; c += blockDim.x * V) {
    if (V == 4) {
      const float4 v = ld4(zr + c);
      st4(yr + c, make_float4(out(v.x), out(v.y), out(v.z), out(v.w)));
    } else {
      st1(yr + c, out(ld1(zr + c)));
    }
  }
}

// o [rows, groups * n] fp32. One warp per (row, group) when a group is narrow, one block per (row, group) else.
// w: [n] shared by the groups (w_per_group 0) or [groups * n]. gate: null or [rows, groups * n] with pitch ld_gate.
template <class T, bool WARP>
__global__ void group_rms_kernel(const float* __restrict__ o, const T* __restrict__ w, int w_per_group,
                                 const T* __restrict__ gate, long long ld_gate, T* __restrict__ y, long long rows,
                                 int groups, int n, float eps) {
  __shared__ float red[33];
  const int nthr = WARP ? 32 : blockDim.x, tid = WARP ? (threadIdx.x & 31) : threadIdx.x;
  const long long unit = WARP ? static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5)
                              : static_cast<long long>(blockIdx.x);
  if (unit >= rows * groups) return;  // whole warps (or no thread) leave
  const long long r = unit / groups;
  const int g = static_cast<int>(unit % groups);
  const long long base = r * groups * n + static_cast<long long>(g) * n;
  float s = 0.f;
  for (int c = tid; c < n; c += nthr) s = fmaf(o[base + c], o[base + c], s);
  s = WARP ? warp_sum(s) : block_sum(s, red);
  const float k = 1.f / sqrtf(s / n + eps);
  for (int c = tid; c < n; c += nthr) {
    float v = o[base + c] * k * ld1(w + (w_per_group ? g * n + c : c));
    if (gate) v *= sigmoid_f(ld1(gate + r * ld_gate + static_cast<long long>(g) * n + c));
    st1(y + base + c, v);
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
  const unsigned grid = grid_for(rows * W, 256, 16);
  if (fp32)
    embed_dyt_kernel<float><<<grid, 256, 0, stream>>>(ids, (const float*)table, vocab, res, (const float*)alpha,
                                                      (const float*)w, (const float*)b, (float*)y, rows, W);
  else
    embed_dyt_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(
        ids, (const __nv_bfloat16*)table, vocab, res, (const __nv_bfloat16*)alpha, (const __nv_bfloat16*)w,
        (const __nv_bfloat16*)b, (__nv_bfloat16*)y, rows, W);
  B200_CHECK(cudaGetLastError());
  return 0;
}

int b200_polynorm(const void* z, long long ldz, const void* coef, void* y, long long rows, int F, float eps, int fp32,
                  cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || F <= 0) return 0;
  const bool v4 = (F % 4 == 0) && (ldz % 4 == 0);
  int block = 1024;
  while (block > 32 && block / 2 * (v4 ? 4 : 1) >= F) block >>= 1;
  if (block > 512 && rows >= 4LL * sm_count()) block = 512;
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

int b200_group_rms(const float* o, const void* w, int w_per_group, const void* gate, long long ld_gate, void* y,
                   long long rows, int groups, int n, float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || groups <= 0 || n <= 0) return 0;
  using bf = __nv_bfloat16;
  const bool warp = n <= 512;
  int block = 256;
  if (!warp) while (block < 1024 && block * 4 < n) block <<= 1;
  const long long units = rows * groups;
  const unsigned grid = static_cast<unsigned>(warp ? (units + 7) / 8 : units);
#define B200_GR(T_, W_)                                                                                             \
  group_rms_kernel<T_, W_><<<grid, block, 0, stream>>>(o, (const T_*)w, w_per_group, (const T_*)gate, ld_gate,      \
                                                       (T_*)y, rows, groups, n, eps)
  if (fp32) { if (warp) B200_GR(float, true); else B200_GR(float, false); }
  else { if (warp) B200_GR(bf, true); else B200_GR(bf, false); }
#undef B200_GR
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // extern "C"
