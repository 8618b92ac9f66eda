// Row kernels of decoders with an fp32 residual stream and layer norms on both sides of a sublayer (the kernel and the
// places that a sublayer's result is read from are in common/residual_row.cuh):
//
//   embed_ln      res = table[id];                            y = LN(res; w, b)
//   residual_ln   res += LN(delta; post_w, post_b);           y = LN(res; w, b)
//
// LN(x) = (x - mean) / sqrt(variance + eps) * w + b with the mean of the squared deviations as variance. And the plain
// activation kernels behind products that have no fused form.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/residual_row.cuh"

extern "C" int b200_gemm_bf16_splitk_partials(const void* A, const void* B, float* workspace, int M, int N, int K,
                                              long long lda, long long ldb, int splits, int* S_out,
                                              long long* stride_out, cudaStream_t stream);

namespace b200 {

template <class T, class Src>
static int launch_residual_ln(const Src& src, const void* pw, const void* pb, float* res, const void* w, const void* b,
                              void* y, long long rows, int W, bool v4, float eps, cudaStream_t stream) {
  return launch_residual_norm<T, kLayerNorm, kLayerNorm>(src, RowNorms{pw, pb, w, b, eps, 1.f}, res, y, rows, W, v4, stream);
}
template <class T>
static int launch_residual_ln(const EmbedSrc<T>& src, const void*, const void*, float* res, const void* w, const void* b,
                              void* y, long long rows, int W, bool v4, float eps, cudaStream_t stream) {
  return launch_residual_norm<T, kNoNorm, kLayerNorm>(src, RowNorms{nullptr, nullptr, w, b, eps, 1.f}, res, y, rows, W, v4,
                                                      stream);
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

template <class T>
__global__ void glu_pairs_kernel(const T* __restrict__ z, T* __restrict__ y, long long n, GluParams p) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n;
       i += static_cast<long long>(gridDim.x) * blockDim.x)
    st1(y + i, glu_act(ld1(z + 2 * i), ld1(z + 2 * i + 1), p, y));
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
    return launch_residual_ln(EmbedSrc<float>{ids, (const float*)table, vocab, W}, nullptr, nullptr, res, w, b, y,
                                     rows, W, true, eps, stream);
  using bf = __nv_bfloat16;
  return launch_residual_ln(EmbedSrc<bf>{ids, (const bf*)table, vocab, W}, nullptr, nullptr, res, w, b, y, rows, W,
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

// delta[t] = sum_j wts[t, j] * rows[dest[t, j]] + an addend (ExpertSrc); rows and add are of the model's dtype.
int b200_experts_residual_ln(const void* rows_y, const int* dest, const float* wts, int k, const void* add,
                             long long ld_add, const float* ws, long long stride, int S, const float* add_gate,
                             const void* pw, const void* pb, float* res, const void* w, const void* b, void* y, long long rows, int W, float eps,
                             int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  const SliceSrc sl{ws, stride, S, W};
  if (fp32)
    return launch_residual_ln<float>(ExpertSrc<float>{(const float*)rows_y, dest, wts, k, W, (const float*)add, ld_add, sl, add_gate},
                                     pw, pb, res, w, b, y, rows, W, true, eps, stream);
  using bf = __nv_bfloat16;
  return launch_residual_ln<bf>(ExpertSrc<bf>{(const bf*)rows_y, dest, wts, k, W, (const bf*)add, ld_add, sl, add_gate}, pw, pb, res,
                                w, b, y, rows, W, true, eps, stream);
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

// y[i] = the gated activation of the pair z[2i], z[2i + 1], i < n
int b200_glu_pairs(const void* z, void* y, long long n, float limit, float alpha, float beta, int fp32,
                   cudaStream_t stream) {
  using namespace b200;
  if (n <= 0) return 0;
  const GluParams p{limit, alpha, beta};
  using bf = __nv_bfloat16;
  if (fp32) glu_pairs_kernel<<<flat_grid(n), 256, 0, stream>>>((const float*)z, (float*)y, n, p);
  else glu_pairs_kernel<<<flat_grid(n), 256, 0, stream>>>((const bf*)z, (bf*)y, n, p);
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
