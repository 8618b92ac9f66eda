// Row kernels of decoders with an fp32 residual stream whose sublayers read the stream itself and whose results are RMS
// normed (the kernel and the places that a sublayer's result is read from are in common/residual_row.cuh):
//
//   embed_rms      res = scale * table[id] + positions[p];     y = OUT(res)
//   residual_rms   res += RMS(delta; post);                    y = OUT(res)
//
// RMS(x; w) = x / sqrt(mean(x^2) + eps) * w. OUT is the residual itself, rounded to the model's dtype (w null), or
// out_scale * RMS(res; w) in front of the head.
#include "common/residual_row.cuh"

namespace b200 {

template <class T, int POST, class Src>
static int launch_residual_rms(const Src& src, const void* post, float* res, const void* w, void* y, long long rows, int W,
                               bool v4, float eps, float out_scale, cudaStream_t stream) {
  const RowNorms n{post, nullptr, w, nullptr, eps, out_scale};
  return w ? launch_residual_norm<T, POST, kRmsNorm>(src, n, res, y, rows, W, v4, stream)
           : launch_residual_norm<T, POST, kNoNorm>(src, n, res, y, rows, W, v4, stream);
}

}  // namespace b200

extern "C" {

// fp32: 1 when tables, weights and y are fp32, 0 for bf16. res [rows, W] is fp32. pos_table (null: none) has `positions`
// rows of W.
int b200_embed_rms(const int* ids, const void* table, long long vocab, float scale, const int* pos, const void* pos_table,
                   long long positions, float* res, const void* w, void* y, long long rows, int W, float eps,
                   float out_scale, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  using bf = __nv_bfloat16;
  if (fp32)
    return launch_residual_rms<float, kNoNorm>(
        ScaledEmbedSrc<float>{{ids, (const float*)table, vocab, W}, scale, pos, (const float*)pos_table, positions}, nullptr,
        res, w, y, rows, W, true, eps, out_scale, stream);
  return launch_residual_rms<bf, kNoNorm>(
      ScaledEmbedSrc<bf>{{ids, (const bf*)table, vocab, W}, scale, pos, (const bf*)pos_table, positions}, nullptr, res, w, y,
      rows, W, true, eps, out_scale, stream);
}

// delta: rows [rows][ld] of bf16 or fp32 (delta_fp32; an fp32 model takes fp32 only), or with S > 0 the sum of S fp32
// slices [rows][W], `stride` numbers apart. res is updated in place.
int b200_residual_rms(const void* delta, int delta_fp32, long long ld, long long stride, int S, const void* post, float* res,
                      const void* w, void* y, long long rows, int W, float eps, float out_scale, int fp32,
                      cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (fp32 && !delta_fp32) return -100;
  using bf = __nv_bfloat16;
  const bool v4 = ld % 4 == 0 && stride % 4 == 0;
  if (S > 0) {
    const SliceSrc src{(const float*)delta, stride, S, W};
    return fp32 ? launch_residual_rms<float, kRmsNorm>(src, post, res, w, y, rows, W, v4, eps, out_scale, stream)
                : launch_residual_rms<bf, kRmsNorm>(src, post, res, w, y, rows, W, v4, eps, out_scale, stream);
  }
  if (fp32)
    return launch_residual_rms<float, kRmsNorm>(RowSrc<float>{(const float*)delta, ld}, post, res, w, y, rows, W, v4, eps,
                                                out_scale, stream);
  if (delta_fp32)
    return launch_residual_rms<bf, kRmsNorm>(RowSrc<float>{(const float*)delta, ld}, post, res, w, y, rows, W, v4, eps,
                                             out_scale, stream);
  return launch_residual_rms<bf, kRmsNorm>(RowSrc<bf>{(const bf*)delta, ld}, post, res, w, y, rows, W, v4, eps, out_scale,
                                           stream);
}

// delta[t] = sum_j wts[t, j] * rows[dest[t, j]] + an addend (ExpertSrc); rows and add are of the model's dtype.
int b200_experts_residual_rms(const void* rows_y, const int* dest, const float* wts, int k, const void* add,
                              long long ld_add, const float* ws, long long stride, int S, const float* add_gate,
                              const void* post, float* res,
                              const void* w, void* y, long long rows, int W, float eps, float out_scale, int fp32,
                              cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  using bf = __nv_bfloat16;
  const SliceSrc sl{ws, stride, S, W};
  if (fp32)
    return launch_residual_rms<float, kRmsNorm>(
        ExpertSrc<float>{(const float*)rows_y, dest, wts, k, W, (const float*)add, ld_add, sl, add_gate}, post, res, w, y, rows, W,
        true, eps, out_scale, stream);
  return launch_residual_rms<bf, kRmsNorm>(ExpertSrc<bf>{(const bf*)rows_y, dest, wts, k, W, (const bf*)add, ld_add, sl, add_gate},
                                           post, res, w, y, rows, W, true, eps, out_scale, stream);
}

}  // extern "C"
