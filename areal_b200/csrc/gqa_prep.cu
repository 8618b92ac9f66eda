// What stands between the input projection of grouped-query attention and the attention itself: rotation of the first
// dimensions of every query and key head (neighbouring pairs, or pairs of one dimension from each half of the rotated
// part), division of each head by its root mean square (optional), and the write of keys and values into their cache pages
//
//   k_cache [blocks, G, block_size, Dp], v_cache [blocks, G, block_size, Vp]      Dp, Vp: D, Dv in steps of 16, zero-filled
//
// One warp per (token, head); everything is computed in fp32 and rounded once.
#include "common/host_utils.h"
#include "common/io.cuh"

namespace b200 {

struct GqaPrepArgs {
  const void* x;                 // [T][ldx]: H * D | G * D | G * Dv | ...
  long long ldx;
  int H, G, D, Dv;
  const float *cosT, *sinT;      // [max_pos, rot / 2]
  const int* pos;
  int max_pos, rot, halves;
  float eps;                     // negative: heads are not normed
  void *q, *k, *v;               // [T][ld] + head * stride; k, v may be null; q, k may be x's own columns
  long long ldq, ldk, ldv;
  int hq, hk, hv;
  int Dp, Vp;
  const long long* slots;        // cache rows (negative: none); null: no cache
  void *k_cache, *v_cache;
  int block_size;
  long long cache_rows;          // blocks * block_size
  int T;
};

template <int V>
struct Vec { float e[V]; };

template <class T, int V>
__device__ __forceinline__ Vec<V> ldvec(const T* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const float4 a = ld4(p);
    r.e[0] = a.x; r.e[1] = a.y; r.e[2] = a.z; r.e[3] = a.w;
  } else {
    r.e[0] = ld1(p);
  }
  return r;
}
template <class T, int V>
__device__ __forceinline__ void stvec(T* p, const Vec<V>& a) {
  if constexpr (V == 4) st4(p, make_float4(a.e[0], a.e[1], a.e[2], a.e[3]));
  else st1(p, a.e[0]);
}

// V: elements per access; N: accesses per lane (32 * V * N >= Dp, Vp)
template <class T, int V, int N>
__global__ void __launch_bounds__(256) gqa_prep_kernel(GqaPrepArgs a) {
  const int units = a.H + 2 * a.G;
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= a.T * units) return;
  const int t = u / units, r = u - t * units;
  const bool is_q = r < a.H, is_v = r >= a.H + a.G;
  const int g = is_q ? r : (is_v ? r - a.H - a.G : r - a.H);
  const int width = is_v ? a.Dv : a.D, padded = is_v ? a.Vp : a.Dp;
  const T* src = static_cast<const T*>(a.x) + t * a.ldx +
                 (is_v ? static_cast<long long>(a.H + a.G) * a.D + static_cast<long long>(g) * a.Dv
                       : static_cast<long long>(r) * a.D);
  T* dst = nullptr;
  if (is_q) dst = static_cast<T*>(a.q) + t * a.ldq + static_cast<long long>(g) * a.hq;
  else if (is_v) dst = a.v ? static_cast<T*>(a.v) + t * a.ldv + static_cast<long long>(g) * a.hv : nullptr;
  else dst = a.k ? static_cast<T*>(a.k) + t * a.ldk + static_cast<long long>(g) * a.hk : nullptr;
  T* page = nullptr;
  if (!is_q && a.slots) {
    const long long slot = a.slots[t];
    if (slot >= 0 && slot < a.cache_rows) {
      const long long blk = slot / a.block_size;
      page = static_cast<T*>(is_v ? a.v_cache : a.k_cache) +
             ((blk * a.G + g) * a.block_size + (slot - blk * a.block_size)) * padded;
    }
  }
  if (!dst && !page) return;

  Vec<V> f[N];
  float s = 0.f;
  const int half = a.rot >> 1, rot = is_v ? 0 : a.rot;
  const int p = min(max(a.pos[t], 0), a.max_pos - 1);
  const float* cr = a.cosT + static_cast<long long>(p) * half;
  const float* sr = a.sinT + static_cast<long long>(p) * half;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 32 + lane) * V;
#pragma unroll
    for (int j = 0; j < V; ++j) f[i].e[j] = 0.f;
    if (c >= width) continue;
    f[i] = ldvec<T, V>(src + c);
    if (c < rot) {
      if (a.halves) {
        const bool low = c < half;
        const int e = low ? c : c - half;
        const Vec<V> o = ldvec<T, V>(src + (low ? c + half : e));
        const Vec<V> cs = ldvec<float, V>(cr + e), sn = ldvec<float, V>(sr + e);
#pragma unroll
        for (int j = 0; j < V; ++j) f[i].e[j] = f[i].e[j] * cs.e[j] + (low ? -o.e[j] : o.e[j]) * sn.e[j];
      } else if constexpr (V == 4) {
        const float2 cs = *reinterpret_cast<const float2*>(cr + (c >> 1)), sn = *reinterpret_cast<const float2*>(sr + (c >> 1));
        const Vec<V> o = f[i];
        f[i].e[0] = o.e[0] * cs.x - o.e[1] * sn.x;
        f[i].e[1] = o.e[1] * cs.x + o.e[0] * sn.x;
        f[i].e[2] = o.e[2] * cs.y - o.e[3] * sn.y;
        f[i].e[3] = o.e[3] * cs.y + o.e[2] * sn.y;
      } else {
        const float o = ld1(src + (c ^ 1)), cs = cr[c >> 1], sn = sr[c >> 1];
        f[i].e[0] = f[i].e[0] * cs + ((c & 1) ? o : -o) * sn;
      }
    }
#pragma unroll
    for (int j = 0; j < V; ++j) s = fmaf(f[i].e[j], f[i].e[j], s);
  }
  if (!is_v && a.eps >= 0.f) {
    // the warp's loads are all done here: the results may overwrite the source
    const float k = 1.f / sqrtf(warp_sum(s) / a.D + a.eps);
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int j = 0; j < V; ++j) f[i].e[j] *= k;
  } else {
    __syncwarp();
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = (i * 32 + lane) * V;
    if (c >= padded) continue;
    if (dst) stvec<T, V>(dst + c, f[i]);
    if (page) stvec<T, V>(page + c, f[i]);
  }
}

}  // namespace b200

extern "C" {

// x [T][ldx]: H * D | G * D | G * Dv | ... Queries go to q (head stride hq; Dp columns are written, zeros past D), keys to k
// and values to v (Vp columns) unless null, keys and values to the caches unless `slots` is null. eps < 0: no norm. q and k
// may be x's own columns when D == Dp. D, Dv <= 512.
int b200_gqa_prep(const void* x, long long ldx, int H, int G, int D, int Dv, const float* cosT, const float* sinT,
                  const int* pos, int max_pos, int rot, int halves, float eps, void* q, long long ldq, int hq, void* k,
                  long long ldk, int hk, void* v, long long ldv, int hv, int Dp, int Vp, const long long* slots,
                  void* k_cache, void* v_cache, int block_size, long long cache_rows, int T, int fp32,
                  cudaStream_t stream) {
  using namespace b200;
  if (T <= 0) return 0;
  if ((rot & 1) || rot > D || H < 1 || G < 1 || Dp < D || Vp < Dv || Dp > 512 || Vp > 512 || block_size < 1) return -100;
  const long long units = static_cast<long long>(T) * (H + 2 * G);
  if (units > 0x7fffffffLL - 8) return -101;
  GqaPrepArgs a{x, ldx, H, G, D, Dv, cosT, sinT, pos, max_pos, rot, halves, eps, q, k, v, ldq, ldk, ldv, hq, hk, hv, Dp, Vp,
                slots, k_cache, v_cache, block_size, cache_rows, T};
  const bool v4 = D % 4 == 0 && Dv % 4 == 0 && rot % 4 == 0 && (!halves || rot % 8 == 0) && ldx % 4 == 0 && ldq % 4 == 0 &&
                  ldk % 4 == 0 && ldv % 4 == 0 && hq % 4 == 0 && hk % 4 == 0 && hv % 4 == 0;
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
  const int w = Dp > Vp ? Dp : Vp;
  using bf = __nv_bfloat16;
#define B200_GP(T_, V_, N_) gqa_prep_kernel<T_, V_, N_><<<grid, 256, 0, stream>>>(a)
#define B200_GPN(T_)                                                                               \
  if (v4) {                                                                                        \
    if (w <= 128) B200_GP(T_, 4, 1); else if (w <= 256) B200_GP(T_, 4, 2); else B200_GP(T_, 4, 4); \
  } else {                                                                                         \
    if (w <= 128) B200_GP(T_, 1, 4); else B200_GP(T_, 1, 16);                                      \
  }
  if (fp32) { B200_GPN(float) } else { B200_GPN(bf) }
#undef B200_GPN
#undef B200_GP
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // extern "C"
