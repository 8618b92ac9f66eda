// What stands between the input projection of grouped-query attention and the attention itself: rotation of the first
// dimensions of every query and key head (neighbouring pairs, or pairs of one dimension from each half of the rotated
// part), division of each head by its root mean square (optional), and the write of keys and values into their cache pages
//
//   k_cache [blocks, G, block_size, Dp], v_cache [blocks, G, block_size, Vp]      Dp, Vp: D, Dv in steps of 16, zero-filled
//
// One warp per (token, head), or for bf16 widths in steps of 8 one part of a warp, eight numbers to a lane; everything is
// computed in fp32 and rounded once.
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
  void *q, *k, *v;               // [T][ld] + head * stride; all may be null; q, k may be x's own columns
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

// a cos + b sin, rounded the same way wherever it is compiled
__device__ __forceinline__ float turned(float a, float b, float c, float s) { return fmaf(a, c, __fmul_rn(b, s)); }

__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 b = __bfloat1622float2(h[j]);
    f[2 * j] = b.x;
    f[2 * j + 1] = b.y;
  }
}
__device__ __forceinline__ void ld8(const float* p, float (&f)[8]) {
  const float4 a = ld4(p), b = ld4(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// LPH: lanes per head (8 * LPH >= Dp, Vp); 32 / LPH heads per warp
template <int LPH>
__global__ void __launch_bounds__(256) gqa_prep8_kernel(GqaPrepArgs a) {
  using T = __nv_bfloat16;
  const int skip = a.q ? 0 : a.H, units = a.H - skip + 2 * a.G, lane = threadIdx.x & 31;
  const int u = (blockIdx.x * 8 + (threadIdx.x >> 5)) * (32 / LPH) + lane / LPH, c = (lane % LPH) * 8;
  const bool live = u < a.T * units;  // (whole warps stay for the shuffles)
  const int t = live ? u / units : 0, r = (live ? u - t * units : 0) + skip;
  const bool is_q = r < a.H, is_v = r >= a.H + a.G;
  const int g = is_q ? r : (is_v ? r - a.H - a.G : r - a.H);
  const int width = is_v ? a.Dv : a.D, padded = is_v ? a.Vp : a.Dp;
  const T* src = static_cast<const T*>(a.x) + t * a.ldx + (is_v ? (a.H + a.G) * a.D + g * a.Dv : r * a.D);
  const bool in = live && c < width;
  float f[8] = {};
  if (in) ld8(src + c, f);
  if (in && !is_v && c < a.rot) {
    const int half = a.rot >> 1;
    const long long at = static_cast<long long>(min(max(a.pos[t], 0), a.max_pos - 1)) * half;
    if (a.halves) {
      const bool low = c < half;
      const int e = low ? c : c - half;
      float o[8], cs[8], sn[8];
      ld8(src + (low ? c + half : e), o);
      ld8(a.cosT + at + e, cs);
      ld8(a.sinT + at + e, sn);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = turned(f[j], low ? -o[j] : o[j], cs[j], sn[j]);
    } else {
      const float4 cs = ld4(a.cosT + at + (c >> 1)), sn = ld4(a.sinT + at + (c >> 1));
      const float cc[4] = {cs.x, cs.y, cs.z, cs.w}, ss[4] = {sn.x, sn.y, sn.z, sn.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float x = f[2 * j], y = f[2 * j + 1];
        f[2 * j] = turned(x, -y, cc[j], ss[j]);
        f[2 * j + 1] = turned(y, x, cc[j], ss[j]);
      }
    }
  }
  if (a.eps >= 0.f) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) s = fmaf(f[j], f[j], s);
#pragma unroll
    for (int d = LPH / 2; d > 0; d >>= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
    // the warp's loads are all done here: the results may overwrite the source
    const float k = is_v ? 1.f : 1.f / sqrtf(s / a.D + a.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= k;
  } else {
    __syncwarp();
  }
  if (!live || c >= padded) return;
  uint4 out;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
  for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(f[2 * j], f[2 * j + 1]);
  T* dst = nullptr;
  if (is_q) dst = static_cast<T*>(a.q) + t * a.ldq + g * a.hq;
  else if (is_v) dst = a.v ? static_cast<T*>(a.v) + t * a.ldv + g * a.hv : nullptr;
  else dst = a.k ? static_cast<T*>(a.k) + t * a.ldk + g * a.hk : nullptr;
  if (dst) *reinterpret_cast<uint4*>(dst + c) = out;
  if (!is_q && a.slots) {
    const long long slot = a.slots[t];
    if (slot >= 0 && slot < a.cache_rows) {
      const int blk = static_cast<int>(slot) / a.block_size, off = static_cast<int>(slot) - blk * a.block_size;
      T* page = static_cast<T*>(is_v ? a.v_cache : a.k_cache) +
                ((static_cast<long long>(blk) * a.G + g) * a.block_size + off) * padded;
      *reinterpret_cast<uint4*>(page + c) = out;
    }
  }
}

// V: elements per access; N: accesses per lane (32 * V * N >= Dp, Vp)
template <class T, int V, int N>
__global__ void __launch_bounds__(256) gqa_prep_kernel(GqaPrepArgs a) {
  const int skip = a.q ? 0 : a.H, units = a.H - skip + 2 * a.G;
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= a.T * units) return;
  const int t = u / units, r = u - t * units + skip;
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
        for (int j = 0; j < V; ++j) f[i].e[j] = turned(f[i].e[j], low ? -o.e[j] : o.e[j], cs.e[j], sn.e[j]);
      } else if constexpr (V == 4) {
        const float2 cs = *reinterpret_cast<const float2*>(cr + (c >> 1)), sn = *reinterpret_cast<const float2*>(sr + (c >> 1));
        const Vec<V> o = f[i];
        f[i].e[0] = turned(o.e[0], -o.e[1], cs.x, sn.x);
        f[i].e[1] = turned(o.e[1], o.e[0], cs.x, sn.x);
        f[i].e[2] = turned(o.e[2], -o.e[3], cs.y, sn.y);
        f[i].e[3] = turned(o.e[3], o.e[2], cs.y, sn.y);
      } else {
        const float o = ld1(src + (c ^ 1)), cs = cr[c >> 1], sn = sr[c >> 1];
        f[i].e[0] = turned(f[i].e[0], (c & 1) ? o : -o, cs, sn);
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

// x [T][ldx]: H * D | G * D | G * Dv | ... Queries go to q (head stride hq; Dp columns are written, zeros past D; null: they stay
// as they are), keys to k and values to v (Vp columns) unless null, keys and values to the caches unless `slots` is null. eps < 0: no norm. q and k
// may be x's own columns when D == Dp. D, Dv <= 512.
int b200_gqa_prep(const void* x, long long ldx, int H, int G, int D, int Dv, const float* cosT, const float* sinT,
                  const int* pos, int max_pos, int rot, int halves, float eps, void* q, long long ldq, int hq, void* k,
                  long long ldk, int hk, void* v, long long ldv, int hv, int Dp, int Vp, const long long* slots,
                  void* k_cache, void* v_cache, int block_size, long long cache_rows, int T, int fp32,
                  cudaStream_t stream) {
  using namespace b200;
  if (T <= 0) return 0;
  if ((rot & 1) || rot > D || H < 1 || G < 1 || Dp < D || Vp < Dv || Dp > 512 || Vp > 512 || block_size < 1) return -100;
  const long long units = static_cast<long long>(T) * ((q ? H : 0) + 2 * G);
  if (units > 0x7fffffffLL - 8) return -101;
  GqaPrepArgs a{x, ldx, H, G, D, Dv, cosT, sinT, pos, max_pos, rot, halves, eps, q, k, v, ldq, ldk, ldv, hq, hk, hv, Dp, Vp,
                slots, k_cache, v_cache, block_size, cache_rows, T};
  const bool v4 = D % 4 == 0 && Dv % 4 == 0 && rot % 4 == 0 && (!halves || rot % 8 == 0) && ldx % 4 == 0 && ldq % 4 == 0 &&
                  ldk % 4 == 0 && ldv % 4 == 0 && hq % 4 == 0 && hk % 4 == 0 && hv % 4 == 0;
  const int w = Dp > Vp ? Dp : Vp;
  const bool v8 = !fp32 && w <= 256 && cache_rows < 0x7fffffff && D % 8 == 0 && Dv % 8 == 0 && rot % (halves ? 16 : 8) == 0 &&
                  !((ldx | ldq | ldk | ldv | hq | hk | hv) & 7) && !(reinterpret_cast<uintptr_t>(x) & 15);
  if (v8) {
    const int lph = w <= 64 ? 8 : (w <= 128 ? 16 : 32);
    const long long heads = 8LL * (32 / lph);
    const unsigned grid8 = static_cast<unsigned>((units + heads - 1) / heads);
    if (lph == 8) gqa_prep8_kernel<8><<<grid8, 256, 0, stream>>>(a);
    else if (lph == 16) gqa_prep8_kernel<16><<<grid8, 256, 0, stream>>>(a);
    else gqa_prep8_kernel<32><<<grid8, 256, 0, stream>>>(a);
    B200_CHECK(cudaGetLastError());
    return 0;
  }
  const unsigned grid = static_cast<unsigned>((units + 7) / 8);
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
