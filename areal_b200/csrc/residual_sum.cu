// Row kernels of decoders whose two sublayers read one layer norm and are added to an fp32 residual stream together:
//
//   embed_sum      res = scale * table[id] + sinusoids(p);                                   y = LN(res)
//   residual_sum   res += mult * (a + f),  or with a pair  mult * (RMS(a; wa) / 2 + RMS(b; wb) / 2 + f);   y = LN(res)
//
// a, b: a mixer's results; f: the feed-forward's. They are read from where the sublayers left them (common/residual_row.cuh).
// A decode step goes on to what the next mixer reads, yc = y + conv(y), a causal convolution over time per channel whose
// last inputs are kept in a ring [slots][taps][W], position p in row p % taps. Everything computed here is fp32; y is rounded
// ahead of the convolution. One block per row; a row stays in registers between the passes.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/residual_row.cuh"
#include "common/scan_inputs.cuh"

namespace b200 {

template <class T>
struct AnySrc {  // rows of the model's dtype, or (x null) the slices of a split product
  const T* x;
  long long ld;
  SliceSrc sl;
  template <int V>
  __device__ __forceinline__ float4 load(long long row, int c) const {
    return x ? ldv(x + row * ld + c, V) : sl.template load<V>(row, c);
  }
};

// How the results are read (V 4 only; kAny asks for each piece): all of them rows, or the experts' uncombined rows with a
// gated addend of rows
enum : int { kAny = 0, kRows = 1, kExperts = 2 };

template <class T>
struct SumArgs {
  EmbedSrc<T> emb;          // kind 0
  float scale;
  const int* pos;           // null: no sinusoids
  const double* turns;      // [ceil(W / 2)] turns per position
  AnySrc<T> a, b;           // kinds 1, 2
  const T *wa, *wb;         // kind 2
  ExpertSrc<T> f;
  float mult, eps;
  float* res;
  const T *w, *bias;
  T* y;
  const T* cw;              // null, or the convolution behind the norm: [W, taps]
  int taps;
  T* ring;
  const int *slots, *cpos;
  T* yc;
  int W;
};

// KIND 0: embedding; 1: one result of the mixer; 2: a pair. V: columns per vector; NV: vectors per thread; FROM: see above
template <class T, int KIND, int V, int NV, int FROM>
__global__ void __launch_bounds__(NV >= 4 ? 512 : 1024) residual_sum_kernel(const SumArgs<T> g) {
  __shared__ float red[4][32];
  const long long row = blockIdx.x;
  const int W = g.W;
  float* rrow = g.res + row * W;
  float4 h[NV];
  auto col = [&](int i) { return (i * static_cast<int>(blockDim.x) + static_cast<int>(threadIdx.x)) * V; };
  auto sq = [](float4 v) { return V == 4 ? (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w) : v.x * v.x; };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  if constexpr (KIND == 0) {
    const double p = g.pos ? static_cast<double>(g.pos[row]) : 0.0;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = col(i);
      h[i] = zero;
      if (c >= W) continue;
      const float4 e = g.emb.template load<V>(row, c);
      h[i] = make_float4(e.x * g.scale, e.y * g.scale, e.z * g.scale, e.w * g.scale);
      if (g.pos) {
        auto wave = [&](int k, float& s, float& co) {  // whole turns are taken off in 64-bit
          const double t = p * g.turns[k];
          sincospif(2.f * static_cast<float>(t - rint(t)), &s, &co);
        };
        float s, co;
        wave(c >> 1, s, co);
        if (V == 4) {
          h[i].x += s;
          h[i].y += co;
          wave((c >> 1) + 1, s, co);
          h[i].z += s;
          h[i].w += co;
        } else {
          h[i].x += (c & 1) ? co : s;
        }
      }
    }
  } else {
    float4 a[NV], b[KIND == 2 ? NV : 1], r[NV];
    const float fg = FROM == kExperts ? 1.f / (1.f + expf(-__ldg(g.f.add_gate + row))) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const bool in = col(i) < W;
      if constexpr (FROM != kAny) {
        a[i] = in ? ldv(g.a.x + row * g.a.ld + col(i), V) : zero;
        if constexpr (KIND == 2) b[i] = in ? ldv(g.b.x + row * g.b.ld + col(i), V) : zero;
        h[i] = in ? ldv(g.f.add + row * g.f.ld_add + col(i), V) : zero;
        if constexpr (FROM == kExperts) { h[i].x *= fg; h[i].y *= fg; h[i].z *= fg; h[i].w *= fg; }
      } else {
        a[i] = in ? g.a.template load<V>(row, col(i)) : zero;
        if constexpr (KIND == 2) b[i] = in ? g.b.template load<V>(row, col(i)) : zero;
        h[i] = in ? g.f.template load<V>(row, col(i)) : zero;
      }
      r[i] = in ? ldv(rrow + col(i), V) : zero;
    }
    if constexpr (FROM == kExperts) {
#pragma unroll 2
      for (int j = 0; j < g.f.k; ++j) {
        const float s = g.f.w ? __ldg(g.f.w + row * g.f.k + j) : 1.f;
        const T* y = g.f.y + static_cast<long long>(__ldg(g.f.dest + row * g.f.k + j)) * W;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          if (col(i) < W) {
            const float4 v = ldv(y + col(i), V);
            h[i].x = fmaf(s, v.x, h[i].x); h[i].y = fmaf(s, v.y, h[i].y); h[i].z = fmaf(s, v.z, h[i].z); h[i].w = fmaf(s, v.w, h[i].w);
          }
      }
    }
    if constexpr (KIND == 2) {
      float sa = 0.f, sb = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        sa += sq(a[i]);
        sb += sq(b[i]);
      }
      const float ka = 0.5f / sqrtf(row_sum(sa, red[0]) / W + g.eps), kb = 0.5f / sqrtf(row_sum(sb, red[1]) / W + g.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (col(i) < W) {
          const float4 u = ldv(g.wa + col(i), V), v = ldv(g.wb + col(i), V);
          h[i].x += a[i].x * ka * u.x + b[i].x * kb * v.x;
          h[i].y += a[i].y * ka * u.y + b[i].y * kb * v.y;
          h[i].z += a[i].z * ka * u.z + b[i].z * kb * v.z;
          h[i].w += a[i].w * ka * u.w + b[i].w * kb * v.w;
        }
    } else {
#pragma unroll
      for (int i = 0; i < NV; ++i) { h[i].x += a[i].x; h[i].y += a[i].y; h[i].z += a[i].z; h[i].w += a[i].w; }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (col(i) < W) {
        h[i] = make_float4(fmaf(g.mult, h[i].x, r[i].x), fmaf(g.mult, h[i].y, r[i].y), fmaf(g.mult, h[i].z, r[i].z),
                           fmaf(g.mult, h[i].w, r[i].w));
      }
  }
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      if (V == 4) st4(rrow + col(i), h[i]);
      else rrow[col(i)] = h[i].x;
      s += V == 4 ? (h[i].x + h[i].y) + (h[i].z + h[i].w) : h[i].x;
    }
  const float mean = row_sum(s, red[2]) / W;
  s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (col(i) < W) {
      h[i] = make_float4(h[i].x - mean, h[i].y - mean, h[i].z - mean, h[i].w - mean);
      s += sq(h[i]);
    }
  const float k = 1.f / sqrtf(row_sum(s, red[3]) / W + g.eps);
  const int slot = g.cw && g.slots ? g.slots[row] : -1, p = g.cw ? g.cpos[row] : 0;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = col(i);
    if (c >= W) continue;
    const float4 ww = ldv(g.w + c, V), bb = ldv(g.bias + c, V);
    float4 v = make_float4(fmaf(h[i].x * k, ww.x, bb.x), fmaf(h[i].y * k, ww.y, bb.y), fmaf(h[i].z * k, ww.z, bb.z),
                           fmaf(h[i].w * k, ww.w, bb.w));
    if (V == 4) st4(g.y + row * W + c, v);
    else st1(g.y + row * W + c, v.x);
    if (!g.cw) continue;
    v = make_float4(round_as(v.x, g.y), round_as(v.y, g.y), round_as(v.z, g.y), round_as(v.w, g.y));
    const T* cw = g.cw + static_cast<long long>(c) * g.taps + g.taps - 1;  // a column's last tap
    float4 o;
    o.x = fmaf(v.x, ld1(cw), v.x);
    if (V == 4) {
      o.y = fmaf(v.y, ld1(cw + g.taps), v.y);
      o.z = fmaf(v.z, ld1(cw + 2 * g.taps), v.z);
      o.w = fmaf(v.w, ld1(cw + 3 * g.taps), v.w);
    }
    if (slot >= 0) {
      T* ring = g.ring + static_cast<long long>(slot) * g.taps * W + c;
      for (int j = 1; j < g.taps && j <= p; ++j) {
        const float4 u = ldv(ring + static_cast<long long>((p - j) % g.taps) * W, V);
        o.x = fmaf(u.x, ld1(cw - j), o.x);
        if (V == 4) {
          o.y = fmaf(u.y, ld1(cw + g.taps - j), o.y);
          o.z = fmaf(u.z, ld1(cw + 2 * g.taps - j), o.z);
          o.w = fmaf(u.w, ld1(cw + 3 * g.taps - j), o.w);
        }
      }
      T* at = ring + static_cast<long long>(p % g.taps) * W;
      if (V == 4) st4(at, v);
      else st1(at, v.x);
    }
    if (V == 4) st4(g.yc + row * W + c, o);
    else st1(g.yc + row * W + c, o.x);
  }
}

template <class T, int KIND>
static int launch_residual_sum(const SumArgs<T>& g, long long rows, bool v4, cudaStream_t stream) {
  v4 = v4 && g.W % 4 == 0;
  const int vecs = v4 ? g.W / 4 : g.W;
  int nv = rows >= 4LL * sm_count() ? 4 : 1;
  if (nv == 4 && vecs <= 64) nv = 2;
  while (nv < 8 && (vecs + nv - 1) / nv > (nv >= 4 ? 512 : 1024)) nv <<= 1;
  const int block = ((vecs + nv - 1) / nv + 31) / 32 * 32;
  if (block > (nv >= 4 ? 512 : 1024)) return -100;
  const unsigned grid = static_cast<unsigned>(rows);
#define B200_RS(V_, N_, F_) residual_sum_kernel<T, KIND, V_, N_, F_><<<grid, block, 0, stream>>>(g)
#define B200_RSN(V_, F_) \
  if (nv == 1) B200_RS(V_, 1, F_); else if (nv == 2) B200_RS(V_, 2, F_); else if (nv == 4) B200_RS(V_, 4, F_); else B200_RS(V_, 8, F_);
  int from = kAny;
  if (KIND && v4 && g.a.x && (KIND == 1 || g.b.x) && g.f.add && !g.f.slices.S) {
    if (g.f.k > 0 && g.f.add_gate) from = kExperts;
    else if (g.f.k == 0 && !g.f.add_gate) from = kRows;
  }
  if (KIND == 0 || from == kAny) {
    if (v4) { B200_RSN(4, kAny) } else { B200_RSN(1, kAny) }
  } else if constexpr (KIND != 0) {
    if (from == kRows) { B200_RSN(4, kRows) } else { B200_RSN(4, kExperts) }
  }
#undef B200_RSN
#undef B200_RS
  B200_CHECK(cudaGetLastError());
  return 0;
}

template <class T>
static void sum_tail(SumArgs<T>& g, float* res, const void* w, const void* bias, void* y, const void* cw, int taps, void* ring,
                     const int* slots, const int* cpos, void* yc, int W, float eps) {
  g.res = res;
  g.w = static_cast<const T*>(w);
  g.bias = static_cast<const T*>(bias);
  g.y = static_cast<T*>(y);
  g.cw = static_cast<const T*>(cw);
  g.taps = taps;
  g.ring = static_cast<T*>(ring);
  g.slots = slots;
  g.cpos = cpos;
  g.yc = static_cast<T*>(yc);
  g.W = W;
  g.eps = eps;
}

}  // namespace b200

extern "C" {

// res [rows, W] fp32; tables, weights, ring, y and yc of the model's dtype (fp32: 1 for fp32, 0 for bf16). cw null: no
// convolution. slots: negative for padding rows.
int b200_embed_sum(const int* ids, const void* table, long long vocab, float scale, const int* pos, const double* turns,
                   float* res, const void* w, const void* bias, void* y, const void* cw, int taps, void* ring,
                   const int* slots, const int* cpos, void* yc, long long rows, int W, float eps, int fp32,
                   cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (cw && taps < 1) return -100;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    SumArgs<T> g{};
    g.emb = EmbedSrc<T>{ids, static_cast<const T*>(table), vocab, W};
    g.scale = scale;
    g.pos = pos;
    g.turns = turns;
    sum_tail(g, res, w, bias, y, cw, taps, ring, slots, cpos, yc, W, eps);
    return launch_residual_sum<T, 0>(g, rows, true, stream);
  };
  return fp32 ? run(float{}) : run(__nv_bfloat16{});
}

// a, b: rows [rows][ld] of the model's dtype, or (a null) the sum of aS fp32 slices [rows][W]; wa null: a alone, not normed.
// rows_y .. add_gate: the feed-forward's result, see ExpertSrc (k 0: the addend alone). res is updated in place.
int b200_residual_sum(const void* a, long long lda, const float* aws, long long astride, int aS, const void* wa, const void* b,
                      long long ldb, const float* bws, long long bstride, int bS, const void* wb, const void* rows_y,
                      const int* dest, const float* wts, int k, const void* add, long long ld_add, const float* ws,
                      long long stride, int S, const float* add_gate, float mult, float* res, const void* w,
                      const void* bias, void* y, const void* cw, int taps, void* ring, const int* slots, const int* cpos,
                      void* yc, long long rows, int W, float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || W <= 0) return 0;
  if (cw && taps < 1) return -100;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    SumArgs<T> g{};
    g.a = AnySrc<T>{static_cast<const T*>(a), lda, SliceSrc{aws, astride, aS, W}};
    g.b = AnySrc<T>{static_cast<const T*>(b), ldb, SliceSrc{bws, bstride, bS, W}};
    g.wa = static_cast<const T*>(wa);
    g.wb = static_cast<const T*>(wb);
    g.f = ExpertSrc<T>{static_cast<const T*>(rows_y), dest, wts, k, W, static_cast<const T*>(add), ld_add,
                       SliceSrc{ws, stride, S, W}, add_gate};
    g.mult = mult;
    sum_tail(g, res, w, bias, y, cw, taps, ring, slots, cpos, yc, W, eps);
    const bool v4 = lda % 4 == 0 && ldb % 4 == 0 && ld_add % 4 == 0;
    return wa ? launch_residual_sum<T, 2>(g, rows, v4, stream) : launch_residual_sum<T, 1>(g, rows, v4, stream);
  };
  return fp32 ? run(float{}) : run(__nv_bfloat16{});
}

}  // extern "C"
