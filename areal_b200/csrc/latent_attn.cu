// Latent attention with a compressed paged cache: per token the normed latent c [rank] followed by one rotated key
// part [rot] shared by all heads (one "kv head" of width rank + rot).
//
//   latent_prep   splits the down projection's row [q_rank | rank | rot]: RMS norm of the query latent, RMS norm of
//                 the key / value latent, rotation of the shared key part, write of (latent | rotated part) into the
//                 cache page of the token
//   latent_qkv_prep  the same for a projection without query latent, [heads * (dim + rot) | rank | rot]: the queries'
//                 rotated parts turn in place
//   rope_pairs    rotates neighbouring pairs (2i, 2i+1) inside a slice of every head, in place
//   attend        softmax attention of any widths, fp32 throughout: one warp per (query, head). Keys come in two
//                 parts (per head, shared) and from rows of a packed batch (prefill) or from pages (decode, where the
//                 per-head part is the latent itself, shared by the heads too, and the queries carry the key
//                 up-projection). The tensor-core kernels cover the widths of real models; this one covers the rest
//                 and fp32. A window bounds how far back a query sees; a gate scales every head's result by a sigmoid.
//                 Grouped-query attention runs here too: keys and values per group of heads, first tokens that a window
//                 keeps, a soft cap on the scores, a sink in the softmax.
#include "common/host_utils.h"
#include "common/io.cuh"

namespace b200 {

// One warp per token; V: elements per load (4 when every part's width and the pitch allow it).
template <class T, int V>
__global__ void latent_prep_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ wq,
                                   const T* __restrict__ wc, const float* __restrict__ cosT,
                                   const float* __restrict__ sinT, const int* __restrict__ pos, int max_pos,
                                   const long long* __restrict__ slot_mapping, T* __restrict__ cq, T* __restrict__ c,
                                   T* __restrict__ kr, T* __restrict__ cache, long long cache_rows, int T_, int q_rank,
                                   int rank, int rot, float eps) {
  const int lane = threadIdx.x & 31;
  const long long t = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (t >= T_) return;
  const T* row = x + t * ldx;
  long long slot = slot_mapping ? slot_mapping[t] : -1;
  if (slot >= cache_rows) slot = -1;
  T* dst = slot >= 0 ? cache + slot * (rank + rot) : nullptr;
  auto sumsq = [&](const T* p, int n) {
    float s = 0.f;
    for (int i = lane * V; i < n; i += 32 * V) {
      if (V == 4) {
        const float4 v = ld4(p + i);
        s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
      } else {
        s = fmaf(ld1(p + i), ld1(p + i), s);
      }
    }
    return warp_sum(s);
  };
  auto scaled = [&](const T* p, const T* w, float k, int i) {
    if (V == 4) {
      const float4 v = ld4(p + i), ww = ld4(w + i);
      return make_float4(v.x * k * ww.x, v.y * k * ww.y, v.z * k * ww.z, v.w * k * ww.w);
    }
    return make_float4(ld1(p + i) * k * ld1(w + i), 0.f, 0.f, 0.f);
  };
  auto put = [&](T* p, float4 v) {
    if (V == 4) st4(p, v);
    else st1(p, v.x);
  };
  const float sq = sumsq(row, q_rank), sc = sumsq(row + q_rank, rank);
  const float kq = 1.f / sqrtf(sq / q_rank + eps), kc = 1.f / sqrtf(sc / rank + eps);
  for (int i = lane * V; i < q_rank; i += 32 * V) put(cq + t * q_rank + i, scaled(row, wq, kq, i));
  row += q_rank;
  for (int i = lane * V; i < rank; i += 32 * V) {
    const float4 v = scaled(row, wc, kc, i);
    if (c) put(c + t * rank + i, v);
    if (dst) put(dst + i, v);
  }
  row += rank;
  const int p = min(max(pos[t], 0), max_pos - 1);
  for (int i = lane; i < rot / 2; i += 32) {
    const float cs = cosT[static_cast<long long>(p) * (rot / 2) + i], sn = sinT[static_cast<long long>(p) * (rot / 2) + i];
    const float u = ld1(row + 2 * i), v = ld1(row + 2 * i + 1);
    const float a = u * cs - v * sn, b = v * cs + u * sn;
    if (kr) { st1(kr + t * rot + 2 * i, a); st1(kr + t * rot + 2 * i + 1, b); }
    if (dst) { st1(dst + rank + 2 * i, a); st1(dst + rank + 2 * i + 1, b); }
  }
}

__device__ __forceinline__ float2 ld_pair(const float* p) { return make_float2(p[0], p[1]); }
__device__ __forceinline__ float2 ld_pair(const __nv_bfloat16* p) {  // 4-byte aligned
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void st_pair(float* p, float a, float b) { p[0] = a; p[1] = b; }
__device__ __forceinline__ void st_pair(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// One block per token; PAIR: pairs are aligned to their size (even pitch, head stride and offset).
template <class T, bool PAIR>
__global__ void rope_pairs_kernel(T* __restrict__ x, long long ldx, int H, int head_stride, int offset, int half,
                                  const float* __restrict__ cosT, const float* __restrict__ sinT,
                                  const int* __restrict__ pos, int max_pos) {
  const long long t = blockIdx.x;
  const int p = min(max(pos[t], 0), max_pos - 1);
  const float* cr = cosT + static_cast<long long>(p) * half;
  const float* sr = sinT + static_cast<long long>(p) * half;
  T* row = x + t * ldx + offset;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, e = i - h * half;
    T* q = row + static_cast<long long>(h) * head_stride + 2 * e;
    const float2 uv = PAIR ? ld_pair(q) : make_float2(ld1(q), ld1(q + 1));
    const float a = uv.x * cr[e] - uv.y * sr[e], b = uv.y * cr[e] + uv.x * sr[e];
    if (PAIR) {
      st_pair(q, a, b);
    } else {
      st1(q, a);
      st1(q + 1, b);
    }
  }
}

// One block per token; warp 0 takes the latent and the shared key part, the others (or, in a block of one warp, warp 0 as
// well) the heads' rotated parts.
template <class T, int V, bool PAIR>
__global__ void latent_qkv_prep_kernel(T* __restrict__ x, long long ldx, int H, int D, const T* __restrict__ wc,
                                       const float* __restrict__ cosT, const float* __restrict__ sinT,
                                       const int* __restrict__ pos, int max_pos,
                                       const long long* __restrict__ slot_mapping, T* __restrict__ c,
                                       T* __restrict__ kr, T* __restrict__ cache, long long cache_rows, int rank,
                                       int rot, float eps) {
  const long long t = blockIdx.x;
  const int half = rot >> 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = min(max(pos[t], 0), max_pos - 1);
  const float* cr = cosT + static_cast<long long>(p) * half;
  const float* sr = sinT + static_cast<long long>(p) * half;
  T* row = x + t * ldx;
  if (warp == 0) {
    long long slot = slot_mapping ? slot_mapping[t] : -1;
    if (slot >= cache_rows) slot = -1;
    T* dst = slot >= 0 ? cache + slot * (rank + rot) : nullptr;
    const T* lat = row + static_cast<long long>(H) * (D + rot);
    float s = 0.f;
    for (int i = lane * V; i < rank; i += 32 * V) {
      if (V == 4) {
        const float4 v = ld4(lat + i);
        s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
      } else {
        s = fmaf(ld1(lat + i), ld1(lat + i), s);
      }
    }
    const float k = 1.f / sqrtf(warp_sum(s) / rank + eps);
    for (int i = lane * V; i < rank; i += 32 * V) {
      if (V == 4) {
        const float4 v = ld4(lat + i), w = ld4(wc + i);
        const float4 y = make_float4(v.x * k * w.x, v.y * k * w.y, v.z * k * w.z, v.w * k * w.w);
        if (c) st4(c + t * rank + i, y);
        if (dst) st4(dst + i, y);
      } else {
        const float y = ld1(lat + i) * k * ld1(wc + i);
        if (c) st1(c + t * rank + i, y);
        if (dst) st1(dst + i, y);
      }
    }
    lat += rank;
    for (int i = lane; i < half; i += 32) {
      const float u = ld1(lat + 2 * i), v = ld1(lat + 2 * i + 1);
      const float a = u * cr[i] - v * sr[i], b = v * cr[i] + u * sr[i];
      if (kr) { st1(kr + t * rot + 2 * i, a); st1(kr + t * rot + 2 * i + 1, b); }
      if (dst) { st1(dst + rank + 2 * i, a); st1(dst + rank + 2 * i + 1, b); }
    }
    if (blockDim.x > 32) return;
  }
  const int first = blockDim.x > 32 ? threadIdx.x - 32 : threadIdx.x;
  const int step = blockDim.x > 32 ? blockDim.x - 32 : blockDim.x;
  if (V == 4 && PAIR && !(half & 1) && !(D & 3)) {  // two pairs at a time
    for (int i = first; i < H * (half >> 1); i += step) {
      const int h = i / (half >> 1), e = (i - h * (half >> 1)) * 2;
      T* q = row + static_cast<long long>(h) * (D + rot) + D + 2 * e;
      const float4 v = ld4(q);
      const float2 cs = *reinterpret_cast<const float2*>(cr + e), sn = *reinterpret_cast<const float2*>(sr + e);
      st4(q, make_float4(v.x * cs.x - v.y * sn.x, v.y * cs.x + v.x * sn.x, v.z * cs.y - v.w * sn.y, v.w * cs.y + v.z * sn.y));
    }
    return;
  }
  for (int i = first; i < H * half; i += step) {
    const int h = i / half, e = i - h * half;
    T* q = row + static_cast<long long>(h) * (D + rot) + D + 2 * e;
    const float2 uv = PAIR ? ld_pair(q) : make_float2(ld1(q), ld1(q + 1));
    const float a = uv.x * cr[e] - uv.y * sr[e], b = uv.y * cr[e] + uv.x * sr[e];
    if (PAIR) {
      st_pair(q, a, b);
    } else {
      st1(q, a);
      st1(q + 1, b);
    }
  }
}

struct AttendArgs {
  const void *qa, *qb;             // query parts: [rows][ld] + h * head stride
  long long ldqa, ldqb;
  int hqa, hqb;
  const void *ka, *kb, *v;         // key parts and values: [rows][ld] + h * head stride (0: shared by the heads)
  long long ldka, ldkb, ldv;
  int hka, hkb, hv;
  int da, db, dv;                  // widths
  const int* seq_start;            // packed: first row of the query's sequence per query row [n]; paged: null
  const int* kv_len;               // visible keys per query row [n]
  const int* block_table;          // paged: [n, max_blocks]; else null
  int max_blocks, block_size;
  float* o_part;                   // [n, H, nsplit, dv] when nsplit > 1
  float* ml_part;                  // [n, H, nsplit, 2]
  void* out;                       // [n][ldo] + h * dv
  long long ldo;
  int H, nsplit;
  float scale;
  int window;                      // a query sees its last `window` keys; 0: all of them
  const void* gate;                // null, or [n][ldg]: head h's result is multiplied by sigmoid(gate[h])
  long long ldg;
  int group;                       // query heads per key / value head (head strides of keys and values count those)
  int page_rows;                   // paged: key rows per page, a multiple of block_size (the heads' rows follow each other)
  int keep;                        // with a window: the first `keep` keys are always visible
  float softcap;                   // score <- softcap * tanh(score / softcap); 0: none
  const void* sink;                // null, or [H]: exp(sink[h]) joins head h's denominator
  const void* sig_bias;            // null: softmax; else [H]: weights are sigmoid(score + sig_bias[h]), not normalised
};

// The factor on a head's accumulators from their reference m and sum l, with the sink's term.
__device__ __forceinline__ float attend_factor(float m, float l, const float* sink) {
  float f = 1.f;
  if (sink) {
    const float mn = fmaxf(m, *sink);
    f = m == -INFINITY ? 0.f : expf(m - mn);
    l = l * f + expf(*sink - mn);
  }
  return l > 0.f ? f / l : 0.f;
}

// grid (n query rows, ceil(H / warps), nsplit)
template <class T>
__global__ void attend_kernel(AttendArgs a) {
  extern __shared__ float sm[];
  const int nw = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * nw + warp;
  const int dq = a.da + a.db;
  float* q = sm + warp * (dq + a.dv);  // this warp's query and accumulator
  float* acc = q + dq;
  if (h >= a.H) return;                // whole warp; no block-wide barrier follows
  const long long r = blockIdx.x;
  const int L = a.kv_len[r];
  const int lo = a.window > 0 ? max(0, L - a.window) : 0;
  const int nk = min(a.keep, lo), n_seen = L - lo + nk;  // kept keys, then those inside the window
  const int per = (n_seen + a.nsplit - 1) / a.nsplit, hg = h / a.group;
  const int k0 = blockIdx.z * per, k1 = min(n_seen, k0 + per);
  for (int i = lane; i < a.da; i += 32) q[i] = ld1(static_cast<const T*>(a.qa) + r * a.ldqa + h * a.hqa + i);
  for (int i = lane; i < a.db; i += 32) q[a.da + i] = ld1(static_cast<const T*>(a.qb) + r * a.ldqb + h * a.hqb + i);
  for (int i = lane; i < a.dv; i += 32) acc[i] = 0.f;
  __syncwarp();
  const long long first = a.seq_start ? a.seq_start[r] : 0;
  const int* bt = a.block_table ? a.block_table + r * a.max_blocks : nullptr;
  float m = a.sig_bias ? 0.f : -INFINITY, l = 0.f;
  const float sig = a.sig_bias ? ld1(static_cast<const T*>(a.sig_bias) + h) : 0.f;
  for (int kb = k0; kb < k1; kb += 32) {
    const int i_seen = kb + lane, j = i_seen < nk ? i_seen : i_seen + lo - nk;
    long long row = 0;
    float s = -INFINITY;
    if (i_seen < k1) {
      row = bt ? static_cast<long long>(bt[j / a.block_size]) * a.page_rows + j % a.block_size : first + j;
      const T* ka = static_cast<const T*>(a.ka) + row * a.ldka + static_cast<long long>(hg) * a.hka;
      const T* kp = static_cast<const T*>(a.kb) + row * a.ldkb + static_cast<long long>(hg) * a.hkb;
      float d = 0.f;
      for (int i = 0; i < a.da; ++i) d = fmaf(q[i], ld1(ka + i), d);
      for (int i = 0; i < a.db; ++i) d = fmaf(q[a.da + i], ld1(kp + i), d);
      s = d * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    }
    float sc = 1.f, p;
    if (a.sig_bias) {
      p = i_seen < k1 ? 1.f / (1.f + expf(-(s + sig))) : 0.f;
    } else {
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float mn = fmaxf(m, mx);
      sc = m == -INFINITY ? 0.f : expf(m - mn);
      p = i_seen < k1 ? expf(s - mn) : 0.f;
      l = l * sc + warp_sum(p);
      m = mn;
    }
    const int n = min(32, k1 - kb);
    for (int i0 = 0; i0 < a.dv; i0 += 32) {
      const int i = i0 + lane;
      float t = 0.f;
      for (int e = 0; e < n; ++e) {
        const long long rr = __shfl_sync(0xffffffffu, row, e);
        const float pe = __shfl_sync(0xffffffffu, p, e);
        if (i < a.dv) t = fmaf(pe, ld1(static_cast<const T*>(a.v) + rr * a.ldv + static_cast<long long>(hg) * a.hv + i), t);
      }
      if (i < a.dv) acc[i] = fmaf(acc[i], sc, t);
    }
  }
  if (a.nsplit == 1) {
    const float sink = a.sink ? ld1(static_cast<const T*>(a.sink) + h) : 0.f;
    float inv = a.sig_bias ? 1.f : attend_factor(m, l, a.sink ? &sink : nullptr);
    if (a.gate) inv *= sigmoid_as(ld1(static_cast<const T*>(a.gate) + r * a.ldg + h), static_cast<const T*>(nullptr));
    for (int i = lane; i < a.dv; i += 32)
      st1(static_cast<T*>(a.out) + r * a.ldo + static_cast<long long>(h) * a.dv + i, acc[i] * inv);
  } else {
    const long long u = (r * a.H + h) * a.nsplit + blockIdx.z;
    for (int i = lane; i < a.dv; i += 32) a.o_part[u * a.dv + i] = acc[i];
    if (lane == 0) { a.ml_part[2 * u] = m; a.ml_part[2 * u + 1] = l; }
  }
}

// Merge of split partials.
template <class T>
__global__ void attend_merge_kernel(const float* __restrict__ o_part, const float* __restrict__ ml, T* __restrict__ out,
                                    long long ldo, int H, int nsplit, int dv, const T* __restrict__ gate,
                                    long long ldg, const T* __restrict__ sink, int sigmoid) {
  const long long u = blockIdx.x;
  const long long r = u / H;
  const int h = static_cast<int>(u % H);
  float m = -INFINITY;
  for (int s = 0; s < nsplit; ++s) m = fmaxf(m, ml[(u * nsplit + s) * 2]);
  float l = 0.f;
  for (int s = 0; s < nsplit; ++s) {
    const float ms = ml[(u * nsplit + s) * 2];
    if (ms != -INFINITY) l += ml[(u * nsplit + s) * 2 + 1] * expf(ms - m);
  }
  const float sv = sink ? ld1(sink + h) : 0.f;
  float inv = sigmoid ? 1.f : attend_factor(m, l, sink ? &sv : nullptr);
  if (gate) inv *= sigmoid_as(ld1(gate + r * ldg + h), gate);
  for (int i = threadIdx.x; i < dv; i += blockDim.x) {
    float t = 0.f;
    for (int s = 0; s < nsplit; ++s) {
      const float ms = ml[(u * nsplit + s) * 2];
      if (ms != -INFINITY) t = fmaf(o_part[(u * nsplit + s) * dv + i], expf(ms - m), t);
    }
    st1(out + r * ldo + static_cast<long long>(h) * dv + i, t * inv);
  }
}

// Launches the attention and, for several splits, their merge.
static int launch_attend(const AttendArgs& a, int n, int fp32, cudaStream_t stream) {
  const int H = a.H, nsplit = a.nsplit;
  int nw = H < 4 ? H : 4;
  const size_t per_warp = static_cast<size_t>(a.da + a.db + a.dv) * sizeof(float);
  while (nw > 1 && per_warp * nw > 48 * 1024) nw >>= 1;
  const size_t smem = per_warp * nw;
  if (smem > 48 * 1024) return -100;
  dim3 grid(n, (H + nw - 1) / nw, nsplit);
  if (fp32) attend_kernel<float><<<grid, nw * 32, smem, stream>>>(a);
  else attend_kernel<__nv_bfloat16><<<grid, nw * 32, smem, stream>>>(a);
  B200_CHECK(cudaGetLastError());
  if (nsplit > 1) {
    if (fp32)
      attend_merge_kernel<float><<<n * H, 128, 0, stream>>>(a.o_part, a.ml_part, (float*)a.out, a.ldo, H, nsplit, a.dv,
                                                            (const float*)a.gate, a.ldg, (const float*)a.sink, a.sig_bias != nullptr);
    else
      attend_merge_kernel<__nv_bfloat16><<<n * H, 128, 0, stream>>>(
          a.o_part, a.ml_part, (__nv_bfloat16*)a.out, a.ldo, H, nsplit, a.dv, (const __nv_bfloat16*)a.gate, a.ldg,
          (const __nv_bfloat16*)a.sink, a.sig_bias != nullptr);
    B200_CHECK(cudaGetLastError());
  }
  return 0;
}

}  // namespace b200

extern "C" {

// x [T][ldx]: [q_rank | rank | rot]. Tables [max_pos, rot / 2]. c, kr, slot_mapping + cache may be null.
int b200_latent_prep(const void* x, long long ldx, const void* wq, const void* wc, const float* cosT, const float* sinT,
                     const int* pos, int max_pos, const long long* slot_mapping, void* cq, void* c, void* kr,
                     void* cache, long long cache_rows, int T, int q_rank, int rank, int rot, float eps, int fp32,
                     cudaStream_t stream) {
  using namespace b200;
  if (T <= 0) return 0;
  if (rot & 1) return -100;
  const bool v4 = q_rank % 4 == 0 && rank % 4 == 0 && rot % 4 == 0 && ldx % 4 == 0;
  const unsigned grid = (T + 7) / 8;
#define B200_LP(T_, V_)                                                                                             \
  latent_prep_kernel<T_, V_><<<grid, 256, 0, stream>>>((const T_*)x, ldx, (const T_*)wq, (const T_*)wc, cosT, sinT, \
                                                       pos, max_pos, slot_mapping, (T_*)cq, (T_*)c, (T_*)kr,        \
                                                       (T_*)cache, cache_rows, T, q_rank, rank, rot, eps)
  if (fp32) { if (v4) B200_LP(float, 4); else B200_LP(float, 1); }
  else { if (v4) B200_LP(__nv_bfloat16, 4); else B200_LP(__nv_bfloat16, 1); }
#undef B200_LP
  B200_CHECK(cudaGetLastError());
  return 0;
}

// x [T][ldx]: [H * (D + rot) | rank | rot | ...]; the heads' last rot columns are rotated in place. c, kr, slot_mapping +
// cache may be null.
int b200_latent_qkv_prep(void* x, long long ldx, int H, int D, const void* wc, const float* cosT, const float* sinT,
                         const int* pos, int max_pos, const long long* slot_mapping, void* c, void* kr, void* cache,
                         long long cache_rows, int T, int rank, int rot, float eps, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0) return 0;
  if ((rot & 1) || H < 1 || D < 0) return -100;
  const long long q = static_cast<long long>(H) * (D + rot);
  const bool v4 = q % 4 == 0 && rank % 4 == 0 && rot % 4 == 0 && ldx % 4 == 0;
  const bool pair = !((ldx | D) & 1);
  int block = 64;
  while (block < 256 && block < 32 + H * (rot / 2)) block <<= 1;
#define B200_LQ(T_, V_, P_)                                                                                         \
  latent_qkv_prep_kernel<T_, V_, P_><<<T, block, 0, stream>>>((T_*)x, ldx, H, D, (const T_*)wc, cosT, sinT, pos,    \
                                                              max_pos, slot_mapping, (T_*)c, (T_*)kr, (T_*)cache,   \
                                                              cache_rows, rank, rot, eps)
#define B200_LQV(T_)                                                                                                \
  if (v4) { if (pair) B200_LQ(T_, 4, true); else B200_LQ(T_, 4, false); }                                           \
  else { if (pair) B200_LQ(T_, 1, true); else B200_LQ(T_, 1, false); }
  if (fp32) { B200_LQV(float) } else { B200_LQV(__nv_bfloat16) }
#undef B200_LQV
#undef B200_LQ
  B200_CHECK(cudaGetLastError());
  return 0;
}

// Rotates columns [offset, offset + dims) of every head of x [rows][ldx] in place; tables [max_pos, dims / 2].
int b200_rope_pairs(void* x, long long ldx, int H, int head_stride, int offset, int dims, const float* cosT,
                    const float* sinT, const int* pos, int max_pos, long long rows, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (rows <= 0 || dims <= 0) return 0;
  if (dims & 1) return -100;
  const bool pair = !((ldx | head_stride | offset) & 1);
  int block = 64;
  while (block < 256 && block < H * (dims / 2)) block <<= 1;
#define B200_RP(T_, P_)                                                                                             \
  rope_pairs_kernel<T_, P_><<<(unsigned)rows, block, 0, stream>>>((T_*)x, ldx, H, head_stride, offset, dims / 2,    \
                                                                  cosT, sinT, pos, max_pos)
  if (fp32) { if (pair) B200_RP(float, true); else B200_RP(float, false); }
  else { if (pair) B200_RP(__nv_bfloat16, true); else B200_RP(__nv_bfloat16, false); }
#undef B200_RP
  B200_CHECK(cudaGetLastError());
  return 0;
}

// General softmax attention; see AttendArgs for the meaning of every operand. n query rows.
int b200_attend(const void* qa, long long ldqa, int hqa, const void* qb, long long ldqb, int hqb, const void* ka,
                long long ldka, int hka, const void* kb, long long ldkb, int hkb, const void* v, long long ldv, int hv,
                int da, int db, int dv, const int* seq_start, const int* kv_len, const int* block_table, int max_blocks,
                int block_size, float* o_part, float* ml_part, void* out, long long ldo, int n, int H, int nsplit,
                float scale, int window, const void* gate, long long ldg, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (n <= 0) return 0;
  AttendArgs a{qa, qb, ldqa, ldqb, hqa, hqb, ka, kb, v, ldka, ldkb, ldv, hka, hkb, hv, da, db, dv, seq_start, kv_len,
               block_table, max_blocks, block_size, o_part, ml_part, out, ldo, H, nsplit, scale, window,
               gate, ldg, 1, block_size, 0, 0.f, nullptr, nullptr};
  return launch_attend(a, n, fp32, stream);
}

// Grouped-query form: q [n][ldq] + h * hq; keys and values per kv head g at g * hk / g * hv of a row. Packed (seq_start): rows
// of the batch. Paged (block_table): page p's rows start at p * page_rows, and hk, hv lead from one head's rows of a page
// to the next one's. window, keep, softcap: 0 for none; sink [H], gate [n][ldg]: null for none; sig_bias: null, or [H] for
// sigmoid weights (without a sink).
int b200_attend_grouped(const void* q, long long ldq, int hq, const void* k, long long ldk, int hk, const void* v,
                        long long ldv, int hv, int d, int dv, const int* seq_start, const int* kv_len,
                        const int* block_table, int max_blocks, int block_size, int page_rows, float* o_part,
                        float* ml_part, void* out, long long ldo, int n, int H, int G, int nsplit, float scale, int window,
                        int keep, float softcap, const void* sink, const void* gate, long long ldg, const void* sig_bias,
                        int fp32, cudaStream_t stream) {
  using namespace b200;
  if (n <= 0) return 0;
  if (G < 1 || H % G || block_size < 1 || (sink && sig_bias)) return -100;
  AttendArgs a{q, nullptr, ldq, 0, hq, 0, k, nullptr, v, ldk, 0, ldv, hk, 0, hv, d, 0, dv, seq_start, kv_len, block_table,
               max_blocks, block_size, o_part, ml_part, out, ldo, H, nsplit, scale, window, gate, ldg, H / G, page_rows,
               keep, softcap, sink, sig_bias};
  return launch_attend(a, n, fp32, stream);
}

}  // extern "C"
