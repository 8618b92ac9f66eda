// Prefill of the recurrences of matrix_state.cu on tensor cores, for bf16 models with key width <= 128.
//
// Sequences are walked in blocks of 16 tokens. With G_i the sum of the log decays of a block up to token i, everything that
// does not depend on the state is prepared for all blocks at once (state_prep_kernel):
//
//   delta rule   A_ij = beta_i e^(G_i - G_j) (k_i . k_j), j < i;   T = (I + A)^-1 diag(beta);   P_ij = e^(G_i - G_j) (q_i . k_j)
//                U = T (V - diag(e^G) K S),   O = diag(e^G) Q S + P U,   S <- e^G16 S + sum_j e^(G16 - G_j) k_j u_j^T
//   mLSTM        P_ij = e^(G_i - G_j + i_j - m_i) (q_i . k_j);   U = V;   the state's factors carry the running maximum alike
//
// so that the walk (state_chunk_kernel) has only products with the state and two with 16 x 16 matrices. One CTA walks a
// sequence for one head and up to 128 value columns; the state stays, transposed, in the accumulators of the warps (warp w: value
// columns 16w .. 16w + 15, all key channels) and is its own operand, and so are W = V - .. and U: the walk needs no exchange
// between warps. q, k and v are bf16 numbers and enter the products exactly, with the factors that make them unit vectors,
// scales and decays applied to the products; fp32 operands (state, W, U, T, P) enter as two bf16 terms.
//
// Few long sequences would leave most SMs idle. The columns of a state are independent, so a head's may be spread over several
// CTAs (its norm is then another kernel's). An mLSTM's state only decays by a number from token to token, so its sequences are
// instead cut into segments: a first pass computes every segment's end state from zero and its decay (the running maximum is
// that of the whole sequence in both passes), a scan over a sequence's segments turns them into the states that the segments
// start from, and the second pass computes the outputs.
//
// The output of a block is normed and gated one block later, behind the barrier that the next block needs anyway.
#include "common/host_utils.h"
#include "common/mma16.cuh"
#include "common/scan_inputs.cuh"
#include "common/state_inputs.cuh"

namespace b200 {

// What the walk reads per (block, head), in floats: P and T as operand fragments (hi, lo; 8 words per lane), then factors per
// token: of K S inside W, of Q S, of the rows that enter the state; the sum of a row of P and e^-m (mLSTM); the state's decay,
// m at the block's end.
enum : int { kRecP = 0, kRecT = 256, kRecK = 512, kRecQ = 528, kRecU = 544, kRecSum = 560, kRecFloor = 576, kRecS = 592, kRecM = 593, kRec = 608 };
constexpr int kMaxThreads = 256, kMaxTokens = 4;  // running maximum: threads, tokens per thread

// ---- mLSTM: log decay, log input gate and running maximum of every token, [T, H, 3]. m_t = max(f_t + m_(t-1), i_t) is the
// composition of maps x -> max(a + x, b), so a chunk of tokens is scanned in parallel. grid (sequences, heads)
template <class T>
__global__ void __launch_bounds__(kMaxThreads) state_running_max_kernel(StateArgs a, const int* __restrict__ cu,
                                                                        float* __restrict__ out) {
  __shared__ float wa[kMaxThreads / 32], wb[kMaxThreads / 32];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = cu[blockIdx.x], t1 = cu[blockIdx.x + 1];
  float m = 0.f;
  for (int base = t0; base < t1; base += kMaxThreads * kMaxTokens) {
    float f[kMaxTokens], g[kMaxTokens], A = 0.f, B = -INFINITY;
#pragma unroll
    for (int e = 0; e < kMaxTokens; ++e) {
      const int t = base + tid * kMaxTokens + e;
      f[e] = 0.f;
      g[e] = -INFINITY;
      if (t < t1) head_gates<T>(a, t, h, f[e], g[e]);
    }
#pragma unroll
    for (int e = 0; e < kMaxTokens; ++e) {
      B = fmaxf(f[e] + B, g[e]);
      A += f[e];
    }
    float sa = A, sb = B;  // inclusive scan over the warp
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, sa, o), pb = __shfl_up_sync(0xffffffffu, sb, o);
      if (lane >= o) {
        sb = fmaxf(sa + pb, sb);
        sa += pa;
      }
    }
    __syncthreads();
    if (lane == 31) {
      wa[warp] = sa;
      wb[warp] = sb;
    }
    __syncthreads();
    float x = m, end = m;  // running maximum ahead of this warp, and behind the chunk
    for (int w = 0; w < kMaxThreads / 32; ++w) {
      end = fmaxf(wa[w] + end, wb[w]);
      if (w < warp) x = fmaxf(wa[w] + x, wb[w]);
    }
    const float pa = __shfl_up_sync(0xffffffffu, sa, 1), pb = __shfl_up_sync(0xffffffffu, sb, 1);
    if (lane > 0) x = fmaxf(pa + x, pb);
#pragma unroll
    for (int e = 0; e < kMaxTokens; ++e) {
      const int t = base + tid * kMaxTokens + e;
      x = fmaxf(f[e] + x, g[e]);
      if (t < t1) {
        float* o = out + (static_cast<long long>(t) * a.H + h) * 3;
        o[0] = f[e];
        o[1] = g[e];
        o[2] = x;
      }
    }
    m = end;
  }
}

__device__ __forceinline__ uint32_t st_s32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void st_cp16(void* dst, const void* src, int bytes) {  // bytes < 16: the rest is zero
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(st_s32(dst)), "l"(src), "r"(bytes) : "memory");
}

// ---- Everything of a block that does not depend on the state. One warp per (block, head).
constexpr int kPrepWarps = 4;
template <int ND>
struct PrepSmem {
  static constexpr int P = ND * 16 + 8;  // pitch of a row
  __nv_bfloat16 q[16 * P], k[16 * P];
  float A[16 * 17], T[16 * 17], beta[16], rk[16], rq[16], li[16], m[16];
  double G[16];
};

template <int ND, bool DELTA>
__global__ void __launch_bounds__(kPrepWarps * 32) state_prep_kernel(StateArgs a, const int4* __restrict__ blocks, int n_blocks,
                                                                     const float* __restrict__ run_max,
                                                                     float* __restrict__ rec) {
  using SM = PrepSmem<ND>;
  constexpr int P = SM::P;
  __shared__ __align__(16) uint8_t raw[kPrepWarps * sizeof(SM)];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long u = static_cast<long long>(blockIdx.x) * kPrepWarps + warp;
  if (u >= static_cast<long long>(n_blocks) * a.H) return;  // whole warps; no block-wide barrier follows
  SM& sm = reinterpret_cast<SM*>(raw)[warp];
  const int h = static_cast<int>(u % a.H), hk = h / (a.H / a.G), D = a.D;
  const int4 blk = blocks[u / a.H];  // first token, tokens, sequence, first block of it
  const __nv_bfloat16* q0 = static_cast<const __nv_bfloat16*>(a.qkv) + static_cast<long long>(blk.x) * a.ldq + hk * D;
  const __nv_bfloat16* k0 = q0 + a.G * D;
  // ---- gates; padding tokens neither decay nor write
  const int tok = lane & 15;
  float lf = 0.f, put = DELTA ? 0.f : -INFINITY, m = 0.f;
  if (tok < blk.y) {
    if constexpr (DELTA) {
      head_gates<__nv_bfloat16>(a, blk.x + tok, h, lf, put);
    } else {
      const float* r = run_max + (static_cast<long long>(blk.x + tok) * a.H + h) * 3;
      lf = r[0];
      put = r[1];
      m = r[2];
    }
  }
  const bool wide = !((D | a.ldq) & 7) && !(reinterpret_cast<uintptr_t>(a.qkv) & 15);
  if (wide) {
    const uint4 zero = make_uint4(0, 0, 0, 0);
    uint4 x[ND], y[ND];  // all loads go out together
#pragma unroll
    for (int j = 0; j < ND; ++j) {
      const int i = lane + 32 * j, t = i / (ND * 2), c = (i % (ND * 2)) * 8;
      const bool in = t < blk.y && c < D;
      x[j] = in ? *reinterpret_cast<const uint4*>(q0 + t * a.ldq + c) : zero;
      y[j] = in ? *reinterpret_cast<const uint4*>(k0 + t * a.ldq + c) : zero;
    }
#pragma unroll
    for (int j = 0; j < ND; ++j) {
      const int i = lane + 32 * j, t = i / (ND * 2), c = (i % (ND * 2)) * 8;
      *reinterpret_cast<uint4*>(sm.q + t * P + c) = x[j];
      *reinterpret_cast<uint4*>(sm.k + t * P + c) = y[j];
    }
  } else {
    for (int i = lane; i < 16 * ND * 16; i += 32) {
      const int t = i / (ND * 16), c = i % (ND * 16);
      const bool in = t < blk.y && c < D;
      sm.q[t * P + c] = in ? q0[t * a.ldq + c] : __float2bfloat16(0.f);
      sm.k[t * P + c] = in ? k0[t * a.ldq + c] : __float2bfloat16(0.f);
    }
  }
  double G = 0.0;
#pragma unroll
  for (int s = 0; s < 16; ++s) {
    const float x = __shfl_sync(0xffffffffu, lf, s);
    if (s <= tok) G += static_cast<double>(x);
  }
  const float scale = 1.f / sqrtf(static_cast<float>(D));
  __syncwarp();
  float rk = 1.f, rq = scale;
  if constexpr (DELTA) {  // a lane takes half of a row
    float sq = 0.f, sk = 0.f;
    for (int c = (lane >> 4) * ND * 8; c < ((lane >> 4) + 1) * ND * 8; c += 4) {
      const float4 x = ld4(sm.q + tok * P + c), y = ld4(sm.k + tok * P + c);
      sq = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, sq))));
      sk = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, fmaf(y.w, y.w, sk))));
    }
    sq += __shfl_xor_sync(0xffffffffu, sq, 16);
    sk += __shfl_xor_sync(0xffffffffu, sk, 16);
    rq = scale / sqrtf(sq + 1e-6f);
    rk = 1.f / sqrtf(sk + 1e-6f);
  }
  if (lane < 16) {
    sm.G[tok] = G;
    sm.rk[tok] = rk;
    sm.rq[tok] = rq;
    if constexpr (DELTA) sm.beta[tok] = put;
    sm.li[tok] = put;
    sm.m[tok] = m;
  }
  __syncwarp();
  // ---- q . k and k . k
  const int g = lane >> 2, t = lane & 3;
  float qk[2][4], kk[2][4];
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) qk[n][c] = kk[n][c] = 0.f;
  const int r8 = (lane & 7) + ((lane >> 4) << 3), c8 = ((lane >> 3) & 1) * 8;
  const uint32_t qa = st_s32(sm.q + (lane & 15) * P + (lane >> 4) * 8), ka = st_s32(sm.k + (lane & 15) * P + (lane >> 4) * 8),
                 kb = st_s32(sm.k + r8 * P + c8);
#pragma unroll
  for (int kt = 0; kt < ND; ++kt) {
    uint32_t x[4], b[4];
    ldm_x4(kb + kt * 32, b);
    ldm_x4(qa + kt * 32, x);
    mma_bf16(qk[0], x, b[0], b[1]);
    mma_bf16(qk[1], x, b[2], b[3]);
    if constexpr (DELTA) {
      ldm_x4(ka + kt * 32, x);
      mma_bf16(kk[0], x, b[0], b[1]);
      mma_bf16(kk[1], x, b[2], b[3]);
    }
  }
  float* out = rec + u * kRec;
  float sum[2] = {0.f, 0.f};
  uint32_t hi[4], lo[4];
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {  // row i, columns j, j + 1
      const int i = g + e * 8, j = n * 8 + 2 * t;
      float p[2];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        p[c] = 0.f;
        if (j + c <= i) {
          const float d = static_cast<float>(sm.G[i] - sm.G[j + c]);
          if constexpr (DELTA) {
            const float w = expf(d);
            p[c] = sm.rq[i] * sm.rk[j + c] * w * qk[n][2 * e + c];
            if (j + c < i) sm.A[i * 17 + j + c] = sm.beta[i] * sm.rk[i] * sm.rk[j + c] * w * kk[n][2 * e + c];
          } else {
            p[c] = scale * expf(d + sm.li[j + c] - sm.m[i]) * qk[n][2 * e + c];
          }
        }
        sum[e] += p[c];
      }
      hi[e * 2 + n] = split2(p[0], p[1], lo[e * 2 + n]);
    }
  *reinterpret_cast<uint4*>(out + kRecP + lane * 8) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
  *reinterpret_cast<uint4*>(out + kRecP + lane * 8 + 4) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  const double G16 = __shfl_sync(0xffffffffu, G, 15);
  if constexpr (DELTA) {
    __syncwarp();
    float col[16];  // column `tok` of (I + A)^-1
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) s = fmaf(sm.A[i * 17 + j], col[j], s);
      col[i] = i < tok ? 0.f : (i == tok ? 1.f : -s);
    }
    if (lane < 16) {
#pragma unroll
      for (int i = 0; i < 16; ++i) sm.T[i * 17 + tok] = col[i] * put;
    }
    __syncwarp();
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = g + (e >> 1) * 8, j = 2 * t + (e & 1) * 8;
      hi[e] = split2(sm.T[i * 17 + j], sm.T[i * 17 + j + 1], lo[e]);
    }
    *reinterpret_cast<uint4*>(out + kRecT + lane * 8) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(out + kRecT + lane * 8 + 4) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    if (lane < 16) {
      const float e = expf(static_cast<float>(G));
      out[kRecK + tok] = e * rk;
      out[kRecQ + tok] = e * rq;
      out[kRecU + tok] = tok < blk.y ? expf(static_cast<float>(G16 - G)) * rk : 0.f;
      out[kRecSum + tok] = 0.f;
      out[kRecFloor + tok] = 0.f;
    }
    if (lane == 0) {
      out[kRecS] = expf(static_cast<float>(G16));
      out[kRecM] = 0.f;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
      sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
      if (t == 0) out[kRecSum + g + e * 8] = sum[e];
    }
    const float before = blk.w ? 0.f : run_max[(static_cast<long long>(blk.x - 1) * a.H + h) * 3 + 2];
    const float after = sm.m[blk.y - 1];
    if (lane < 16) {
      const bool in = tok < blk.y;
      out[kRecK + tok] = 0.f;
      out[kRecQ + tok] = in ? scale * expf(static_cast<float>(G) + before - m) : 0.f;
      out[kRecU + tok] = in ? expf(static_cast<float>(G16 - G) + put - after) : 0.f;
      out[kRecFloor + tok] = in ? expf(-m) : 1.f;
    }
    if (lane == 0) {
      out[kRecS] = expf(static_cast<float>(G16) + before - after);
      out[kRecM] = after;
    }
  }
}

// ---- The walk
struct StateChunkArgs {
  const __nv_bfloat16* qkv;   // [T][ldq]: q, k (G * D each) | v (H * Dv)
  long long ldq;
  const __nv_bfloat16* gate;  // [T][ldg], H * Dv
  long long ldg;
  const float* rec;           // [blocks, H, kRec]
  const int4* blocks;
  const int4* segs;           // first block, blocks, sequence, 1 for the last segment of its sequence
  const int* slots;           // may be null
  float *seg_S, *seg_n, *seg_f;  // per segment: [H, D, Dv], [H, D], [H]; the first pass writes, the second reads S and n (null:
                                 // segments are whole sequences)
  float *S, *n, *m;
  const __nv_bfloat16* norm;  // with it y gets the normed and gated heads
  __nv_bfloat16* y;           // [T, H * Dv]
  float* o;                   // without it: the plain outputs
  float eps;
  int H, G, D, Dv, cols;      // cols: value columns per CTA, a multiple of 16 up to 128
};

template <int ND>
struct StateSmem {
  static constexpr int DP = ND * 16, P = DP + 8;
  __nv_bfloat16 q[2][16 * P], k[2][16 * P], v[2][16 * 136];
  float rec[2][kRec];
  float o[2][16 * 132], inv[2][16], n[2][DP];
};

// STATE_ONLY: the first pass over segments
template <int ND, bool DELTA, int WARPS, bool STATE_ONLY>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 8 ? 2 : 3) state_chunk_kernel(const StateChunkArgs a) {
  using SM = StateSmem<ND>;
  constexpr int P = SM::P, PB = P * 2;
  extern __shared__ __align__(16) uint8_t raw[];
  SM& sm = *reinterpret_cast<SM*>(raw);
  const int4 seg = a.segs[blockIdx.x];
  const int seq = seg.z, h = blockIdx.y, vb = blockIdx.z * a.cols, D = a.D, Dv = a.Dv, H = a.H, hk = h / (H / a.G);
  constexpr int nthr = WARPS * 32, nw = WARPS, TPW = 16 / WARPS;  // TPW: tokens of a block whose outputs a warp writes
  const int nv = min(a.cols, Dv - vb);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const bool mma = warp * 16 < nv;
  const int b0 = seg.x, nblk = seg.y;
  if (nblk == 0 || (STATE_ONLY && seg.w)) return;  // (nothing starts from the last segment's end state)
  const int t0 = a.blocks[b0].x, len = a.blocks[b0 + nblk - 1].x + a.blocks[b0 + nblk - 1].y - t0;  // the segment's tokens
  const long long sgh = static_cast<long long>(blockIdx.x) * H + h;
  for (int i = tid; i < static_cast<int>(sizeof(SM) / 16); i += nthr) reinterpret_cast<uint4*>(raw)[i] = make_uint4(0, 0, 0, 0);
  float S[2 * ND][4];
#pragma unroll
  for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) S[i][c] = 0.f;
  const int at_q = hk * D, at_k = (a.G + hk) * D, at_v = 2 * a.G * D + h * Dv + vb;
  const bool wide = !((D | Dv | a.ldq) & 7) && !(reinterpret_cast<uintptr_t>(a.qkv) & 15);
  const int dc = D >> 3, vc = nv >> 3;
  __syncthreads();
  if (!STATE_ONLY && !DELTA && a.seg_S) {
    if (mma) {
#pragma unroll
      for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int d = i * 8 + 2 * t + (c & 1), col = vb + warp * 16 + g + (c >> 1) * 8;
          if (d < D && col < Dv) S[i][c] = a.seg_S[(sgh * D + d) * Dv + col];
        }
    }
    for (int d = tid; d < D; d += nthr) sm.n[0][d] = a.seg_n[sgh * D + d];
  }
  float seg_f = 1.f;
  constexpr int LPT = nthr / 16;  // threads that load a token
  const int ltok = tid / LPT, lc = tid % LPT;
  const float* rec_base = a.rec + (static_cast<long long>(b0) * H + h) * kRec;
  auto load = [&](int b, int st) {
    const int n = len - b * 16;  // tokens from here to the end
    const __nv_bfloat16* x = a.qkv + static_cast<long long>(t0 + b * 16) * a.ldq;
    if (wide) {
      const __nv_bfloat16* row = x + min(ltok, n - 1) * a.ldq;
      const int bytes = ltok < n ? 16 : 0;
#pragma unroll 1
      for (int c = lc; c < dc; c += LPT) {
        st_cp16(&sm.q[st][ltok * P + c * 8], row + at_q + c * 8, bytes);
        st_cp16(&sm.k[st][ltok * P + c * 8], row + at_k + c * 8, bytes);
      }
#pragma unroll 1
      for (int c = lc; c < vc; c += LPT) st_cp16(&sm.v[st][ltok * 136 + c * 8], row + at_v + c * 8, bytes);
    } else {
      const __nv_bfloat16 zero = __float2bfloat16(0.f);
      for (int i = tid; i < 16 * D; i += nthr) {
        const int tok = i / D, c = i - tok * D;
        sm.q[st][tok * P + c] = tok < n ? x[tok * a.ldq + at_q + c] : zero;
        sm.k[st][tok * P + c] = tok < n ? x[tok * a.ldq + at_k + c] : zero;
      }
      for (int i = tid; i < 16 * nv; i += nthr) {
        const int tok = i / nv, c = i - tok * nv;
        sm.v[st][tok * 136 + c] = tok < n ? x[tok * a.ldq + at_v + c] : zero;
      }
    }
    const float* rec = rec_base + static_cast<long long>(b) * H * kRec;
    for (int i = tid; i < kRec / 4; i += nthr)
      if (DELTA || i < kRecT / 4 || i >= kRecK / 4) st_cp16(&sm.rec[st][i * 4], rec + i * 4, 16);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // the norm's weights and the gates of the four columns that this lane writes
  float nw4[4] = {0.f, 0.f, 0.f, 0.f};
  const int oc = lane * 4;
  if (a.norm)
    for (int c = 0; c < 4; ++c)
      if (oc + c < nv) nw4[c] = ld1(a.norm + (DELTA ? 0 : h * Dv) + oc + c);
  const bool v4 = !(Dv & 3), gate4 = v4 && !(a.ldg & 3) && !(reinterpret_cast<uintptr_t>(a.gate) & 7);
  // gates of a block's outputs, fetched a block ahead of their use; bf16 pairs
  uint2 gates[TPW];
  auto fetch_gates = [&](int b) {
#pragma unroll
    for (int e = 0; e < TPW; ++e) {
      const int i = b * 16 + warp + e * nw;
      gates[e] = make_uint2(0, 0);
      if (!a.norm || i >= len || oc >= nv) continue;
      const __nv_bfloat16* gp = a.gate + (t0 + i) * a.ldg + h * Dv + oc;
      if (gate4) {
        gates[e] = *reinterpret_cast<const uint2*>(gp);
      } else {
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        for (int c = 0; c < 4; ++c)
          if (oc + c < nv) f[c] = ld1(gp + c);
        gates[e] = make_uint2(pack2(f[0], f[1]), pack2(f[2], f[3]));
      }
    }
  };
  // normed and gated outputs of a block: tokens over the warps, columns over the lanes
  auto output = [&](int b, int st) {
#pragma unroll
    for (int e = 0; e < TPW; ++e) {
      const int i = warp + e * nw;
      if (b * 16 + i >= len) break;
      float4 v = *reinterpret_cast<const float4*>(&sm.o[st][i * 132 + oc]);
      if (!DELTA) {
        const float f = sm.inv[st][i];
        v.x *= f; v.y *= f; v.z *= f; v.w *= f;
      }
      if (oc >= nv) v.x = 0.f;
      if (oc + 1 >= nv) v.y = 0.f;
      if (oc + 2 >= nv) v.z = 0.f;
      if (oc + 3 >= nv) v.w = 0.f;
      const long long at = (static_cast<long long>(t0 + b * 16 + i) * H + h) * Dv + vb + oc;
      float u[4] = {v.x, v.y, v.z, v.w};
      if (a.norm) {
        const float k = 1.f / sqrtf(warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)))) / nv + a.eps);
        const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gates[e].x)),
                     g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gates[e].y));
        const float gt[4] = {g0.x, g0.y, g1.x, g1.y};
#pragma unroll
        for (int c = 0; c < 4; ++c) u[c] *= k * nw4[c] * out_gate(gt[c], DELTA, a.gate);
      }
      if (v4) {
        if (oc < nv) {
          if (a.norm) st4(a.y + at, make_float4(u[0], u[1], u[2], u[3]));
          else st4(a.o + at, make_float4(u[0], u[1], u[2], u[3]));
        }
      } else {
        for (int c = 0; c < 4 && oc + c < nv; ++c) {
          if (a.norm) st1(a.y + at + c, u[c]);
          else a.o[at + c] = u[c];
        }
      }
    }
  };
  load(0, 0);
  const int r8 = (lane & 7) + ((lane >> 4) << 3), c8 = ((lane >> 3) & 1) * 8;
  for (int b = 0; b < nblk; ++b) {
    const int st = b & 1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this block's inputs are here, the last block's outputs too; every warp has left the block before
    if (b + 1 < nblk) load(b + 1, st ^ 1);
    if (!STATE_ONLY) {
      if (b > 0) output(b - 1, st ^ 1);
      fetch_gates(b);
    }
    const float* rec = sm.rec[st];
    if (STATE_ONLY) seg_f *= rec[kRecS];
    if (!DELTA) {  // 1 / the denominators, then the normaliser behind this block (no one reads that copy before the barrier)
      for (int i = STATE_ONLY ? 16 : warp; i < 16; i += nw) {
        float x = 0.f;
        for (int d = lane; d < D; d += 32) x = fmaf(sm.n[st][d], __bfloat162float(sm.q[st][i * P + d]), x);
        x = fmaf(warp_sum(x), rec[kRecQ + i], rec[kRecSum + i]);
        if (lane == 0) sm.inv[st][i] = 1.f / (fmaxf(fabsf(x), rec[kRecFloor + i]) + 1e-6f);
      }
      for (int d = tid; d < D; d += nthr) {
        float x = rec[kRecS] * sm.n[st][d];
#pragma unroll
        for (int j = 0; j < 16; ++j) x = fmaf(rec[kRecU + j], __bfloat162float(sm.k[st][j * P + d]), x);
        sm.n[st ^ 1][d] = x;
      }
    }
    if (mma) {
      const uint32_t qb = st_s32(sm.q[st]) + r8 * PB + c8 * 2, kb = st_s32(sm.k[st]) + r8 * PB + c8 * 2;
      float ks[2][4], o[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) ks[n][c] = o[n][c] = 0.f;
      // ---- K S and Q S, transposed: [value column, token]
#pragma unroll
      for (int kt = 0; kt < (STATE_ONLY ? 0 : ND); ++kt) {
        uint32_t hi[4], lo[4], bq[4], bk[4];
        hi[0] = split2(S[2 * kt][0], S[2 * kt][1], lo[0]);
        hi[1] = split2(S[2 * kt][2], S[2 * kt][3], lo[1]);
        hi[2] = split2(S[2 * kt + 1][0], S[2 * kt + 1][1], lo[2]);
        hi[3] = split2(S[2 * kt + 1][2], S[2 * kt + 1][3], lo[3]);
        ldm_x4(qb + kt * 32, bq);
        if (DELTA) ldm_x4(kb + kt * 32, bk);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (DELTA) mma_bf16(ks[n], hi, bk[2 * n], bk[2 * n + 1]);
          mma_bf16(o[n], hi, bq[2 * n], bq[2 * n + 1]);
          if (DELTA) mma_bf16(ks[n], lo, bk[2 * n], bk[2 * n + 1]);
          mma_bf16(o[n], lo, bq[2 * n], bq[2 * n + 1]);
        }
      }
      uint32_t vt[4], uh[4], ul[4], xh[4], xl[4];
      ldm_x4_t(st_s32(sm.v[st] + r8 * 136 + warp * 16 + c8), vt);
      float2 fu[2];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const float2 fq = *reinterpret_cast<const float2*>(rec + kRecQ + n * 8 + 2 * t);
        fu[n] = *reinterpret_cast<const float2*>(rec + kRecU + n * 8 + 2 * t);
        o[n][0] *= fq.x; o[n][1] *= fq.y; o[n][2] *= fq.x; o[n][3] *= fq.y;
      }
      if constexpr (DELTA) {
        uint32_t wh[4], wl[4], th[4], tl[4];
        *reinterpret_cast<uint4*>(th) = *reinterpret_cast<const uint4*>(rec + kRecT + lane * 8);
        *reinterpret_cast<uint4*>(tl) = *reinterpret_cast<const uint4*>(rec + kRecT + lane * 8 + 4);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const float2 fk = *reinterpret_cast<const float2*>(rec + kRecK + n * 8 + 2 * t);
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vt[n * 2 + r]));
            wh[n * 2 + r] = split2(fmaf(-fk.x, ks[n][2 * r], v.x), fmaf(-fk.y, ks[n][2 * r + 1], v.y), wl[n * 2 + r]);
          }
        }
        float u[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
#pragma unroll
          for (int c = 0; c < 4; ++c) u[n][c] = 0.f;
          mma_bf16(u[n], wh, th[2 * n], th[2 * n + 1]);
          mma_bf16(u[n], wl, th[2 * n], th[2 * n + 1]);
          mma_bf16(u[n], wh, tl[2 * n], tl[2 * n + 1]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            uh[n * 2 + r] = split2(u[n][2 * r], u[n][2 * r + 1], ul[n * 2 + r]);
            xh[n * 2 + r] = split2(fu[n].x * u[n][2 * r], fu[n].y * u[n][2 * r + 1], xl[n * 2 + r]);
          }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vt[e]));
          uh[e] = vt[e];
          xh[e] = split2(fu[e >> 1].x * v.x, fu[e >> 1].y * v.y, xl[e]);
        }
      }
      // ---- outputs of the block itself
      if constexpr (!STATE_ONLY) {
        uint32_t ph[4], pl[4];
        *reinterpret_cast<uint4*>(ph) = *reinterpret_cast<const uint4*>(rec + kRecP + lane * 8);
        *reinterpret_cast<uint4*>(pl) = *reinterpret_cast<const uint4*>(rec + kRecP + lane * 8 + 4);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16(o[n], uh, ph[2 * n], ph[2 * n + 1]);
          if (DELTA) mma_bf16(o[n], ul, ph[2 * n], ph[2 * n + 1]);
          mma_bf16(o[n], uh, pl[2 * n], pl[2 * n + 1]);
#pragma unroll
          for (int c = 0; c < 4; ++c) sm.o[st][(n * 8 + 2 * t + (c & 1)) * 132 + warp * 16 + g + (c >> 1) * 8] = o[n][c];
        }
      }
      // ---- the state behind the block
      const float fs = rec[kRecS];
      const uint32_t ka = st_s32(sm.k[st]) + (lane & 15) * PB + (lane >> 4) * 16;
#pragma unroll
      for (int nt = 0; nt < ND; ++nt) {
        uint32_t bk[4];
        ldm_x4_t(ka + nt * 32, bk);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float(&c)[4] = S[2 * nt + n];
          c[0] *= fs; c[1] *= fs; c[2] *= fs; c[3] *= fs;
          mma_bf16(c, xh, bk[2 * n], bk[2 * n + 1]);
          mma_bf16(c, xl, bk[2 * n], bk[2 * n + 1]);
        }
      }
    }
  }
  __syncthreads();
  if (!STATE_ONLY) output(nblk - 1, (nblk - 1) & 1);
  const int slot = !STATE_ONLY && a.slots && seg.w ? a.slots[seq] : -1;
  if (!STATE_ONLY && slot < 0) return;
  const long long sh = STATE_ONLY ? sgh : static_cast<long long>(slot) * H + h;
  float *dS = STATE_ONLY ? a.seg_S : a.S, *dn = STATE_ONLY ? a.seg_n : a.n;
  if (mma) {
#pragma unroll
    for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int d = i * 8 + 2 * t + (c & 1), col = vb + warp * 16 + g + (c >> 1) * 8;
        if (d < D && col < Dv) dS[(sh * D + d) * Dv + col] = S[i][c];
      }
  }
  if (!DELTA && blockIdx.z == 0) {
    for (int d = tid; d < D; d += nthr) dn[sh * D + d] = sm.n[nblk & 1][d];
    if (tid == 0) {
      if (STATE_ONLY) a.seg_f[sgh] = seg_f;
      else a.m[sh] = sm.rec[(nblk - 1) & 1][kRecM];
    }
  }
}

// End states of segments from zero -> the states that the segments start from. grid (elements of S and n / 256, sequences)
__global__ void state_segments_kernel(float* __restrict__ S, float* __restrict__ n, const float* __restrict__ f,
                                      const int* __restrict__ first, int H, int D, int Dv) {
  const long long ns = static_cast<long long>(H) * D * Dv, nn = static_cast<long long>(H) * D;
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (e >= ns + nn) return;
  const bool is_s = e < ns;
  const long long at = is_s ? e : e - ns, size = is_s ? ns : nn;
  const int h = static_cast<int>(at / (size / H)), s1 = first[blockIdx.y + 1];
  float* x = (is_s ? S : n) + at;
  float run = 0.f;
  for (int s = first[blockIdx.y]; s < s1; ++s) {
    const float add = s + 1 < s1 ? x[s * size] : 0.f;
    x[s * size] = run;
    if (s + 1 < s1) run = fmaf(f[static_cast<long long>(s) * H + h], run, add);
  }
}

template <int ND, bool DELTA, int WARPS, bool STATE_ONLY>
static int launch_state_chunk(const StateChunkArgs& a, int n_seg, cudaStream_t stream) {
  constexpr int smem = static_cast<int>(sizeof(StateSmem<ND>));
  static_assert(smem % 16 == 0, "cleared in 16-byte steps");
  B200_CHECK(cudaFuncSetAttribute(state_chunk_kernel<ND, DELTA, WARPS, STATE_ONLY>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  state_chunk_kernel<ND, DELTA, WARPS, STATE_ONLY><<<dim3(n_seg, a.H, (a.Dv + a.cols - 1) / a.cols), WARPS * 32, smem, stream>>>(a);
  B200_CHECK(cudaGetLastError());
  return 0;
}

template <bool DELTA, bool STATE_ONLY>
static int pick_state_chunk(const StateChunkArgs& a, int n_seg, cudaStream_t stream) {
  const bool wide = a.cols > 64 && a.Dv > 64;
#define B200_SW(ND_)                                                               \
  (wide ? launch_state_chunk<ND_, DELTA, 8, STATE_ONLY>(a, n_seg, stream)          \
        : launch_state_chunk<ND_, DELTA, 4, STATE_ONLY>(a, n_seg, stream))
  if (a.D <= 32) return B200_SW(2);
  if (a.D <= 64) return B200_SW(4);
  return B200_SW(8);
#undef B200_SW
}

}  // namespace b200

extern "C" {

int b200_state_record_floats() { return b200::kRec; }

// qkv, g0, g1, p0, p1: see StateArgs (bf16). run_max: mLSTM, scratch [T, H, 3]. rec: [n_blocks, H, b200_state_record_floats()].
// blocks: int32 [n_blocks, 4]: first token, tokens (1 .. 16), sequence, 1 for the first block of its sequence.
int b200_state_chunk_prep(const void* qkv, long long ldq, const void* g0, const void* g1, long long ldx, const void* p0,
                          const void* p1, float cap, int delta, const int* blocks, int n_blocks, const int* cu, int n_seq,
                          float* run_max, float* rec, int H, int G, int D, int Dv, cudaStream_t stream) {
  using namespace b200;
  if (n_blocks <= 0 || n_seq <= 0) return 0;
  if (G < 1 || H % G || D < 1 || D > 128) return -100;
  const StateArgs a{qkv, ldq, g0, g1, ldx, p0, p1, cap, delta, H, G, D, Dv};
  if (!delta) {
    state_running_max_kernel<__nv_bfloat16><<<dim3(n_seq, H), kMaxThreads, 0, stream>>>(a, cu, run_max);
    B200_CHECK(cudaGetLastError());
  }
  const long long units = static_cast<long long>(n_blocks) * H;
  const unsigned grid = static_cast<unsigned>((units + kPrepWarps - 1) / kPrepWarps);
  const int4* blk = reinterpret_cast<const int4*>(blocks);
#define B200_SP(ND_)                                                                                                  \
  {                                                                                                                   \
    if (delta) state_prep_kernel<ND_, true><<<grid, kPrepWarps * 32, 0, stream>>>(a, blk, n_blocks, run_max, rec);    \
    else state_prep_kernel<ND_, false><<<grid, kPrepWarps * 32, 0, stream>>>(a, blk, n_blocks, run_max, rec);         \
  }
  if (D <= 32) B200_SP(2)
  else if (D <= 64) B200_SP(4)
  else B200_SP(8)
#undef B200_SP
  B200_CHECK(cudaGetLastError());
  return 0;
}

// norm (Dv <= cols): out is the normed and gated heads in bf16; null: out is the plain outputs in fp32. cols: value columns per
// CTA, a multiple of 16 up to 128. segs: int32 [n_seg, 4] as in StateChunkArgs. seg_first: [n_seq + 1] first segment of every
// sequence; seg_S, seg_n, seg_f: scratch, all null when every segment is a whole sequence (mLSTM only). slots null: no state is
// kept.
int b200_state_chunk(const void* qkv, long long ldq, const void* gate, long long ldg, const float* rec, const int* blocks,
                     const int* segs, int n_seg, const int* seg_first, int n_seq, float* seg_S, float* seg_n, float* seg_f,
                     const int* slots, float* S, float* n, float* m, const void* norm, void* out, int cols, float eps,
                     int delta, int H, int G, int D, int Dv, cudaStream_t stream) {
  using namespace b200;
  if (n_seg <= 0 || n_seq <= 0) return 0;
  if (delta && seg_S) return -100;
  if (G < 1 || H % G || D < 1 || D > 128 || Dv < 1 || cols < 16 || cols > 128 || cols % 16 || (norm && Dv > cols)) return -100;
  using bf = __nv_bfloat16;
  const StateChunkArgs a{(const bf*)qkv, ldq, (const bf*)gate, ldg, rec, reinterpret_cast<const int4*>(blocks),
                         reinterpret_cast<const int4*>(segs), slots, seg_S, seg_n, seg_f, S, n, m, (const bf*)norm, (bf*)out, (float*)out, eps, H, G, D, Dv, cols};
  if (delta) return pick_state_chunk<true, false>(a, n_seg, stream);
  if (seg_S) {
    const int rc = pick_state_chunk<false, true>(a, n_seg, stream);
    if (rc) return rc;
    const long long e = static_cast<long long>(H) * D * (Dv + 1);
    state_segments_kernel<<<dim3(static_cast<unsigned>((e + 255) / 256), n_seq), 256, 0, stream>>>(seg_S, seg_n, seg_f, seg_first,
                                                                                                  H, D, Dv);
    B200_CHECK(cudaGetLastError());
  }
  return pick_state_chunk<false, false>(a, n_seg, stream);
}

}  // extern "C"
