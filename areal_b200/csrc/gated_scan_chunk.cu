// Prefill of the gated linear recurrences (gated_scan.cu) on tensor cores, for bf16 models with key width <= 128.
//
// A sequence (or a segment of one) is walked 16 tokens at a time by one CTA per (segment, head, 128 value columns); the
// fp32 state stays in the accumulator registers of the warps for the whole walk, transposed, so that it can be used as
// an operand without a shuffle: warp w owns value columns 16w..16w+15 and all key channels. With P_i the product of the
// gates of the block up to token i, R_j that of the gates after token j, F that of all 16 (all per channel):
//
//   O^T = S^T (q_i P_i)^T + V^T A^T,   A_ij = sum_d q_id k_jd prod_{j < t <= i} f_td  (j <= i)
//   S^T <- S^T diag(F) + V^T (k_j R_j)
//
// fp32 operands enter the bf16 products as two terms (hi + lo, three products where both sides have two); values are bf16
// numbers and enter exactly. A is a product of (q_i P_i / F) with (k_j R_j): every term has the size of the true weight,
// only the factors need range, so this holds as long as F stays inside the exponent range. A block in which some channel
// forgets more than that (F < 2^-90) takes a slow path that multiplies the gates up pair by pair, in fp32.
//
// Few long sequences would leave most SMs idle: they are cut into segments. A first pass computes every segment's state
// from zero and its gate product, a scan over a sequence's segments turns them into the states the segments start
// from, and the second pass computes the outputs.
#include "common/host_utils.h"
#include "common/mma16.cuh"
#include "common/scan_inputs.cuh"

namespace b200 {

constexpr int kScThreads = 256;

struct ScanChunkArgs {
  ScanArgs s;
  const int4* segs;          // (first token, tokens, sequence, 1 for the last segment of its sequence)
  float* seg_state;          // [n_seg, H, D, Dv]: pass 1 writes, pass 2 reads (null: segments are whole sequences)
  float* seg_decay;          // [n_seg, H, D]
  const __nv_bfloat16* norm_w;  // [Dv] or null; with it y gets the normed heads
  __nv_bfloat16* y;          // [T, H * Dv]
  float eps;
};

__device__ __forceinline__ uint32_t s32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }

template <int ND>
struct ScanSmem {
  static constexpr int DP = ND * 16, PB = (DP + 8) * 2;  // padded channels, bytes of a bf16 row
  __nv_bfloat16 raw[2][3][16 * 128];                     // double-buffered projections: q, f / k, v
  __nv_bfloat16 q[2][16 * (DP + 8)], k[2][16 * (DP + 8)], s[2][16 * (DP + 8)];  // hi, lo of q P, k R, q P / F
  __nv_bfloat16 v[16 * 136];
  float A[4][16 * 16];  // partial sums over channels
  float tot[2][DP], F[DP];
  float o[16 * 132];
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {  // bytes < 16: the rest is zero
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void put_split(__nv_bfloat16* hi, __nv_bfloat16* lo, int at, float v) {
  const __nv_bfloat16 h = __float2bfloat16(v);
  hi[at] = h;
  lo[at] = __float2bfloat16(v - __bfloat162float(h));
}

// STATE_ONLY: pass 1 (no outputs; starts from zero; writes seg_state and seg_decay)
template <int ND, bool STATE_ONLY>
__global__ void __launch_bounds__(kScThreads, 2) scan_chunk_kernel(ScanChunkArgs a) {
  using SM = ScanSmem<ND>;
  constexpr int DP = SM::DP, PB = SM::PB;
  extern __shared__ __align__(16) uint8_t raw[];
  SM& sm = *reinterpret_cast<SM*>(raw);
  const int4 seg = a.segs[blockIdx.x];
  if (STATE_ONLY && seg.w) return;  // nothing starts from the last segment's end state here
  const int h = blockIdx.y, vb = blockIdx.z * 128, D = a.s.D, Dv = a.s.Dv, H = a.s.H;
  const int nv = min(128, Dv - vb);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const bool mma = warp * 16 < nv;
  const __nv_bfloat16* x = static_cast<const __nv_bfloat16*>(a.s.x);
  const int mode = a.s.mode;

  // this thread's channel and half of a 16-token block
  const int d = tid & 127, half = tid >> 7;
  const bool dch = d < D;
  float bias = 0.f, low = 0.f, decay = 0.f;
  const float decay_h = mode == 0 ? 0.f : a.s.decay[h];
  if (dch) {
    if (mode == 0) {
      bias = ld1(static_cast<const __nv_bfloat16*>(a.s.bias) + h * D + d);
      low = ld1(static_cast<const __nv_bfloat16*>(a.s.lower) + h * D + d);
    } else {
      decay = decay_h;
    }
  }
  float S[2 * ND][4];
#pragma unroll
  for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) S[i][c] = 0.f;
  auto state_at = [&](int i, int c) {  // (channel, column) of accumulator element c of tile i
    return make_int2(i * 8 + 2 * t + (c & 1), vb + warp * 16 + g + (c >> 1) * 8);
  };
  const long long seg_base = (static_cast<long long>(blockIdx.x) * H + h) * D * Dv;
  if (!STATE_ONLY && a.seg_state && mma) {
#pragma unroll
    for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int2 p = state_at(i, c);
        if (p.x < D && p.y < Dv) S[i][c] = a.seg_state[seg_base + static_cast<long long>(p.x) * Dv + p.y];
      }
  }
  float seg_f = 1.f;  // product of all gates of the segment (threads of half 0)
  float nw[4] = {0.f, 0.f, 0.f, 0.f};  // the norm's weights of the columns this lane writes
  if (!STATE_ONLY && a.norm_w)
    for (int c = 0; c < 4; ++c)
      if (lane * 4 + c < nv) nw[c] = ld1(a.norm_w + lane * 4 + c);
  // projections of 16 tokens into a stage; tokens past the end become zeros
  const bool wide = !((D | Dv | a.s.ldx) & 7) && !(reinterpret_cast<uintptr_t>(x) & 15);
  auto load = [&](int t0, int st) {
    if (wide) {
      for (int i = tid; i < 3 * 16 * 16; i += kScThreads) {
        const int part = i >> 8, tok = (i >> 4) & 15, c = (i & 15) * 8;
        if (c < (part == 2 ? nv : D)) {
          const long long row = static_cast<long long>(seg.x) + min(t0 + tok, seg.y - 1);
          const int col = part == 2 ? 2 * H * D + h * Dv + vb + c : part * H * D + h * D + c;
          cp_async16(&sm.raw[st][part][tok * 128 + c], x + row * a.s.ldx + col, t0 + tok < seg.y ? 16 : 0);
        }
      }
    } else {
      for (int i = tid; i < 3 * 16 * 128; i += kScThreads) {
        const int part = i >> 11, tok = (i >> 7) & 15, c = i & 127;
        if (c < (part == 2 ? nv : D)) {
          const long long row = static_cast<long long>(seg.x) + t0 + tok;
          const int col = part == 2 ? 2 * H * D + h * Dv + vb + c : part * H * D + h * D + c;
          sm.raw[st][part][tok * 128 + c] = t0 + tok < seg.y ? x[row * a.s.ldx + col] : __float2bfloat16(0.f);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(0, 0);
  int st = 0;
  for (int t0 = 0; t0 < seg.y; t0 += 16, st ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this block's projections are here; every warp has left the block before
    if (t0 + 16 < seg.y) load(t0 + 16, st ^ 1);
    // ---- activations, running products of the gates inside this half
    float q[8], k[8], f[8], run = 1.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int tok = half * 8 + i;
      q[i] = 0.f; k[i] = 0.f; f[i] = 1.f;
      if (dch && t0 + tok < seg.y)
        scan_activate(x, mode, __bfloat162float(sm.raw[st][0][tok * 128 + d]), __bfloat162float(sm.raw[st][1][tok * 128 + d]),
                      bias, low, decay, q[i], f[i], k[i]);
      run *= f[i];
      q[i] *= run;  // q_i P_i, still without the gates of the first half
    }
    float suf = 1.f;
#pragma unroll
    for (int i = 7; i >= 0; --i) {
      k[i] *= suf;
      suf *= f[i];
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int tok = half * 8 + i;
      __nv_bfloat16 v = __float2bfloat16(0.f);
      if (d < nv) {
        v = sm.raw[st][2][tok * 128 + d];
        if (mode != 0) v = __float2bfloat16(silu_fast(__bfloat162float(v)));
      }
      sm.v[tok * 136 + d] = v;
    }
    if (d < DP) sm.tot[half][d] = run;
    __syncthreads();
    // ---- operands: the other half's gates, then two bf16 terms
    bool far = false;
    if (d < DP) {
      const float other = sm.tot[half ^ 1][d], F = run * other;
      far = F < 0x1p-90f;
      const float inv = far ? 0.f : rcp_fast(F);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int at = (half * 8 + i) * (DP + 8) + d;
        if (!STATE_ONLY) {
          const float qq = half ? q[i] * other : q[i];
          put_split(sm.q[0], sm.q[1], at, qq);
          put_split(sm.s[0], sm.s[1], at, qq * inv);
        }
        put_split(sm.k[0], sm.k[1], at, half ? k[i] : k[i] * other);
      }
      if (half == 0) {
        sm.F[d] = F;
        seg_f *= F;
      }
    }
    bool slow = false;
    if (STATE_ONLY) __syncthreads();
    else slow = __syncthreads_or(far);
    const int r8 = (lane & 7) + ((lane >> 4) << 3), c8 = ((lane >> 3) & 1) * 8;
    float o[2][4];
    if (!STATE_ONLY) {
      if (!slow) {
        // ---- A: warp w computes keys 8 (w & 1) .. over channels 32 (w >> 1) ..
        if ((warp >> 1) * 32 < DP) {
          float acc[4] = {0.f, 0.f, 0.f, 0.f};
          const uint32_t sh = s32(sm.s[0]) + (lane & 15) * PB + (lane >> 4) * 16, sl = s32(sm.s[1]) + (lane & 15) * PB + (lane >> 4) * 16;
          const int kr = ((warp & 1) * 8 + (lane & 7)) * PB + (lane >> 3) * 16;
          uint32_t bh[4], bl[4], ah[4], al[4];
          const int c0 = (warp >> 1) * 64;  // bytes: two reduction blocks of 16 channels
          ldm_x4(s32(sm.k[0]) + kr + c0, bh);
          ldm_x4(s32(sm.k[1]) + kr + c0, bl);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            ldm_x4(sh + c0 + e * 32, ah);
            ldm_x4(sl + c0 + e * 32, al);
            mma_bf16(acc, ah, bh[2 * e], bh[2 * e + 1]);
            mma_bf16(acc, al, bh[2 * e], bh[2 * e + 1]);
            mma_bf16(acc, ah, bl[2 * e], bl[2 * e + 1]);
          }
          float* A = sm.A[warp >> 1] + (warp & 1) * 8 + 2 * t;
          *reinterpret_cast<float2*>(A + g * 16) = make_float2(acc[0], acc[1]);
          *reinterpret_cast<float2*>(A + (g + 8) * 16) = make_float2(acc[2], acc[3]);
        }
      } else {
        // some channel forgets everything inside the block: pair by pair, lanes over channels
        for (int j = warp; j < 16; j += 8) {
          float w[4], acc = 0.f;
          for (int i = j; i < 16; ++i) {
            acc = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int c = lane + 32 * e;
              if (c < D && t0 + i < seg.y) {
                float qq, ff, kk;
                const bool gated = mode == 0;
                const int hd = h * D + c;
                scan_activate(x, mode, __bfloat162float(sm.raw[st][0][i * 128 + c]), __bfloat162float(sm.raw[st][1][i * 128 + c]),
                              gated ? ld1(static_cast<const __nv_bfloat16*>(a.s.bias) + hd) : 0.f,
                              gated ? ld1(static_cast<const __nv_bfloat16*>(a.s.lower) + hd) : 0.f, decay_h, qq, ff, kk);
                w[e] = i == j ? kk : w[e] * ff;
                acc = fmaf(qq, w[e], acc);
              }
            }
            acc = warp_sum(acc);
            if (lane == 0) {
              sm.A[0][i * 16 + j] = acc;
#pragma unroll
              for (int c = 1; c < 4; ++c) sm.A[c][i * 16 + j] = 0.f;
            }
          }
        }
      }
      // ---- outputs from the state at the block's start
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[n][c] = 0.f;
      if (mma) {
        const uint32_t qh = s32(sm.q[0]) + r8 * PB + c8 * 2, ql = s32(sm.q[1]) + r8 * PB + c8 * 2;
#pragma unroll
        for (int kt = 0; kt < ND; ++kt) {
          uint32_t hi[4], lo[4], bh[4], bl[4];
          hi[0] = split2(S[2 * kt][0], S[2 * kt][1], lo[0]);
          hi[1] = split2(S[2 * kt][2], S[2 * kt][3], lo[1]);
          hi[2] = split2(S[2 * kt + 1][0], S[2 * kt + 1][1], lo[2]);
          hi[3] = split2(S[2 * kt + 1][2], S[2 * kt + 1][3], lo[3]);
          ldm_x4(qh + kt * 32, bh);
          ldm_x4(ql + kt * 32, bl);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma_bf16(o[n], hi, bh[2 * n], bh[2 * n + 1]);
            mma_bf16(o[n], lo, bh[2 * n], bh[2 * n + 1]);
            mma_bf16(o[n], hi, bl[2 * n], bl[2 * n + 1]);
          }
        }
      }
      __syncthreads();
    }
    if (mma) {
      uint32_t vt[4];
      ldm_x4_t(s32(sm.v + r8 * 136 + warp * 16 + c8), vt);
      if (!STATE_ONLY) {
        // ---- outputs from the block itself: A as the second operand, entries (i = g + 8n, j = 2t + 8c, +1), j <= i
        uint32_t ah[4], al[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = g + (e >> 1) * 8, j = 2 * t + (e & 1) * 8;
          float2 sum = *reinterpret_cast<const float2*>(&sm.A[0][i * 16 + j]);
#pragma unroll
          for (int c = 1; c < (DP + 31) / 32; ++c) {
            const float2 p = *reinterpret_cast<const float2*>(&sm.A[c][i * 16 + j]);
            sum.x += p.x;
            sum.y += p.y;
          }
          ah[e] = split2(j <= i ? sum.x : 0.f, j + 1 <= i ? sum.y : 0.f, al[e]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16(o[n], vt, ah[2 * n], ah[2 * n + 1]);
          mma_bf16(o[n], vt, al[2 * n], al[2 * n + 1]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int c = 0; c < 4; ++c) sm.o[(n * 8 + 2 * t + (c & 1)) * 132 + warp * 16 + g + (c >> 1) * 8] = o[n][c];
      }
      // ---- the state at the block's end
      const uint32_t kh = s32(sm.k[0]) + (lane & 15) * PB + (lane >> 4) * 16,
                     kl = s32(sm.k[1]) + (lane & 15) * PB + (lane >> 4) * 16;
#pragma unroll
      for (int nt = 0; nt < ND; ++nt) {
        uint32_t bh[4], bl[4];
        ldm_x4_t(kh + nt * 32, bh);
        ldm_x4_t(kl + nt * 32, bl);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float(&c)[4] = S[2 * nt + n];
          const float2 F = *reinterpret_cast<const float2*>(&sm.F[nt * 16 + n * 8 + 2 * t]);
          c[0] *= F.x; c[1] *= F.y; c[2] *= F.x; c[3] *= F.y;
          mma_bf16(c, vt, bh[2 * n], bh[2 * n + 1]);
          mma_bf16(c, vt, bl[2 * n], bl[2 * n + 1]);
        }
      }
    }
    if (!STATE_ONLY) {
      __syncthreads();
      // ---- warp w writes tokens w and w + 8, a lane four columns
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = warp + 8 * e, c = lane * 4;
        if (t0 + i < seg.y) {
          const long long at = ((static_cast<long long>(seg.x) + t0 + i) * H + h) * Dv + vb + c;
          float4 v = *reinterpret_cast<const float4*>(&sm.o[i * 132 + c]);
          if (c >= nv) v.x = 0.f;
          if (c + 1 >= nv) v.y = 0.f;
          if (c + 2 >= nv) v.z = 0.f;
          if (c + 3 >= nv) v.w = 0.f;
          if (a.norm_w) {
            const float r = rsqrtf(warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)))) / nv + a.eps);
            v.x *= r * nw[0]; v.y *= r * nw[1]; v.z *= r * nw[2]; v.w *= r * nw[3];
          }
          if (!(Dv & 3)) {
            if (c < nv) {
              if (a.norm_w) st4(a.y + at, v);
              else st4(a.s.o + at, v);
            }
          } else {
            const float u[4] = {v.x, v.y, v.z, v.w};
            for (int n = 0; n < 4 && c + n < nv; ++n) {
              if (a.norm_w) st1(a.y + at + n, u[n]);
              else a.s.o[at + n] = u[n];
            }
          }
        }
      }
    }
  }
  // ---- end state
  float* dst = nullptr;
  if (STATE_ONLY) {
    dst = a.seg_state + seg_base;
    if (half == 0 && dch && blockIdx.z == 0) a.seg_decay[(static_cast<long long>(blockIdx.x) * H + h) * D + d] = seg_f;
  } else if (seg.w && a.s.slots) {
    const int slot = a.s.slots[seg.z];
    if (slot >= 0) dst = a.s.state + (static_cast<long long>(slot) * H + h) * D * Dv;
  }
  if (dst && mma) {
#pragma unroll
    for (int i = 0; i < 2 * ND; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int2 p = state_at(i, c);
        if (p.x < D && p.y < Dv) dst[static_cast<long long>(p.x) * Dv + p.y] = S[i][c];
      }
  }
}

// seg_state[s] (end state of segment s from zero) -> the state segment s starts from. One thread per state element.
__global__ void scan_segments_kernel(float* __restrict__ seg_state, const float* __restrict__ seg_decay,
                                     const int* __restrict__ first, int H, int D, int Dv) {
  const int seq = blockIdx.y;
  const long long n = static_cast<long long>(H) * D * Dv;
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (e >= n) return;
  const long long hd = e / Dv;
  float S = 0.f;
  const int s1 = first[seq + 1];
  for (int s = first[seq]; s < s1; ++s) {
    float* p = seg_state + s * n + e;
    const float add = s + 1 < s1 ? *p : 0.f;
    *p = S;
    if (s + 1 < s1) S = fmaf(seg_decay[static_cast<long long>(s) * H * D + hd], S, add);
  }
}

}  // namespace b200

extern "C" {

int b200_scan_chunk_ok(int D, int Dv) { return (D >= 1 && D <= 128 && Dv >= 1) ? 0 : -100; }

// segs: int32 [n_seg, 4]; seg_first: [n_seq + 1] first segment of every sequence. seg_state / seg_decay: null when every
// segment is a whole sequence. Either norm_w + y (Dv <= 128) or o (fp32). bf16 models.
int b200_scan_chunk(const void* x, long long ldx, const void* bias, const void* lower, const float* decay,
                    const int* segs, int n_seg, const int* seg_first, int n_seq, const int* slots, float* state,
                    float* seg_state, float* seg_decay, float* o, const void* norm_w, void* y, float eps, int H, int D,
                    int Dv, int mode, cudaStream_t stream) {
  using namespace b200;
  if (n_seg <= 0) return 0;
  if (b200_scan_chunk_ok(D, Dv) || (norm_w && Dv > 128)) return -100;
  ScanChunkArgs a{ScanArgs{x, ldx, bias, lower, decay, nullptr, slots, state, o, H, D, Dv, mode},
                  reinterpret_cast<const int4*>(segs), seg_state, seg_decay, (const __nv_bfloat16*)norm_w,
                  (__nv_bfloat16*)y, eps};
  dim3 grid(n_seg, H, (Dv + 127) / 128);
#define B200_SC(ND_, ONLY_)                                                                                         \
  {                                                                                                                 \
    B200_CHECK(cudaFuncSetAttribute(scan_chunk_kernel<ND_, ONLY_>, cudaFuncAttributeMaxDynamicSharedMemorySize,     \
                                    (int)sizeof(ScanSmem<ND_>)));                                                   \
    scan_chunk_kernel<ND_, ONLY_><<<grid, kScThreads, sizeof(ScanSmem<ND_>), stream>>>(a);                          \
    B200_CHECK(cudaGetLastError());                                                                                 \
  }
#define B200_SCD(ONLY_)                                                                                             \
  if (D <= 32) B200_SC(2, ONLY_)                                                                                    \
  else if (D <= 64) B200_SC(4, ONLY_)                                                                               \
  else B200_SC(8, ONLY_)
  if (seg_state) {
    B200_SCD(true)
    const long long n = static_cast<long long>(H) * D * Dv;
    scan_segments_kernel<<<dim3((unsigned)((n + 255) / 256), n_seq), 256, 0, stream>>>(seg_state, seg_decay, seg_first,
                                                                                      H, D, Dv);
    B200_CHECK(cudaGetLastError());
  }
  B200_SCD(false)
#undef B200_SCD
#undef B200_SC
  return 0;
}

}  // extern "C"
