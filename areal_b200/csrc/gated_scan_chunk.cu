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
// Products of gates only ever run forward (no quotients, no logarithms), so nothing overflows or loses precision when
// gates close. fp32 operands enter the bf16 products as two terms (hi + lo, three products where both sides have two);
// values are bf16 numbers and enter exactly. A is computed in fp32 on the CUDA
// cores: inside a half block with running products held in registers, between the halves as plain products.
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
  __nv_bfloat16 q[2][16 * (DP + 8)], k[2][16 * (DP + 8)];  // hi, lo
  __nv_bfloat16 v[16 * 136];
  float A[4][16 * 16];        // partial sums over 32 channels each; the part above the diagonal stays zero
  float qx[8 * 128], kx[8 * 128];  // second half's q and first half's k with the gates of their own half
  float tot[2][DP], F[DP];
  float o[16 * 132];
};

// Sums 16 per-lane values over the warp: every lane ends with the total of value (lane >> 1). Halves the values while
// doubling the lanes that share one.
__device__ __forceinline__ float warp_sum16(float (&v)[16], int lane) {
#pragma unroll
  for (int s = 8; s >= 1; s >>= 1) {
    const bool up = lane & (2 * s);
#pragma unroll
    for (int r = 0; r < s; ++r) {
      const float give = up ? v[r] : v[r + s];
      const float keep = up ? v[r + s] : v[r];
      v[r] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * s);
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 1);
}
// The 36 entries (i, j), j <= i < 8, of a half block's triangle in three batches of whole columns: columns 0, 1, 7; then
// 2, 3, 5, 6; then 4. Entry e of a batch as i * 16 + j.
__device__ __forceinline__ int tri_entry(int batch, int e) {
  if (batch == 0) return e < 8 ? e * 16 : e < 15 ? (e - 7) * 16 + 1 : 7 * 16 + 7;
  if (batch == 1) return e < 6 ? (e + 2) * 16 + 2 : e < 11 ? (e - 3) * 16 + 3 : e < 14 ? (e - 6) * 16 + 5 : (e - 8) * 16 + 6;
  return (e + 4) * 16 + 4;
}
// One column j of the triangle: q_i k_j prod_{j < t <= i} f_t for i = j..7 into v[at..]
template <int J>
__device__ __forceinline__ void tri_column(const float (&q)[8], const float (&f)[8], const float (&k)[8], float (&v)[16], int at) {
  float w = k[J];
#pragma unroll
  for (int i = J; i < 8; ++i) {
    if (i > J) w *= f[i];
    v[at + i - J] = q[i] * w;
  }
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
  if (dch) {
    if (mode == 0) {
      bias = ld1(static_cast<const __nv_bfloat16*>(a.s.bias) + h * D + d);
      low = ld1(static_cast<const __nv_bfloat16*>(a.s.lower) + h * D + d);
    } else {
      decay = a.s.decay[h];
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
  const bool warp_live = (warp & 3) * 32 < DP;  // this warp has channels
  if (!STATE_ONLY)
    for (int i = tid; i < 4 * 256; i += kScThreads) (&sm.A[0][0])[i] = 0.f;
  __syncthreads();
  float seg_f = 1.f;  // product of all gates of the segment (threads of half 0)

  __nv_bfloat16 rq[8], rf[8], rv[8];
  const __nv_bfloat16 zero = __float2bfloat16(0.f);
  auto load = [&](int t0) {  // raw projections of the block that starts at token t0 of the segment
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int tok = t0 + half * 8 + i;
      const __nv_bfloat16* row = x + (static_cast<long long>(seg.x) + tok) * a.s.ldx + h * D + d;
      const bool in = tok < seg.y;
      rq[i] = in && dch ? row[0] : zero;
      rf[i] = in && dch ? row[H * D] : zero;
      rv[i] = in && d < nv ? x[(static_cast<long long>(seg.x) + tok) * a.s.ldx + 2 * H * D + h * Dv + vb + d] : zero;
    }
  };
  load(0);
  for (int t0 = 0; t0 < seg.y; t0 += 16) {
    // ---- activations; the triangle of A inside this half; running products of the gates inside the half
    float q[8], f[8], k[8];
    float run = 1.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int tok = half * 8 + i;
      q[i] = 0.f; k[i] = 0.f; f[i] = 1.f;
      if (dch && t0 + tok < seg.y)
        scan_activate(mode, __bfloat162float(rq[i]), __bfloat162float(rf[i]), bias, low, decay, q[i], f[i], k[i]);
    }
    if (!STATE_ONLY && warp_live) {
      float* A = sm.A[warp & 3] + half * (8 * 16 + 8);
#pragma unroll
      for (int batch = 0; batch < 3; ++batch) {
        float v[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) v[e] = 0.f;
        if (batch == 0) {
          tri_column<0>(q, f, k, v, 0);
          tri_column<1>(q, f, k, v, 8);
          tri_column<7>(q, f, k, v, 15);
        } else if (batch == 1) {
          tri_column<2>(q, f, k, v, 0);
          tri_column<3>(q, f, k, v, 6);
          tri_column<5>(q, f, k, v, 11);
          tri_column<6>(q, f, k, v, 14);
        } else {
          tri_column<4>(q, f, k, v, 0);
        }
        const float sum = warp_sum16(v, lane);
        const int e = lane >> 1;
        if (!(lane & 1) && (batch < 2 || e < 4)) A[tri_entry(batch, e)] = sum;
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      run *= f[i];
      if (!STATE_ONLY) q[i] *= run;  // q_i P_i, still without the gates of the first half
    }
    float suf = 1.f;
#pragma unroll
    for (int i = 7; i >= 0; --i) {
      k[i] *= suf;
      suf *= f[i];
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float v = __bfloat162float(rv[i]);
      if (mode != 0) v = silu_fast(v);
      sm.v[(half * 8 + i) * 136 + d] = d < nv ? __float2bfloat16(v) : zero;
    }
    if (d < DP) sm.tot[half][d] = run;
    if (!STATE_ONLY) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (half) sm.qx[i * 128 + d] = q[i];
        else sm.kx[i * 128 + d] = k[i];
      }
    }
    __syncthreads();
    if (t0 + 16 < seg.y) load(t0 + 16);
    // ---- operands: the other half's gates, then two bf16 terms
    if (d < DP) {
      const float other = sm.tot[half ^ 1][d];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int at = (half * 8 + i) * (DP + 8) + d;
        if (!STATE_ONLY) {
          const float qq = half ? q[i] * other : q[i];
          const __nv_bfloat16 hi = __float2bfloat16(qq);
          sm.q[0][at] = hi;
          sm.q[1][at] = __float2bfloat16(qq - __bfloat162float(hi));
        }
        const float kk = half ? k[i] : k[i] * other;
        const __nv_bfloat16 hi = __float2bfloat16(kk);
        sm.k[0][at] = hi;
        sm.k[1][at] = __float2bfloat16(kk - __bfloat162float(hi));
      }
      if (half == 0) {
        sm.F[d] = run * other;
        seg_f *= run * other;
      }
    }
    // ---- A between the halves: q_i of the second against k_j of the first; half h of the threads takes i = 8 + 4h ..
    if (!STATE_ONLY && warp_live) {
      float kj[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) kj[j] = sm.kx[j * 128 + d];
      float* A = sm.A[warp & 3] + (8 + half * 4) * 16;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float q0 = sm.qx[(half * 4 + e * 2) * 128 + d], q1 = sm.qx[(half * 4 + e * 2 + 1) * 128 + d];
        float v[16];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          v[j] = q0 * kj[j];
          v[8 + j] = q1 * kj[j];
        }
        const float sum = warp_sum16(v, lane);
        const int x = lane >> 1;
        if (!(lane & 1)) A[(e * 2 + (x >> 3)) * 16 + (x & 7)] = sum;
      }
    }
    __syncthreads();
    // ---- products
    if (mma) {
      const int r8 = (lane & 7) + ((lane >> 4) << 3), c8 = ((lane >> 3) & 1) * 8;
      uint32_t vt[4];
      ldm_x4_t(s32(sm.v + r8 * 136 + warp * 16 + c8), vt);
      if (!STATE_ONLY) {
        float o[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int c = 0; c < 4; ++c) o[n][c] = 0.f;
        uint32_t ah[4], al[4];
        // A as the second operand: entries (i = g + 8n, j = 2t + 8c, +1) of the channel groups' partial sums
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int at = (g + (e >> 1) * 8) * 16 + 2 * t + (e & 1) * 8;
          float2 sum = *reinterpret_cast<const float2*>(&sm.A[0][at]);
#pragma unroll
          for (int c = 1; c < (ND * 16 + 31) / 32; ++c) {
            const float2 p = *reinterpret_cast<const float2*>(&sm.A[c][at]);
            sum.x += p.x;
            sum.y += p.y;
          }
          ah[e] = split2(sum.x, sum.y, al[e]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          mma_bf16(o[n], vt, ah[2 * n], ah[2 * n + 1]);
          mma_bf16(o[n], vt, al[2 * n], al[2 * n + 1]);
        }
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
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int c = 0; c < 4; ++c) sm.o[(n * 8 + 2 * t + (c & 1)) * 132 + warp * 16 + g + (c >> 1) * 8] = o[n][c];
      }
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
    __syncthreads();
    // ---- outputs: warp w writes tokens w and w + 8
    if (!STATE_ONLY) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = warp + 8 * e;
        if (t0 + i < seg.y) {
          const long long at = ((static_cast<long long>(seg.x) + t0 + i) * H + h) * Dv + vb;
          if (a.norm_w) {
            float ss = 0.f;
            for (int c = lane; c < nv; c += 32) ss = fmaf(sm.o[i * 132 + c], sm.o[i * 132 + c], ss);
            const float r = rsqrtf(warp_sum(ss) / nv + a.eps);
            for (int c = lane; c < nv; c += 32) a.y[at + c] = __float2bfloat16(sm.o[i * 132 + c] * r * ld1(a.norm_w + c));
          } else {
            for (int c = lane; c < nv; c += 32) a.s.o[at + c] = sm.o[i * 132 + c];
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
