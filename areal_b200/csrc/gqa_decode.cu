// Decode attention over a paged cache for grouped-query heads of up to 256 with the options of ops/gqa.py: a window that
// keeps the first tokens, a soft cap on the scores, a sink, a gate per head, sigmoids as weights. One query token per
// sequence.
//
//   k_cache [blocks, G, block_size, D], v_cache [blocks, G, block_size, Dv]   bf16, D and Dv in steps of 16
//
// Same shape as paged_decode.cu: one CTA per (sequence, key / value head, split), four warps, and every warp is its own
// pipeline over slabs of 16 tokens that lane 0 fills with TMA (128-byte swizzle). Up to 16 query heads of the group are
// the rows of an m16n8k16 tile (groups past 16 take several CTAs). What differs:
//   * the walk over slabs has two parts: those of the first tokens that a window keeps, then those inside the window;
//   * softmax weights enter the second product as two bf16 terms (hi + lo), so they keep fp32-like precision;
//   * the sink joins the denominator once, and the gate scales a head's result, where the splits meet;
//   * sigmoid weights count as they are: neither maxima nor sums are kept (the reference stays 0).
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/mma16.cuh"
#include "common/ptx.cuh"

namespace b200 {

constexpr int kGdSlab = 16, kGdWarps = 4, kGdBox = kGdSlab * 128;  // tokens per slab; bytes of 64 columns of a slab

struct GqaDecodeArgs {
  const __nv_bfloat16* q;      // [B][ldq] + h * hq, zeros between a head's width and D
  long long ldq;
  int hq;
  const int *block_table, *seq_lens;
  __nv_bfloat16* out;          // [B, H * dv]
  float *o_part, *ml_part;     // [B, H, nsplit, Dv], [B, H, nsplit, 2]
  int H, G, D, Dv, dv, block_size, max_blocks, nsplit;  // dv: numbers of a head's result
  float scale, cap;
  int window, keep;
  const __nv_bfloat16 *sink, *gate;
  long long ldg;
  const __nv_bfloat16* sig_bias;  // null: softmax; else [H], added to the scores
};

// Result of a head from its accumulated sum `l` (against the reference m, in units of log 2): the factor on the
// accumulators, with the sink's term and the gate.
__device__ __forceinline__ float gqa_final(float m, float l, int h, long long row, const __nv_bfloat16* sink,
                                           const __nv_bfloat16* gate, long long ldg, bool sigmoid) {
  float f = 1.f;
  if (sigmoid) return gate ? sigmoid_as(__bfloat162float(gate[row * ldg + h]), gate) : 1.f;
  if (sink) {
    const float sv = __bfloat162float(sink[h]) * 1.4426950408889634f, mn = fmaxf(m, sv);
    f = m == -INFINITY ? 0.f : ex2_fast(m - mn);
    l = l * f + ex2_fast(sv - mn);
  }
  f = l > 0.f ? f / l : 0.f;
  return gate ? f * sigmoid_as(__bfloat162float(gate[row * ldg + h]), gate) : f;
}

// KB / VB: 64-column boxes of keys / values; SLOTS: slabs in flight per warp; R16: rows 8-15 of the tile are in use
template <int KB, int VB, int SLOTS, bool R16>
__global__ void __launch_bounds__(kGdWarps * 32, KB + VB > 4 ? 1 : 2)
gqa_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const GqaDecodeArgs a,
                  int* status) {
  constexpr int kSlabB = (KB + VB) * kGdBox, kRows = R16 ? 16 : 8;
  extern __shared__ uint8_t dsm_raw[];
  uint8_t* dsm = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(dsm_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(dsm + kGdWarps * SLOTS * kSlabB);  // [warp][slot]
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars + kGdWarps * SLOTS);

  const int group = a.H / a.G, parts = (group + 15) / 16;
  const int b = blockIdx.x, hk = blockIdx.y / parts, h0 = hk * group + (blockIdx.y % parts) * 16, split = blockIdx.z;
  const int nh = min(16, hk * group + group - h0);  // query heads of this CTA
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int L = a.seq_lens[b];
  const int lo = a.window > 0 ? max(0, L - a.window) : 0;
  const int s0 = lo / kGdSlab, nkeep = min((a.keep + kGdSlab - 1) / kGdSlab, s0);
  const int slabs = (L + kGdSlab - 1) / kGdSlab - s0 + nkeep, skip = s0 - nkeep;
  const int per = (slabs + a.nsplit - 1) / a.nsplit;
  const int i_begin = split * per, i_end = min(slabs, i_begin + per);
  const int spp = a.block_size / kGdSlab;  // slabs per page
  const int* bt = a.block_table + static_cast<long long>(b) * a.max_blocks;
  const int kboxes = (a.D + 63) >> 6, vboxes = (a.Dv + 63) >> 6, ksteps = a.D >> 4, vtiles = a.Dv >> 4;

  if (threadIdx.x == 0) {
    for (int i = 0; i < kGdWarps * SLOTS; ++i) mbar_init(&bars[i], 1);
    *abort_flag = 0;
    fence_mbar_init();
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
  }
  __syncthreads();

  uint8_t* ring = dsm + warp * SLOTS * kSlabB;
  uint64_t* full = bars + warp * SLOTS;
  const int first = i_begin + warp;
  const int count = first < i_end ? (i_end - first + kGdWarps - 1) / kGdWarps : 0;
  auto slab_of = [&](int j) {
    const int i = first + j * kGdWarps;
    return i < nkeep ? i : i + skip;
  };
  auto issue = [&](int j) {  // lane 0 only
    const int sl = slab_of(j);
    const int y = (__ldg(bt + sl / spp) * a.G + hk) * a.block_size + (sl % spp) * kGdSlab;
    uint8_t* dst = ring + (j % SLOTS) * kSlabB;
    uint64_t* bar = &full[j % SLOTS];
    mbar_arrive_expect_tx(bar, (kboxes + vboxes) * kGdBox);
    for (int c = 0; c < kboxes; ++c) tma_load_2d(dst + c * kGdBox, &tmK, bar, c * 64, y);
    for (int c = 0; c < vboxes; ++c) tma_load_2d(dst + (KB + c) * kGdBox, &tmV, bar, c * 64, y);
  };
  if (lane == 0)
    for (int j = 0; j < SLOTS && j < count; ++j) issue(j);

  // query fragments: rows lane / 4 and lane / 4 + 8 are heads of the group (rows past its end are zero)
  const int row = lane >> 2, cq = (lane & 3) * 2;
  uint32_t qa[KB * 4][R16 ? 4 : 2];
#pragma unroll
  for (int kk = 0; kk < KB * 4; ++kk)
#pragma unroll
    for (int e = 0; e < (R16 ? 4 : 2); ++e) {  // (row, k), (row, k + 8), (row + 8, k), (row + 8, k + 8)
      const int r = row + (e >> 1) * 8;
      qa[kk][e] = 0u;
      if (r < nh && kk < ksteps)
        qa[kk][e] = *reinterpret_cast<const uint32_t*>(a.q + b * a.ldq + static_cast<long long>(h0 + r) * a.hq + kk * 16 +
                                                       cq + (e & 1) * 8);
    }
  float o[VB * 8][4];
#pragma unroll
  for (int i = 0; i < VB * 8; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[i][c] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  constexpr float kLog2e = 1.4426950408889634f;
  float sig[2] = {0.f, 0.f};
  if (a.sig_bias) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      m[e] = 0.f;
      if (row + e * 8 < nh) sig[e] = __bfloat162float(a.sig_bias[h0 + row + e * 8]) * kLog2e;
    }
  }
  const float scale_log2 = a.scale * kLog2e, cap_log2 = a.cap * kLog2e, to_cap = a.cap > 0.f ? a.scale / a.cap : 0.f;

  const int lm = lane >> 3, lr = lane & 7;  // ldmatrix: matrix and row in it
  bool ok = true;
  for (int j = 0; j < count; ++j) {
    const int slot = j % SLOTS;
    if (!mbar_wait(&full[slot], (j / SLOTS) & 1, abort_flag)) { ok = false; break; }
    const uint32_t kbase = smem_u32(ring + slot * kSlabB), vbase = kbase + KB * kGdBox;
    float s[2][4];
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[t][c] = 0.f;
#pragma unroll
    for (int kk = 0; kk < KB * 4; ++kk) {
      if (kk < ksteps) {
        // matrices: (tokens 0-7, dims k..k+7), (0-7, k+8..), (8-15, k..), (8-15, k+8..)
        const int tok = ((lm >> 1) << 3) + lr, chunk = ((kk & 3) << 1) + (lm & 1);
        uint32_t kb[4];
        ldm_x4(kbase + (kk >> 2) * kGdBox + tok * 128 + ((chunk ^ (tok & 7)) << 4), kb);
        const uint32_t qf[4] = {qa[kk][0], R16 ? qa[kk][R16 ? 2 : 0] : 0u, qa[kk][1], R16 ? qa[kk][R16 ? 3 : 0] : 0u};
        mma_bf16(s[0], qf, kb[0], kb[1]);
        mma_bf16(s[1], qf, kb[2], kb[3]);
      }
    }
    const int tok0 = slab_of(j) * kGdSlab + cq;
    uint32_t hi[4] = {0u, 0u, 0u, 0u}, low[4] = {0u, 0u, 0u, 0u};
#pragma unroll
    for (int e = 0; e < (R16 ? 2 : 1); ++e) {
      float v[4] = {s[0][2 * e], s[0][2 * e + 1], s[1][2 * e], s[1][2 * e + 1]};  // tokens tok0, +1, +8, +9
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int tok = tok0 + (c & 1) + (c >> 1) * 8;
        v[c] = a.cap > 0.f ? cap_log2 * tanh_as(v[c] * to_cap, a.q) : v[c] * scale_log2;
        if (tok >= L || (tok < lo && tok >= a.keep)) v[c] = -INFINITY;
      }
      float p[4];
      if (a.sig_bias) {
#pragma unroll
        for (int c = 0; c < 4; ++c) p[c] = rcp_fast(1.f + ex2_fast(-(v[c] + sig[e])));  // -inf: 0
        hi[e] = split2(p[0], p[1], low[e]);
        hi[2 + e] = split2(p[2], p[3], low[2 + e]);
        continue;
      }
      float mx = fmaxf(fmaxf(v[0], v[1]), fmaxf(v[2], v[3]));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      // the running maximum is raised only when a score passes it by 2^8
      const bool raise = mx > m[e] + 8.f;
      if (__any_sync(0xffffffffu, raise)) {
        const float mn = raise ? mx : m[e];
        const float sc = m[e] == -INFINITY ? 0.f : ex2_fast(m[e] - mn);
        l[e] *= sc;
#pragma unroll
        for (int i = 0; i < VB * 8; ++i) { o[i][2 * e] *= sc; o[i][2 * e + 1] *= sc; }
        m[e] = mn;
      }
      const float mref = m[e] == -INFINITY ? 0.f : m[e];
#pragma unroll
      for (int c = 0; c < 4; ++c) p[c] = ex2_fast(v[c] - mref);
      l[e] += (p[0] + p[1]) + (p[2] + p[3]);
      hi[e] = split2(p[0], p[1], low[e]);
      hi[2 + e] = split2(p[2], p[3], low[2 + e]);
    }
#pragma unroll
    for (int nd = 0; nd < VB * 4; ++nd) {
      if (nd < vtiles) {
        // matrices: (tokens 0-7, dims d..d+7), (8-15, d..), (0-7, d+8..), (8-15, d+8..), transposed on load
        const int tok = ((lm & 1) << 3) + lr, dchunk = (nd << 1) + (lm >> 1);
        uint32_t v[4];
        ldm_x4_t(vbase + (dchunk >> 3) * kGdBox + tok * 128 + (((dchunk & 7) ^ (tok & 7)) << 4), v);
        mma_bf16(o[2 * nd], hi, v[0], v[1]);
        mma_bf16(o[2 * nd + 1], hi, v[2], v[3]);
        mma_bf16(o[2 * nd], low, v[0], v[1]);
        mma_bf16(o[2 * nd + 1], low, v[2], v[3]);
      }
    }
    __syncwarp();
    if (lane == 0 && j + SLOTS < count) {
      fence_proxy_async_smem();  // the slab was read through the generic proxy; TMA writes through the async one
      issue(j + SLOTS);
    }
  }
  if (!ok) {
    *abort_flag = 1;
    if (lane == 0) atomicCAS(status, 0, kErrMbarTimeoutEpilogue);
    const unsigned long long t0 = globaltimer_ns();  // let copies already in flight land before the CTA retires
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
#pragma unroll
  for (int e = 0; e < (R16 ? 2 : 1); ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
  }
  __syncthreads();  // every warp is done with its ring: reuse it for the cross-warp merge
  constexpr int kOW = VB * 64;
  float* s_o = reinterpret_cast<float*>(dsm);       // [warp][kRows][kOW]
  float* s_ml = s_o + kGdWarps * kRows * kOW;       // [warp][kRows][2]
#pragma unroll
  for (int e = 0; e < (R16 ? 2 : 1); ++e) {
    const int r = row + e * 8;
#pragma unroll
    for (int i = 0; i < VB * 8; ++i)
      *reinterpret_cast<float2*>(s_o + (warp * kRows + r) * kOW + i * 8 + cq) = make_float2(o[i][2 * e], o[i][2 * e + 1]);
    if ((lane & 3) == 0) {
      s_ml[(warp * kRows + r) * 2] = m[e];
      s_ml[(warp * kRows + r) * 2 + 1] = l[e];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < nh * a.Dv; idx += blockDim.x) {
    const int g = idx / a.Dv, d = idx - g * a.Dv;
    float mn = -INFINITY;
#pragma unroll
    for (int w = 0; w < kGdWarps; ++w) mn = fmaxf(mn, s_ml[(w * kRows + g) * 2]);
    float lt = 0.f, at = 0.f;
#pragma unroll
    for (int w = 0; w < kGdWarps; ++w) {
      const float mw = s_ml[(w * kRows + g) * 2];
      const float sc = mw == -INFINITY ? 0.f : ex2_fast(mw - mn);
      lt += s_ml[(w * kRows + g) * 2 + 1] * sc;
      at += s_o[(w * kRows + g) * kOW + d] * sc;
    }
    const long long bh = static_cast<long long>(b) * a.H + h0 + g;
    if (a.nsplit == 1) {
      if (d < a.dv) a.out[bh * a.dv + d] = __float2bfloat16(at * gqa_final(mn, lt, h0 + g, b, a.sink, a.gate, a.ldg, a.sig_bias));
    } else {
      const long long u = bh * a.nsplit + split;
      a.o_part[u * a.Dv + d] = at;
      if (d == 0) {
        a.ml_part[u * 2] = mn;
        a.ml_part[u * 2 + 1] = lt;
      }
    }
  }
}

// One block per (sequence, head)
__global__ void gqa_merge_kernel(const GqaDecodeArgs a) {
  __shared__ float w[64];
  const long long u = blockIdx.x;
  const int h = static_cast<int>(u % a.H);
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < a.nsplit; ++s) m = fmaxf(m, a.ml_part[(u * a.nsplit + s) * 2]);
  for (int s = 0; s < a.nsplit; ++s) {
    const float ms = a.ml_part[(u * a.nsplit + s) * 2];
    const float e = ms == -INFINITY ? 0.f : ex2_fast(ms - m);
    l += a.ml_part[(u * a.nsplit + s) * 2 + 1] * e;
    if (threadIdx.x == 0) w[s] = e;
  }
  __syncthreads();
  const float f = gqa_final(m, l, h, u / a.H, a.sink, a.gate, a.ldg, a.sig_bias);
  for (int d = threadIdx.x; d < a.dv; d += blockDim.x) {
    float t = 0.f;
    for (int s = 0; s < a.nsplit; ++s)
      if (w[s] != 0.f) t = fmaf(a.o_part[(u * a.nsplit + s) * a.Dv + d], w[s], t);  // 0: an empty split
    a.out[u * a.dv + d] = __float2bfloat16(t * f);
  }
}

template <int KB, int VB, int SLOTS>
static int launch_gqa_decode(const CUtensorMap& tmK, const CUtensorMap& tmV, const GqaDecodeArgs& a, int B,
                             cudaStream_t stream) {
  constexpr int smem = kGdWarps * SLOTS * (KB + VB) * kGdBox + 1024 + 256;
  // the cross-warp merge reuses the ring
  static_assert(kGdWarps * 16 * (VB * 64 + 2) * 4 <= kGdWarps * SLOTS * (KB + VB) * kGdBox, "ring too small");
  int* status = device_status_word();
  if (!status) return -3;
  const int group = a.H / a.G;
  const dim3 grid(B, a.G * ((group + 15) / 16), a.nsplit);
#define B200_GD(R_)                                                                                              \
  {                                                                                                              \
    B200_CHECK(cudaFuncSetAttribute(gqa_decode_kernel<KB, VB, SLOTS, R_>,                                        \
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, smem));                         \
    gqa_decode_kernel<KB, VB, SLOTS, R_><<<grid, kGdWarps * 32, smem, stream>>>(tmK, tmV, a, status);            \
  }
  if (group > 8) B200_GD(true) else B200_GD(false)
#undef B200_GD
  B200_CHECK(cudaGetLastError());
  if (a.nsplit > 1) {
    gqa_merge_kernel<<<B * a.H, a.dv > 64 ? 128 : 64, 0, stream>>>(a);
    B200_CHECK(cudaGetLastError());
  }
  return 0;
}

}  // namespace b200

extern "C" {

// q [B][ldq] + h * hq (multiples of 8, zeros between a head's width and D); caches as above, 16-byte aligned; out [B, H *
// dv], dv <= Dv. o_part fp32 [B, H, nsplit, Dv] and ml_part [B, H, nsplit, 2] when nsplit > 1 (at most 64). window 0: none;
// keep counts only with a window. softcap 0: none. sink: null or [H]; gate: null or [B][ldg]; sig_bias: null, or [H] for
// sigmoid weights (without a sink).
int b200_gqa_decode(const void* q, long long ldq, int hq, const void* k_cache, const void* v_cache, const int* block_table,
                    int max_blocks, int block_size, int num_blocks, const int* seq_lens, void* out, float* o_part,
                    float* ml_part, int B, int H, int G, int D, int Dv, int dv, int nsplit, float scale, int window,
                    int keep, float softcap, const void* sink, const void* gate, long long ldg, const void* sig_bias,
                    cudaStream_t stream) {
  using namespace b200;
  if (B <= 0) return 0;
  if (G < 1 || H % G || D < 16 || Dv < 16 || D % 16 || Dv % 16 || D > 256 || Dv > 256 || dv > Dv || block_size % kGdSlab ||
      ((ldq | hq) & 7) || nsplit < 1 || nsplit > 64 || (sink && sig_bias))
    return -100;
  using bf = __nv_bfloat16;
  const auto dt = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const uint64_t rows = static_cast<uint64_t>(num_blocks) * G * block_size;
  CUtensorMap tmK, tmV;
  int rc = make_tmap_2d(&tmK, k_cache, dt, 2, rows, D, static_cast<uint64_t>(D) * 2, kGdSlab, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tmV, v_cache, dt, 2, rows, Dv, static_cast<uint64_t>(Dv) * 2, kGdSlab, 64);
  if (rc) return rc;
  const GqaDecodeArgs a{(const bf*)q, ldq, hq, block_table, seq_lens, (bf*)out, o_part, ml_part, H, G, D, Dv, dv, block_size,
                        max_blocks, nsplit, scale, softcap, window, keep, (const bf*)sink, (const bf*)gate, ldg,
                        (const bf*)sig_bias};
  if (D > 128 || Dv > 128) return launch_gqa_decode<4, 4, 3>(tmK, tmV, a, B, stream);
  if (D <= 64)
    return Dv <= 64 ? launch_gqa_decode<1, 1, 6>(tmK, tmV, a, B, stream) : launch_gqa_decode<1, 2, 4>(tmK, tmV, a, B, stream);
  return Dv <= 64 ? launch_gqa_decode<2, 1, 4>(tmK, tmV, a, B, stream) : launch_gqa_decode<2, 2, 3>(tmK, tmV, a, B, stream);
}

}  // extern "C"
