// Causal grouped-query attention of packed prompts (tcgen05 + TMEM, sm_100a) for heads of up to 256 with the options of
// ops/gqa.py: a window that keeps the first tokens, a soft cap on the scores, a sink, a gate per head, sigmoids as weights.
//
//   q [T, H heads], k [T, G heads], v [T, G heads], each head at its own stride inside a row  ->  o [T, H * Dv], all bf16
//
// Same shape as latent_prefill.cu: one CTA per (128-query tile, head), 64 keys per block, scores double-buffered in TMEM,
// one softmax thread per query row, softmax weights as two bf16 terms (hi, lo) in TMEM, from where the second product
// reads them. What differs:
//   * heads are read where they lie: 64-column boxes may run into the next head, the products stop at the head's own
//     width (steps of 16).
//   * the walk over key blocks has two parts: the blocks of the first tokens that a window keeps, then those that any
//     query of the tile sees through its window.
//   * scores that cannot be large (q and k of unit mean square, or capped) need no running maximum: the weights are
//     2^score, and neither maxima nor rescaled accumulators are needed (kBounded). Sigmoid weights (kSigmoid) need neither
//     these nor a sum.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/mma16.cuh"
#include "common/ptx.cuh"

namespace b200 {

constexpr int kGpQ = 128, kGpK = 64, kGpThreads = 192;

enum : int { kRunningMax = 0, kBounded = 1, kSigmoid = 2 };

struct GqaTile {  // one record of VarlenMeta.fwd_tiles
  int q_start, q_len, kv_start, kv_len, q_off, pad0, pad1, pad2;
};

// D[tmem] (+)= A[tmem] * B[smem desc]: A holds two bf16 per 32-bit column, 8 columns per 16-wide reduction step
__device__ __forceinline__ void gqa_umma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n"
      ".reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n"
      "}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// ND / NV: 64-column blocks of queries and keys / values
template <int ND, int NV>
struct GpCfg {
  static constexpr int kQBlk = kGpQ * 128, kKBlk = kGpK * 128;  // bytes of one 64-column block
  static constexpr int kQ = ND * kQBlk, kK = ND * kKBlk, kV = NV * kKBlk;
  static constexpr bool kWide = ND > 2 || NV > 2;
  static constexpr int kVStages = kWide ? 1 : 2;
  static constexpr int kTmem = kWide ? 512 : 256;
  static constexpr int kSmem = kQ + 2 * kK + kVStages * kV;
};

struct GqaPrefillArgs {
  const GqaTile* tiles;
  __nv_bfloat16* o;
  int H, group, D, Dv;     // D in steps of 16
  int hq, hk, hv;          // head strides
  float scale, cap;        // cap: 0 for none
  int cap_terms;           // > 0: |score / cap| is small enough for the first 4 or 6 terms of tanh's series, whose
  float cap_c[6];          // coefficients, in powers of (q . k)^2, give the capped score over q . k in units of log 2
  int window, keep;        // 0: none
  const __nv_bfloat16* sink;
  const __nv_bfloat16* gate;
  long long ldg;
  const __nv_bfloat16* sig_bias;  // kSigmoid: [H], added to the scores
};

template <int N>
__device__ __forceinline__ float cap_series(float x, const float* c) {
  const float u = x * x;
  float p = c[N - 1];
#pragma unroll
  for (int i = N - 2; i >= 0; --i) p = fmaf(u, p, c[i]);
  return x * p;
}

template <int ND, int NV, int MODE>
__global__ void __launch_bounds__(kGpThreads, GpCfg<ND, NV>::kWide ? 1 : 2)
gqa_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, const GqaPrefillArgs a, int* status) {
  using C = GpCfg<ND, NV>;
  constexpr bool BOUNDED = MODE != kRunningMax;
  constexpr int VS = C::kVStages;
  constexpr float kLog2e = 1.4426950408889634f;
  extern __shared__ __align__(1024) uint8_t smem[];
  __shared__ uint64_t bars[16];
  __shared__ uint32_t tmem_holder;
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + C::kQ;
  uint8_t* sV = sK + 2 * C::kK;
  uint64_t *q_full = &bars[0], *k_full = &bars[1], *k_empty = &bars[3], *v_full = &bars[5], *v_empty = &bars[7],
           *s_full = &bars[9], *p_ready = &bars[11], *pv_done = &bars[13];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const GqaTile tile = a.tiles[blockIdx.x];
  const int h = blockIdx.y, hk = h / a.group;
  // first block inside the window of any query, and the blocks of kept tokens ahead of it
  const int blk0 = a.window > 0 ? max(0, tile.q_off - a.window + 1) / kGpK : 0;
  const int nkeep = min((a.keep + kGpK - 1) / kGpK, blk0);
  const int nblk = (tile.kv_len + kGpK - 1) / kGpK - blk0 + nkeep;
  const int skip = blk0 - nkeep;
  auto block_of = [&](int j) { return j < nkeep ? j : j + skip; };
  const int kboxes = (a.D + 63) >> 6, vboxes = (a.Dv + 63) >> 6;

  if (threadIdx.x == 0) {
    abort_word = 0;
    if (smem_u32(smem) & 1023) {
      atomicCAS(status, 0, kErrBounds);
      abort_word = 1;
    }
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1);
      // one per score buffer: a role may be a whole block ahead of what another has looked at
      mbar_init(&p_ready[i], 128);
      mbar_init(&pv_done[i], 1);
    }
    fence_mbar_init();
    prefetch_tmap(&tmQ);
    prefetch_tmap(&tmK);
    prefetch_tmap(&tmV);
  }
  if (warp == 5) {
    tmem_alloc(&tmem_holder, C::kTmem);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_holder, tmem_O = tmem_base + 128;
  const bool bad = abort_word != 0;

  if (bad) {
    // fall through to teardown
  } else if (warp == 4) {
    // ------------------------------------------------------ TMA producer --
    if (elect_one_sync()) {
      mbar_arrive_expect_tx(q_full, kboxes * C::kQBlk);
      for (int c = 0; c < kboxes; ++c) tma_load_2d(sQ + c * C::kQBlk, &tmQ, q_full, h * a.hq + c * 64, tile.q_start);
      bool ok = true;
      for (int j = 0; j < nblk; ++j) {
        const int st = j & 1, row = tile.kv_start + block_of(j) * kGpK;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_arrive_expect_tx(&k_full[st], kboxes * C::kKBlk);
        for (int c = 0; c < kboxes; ++c)
          tma_load_2d(sK + st * C::kK + c * C::kKBlk, &tmK, &k_full[st], hk * a.hk + c * 64, row);
        const int vs = j % VS;
        if (!mbar_wait(&v_empty[vs], ((j / VS) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_arrive_expect_tx(&v_full[vs], vboxes * C::kKBlk);
        for (int c = 0; c < vboxes; ++c)
          tma_load_2d(sV + vs * C::kV + c * C::kKBlk, &tmV, &v_full[vs], hk * a.hv + c * 64, row);
      }
      if (!ok) {
        *abort_flag = 1;
        atomicCAS(status, 0, kErrMbarTimeoutProducer);
        const unsigned long long t0 = globaltimer_ns();  // copies in flight land before the CTA retires
        while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
      }
    }
  } else if (warp == 5) {
    // -------------------------------------------------------- MMA issuer --
    if (elect_one_sync()) {
      constexpr uint32_t idesc_s = make_idesc(1, 1, 0, 0, kGpQ, kGpK);
      const uint32_t idesc_o = make_idesc(1, 1, 0, 1, kGpQ, (a.Dv + 15) & ~15);
      const int ksteps = a.D >> 4;
      bool ok = mbar_wait(q_full, 0, abort_flag);
      const uint32_t q_addr = smem_u32(sQ);
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + st * C::kK);
        for (int k = 0; k < ksteps; ++k) {
          const uint64_t ad = make_sdesc_sw128(q_addr + (k >> 2) * C::kQBlk + (k & 3) * 32, 16, 1024);
          const uint64_t bd = make_sdesc_sw128(k_addr + (k >> 2) * C::kKBlk + (k & 3) * 32, 16, 1024);
          umma_f16(tmem_base + st * kGpK, ad, bd, idesc_s, k > 0 ? 1u : 0u);
        }
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[st]);
        return true;
      };
      if (ok && nblk > 0) ok = issue_s(0);
      for (int j = 0; j < nblk && ok; ++j) {
        const int vs = j % VS;
        // the other score buffer held the weights of block j - 1, whose product was issued before this one: products
        // of one CTA run in issue order
        if (j + 1 < nblk && !issue_s(j + 1)) { ok = false; break; }
        if (!mbar_wait(&p_ready[j & 1], (j >> 1) & 1, abort_flag)) { ok = false; break; }
        if (!mbar_wait(&v_full[vs], (j / VS) & 1, abort_flag)) { ok = false; break; }
        tc_fence_after();
        const uint32_t v_addr = smem_u32(sV + vs * C::kV), p_addr = tmem_base + (j & 1) * kGpK;
#pragma unroll
        for (int k = 0; k < 8; ++k) {  // 4 reduction steps with the leading terms, 4 with the remainders
          const uint64_t b = make_sdesc_sw128(v_addr + (k & 3) * 2048, C::kKBlk, 1024);
          gqa_umma_ts(tmem_O, p_addr + k * 8, b, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
        }
        umma_commit(&v_empty[vs]);
        umma_commit(&pv_done[j & 1]);
      }
      if (!ok) {
        *abort_flag = 1;
        atomicCAS(status, 0, kErrMbarTimeoutMma);
      }
    }
  } else {
    // ----------------------------------------------------------- softmax --
    const int r = warp * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    const int q_pos = tile.q_off + r, q_lo = a.window > 0 ? q_pos - a.window + 1 : 0;
    const float scale_log2 = a.scale * kLog2e, cap_log2 = a.cap * kLog2e, to_cap = a.cap > 0.f ? a.scale / a.cap : 0.f;
    const float sig_log2 = MODE == kSigmoid ? __bfloat162float(a.sig_bias[h]) * kLog2e : 0.f;
    float m = BOUNDED ? 0.f : -INFINITY, l = MODE == kSigmoid ? 1.f : 0.f;
    bool ok = true;
    for (int j = 0; j < nblk; ++j) {
      const uint32_t s_addr = tmem_base + lane_addr + (j & 1) * kGpK;
      if (!mbar_wait(&s_full[j & 1], (j >> 1) & 1, abort_flag)) { ok = false; break; }
      tc_fence_after();
      float s[kGpK];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t raw[32];
        tmem_ld_32x32(s_addr + c * 32, raw);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[c * 32 + i] = __uint_as_float(raw[i]);
      }
      // scores in units of log 2
      if (a.cap <= 0.f) {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) s[i] *= scale_log2;
      } else if (a.cap_terms == 4) {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) s[i] = cap_series<4>(s[i], a.cap_c);
      } else if (a.cap_terms == 6) {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) s[i] = cap_series<6>(s[i], a.cap_c);
      } else {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) s[i] = cap_log2 * tanh_as(s[i] * to_cap, a.o);
      }
      if constexpr (MODE == kSigmoid) {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) s[i] += sig_log2;
      }
      const int kv0 = block_of(j) * kGpK;
      // the diagonal, the end of the tile's keys, or the window's edge for the tile's last query
      if (kv0 + kGpK - 1 > tile.q_off || kv0 + kGpK > tile.kv_len ||
          (a.window > 0 && kv0 < tile.q_off + kGpQ - a.window && kv0 + kGpK > a.keep)) {
#pragma unroll
        for (int i = 0; i < kGpK; ++i) {
          const int kv = kv0 + i;
          if (kv > q_pos || kv >= tile.kv_len || (kv < q_lo && kv >= a.keep)) s[i] = -INFINITY;
        }
      }
      if constexpr (!BOUNDED) {
        float mx = s[0];
#pragma unroll
        for (int i = 1; i < kGpK; ++i) mx = fmaxf(mx, s[i]);
        // The row maximum is raised when it grows by 2^8. The accumulator may be rescaled only between two products:
        // that of block j - 2 is complete (the scores of block j were issued behind it), j - 1 is waited for here. The
        // weights themselves need no wait: their buffer was last read by block j - 2.
        const bool grow = mx > m + 8.f;
        if (__any_sync(0xffffffffu, grow)) {
          if (j > 0) {
            if (!mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, abort_flag)) { ok = false; break; }
            tc_fence_after();
          }
          const float mn = grow ? mx : m;
          const float alpha = m == -INFINITY ? (mn == -INFINITY ? 1.f : 0.f) : ex2_fast(m - mn);
          l *= alpha;
          m = mn;
          if (j > 0) {
#pragma unroll 1
            for (int c = 0; c < NV * 2; ++c) {
              uint32_t raw[32];
              tmem_ld_32x32(tmem_O + lane_addr + c * 32, raw);
              tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) raw[i] = __float_as_uint(__uint_as_float(raw[i]) * alpha);
              tmem_st_32x32(tmem_O + lane_addr + c * 32, raw);
            }
          }
        }
      }
      const float mref = m == -INFINITY ? 0.f : m;
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        float x, y;
        if constexpr (MODE == kSigmoid) {
          // 1 / (1 + 2^-s) for two scores with one reciprocal; weights below 2^-60 become 0
          const float u = 1.f + ex2_fast(fminf(-s[2 * i], 60.f)), v = 1.f + ex2_fast(fminf(-s[2 * i + 1], 60.f));
          const float r = rcp_fast(u * v);
          x = s[2 * i] < -60.f ? 0.f : v * r;
          y = s[2 * i + 1] < -60.f ? 0.f : u * r;
        } else {
          x = ex2_fast(BOUNDED ? s[2 * i] : s[2 * i] - mref);
          y = ex2_fast(BOUNDED ? s[2 * i + 1] : s[2 * i + 1] - mref);
          l += x + y;
        }
        hi[i] = split2(x, y, lo[i]);
      }
      tmem_st_32x32(s_addr, hi);
      tmem_st_32x32(s_addr + 32, lo);
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_ready[j & 1]);
    }
    if (ok && nblk > 0) {
      ok = mbar_wait(&pv_done[(nblk - 1) & 1], ((nblk - 1) >> 1) & 1, abort_flag);  // products run in issue order
      tc_fence_after();
    }
    if (ok) {
      float f = 1.f;  // on the accumulators
      if (a.sink) {   // one more term in the denominator, against the larger of both references
        const float sv = __bfloat162float(a.sink[h]) * kLog2e, mn = fmaxf(m, sv);
        f = m == -INFINITY ? 0.f : ex2_fast(m - mn);
        l = l * f + ex2_fast(sv - mn);
      }
      float inv = l > 0.f ? f / l : 0.f;
      if (a.gate && r < tile.q_len)
        inv *= sigmoid_as(__bfloat162float(a.gate[static_cast<long long>(tile.q_start + r) * a.ldg + h]), a.gate);
      __nv_bfloat16* orow = a.o + (static_cast<long long>(tile.q_start + r) * a.H + h) * a.Dv;
      const bool vec = (a.Dv & 7) == 0;
#pragma unroll 1
      for (int c = 0; c * 32 < a.Dv; ++c) {
        uint32_t raw[32];
        tmem_ld_32x32(tmem_O + lane_addr + c * 32, raw);
        tmem_ld_wait();
        if (r < tile.q_len) {
          if (vec) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              if (c * 32 + i * 8 < a.Dv) {
                uint4 pk;
                pk.x = pack2(__uint_as_float(raw[i * 8]) * inv, __uint_as_float(raw[i * 8 + 1]) * inv);
                pk.y = pack2(__uint_as_float(raw[i * 8 + 2]) * inv, __uint_as_float(raw[i * 8 + 3]) * inv);
                pk.z = pack2(__uint_as_float(raw[i * 8 + 4]) * inv, __uint_as_float(raw[i * 8 + 5]) * inv);
                pk.w = pack2(__uint_as_float(raw[i * 8 + 6]) * inv, __uint_as_float(raw[i * 8 + 7]) * inv);
                *reinterpret_cast<uint4*>(orow + c * 32 + i * 8) = pk;
              }
            }
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (c * 32 + i < a.Dv) orow[c * 32 + i] = __float2bfloat16(__uint_as_float(raw[i]) * inv);
          }
        }
      }
    } else if (lane == 0) {
      *abort_flag = 1;
      atomicCAS(status, 0, kErrMbarTimeoutEpilogue);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::kTmem);
  }
}

template <int ND, int NV, int MODE>
static int launch_gqa_prefill(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV,
                              const GqaPrefillArgs& a, int n_tiles, cudaStream_t stream) {
  constexpr int smem = GpCfg<ND, NV>::kSmem;
  B200_CHECK(cudaFuncSetAttribute(gqa_prefill_kernel<ND, NV, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  int* status = device_status_word();
  if (!status) return -3;
  gqa_prefill_kernel<ND, NV, MODE><<<dim3(n_tiles, a.H), kGpThreads, smem, stream>>>(tmQ, tmK, tmV, a, status);
  B200_CHECK(cudaGetLastError());
  return 0;
}

template <int MODE>
static int pick_gqa_prefill(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV, const GqaPrefillArgs& a,
                            int n_tiles, cudaStream_t stream) {
  if (a.D > 128 || a.Dv > 128) return launch_gqa_prefill<4, 4, MODE>(tmQ, tmK, tmV, a, n_tiles, stream);
  if (a.D <= 64)
    return a.Dv <= 64 ? launch_gqa_prefill<1, 1, MODE>(tmQ, tmK, tmV, a, n_tiles, stream)
                      : launch_gqa_prefill<1, 2, MODE>(tmQ, tmK, tmV, a, n_tiles, stream);
  return a.Dv <= 64 ? launch_gqa_prefill<2, 1, MODE>(tmQ, tmK, tmV, a, n_tiles, stream)
                    : launch_gqa_prefill<2, 2, MODE>(tmQ, tmK, tmV, a, n_tiles, stream);
}

}  // namespace b200

extern "C" {

// q [T][ldq] + h * hq, k [T][ldk] + g * hk, v [T][ldv] + g * hv, all bf16 and 16-byte aligned with pitches and strides in
// multiples of 8; columns of q and k between a head's width and D (a multiple of 16) are zeros. o [T, H * Dv] contiguous.
// score_bound: largest |scale * q . k| (0: unknown). window 0: none; keep counts only with a window. softcap 0: none.
// sink: null or [H]; gate: null or [T][ldg]; sig_bias: null, or [H] for sigmoid weights (without a sink).
int b200_gqa_prefill(const void* q, long long ldq, int hq, const void* k, long long ldk, int hk, const void* v,
                     long long ldv, int hv, void* o, const void* tiles, int n_tiles, int T, int H, int G, int D, int Dv,
                     float scale, float score_bound, int window, int keep, float softcap, const void* sink,
                     const void* gate, long long ldg, const void* sig_bias, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || n_tiles <= 0) return 0;
  if (D < 16 || D > 256 || D % 16 || Dv < 1 || Dv > 256 || G < 1 || H % G || ((ldq | hq | ldk | hk | ldv | hv) & 7) ||
      (sink && sig_bias))
    return -100;
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  CUtensorMap tmQ, tmK, tmV;
  int rc = make_tmap_2d(&tmQ, q, bf, 2, T, static_cast<uint64_t>(H - 1) * hq + D, static_cast<uint64_t>(ldq) * 2, kGpQ, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tmK, k, bf, 2, T, static_cast<uint64_t>(G - 1) * hk + D, static_cast<uint64_t>(ldk) * 2, kGpK, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tmV, v, bf, 2, T, static_cast<uint64_t>(G - 1) * hv + Dv, static_cast<uint64_t>(ldv) * 2, kGpK, 64);
  if (rc) return rc;
  const float log2e = 1.4426950408889634f;
  float bound = score_bound;
  if (softcap > 0.f && (bound <= 0.f || softcap < bound)) bound = softcap;
  GqaPrefillArgs a{reinterpret_cast<const GqaTile*>(tiles), (__nv_bfloat16*)o, H, H / G, D, Dv, hq, hk, hv, scale, softcap,
                   0, {}, window, keep, (const __nv_bfloat16*)sink, (const __nv_bfloat16*)gate, ldg,
                   (const __nv_bfloat16*)sig_bias};
  if (softcap > 0.f && score_bound > 0.f && score_bound <= 0.5f * softcap) {
    // cap * tanh(s / cap) = s (1 - r / 3 + 2 r^2 / 15 - 17 r^3 / 315 + ...), r = (s / cap)^2. What is left out is below 1e-6
    // of the score: 4 terms up to s / cap = 0.25, 6 terms up to 0.5.
    const double c[6] = {1.0, -1.0 / 3, 2.0 / 15, -17.0 / 315, 62.0 / 2835, -1382.0 / 155925};
    const double r = static_cast<double>(scale) / softcap;
    double f = static_cast<double>(scale) * 1.4426950408889634;
    for (int i = 0; i < 6; ++i, f *= r * r) a.cap_c[i] = static_cast<float>(c[i] * f);
    a.cap_terms = score_bound <= 0.25f * softcap ? 4 : 6;
  }
  if (sig_bias) return pick_gqa_prefill<kSigmoid>(tmQ, tmK, tmV, a, n_tiles, stream);
  // 2^(-64 .. 64): neither the weights, their sums nor the two-term split leave the range of fp32 and bf16
  return bound > 0.f && bound * log2e <= 64.f ? pick_gqa_prefill<kBounded>(tmQ, tmK, tmV, a, n_tiles, stream)
                                              : pick_gqa_prefill<kRunningMax>(tmQ, tmK, tmV, a, n_tiles, stream);
}

}  // extern "C"
