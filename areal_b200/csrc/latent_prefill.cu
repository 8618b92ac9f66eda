// Causal attention of packed prompts for latent attention heads (tcgen05 + TMEM, sm_100a): a query / key is an unrotated
// part of D = 64 or 128 numbers per head and a rotated part of up to 64 whose key side is shared by all heads; values
// are up to 128 wide.
//
//   q [T, H * (D + R)], kv [T, H * D | H * Dv] (expanded from the latents), kr [T, R]  ->  o [T, H * Dv], all bf16
//
// Same shape as the general attention kernel (attn_fwd.cu): one CTA per (128-query tile, head), 64 keys per block, the
// scores double-buffered in TMEM, two CTAs per SM, one softmax thread per query row. What differs:
//   * S = Qn Kn^T + Qr Kr^T: the shared rotated keys are a second TMA tile, never copied per head. A rotated part
//     narrower than 64 is read as 64 columns: the columns past R are zero on the key side (out-of-range fill).
//   * the softmax weights stay in TMEM. They overwrite their own score buffer as two bf16 terms, hi (32 columns) and lo
//     (32 columns), and P V is two products with the A operand read from TMEM, so the weights keep fp32-like precision
//     and take no shared memory.
//   * a window (query i sees keys i - window + 1 .. i) starts a tile's walk at the first block that any of its queries
//     sees; a gate scales a head's result by sigmoid(gate[token, head]) on the way out.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/mma16.cuh"
#include "common/ptx.cuh"

namespace b200 {

constexpr int kLpQ = 128, kLpK = 64, kLpThreads = 192;

struct LatentTile {  // one record of VarlenMeta.fwd_tiles
  int q_start, q_len, kv_start, kv_len, q_off, pad0, pad1, pad2;
};

// D[tmem] (+)= A[tmem] * B[smem desc]: A holds two bf16 per 32-bit column, 8 columns per 16-wide reduction step
__device__ __forceinline__ void umma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc,
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

// ND: 64-column blocks of the unrotated part; NV: 64-column blocks of the values
template <int ND, int NV>
struct LpCfg {
  static constexpr int kQBlk = kLpQ * 128, kKBlk = kLpK * 128;  // bytes of one 64-column block
  static constexpr int kQ = (ND + 1) * kQBlk, kK = (ND + 1) * kKBlk, kV = NV * kKBlk;
  static constexpr int kVStages = ND + NV <= 3 ? 2 : 1;
  static constexpr int kSmem = kQ + 2 * kK + kVStages * kV;
};

template <int ND, int NV>
__global__ void __launch_bounds__(kLpThreads, 2)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV,
                      const __grid_constant__ CUtensorMap tmR, const LatentTile* __restrict__ tiles,
                      __nv_bfloat16* __restrict__ o, int H, int R, int Dv, float scale_log2, int window,
                      const __nv_bfloat16* __restrict__ gate, long long ldg, int* status) {
  using C = LpCfg<ND, NV>;
  constexpr int D = ND * 64, VS = C::kVStages;
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
  const LatentTile tile = tiles[blockIdx.x];
  const int h = blockIdx.y;
  const int blk0 = window > 0 ? max(0, tile.q_off - window + 1) / kLpK : 0;  // first block that a query of the tile sees
  const int nblk = (tile.kv_len + kLpK - 1) / kLpK - blk0;

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
    prefetch_tmap(&tmKV);
    prefetch_tmap(&tmR);
  }
  if (warp == 5) {
    tmem_alloc(&tmem_holder, 256);
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
      mbar_arrive_expect_tx(q_full, C::kQ);
#pragma unroll
      for (int c = 0; c <= ND; ++c) tma_load_2d(sQ + c * C::kQBlk, &tmQ, q_full, h * (D + R) + c * 64, tile.q_start);
      bool ok = true;
      for (int j = 0; j < nblk; ++j) {
        const int st = j & 1, row = tile.kv_start + (blk0 + j) * kLpK;
        if (!mbar_wait(&k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_arrive_expect_tx(&k_full[st], C::kK);
        uint8_t* k = sK + st * C::kK;
#pragma unroll
        for (int c = 0; c < ND; ++c) tma_load_2d(k + c * C::kKBlk, &tmKV, &k_full[st], h * D + c * 64, row);
        tma_load_2d(k + ND * C::kKBlk, &tmR, &k_full[st], 0, row);
        const int vs = j % VS;
        if (!mbar_wait(&v_empty[vs], ((j / VS) & 1) ^ 1, abort_flag)) { ok = false; break; }
        mbar_arrive_expect_tx(&v_full[vs], C::kV);
#pragma unroll
        for (int c = 0; c < NV; ++c)
          tma_load_2d(sV + vs * C::kV + c * C::kKBlk, &tmKV, &v_full[vs], H * D + h * Dv + c * 64, row);
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
      constexpr uint32_t idesc_s = make_idesc(1, 1, 0, 0, kLpQ, kLpK);
      constexpr uint32_t idesc_o = make_idesc(1, 1, 0, 1, kLpQ, NV * 64);
      bool ok = mbar_wait(q_full, 0, abort_flag);
      const uint32_t q_addr = smem_u32(sQ);
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1, abort_flag)) return false;
        tc_fence_after();
        const uint32_t k_addr = smem_u32(sK + st * C::kK);
#pragma unroll
        for (int k = 0; k < (ND + 1) * 4; ++k) {
          const uint64_t a = make_sdesc_sw128(q_addr + (k >> 2) * C::kQBlk + (k & 3) * 32, 16, 1024);
          const uint64_t b = make_sdesc_sw128(k_addr + (k >> 2) * C::kKBlk + (k & 3) * 32, 16, 1024);
          umma_f16(tmem_base + st * kLpK, a, b, idesc_s, k > 0 ? 1u : 0u);
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
        const uint32_t v_addr = smem_u32(sV + vs * C::kV), p_addr = tmem_base + (j & 1) * kLpK;
#pragma unroll
        for (int k = 0; k < 8; ++k) {  // 4 reduction steps with the leading terms, 4 with the remainders
          const uint64_t b = make_sdesc_sw128(v_addr + (k & 3) * 2048, C::kKBlk, 1024);
          umma_f16_ts(tmem_O, p_addr + k * 8, b, idesc_o, (j > 0 || k > 0) ? 1u : 0u);
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
    const int q_pos = tile.q_off + r, q_lo = window > 0 ? q_pos - window + 1 : 0;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nblk; ++j) {
      const uint32_t s_addr = tmem_base + lane_addr + (j & 1) * kLpK;
      if (!mbar_wait(&s_full[j & 1], (j >> 1) & 1, abort_flag)) { ok = false; break; }
      tc_fence_after();
      float s[kLpK];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t raw[32];
        tmem_ld_32x32(s_addr + c * 32, raw);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[c * 32 + i] = __uint_as_float(raw[i]) * scale_log2;
      }
      const int kv0 = (blk0 + j) * kLpK;
      // the diagonal, the end of the tile's keys, or the window's edge for the tile's last query
      if (kv0 + kLpK - 1 > tile.q_off || kv0 + kLpK > tile.kv_len ||
          (window > 0 && kv0 < tile.q_off + kLpQ - window)) {
#pragma unroll
        for (int i = 0; i < kLpK; ++i)
          if (kv0 + i > q_pos || kv0 + i >= tile.kv_len || kv0 + i < q_lo) s[i] = -INFINITY;
      }
      float mx = s[0];
#pragma unroll
      for (int i = 1; i < kLpK; ++i) mx = fmaxf(mx, s[i]);
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
      const float mref = m == -INFINITY ? 0.f : m;
      uint32_t hi[32], lo[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float a = ex2_fast(s[2 * i] - mref), b = ex2_fast(s[2 * i + 1] - mref);
        l += a + b;
        hi[i] = split2(a, b, lo[i]);
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
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (gate && r < tile.q_len)
        inv *= sigmoid_as(__bfloat162float(gate[static_cast<long long>(tile.q_start + r) * ldg + h]), gate);
      __nv_bfloat16* orow = o + (static_cast<long long>(tile.q_start + r) * H + h) * Dv;
#pragma unroll 1
      for (int c = 0; c < NV * 2; ++c) {
        uint32_t raw[32];
        tmem_ld_32x32(tmem_O + lane_addr + c * 32, raw);
        tmem_ld_wait();
        if (r < tile.q_len) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 < Dv) {
              uint4 pk;
              pk.x = pack2(__uint_as_float(raw[i * 8]) * inv, __uint_as_float(raw[i * 8 + 1]) * inv);
              pk.y = pack2(__uint_as_float(raw[i * 8 + 2]) * inv, __uint_as_float(raw[i * 8 + 3]) * inv);
              pk.z = pack2(__uint_as_float(raw[i * 8 + 4]) * inv, __uint_as_float(raw[i * 8 + 5]) * inv);
              pk.w = pack2(__uint_as_float(raw[i * 8 + 6]) * inv, __uint_as_float(raw[i * 8 + 7]) * inv);
              *reinterpret_cast<uint4*>(orow + c * 32 + i * 8) = pk;
            }
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
    tmem_dealloc(tmem_base, 256);
  }
}

template <int ND, int NV>
static int launch_latent_prefill(const CUtensorMap& tmQ, const CUtensorMap& tmKV, const CUtensorMap& tmR, const void* tiles,
                                 int n_tiles, void* o, int H, int R, int Dv, float scale, int window,
                                 const void* gate, long long ldg, cudaStream_t stream) {
  constexpr int smem = LpCfg<ND, NV>::kSmem;
  B200_CHECK(cudaFuncSetAttribute(latent_prefill_kernel<ND, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  int* status = device_status_word();
  if (!status) return -3;
  latent_prefill_kernel<ND, NV><<<dim3(n_tiles, H), kLpThreads, smem, stream>>>(
      tmQ, tmKV, tmR, reinterpret_cast<const LatentTile*>(tiles), (__nv_bfloat16*)o, H, R, Dv,
      scale * 1.4426950408889634f, window, (const __nv_bfloat16*)gate, ldg, status);
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace b200

extern "C" {

// q [T][ldq] (H * (D + R) columns, pitch a multiple of 8); contiguous kv [T, H * (D + Dv)], kr [T, R], o [T, H * Dv]; all
// 16-byte aligned. window: 0 for none. gate: null or [T][ldg], one number per head.
int b200_latent_prefill(const void* q, long long ldq, const void* kv, const void* kr, void* o, const void* tiles,
                        int n_tiles, int T, int H, int D, int R, int Dv, float scale, int window, const void* gate,
                        long long ldg, cudaStream_t stream) {
  using namespace b200;
  if (T <= 0 || n_tiles <= 0) return 0;
  if ((D != 64 && D != 128) || R < 8 || R > 64 || R % 8 || (ldq & 7) || Dv < 8 || Dv > 128 || Dv % 8) return -100;
  CUtensorMap tmQ, tmKV, tmR;
  const auto bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const uint64_t wq = static_cast<uint64_t>(H) * (D + R), wkv = static_cast<uint64_t>(H) * (D + Dv);
  int rc = make_tmap_2d(&tmQ, q, bf, 2, T, wq, static_cast<uint64_t>(ldq) * 2, kLpQ, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tmKV, kv, bf, 2, T, wkv, wkv * 2, kLpK, 64);
  if (rc) return rc;
  rc = make_tmap_2d(&tmR, kr, bf, 2, T, R, static_cast<uint64_t>(R) * 2, kLpK, 64);
  if (rc) return rc;
  if (D == 64)
    return Dv <= 64 ? launch_latent_prefill<1, 1>(tmQ, tmKV, tmR, tiles, n_tiles, o, H, R, Dv, scale, window, gate, ldg, stream)
                    : launch_latent_prefill<1, 2>(tmQ, tmKV, tmR, tiles, n_tiles, o, H, R, Dv, scale, window, gate, ldg, stream);
  return Dv <= 64 ? launch_latent_prefill<2, 1>(tmQ, tmKV, tmR, tiles, n_tiles, o, H, R, Dv, scale, window, gate, ldg, stream)
                  : launch_latent_prefill<2, 2>(tmQ, tmKV, tmR, tiles, n_tiles, o, H, R, Dv, scale, window, gate, ldg, stream);
}

}  // extern "C"
