// Decode attention over the compressed latent cache on tensor cores: one query token per sequence, all heads of it
// against the same cached rows [rank | rot] (see latent_attn.cu). A cached row is read once for 16 heads and serves as
// key (all of it) and value (its first `rank` numbers), so the kernel is bound by the cache stream.
//
// One CTA per (sequence, group of 16 heads, split): 8 warps, tiles of 32 tokens in a ring of stages filled by cp.async
// (rows are padded to an odd number of 16-byte units so that ldmatrix is free of bank conflicts). A warp computes the
// scores of 8 tokens over half of the width; the [16, 32] scores meet in shared memory, every warp takes the softmax of two
// heads (max, sum and weights in fp32, a lane per token) and, with all heads' weights, multiplies its share of the value
// columns. The weights enter the product as two bf16 terms
// (hi + lo), so they keep fp32-like precision. With a window the walk starts at the tile of the first visible token; a
// gate scales a head's result by sigmoid(gate[sequence, head]) when it is written.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/mma16.cuh"

namespace b200 {

constexpr int kLdTok = 32;     // tokens per tile
constexpr int kLdWarps = 8;
constexpr int kLdSPitch = 40;  // floats per score row
constexpr int kLdPPitch = 80;  // bytes per row of weights (32 bf16 and padding)
// shared memory ahead of the queries: scores of both width halves, weights (hi, lo), correction factors, row statistics
constexpr int kLdFixed = 2 * 16 * kLdSPitch * 4 + 2 * 16 * kLdPPitch + 16 * 4 + 32 * 4 + 64;

struct LatentDecodeArgs {
  const __nv_bfloat16 *qa, *q, *cache;
  long long ldqa, ldq;
  int q_stride, q_off;  // rotated query part of head h: q + h * q_stride + q_off
  const int *block_table, *seq_lens;
  __nv_bfloat16* out;   // [B, H * rank]
  float *o_part, *ml_part;
  int H, rank, rot, block_size, max_blocks, nsplit, pitch;  // pitch: bytes of a row in shared memory
  float scale_log2;
  int window;           // 0: every cached token is visible
  const __nv_bfloat16* gate;  // null or [B][ldg]
  long long ldg;
};

__device__ __forceinline__ uint32_t sa32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }

// NP: pairs of value column tiles (16 columns) per warp; ST: stages
template <int NP, int ST>
__global__ void __launch_bounds__(kLdWarps * 32, 2) latent_decode_kernel(LatentDecodeArgs a) {
  extern __shared__ __align__(128) uint8_t sm[];
  const int W = a.rank + a.rot, pitch = a.pitch;
  float* sS = reinterpret_cast<float*>(sm);             // [width half][16][kLdSPitch]
  uint8_t* sP = sm + 2 * 16 * kLdSPitch * 4;            // [hi, lo][16][kLdPPitch]
  float* sC = reinterpret_cast<float*>(sP + 2 * 16 * kLdPPitch);  // [16] factor for what a head has accumulated
  float* sML = sC + 16;                                 // [16][2] maximum and sum at the end
  uint8_t* sQ = sm + kLdFixed;                          // [16][pitch]
  uint8_t* ring = sQ + 16 * pitch;                      // [ST][32][pitch]
  const int b = blockIdx.x, h0 = blockIdx.y * 16, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int L = a.seq_lens[b];
  const int lo = a.window > 0 ? max(0, L - a.window) : 0;  // first visible token
  const int tiles = (L + kLdTok - 1) / kLdTok, t0 = lo / kLdTok, per = (tiles - t0 + a.nsplit - 1) / a.nsplit;
  const int j0 = t0 + split * per, n = max(0, min(tiles, j0 + per) - j0);
  const int* bt = a.block_table + static_cast<long long>(b) * a.max_blocks;
  // queries: 16 rows of W, zero for heads past the last
  for (int i = threadIdx.x; i < 16 * (W / 8); i += blockDim.x) {
    const int r = i / (W / 8), c = (i % (W / 8)) * 8, h = h0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (h < a.H)
      v = c < a.rank ? *reinterpret_cast<const uint4*>(a.qa + b * a.ldqa + static_cast<long long>(h) * a.rank + c)
                     : *reinterpret_cast<const uint4*>(a.q + b * a.ldq + static_cast<long long>(h) * a.q_stride + a.q_off + c - a.rank);
    *reinterpret_cast<uint4*>(sQ + r * pitch + c * 2) = v;
  }

  // eight threads per row; rows past the end become zeros (a weight of 0 must meet a number)
  const int fr = threadIdx.x >> 3, fc = threadIdx.x & 7;
  auto page_of = [&](int j) {  // page of this thread's row of tile j (any page past the end: the row is zeroed)
    return j < n ? __ldg(bt + min((j0 + j) * kLdTok + fr, L - 1) / a.block_size) : 0;
  };
  int page = page_of(0);  // looked up one tile ahead: its latency would delay every copy
  auto fill = [&](int j) {
    if (j < n) {
      const int tok = (j0 + j) * kLdTok + fr;
      const bool in = tok < L;
      const int tk = in ? tok : L - 1;
      const __nv_bfloat16* src = a.cache + (static_cast<long long>(page) * a.block_size + tk % a.block_size) * W;
      page = page_of(j + 1);
      const uint32_t dst = sa32(ring + ((j % ST) * kLdTok + fr) * pitch);
#pragma unroll 4
      for (int c = fc; c < W / 8; c += 8)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + c * 16), "l"(src + c * 8), "r"(in ? 16 : 0)
                     : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int j = 0; j < ST - 1; ++j) fill(j);

  float o[2 * NP][4];
#pragma unroll
  for (int i = 0; i < 2 * NP; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[i][c] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // heads 2 * warp and 2 * warp + 1; l: this lane's tokens
  const int g = lane >> 2, t = lane & 3;
  const int pairs = a.rank >> 4;
  const uint32_t qrow = sa32(sQ) + (lane & 15) * pitch + (lane >> 4) * 16;
  for (int j = 0; j < n; ++j) {
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
    __syncthreads();  // tile j is here for everyone; every warp has left tile j - 1
    fill(j + ST - 1);
    const uint32_t base = sa32(ring + (j % ST) * kLdTok * pitch);
    // scores of this warp's 8 tokens over its half of the width: two blocks of 16 per ldmatrix, two chains against the
    // tensor-core latency
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
    const int tg = warp & 3, wh = warp >> 2;
    const uint32_t krow = base + (tg * 8 + (lane & 7)) * pitch + (lane >> 3) * 16;
    const int mid = (((W >> 4) + 3) >> 2) * 2, kt = wh ? W >> 4 : min(mid, W >> 4);
    int k = wh ? min(mid, W >> 4) : 0;
#pragma unroll 4
    for (; k + 2 <= kt; k += 2) {
      uint32_t kb[4], q0[4], q1[4];
      ldm_x4(krow + k * 32, kb);
      ldm_x4(qrow + k * 32, q0);
      ldm_x4(qrow + k * 32 + 32, q1);
      mma_bf16(s, q0, kb[0], kb[1]);
      mma_bf16(s2, q1, kb[2], kb[3]);
    }
    if (k < kt) {
      uint32_t kb[2], q0[4];
      ldm_x2(base + (tg * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16 + k * 32, kb);
      ldm_x4(qrow + k * 32, q0);
      mma_bf16(s, q0, kb[0], kb[1]);
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) s[c] += s2[c];
    constexpr int kHalf = 16 * kLdSPitch;
    *reinterpret_cast<float2*>(sS + wh * kHalf + g * kLdSPitch + tg * 8 + 2 * t) = make_float2(s[0], s[1]);
    *reinterpret_cast<float2*>(sS + wh * kHalf + (g + 8) * kLdSPitch + tg * 8 + 2 * t) = make_float2(s[2], s[3]);
    __syncthreads();  // scores complete
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = 2 * warp + e;
      const int tok = (j0 + j) * kLdTok + lane;
      const bool in = tok < L && tok >= lo;
      const float x = in ? (sS[r * kLdSPitch + lane] + sS[kHalf + r * kLdSPitch + lane]) * a.scale_log2 : -INFINITY;
      float mx = x;
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      // the running maximum is raised only when a score passes it by 2^8 (every tile holds at least one token)
      float corr = 1.f;
      if (mx > m[e] + 8.f) {
        corr = m[e] == -INFINITY ? 0.f : ex2_fast(m[e] - mx);
        m[e] = mx;
      }
      const float w = ex2_fast(x - m[e]);
      l[e] = l[e] * corr + w;
      const __nv_bfloat16 hi = __float2bfloat16(w);
      reinterpret_cast<__nv_bfloat16*>(sP + r * kLdPPitch)[lane] = hi;
      reinterpret_cast<__nv_bfloat16*>(sP + (16 + r) * kLdPPitch)[lane] = __float2bfloat16(w - __bfloat162float(hi));
      if (lane == 0) sC[r] = corr;
    }
    __syncthreads();  // weights complete
    const float c0 = sC[g], c1 = sC[g + 8];
    if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
      for (int i = 0; i < 2 * NP; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
    }
    uint32_t hi[2][4], lo[2][4];
    const uint32_t prow = sa32(sP) + (lane & 15) * kLdPPitch + (lane >> 4) * 16;
#pragma unroll
    for (int kb = 0; kb < 2; ++kb) {
      ldm_x4(prow + kb * 32, hi[kb]);
      ldm_x4(prow + 16 * kLdPPitch + kb * 32, lo[kb]);
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int pr = warp + i * kLdWarps;
      if (pr < pairs) {
#pragma unroll
        for (int kb = 0; kb < 2; ++kb) {
          uint32_t v[4];  // tokens 0-7 / 8-15 of the block x columns 0-7, then columns 8-15
          ldm_x4_t(base + (kb * 16 + (lane & 15)) * pitch + (pr * 16 + (lane >> 4) * 8) * 2, v);
          mma_bf16(o[2 * i], hi[kb], v[0], v[1]);
          mma_bf16(o[2 * i + 1], hi[kb], v[2], v[3]);
          mma_bf16(o[2 * i], lo[kb], v[0], v[1]);
          mma_bf16(o[2 * i + 1], lo[kb], v[2], v[3]);
        }
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const float sum = warp_sum(l[e]);
    if (lane == 0) {
      sML[(2 * warp + e) * 2] = m[e];
      sML[(2 * warp + e) * 2 + 1] = sum;
    }
  }
  __syncthreads();
  const bool direct = a.nsplit == 1;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int h = h0 + g + half * 8;
    if (h >= a.H) continue;
    const long long u = (static_cast<long long>(b) * a.H + h);
    const float sum = sML[(g + half * 8) * 2 + 1];
    float inv = sum > 0.f ? 1.f / sum : 0.f;
    if (direct && a.gate) inv *= sigmoid_as(__bfloat162float(a.gate[b * a.ldg + h]), a.gate);
#pragma unroll
    for (int i = 0; i < 2 * NP; ++i) {
      const int pr = warp + (i >> 1) * kLdWarps;
      if (pr >= pairs) continue;
      const int c = pr * 16 + (i & 1) * 8 + 2 * t;
      const float v0 = o[i][half * 2], v1 = o[i][half * 2 + 1];
      if (direct)
        *reinterpret_cast<uint32_t*>(a.out + u * a.rank + c) = pack2(v0 * inv, v1 * inv);
      else
        *reinterpret_cast<float2*>(a.o_part + (u * a.nsplit + split) * a.rank + c) = make_float2(v0, v1);
    }
    if (!direct && warp == 0 && t == 0) {
      a.ml_part[(u * a.nsplit + split) * 2] = sML[(g + half * 8) * 2];
      a.ml_part[(u * a.nsplit + split) * 2 + 1] = sum;
    }
  }
}

// One block per (sequence, head); threads over the columns, two at a time.
__global__ void latent_merge_kernel(const float* __restrict__ o_part, const float* __restrict__ ml,
                                    __nv_bfloat16* __restrict__ out, int nsplit, int rank,
                                    const __nv_bfloat16* __restrict__ gate, long long ldg, int H) {
  __shared__ float w[64];
  const long long u = blockIdx.x;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < nsplit; ++s) m = fmaxf(m, ml[(u * nsplit + s) * 2]);
  for (int s = 0; s < nsplit; ++s) {
    const float ms = ml[(u * nsplit + s) * 2];
    const float e = ms == -INFINITY ? 0.f : ex2_fast(ms - m);
    l += ml[(u * nsplit + s) * 2 + 1] * e;
    if (threadIdx.x == 0) w[s] = e;
  }
  __syncthreads();
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (gate) inv *= sigmoid_as(__bfloat162float(gate[u / H * ldg + u % H]), gate);
  for (int c = threadIdx.x * 2; c < rank; c += blockDim.x * 2) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < nsplit; ++s) {
      if (w[s] == 0.f) continue;  // an empty split
      const float2 v = *reinterpret_cast<const float2*>(o_part + (u * nsplit + s) * rank + c);
      x = fmaf(v.x, w[s], x);
      y = fmaf(v.y, w[s], y);
    }
    *reinterpret_cast<uint32_t*>(out + u * rank + c) = pack2(x * inv, y * inv);
  }
}

}  // namespace b200

extern "C" {

// 0 when the kernel takes these widths (bf16), negative otherwise.
int b200_latent_decode_ok(int rank, int rot) {
  using namespace b200;
  return (rank % 16 == 0 && rot % 16 == 0 && rank >= 16 && rank <= 512 && rot <= 128) ? 0 : -100;
}

// qa [B][ldqa]: head h at h * rank; q [B][ldq]: rotated part of head h at h * q_stride + q_off. All bf16, 16-byte
// aligned, pitches and strides multiples of 8. cache rows are rank + rot wide. nsplit <= 64.
int b200_latent_decode(const void* qa, long long ldqa, const void* q, long long ldq, int q_stride, int q_off,
                       const void* cache, const int* block_table, int max_blocks, int block_size, const int* seq_lens,
                       void* out, float* o_part, float* ml_part, int B, int H, int rank, int rot, int nsplit,
                       float scale, int window, const void* gate, long long ldg, cudaStream_t stream) {
  using namespace b200;
  if (B <= 0) return 0;
  if (b200_latent_decode_ok(rank, rot) || (ldqa & 7) || (ldq & 7) || (q_stride & 7) || (q_off & 7) || nsplit < 1 || nsplit > 64)
    return -100;
  using bf = __nv_bfloat16;
  const int W = rank + rot, pitch = ((W / 8) | 1) * 16;
  const int fixed = kLdFixed + 16 * pitch, stage = kLdTok * pitch;
  const int stages = fixed + 3 * stage <= 113 * 1024 ? 3 : 2;
  const int smem = fixed + stages * stage;
  LatentDecodeArgs a{(const bf*)qa, (const bf*)q, (const bf*)cache, ldqa, ldq, q_stride, q_off, block_table, seq_lens,
                     (bf*)out, o_part, ml_part, H, rank, rot, block_size, max_blocks, nsplit, pitch,
                     scale * 1.4426950408889634f, window, (const bf*)gate, ldg};
  dim3 grid(B, (H + 15) / 16, nsplit);
  const int np = (rank / 16 + kLdWarps - 1) / kLdWarps;
#define B200_LDS(NP_, ST_)                                                                                          \
  {                                                                                                                 \
    B200_CHECK(cudaFuncSetAttribute(latent_decode_kernel<NP_, ST_>, cudaFuncAttributeMaxDynamicSharedMemorySize,    \
                                    smem));                                                                         \
    latent_decode_kernel<NP_, ST_><<<grid, kLdWarps * 32, smem, stream>>>(a);                                       \
  }
#define B200_LD(NP_)                                                                                                \
  if (stages == 3) B200_LDS(NP_, 3) else B200_LDS(NP_, 2)
  if (np <= 1) { B200_LD(1) }
  else if (np <= 2) { B200_LD(2) }
  else { B200_LD(4) }
#undef B200_LD
#undef B200_LDS
  B200_CHECK(cudaGetLastError());
  if (nsplit > 1) {
    latent_merge_kernel<<<B * H, rank >= 256 ? 256 : 128, 0, stream>>>(o_part, ml_part, (bf*)out, nsplit, rank,
                                                                                (const bf*)gate, ldg, H);
    B200_CHECK(cudaGetLastError());
  }
  return 0;
}

}  // extern "C"
