// Gated linear recurrences with an outer-product write, on packed variable-length sequences and for single decode
// steps:
//
//   S_t = diag(f_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t        per head, S [D, Dv] fp32
//
//   mode 0, HGRN2 (Qin et al., "HGRN2: Gated Linear RNNs with State Expansion"): the input row of a token holds
//     [q | f | v];  q <- silu(q),  f <- l + (1 - l) sigmoid(f + bias) per channel,  k = 1 - f.
//   mode 1, lightning attention with one constant decay per head: the row holds [q | k | v | gate];
//     q, k, v <- silu, f = decay[head].
//
// The activations are applied on load; the state and everything that enters it is fp32. The state of a sequence
// lives in state[slot] ([slots, H, D, Dv]); a prefill starts from zero and leaves the final state there, a decode
// step advances it in place. The linear-attention kernels beside this one (linear_attn.cu) cover a scalar decay per
// token with bf16 inputs that were activated beforehand.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/scan_inputs.cuh"

namespace b200 {

// Token-by-token form for any D and Dv: one block per (sequence, head, 32 value columns). Lane = column, the warps
// split the rows; the state slice [D][32] stays in shared memory. Tokens come in groups of kGrp whose activations are
// computed together.
constexpr int kGrp = 8;
template <class T>
__global__ void scan_tokens_kernel(ScanArgs a) {
  extern __shared__ float sm[];
  const int D = a.D, nw = blockDim.x >> 5, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* S = sm;                    // [D][32]
  float* sq = S + D * 32;           // [kGrp][D]
  float* sf = sq + kGrp * D;
  float* sk = sf + kGrp * D;
  float* part = sk + kGrp * D;      // [kGrp][nw][32]
  const int seq = blockIdx.x, h = blockIdx.y, j = blockIdx.z * 32 + lane;
  const int t0 = a.cu[seq], t1 = a.cu[seq + 1];
  for (int i = threadIdx.x; i < D * 32; i += blockDim.x) S[i] = 0.f;
  for (int tb = t0; tb < t1; tb += kGrp) {
    const int n = min(kGrp, t1 - tb);
    __syncthreads();
    for (int i = threadIdx.x; i < n * D; i += blockDim.x) {
      const int g = i / D, d = i % D;
      scan_channel(a, static_cast<const T*>(a.x) + (tb + g) * a.ldx, h, d, sq[g * D + d], sf[g * D + d], sk[g * D + d]);
    }
    __syncthreads();
    for (int g = 0; g < n; ++g) {
      const float v = j < a.Dv ? scan_value(a, static_cast<const T*>(a.x) + (tb + g) * a.ldx, h, j) : 0.f;
      float acc = 0.f;
      for (int d = warp; d < D; d += nw) {
        const float s = fmaf(sf[g * D + d], S[d * 32 + lane], sk[g * D + d] * v);
        S[d * 32 + lane] = s;
        acc = fmaf(s, sq[g * D + d], acc);
      }
      part[(g * nw + warp) * 32 + lane] = acc;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n * 32; i += blockDim.x) {
      const int g = i >> 5, c = blockIdx.z * 32 + (i & 31);
      float acc = 0.f;
      for (int w = 0; w < nw; ++w) acc += part[(g * nw + w) * 32 + (i & 31)];
      if (c < a.Dv) a.o[(static_cast<long long>(tb + g) * a.H + h) * a.Dv + c] = acc;
    }
  }
  __syncthreads();
  const int slot = a.slots ? a.slots[seq] : -1;
  if (slot >= 0)
    for (int i = threadIdx.x; i < D * 32; i += blockDim.x) {
      const int d = i >> 5, c = blockIdx.z * 32 + (i & 31);
      if (c < a.Dv) a.state[((static_cast<long long>(slot) * a.H + h) * D + d) * a.Dv + c] = S[i];
    }
}

// Decode step: one block per (sequence, head). Threads form rows x column groups of V; the state is streamed once
// through registers and written back in place. With norm_w (mode 0) the head's RMS norm is applied here and y gets the
// model's dtype; without it the raw fp32 output goes to o.
template <class T, int V>
__global__ void scan_step_kernel(ScanArgs a, const T* __restrict__ norm_w, T* __restrict__ y, float eps) {
  extern __shared__ float sm[];
  __shared__ float red[33];
  const int D = a.D, Dv = a.Dv, b = blockIdx.x, h = blockIdx.y;
  float* sq = sm;
  float* sf = sq + D;
  float* sk = sf + D;
  float* sv = sk + D;         // [Dv]
  float* part = sv + Dv;      // [row groups][Dv]
  const int slot = a.slots[b];
  const long long ob = (static_cast<long long>(b) * a.H + h) * Dv;
  if (slot < 0) {             // padding row of a fixed-size batch
    for (int c = threadIdx.x; c < Dv; c += blockDim.x) {
      if (norm_w) st1(y + ob + c, 0.f);
      else a.o[ob + c] = 0.f;
    }
    return;
  }
  const T* row = static_cast<const T*>(a.x) + b * a.ldx;
  for (int d = threadIdx.x; d < D; d += blockDim.x) scan_channel(a, row, h, d, sq[d], sf[d], sk[d]);
  for (int c = threadIdx.x; c < Dv; c += blockDim.x) sv[c] = scan_value(a, row, h, c);
  __syncthreads();
  float* S = a.state + (static_cast<long long>(slot) * a.H + h) * D * Dv;
  const int ncg = Dv / V;                                  // column groups
  const int cgt = ncg < (int)blockDim.x ? ncg : blockDim.x;  // threads along the columns
  const int nrg = blockDim.x / cgt;                        // row groups
  const int rg = threadIdx.x / cgt;
  if (rg < nrg) {
    for (int cg = threadIdx.x % cgt; cg < ncg; cg += cgt) {
      float acc[V], v[V];
#pragma unroll
      for (int i = 0; i < V; ++i) { acc[i] = 0.f; v[i] = sv[cg * V + i]; }
      if (V == 4) {
        constexpr int U = 8;                               // independent 16-byte loads in flight
        for (int d0 = rg; d0 < D; d0 += nrg * U) {
          float4 s[U];
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int d = d0 + u * nrg;
            if (d < D) s[u] = __ldcs(reinterpret_cast<const float4*>(S + static_cast<long long>(d) * Dv + cg * 4));
          }
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int d = d0 + u * nrg;
            if (d < D) {
              const float f = sf[d], k = sk[d], q = sq[d];
              s[u].x = fmaf(f, s[u].x, k * v[0]); s[u].y = fmaf(f, s[u].y, k * v[1 % V]);
              s[u].z = fmaf(f, s[u].z, k * v[2 % V]); s[u].w = fmaf(f, s[u].w, k * v[3 % V]);
              acc[0] = fmaf(s[u].x, q, acc[0]); acc[1 % V] = fmaf(s[u].y, q, acc[1 % V]);
              acc[2 % V] = fmaf(s[u].z, q, acc[2 % V]); acc[3 % V] = fmaf(s[u].w, q, acc[3 % V]);
              __stcs(reinterpret_cast<float4*>(S + static_cast<long long>(d) * Dv + cg * 4), s[u]);
            }
          }
        }
      } else {
        for (int d = rg; d < D; d += nrg) {
          const float s = fmaf(sf[d], S[static_cast<long long>(d) * Dv + cg], sk[d] * v[0]);
          S[static_cast<long long>(d) * Dv + cg] = s;
          acc[0] = fmaf(s, sq[d], acc[0]);
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) part[rg * Dv + cg * V + i] = acc[i];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x; c < Dv; c += blockDim.x) {
    float t = 0.f;
    for (int r = 0; r < nrg; ++r) t += part[r * Dv + c];
    sv[c] = t;  // only this thread reads it again
    ss = fmaf(t, t, ss);
    if (!norm_w) a.o[ob + c] = t;
  }
  if (norm_w) {
    ss = block_sum(ss, red);
    const float k = 1.f / sqrtf(ss / Dv + eps);
    for (int c = threadIdx.x; c < Dv; c += blockDim.x) st1(y + ob + c, sv[c] * k * ld1(norm_w + c));
  }
}

constexpr int kMaxSmem = 227 * 1024;

}  // namespace b200

extern "C" {

// Token-by-token prefill. cu: [n_seq + 1]; slots: [n_seq] or null; o: [T, H, Dv] fp32.
int b200_scan_tokens(const void* x, long long ldx, const void* bias, const void* lower, const float* decay,
                     const int* cu, const int* slots, float* state, float* o, int n_seq, int H, int D, int Dv, int mode,
                     int fp32, cudaStream_t stream) {
  using namespace b200;
  if (n_seq <= 0) return 0;
  ScanArgs a{x, ldx, bias, lower, decay, cu, slots, state, o, H, D, Dv, mode};
  const int nw = D >= 64 ? 8 : 4;
  const size_t smem = (static_cast<size_t>(D) * 32 + 3 * kGrp * D + kGrp * nw * 32) * sizeof(float);
  if (smem > kMaxSmem) return -100;
  dim3 grid(n_seq, H, (Dv + 31) / 32);
  if (fp32) {
    B200_CHECK(cudaFuncSetAttribute(scan_tokens_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    scan_tokens_kernel<float><<<grid, nw * 32, smem, stream>>>(a);
  } else {
    B200_CHECK(cudaFuncSetAttribute(scan_tokens_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    (int)smem));
    scan_tokens_kernel<__nv_bfloat16><<<grid, nw * 32, smem, stream>>>(a);
  }
  B200_CHECK(cudaGetLastError());
  return 0;
}

// One token per sequence. norm_w [Dv] and y (model dtype) or null and o (fp32).
int b200_scan_step(const void* x, long long ldx, const void* bias, const void* lower, const float* decay,
                   const int* slots, float* state, float* o, const void* norm_w, void* y, float eps, int B, int H, int D,
                   int Dv, int mode, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (B <= 0) return 0;
  ScanArgs a{x, ldx, bias, lower, decay, nullptr, slots, state, o, H, D, Dv, mode};
  const bool v4 = Dv % 4 == 0;
  const int ncg = v4 ? Dv / 4 : Dv;
  const int block = 256;
  const int nrg = ncg < block ? block / ncg : 1;
  const size_t smem = (3 * static_cast<size_t>(D) + Dv + static_cast<size_t>(nrg) * Dv) * sizeof(float);
  if (smem > kMaxSmem) return -100;
  dim3 grid(B, H);
#define B200_SS(T_, V_)                                                                                             \
  {                                                                                                                 \
    B200_CHECK(cudaFuncSetAttribute(scan_step_kernel<T_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize,          \
                                    (int)smem));                                                                    \
    scan_step_kernel<T_, V_><<<grid, block, smem, stream>>>(a, (const T_*)norm_w, (T_*)y, eps);                     \
  }
  if (fp32) { if (v4) B200_SS(float, 4) else B200_SS(float, 1) }
  else { if (v4) B200_SS(__nv_bfloat16, 4) else B200_SS(__nv_bfloat16, 1) }
#undef B200_SS
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // extern "C"
