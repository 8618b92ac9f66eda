// Recurrences with one matrix state S [D, Dv] per head, fp32, and one decay per head and token:
//
//   gated delta rule   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          unit q and k
//   mLSTM              m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n likewise with k alone;
//                      o = S^T q / (max(|n . q|, e^-m') + 1e-6)
//
// Here: single decode steps with everything from the projections to the gated output in one kernel, and a token-by-token
// prefill for 32-bit models and head widths that the tensor-core kernels (matrix_state_chunk.cu) do not take.
#include "common/host_utils.h"
#include "common/io.cuh"
#include "common/scan_inputs.cuh"
#include "common/state_inputs.cuh"

namespace b200 {

constexpr int kStGrp = 8, kStMaxSmem = 227 * 1024;

struct StateOut {
  const int *cu, *slots;
  float *S, *n, *m;   // [slots, H, D, Dv], [slots, H, D], [slots, H]; n, m: mLSTM
  float* o;           // [T, H, Dv]
};

// One block per (sequence, head, 32 value columns). Lane = column, the warps split the rows; the state slice [D][32] stays in
// shared memory. Tokens come in groups whose inputs are prepared together.
template <class T>
__global__ void state_tokens_kernel(StateArgs a, StateOut out) {
  extern __shared__ float sm[];
  const int D = a.D, nw = blockDim.x >> 5, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* S = sm;                      // [D][32]
  float* n = S + D * 32;              // [D]
  float* sq = n + D;                  // [kStGrp][D]
  float* sk = sq + kStGrp * D;
  float* part = sk + kStGrp * D;      // [2][nw][32]
  float* op = part + 2 * nw * 32;     // [kStGrp][nw][32]
  float* np = op + kStGrp * nw * 32;  // [kStGrp][nw]
  float* gates = np + kStGrp * nw;    // [kStGrp][2]
  float* floor_ = gates + kStGrp * 2; // [kStGrp]
  const int seq = blockIdx.x, h = blockIdx.y, hk = h / (a.H / a.G), j = blockIdx.z * 32 + lane;
  const int t0 = out.cu[seq], t1 = out.cu[seq + 1];
  for (int i = threadIdx.x; i < D * 33; i += blockDim.x) sm[i] = 0.f;  // S and n
  float m = 0.f;
  const float qscale = 1.f / sqrtf(static_cast<float>(D));
  for (int tb = t0; tb < t1; tb += kStGrp) {
    const int cnt = min(kStGrp, t1 - tb);
    __syncthreads();
    for (int g = warp; g < cnt; g += nw) {  // a warp per token: q and k, made unit vectors for the delta rule
      const T* row = static_cast<const T*>(a.qkv) + (tb + g) * a.ldq + hk * D;
      float s0 = 0.f, s1 = 0.f;
      for (int d = lane; d < D; d += 32) {
        const float q = ld1(row + d), k = ld1(row + a.G * D + d);
        sq[g * D + d] = q;
        sk[g * D + d] = k;
        s0 = fmaf(q, q, s0);
        s1 = fmaf(k, k, s1);
      }
      const float kq = (a.delta ? 1.f / sqrtf(warp_sum(s0) + 1e-6f) : 1.f) * qscale;
      const float kk = a.delta ? 1.f / sqrtf(warp_sum(s1) + 1e-6f) : 1.f;
      for (int d = lane; d < D; d += 32) {
        sq[g * D + d] *= kq;
        sk[g * D + d] *= kk;
      }
      if (lane == 0) head_gates<T>(a, tb + g, h, gates[2 * g], gates[2 * g + 1]);
    }
    __syncthreads();
    for (int g = 0; g < cnt; ++g) {
      const float* q = sq + g * D;
      const float* k = sk + g * D;
      const float v = j < a.Dv ? ld1(static_cast<const T*>(a.qkv) + (tb + g) * a.ldq + 2 * a.G * D + h * a.Dv + j) : 0.f;
      float keep, u;
      if (a.delta) {
        keep = expf(gates[2 * g]);
        float acc = 0.f;
        for (int d = warp; d < D; d += nw) acc = fmaf(keep * S[d * 32 + lane], k[d], acc);
        float* p = part + (g & 1) * nw * 32;
        p[warp * 32 + lane] = acc;
        __syncthreads();
        acc = 0.f;
        for (int w = 0; w < nw; ++w) acc += p[w * 32 + lane];
        u = gates[2 * g + 1] * (v - acc);
      } else {
        const float next = fmaxf(gates[2 * g] + m, gates[2 * g + 1]), put = expf(gates[2 * g + 1] - next);
        keep = expf(gates[2 * g] + m - next);
        m = next;
        u = put * v;
        float acc = 0.f;
        for (int d = threadIdx.x; d < D; d += blockDim.x) {
          const float x = fmaf(keep, n[d], put * k[d]);
          n[d] = x;
          acc = fmaf(x, q[d], acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) np[g * nw + warp] = acc;
        if (threadIdx.x == 0) floor_[g] = expf(-m);
      }
      float o = 0.f;
      for (int d = warp; d < D; d += nw) {
        const float s = fmaf(keep, S[d * 32 + lane], k[d] * u);
        S[d * 32 + lane] = s;
        o = fmaf(s, q[d], o);
      }
      op[(g * nw + warp) * 32 + lane] = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < cnt * 32; i += blockDim.x) {
      const int g = i >> 5, c = blockIdx.z * 32 + (i & 31);
      float o = 0.f;
      for (int w = 0; w < nw; ++w) o += op[(g * nw + w) * 32 + (i & 31)];
      if (!a.delta) {
        float den = 0.f;
        for (int w = 0; w < nw; ++w) den += np[g * nw + w];
        o /= fmaxf(fabsf(den), floor_[g]) + 1e-6f;
      }
      if (c < a.Dv) out.o[(static_cast<long long>(tb + g) * a.H + h) * a.Dv + c] = o;
    }
  }
  __syncthreads();
  const int slot = out.slots ? out.slots[seq] : -1;
  if (slot < 0) return;
  const long long sh = static_cast<long long>(slot) * a.H + h;
  for (int i = threadIdx.x; i < D * 32; i += blockDim.x) {
    const int d = i >> 5, c = blockIdx.z * 32 + (i & 31);
    if (c < a.Dv) out.S[(sh * D + d) * a.Dv + c] = S[i];
  }
  if (!a.delta && blockIdx.z == 0) {
    for (int d = threadIdx.x; d < D; d += blockDim.x) out.n[sh * D + d] = n[d];
    if (threadIdx.x == 0) out.m[sh] = m;
  }
}

struct StepArgs {
  const void* x;           // [B][ldx]: q, k (G * D) | v (H * Dv) | gate (H * Dv) | ...; g0, g1 of StateArgs point into it
  const void* conv;        // delta rule: [2 G D + H Dv, taps]
  void* ring;              // [slots][taps][2 G D + H Dv], position p in row p % taps
  int taps;
  const int *pos, *slots;  // [B]; negative slots: padding rows
  float *S, *n, *m;
  const void* norm;        // delta rule: [Dv]; mLSTM: [H * Dv]
  void* y;                 // [B, H * Dv]
  float eps;
};

// One token's channel c behind the short convolution and SiLU, rounded to the model's dtype; `keep`: its input goes to the
// ring (the row that is written is none of those that are read, so heads may share channels).
template <class T>
__device__ __forceinline__ float conv_channel(const StepArgs& s, const T* x, int c, int C, int slot, int p, bool keep) {
  const T* w = static_cast<const T*>(s.conv) + static_cast<long long>(c) * s.taps + s.taps - 1;
  T* ring = static_cast<T*>(s.ring) + static_cast<long long>(slot) * s.taps * C + c;
  float acc = ld1(x + c) * ld1(w);
  if (s.taps <= 4) {  // the loads go out together
    float f[3], u[3];
#pragma unroll
    for (int j = 1; j < 4; ++j) {
      const bool in = j < s.taps && j <= p;
      f[j - 1] = in ? ld1(ring + static_cast<long long>((p - j) % s.taps) * C) : 0.f;
      u[j - 1] = in ? ld1(w - j) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 3; ++j) acc = fmaf(f[j], u[j], acc);
  } else {
    for (int j = 1; j < s.taps && j <= p; ++j)
      acc = fmaf(ld1(ring + static_cast<long long>((p - j) % s.taps) * C), ld1(w - j), acc);
  }
  if (keep) ring[static_cast<long long>(p % s.taps) * C] = x[c];
  return round_as(silu_as(acc, x), x);
}

// Decode step: one block per (sequence, head). Threads form row groups x column groups of V; with R > 0 a thread keeps its R
// rows of the state in registers between the read (S^T k, S^T q) and the update, with R 0 it reads them twice.
template <class T, int V, int R, int NT>
__global__ void __launch_bounds__(NT, 2) state_step_kernel(StateArgs a, StepArgs s) {
  extern __shared__ float sm[];
  __shared__ float red[3][NT / 32], red2[33];
  const int D = a.D, Dv = a.Dv, H = a.H, b = blockIdx.x, h = blockIdx.y, group = H / a.G, hk = h / group;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* sq = sm;            // [D]
  float* sk = sq + D;        // [D]
  float* sv = sk + D;        // [Dv]: v, then u
  float* part = sv + Dv;     // [2][row groups][Dv]
  const int slot = s.slots[b];
  T* y = static_cast<T*>(s.y) + (static_cast<long long>(b) * H + h) * Dv;
  if (slot < 0) {            // padding row of a fixed-size batch
    for (int c = tid; c < Dv; c += blockDim.x) st1(y + c, 0.f);
    return;
  }
  const T* x = static_cast<const T*>(s.x) + b * a.ldx;
  const int q0 = hk * D, k0 = (a.G + hk) * D, v0 = 2 * a.G * D + h * Dv, C = 2 * a.G * D + H * Dv;
  const long long sh = static_cast<long long>(slot) * H + h;
  const int ncg = Dv / V, cgt = ncg < NT ? ncg : NT, nrg = NT / cgt, rg = tid / cgt;
  float* S = s.S + sh * D * Dv;
  // the state is on its way while q, k and v are prepared
  float st[R > 0 ? R : 1][V];
  const int cg = tid % cgt;
  if constexpr (R > 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int d = rg + r * nrg;
#pragma unroll
      for (int e = 0; e < V; ++e) st[r][e] = 0.f;
      if (rg < nrg && d < D) {
        if constexpr (V == 4) {
          const float4 f = __ldcs(reinterpret_cast<const float4*>(S + static_cast<long long>(d) * Dv + cg * 4));
          st[r][0] = f.x; st[r][1] = f.y; st[r][2] = f.z; st[r][3] = f.w;
        } else {
          st[r][0] = S[static_cast<long long>(d) * Dv + cg];
        }
      }
    }
  }
  float log_decay, write;
  head_gates<T>(a, b, h, log_decay, write);
  float r0 = 0.f, r1 = 0.f, r2 = 0.f;  // q . q, k . k, k . q, or n . q in the first
  const int p = a.delta ? s.pos[b] : 0;
  const bool owner = h == hk * group;  // one of the heads that share q and k keeps their inputs
  // values by the last threads, queries and keys by the first: different warps where there are enough
  for (int c = NT - 1 - tid; c < Dv; c += NT) sv[c] = a.delta ? conv_channel(s, x, v0 + c, C, slot, p, true) : ld1(x + v0 + c);
  for (int d = tid; d < D; d += NT) {
    float q, k;
    if (a.delta) {
      q = conv_channel(s, x, q0 + d, C, slot, p, owner);
      k = conv_channel(s, x, k0 + d, C, slot, p, owner);
      r0 = fmaf(q, q, r0);
      r1 = fmaf(k, k, r1);
    } else {
      q = ld1(x + q0 + d);
      k = ld1(x + k0 + d);
      r0 = fmaf(s.n[sh * D + d], q, r0);
    }
    r2 = fmaf(k, q, r2);
    sq[d] = q;
    sk[d] = k;
  }
  r0 = warp_sum(r0);
  r1 = warp_sum(r1);
  r2 = warp_sum(r2);
  if (lane == 0) { red[0][warp] = r0; red[1][warp] = r1; red[2][warp] = r2; }
  const float m0 = a.delta ? 0.f : s.m[sh];
  __syncthreads();
  r0 = r1 = r2 = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) { r0 += red[0][w]; r1 += red[1][w]; r2 += red[2][w]; }
  // S' = keep S + wk k~ u^T with the raw vectors k~, q~;  o = fq (keep S^T q~ + wk (k~ . q~) u)
  float fq = 1.f / sqrtf(static_cast<float>(D)), wk = 1.f, keep, inv = 1.f, next = 0.f;
  if (a.delta) {
    fq /= sqrtf(r0 + 1e-6f);
    wk = 1.f / sqrtf(r1 + 1e-6f);
    keep = expf(log_decay);
  } else {
    next = fmaxf(log_decay + m0, write);
    keep = expf(log_decay + m0 - next);
    wk = expf(write - next);
    inv = 1.f / (fmaxf(fabsf(fq * fmaf(keep, r0, wk * r2)), expf(-next)) + 1e-6f);
  }
  // ---- S^T k~ and S^T q~
  if (rg < nrg) {
    auto put = [&](int col, const float (&ka)[V], const float (&qa)[V]) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        part[rg * Dv + col * V + e] = ka[e];
        part[(nrg + rg) * Dv + col * V + e] = qa[e];
      }
    };
    if constexpr (R > 0) {
      float ka[V], qa[V];
#pragma unroll
      for (int e = 0; e < V; ++e) ka[e] = qa[e] = 0.f;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int d = rg + r * nrg;
        if (d < D) {
          const float k = sk[d], q = sq[d];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            ka[e] = fmaf(st[r][e], k, ka[e]);
            qa[e] = fmaf(st[r][e], q, qa[e]);
          }
        }
      }
      put(cg, ka, qa);
    } else {
      for (int col = cg; col < ncg; col += cgt) {
        float ka[V], qa[V];
#pragma unroll
        for (int e = 0; e < V; ++e) ka[e] = qa[e] = 0.f;
        for (int d = rg; d < D; d += nrg) {
          float f[V];
          if constexpr (V == 4) {
            const float4 t = ld4(S + static_cast<long long>(d) * Dv + col * 4);
            f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
          } else {
            f[0] = S[static_cast<long long>(d) * Dv + col];
          }
#pragma unroll
          for (int e = 0; e < V; ++e) {
            ka[e] = fmaf(f[e], sk[d], ka[e]);
            qa[e] = fmaf(f[e], sq[d], qa[e]);
          }
        }
        put(col, ka, qa);
      }
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < Dv; c += blockDim.x) {
    float ks = 0.f, qs = 0.f;
    for (int r = 0; r < nrg; ++r) {
      ks += part[r * Dv + c];
      qs += part[(nrg + r) * Dv + c];
    }
    float u = sv[c];
    if (a.delta) u = write * (u - keep * wk * ks);
    sv[c] = u;
    const float o = fq * fmaf(keep, qs, wk * r2 * u) * inv;
    part[c] = o;  // only this thread reads the column again
    ss = fmaf(o, o, ss);
  }
  ss = block_sum(ss, red2);  // (its barriers also publish u)
  const float k = 1.f / sqrtf(ss / Dv + s.eps);
  const T* norm = static_cast<const T*>(s.norm) + (a.delta ? 0 : h * Dv);
  const T* gate = x + C + h * Dv;
  for (int c = tid; c < Dv; c += blockDim.x) st1(y + c, part[c] * k * ld1(norm + c) * out_gate(ld1(gate + c), a.delta, x));
  // ---- the new state
  if (rg < nrg) {
    if constexpr (R > 0) {
      float u[V];
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] = wk * sv[cg * V + e];
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int d = rg + r * nrg;
        if (d < D) {
          const float kd = sk[d];
#pragma unroll
          for (int e = 0; e < V; ++e) st[r][e] = fmaf(keep, st[r][e], kd * u[e]);
          if constexpr (V == 4)
            __stcs(reinterpret_cast<float4*>(S + static_cast<long long>(d) * Dv + cg * 4),
                   make_float4(st[r][0], st[r][1], st[r][2], st[r][3]));
          else
            S[static_cast<long long>(d) * Dv + cg] = st[r][0];
        }
      }
    } else {
      for (int col = cg; col < ncg; col += cgt)
        for (int d = rg; d < D; d += nrg)
#pragma unroll
          for (int e = 0; e < V; ++e) {
            float* at = S + static_cast<long long>(d) * Dv + col * V + e;
            *at = fmaf(keep, *at, sk[d] * wk * sv[col * V + e]);
          }
    }
  }
  if (!a.delta) {
    for (int d = tid; d < D; d += blockDim.x) s.n[sh * D + d] = fmaf(keep, s.n[sh * D + d], wk * sk[d]);
    if (tid == 0) s.m[sh] = next;
  }
}

template <class T, int V, int NT>
static int launch_state_step(const StateArgs& a, const StepArgs& s, int B, cudaStream_t stream) {
  const int ncg = a.Dv / V, cgt = ncg < NT ? ncg : NT, nrg = NT / cgt, rows = (a.D + nrg - 1) / nrg;
  const size_t smem = (2 * static_cast<size_t>(a.D) + a.Dv + 2 * static_cast<size_t>(nrg) * a.Dv) * sizeof(float);
  if (smem > kStMaxSmem) return -100;
  const dim3 grid(B, a.H);
#define B200_ST(R_)                                                                                                     \
  {                                                                                                                     \
    B200_CHECK(cudaFuncSetAttribute(state_step_kernel<T, V, R_, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    state_step_kernel<T, V, R_, NT><<<grid, NT, smem, stream>>>(a, s);                                                  \
  }
  if (ncg > NT || rows > 8) B200_ST(0)
  else if (rows > 4) B200_ST(8)
  else B200_ST(4)
#undef B200_ST
  B200_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace b200

extern "C" {

// Token-by-token prefill; o [T, H, Dv] fp32 (not normed). For the meaning of the operands see StateArgs and StateOut.
int b200_state_tokens(const void* qkv, long long ldq, const void* g0, const void* g1, long long ldx, const void* p0,
                      const void* p1, float cap, int delta, const int* cu, int n_seq, const int* slots, float* S, float* n,
                      float* m, float* o, int H, int G, int D, int Dv, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (n_seq <= 0) return 0;
  if (G < 1 || H % G || D < 1 || Dv < 1) return -100;
  const StateArgs a{qkv, ldq, g0, g1, ldx, p0, p1, cap, delta, H, G, D, Dv};
  const StateOut out{cu, slots, S, n, m, o};
  const int nw = D >= 64 ? 8 : 4;
  const size_t smem =
      (static_cast<size_t>(D) * (33 + 2 * kStGrp) + 2 * nw * 32 + kStGrp * (nw * 33 + 3)) * sizeof(float);
  if (smem > kStMaxSmem) return -101;
  const dim3 grid(n_seq, H, (Dv + 31) / 32);
#define B200_TK(T_)                                                                                                  \
  {                                                                                                                  \
    B200_CHECK(cudaFuncSetAttribute(state_tokens_kernel<T_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    state_tokens_kernel<T_><<<grid, nw * 32, smem, stream>>>(a, out);                                                \
  }
  if (fp32) B200_TK(float) else B200_TK(__nv_bfloat16)
#undef B200_TK
  B200_CHECK(cudaGetLastError());
  return 0;
}

// One token per sequence: x [B][ldx] as in StepArgs; g0, g1 follow from the row's layout. conv, ring, pos: delta rule.
int b200_state_step(const void* x, long long ldx, const void* p0, const void* p1, float cap, int delta, const void* conv,
                    void* ring, int taps, const int* pos, const int* slots, float* S, float* n, float* m, const void* norm,
                    void* y, float eps, int B, int H, int G, int D, int Dv, int fp32, cudaStream_t stream) {
  using namespace b200;
  if (B <= 0) return 0;
  if (G < 1 || H % G || D < 1 || Dv < 1 || (delta && taps < 1)) return -100;
  const long long at = 2LL * G * D + 2LL * H * Dv, size = fp32 ? 4 : 2;
  const char* g0 = static_cast<const char*>(x) + at * size;
  const StateArgs a{x, ldx, g0, g0 + H * size, ldx, p0, p1, cap, delta, H, G, D, Dv};
  const StepArgs s{x, conv, ring, taps, pos, slots, S, n, m, norm, y, eps};
  auto run = [&](auto tag) {
    using T = decltype(tag);
    if (Dv % 4) return launch_state_step<T, 1, 256>(a, s, B, stream);
    return D * Dv > 8192 ? launch_state_step<T, 4, 512>(a, s, B, stream) : launch_state_step<T, 4, 256>(a, s, B, stream);
  };
  return fp32 ? run(float{}) : run(__nv_bfloat16{});
}

}  // extern "C"
