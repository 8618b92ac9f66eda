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
#include "common/ptx.cuh"
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

// What a decode step of one (sequence, head) prepares ahead of the state: q~ and k~ (raw, in shared memory), v, and the factors
//   S' = keep S + wk k~ u^T,   o = fq (keep S^T q~ + wk (k~ . q~) u) inv,   u = write (v - keep wk S^T k~) or (mLSTM) v
struct StepFactors {
  float fq, wk, keep, inv, write, kq, next;
};

template <class T, int NT>
__device__ __forceinline__ StepFactors step_inputs(const StateArgs& a, const StepArgs& s, const T* x, int b, int h, int slot,
                                                   float* sq, float* sk, float* sv, float (&red)[3][NT / 32]) {
  const int D = a.D, Dv = a.Dv, H = a.H, group = H / a.G, hk = h / group, tid = threadIdx.x, warp = tid >> 5;
  const int q0 = hk * D, k0 = (a.G + hk) * D, v0 = 2 * a.G * D + h * Dv, C = 2 * a.G * D + H * Dv;
  const long long sh = static_cast<long long>(slot) * H + h;
  StepFactors f;
  float log_decay;
  head_gates<T>(a, b, h, log_decay, f.write);
  float r0 = 0.f, r1 = 0.f, r2 = 0.f;  // q . q (mLSTM: n . q), k . k, k . q
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
  const float m0 = a.delta ? 0.f : s.m[sh];
  r0 = warp_sum(r0);
  r1 = warp_sum(r1);
  r2 = warp_sum(r2);
  if ((tid & 31) == 0) { red[0][warp] = r0; red[1][warp] = r1; red[2][warp] = r2; }
  __syncthreads();
  r0 = r1 = r2 = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) { r0 += red[0][w]; r1 += red[1][w]; r2 += red[2][w]; }
  f.fq = 1.f / sqrtf(static_cast<float>(D));
  f.inv = 1.f;
  f.next = 0.f;
  f.kq = r2;
  if (a.delta) {
    f.fq /= sqrtf(r0 + 1e-6f);
    f.wk = 1.f / sqrtf(r1 + 1e-6f);
    f.keep = expf(log_decay);
  } else {
    f.next = fmaxf(log_decay + m0, f.write);
    f.keep = expf(log_decay + m0 - f.next);
    f.wk = expf(f.write - f.next);
    f.inv = 1.f / (fmaxf(fabsf(f.fq * fmaf(f.keep, r0, f.wk * r2)), expf(-f.next)) + 1e-6f);
  }
  return f;
}

// From the row groups' partial sums part [2][nrg][Dv] of S^T k~ and S^T q~: u (over v), and the head's normed and gated output.
// Ends behind a barrier.
template <class T, int NT>
__device__ __forceinline__ void step_outputs(const StateArgs& a, const StepArgs& s, const T* x, int b, int h, const StepFactors& f,
                                             int nrg, float* sv, float* part, float* red2) {
  const int Dv = a.Dv, C = 2 * a.G * a.D + a.H * Dv, tid = threadIdx.x;
  float ss = 0.f;
  for (int c = tid; c < Dv; c += NT) {
    float ks = 0.f, qs = 0.f;
    for (int r = 0; r < nrg; ++r) {
      ks += part[r * Dv + c];
      qs += part[(nrg + r) * Dv + c];
    }
    float u = sv[c];
    if (a.delta) u = f.write * (u - f.keep * f.wk * ks);
    sv[c] = u;
    const float o = f.fq * fmaf(f.keep, qs, f.wk * f.kq * u) * f.inv;
    part[c] = o;  // only this thread reads the column again
    ss = fmaf(o, o, ss);
  }
  ss = block_sum(ss, red2);  // (its barriers also publish u)
  const float k = 1.f / sqrtf(ss / Dv + s.eps);
  const T* norm = static_cast<const T*>(s.norm) + (a.delta ? 0 : h * Dv);
  const T* gate = x + C + h * Dv;
  T* y = static_cast<T*>(s.y) + (static_cast<long long>(b) * a.H + h) * Dv;
  for (int c = tid; c < Dv; c += NT) st1(y + c, part[c] * k * ld1(norm + c) * out_gate(ld1(gate + c), a.delta, x));
}

template <class T, int NT>
__device__ __forceinline__ void step_normaliser(const StateArgs& a, const StepArgs& s, long long sh, const StepFactors& f,
                                                const float* sk) {
  if (a.delta) return;
  for (int d = threadIdx.x; d < a.D; d += NT) s.n[sh * a.D + d] = fmaf(f.keep, s.n[sh * a.D + d], f.wk * sk[d]);
  if (threadIdx.x == 0) s.m[sh] = f.next;
}

// Decode step, one block per (sequence, head), for states that fit shared memory: one bulk copy brings the state in while q, k
// and v are prepared, it is read and updated there, and one bulk copy takes it back. Dv in steps of 4. Threads form row groups
// x groups of four columns.
template <class T, int NT>
__global__ void __launch_bounds__(NT) state_step_kernel(StateArgs a, StepArgs s, int* status) {
  extern __shared__ __align__(128) float sm[];
  __shared__ float red[3][NT / 32], red2[33];
  __shared__ uint64_t bar;
  __shared__ int abort_word;
  const int D = a.D, Dv = a.Dv, b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  float* S = sm;             // [D][Dv]
  float* sq = S + D * Dv;    // [D]
  float* sk = sq + D;        // [D]
  float* sv = sk + D;        // [Dv]: v, then u
  float* part = sv + Dv;     // [2][row groups][Dv]
  const int slot = s.slots[b];
  if (slot < 0) {            // padding row of a fixed-size batch
    T* y = static_cast<T*>(s.y) + (static_cast<long long>(b) * a.H + h) * Dv;
    for (int c = tid; c < Dv; c += NT) st1(y + c, 0.f);
    return;
  }
  const long long sh = static_cast<long long>(slot) * a.H + h;
  float* home = s.S + sh * D * Dv;
  const uint32_t bytes = static_cast<uint32_t>(D) * Dv * 4;
  if (tid == 0) {
    abort_word = 0;
    mbar_init(&bar, 1);
    fence_mbar_init();
    mbar_arrive_expect_tx(&bar, bytes);
    bulk_load(S, home, bytes, &bar);
  }
  const T* x = static_cast<const T*>(s.x) + b * a.ldx;
  const StepFactors f = step_inputs<T, NT>(a, s, x, b, h, slot, sq, sk, sv, red);
  if (!mbar_wait(&bar, 0, &abort_word)) {
    abort_word = 1;
    if (tid == 0) {
      atomicCAS(status, 0, kErrMbarTimeoutProducer);
      const unsigned long long t0 = globaltimer_ns();  // the copy in flight lands before the CTA retires
      while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
    }
    __syncthreads();
    return;
  }
  const int ncg = Dv / 4, cgt = ncg < NT ? ncg : NT, nrg = NT / cgt, rg = tid / cgt;
  if (rg < nrg) {
    for (int col = tid % cgt; col < ncg; col += cgt) {
      float4 ka = make_float4(0.f, 0.f, 0.f, 0.f), qa = ka;
#pragma unroll 4
      for (int d = rg; d < D; d += nrg) {
        const float4 t = *reinterpret_cast<const float4*>(S + d * Dv + col * 4);
        const float k = sk[d], q = sq[d];
        ka.x = fmaf(t.x, k, ka.x); ka.y = fmaf(t.y, k, ka.y); ka.z = fmaf(t.z, k, ka.z); ka.w = fmaf(t.w, k, ka.w);
        qa.x = fmaf(t.x, q, qa.x); qa.y = fmaf(t.y, q, qa.y); qa.z = fmaf(t.z, q, qa.z); qa.w = fmaf(t.w, q, qa.w);
      }
      *reinterpret_cast<float4*>(part + rg * Dv + col * 4) = ka;
      *reinterpret_cast<float4*>(part + (nrg + rg) * Dv + col * 4) = qa;
    }
  }
  __syncthreads();
  step_outputs<T, NT>(a, s, x, b, h, f, nrg, sv, part, red2);
  if (rg < nrg) {
    for (int col = tid % cgt; col < ncg; col += cgt) {
      const float4 v = *reinterpret_cast<const float4*>(sv + col * 4);
      const float4 u = make_float4(f.wk * v.x, f.wk * v.y, f.wk * v.z, f.wk * v.w);
#pragma unroll 4
      for (int d = rg; d < D; d += nrg) {
        float4* at = reinterpret_cast<float4*>(S + d * Dv + col * 4);
        const float k = sk[d];
        const float4 t = *at;
        *at = make_float4(fmaf(f.keep, t.x, k * u.x), fmaf(f.keep, t.y, k * u.y), fmaf(f.keep, t.z, k * u.z),
                          fmaf(f.keep, t.w, k * u.w));
      }
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 0) {
    bulk_store(home, S, bytes);
    tma_store_commit();
  }
  step_normaliser<T, NT>(a, s, sh, f, sk);
  if (tid == 0) tma_store_wait_read<0>();
}

// The same for any width: the state is read where it lies, twice.
template <class T, int NT>
__global__ void __launch_bounds__(NT) state_step_wide_kernel(StateArgs a, StepArgs s) {
  extern __shared__ float sm[];
  __shared__ float red[3][NT / 32], red2[33];
  const int D = a.D, Dv = a.Dv, b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  float* sq = sm;            // [D]
  float* sk = sq + D;        // [D]
  float* sv = sk + D;        // [Dv]: v, then u
  float* part = sv + Dv;     // [2][row groups][Dv]
  const int slot = s.slots[b];
  if (slot < 0) {
    T* y = static_cast<T*>(s.y) + (static_cast<long long>(b) * a.H + h) * Dv;
    for (int c = tid; c < Dv; c += NT) st1(y + c, 0.f);
    return;
  }
  const long long sh = static_cast<long long>(slot) * a.H + h;
  float* S = s.S + sh * D * Dv;
  const T* x = static_cast<const T*>(s.x) + b * a.ldx;
  const StepFactors f = step_inputs<T, NT>(a, s, x, b, h, slot, sq, sk, sv, red);
  const int cgt = Dv < NT ? Dv : NT, nrg = NT / cgt, rg = tid / cgt;
  if (rg < nrg) {
    for (int c = tid % cgt; c < Dv; c += cgt) {
      float ka = 0.f, qa = 0.f;
#pragma unroll 4
      for (int d = rg; d < D; d += nrg) {
        const float t = S[static_cast<long long>(d) * Dv + c];
        ka = fmaf(t, sk[d], ka);
        qa = fmaf(t, sq[d], qa);
      }
      part[rg * Dv + c] = ka;
      part[(nrg + rg) * Dv + c] = qa;
    }
  }
  __syncthreads();
  step_outputs<T, NT>(a, s, x, b, h, f, nrg, sv, part, red2);
  if (rg < nrg) {
    for (int c = tid % cgt; c < Dv; c += cgt) {
      const float u = f.wk * sv[c];
#pragma unroll 4
      for (int d = rg; d < D; d += nrg) {
        float* at = S + static_cast<long long>(d) * Dv + c;
        *at = fmaf(f.keep, *at, sk[d] * u);
      }
    }
  }
  step_normaliser<T, NT>(a, s, sh, f, sk);
}

template <class T>
static int launch_state_step(const StateArgs& a, const StepArgs& s, int B, cudaStream_t stream) {
  constexpr int NT = 256;
  const dim3 grid(B, a.H);
  const bool v4 = a.Dv % 4 == 0;
  const int ncg = v4 ? a.Dv / 4 : a.Dv, nrg = NT / (ncg < NT ? ncg : NT);
  const size_t vecs = (2 * static_cast<size_t>(a.D) + a.Dv + 2 * static_cast<size_t>(nrg) * a.Dv) * sizeof(float);
  const size_t whole = static_cast<size_t>(a.D) * a.Dv * sizeof(float) + vecs;
  // (shared memory is carved up in floats: 16-byte accesses behind q and k want D in steps of 2 as well)
  if (v4 && a.D % 2 == 0 && whole <= 200 * 1024 && !(reinterpret_cast<uintptr_t>(s.S) & 15)) {
    int* status = device_status_word();
    if (!status) return -3;
    B200_CHECK(cudaFuncSetAttribute(state_step_kernel<T, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)whole));
    state_step_kernel<T, NT><<<grid, NT, whole, stream>>>(a, s, status);
    B200_CHECK(cudaGetLastError());
    return 0;
  }
  const int wide_nrg = NT / (a.Dv < NT ? a.Dv : NT);
  const size_t smem = (2 * static_cast<size_t>(a.D) + a.Dv + 2 * static_cast<size_t>(wide_nrg) * a.Dv) * sizeof(float);
  if (smem > kStMaxSmem) return -100;
  B200_CHECK(cudaFuncSetAttribute(state_step_wide_kernel<T, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  state_step_wide_kernel<T, NT><<<grid, NT, smem, stream>>>(a, s);
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
  return fp32 ? launch_state_step<float>(a, s, B, stream) : launch_state_step<__nv_bfloat16>(a, s, B, stream);
}

}  // extern "C"
