// polyrl_b200 — selective scan (Mamba): a state vector per channel, input-dependent step sizes, input and output maps shared by all channels.
//
//   d = softplus(dt + bias),  S[c, n] = exp(d_c A[c, n]) S[c, n] + d_c x_c B_n,  y_c = sum_n S[c, n] C_n + D_c x_c,  out = y silu(z)
//
// The recurrence is element-wise in (c, n), so it has no matrix form: a prompt's cost is one exponential per token, channel and state entry.
// LPC neighbouring lanes share a channel, SN state entries each, in registers from the first token to the last.  Tokens are taken TT at a
// time: what depends on a token and a channel only (step size, d x, D x, the gate) is computed once while the next tile's loads are in flight,
// B and C of a tile lie in shared memory as fp32, outputs leave through shared memory in whole rows.
// mix_selective_step_kernel serves spans of one token: the state streams through registers once.
#include "mixers.cuh"

namespace prl {

constexpr int kSelThreads = 256;

// exp(d A): a slow decay to the last bit in fp32 runs, ex2.approx (relative error 2^-22) beside bf16 activations
template <class T>
__device__ __forceinline__ float sel_decay(float x) {
  if constexpr (sizeof(T) == 2) return fast_exp2(x);         // x is scaled by log2 e already
  else return decay_f(x);
}
template <class T>
__device__ __forceinline__ float sel_softplus(float z) {
  if constexpr (sizeof(T) == 2) return softplus_series(z);
  else return softplus_f(z);
}

template <class T, int LPC, int SN, int TT>
__global__ void __launch_bounds__(kSelThreads) mix_selective_kernel(SelectiveParams p) {
  constexpr int CB = kSelThreads / LPC, NP = LPC * SN;       // channels of a CTA, padded state entries
  constexpr int ROWS = kSelThreads / CB, PX = (TT + ROWS - 1) / ROWS, PB = (TT * NP + kSelThreads - 1) / kSelThreads;
  constexpr float kScale = sizeof(T) == 2 ? 1.4426950408889634f : 1.f;
  __shared__ alignas(16) float sB[TT][NP], sC[TT][NP];
  __shared__ float sd[TT][CB], sdx[TT][CB], sy[TT][CB], sg[TT][CB];
  const int s = blockIdx.y, c0 = blockIdx.x * CB, tid = threadIdx.x;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int ch = tid / LPC, part = tid % LPC, c = c0 + ch;
  const bool on = c < p.C;
  float* Sg = p.S + (p.slot[s] * p.C + c) * static_cast<int64_t>(p.N);
  float S[SN], A[SN];
#pragma unroll
  for (int i = 0; i < SN; ++i) {
    const int n = part * SN + i;
    S[i] = on && !fresh && n < p.N ? Sg[n] : 0.f;
    A[i] = on && n < p.N ? p.a_neg[static_cast<int64_t>(c) * p.N + n] * kScale : 0.f;
  }
  // the tile's loads: column tid % CB of rows tid / CB, + ROWS, ...
  const int lc = c0 + tid % CB, lr = tid / CB;
  const bool lon = lc < p.C;
  const float bias = lon ? p.dt_bias[lc] : 0.f, skip = lon ? p.d_skip[lc] : 0.f;
  float rx[PX], rd[PX], rz[PX], rb[PB], rc[PB];
  auto fetch = [&](int at) {
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int r = lr + i * ROWS, t = at + r;
      const bool ok = lon && r < TT && t < len;
      const int64_t row = t0 + (ok ? t : 0);
      rx[i] = ok ? to_f<T>(static_cast<const T*>(p.x)[row * p.ldx + lc]) : 0.f;
      rd[i] = ok ? p.dt[row * p.ldd + lc] : 0.f;
      rz[i] = ok ? to_f<T>(static_cast<const T*>(p.z)[row * p.ldz + lc]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < PB; ++i) {
      const int e = tid + i * kSelThreads, t = at + e / NP, n = e % NP;
      const bool ok = e < TT * NP && t < len && n < p.N;
      const int64_t row = t0 + (ok ? t : 0);
      rb[i] = ok ? to_f<T>(static_cast<const T*>(p.b)[row * p.ldb + n]) : 0.f;
      rc[i] = ok ? to_f<T>(static_cast<const T*>(p.c)[row * p.ldc + n]) : 0.f;
    }
  };
  fetch(0);
  for (int at = 0; at < len; at += TT) {
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int r = lr + i * ROWS, k = tid % CB;
      if (r >= TT) break;
      const float d = at + r < len ? sel_softplus<T>(rd[i] + bias) : 0.f;      // (d = 0 leaves the state as it is)
      sd[r][k] = d;
      sdx[r][k] = d * rx[i];
      sy[r][k] = skip * rx[i];
      sg[r][k] = silu_t<T>(rz[i]);
    }
#pragma unroll
    for (int i = 0; i < PB; ++i) {
      const int e = tid + i * kSelThreads;
      if (e < TT * NP) { (&sB[0][0])[e] = rb[i]; (&sC[0][0])[e] = rc[i]; }
    }
    __syncthreads();
    if (at + TT < len) fetch(at + TT);
    const int nt = min(TT, len - at);
#pragma unroll 4
    for (int t = 0; t < nt; ++t) {
      const float d = sd[t][ch], dx = sdx[t][ch];
      float bv[SN], cv[SN], y = 0.f;
      if constexpr (SN % 4 == 0) {
#pragma unroll
        for (int i = 0; i < SN; i += 4) {
          const float4 q = *reinterpret_cast<const float4*>(&sB[t][part * SN + i]), w = *reinterpret_cast<const float4*>(&sC[t][part * SN + i]);
          bv[i] = q.x; bv[i + 1] = q.y; bv[i + 2] = q.z; bv[i + 3] = q.w;
          cv[i] = w.x; cv[i + 1] = w.y; cv[i + 2] = w.z; cv[i + 3] = w.w;
        }
      } else {
#pragma unroll
        for (int i = 0; i < SN; ++i) { bv[i] = sB[t][part * SN + i]; cv[i] = sC[t][part * SN + i]; }
      }
#pragma unroll
      for (int i = 0; i < SN; ++i) {
        S[i] = sel_decay<T>(d * A[i]) * S[i] + dx * bv[i];
        y += S[i] * cv[i];
      }
#pragma unroll
      for (int o = LPC / 2; o; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (part == 0) sy[t][ch] += y;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int r = lr + i * ROWS, k = tid % CB, t = at + r;
      if (lon && r < TT && t < len) static_cast<T*>(p.out)[(t0 + t) * p.ldo + lc] = from_f<T>(sy[r][k] * sg[r][k]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < SN; ++i) {
    const int n = part * SN + i;
    if (on && n < p.N) Sg[n] = S[i];
  }
}

// one token per span: LPC lanes per channel, VEC neighbouring state entries per lane and step
template <class T, int LPC, int VEC>
__global__ void __launch_bounds__(kSelThreads) mix_selective_step_kernel(SelectiveParams p) {
  constexpr int CB = kSelThreads / LPC;
  constexpr float kScale = sizeof(T) == 2 ? 1.4426950408889634f : 1.f;
  const int s = blockIdx.y, part = threadIdx.x % LPC, c = blockIdx.x * CB + threadIdx.x / LPC;
  const int64_t t = p.cu[s];
  if (p.cu[s + 1] <= t) return;
  const bool on = c < p.C, fresh = p.start[s] == 0;
  const int64_t cc = on ? c : 0;
  float* Sg = p.S + (p.slot[s] * p.C + cc) * p.N;
  const float* A = p.a_neg + cc * p.N;
  const T *B = static_cast<const T*>(p.b) + t * p.ldb, *Cm = static_cast<const T*>(p.c) + t * p.ldc;
  const float x = to_f<T>(static_cast<const T*>(p.x)[t * p.ldx + cc]), z = to_f<T>(static_cast<const T*>(p.z)[t * p.ldz + cc]);
  const float d = sel_softplus<T>(p.dt[t * p.ldd + cc] + p.dt_bias[cc]);
  float y = 0.f;
  for (int n = part * VEC; n < p.N; n += LPC * VEC) {          // N is a multiple of VEC
    float v[VEC], a[VEC];
    if constexpr (VEC == 4) {
      const float4 q = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcs(reinterpret_cast<const float4*>(Sg + n)), w = *reinterpret_cast<const float4*>(A + n);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
      a[0] = w.x; a[1] = w.y; a[2] = w.z; a[3] = w.w;
    } else {
      v[0] = fresh ? 0.f : Sg[n];
      a[0] = A[n];
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v[i] = sel_decay<T>(d * (a[i] * kScale)) * v[i] + (d * x) * to_f<T>(B[n + i]);
      y += v[i] * to_f<T>(Cm[n + i]);
    }
    if (on) {
      if constexpr (VEC == 4) __stcs(reinterpret_cast<float4*>(Sg + n), make_float4(v[0], v[1], v[2], v[3]));
      else Sg[n] = v[0];
    }
  }
#pragma unroll
  for (int o = LPC / 2; o; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (on && part == 0) static_cast<T*>(p.out)[t * p.ldo + c] = from_f<T>((y + p.d_skip[c] * x) * silu_t<T>(z));
}

template <class T, int LPC, int SN, int TT>
static int run_sel(const SelectiveParams& p, cudaStream_t st) {
  constexpr int CB = kSelThreads / LPC;
  mix_selective_kernel<T, LPC, SN, TT><<<dim3((p.C + CB - 1) / CB, p.spans), kSelThreads, 0, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <class T>
static int pick_sel(const SelectiveParams& p, cudaStream_t st) {
  if (p.N <= 4) return run_sel<T, 4, 1, 32>(p, st);
  if (p.N <= 8) return run_sel<T, 4, 2, 32>(p, st);
  if (p.N <= 16) return run_sel<T, 4, 4, 32>(p, st);
  if (p.N <= 32) return run_sel<T, 4, 8, 16>(p, st);
  if (p.N <= 64) return run_sel<T, 8, 8, 16>(p, st);
  if (p.N <= 128) return run_sel<T, 16, 8, 16>(p, st);
  return run_sel<T, 32, 16, 8>(p, st);
}
template <class T>
static int step_sel(const SelectiveParams& p, cudaStream_t st) {
  const bool vec = p.N % 4 == 0 && (reinterpret_cast<uintptr_t>(p.S) & 15) == 0 && (reinterpret_cast<uintptr_t>(p.a_neg) & 15) == 0;
  if (vec) mix_selective_step_kernel<T, 4, 4><<<dim3((p.C + 63) / 64, p.spans), kSelThreads, 0, st>>>(p);
  else mix_selective_step_kernel<T, 8, 1><<<dim3((p.C + 31) / 32, p.spans), kSelThreads, 0, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

// dtype: 0 = bf16, 1 = fp32 activations; single: every span is one token
extern "C" int prl_mix_selective(const SelectiveParams* p, int dtype, int single, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->N < 1 || p->N > 512 || p->C < 1) return -300;
  if (single) return dtype == 0 ? step_sel<__nv_bfloat16>(*p, st) : step_sel<float>(*p, st);
  return dtype == 0 ? pick_sel<__nv_bfloat16>(*p, st) : pick_sel<float>(*p, st);
}
