// polyrl_b200 — selective scan (Mamba): a state vector per channel, input-dependent step sizes, input and output maps shared by all channels.
//
//   d = softplus(dt + bias),  S[c, n] = exp(d_c A[c, n]) S[c, n] + d_c x_c B_n,  y_c = sum_n S[c, n] C_n + D_c x_c,  out = y silu(z)
//
// The recurrence is element-wise in (c, n), so it has no matrix form: a prompt's cost is one exponential per token, channel and state entry.
// LPC neighbouring lanes share a channel, SN state entries each, in registers from the first token to the last.  Tokens are taken TT at a
// time: what depends on a token and a channel only (step size, d x, D x, the gate) is computed once while the next tile's loads are in flight,
// B and C of a tile lie in shared memory as fp32, outputs leave through shared memory in whole rows.
// mix_selective_step_kernel serves spans of one token: the state streams through registers once.
#include <type_traits>

#include "mixers.cuh"

namespace prl {

constexpr int kSelThreads = 128;

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

// two fp32 values in one register pair: Blackwell's packed arithmetic
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
template <class T>
__device__ __forceinline__ f32x2 sel_decay2(f32x2 x) {
  const float2 v = unpack2(x);
  return pack2(sel_decay<T>(v.x), sel_decay<T>(v.y));
}
// W neighbouring channels, raw
template <class T, int W>
__device__ __forceinline__ void ld_raw(const T* p, bool ok, float (&v)[W]) {
  if constexpr (W == 2 && sizeof(T) == 2) {
    const float2 a = unpack_bf16(ok ? *reinterpret_cast<const uint32_t*>(p) : 0u);
    v[0] = a.x; v[1] = a.y;
  } else if constexpr (W == 2) {
    const float2 a = ok ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
    v[0] = a.x; v[1] = a.y;
  } else {
    v[0] = ok ? to_f<T>(*p) : 0.f;
  }
}
template <class T, int W>
struct SelRaw {                                              // a thread's share of a tile, as loaded: it waits in registers while the tile before it runs
  using Word = std::conditional_t<sizeof(T) == 2 && W == 2, uint32_t, std::conditional_t<W == 2, float2, T>>;
};

// W: channels per load (2 where rows allow it)
template <class T, int LPC, int SN, int TT, int W>
__global__ void __launch_bounds__(kSelThreads) mix_selective_kernel(SelectiveParams p) {
  constexpr int CB = kSelThreads / LPC, NP = LPC * SN, U = CB / W;       // channels of a CTA, padded state entries, loads per row
  constexpr int TG = SN <= 8 ? 4 : 2;
  constexpr int ROWS = kSelThreads / U, PX = (TT + ROWS - 1) / ROWS, PB = (TT * NP + kSelThreads - 1) / kSelThreads;
  constexpr float kScale = sizeof(T) == 2 ? 1.4426950408889634f : 1.f;
  using Word = typename SelRaw<T, W>::Word;
  __shared__ alignas(16) float sB[TT][NP], sC[TT][NP];
  __shared__ alignas(16) float2 sd[TT][CB], sg[TT][CB];       // (d, d x), (gate, D x)
  __shared__ alignas(16) float sy[TT][CB];
  const int s = blockIdx.y, c0 = blockIdx.x * CB, tid = threadIdx.x;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int ch = tid / LPC, part = tid % LPC, c = c0 + ch;
  const bool on = c < p.C;
  float* Sg = p.S + (p.slot[s] * p.C + c) * static_cast<int64_t>(p.N);
  f32x2 S[SN / 2], A[SN / 2];
#pragma unroll
  for (int i = 0; i < SN; i += 2) {
    float v[2], a[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = part * SN + i + e;
      v[e] = on && !fresh && n < p.N ? Sg[n] : 0.f;
      a[e] = on && n < p.N ? p.a_neg[static_cast<int64_t>(c) * p.N + n] * kScale : 0.f;
    }
    S[i / 2] = pack2(v[0], v[1]);
    A[i / 2] = pack2(a[0], a[1]);
  }
  // the tile's loads: channels lc, lc + 1 of rows lr, lr + ROWS, ...
  const int lk = tid % U * W, lc = c0 + lk, lr = tid / U;
  const bool lon = lc < p.C;                                  // (C is even where W = 2)
  float bias[W], skip[W];
#pragma unroll
  for (int e = 0; e < W; ++e) { bias[e] = lon ? p.dt_bias[lc + e] : 0.f; skip[e] = lon ? p.d_skip[lc + e] : 0.f; }
  Word rx[PX], rz[PX];
  float rd[PX][W], rb[PB], rc[PB];
  auto fetch = [&](int at) {
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int r = lr + i * ROWS, t = at + r;
      const bool ok = lon && r < TT && t < len;
      const int64_t row = t0 + (ok ? t : 0);
      rx[i] = ok ? *reinterpret_cast<const Word*>(static_cast<const T*>(p.x) + row * p.ldx + lc) : Word{};
      rz[i] = ok ? *reinterpret_cast<const Word*>(static_cast<const T*>(p.z) + row * p.ldz + lc) : Word{};
      ld_raw<float, W>(p.dt + row * p.ldd + (ok ? lc : 0), ok, rd[i]);
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
      const int r = lr + i * ROWS;
      if (r >= TT) break;
      float x[W], z[W];
      ld_raw<T, W>(reinterpret_cast<const T*>(&rx[i]), true, x);
      ld_raw<T, W>(reinterpret_cast<const T*>(&rz[i]), true, z);
#pragma unroll
      for (int e = 0; e < W; ++e) {
        const float d = at + r < len ? sel_softplus<T>(rd[i][e] + bias[e]) : 0.f;
        sd[r][lk + e] = make_float2(d, d * x[e]);
        sg[r][lk + e] = make_float2(silu_t<T>(z[e]), skip[e] * x[e]);
      }
    }
#pragma unroll
    for (int i = 0; i < PB; ++i) {
      const int e = tid + i * kSelThreads;
      if (e < TT * NP) { (&sB[0][0])[e] = rb[i]; (&sC[0][0])[e] = rc[i]; }
    }
    __syncthreads();
    if (at + TT < len) fetch(at + TT);
    // TG tokens at a time: what does not wait for the state first.  Tokens behind the span's end have d = 0 and change nothing
    const int nt = min(TT, (len - at + TG - 1) / TG * TG);
#pragma unroll 1
    for (int t = 0; t < nt; t += TG) {
      f32x2 e[TG][SN / 2], f[TG][SN / 2];
#pragma unroll
      for (int k = 0; k < TG; ++k) {
        const float2 dd = sd[t + k][ch];
        const f32x2 d = pack2(dd.x, dd.x), dx = pack2(dd.y, dd.y);
#pragma unroll
        for (int i = 0; i < SN; i += 4) {
          const ulonglong2 b = *reinterpret_cast<const ulonglong2*>(&sB[t + k][part * SN + i]);
          e[k][i / 2] = sel_decay2<T>(mul2(A[i / 2], d));
          e[k][i / 2 + 1] = sel_decay2<T>(mul2(A[i / 2 + 1], d));
          f[k][i / 2] = mul2(dx, b.x);
          f[k][i / 2 + 1] = mul2(dx, b.y);
        }
      }
      float o[TG];
#pragma unroll
      for (int k = 0; k < TG; ++k) {
        f32x2 y0 = 0, y1 = 0;
#pragma unroll
        for (int i = 0; i < SN; i += 4) {
          const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(&sC[t + k][part * SN + i]);
          S[i / 2] = fma2(e[k][i / 2], S[i / 2], f[k][i / 2]);
          S[i / 2 + 1] = fma2(e[k][i / 2 + 1], S[i / 2 + 1], f[k][i / 2 + 1]);
          y0 = fma2(S[i / 2], w.x, y0);
          y1 = fma2(S[i / 2 + 1], w.y, y1);
        }
        const float2 a = unpack2(y0), c2 = unpack2(y1);
        o[k] = (a.x + a.y) + (c2.x + c2.y);
      }
#pragma unroll
      for (int m = LPC / 2; m; m >>= 1)
#pragma unroll
        for (int k = 0; k < TG; ++k) o[k] += __shfl_xor_sync(0xffffffffu, o[k], m);
      if (part == 0)
#pragma unroll
        for (int k = 0; k < TG; ++k) sy[t + k][ch] = o[k];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int r = lr + i * ROWS, t = at + r;
      if (!lon || r >= TT || t >= len) continue;
      float o[W];
#pragma unroll
      for (int e = 0; e < W; ++e) {
        const float2 g = sg[r][lk + e];
        o[e] = (sy[r][lk + e] + g.y) * g.x;
      }
      T* dst = static_cast<T*>(p.out) + (t0 + t) * p.ldo + lc;
      if constexpr (W == 2 && sizeof(T) == 2) {
        *reinterpret_cast<uint32_t*>(dst) = pack_bf16(o[0], o[1]);
      } else {
#pragma unroll
        for (int e = 0; e < W; ++e) dst[e] = from_f<T>(o[e]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < SN; i += 2) {
    const float2 v = unpack2(S[i / 2]);
    const int n = part * SN + i;
    if (on && n < p.N) Sg[n] = v.x;
    if (on && n + 1 < p.N) Sg[n + 1] = v.y;
  }
}

// one token per span: LPC lanes per channel, VEC neighbouring state entries per lane and step, CH channels per lane group with their loads in flight
// together (a span's B and C are read once for all of them)
template <class T, int LPC, int VEC, int CH>
__global__ void __launch_bounds__(256, CH == 1 ? 5 : 3) mix_selective_step_kernel(SelectiveParams p) {
  constexpr int CB = 256 / LPC;
  constexpr float kScale = sizeof(T) == 2 ? 1.4426950408889634f : 1.f;
  const int s = blockIdx.y, part = threadIdx.x % LPC, c0 = blockIdx.x * CB * CH + threadIdx.x / LPC;
  const int64_t t = p.cu[s], slot = p.slot[s];
  const bool live = p.cu[s + 1] > t, fresh = p.start[s] == 0;
  if (!live) return;
  float* Sg = p.S + slot * p.C * p.N;
  float x[CH], z[CH], d[CH], y[CH], skip[CH];
#pragma unroll
  for (int i = 0; i < CH; ++i) {
    const int64_t c = min(c0 + i * CB, p.C - 1);
    x[i] = to_f<T>(static_cast<const T*>(p.x)[t * p.ldx + c]);
    z[i] = to_f<T>(static_cast<const T*>(p.z)[t * p.ldz + c]);
    d[i] = p.dt[t * p.ldd + c] + p.dt_bias[c];
    skip[i] = p.d_skip[c];
    y[i] = 0.f;
  }
  for (int n = part * VEC; n < p.N; n += LPC * VEC) {          // N is a multiple of VEC
    float v[CH][VEC], a[CH][VEC], b[VEC], w[VEC];
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const int64_t at = static_cast<int64_t>(min(c0 + i * CB, p.C - 1)) * p.N + n;
      if constexpr (VEC % 4 == 0) {
#pragma unroll
        for (int e = 0; e < VEC; e += 4) {
          const float4 q = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcs(reinterpret_cast<const float4*>(Sg + at + e));
          const float4 m = *reinterpret_cast<const float4*>(p.a_neg + at + e);
          v[i][e] = q.x; v[i][e + 1] = q.y; v[i][e + 2] = q.z; v[i][e + 3] = q.w;
          a[i][e] = m.x; a[i][e + 1] = m.y; a[i][e + 2] = m.z; a[i][e + 3] = m.w;
        }
      } else {
        v[i][0] = fresh ? 0.f : Sg[at];
        a[i][0] = p.a_neg[at];
      }
    }
    if constexpr (VEC == 8) {
      ld_vec<T, 8>(static_cast<const T*>(p.b) + t * p.ldb + n, b);
      ld_vec<T, 8>(static_cast<const T*>(p.c) + t * p.ldc + n, w);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        b[e] = to_f<T>(static_cast<const T*>(p.b)[t * p.ldb + n + e]);
        w[e] = to_f<T>(static_cast<const T*>(p.c)[t * p.ldc + n + e]);
      }
    }
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const float dd = sel_softplus<T>(d[i]), dx = dd * x[i];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        v[i][e] = sel_decay<T>(dd * (a[i][e] * kScale)) * v[i][e] + dx * b[e];
        y[i] += v[i][e] * w[e];
      }
      const int c = c0 + i * CB;
      if (c < p.C) {
        float* dst = Sg + static_cast<int64_t>(c) * p.N + n;
        if constexpr (VEC % 4 == 0) {
#pragma unroll
          for (int e = 0; e < VEC; e += 4) __stcs(reinterpret_cast<float4*>(dst + e), make_float4(v[i][e], v[i][e + 1], v[i][e + 2], v[i][e + 3]));
        } else {
          *dst = v[i][0];
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < CH; ++i) {
#pragma unroll
    for (int o = LPC / 2; o; o >>= 1) y[i] += __shfl_xor_sync(0xffffffffu, y[i], o);
    const int c = c0 + i * CB;
    if (c < p.C && part == 0) static_cast<T*>(p.out)[t * p.ldo + c] = from_f<T>((y[i] + skip[i] * x[i]) * silu_t<T>(z[i]));
  }
}

template <class T, int LPC, int SN, int TT>
static int run_sel(const SelectiveParams& p, cudaStream_t st) {
  constexpr int CB = kSelThreads / LPC;
  auto al = [](const void* q, int64_t ld, int bytes) { return (reinterpret_cast<uintptr_t>(q) & (bytes - 1)) == 0 && ld % 2 == 0; };
  constexpr int E = 2 * sizeof(T);
  const bool two = CB % 2 == 0 && p.C % 2 == 0 && al(p.x, p.ldx, E) && al(p.z, p.ldz, E) && al(p.out, p.ldo, E) && al(p.dt, p.ldd, 8);
  const dim3 grid((p.C + CB - 1) / CB, p.spans);
  if (two) mix_selective_kernel<T, LPC, SN, TT, 2><<<grid, kSelThreads, 0, st>>>(p);
  else mix_selective_kernel<T, LPC, SN, TT, 1><<<grid, kSelThreads, 0, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <class T>
static int pick_sel(const SelectiveParams& p, cudaStream_t st) {
  if (p.N <= 4) return run_sel<T, 1, 4, 16>(p, st);
  if (p.N <= 8) return run_sel<T, 1, 8, 16>(p, st);
  if (p.N <= 16) return run_sel<T, 2, 8, 32>(p, st);
  if (p.N <= 24) return run_sel<T, 2, 12, 32>(p, st);
  if (p.N <= 32) return run_sel<T, 4, 8, 32>(p, st);
  if (p.N <= 64) return run_sel<T, 8, 8, 16>(p, st);
  if (p.N <= 128) return run_sel<T, 16, 8, 16>(p, st);
  return run_sel<T, 32, 16, 8>(p, st);
}
template <class T>
static int step_sel(const SelectiveParams& p, cudaStream_t st) {
  const bool vec = p.N % 4 == 0 && al16(p.S) && al16(p.a_neg);
  const bool many = p.spans >= 16;                            // few spans: more CTAs
#define MIX_SEL_STEP(LPC, VEC, CH) \
  mix_selective_step_kernel<T, LPC, VEC, CH><<<dim3((p.C + 256 / LPC * CH - 1) / (256 / LPC * CH), p.spans), 256, 0, st>>>(p)
  const bool wide = vec && p.N % 8 == 0 && al16(p.b) && al16(p.c) && p.ldb % 8 == 0 && p.ldc % 8 == 0;
  if (wide && many) MIX_SEL_STEP(2, 8, 2);
  else if (wide) MIX_SEL_STEP(2, 8, 1);
  else if (vec && many) MIX_SEL_STEP(4, 4, 2);
  else if (vec) MIX_SEL_STEP(4, 4, 1);
  else if (many) MIX_SEL_STEP(8, 1, 2);
  else MIX_SEL_STEP(8, 1, 1);
#undef MIX_SEL_STEP
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
