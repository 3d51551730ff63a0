// polyrl_b200 — gated linear recurrences, token by token: decode steps, short spans, fp32 runs and any head size.
//
//   kSsd   (Mamba-2 / state-space duality)   S = exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x
//   kMlstm (xLSTM matrix memory)             m' = max(f + m, i),  S = e^(f+m-m') S + e^(i-m') k v^T,  n likewise with k alone,
//                                            y = S^T q / (max(|n . q|, e^(-m')) + 1e-6);  m starts at 0
//   kDelta (gated delta rule)                k' = k / |k|, q' = scale q / |q|,  S = keep S + k' u^T,  u = beta (v - keep S^T k'),  y = S^T q'
//                                            with keep = exp(-exp(A_log) softplus(a + bias)), beta = sigmoid(b).  With S the state before the
//                                            token, y = keep S^T q' + (k' . q') u, so one pass over S gives both products.
//   kDecay (constant decay)                  S = e^a S + k v^T,  y = S^T q, a per head; single tokens may come ahead of their silu
//   kGla   (decay per state row)             S = diag(keep) S + k v^T,  y = S^T q with keep = sigmoid(g + bias)^(1 / tau)
//
// mix_step_kernel (mix_delta_step_kernel for kDelta) serves spans of one token (decode): every state byte is read and written once, streaming.
// mix_scan_kernel: one CTA = one (span, head, 32 value columns): lane = value column, warp w owns the state rows w, w + 8, ... in registers
// from the first token to the last.
#include "mixers.cuh"

namespace prl {

constexpr int kScanWarps = 8;
constexpr int kScanVT = 32;

__device__ __forceinline__ float gla_keep(const ScanParams& p, int64_t t, int h, int n) {
  const int64_t c = static_cast<int64_t>(h) * p.N + n;
  return decay_f(logsigmoid_f(p.g0[t * p.ldg + c] + (p.b0 ? p.b0[c] : 0.f)) / p.cap);
}

template <class T, int MODE, int RN>
__global__ void __launch_bounds__(kScanWarps * 32)
mix_scan_kernel(ScanParams p) {
  constexpr int NMAX = RN * kScanWarps;
  __shared__ float s_q[2][NMAX], s_k[2][NMAX], s_n[NMAX], s_w[MODE == kGla ? 2 : 1][MODE == kGla ? NMAX : 1];
  constexpr int ND = MODE == kDelta ? 3 : 1;
  __shared__ float s_red[2][kScanWarps][33], s_dot[2][ND][kScanWarps], s_red2[MODE == kDelta ? 2 : 1][kScanWarps][33];
  const int vt = blockIdx.x, h = blockIdx.y, s = blockIdx.z;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int t0 = p.cu[s], t1 = p.cu[s + 1];
  if (t1 <= t0) return;
  const bool fresh = p.start[s] == 0;
  const int64_t slot = p.slot[s];
  const int col = vt * kScanVT + lane;
  const bool col_ok = col < p.V;
  float* Sg = p.S + (slot * p.H + h) * static_cast<int64_t>(p.N) * p.V + col;
  const T* q = static_cast<const T*>(p.q) + static_cast<int64_t>(h / p.rep) * p.N;
  const T* k = static_cast<const T*>(p.k) + static_cast<int64_t>(h / p.rep) * p.N;
  const T* v = static_cast<const T*>(p.v) + static_cast<int64_t>(h) * p.V;
  T* out = static_cast<T*>(p.out) + static_cast<int64_t>(h) * p.V;

  float S[RN];
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const int n = i * kScanWarps + w;
    S[i] = (!fresh && col_ok && n < p.N) ? Sg[static_cast<int64_t>(n) * p.V] : 0.f;
  }
  float m = 0.f;
  if constexpr (MODE == kMlstm) {
    const int64_t hb = slot * p.H + h;
    if (!fresh) m = p.mst[hb];
    for (int n = tid; n < NMAX; n += kScanWarps * 32) s_n[n] = (!fresh && n < p.N) ? p.nst[hb * p.N + n] : 0.f;
  }
  const float b0 = MODE != kGla && p.b0 ? p.b0[h] : 0.f, b1 = p.b1 ? p.b1[h] : 0.f;
  const float a_neg = MODE == kSsd || MODE == kDelta ? -expf(p.a_log[h]) : 0.f;
  const float fixed = MODE == kDecay ? decay_f(p.a_log[h]) : 1.f;
  const float skip = (MODE == kSsd && p.d_skip) ? p.d_skip[h] : 0.f;

  for (int t = t0; t < t1; ++t) {
    const int b = t & 1;
    if constexpr (MODE == kDelta) {
      float kk = 0.f, qq = 0.f, kq = 0.f;
      for (int n = tid; n < NMAX; n += kScanWarps * 32) {
        const float qn = n < p.N ? to_f<T>(q[static_cast<int64_t>(t) * p.ldq + n]) : 0.f;
        const float kn = n < p.N ? to_f<T>(k[static_cast<int64_t>(t) * p.ldk + n]) : 0.f;
        s_q[b][n] = qn;
        s_k[b][n] = kn;
        kk += kn * kn; qq += qn * qn; kq += kn * qn;
      }
      kk = warp_sum(kk); qq = warp_sum(qq); kq = warp_sum(kq);
      if (lane == 0) { s_dot[b][0][w] = kk; s_dot[b][1][w] = qq; s_dot[b][2][w] = kq; }
      const float vv = col_ok ? to_f<T>(v[static_cast<int64_t>(t) * p.ldv + col]) : 0.f;
      const float keep = decay_f(a_neg * softplus_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + b0));
      const float beta = sigmoid_f(p.g1[static_cast<int64_t>(t) * p.ldg + h] + b1);
      __syncthreads();
      float ak = 0.f, aq = 0.f;
#pragma unroll
      for (int i = 0; i < RN; ++i) {
        const int n = i * kScanWarps + w;
        ak += s_k[b][n] * S[i];
        aq += s_q[b][n] * S[i];
      }
      s_red[b][w][lane] = ak;
      s_red2[b][w][lane] = aq;
      __syncthreads();
      ak = aq = kk = qq = kq = 0.f;
#pragma unroll
      for (int i = 0; i < kScanWarps; ++i) {
        ak += s_red[b][i][lane]; aq += s_red2[b][i][lane];
        kk += s_dot[b][0][i]; qq += s_dot[b][1][i]; kq += s_dot[b][2][i];
      }
      const float rk = rsqrtf(kk + kUnitEps), rq = rsqrtf(qq + kUnitEps) * p.qscale;
      const float u = beta * (vv - keep * rk * ak), uk = u * rk;
#pragma unroll
      for (int i = 0; i < RN; ++i) S[i] = keep * S[i] + uk * s_k[b][i * kScanWarps + w];
      if (w == 0 && col_ok) out[static_cast<int64_t>(t) * p.ldo + col] = from_f<T>(rq * (keep * aq + uk * kq));
      continue;
    }
    for (int n = tid; n < NMAX; n += kScanWarps * 32) {
      s_q[b][n] = n < p.N ? to_f<T>(q[static_cast<int64_t>(t) * p.ldq + n]) * p.qscale : 0.f;
      s_k[b][n] = n < p.N ? to_f<T>(k[static_cast<int64_t>(t) * p.ldk + n]) : 0.f;
      if constexpr (MODE == kGla) s_w[b][n] = n < p.N ? gla_keep(p, t, h, n) : 1.f;
    }
    const float vv = col_ok ? to_f<T>(v[static_cast<int64_t>(t) * p.ldv + col]) : 0.f;
    float keep, add, floor_ = 0.f;
    if constexpr (MODE == kDecay || MODE == kGla) {
      keep = fixed;
      add = 1.f;
    } else if constexpr (MODE == kSsd) {
      add = softplus_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + b0);
      keep = expf(a_neg * add);
    } else {
      const float gi = softcap_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + b0, p.cap);
      const float gf = logsigmoid_f(softcap_f(p.g1[static_cast<int64_t>(t) * p.ldg + h] + b1, p.cap));
      const float m2 = fmaxf(gf + m, gi);
      keep = expf(gf + m - m2);
      add = expf(gi - m2);
      m = m2;
      floor_ = expf(-m2);
    }
    __syncthreads();
    const float av = add * vv;
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < RN; ++i) {
      const int n = i * kScanWarps + w;
      S[i] = (MODE == kGla ? s_w[b][n] : keep) * S[i] + av * s_k[b][n];
      acc += s_q[b][n] * S[i];
    }
    s_red[b][w][lane] = acc;
    if constexpr (MODE == kMlstm) {
      float d = 0.f;
      for (int n = tid; n < NMAX; n += kScanWarps * 32) {        // the same thread owns s_n[n] for every token
        const float nn = keep * s_n[n] + add * s_k[b][n];
        s_n[n] = nn;
        d += nn * s_q[b][n];
      }
      d = warp_sum(d);
      if (lane == 0) s_dot[b][0][w] = d;
    }
    __syncthreads();
    if (w == 0 && col_ok) {
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < kScanWarps; ++i) y += s_red[b][i][lane];
      if constexpr (MODE == kSsd) {
        y += skip * vv;
      } else if constexpr (MODE == kMlstm) {
        float d = 0.f;
#pragma unroll
        for (int i = 0; i < kScanWarps; ++i) d += s_dot[b][0][i];
        y /= fmaxf(fabsf(d), floor_) + 1e-6f;
      }
      out[static_cast<int64_t>(t) * p.ldo + col] = from_f<T>(y);
    }
  }
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const int n = i * kScanWarps + w;
    if (col_ok && n < p.N) Sg[static_cast<int64_t>(n) * p.V] = S[i];
  }
  if constexpr (MODE == kMlstm) {
    if (last_tile(p.counter + s * p.H + h, gridDim.x)) {
      const int64_t hb = slot * p.H + h;
      for (int n = tid; n < p.N; n += kScanWarps * 32) p.nst[hb * p.N + n] = s_n[n];
      if (tid == 0) p.mst[hb] = m;
    }
  }
}

// ---- one token per span: the state streams through registers, CPL neighbouring value columns per lane
template <int CPL>
__device__ __forceinline__ void ld_cols(const float* p, float (&v)[CPL]) {
  if constexpr (CPL == 4) { const float4 q = __ldcs(reinterpret_cast<const float4*>(p)); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
  else if constexpr (CPL == 2) { const float2 q = __ldcs(reinterpret_cast<const float2*>(p)); v[0] = q.x; v[1] = q.y; }
  else v[0] = __ldcs(p);
}
template <int CPL>
__device__ __forceinline__ void st_cols(float* p, const float (&v)[CPL]) {
  if constexpr (CPL == 4) __stcs(reinterpret_cast<float4*>(p), make_float4(v[0], v[1], v[2], v[3]));
  else if constexpr (CPL == 2) __stcs(reinterpret_cast<float2*>(p), make_float2(v[0], v[1]));
  else __stcs(p, v[0]);
}

template <class T, int MODE, int CPL>
__global__ void __launch_bounds__(kScanWarps * 32)
mix_step_kernel(ScanParams p) {
  constexpr int U = 8;                                   // state rows in flight per warp
  __shared__ float s_q[512], s_k[512], s_n[512], s_w[MODE == kGla ? 512 : 1];
  __shared__ float s_red[kScanWarps][32 * CPL + 1], s_dot[kScanWarps];
  const int vt = blockIdx.x, h = blockIdx.y, s = blockIdx.z;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int t = p.cu[s];
  if (p.cu[s + 1] <= t) return;
  const bool fresh = p.start[s] == 0;
  const int64_t slot = p.slot[s], hb = slot * p.H + h;
  const int col = vt * 32 * CPL + lane * CPL;
  const bool ok = col < p.V;                             // V is a multiple of CPL
  float* Sg = p.S + hb * static_cast<int64_t>(p.N) * p.V + col;
  float st[U][CPL];
  auto load = [&](int n0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int n = n0 + u * kScanWarps + w;
#pragma unroll
      for (int c = 0; c < CPL; ++c) st[u][c] = 0.f;
      if (!fresh && ok && n < p.N) ld_cols<CPL>(Sg + static_cast<int64_t>(n) * p.V, st[u]);
    }
  };
  load(0);
  const T* q = static_cast<const T*>(p.q) + static_cast<int64_t>(t) * p.ldq + static_cast<int64_t>(h / p.rep) * p.N;
  const T* k = static_cast<const T*>(p.k) + static_cast<int64_t>(t) * p.ldk + static_cast<int64_t>(h / p.rep) * p.N;
  const T* v = static_cast<const T*>(p.v) + static_cast<int64_t>(t) * p.ldv + static_cast<int64_t>(h) * p.V;
  float vv[CPL];
  auto act = [&](float x) { return MODE == kDecay && p.raw ? to_f<T>(from_f<T>(silu_f(x))) : x; };         // (rounded like an activated row)
#pragma unroll
  for (int c = 0; c < CPL; ++c) vv[c] = ok ? act(to_f<T>(v[col + c])) : 0.f;
  float keep, add, floor_ = 0.f, m2 = 0.f;
  const float b0 = MODE != kGla && p.b0 ? p.b0[h] : 0.f;
  if constexpr (MODE == kDecay || MODE == kGla) {
    keep = MODE == kDecay ? decay_f(p.a_log[h]) : 1.f;
    add = 1.f;
  } else if constexpr (MODE == kSsd) {
    add = softplus_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + b0);
    keep = expf(-expf(p.a_log[h]) * add);
  } else {
    const float m = fresh ? 0.f : p.mst[hb];
    const float gi = softcap_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + b0, p.cap);
    const float gf = logsigmoid_f(softcap_f(p.g1[static_cast<int64_t>(t) * p.ldg + h] + (p.b1 ? p.b1[h] : 0.f), p.cap));
    m2 = fmaxf(gf + m, gi);
    keep = expf(gf + m - m2);
    add = expf(gi - m2);
    floor_ = expf(-m2);
  }
  float dot = 0.f;
  for (int n = tid; n < p.N; n += kScanWarps * 32) {
    const float qn = act(to_f<T>(q[n])) * p.qscale, kn = act(to_f<T>(k[n]));
    s_q[n] = qn;
    s_k[n] = kn;
    if constexpr (MODE == kGla) s_w[n] = gla_keep(p, t, h, n);
    if constexpr (MODE == kMlstm) {
      const float nn = keep * (fresh ? 0.f : p.nst[hb * p.N + n]) + add * kn;
      s_n[n] = nn;
      dot += nn * qn;
    }
  }
  if constexpr (MODE == kMlstm) {
    dot = warp_sum(dot);
    if (lane == 0) s_dot[w] = dot;
  }
  __syncthreads();
  float acc[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) acc[c] = 0.f;
  for (int n0 = 0; n0 < p.N; n0 += U * kScanWarps) {
    if (n0) load(n0);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int n = n0 + u * kScanWarps + w;
      if (n < p.N) {
        const float ak = add * s_k[n], qn = s_q[n];
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          st[u][c] = (MODE == kGla ? s_w[n] : keep) * st[u][c] + ak * vv[c];
          acc[c] += qn * st[u][c];
        }
        if (ok) st_cols<CPL>(Sg + static_cast<int64_t>(n) * p.V, st[u]);
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) s_red[w][lane * CPL + c] = acc[c];
  __syncthreads();
  for (int c = tid; c < 32 * CPL; c += kScanWarps * 32) {
    const int gc = vt * 32 * CPL + c;
    if (gc < p.V) {
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < kScanWarps; ++i) y += s_red[i][c];
      if constexpr (MODE == kSsd) {
        if (p.d_skip) y += p.d_skip[h] * to_f<T>(v[gc]);
      } else if constexpr (MODE == kMlstm) {
        float d = 0.f;
#pragma unroll
        for (int i = 0; i < kScanWarps; ++i) d += s_dot[i];
        y /= fmaxf(fabsf(d), floor_) + 1e-6f;
      }
      static_cast<T*>(p.out)[static_cast<int64_t>(t) * p.ldo + static_cast<int64_t>(h) * p.V + gc] = from_f<T>(y);
    }
  }
  if constexpr (MODE == kMlstm) {
    if (last_tile(p.counter + s * p.H + h, gridDim.x)) {
      for (int n = tid; n < p.N; n += kScanWarps * 32) p.nst[hb * p.N + n] = s_n[n];
      if (tid == 0) p.mst[hb] = m2;
    }
  }
}

// ---- kDelta, one token per span: the state tile waits in registers for its two products, then is updated and written back
template <class T, int RN, int CPL>
__global__ void __launch_bounds__(kScanWarps * 32)
mix_delta_step_kernel(ScanParams p) {
  __shared__ float s_q[RN * kScanWarps], s_k[RN * kScanWarps], s_dot[3][kScanWarps];
  __shared__ alignas(16) float s_red[2][kScanWarps][32 * CPL];
  const int vt = blockIdx.x, h = blockIdx.y, s = blockIdx.z;
  const int w = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int t = p.cu[s];
  if (p.cu[s + 1] <= t) return;
  const bool fresh = p.start[s] == 0;
  const int64_t hb = p.slot[s] * p.H + h;
  const int col = vt * 32 * CPL + lane * CPL;
  const bool ok = col < p.V;                             // V is a multiple of CPL
  float* Sg = p.S + hb * static_cast<int64_t>(p.N) * p.V + col;
  float st[RN][CPL];
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const int n = i * kScanWarps + w;
#pragma unroll
    for (int c = 0; c < CPL; ++c) st[i][c] = 0.f;
    if (!fresh && ok && n < p.N) ld_cols<CPL>(Sg + static_cast<int64_t>(n) * p.V, st[i]);
  }
  const T* q = static_cast<const T*>(p.q) + static_cast<int64_t>(t) * p.ldq + static_cast<int64_t>(h / p.rep) * p.N;
  const T* k = static_cast<const T*>(p.k) + static_cast<int64_t>(t) * p.ldk + static_cast<int64_t>(h / p.rep) * p.N;
  const T* v = static_cast<const T*>(p.v) + static_cast<int64_t>(t) * p.ldv + static_cast<int64_t>(h) * p.V;
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int n = tid; n < RN * kScanWarps; n += kScanWarps * 32) {
    const float qn = n < p.N ? to_f<T>(q[n]) : 0.f, kn = n < p.N ? to_f<T>(k[n]) : 0.f;
    s_q[n] = qn;
    s_k[n] = kn;
    kk += kn * kn; qq += qn * qn; kq += kn * qn;
  }
  kk = warp_sum(kk); qq = warp_sum(qq); kq = warp_sum(kq);
  if (lane == 0) { s_dot[0][w] = kk; s_dot[1][w] = qq; s_dot[2][w] = kq; }
  float vv[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) vv[c] = ok ? to_f<T>(v[col + c]) : 0.f;
  const float keep = decay_f(-expf(p.a_log[h]) * softplus_f(p.g0[static_cast<int64_t>(t) * p.ldg + h] + (p.b0 ? p.b0[h] : 0.f)));
  const float beta = sigmoid_f(p.g1[static_cast<int64_t>(t) * p.ldg + h] + (p.b1 ? p.b1[h] : 0.f));
  __syncthreads();
  float ak[CPL], aq[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) ak[c] = aq[c] = 0.f;
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const float kn = s_k[i * kScanWarps + w], qn = s_q[i * kScanWarps + w];
#pragma unroll
    for (int c = 0; c < CPL; ++c) { ak[c] += kn * st[i][c]; aq[c] += qn * st[i][c]; }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) { s_red[0][w][lane * CPL + c] = ak[c]; s_red[1][w][lane * CPL + c] = aq[c]; ak[c] = aq[c] = 0.f; }
  __syncthreads();
  kk = qq = kq = 0.f;
#pragma unroll
  for (int i = 0; i < kScanWarps; ++i) {
#pragma unroll
    for (int c = 0; c < CPL; ++c) { ak[c] += s_red[0][i][lane * CPL + c]; aq[c] += s_red[1][i][lane * CPL + c]; }
    kk += s_dot[0][i]; qq += s_dot[1][i]; kq += s_dot[2][i];
  }
  const float rk = rsqrtf(kk + kUnitEps), rq = rsqrtf(qq + kUnitEps) * p.qscale;
  float uk[CPL];
#pragma unroll
  for (int c = 0; c < CPL; ++c) uk[c] = beta * (vv[c] - keep * rk * ak[c]) * rk;
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const int n = i * kScanWarps + w;
    const float kn = s_k[n];
#pragma unroll
    for (int c = 0; c < CPL; ++c) st[i][c] = keep * st[i][c] + uk[c] * kn;
    if (ok && n < p.N) st_cols<CPL>(Sg + static_cast<int64_t>(n) * p.V, st[i]);
  }
  if (w == 0 && ok) {
    T* o = static_cast<T*>(p.out) + static_cast<int64_t>(t) * p.ldo + static_cast<int64_t>(h) * p.V + col;
#pragma unroll
    for (int c = 0; c < CPL; ++c) o[c] = from_f<T>(rq * (keep * aq[c] + uk[c] * kq));
  }
}
template <class T, int RN>
static int launch_delta_step(const ScanParams& p, cudaStream_t st) {
  constexpr int C4 = RN <= 16 ? 4 : 1, C2 = RN <= 32 ? 2 : 1;          // (at most 64 state entries per thread)
  const bool al = (reinterpret_cast<uintptr_t>(p.S) & 15) == 0;
  const int threads = kScanWarps * 32;
  if (al && C4 == 4 && p.V % 4 == 0 && p.V > 64) mix_delta_step_kernel<T, RN, C4><<<dim3((p.V + 127) / 128, p.H, p.spans), threads, 0, st>>>(p);
  else if (al && C2 == 2 && p.V % 2 == 0 && p.V > 32) mix_delta_step_kernel<T, RN, C2><<<dim3((p.V + 63) / 64, p.H, p.spans), threads, 0, st>>>(p);
  else mix_delta_step_kernel<T, RN, 1><<<dim3((p.V + 31) / 32, p.H, p.spans), threads, 0, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <class T>
static int launch_delta_step(const ScanParams& p, cudaStream_t st) {
  if (p.N <= 64) return launch_delta_step<T, 8>(p, st);
  if (p.N <= 128) return launch_delta_step<T, 16>(p, st);
  if (p.N <= 256) return launch_delta_step<T, 32>(p, st);
  if (p.N <= 512) return launch_delta_step<T, 64>(p, st);
  return -203;
}

template <class T, int MODE>
static int launch_step(const ScanParams& p, cudaStream_t st) {
  const bool al = (reinterpret_cast<uintptr_t>(p.S) & 15) == 0;
  const int threads = kScanWarps * 32;
  if (p.N > 512) return -203;
  if (al && p.V % 4 == 0 && p.V > 64) mix_step_kernel<T, MODE, 4><<<dim3((p.V + 127) / 128, p.H, p.spans), threads, 0, st>>>(p);
  else if (al && p.V % 2 == 0 && p.V > 32) mix_step_kernel<T, MODE, 2><<<dim3((p.V + 63) / 64, p.H, p.spans), threads, 0, st>>>(p);
  else mix_step_kernel<T, MODE, 1><<<dim3((p.V + 31) / 32, p.H, p.spans), threads, 0, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

template <class T, int MODE>
static int launch_scan(const ScanParams& p, cudaStream_t st) {
  dim3 grid((p.V + kScanVT - 1) / kScanVT, p.H, p.spans);
  const int threads = kScanWarps * 32;
  if (p.N <= 32) mix_scan_kernel<T, MODE, 4><<<grid, threads, 0, st>>>(p);
  else if (p.N <= 64) mix_scan_kernel<T, MODE, 8><<<grid, threads, 0, st>>>(p);
  else if (p.N <= 128) mix_scan_kernel<T, MODE, 16><<<grid, threads, 0, st>>>(p);
  else if (p.N <= 256) mix_scan_kernel<T, MODE, 32><<<grid, threads, 0, st>>>(p);
  else if (p.N <= 512) mix_scan_kernel<T, MODE, 64><<<grid, threads, 0, st>>>(p);
  else return -201;
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

template <class T>
static int run_scan(const ScanParams& p, int mode, int single, cudaStream_t st) {
  if (mode == kDelta) return single ? launch_delta_step<T>(p, st) : launch_scan<T, kDelta>(p, st);
  if (mode == kDecay) return single ? launch_step<T, kDecay>(p, st) : launch_scan<T, kDecay>(p, st);
  if (mode == kGla) return single ? launch_step<T, kGla>(p, st) : launch_scan<T, kGla>(p, st);
  if (single) return mode == kSsd ? launch_step<T, kSsd>(p, st) : launch_step<T, kMlstm>(p, st);
  return mode == kSsd ? launch_scan<T, kSsd>(p, st) : launch_scan<T, kMlstm>(p, st);
}
// dtype: 0 = bf16, 1 = fp32 activations; mode: kSsd / kMlstm / kDelta / kDecay / kGla; single: every span is one token
extern "C" int prl_mix_scan(const ScanParams* p, int mode, int dtype, int single, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || (p->raw && !(mode == kDecay && single))) return -202;
  return dtype == 0 ? run_scan<__nv_bfloat16>(*p, mode, single, st) : run_scan<float>(*p, mode, single, st);
}
