// polyrl_b200 — row-wise kernels of the mixer stacks: embedding, output-norm + residual add, gated group norm, causal
// convolution with carried taps, latent-attention row preparation, GELU.  The residual stream is fp32.
#include "mixers.cuh"

namespace prl {

// ---- x = embed[id] (fp32), h = the same in T (h may be null when T is fp32 and x is used directly), or T(rms(x) * w) when w is given
template <class T, int VEC>
__global__ void __launch_bounds__(128) mix_embed_kernel(const int64_t* __restrict__ ids, const T* __restrict__ emb, const float* __restrict__ w,
                                                        float* __restrict__ x, T* __restrict__ h, int W, float eps) {
  __shared__ float red[4];
  const int64_t row = blockIdx.x;
  const T* src = emb + ids[row] * W;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += 128 * VEC) {
    float v[VEC];
    ld_vec<T, VEC>(src + c, v);
    st_vec<float, VEC>(x + row * W + c, v);
    if (h && !w) st_vec<T, VEC>(h + row * W + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
  }
  if (!w) return;
  const float r = rsqrtf(block_sum<4>(ss, red) / W + eps);
  for (int c = threadIdx.x * VEC; c < W; c += 128 * VEC) {
    float v[VEC], g[VEC];
    ld_vec<T, VEC>(src + c, v);
    ld_vec<float, VEC>(w + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] *= r * g[i];
    st_vec<T, VEC>(h + row * W + c, v);
  }
}

// ---- x += rms(y) * w;  h = T(x), or T(rms(x) * w_next) when w_next is given (the model's final norm)
template <class T, int VEC>
__global__ void __launch_bounds__(256) mix_norm_add_kernel(const T* __restrict__ y, int64_t ldy, float* __restrict__ x, const float* __restrict__ w,
                                                           const float* __restrict__ w_next, T* __restrict__ h, int W, float eps) {
  __shared__ float red[8];
  const int64_t row = blockIdx.x;
  const T* yr = y + row * ldy;
  float* xr = x + row * W;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
    float v[VEC];
    ld_vec<T, VEC>(yr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += v[i] * v[i];
  }
  const float r = rsqrtf(block_sum<8>(ss, red) / W + eps);
  float s2 = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
    float v[VEC], g[VEC], xx[VEC];
    ld_vec<T, VEC>(yr + c, v);
    ld_vec<float, VEC>(w + c, g);
    ld_vec<float, VEC>(xr + c, xx);
#pragma unroll
    for (int i = 0; i < VEC; ++i) { xx[i] += v[i] * r * g[i]; s2 += xx[i] * xx[i]; }
    st_vec<float, VEC>(xr + c, xx);
    if (h && !w_next) st_vec<T, VEC>(h + row * W + c, xx);
  }
  if (!w_next) return;
  const float r2 = rsqrtf(block_sum<8>(s2, red) / W + eps);
  for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
    float g[VEC], xx[VEC];
    ld_vec<float, VEC>(xr + c, xx);
    ld_vec<float, VEC>(w_next + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) xx[i] *= r2 * g[i];
    st_vec<T, VEC>(h + row * W + c, xx);
  }
}

// ---- h = T(rms(x) * w) of fp32 rows; center: of x minus its mean
template <class T, int VEC>
__global__ void __launch_bounds__(256) mix_rms_kernel(const float* __restrict__ x, const float* __restrict__ w, T* __restrict__ h, int W, float eps,
                                                      int center) {
  __shared__ float red[8];
  const int64_t row = blockIdx.x;
  const float* xr = x + row * W;
  float ss = 0.f, mean = 0.f;
  if (center) {
    float s = 0.f;
    for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
      float v[VEC];
      ld_vec<float, VEC>(xr + c, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) s += v[i];
    }
    mean = block_sum<8>(s, red) / W;
  }
  for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
    float v[VEC];
    ld_vec<float, VEC>(xr + c, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += (v[i] - mean) * (v[i] - mean);
  }
  const float r = rsqrtf(block_sum<8>(ss, red) / W + eps);
  for (int c = threadIdx.x * VEC; c < W; c += 256 * VEC) {
    float v[VEC], g[VEC];
    ld_vec<float, VEC>(xr + c, v);
    ld_vec<float, VEC>(w + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = (v[i] - mean) * (r * g[i]);
    st_vec<T, VEC>(h + row * W + c, v);
  }
}

// ---- group norm of mixer outputs with a gate: kSiluFirst  rms(y silu(z)) w,   else  rms(y) w sigmoid(z)  or  rms(y) w silu(z)
// WPG warps share one (row, group); 8 / WPG groups per CTA
enum : int { kSigmoidLast = 0, kSiluFirst = 1, kSiluLast = 2 };
template <class T, int VEC, int GATE, int WPG>
__global__ void __launch_bounds__(256) mix_gated_norm_kernel(const T* __restrict__ y, int64_t ldy, const T* __restrict__ z, int64_t ldz,
                                                             const float* __restrict__ w, T* __restrict__ out, int64_t ldo, int64_t items, int groups,
                                                             int gs, float eps) {
  constexpr bool GATE_FIRST = GATE == kSiluFirst;
  __shared__ float red[8];
  const int64_t item = static_cast<int64_t>(blockIdx.x) * (8 / WPG) + (threadIdx.x >> 5) / WPG;
  if (WPG == 1 && item >= items) return;                // (WPG == 8: one item per CTA, the grid is exact)
  const int64_t row = item / groups;
  const int c0 = static_cast<int>(item % groups) * gs;
  const int t = threadIdx.x % (32 * WPG);
  const T* yr = y + row * ldy + c0;
  const T* zr = z + row * ldz + c0;
  T* orow = out + row * ldo + c0;
  float ss = 0.f;
  if constexpr (VEC == 8) {
    constexpr int HOLD = 4;                              // groups of up to 32 * WPG * 8 * HOLD elements stay in registers
    if (gs <= 32 * WPG * VEC * HOLD) {
      float u[HOLD][VEC];
#pragma unroll
      for (int k = 0; k < HOLD; ++k) {
        const int c = (k * 32 * WPG + t) * VEC;
        if (c < gs) {
          float g[VEC];
          ld_vec<T, VEC>(yr + c, u[k]);
          ld_vec<T, VEC>(zr + c, g);
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            const float f = GATE == kSigmoidLast ? sigmoid_t<T>(g[i]) : silu_t<T>(g[i]);
            if (!GATE_FIRST) ss += u[k][i] * u[k][i];
            u[k][i] *= f;
            if (GATE_FIRST) ss += u[k][i] * u[k][i];
          }
        }
      }
      const float r = rsqrtf(block_sum<WPG>(ss, red) / gs + eps);
#pragma unroll
      for (int k = 0; k < HOLD; ++k) {
        const int c = (k * 32 * WPG + t) * VEC;
        if (c < gs) {
          float ww[VEC];
          ld_vec<float, VEC>(w + c0 + c, ww);
#pragma unroll
          for (int i = 0; i < VEC; ++i) u[k][i] *= r * ww[i];
          st_vec<T, VEC>(orow + c, u[k]);
        }
      }
      return;
    }
  }
  for (int c = t * VEC; c < gs; c += 32 * WPG * VEC) {
    float v[VEC], g[VEC];
    ld_vec<T, VEC>(yr + c, v);
    if constexpr (GATE_FIRST) ld_vec<T, VEC>(zr + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float u = GATE_FIRST ? v[i] * silu_f(g[i]) : v[i];
      ss += u * u;
    }
  }
  const float r = rsqrtf(block_sum<WPG>(ss, red) / gs + eps);
  for (int c = t * VEC; c < gs; c += 32 * WPG * VEC) {
    float v[VEC], g[VEC], ww[VEC];
    ld_vec<T, VEC>(yr + c, v);
    ld_vec<T, VEC>(zr + c, g);
    ld_vec<float, VEC>(w + c0 + c, ww);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = v[i] * (GATE == kSigmoidLast ? sigmoid_f(g[i]) : silu_f(g[i])) * r * ww[i];
    st_vec<T, VEC>(orow + c, v);
  }
}

// the same for groups of at most 128 elements: 16 lanes per group, two groups in flight
template <class T, int GATE>
__global__ void __launch_bounds__(256) mix_gated_norm_narrow_kernel(const T* __restrict__ y, int64_t ldy, const T* __restrict__ z, int64_t ldz,
                                                                    const float* __restrict__ w, T* __restrict__ out, int64_t ldo, int64_t items, int groups,
                                                                    int gs, float eps) {
  const int c = (threadIdx.x & 15) * 8;
  const int64_t first = static_cast<int64_t>(blockIdx.x) * 32 + (threadIdx.x >> 4);
  float u[2][8], g[2][8], ss[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int64_t item = first + k * 16;
    ss[k] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) u[k][i] = g[k][i] = 0.f;
    if (item < items && c < gs) {
      const int64_t row = item / groups, at = item % groups * gs + c;
      ld_vec<T, 8>(y + row * ldy + at, u[k]);
      ld_vec<T, 8>(z + row * ldz + at, g[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float f = GATE == kSigmoidLast ? sigmoid_t<T>(g[k][i]) : silu_t<T>(g[k][i]);
      if (GATE != kSiluFirst) ss[k] += u[k][i] * u[k][i];
      u[k][i] *= f;
      if (GATE == kSiluFirst) ss[k] += u[k][i] * u[k][i];
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss[k] += __shfl_xor_sync(0xffffffffu, ss[k], o);
    const int64_t item = first + k * 16;
    if (item < items && c < gs) {
      const int64_t row = item / groups, at = item % groups * gs + c;
      const float r = rsqrtf(ss[k] / gs + eps);
      float ww[8];
      ld_vec<float, 8>(w + at, ww);
#pragma unroll
      for (int i = 0; i < 8; ++i) u[k][i] *= r * ww[i];
      st_vec<T, 8>(out + row * ldo + at, u[k]);
    }
  }
}

template <int VEC>
__device__ __forceinline__ void ld_bias(const float* bias, int c, float (&v)[VEC]) {
  if (bias) {
    ld_vec<float, VEC>(bias + c, v);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = 0.f;
  }
}
// ---- causal convolution per channel + silu (bias may be null); w [taps, ch] (row taps - 1 = current token), state [slots, taps - 1, ch]
template <class T, int VEC, int TT>
__global__ void __launch_bounds__(128) mix_conv_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w, const float* __restrict__ bias,
                                                       const T* __restrict__ state, const int32_t* __restrict__ cu, const int32_t* __restrict__ start,
                                                       const int64_t* __restrict__ slot, const int32_t* __restrict__ seq_of, T* __restrict__ out,
                                                       int64_t ldo, int ch, int taps, int total) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (c >= ch) return;
  const int tb = blockIdx.y * TT, te = min(total, tb + TT);
  for (int t = tb; t < te; ++t) {
    const int s = seq_of[t];
    const int t0 = cu[s];
    const bool fresh = start[s] == 0;
    float acc[VEC];
    ld_bias<VEC>(bias, c, acc);
    for (int j = 0; j < taps; ++j) {
      const int u = t - (taps - 1) + j;
      float v[VEC], g[VEC];
      if (u >= t0) {
        ld_vec<T, VEC>(x + static_cast<int64_t>(u) * ldx + c, v);
      } else {
        if (fresh) continue;
        ld_vec<T, VEC>(state + (slot[s] * (taps - 1) + (u - t0 + taps - 1)) * ch + c, v);
      }
      ld_vec<float, VEC>(w + static_cast<int64_t>(j) * ch + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] += g[i] * v[i];
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] = silu_f(acc[i]);
    st_vec<T, VEC>(out + static_cast<int64_t>(t) * ldo + c, acc);
  }
}
// the same for a fixed small tap count: 8 channels per thread, TT tokens with the window and the taps in registers
template <class T, int TAPS, int TT>
__global__ void __launch_bounds__(128) mix_conv_window_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w, const float* __restrict__ bias,
                                                              const T* __restrict__ state, const int32_t* __restrict__ cu, const int32_t* __restrict__ start,
                                                              const int64_t* __restrict__ slot, const int32_t* __restrict__ seq_of, T* __restrict__ out,
                                                              int64_t ldo, int ch, int total) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= ch) return;
  const int tb = blockIdx.y * TT, te = min(total, tb + TT);
  float wt[TAPS][8], bs[8], win[TAPS][8];               // win[j]: input of token t - (TAPS - 1) + j
#pragma unroll
  for (int j = 0; j < TAPS; ++j) ld_vec<float, 8>(w + static_cast<int64_t>(j) * ch + c, wt[j]);
  ld_bias<8>(bias, c, bs);
  int cur = -1;
#pragma unroll 4
  for (int t = tb; t < te; ++t) {
    const int s = seq_of[t];
    if (s != cur) {                                      // (re)fill the window at a span's start or at the tile's first token
      cur = s;
      const int t0 = cu[s];
      const bool fresh = start[s] == 0;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int u = t - (TAPS - 1) + j;
        if (u >= t0) {
          ld_vec<T, 8>(x + static_cast<int64_t>(u) * ldx + c, win[j]);
        } else if (!fresh) {
          ld_vec<T, 8>(state + (slot[s] * (TAPS - 1) + (u - t0 + TAPS - 1)) * ch + c, win[j]);
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) win[j][i] = 0.f;
        }
      }
    }
    ld_vec<T, 8>(x + static_cast<int64_t>(t) * ldx + c, win[TAPS - 1]);
    float acc[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = bs[i];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] += wt[j][i] * win[j][i];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = silu_t<T>(acc[i]);
    st_vec<T, 8>(out + static_cast<int64_t>(t) * ldo + c, acc);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
  }
}
// the last taps - 1 inputs of every span become its slot's state (row j of the new state is input len - (taps - 1) + j)
template <class T>
__global__ void mix_conv_state_kernel(const T* __restrict__ x, int64_t ldx, T* __restrict__ state, const int32_t* __restrict__ cu,
                                      const int32_t* __restrict__ start, const int64_t* __restrict__ slot, int ch, int taps) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
  if (c >= ch) return;
  const int t0 = cu[s], len = cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = start[s] == 0;
  T* st = state + slot[s] * static_cast<int64_t>(taps - 1) * ch + c;
  for (int j = 0; j < taps - 1; ++j) {                  // reads row j + len > j: in place in increasing order
    const int u = len - (taps - 1) + j;
    T v = from_f<T>(0.f);
    if (u >= 0) v = x[static_cast<int64_t>(t0 + u) * ldx + c];
    else if (!fresh) v = st[static_cast<int64_t>(j + len) * ch];
    st[static_cast<int64_t>(j) * ch] = v;
  }
}
// one token per span: convolution and state shift in one pass
template <class T, int VEC>
__global__ void __launch_bounds__(128) mix_conv_step_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w, const float* __restrict__ bias,
                                                            T* __restrict__ state, const int32_t* __restrict__ start, const int64_t* __restrict__ slot,
                                                            T* __restrict__ out, int64_t ldo, int ch, int taps) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, s = blockIdx.y;
  if (c >= ch) return;
  const bool fresh = start[s] == 0;
  T* st = state + slot[s] * static_cast<int64_t>(taps - 1) * ch + c;
  float acc[VEC], g[VEC], cur[VEC];
  ld_bias<VEC>(bias, c, acc);
  ld_vec<T, VEC>(x + static_cast<int64_t>(s) * ldx + c, cur);
  for (int j = 0; j < taps - 1; ++j) {
    float v[VEC];
    if (fresh) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    } else {
      ld_vec<T, VEC>(st + static_cast<int64_t>(j) * ch, v);
    }
    ld_vec<float, VEC>(w + static_cast<int64_t>(j) * ch + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc[i] += g[i] * v[i];
    if (j > 0) st_vec<T, VEC>(st + static_cast<int64_t>(j - 1) * ch, v);
  }
  ld_vec<float, VEC>(w + static_cast<int64_t>(taps - 1) * ch + c, g);
#pragma unroll
  for (int i = 0; i < VEC; ++i) acc[i] = silu_f(acc[i] + g[i] * cur[i]);
  if (taps > 1) st_vec<T, VEC>(st + static_cast<int64_t>(taps - 2) * ch, cur);
  st_vec<T, VEC>(out + static_cast<int64_t>(s) * ldo + c, acc);
}

// ---- latent attention, per token: a = [query latent qr | key-value latent r | shared rotary key rd]
//   cq = rms(a_q) wq;   entry = [rms(a_kv) wkv | rotate(a_rot)] -> pool row kvslot[t] (and a packed copy when asked for)
__device__ __forceinline__ void rope_cs(int64_t pos, double f, float& c, float& s) {
  double a = static_cast<double>(pos) * f;
  a -= 6.283185307179586 * rint(a * 0.15915494309189535);
  sincosf(static_cast<float>(a), &s, &c);
}
template <class T>
__global__ void __launch_bounds__(128) mix_latent_prep_kernel(const T* __restrict__ a, int64_t lda, int qr, int r, int rd, const float* __restrict__ wq,
                                                              const float* __restrict__ wkv, const double* __restrict__ freq,
                                                              const int64_t* __restrict__ pos, const int64_t* __restrict__ kvslot, T* __restrict__ cq,
                                                              T* __restrict__ entry, T* __restrict__ pool, float eps) {
  __shared__ float red[4];
  const int64_t t = blockIdx.x;
  const T* row = a + t * lda;
  float ss = 0.f;
  for (int c = threadIdx.x; c < qr; c += 128) { const float v = to_f<T>(row[c]); ss += v * v; }
  float g = rsqrtf(block_sum<4>(ss, red) / qr + eps);
  for (int c = threadIdx.x; c < qr; c += 128) cq[t * qr + c] = from_f<T>(to_f<T>(row[c]) * g * wq[c]);
  row += qr;
  ss = 0.f;
  for (int c = threadIdx.x; c < r; c += 128) { const float v = to_f<T>(row[c]); ss += v * v; }
  g = rsqrtf(block_sum<4>(ss, red) / r + eps);
  T* pe = pool + kvslot[t] * (r + rd);
  T* en = entry ? entry + t * (r + rd) : nullptr;
  for (int c = threadIdx.x; c < r; c += 128) {
    const T v = from_f<T>(to_f<T>(row[c]) * g * wkv[c]);
    pe[c] = v;
    if (en) en[c] = v;
  }
  const int half = rd / 2;
  for (int i = threadIdx.x; i < half; i += 128) {
    float cs, sn;
    rope_cs(pos[t], freq[i], cs, sn);
    const float u = to_f<T>(row[r + i]), v = to_f<T>(row[r + half + i]);
    const T x0 = from_f<T>(u * cs - v * sn), x1 = from_f<T>(v * cs + u * sn);
    pe[r + i] = x0; pe[r + half + i] = x1;
    if (en) { en[r + i] = x0; en[r + half + i] = x1; }
  }
}
// rotate columns [d, d + rd) of every head of q [T, H, dq] in place
template <class T>
__global__ void __launch_bounds__(128) mix_rope_kernel(T* __restrict__ q, int64_t ldq, int H, int dq, int d, int rd, const double* __restrict__ freq,
                                                       const int64_t* __restrict__ pos) {
  const int64_t t = blockIdx.x;
  const int half = rd / 2;
  __shared__ float sc[256], ss[256];
  for (int i = threadIdx.x; i < half; i += 128) rope_cs(pos[t], freq[i], sc[i], ss[i]);
  __syncthreads();
  for (int e = threadIdx.x; e < H * half; e += 128) {
    const int h = e / half, i = e % half;
    T* p = q + t * ldq + static_cast<int64_t>(h) * dq + d;
    const float u = to_f<T>(p[i]), v = to_f<T>(p[half + i]);
    p[i] = from_f<T>(u * sc[i] - v * ss[i]);
    p[half + i] = from_f<T>(v * sc[i] + u * ss[i]);
  }
}

// ---- windowed attention, per token: p = [queries heads x dim | keys kheads x dim].  Queries and keys are RMS-normed over the whole row
// and rotated in neighbouring pairs; q, k [T, heads, width] and the cached rows are zero beyond dim, values are the keys as projected.
// Pools are [pages, kheads, 16, width]; kp / vp (packed keys and values) may be null.
template <class T>
__global__ void __launch_bounds__(256) mix_qk_prep_kernel(const T* __restrict__ p, int64_t ldp, int heads, int kheads, int dim, int width, int rd,
                                                          const float* __restrict__ wq, const float* __restrict__ wk, const double* __restrict__ freq,
                                                          const int64_t* __restrict__ pos, const int64_t* __restrict__ kvslot, T* __restrict__ q,
                                                          T* __restrict__ kp, T* __restrict__ vp, T* __restrict__ k_pool, T* __restrict__ v_pool, float eps) {
  __shared__ float sc[256], sn[256], red[8];
  const int64_t t = blockIdx.x;
  const T* row = p + t * ldp;
  const int nq = heads * dim, nk = kheads * dim;
  for (int i = threadIdx.x; i < rd / 2; i += 256) rope_cs(pos[t], freq[i], sc[i], sn[i]);
  const bool vec = sizeof(T) == 2 && dim % 8 == 0 && ldp % 8 == 0 && rd % 8 == 0 && (reinterpret_cast<uintptr_t>(p) & 15) == 0;
  float sq = 0.f, sk = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 8; c < nq + nk; c += 2048) {
      float v[8];
      ld_vec<T, 8>(row + c, v);
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) a += v[i] * v[i];
      if (c < nq) sq += a; else sk += a;
    }
  } else {
    for (int c = threadIdx.x; c < nq + nk; c += 256) {
      const float v = to_f<T>(row[c]);
      if (c < nq) sq += v * v; else sk += v * v;
    }
  }
  const float rq = rsqrtf(block_sum<8>(sq, red) / nq + eps);
  const float rk = rsqrtf(block_sum<8>(sk, red) / nk + eps);           // (both sums end in a barrier: the angles are in place)
  const int64_t slot = kvslot[t], page = slot / 16, off = slot % 16;
  auto dst = [&](int g) { return ((page * kheads + g) * 16 + off) * width; };
  if (vec) {
    const int wu = width / 8;                                          // 16-byte units of a head
    for (int u = threadIdx.x; u < (heads + kheads) * wu; u += 256) {
      const int hd = u / wu, c = (u % wu) * 8;
      const bool key = hd >= heads;
      float x[8], y[8];
      if (c < dim) {
        float w[8];
        ld_vec<T, 8>(row + hd * dim + c, x);
        ld_vec<float, 8>(key ? wk + (hd - heads) * dim + c : wq + hd * dim + c, w);
        const float r = key ? rk : rq;
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = x[i] * r * w[i];
        if (c < rd) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float cs = sc[c / 2 + i], s = sn[c / 2 + i], a = y[2 * i], b = y[2 * i + 1];
            y[2 * i] = a * cs - b * s;
            y[2 * i + 1] = b * cs + a * s;
          }
        }
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = y[i] = 0.f;
      }
      if (!key) {
        st_vec<T, 8>(q + (t * heads + hd) * width + c, y);
      } else {
        const int g = hd - heads;
        st_vec<T, 8>(k_pool + dst(g) + c, y);
        st_vec<T, 8>(v_pool + dst(g) + c, x);
        if (kp) {
          st_vec<T, 8>(kp + (t * kheads + g) * width + c, y);
          st_vec<T, 8>(vp + (t * kheads + g) * width + c, x);
        }
      }
    }
    return;
  }
  for (int e = threadIdx.x; e < (heads + kheads) * width; e += 256) {
    const int hd = e / width, c = e % width;
    const bool key = hd >= heads;
    float x = 0.f, y = 0.f;
    if (c < dim) {
      const T* src = row + hd * dim;
      const float* w = key ? wk + (hd - heads) * dim : wq + hd * dim;
      const float r = key ? rk : rq;
      x = to_f<T>(src[c]);
      y = x * r * w[c];
      if (c < rd) {
        const int o = c ^ 1;
        const float z = to_f<T>(src[o]) * r * w[o], cs = sc[c / 2], s = sn[c / 2];
        y = (c & 1) ? y * cs + z * s : y * cs - z * s;
      }
    }
    if (!key) {
      q[(t * heads + hd) * width + c] = from_f<T>(y);
    } else {
      const int g = hd - heads;
      k_pool[dst(g) + c] = from_f<T>(y);
      v_pool[dst(g) + c] = from_f<T>(x);
      if (kp) {
        kp[(t * kheads + g) * width + c] = from_f<T>(y);
        vp[(t * kheads + g) * width + c] = from_f<T>(x);
      }
    }
  }
}
// packed keys and values of flat cache rows; ku / vu 16-byte units per head
__global__ void __launch_bounds__(256) mix_gather_keys_kernel(const uint4* __restrict__ k_pool, const uint4* __restrict__ v_pool,
                                                              const int64_t* __restrict__ rows, uint4* __restrict__ k, uint4* __restrict__ v, int64_t n,
                                                              int kheads, int ku, int vu) {
  const int64_t per = static_cast<int64_t>(kheads) * (ku + vu);
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x; i < n * per; i += static_cast<int64_t>(gridDim.x) * 256) {
    const int64_t at = i / per, r = rows[at];
    int rest = static_cast<int>(i % per);
    const bool value = rest >= kheads * ku;
    const int units = value ? vu : ku;
    if (value) rest -= kheads * ku;
    const int64_t src = ((r / 16 * kheads + rest / units) * 16 + r % 16) * units + rest % units, dst = at * kheads * units + rest;
    if (value) v[dst] = v_pool[src]; else k[dst] = k_pool[src];
  }
}

// gate and up columns interleaved in blocks of blk: y = g sigmoid(alpha g) (u + 1), g = min(gate, limit), u = clamp(up, -limit, limit)
template <class T>
__global__ void mix_clamped_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int64_t rows, int F, int blk, float limit, float alpha) {
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < rows * F; i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = i / F;
    const int c = static_cast<int>(i % F);
    const T* src = gu + r * 2 * F + (c / blk) * 2 * blk + c % blk;
    const float g = fminf(to_f<T>(src[0]), limit), u = fminf(fmaxf(to_f<T>(src[blk]), -limit), limit);
    out[i] = from_f<T>(g * sigmoid_f(alpha * g) * (u + 1.f));
  }
}

// x = gelu(x) or silu(x) in place
template <class T, int VEC, bool SILU>
__global__ void mix_act_kernel(T* __restrict__ x, int64_t n) {
  for (int64_t i = (static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x) * VEC; i < n; i += static_cast<int64_t>(gridDim.x) * blockDim.x * VEC) {
    float v[VEC];
    ld_vec<T, VEC>(x + i, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = SILU ? silu_f(v[j]) : gelu_tanh_f(v[j]);
    st_vec<T, VEC>(x + i, v);
  }
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_embed(const int64_t* ids, const void* emb, const float* w, float* x, void* h, int rows, int W, float eps, int dtype,
                             cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = W % 8 == 0 && al16(emb) && al16(x) && al16(h) && al16(w);
  MIX_DISPATCH(vec, (mix_embed_kernel<T, VEC><<<rows, 128, 0, st>>>(ids, static_cast<const T*>(emb), w, x, static_cast<T*>(h), W, eps)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_norm_add(const void* y, int64_t ldy, float* x, const float* w, const float* w_next, void* h, int rows, int W, float eps,
                                int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = W % 8 == 0 && ldy % 8 == 0 && al16(y) && al16(x) && al16(w) && al16(w_next) && al16(h);
  MIX_DISPATCH(vec, (mix_norm_add_kernel<T, VEC><<<rows, 256, 0, st>>>(static_cast<const T*>(y), ldy, x, w, w_next, static_cast<T*>(h), W, eps)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_rms(const float* x, const float* w, void* h, int rows, int W, float eps, int center, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = W % 8 == 0 && al16(x) && al16(w) && al16(h);
  MIX_DISPATCH(vec, (mix_rms_kernel<T, VEC><<<rows, 256, 0, st>>>(x, w, static_cast<T*>(h), W, eps, center)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_gated_norm(const void* y, int64_t ldy, const void* z, int64_t ldz, const float* w, void* out, int64_t ldo, int rows, int groups,
                                  int gs, float eps, int gate, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  const int64_t items = static_cast<int64_t>(rows) * groups;
  const bool vec = gs % 8 == 0 && ldy % 8 == 0 && ldz % 8 == 0 && ldo % 8 == 0 && al16(y) && al16(z) && al16(w) && al16(out);
  const bool wide = gs > 1024;
  const int64_t grid = wide ? items : (items + 7) / 8;
  if (vec && dtype == 0 && gs <= 128 && gate >= kSigmoidLast && gate <= kSiluLast) {
    using T = __nv_bfloat16;
    const unsigned blocks = static_cast<unsigned>((items + 31) / 32);
#define MIX_GNN(G)                                                                                                                        \
  mix_gated_norm_narrow_kernel<T, G><<<blocks, 256, 0, st>>>(static_cast<const T*>(y), ldy, static_cast<const T*>(z), ldz, w,              \
                                                             static_cast<T*>(out), ldo, items, groups, gs, eps)
    if (gate == kSiluFirst) MIX_GNN(kSiluFirst);
    else if (gate == kSiluLast) MIX_GNN(kSiluLast);
    else MIX_GNN(kSigmoidLast);
#undef MIX_GNN
    PRL_CUDA_CHECK(cudaGetLastError());
    return 0;
  }
#define MIX_GN(GF, WPG)                                                                                                                   \
  MIX_DISPATCH(vec, (mix_gated_norm_kernel<T, VEC, GF, WPG><<<static_cast<unsigned>(grid), 256, 0, st>>>(                                 \
                        static_cast<const T*>(y), ldy, static_cast<const T*>(z), ldz, w, static_cast<T*>(out), ldo, items, groups, gs, eps)))
  if (gate == kSiluFirst) {
    if (wide) MIX_GN(kSiluFirst, 8); else MIX_GN(kSiluFirst, 1);
  } else if (gate == kSiluLast) {
    if (wide) MIX_GN(kSiluLast, 8); else MIX_GN(kSiluLast, 1);
  } else if (gate == kSigmoidLast) {
    if (wide) MIX_GN(kSigmoidLast, 8); else MIX_GN(kSigmoidLast, 1);
  } else {
    return -223;
  }
#undef MIX_GN
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
// the last taps - 1 inputs of every span become its slot's state
extern "C" int prl_mix_conv_state(const void* x, int64_t ldx, void* state, const int32_t* cu, const int32_t* start, const int64_t* slot, int ch, int taps,
                                  int spans, int dtype, cudaStream_t st) {
  if (taps <= 1 || spans <= 0) return 0;
  if (spans > 65535) return -220;
  dim3 g2((ch + 127) / 128, spans);
  if (dtype == 0)
    mix_conv_state_kernel<__nv_bfloat16><<<g2, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(x), ldx, static_cast<__nv_bfloat16*>(state), cu, start, slot, ch,
                                                             taps);
  else
    mix_conv_state_kernel<float><<<g2, 128, 0, st>>>(static_cast<const float*>(x), ldx, static_cast<float*>(state), cu, start, slot, ch, taps);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
// x [total, ldx] -> out [total, ldo] and the carried taps of every span.  seq_of == nullptr: one token per span.
extern "C" int prl_mix_conv(const void* x, int64_t ldx, const float* w, const float* bias, void* state, const int32_t* cu, const int32_t* start,
                            const int64_t* slot, const int32_t* seq_of, void* out, int64_t ldo, int ch, int taps, int total, int spans, int dtype,
                            cudaStream_t st) {
  if (total <= 0 || spans <= 0) return 0;
  if (spans > 65535 || taps < 1) return -220;
  const bool vec = ch % 8 == 0 && ldx % 8 == 0 && ldo % 8 == 0 && al16(x) && al16(w) && al16(bias) && al16(state) && al16(out);
  const int per = 128 * (vec ? 8 : 1);
  const unsigned gx = (ch + per - 1) / per;
  if (seq_of == nullptr) {
    MIX_DISPATCH(vec, (mix_conv_step_kernel<T, VEC><<<dim3(gx, spans), 128, 0, st>>>(static_cast<const T*>(x), ldx, w, bias, static_cast<T*>(state), start,
                                                                                    slot, static_cast<T*>(out), ldo, ch, taps)));
    PRL_CUDA_CHECK(cudaGetLastError());
    return 0;
  }
  if (vec && taps >= 2 && taps <= 4 && total <= 65535 * 16) {
    dim3 gw(gx, (total + 15) / 16);
#define MIX_CW(TAPS)                                                                                                                     \
  do {                                                                                                                                   \
    if (dtype == 0) {                                                                                                                    \
      using T = __nv_bfloat16;                                                                                                           \
      mix_conv_window_kernel<T, TAPS, 16><<<gw, 128, 0, st>>>(static_cast<const T*>(x), ldx, w, bias, static_cast<const T*>(state), cu,   \
                                                              start, slot, seq_of, static_cast<T*>(out), ldo, ch, total);                \
    } else {                                                                                                                             \
      using T = float;                                                                                                                   \
      mix_conv_window_kernel<T, TAPS, 16><<<gw, 128, 0, st>>>(static_cast<const T*>(x), ldx, w, bias, static_cast<const T*>(state), cu,   \
                                                              start, slot, seq_of, static_cast<T*>(out), ldo, ch, total);                \
    }                                                                                                                                    \
  } while (0)
    if (taps == 2) MIX_CW(2);
    else if (taps == 3) MIX_CW(3);
    else MIX_CW(4);
#undef MIX_CW
    PRL_CUDA_CHECK(cudaGetLastError());
  } else {
    const int TT = total > 65535 * 4 ? 32 : 4;
    const unsigned gy = (total + TT - 1) / TT;
    if (gy > 65535) return -221;
    if (TT == 4)
      MIX_DISPATCH(vec, (mix_conv_kernel<T, VEC, 4><<<dim3(gx, gy), 128, 0, st>>>(static_cast<const T*>(x), ldx, w, bias, static_cast<const T*>(state), cu,
                                                                                 start, slot, seq_of, static_cast<T*>(out), ldo, ch, taps, total)));
    else
      MIX_DISPATCH(vec, (mix_conv_kernel<T, VEC, 32><<<dim3(gx, gy), 128, 0, st>>>(static_cast<const T*>(x), ldx, w, bias, static_cast<const T*>(state), cu,
                                                                                  start, slot, seq_of, static_cast<T*>(out), ldo, ch, taps, total)));
    PRL_CUDA_CHECK(cudaGetLastError());
  }
  return prl_mix_conv_state(x, ldx, state, cu, start, slot, ch, taps, spans, dtype, st);
}

extern "C" int prl_mix_latent_prep(const void* a, int64_t lda, int qr, int r, int rd, const float* wq, const float* wkv, const double* freq,
                                   const int64_t* pos, const int64_t* kvslot, void* cq, void* entry, void* pool, int rows, float eps, int dtype,
                                   cudaStream_t st) {
  if (rows <= 0) return 0;
  if (dtype == 0)
    mix_latent_prep_kernel<__nv_bfloat16><<<rows, 128, 0, st>>>(static_cast<const __nv_bfloat16*>(a), lda, qr, r, rd, wq, wkv, freq, pos, kvslot,
                                                                static_cast<__nv_bfloat16*>(cq), static_cast<__nv_bfloat16*>(entry),
                                                                static_cast<__nv_bfloat16*>(pool), eps);
  else
    mix_latent_prep_kernel<float><<<rows, 128, 0, st>>>(static_cast<const float*>(a), lda, qr, r, rd, wq, wkv, freq, pos, kvslot,
                                                        static_cast<float*>(cq), static_cast<float*>(entry), static_cast<float*>(pool), eps);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_rope(void* q, int64_t ldq, int H, int dq, int d, int rd, const double* freq, const int64_t* pos, int rows, int dtype,
                            cudaStream_t st) {
  if (rows <= 0 || rd <= 0) return 0;
  if (rd > 512) return -222;
  if (dtype == 0) mix_rope_kernel<__nv_bfloat16><<<rows, 128, 0, st>>>(static_cast<__nv_bfloat16*>(q), ldq, H, dq, d, rd, freq, pos);
  else mix_rope_kernel<float><<<rows, 128, 0, st>>>(static_cast<float*>(q), ldq, H, dq, d, rd, freq, pos);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_qk_prep(const void* p, int64_t ldp, int heads, int kheads, int dim, int width, int rd, const float* wq, const float* wk,
                               const double* freq, const int64_t* pos, const int64_t* kvslot, void* q, void* kp, void* vp, void* k_pool, void* v_pool, int rows,
                               float eps, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (rd > 512 || rd > dim || width < dim) return -224;
  if (dtype == 0) {
    using T = __nv_bfloat16;
    mix_qk_prep_kernel<T><<<rows, 256, 0, st>>>(static_cast<const T*>(p), ldp, heads, kheads, dim, width, rd, wq, wk, freq, pos, kvslot, static_cast<T*>(q),
                                                static_cast<T*>(kp), static_cast<T*>(vp), static_cast<T*>(k_pool), static_cast<T*>(v_pool), eps);
  } else {
    using T = float;
    mix_qk_prep_kernel<T><<<rows, 256, 0, st>>>(static_cast<const T*>(p), ldp, heads, kheads, dim, width, rd, wq, wk, freq, pos, kvslot, static_cast<T*>(q),
                                                static_cast<T*>(kp), static_cast<T*>(vp), static_cast<T*>(k_pool), static_cast<T*>(v_pool), eps);
  }
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
// row_bytes: bytes of one head's key, a multiple of 16
extern "C" int prl_mix_gather_keys(const void* k_pool, const void* v_pool, const int64_t* rows, void* k, void* v, int64_t n, int kheads, int k_bytes,
                                   int v_bytes, cudaStream_t st) {
  if (n <= 0) return 0;
  if (k_bytes % 16 || v_bytes % 16 || !al16(k_pool) || !al16(v_pool) || !al16(k) || !al16(v)) return -225;
  const int64_t blocks = (n * kheads * ((k_bytes + v_bytes) / 16) + 255) / 256;
  mix_gather_keys_kernel<<<static_cast<unsigned>(blocks < 148 * 32 ? blocks : 148 * 32), 256, 0, st>>>(
      static_cast<const uint4*>(k_pool), static_cast<const uint4*>(v_pool), rows, static_cast<uint4*>(k), static_cast<uint4*>(v), n, kheads, k_bytes / 16,
      v_bytes / 16);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int prl_mix_clamped_glu(const void* gu, void* out, int64_t rows, int F, int blk, float limit, float alpha, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (F <= 0 || blk <= 0 || F % blk) return -226;
  const int64_t blocks = (rows * F + 255) / 256;
  const unsigned grid = static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16);
  if (dtype == 0)
    mix_clamped_glu_kernel<<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(out), rows, F, blk, limit, alpha);
  else
    mix_clamped_glu_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(gu), static_cast<float*>(out), rows, F, blk, limit, alpha);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
extern "C" int prl_mix_gelu(void* x, int64_t n, int silu, int dtype, cudaStream_t st) {
  if (n <= 0) return 0;
  const bool vec = n % 8 == 0 && al16(x);
  const int64_t blocks = (n / (vec ? 8 : 1) + 255) / 256;
  const unsigned grid = static_cast<unsigned>(blocks < 148 * 16 ? blocks : 148 * 16);
  if (silu) MIX_DISPATCH(vec, (mix_act_kernel<T, VEC, true><<<grid > 0 ? grid : 1, 256, 0, st>>>(static_cast<T*>(x), n)));
  else MIX_DISPATCH(vec, (mix_act_kernel<T, VEC, false><<<grid > 0 ? grid : 1, 256, 0, st>>>(static_cast<T*>(x), n)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
