// polyrl_b200 — parallel blocks: the kernel between two layers, input convolutions, the polynomial activation, silu-gated rows.
//
// A layer's results are added, scaled, to its input x; the next layer reads a learned average over the embedding output and all
// results so far.  x is such an average itself, so it is recomputed from the stored results (fp32) by the kernel that reads them
// anyway, and never stored.  One CTA owns a token: it keeps the new row in shared memory, norms it and, when every span is a
// single token, runs the next layer's two input convolutions on it as well (their taps lie in the state slots).
#include "mixers.cuh"

namespace prl {

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// NT threads per token; the results are read four layers at a time, their coefficients lie in shared memory
template <class T, int VEC, int NT>
__global__ void __launch_bounds__(NT, 1024 / NT) mix_block_kernel(BlockParams p) {
  extern __shared__ float sh[];                        // row [W], then a_prev [n + 1] and a_cur [n + 2]
  __shared__ float red[NT / 32];
  float* ap = sh + (p.W + 3) / 4 * 4;
  float* ac = ap + p.n + 1;
  const int64_t row = blockIdx.x;
  const int W = p.W;
  float* xr = p.past + row * W;
  if (p.a_prev) for (int j = threadIdx.x; j <= p.n; j += NT) ap[j] = p.a_prev[j];
  if (p.a_cur) for (int j = threadIdx.x; j <= p.n + 1; j += NT) ac[j] = p.a_cur[j];
  if (p.c1) {                                           // what the convolution reads after the norm
    const T* st = static_cast<const T*>(p.state) + p.slot[row] * static_cast<int64_t>(p.taps - 1) * W;
    for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {
      prefetch_l2(p.w_next + c);
      for (int j = 0; j < p.taps; ++j) {
        if (j + 1 < p.taps) prefetch_l2(st + static_cast<int64_t>(j) * W + c);
        prefetch_l2(p.c1 + static_cast<int64_t>(j) * W + c);
        if (p.c2) prefetch_l2(p.c2 + static_cast<int64_t>(j) * W + c);
      }
    }
  }
  __syncthreads();
  float s = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {
    float x[VEC], avg[VEC];
    if (p.ids) {
      ld_vec<T, VEC>(static_cast<const T*>(p.emb) + p.ids[row] * W + c, x);
      st_vec<float, VEC>(xr + c, x);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) avg[i] = 0.f;
      if (p.a_prev || p.a_cur) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = 0.f;
#pragma unroll 4
        for (int j = 0; j <= p.n; ++j) {
          float v[VEC];
          ld_vec<float, VEC>(xr + j * p.stride + c, v);
          const float b = p.a_cur ? ac[j] : 0.f, a = p.a_prev ? ap[j] : (j == 0 ? 1.f : 0.f);
#pragma unroll
          for (int i = 0; i < VEC; ++i) { x[i] += a * v[i]; avg[i] += b * v[i]; }
        }
      } else {
        ld_vec<float, VEC>(xr + c, x);
      }
      float y[VEC];
      ld_vec<T, VEC>(static_cast<const T*>(p.y1) + row * p.ld1 + c, y);
      if (p.s1) {
        float g[VEC];
        ld_vec<float, VEC>(p.s1 + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] *= g[i];
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] += y[i];
      if (p.y2 || p.rows) {
        float f[VEC];
        if (p.y2) {
          ld_vec<T, VEC>(static_cast<const T*>(p.y2) + row * p.ld2 + c, f);
        } else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) f[i] = 0.f;
        }
        if (p.rows) {
          for (int j = 0; j < p.top; ++j) {
            float v[VEC];
            ld_vec<T, VEC>(static_cast<const T*>(p.rows) + static_cast<int64_t>(p.pos[row * p.top + j]) * W + c, v);
#pragma unroll
            for (int i = 0; i < VEC; ++i) f[i] += v[i];
          }
        }
        if (p.s2) {
          float g[VEC];
          ld_vec<float, VEC>(p.s2 + c, g);
#pragma unroll
          for (int i = 0; i < VEC; ++i) f[i] *= g[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] += f[i];
      }
      st_vec<float, VEC>(xr + (p.a_cur ? (p.n + 1) * p.stride : 0) + c, x);
      if (p.a_cur) {
        const float b = ac[p.n + 1];
#pragma unroll
        for (int i = 0; i < VEC; ++i) x[i] = avg[i] + b * x[i];
      }
      if (p.x_out) st_vec<float, VEC>(p.x_out + row * W + c, x);
    }
    st_vec<float, VEC>(sh + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) s += x[i];
  }
  if (!p.w_next) return;
  // a thread reads back only what it wrote to the row
  const float mean = p.center ? block_sum<NT / 32>(s, red) / W : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {
    float x[VEC];
    ld_vec<float, VEC>(sh + c, x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += (x[i] - mean) * (x[i] - mean);
  }
  const float r = rsqrtf(block_sum<NT / 32>(ss, red) / W + p.eps);
  const bool fresh = p.c1 && p.start[row] == 0;
  T* st = p.c1 ? static_cast<T*>(p.state) + p.slot[row] * static_cast<int64_t>(p.taps - 1) * W : nullptr;
  for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {
    float x[VEC], g[VEC];
    ld_vec<float, VEC>(sh + c, x);
    ld_vec<float, VEC>(p.w_next + c, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) x[i] = to_f<T>(from_f<T>((x[i] - mean) * r * g[i]));      // what a prompt's convolution reads
    if (!p.c1) {
      st_vec<T, VEC>(static_cast<T*>(p.h) + row * W + c, x);
      continue;
    }
    float u1[VEC], u2[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) u1[i] = u2[i] = x[i];
    for (int j = 0; j < p.taps; ++j) {
      float v[VEC];
      if (j + 1 == p.taps) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = x[i];
      } else if (fresh) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      } else {
        ld_vec<T, VEC>(st + static_cast<int64_t>(j) * W + c, v);
      }
      ld_vec<float, VEC>(p.c1 + static_cast<int64_t>(j) * W + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) u1[i] += g[i] * v[i];
      if (p.c2) {
        ld_vec<float, VEC>(p.c2 + static_cast<int64_t>(j) * W + c, g);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u2[i] += g[i] * v[i];
      }
      if (j > 0) st_vec<T, VEC>(st + static_cast<int64_t>(j - 1) * W + c, v);
    }
    st_vec<T, VEC>(static_cast<T*>(p.h) + row * W + c, u1);
    if (p.c2) st_vec<T, VEC>(static_cast<T*>(p.h2) + row * W + c, u2);
  }
}

// ---- h + causal convolution per channel, for two sublayers that read the same h; w [taps, ch], state [slots, taps - 1, ch]
template <class T, int VEC>
__global__ void __launch_bounds__(128) mix_input_conv_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w1, const float* __restrict__ w2,
                                                             const T* __restrict__ state, const int32_t* __restrict__ cu, const int32_t* __restrict__ start,
                                                             const int64_t* __restrict__ slot, const int32_t* __restrict__ seq_of, T* __restrict__ o1,
                                                             T* __restrict__ o2, int ch, int taps, int total) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC;
  if (c >= ch) return;
  for (int t = blockIdx.y; t < total; t += gridDim.y) {
    const int s = seq_of ? seq_of[t] : t, t0 = cu[s];
    const bool fresh = start[s] == 0;
    float a[VEC], b[VEC];
    ld_vec<T, VEC>(x + static_cast<int64_t>(t) * ldx + c, a);
#pragma unroll
    for (int i = 0; i < VEC; ++i) b[i] = a[i];
    for (int j = 0; j < taps; ++j) {
      const int u = t - (taps - 1) + j;
      float v[VEC], g[VEC];
      if (u >= t0) {
        ld_vec<T, VEC>(x + static_cast<int64_t>(u) * ldx + c, v);
      } else {
        if (fresh) continue;
        ld_vec<T, VEC>(state + (slot[s] * (taps - 1) + (u - t0 + taps - 1)) * ch + c, v);
      }
      ld_vec<float, VEC>(w1 + static_cast<int64_t>(j) * ch + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) a[i] += g[i] * v[i];
      if (!w2) continue;
      ld_vec<float, VEC>(w2 + static_cast<int64_t>(j) * ch + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) b[i] += g[i] * v[i];
    }
    st_vec<T, VEC>(o1 + static_cast<int64_t>(t) * ch + c, a);
    if (w2) st_vec<T, VEC>(o2 + static_cast<int64_t>(t) * ch + c, b);
  }
}
// the same for a fixed small tap count: 8 channels per thread, TT tokens with the window and the taps in registers
template <class T, int TAPS, bool TWO, int TT>
__global__ void __launch_bounds__(128) mix_input_conv_window_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w1,
                                                                    const float* __restrict__ w2, const T* __restrict__ state,
                                                                    const int32_t* __restrict__ cu, const int32_t* __restrict__ start,
                                                                    const int64_t* __restrict__ slot, const int32_t* __restrict__ seq_of,
                                                                    T* __restrict__ o1, T* __restrict__ o2, int ch, int total) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= ch) return;
  const int tb = blockIdx.y * TT, te = min(total, tb + TT);
  float wa[TAPS][8], wb[TAPS][8], win[TAPS][8];         // win[j]: input of token t - (TAPS - 1) + j
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    ld_vec<float, 8>(w1 + static_cast<int64_t>(j) * ch + c, wa[j]);
    if constexpr (TWO) ld_vec<float, 8>(w2 + static_cast<int64_t>(j) * ch + c, wb[j]);
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {                        // the token itself
    wa[TAPS - 1][i] += 1.f;
    if constexpr (TWO) wb[TAPS - 1][i] += 1.f;
  }
  int cur = -1;
#pragma unroll 4
  for (int t = tb; t < te; ++t) {
    const int s = seq_of[t];
    if (s != cur) {                                     // (re)fill the window at a span's start or at the tile's first token
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
    float a[8], b[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = b[i] = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        a[i] += wa[j][i] * win[j][i];
        if constexpr (TWO) b[i] += wb[j][i] * win[j][i];
      }
    st_vec<T, 8>(o1 + static_cast<int64_t>(t) * ch + c, a);
    if constexpr (TWO) st_vec<T, 8>(o2 + static_cast<int64_t>(t) * ch + c, b);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
  }
}

// ---- a N(z) + b N(z^2) + c N(z^3) + e over rows, N(u) = u / sqrt(mean(u^2) + eps); rows of up to 256 * VEC * HOLD stay in registers
template <class T, int VEC, int HOLD>
__global__ void __launch_bounds__(256) mix_poly_norm_kernel(const T* __restrict__ z, int64_t ldz, const float* __restrict__ act, T* __restrict__ out, int F,
                                                            float eps) {
  __shared__ float red[8][3];
  const int64_t row = blockIdx.x;
  const T* zr = z + row * ldz;
  constexpr int U = sizeof(T) * VEC % 16 == 0 ? sizeof(T) * VEC / 16 : 0;      // held as loaded: 16-byte units, or one element
  uint4 raw[HOLD][U ? U : 1];
  T one[HOLD];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto get = [&](int k, float (&v)[VEC]) {
    if constexpr (U > 0) ld_vec<T, VEC>(reinterpret_cast<const T*>(&raw[k][0]), v);
    else v[0] = to_f<T>(one[k]);
  };
  const bool held = F <= 256 * VEC * HOLD;
  auto add = [&](const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float q = v[i] * v[i], q2 = q * q;
      s1 += q; s2 += q2; s3 += q2 * q;
    }
  };
  if (held) {
#pragma unroll
    for (int k = 0; k < HOLD; ++k) {
      const int c = (k * 256 + threadIdx.x) * VEC;
      if (c < F) {
        if constexpr (U > 0) {
#pragma unroll
          for (int u = 0; u < U; ++u) raw[k][u] = reinterpret_cast<const uint4*>(zr + c)[u];
        } else {
          one[k] = zr[c];
        }
      }
    }
#pragma unroll
    for (int k = 0; k < HOLD; ++k) {
      if ((k * 256 + threadIdx.x) * VEC < F) {
        float v[VEC];
        get(k, v);
        add(v);
      }
    }
  } else {
    for (int c = threadIdx.x * VEC; c < F; c += 256 * VEC) {
      float v[VEC];
      ld_vec<T, VEC>(zr + c, v);
      add(v);
    }
  }
  s1 = warp_sum(s1); s2 = warp_sum(s2); s3 = warp_sum(s3);
  if ((threadIdx.x & 31) == 0) { red[threadIdx.x >> 5][0] = s1; red[threadIdx.x >> 5][1] = s2; red[threadIdx.x >> 5][2] = s3; }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { s1 += red[i][0]; s2 += red[i][1]; s3 += red[i][2]; }
  const float a = act[0] * rsqrtf(s1 / F + eps), b = act[1] * rsqrtf(s2 / F + eps), d = act[2] * rsqrtf(s3 / F + eps), e = act[3];
  auto put = [&](float (&v)[VEC], int c) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = e + v[i] * (a + v[i] * (b + v[i] * d));
    st_vec<T, VEC>(out + row * F + c, v);
  };
  if (held) {
#pragma unroll
    for (int k = 0; k < HOLD; ++k) {
      const int c = (k * 256 + threadIdx.x) * VEC;
      if (c < F) {
        float v[VEC];
        get(k, v);
        put(v, c);
      }
    }
  } else {
    for (int c = threadIdx.x * VEC; c < F; c += 256 * VEC) {
      float v[VEC];
      ld_vec<T, VEC>(zr + c, v);
      put(v, c);
    }
  }
}

// gate and up columns interleaved in blocks of blk: y = silu(g) u
template <class T>
__global__ void mix_silu_glu_kernel(const T* __restrict__ gu, T* __restrict__ out, int64_t rows, int F, int blk) {
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < rows * F; i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t r = i / F;
    const int c = static_cast<int>(i % F);
    const T* src = gu + r * 2 * F + (c / blk) * 2 * blk + c % blk;
    out[i] = from_f<T>(silu_f(to_f<T>(src[0])) * to_f<T>(src[blk]));
  }
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_conv_state(const void*, int64_t, void*, const int32_t*, const int32_t*, const int64_t*, int, int, int, int, cudaStream_t);

extern "C" int prl_mix_block(const BlockParams* bp, int dtype, cudaStream_t st) {
  const BlockParams& p = *bp;
  if (p.R <= 0) return 0;
  if (p.W < 1 || p.n < 0 || (p.c1 && p.taps < 1)) return -260;
  bool vec = p.W % 8 == 0 && p.stride % 8 == 0 && p.ld1 % 8 == 0 && p.ld2 % 8 == 0;
  for (const void* q : {static_cast<const void*>(p.past), p.emb, p.y1, p.y2, p.rows, static_cast<const void*>(p.s1), static_cast<const void*>(p.s2),
                        static_cast<const void*>(p.w_next), static_cast<const void*>(p.x_out), static_cast<const void*>(p.h), static_cast<const void*>(p.h2),
                        static_cast<const void*>(p.c1), static_cast<const void*>(p.c2), static_cast<const void*>(p.state)})
    vec = vec && al16(q);
  const int smem = ((p.W + 3) / 4 * 4 + 2 * p.n + 3) * 4;
  if (smem > 200 * 1024) return -261;
  // few rows: one vector per thread where the width allows it (latency); many: small CTAs that overlap one another's barriers
  const bool few = p.R <= 4 * 148;
#define MIX_BLOCK(NT)                                                                                                            \
  do {                                                                                                                           \
    if (smem > 40 * 1024)                                                                                                        \
      PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_block_kernel<T, VEC, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));     \
    mix_block_kernel<T, VEC, NT><<<p.R, NT, smem, st>>>(p);                                                                      \
  } while (0)
  MIX_DISPATCH(vec, {
    if (p.W <= 128 * VEC || !few) MIX_BLOCK(128);
    else if (p.W <= 256 * VEC) MIX_BLOCK(256);
    else MIX_BLOCK(512);
  });
#undef MIX_BLOCK
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

// x [total, ldx] -> x + conv(x) with w1 (o1) and, when given, w2 (o2), both [total, ch]; the carried taps of every span.  seq_of == nullptr: one
// token per span
extern "C" int prl_mix_input_conv(const void* x, int64_t ldx, const float* w1, const float* w2, void* state, const int32_t* cu, const int32_t* start,
                                  const int64_t* slot, const int32_t* seq_of, void* o1, void* o2, int ch, int taps, int total, int spans, int dtype,
                                  cudaStream_t st) {
  if (total <= 0 || spans <= 0) return 0;
  if (taps < 1) return -262;
  const bool vec = ch % 8 == 0 && ldx % 8 == 0 && al16(x) && al16(w1) && al16(w2) && al16(state) && al16(o1) && al16(o2);
  const int per = 128 * (vec ? 8 : 1);
  const unsigned gx = (ch + per - 1) / per;
  if (vec && seq_of && taps >= 2 && taps <= 4 && total <= 65535 * 16) {
    const dim3 grid(gx, (total + 15) / 16);
#define MIX_IC(T, TAPS, TWO)                                                                                                                              \
  mix_input_conv_window_kernel<T, TAPS, TWO, 16><<<grid, 128, 0, st>>>(static_cast<const T*>(x), ldx, w1, w2, static_cast<const T*>(state), cu, start, slot, \
                                                                       seq_of, static_cast<T*>(o1), static_cast<T*>(o2), ch, total)
#define MIX_IC_T(T)                                                                                                                                       \
  do {                                                                                                                                                    \
    if (taps == 2) { if (w2) MIX_IC(T, 2, true); else MIX_IC(T, 2, false); }                                                                              \
    else if (taps == 3) { if (w2) MIX_IC(T, 3, true); else MIX_IC(T, 3, false); }                                                                         \
    else { if (w2) MIX_IC(T, 4, true); else MIX_IC(T, 4, false); }                                                                                        \
  } while (0)
    if (dtype == 0) MIX_IC_T(__nv_bfloat16);
    else MIX_IC_T(float);
#undef MIX_IC_T
#undef MIX_IC
  } else {
    const dim3 grid(gx, total < 65535 ? total : 65535);
    MIX_DISPATCH(vec, (mix_input_conv_kernel<T, VEC><<<grid, 128, 0, st>>>(static_cast<const T*>(x), ldx, w1, w2, static_cast<const T*>(state), cu, start,
                                                                           slot, seq_of, static_cast<T*>(o1), static_cast<T*>(o2), ch, taps, total)));
  }
  PRL_CUDA_CHECK(cudaGetLastError());
  return prl_mix_conv_state(x, ldx, state, cu, start, slot, ch, taps, spans, dtype, st);
}

extern "C" int prl_mix_poly_norm(const void* z, int64_t ldz, const float* act, void* out, int rows, int F, float eps, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  const bool vec = F % 8 == 0 && ldz % 8 == 0 && al16(z) && al16(out);
#define MIX_PN(T, VEC, HOLD) mix_poly_norm_kernel<T, VEC, HOLD><<<rows, 256, 0, st>>>(static_cast<const T*>(z), ldz, act, static_cast<T*>(out), F, eps)
  if (dtype == 0) {
    using T = __nv_bfloat16;
    if (!vec) MIX_PN(T, 1, 8);
    else if (F <= 256 * 8) MIX_PN(T, 8, 1);
    else if (F <= 256 * 8 * 4) MIX_PN(T, 8, 4);
    else MIX_PN(T, 8, 8);
  } else if (vec) {
    MIX_PN(float, 8, 2);
  } else {
    MIX_PN(float, 1, 8);
  }
#undef MIX_PN
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int prl_mix_silu_glu(const void* gu, void* out, int64_t rows, int F, int blk, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (F <= 0 || blk <= 0 || F % blk) return -263;
  const int64_t n = (rows * F + 255) / 256;
  const unsigned grid = static_cast<unsigned>(n < 148 * 32 ? n : 148 * 32);
  if (dtype == 0) mix_silu_glu_kernel<<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(gu), static_cast<__nv_bfloat16*>(out), rows, F, blk);
  else mix_silu_glu_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(gu), static_cast<float*>(out), rows, F, blk);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
