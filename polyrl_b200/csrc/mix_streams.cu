// polyrl_b200 — residual streams with hyper-connections: the end of one sublayer and the beginning of the next.
//
//   X_t = sum_s mix[s, t] x_s + out[t] (y + bias + weighted routed rows),     h = norm(sum_t win[t] X_t) * g
//
// One CTA owns a token: every stream of it is read and written once (fp32), the row that the next sublayer reads stays in shared memory for
// its norm.  Until the first sublayer has ended all streams are the embedding output and are held once (stride 0 between streams); after the
// last one only their sum is written.
#include "mixers.cuh"

namespace prl {

template <class T, int VEC, int SM, int NT>
__global__ void __launch_bounds__(NT, SM * VEC > 32 ? 1 : 1024 / NT) mix_streams_kernel(StreamsParams p) {
  extern __shared__ float sh[];                        // row [W], mix [SM][SM] (from, to), out [SM], win [SM]
  __shared__ float red[NT / 32];
  float* cm = sh + (p.W + 3) / 4 * 4;
  float *co = cm + SM * SM, *ci = co + SM;
  const int64_t row = blockIdx.x;
  const int W = p.W, S = p.S;
  for (int i = threadIdx.x; i < SM * SM; i += NT) {
    const int s = i / SM, t = i % SM;
    cm[i] = p.mix && s < S && t < S ? p.mix[s * S + t] : 0.f;
  }
  if (threadIdx.x < SM) {
    co[threadIdx.x] = p.out && threadIdx.x < S ? p.out[threadIdx.x] : 0.f;
    ci[threadIdx.x] = threadIdx.x < S ? (p.win ? p.win[threadIdx.x] : 1.f) : 0.f;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {
    float u[VEC];
    if (p.ids) {
      float x[VEC], sum = 0.f;
      ld_vec<T, VEC>(static_cast<const T*>(p.emb) + p.ids[row] * W + c, x);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] *= p.scale;
      st_vec<float, VEC>(p.x_out + row * p.row_out + c, x);
#pragma unroll
      for (int s = 0; s < SM; ++s) sum += ci[s];
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[i] = sum * x[i];
    } else {
      float x[SM][VEC], y[VEC];
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s < S && (s == 0 || p.stream_in)) {
          ld_vec<float, VEC>(p.x_in + row * p.row_in + s * p.stream_in + c, x[s]);
        } else {
#pragma unroll
          for (int i = 0; i < VEC; ++i) x[s][i] = s < S ? x[0][i] : 0.f;
        }
      }
      if (p.y) {
        ld_vec<T, VEC>(static_cast<const T*>(p.y) + row * p.ldy + c, y);
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] = 0.f;
      }
      if (p.bias) {
        float v[VEC];
        ld_vec<float, VEC>(p.bias + c, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y[i] += v[i];
      }
      if (p.rows) {
        for (int j = 0; j < p.top; ++j) {
          const int64_t at = row * p.top + j;
          const float g = p.weight ? p.weight[at] : 1.f;
          float v[VEC];
          ld_vec<T, VEC>(static_cast<const T*>(p.rows) + static_cast<int64_t>(p.pos[at]) * W + c, v);
#pragma unroll
          for (int i = 0; i < VEC; ++i) y[i] += g * v[i];
        }
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) u[i] = 0.f;
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) break;
        float z[VEC];
        const float o = co[t], w = ci[t];
#pragma unroll
        for (int i = 0; i < VEC; ++i) z[i] = o * y[i];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          const float m = cm[s * SM + t];
#pragma unroll
          for (int i = 0; i < VEC; ++i) z[i] += m * x[s][i];
        }
        if (p.x_out) st_vec<float, VEC>(p.x_out + row * p.row_out + static_cast<int64_t>(t) * W + c, z);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u[i] += w * z[i];
      }
      if (p.sum) st_vec<float, VEC>(p.sum + row * W + c, u);
    }
    st_vec<float, VEC>(sh + c, u);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss += u[i] * u[i];
  }
  if (!p.w_next) return;
  const float r = rsqrtf(block_sum<NT / 32>(ss, red) / W + p.eps);
  const float one = p.w_scalar ? p.w_next[0] * r : r;
  for (int c = threadIdx.x * VEC; c < W; c += NT * VEC) {          // (a thread reads back only what it wrote)
    float x[VEC];
    ld_vec<float, VEC>(sh + c, x);
    if (p.w_scalar) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] *= one;
    } else {
      float g[VEC];
      ld_vec<float, VEC>(p.w_next + c, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) x[i] *= r * g[i];
    }
    st_vec<T, VEC>(static_cast<T*>(p.h) + row * W + c, x);
  }
}

template <class T, int VEC, int SM>
static int run_streams(const StreamsParams& p, cudaStream_t st) {
  const int smem = ((p.W + 3) / 4 * 4 + SM * SM + 2 * SM) * 4;
  if (smem > 200 * 1024) return -291;
  // few rows: one vector per thread where the width allows it (latency); many: small CTAs that overlap one another's barriers
  const bool few = p.R <= 4 * 148;
#define MIX_STREAMS(NT)                                                                                                                  \
  do {                                                                                                                                   \
    if (smem > 40 * 1024)                                                                                                                \
      PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_streams_kernel<T, VEC, SM, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));       \
    mix_streams_kernel<T, VEC, SM, NT><<<p.R, NT, smem, st>>>(p);                                                                        \
  } while (0)
  if (p.W <= 128 * VEC || !few) MIX_STREAMS(128);
  else if (p.W <= 256 * VEC) MIX_STREAMS(256);
  else MIX_STREAMS(512);
#undef MIX_STREAMS
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <class T>
static int pick_streams(const StreamsParams& p, bool vec, cudaStream_t st) {
  if (!vec || p.S > 8) return run_streams<T, 1, 16>(p, st);
  if (p.S <= 1) return run_streams<T, 8, 1>(p, st);
  if (p.S <= 2) return run_streams<T, 8, 2>(p, st);
  if (p.S <= 4) return run_streams<T, 8, 4>(p, st);
  return run_streams<T, 8, 8>(p, st);
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_streams(const StreamsParams* sp, int dtype, cudaStream_t st) {
  const StreamsParams& p = *sp;
  if (p.R <= 0) return 0;
  if (p.W < 1 || p.S < 1 || p.S > 16) return -290;
  bool vec = p.W % 8 == 0 && p.ldy % 8 == 0;
  for (const void* q : {static_cast<const void*>(p.x_in), static_cast<const void*>(p.x_out), static_cast<const void*>(p.sum), p.emb, p.y, p.rows,
                        static_cast<const void*>(p.bias), static_cast<const void*>(p.w_scalar ? nullptr : p.w_next), static_cast<const void*>(p.h)})
    vec = vec && al16(q);
  return dtype == 0 ? pick_streams<__nv_bfloat16>(p, vec, st) : pick_streams<float>(p, vec, st);
}
