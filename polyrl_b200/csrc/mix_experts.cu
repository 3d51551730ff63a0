// polyrl_b200 — mixture of experts without host synchronisation: routing, rows in the experts' order, a plain grouped product.
//
// The plan of a step is device data: plan[0] = number of 128-row tiles, plan[1 + e] = first row of expert e (a multiple of 128),
// plan[1 + E + i] = expert of tile i, and above its 16 bits the tile's rows in use.  Grids are sized for the worst case and leave early, so a decode step can be captured.
// The order of an expert's rows depends on arrival; every row is computed by itself, so results do not.
#include "mixers.cuh"

namespace prl {

constexpr int kMoeTile = 128;
// a warp per token, `per` tokens per CTA: the `top` largest logits (ties: the lower index); s = sigmoid, or the softmax over all experts divided by
// the sum of the chosen ones (+ 1e-20); counts [E + 1] are zero between launches
template <int RN, bool SOFTMAX>
__global__ void __launch_bounds__(256) mix_route_kernel(const float* __restrict__ logits, int64_t ld, int T, int E, int top, int per, int32_t* __restrict__ pick,
                                                        float* __restrict__ score, int32_t* __restrict__ rank, int32_t* __restrict__ counts,
                                                        int32_t* __restrict__ plan) {
  extern __shared__ int hist[];                         // [E]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < E; e += 256) hist[e] = 0;
  __syncthreads();
  for (int i = warp; i < per; i += 8) {
    const int t = blockIdx.x * per + i;
    if (t >= T) break;
    float v[RN], top_v = 0.f, all = 0.f, chosen = 0.f;
    uint32_t taken = 0;
#pragma unroll
    for (int r = 0; r < RN; ++r) {
      const int e = r * 32 + lane;
      v[r] = e < E ? logits[t * ld + e] : 0.f;
      if (!(v[r] == v[r])) v[r] = -INFINITY;
      if (e >= E) taken |= 1u << r;
    }
    if (SOFTMAX) {
      top_v = -INFINITY;
#pragma unroll
      for (int r = 0; r < RN; ++r)
        if (r * 32 + lane < E) top_v = fmaxf(top_v, v[r]);
      top_v = warp_max(top_v);
#pragma unroll
      for (int r = 0; r < RN; ++r)
        if (r * 32 + lane < E) all += expf(v[r] - top_v);
      all = warp_sum(all);
    }
    for (int k = 0; k < top; ++k) {
      float bv = -INFINITY;
      int be = 0x7fffffff;
#pragma unroll
      for (int r = 0; r < RN; ++r) {
        const int e = r * 32 + lane;
        if (!(taken >> r & 1) && (v[r] > bv || (v[r] == bv && e < be))) { bv = v[r]; be = e; }
      }
#pragma unroll
      for (int o = 16; o; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ov > bv || (ov == bv && oe < be)) { bv = ov; be = oe; }
      }
      if ((be & 31) == lane) taken |= 1u << (be >> 5);
      const float s = SOFTMAX ? expf(bv - top_v) / all : sigmoid_f(bv);
      chosen += s;
      if (lane == 0) {
        const int64_t at = static_cast<int64_t>(t) * top + k;
        pick[at] = be;
        score[at] = s;
        rank[at] = atomicAdd(&hist[be], 1);
      }
    }
    if (SOFTMAX && lane == 0)
      for (int k = 0; k < top; ++k) score[static_cast<int64_t>(t) * top + k] /= chosen + 1e-20f;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256)
    if (hist[e]) hist[e] = atomicAdd(&counts[e], hist[e]);
  __syncthreads();
  if (lane == 0) {
    for (int i = warp; i < per; i += 8) {
      const int t = blockIdx.x * per + i;
      if (t >= T) break;
      for (int k = 0; k < top; ++k) {
        const int64_t at = static_cast<int64_t>(t) * top + k;
        rank[at] += hist[pick[at]];
      }
    }
  }
  if (!last_tile(&counts[E], gridDim.x)) return;
  // the last CTA to arrive has everybody's counts: first rows by a warp scan, then the experts of the tiles
  if (warp == 0) {
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      const int rows = e < E ? atomicAdd(&counts[e], 0) : 0, tiles = (rows + kMoeTile - 1) / kMoeTile;
      int sum = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      if (e < E) {
        plan[1 + e] = (base + sum - tiles) * kMoeTile;
        hist[e] = rows;
        counts[e] = 0;
      }
      base += __shfl_sync(0xffffffffu, sum, 31);
    }
    if (lane == 0) plan[0] = base;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256) {
    const int first = plan[1 + e] / kMoeTile;
    for (int r = 0; r < hist[e]; r += kMoeTile) plan[1 + E + first + r / kMoeTile] = e | min(kMoeTile, hist[e] - r) << 16;
  }
}

// rows[first row of the expert + rank] = h[t], times its score where there are scores
template <class T, int VEC>
__global__ void __launch_bounds__(128) mix_expert_rows_kernel(const T* __restrict__ h, int64_t ldh, const int32_t* __restrict__ pick,
                                                              const float* __restrict__ score, const int32_t* __restrict__ rank,
                                                              const int32_t* __restrict__ plan, T* __restrict__ rows, int32_t* __restrict__ pos, int top,
                                                              int W) {
  const int64_t t = blockIdx.x;
  for (int k = threadIdx.x; k < top; k += 128) pos[t * top + k] = plan[1 + pick[t * top + k]] + rank[t * top + k];
  __syncthreads();
  for (int c = threadIdx.x * VEC; c < W; c += 128 * VEC) {
    float v[VEC];
    ld_vec<T, VEC>(h + t * ldh + c, v);
    for (int k = 0; k < top; ++k) {
      const float s = score ? score[t * top + k] : 1.f;
      float y[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) y[i] = v[i] * s;
      st_vec<T, VEC>(rows + static_cast<int64_t>(plan[1 + pick[t * top + k]] + rank[t * top + k]) * W + c, y);
    }
  }
}

// out[r, n] = sum_k x[r, k] w[expert of r's tile * N + n, k]; 64 x 64 tiles, fp32 products and sums
template <class T>
__global__ void __launch_bounds__(256) mix_expert_gemm_kernel(const T* __restrict__ x, const T* __restrict__ w, const int32_t* __restrict__ plan,
                                                              T* __restrict__ out, int E, int N, int K) {
  __shared__ float sa[16][68], sb[16][68];
  if (static_cast<int>(blockIdx.y) / 2 >= plan[0]) return;
  const int64_t r0 = static_cast<int64_t>(blockIdx.y) * 64;
  const int n0 = blockIdx.x * 64;
  const int64_t w0 = static_cast<int64_t>(plan[1 + E + blockIdx.y / 2] & 0xffff) * N;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256, r = idx >> 4, k = idx & 15;
      sa[k][r] = k0 + k < K ? to_f<T>(x[(r0 + r) * K + k0 + k]) : 0.f;
      sb[k][r] = k0 + k < K && n0 + r < N ? to_f<T>(w[(w0 + n0 + r) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sa[k][ty * 4 + i]; b[i] = sb[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * b[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tx * 4 + j < N) out[(r0 + ty * 4 + i) * N + n0 + tx * 4 + j] = from_f<T>(acc[i][j]);
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_route_tiles(int64_t rows, int64_t experts) {         // upper bound on the tiles of `rows` routed rows
  return static_cast<int>(rows / kMoeTile + (rows < experts ? rows : experts));
}

extern "C" int prl_mix_route(const float* logits, int64_t ld, int T, int E, int top, int32_t* pick, float* score, int32_t* rank, int32_t* counts, int32_t* plan,
                             int softmax, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E < 1 || E > 1024 || top < 1 || top > E) return -270;
  const int per = T <= 8 * 148 ? 8 : 32, grid = (T + per - 1) / per;
#define MIX_RT(RN)                                                                                                                        \
  do {                                                                                                                                    \
    if (softmax) mix_route_kernel<RN, true><<<grid, 256, E * 4, st>>>(logits, ld, T, E, top, per, pick, score, rank, counts, plan);        \
    else mix_route_kernel<RN, false><<<grid, 256, E * 4, st>>>(logits, ld, T, E, top, per, pick, score, rank, counts, plan);               \
  } while (0)
  if (E <= 32) MIX_RT(1);
  else if (E <= 128) MIX_RT(4);
  else MIX_RT(32);
#undef MIX_RT
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int prl_mix_expert_rows(const void* h, int64_t ldh, const int32_t* pick, const float* score, const int32_t* rank, const int32_t* plan, void* rows,
                                   int32_t* pos, int tokens, int top, int W, int dtype, cudaStream_t st) {
  if (tokens <= 0) return 0;
  const bool vec = W % 8 == 0 && ldh % 8 == 0 && al16(h) && al16(rows);
  MIX_DISPATCH(vec, (mix_expert_rows_kernel<T, VEC><<<tokens, 128, 0, st>>>(static_cast<const T*>(h), ldh, pick, score, rank, plan, static_cast<T*>(rows), pos, top,
                                                                       W)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int prl_mix_expert_gemm(const void* x, const void* w, const int32_t* plan, void* out, int tiles, int E, int N, int K, int dtype, cudaStream_t st) {
  if (tiles <= 0 || N <= 0) return 0;
  if (tiles > 32767 || K < 1) return -271;
  const dim3 grid((N + 63) / 64, 2 * tiles);
  if (dtype == 0)
    mix_expert_gemm_kernel<<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(w), plan,
                                                 static_cast<__nv_bfloat16*>(out), E, N, K);
  else
    mix_expert_gemm_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(x), static_cast<const float*>(w), plan, static_cast<float*>(out), E, N, K);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
