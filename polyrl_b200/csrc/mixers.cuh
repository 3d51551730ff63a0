// polyrl_b200 — shared pieces of the sequence-mixer kernels (mix_elem.cu, mix_scan.cu, mix_chunk.cu, mix_latent.cu).
//
// Every kernel works on a PACKED batch of spans: span s holds the tokens [cu[s], cu[s+1]) of one sequence, whose first
// start[s] tokens were processed by earlier steps.  A decoded token is a span of length one, so prefill portions and
// decoded tokens share one launch.  Recurrent state lives in pools indexed by slot[s]; a span with start == 0 begins from
// the zero state whatever its slot held before.  Activations are T = bf16 or fp32; states, gates and norms are fp32.
#pragma once
#include "common.cuh"
#include "mix_params.hpp"

namespace prl {

template <class T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <class T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// VEC consecutive elements <-> fp32 registers (VEC * sizeof(T) <= 32 bytes, aligned when VEC > 1)
template <class T, int VEC>
__device__ __forceinline__ void ld_vec(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    v[0] = to_f<T>(p[0]);
  } else if constexpr (sizeof(T) == 2) {
    const uint4 q = *reinterpret_cast<const uint4*>(p);
    const float2 a = unpack_bf16(q.x), b = unpack_bf16(q.y), c = unpack_bf16(q.z), d = unpack_bf16(q.w);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y; v[4] = c.x; v[5] = c.y; v[6] = d.x; v[7] = d.y;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 q = *reinterpret_cast<const float4*>(p + i);
      v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
    }
  }
}
template <class T, int VEC>
__device__ __forceinline__ void st_vec(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 1) {
    p[0] = from_f<T>(v[0]);
  } else if constexpr (sizeof(T) == 2) {
    uint4 q;
    q.x = pack_bf16(v[0], v[1]); q.y = pack_bf16(v[2], v[3]); q.z = pack_bf16(v[4], v[5]); q.w = pack_bf16(v[6], v[7]);
    *reinterpret_cast<uint4*>(p) = q;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  }
}

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// bf16 outputs: the fast exponential and division (relative error about 2^-21) are far below the output's rounding
template <class T>
__device__ __forceinline__ float sigmoid_t(float z) {
  return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(fminf(-z, 80.f))) : sigmoid_f(z);
}
template <class T>
__device__ __forceinline__ float silu_t(float z) { return z * sigmoid_t<T>(z); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float logsigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// softplus by log(1 + e) = 2 artanh(e / (2 + e)), e = exp(-|z|) <= 1: seven terms of the series, below 2e-8 relative
__device__ __forceinline__ float softplus_series(float z) {
  const float e = __expf(-fabsf(z)), s = __fdividef(e, 2.f + e), q = s * s;
  float a = 1.f / 13.f;
  a = a * q + 1.f / 11.f;
  a = a * q + 1.f / 9.f;
  a = a * q + 1.f / 7.f;
  a = a * q + 1.f / 5.f;
  a = a * q + 1.f / 3.f;
  a = a * q + 1.f;
  return fmaxf(z, 0.f) + 2.f * s * a;
}
// exp of x <= 0, to the last bit near 1: a slow decay is the distance from 1, and its rounding adds up over a sequence
__device__ __forceinline__ float decay_f(float x) { return x > -0.5f ? 1.f + expm1f(x) : expf(x); }
__device__ __forceinline__ float softcap_f(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// sum over a block of WARPS warps; every thread gets the result.  `red` is WARPS floats of shared memory.
template <int WARPS>
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if constexpr (WARPS == 1) return v;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < WARPS; ++i) s += red[i];
  return s;
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// dtype: 0 = bf16, 1 = fp32.  VEC = 8 when every row of every operand starts on a 16-byte boundary.
#define MIX_DISPATCH(vec_, ...)                                                                      \
  do {                                                                                               \
    if (dtype == 0) {                                                                                \
      using T = __nv_bfloat16;                                                                       \
      if (vec_) { constexpr int VEC = 8; __VA_ARGS__; } else { constexpr int VEC = 1; __VA_ARGS__; } \
    } else {                                                                                         \
      using T = float;                                                                               \
      if (vec_) { constexpr int VEC = 8; __VA_ARGS__; } else { constexpr int VEC = 1; __VA_ARGS__; } \
    }                                                                                                \
  } while (0)

// The gated linear recurrences served by mix_scan.cu / mix_chunk.cu / mix_delta.cu:
//   S_t = keep_t S_(t-1) + add_t k_t v_t^T,     y_t = S_t^T q_t
//   kSsd    state-space duality: dt = softplus(g0 + b0), keep = exp(-exp(A_log) dt), add = dt;   y += D v
//   kMlstm  matrix memory with a running maximum m and normaliser n (csrc/mix_scan.cu)
//   kDelta  gated delta rule: unit k and q, the write corrects what the decayed state already answers for k (csrc/mix_scan.cu)
//   kDecay  constant decay per head: keep = exp(a_log), add = 1
//   kGla    a decay for every state row: keep_n = sigmoid(g0_n + b0_n)^(1 / cap), add = 1
enum : int { kSsd = 0, kMlstm = 1, kDelta = 2, kDecay = 3, kGla = 4 };
constexpr float kUnitEps = 1e-6f;        // under the root of a unit vector's norm

// n and m are read by every value tile of a head and may be overwritten only after the last tile has read them: the last
// CTA of a (span, head) to finish writes them (all tiles compute the same values).  Returns true for that CTA.
__device__ __forceinline__ bool last_tile(int32_t* counter, int tiles) {
  __shared__ int s_last;
  __syncthreads();
  if (threadIdx.x == 0) {
    __threadfence();
    const int old = atomicAdd(counter, 1);
    s_last = old == tiles - 1;
    if (s_last) *counter = 0;
    __threadfence();
  }
  __syncthreads();
  return s_last != 0;
}

}  // namespace prl
