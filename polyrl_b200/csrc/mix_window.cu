// polyrl_b200 — paged grouped-query attention of any head width, bf16 or fp32: in a sliding window with kept first tokens, or with a sink.
//
// A query row sees its last `window` keys (its own included) and the first `keep_first` keys of its sequence.  One CTA per (head, row),
// one key per warp and step, fp32 throughout.  bf16 rows of width 64 and 128 take the tensor-core kernels instead: decode_attn.cu for
// single tokens, attn_fwd.cu for prompt portions.
#include "mixers.cuh"

namespace prl {

constexpr int kWnWarps = 8;

template <class T, int RN>
__global__ void __launch_bounds__(kWnWarps * 32) mix_window_row_kernel(WindowParams p) {
  extern __shared__ float sh[];                   // [kWnWarps][D]
  __shared__ float sm[kWnWarps], sl[kWnWarps];
  const int h = blockIdx.x, row = blockIdx.y, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G);
  const T* qr = static_cast<const T*>(p.q) + (static_cast<int64_t>(row) * p.H + h) * p.D;
  float q[RN], o[RN];
#pragma unroll
  for (int i = 0; i < RN; ++i) {
    const int c = i * 32 + lane;
    q[i] = c < p.D ? to_f<T>(qr[c]) * p.scale : 0.f;
    o[i] = 0.f;
  }
  const int len = p.kv_len[row];
  const int first = max(0, len - p.window), kept = min(p.keep_first, first);
  const int n = kept + len - first;               // visible keys: [0, kept) and [first, len)
  const int32_t* bt = p.table + static_cast<int64_t>(p.seq_of ? p.seq_of[row] : row) * p.ld_table;
  const T* kp = static_cast<const T*>(p.k_pool);
  const T* vp = static_cast<const T*>(p.v_pool);
  float m = -INFINITY, l = 0.f;
  for (int e = w; e < n; e += kWnWarps) {
    const int j = e < kept ? e : e - kept + first;
    const int64_t at = ((static_cast<int64_t>(bt[j / 16]) * p.G + g) * 16 + j % 16) * p.D;
    float s = 0.f, v[RN];
#pragma unroll
    for (int i = 0; i < RN; ++i) {
      const int c = i * 32 + lane;
      v[i] = c < p.D ? to_f<T>(vp[at + c]) : 0.f;
      s += c < p.D ? q[i] * to_f<T>(kp[at + c]) : 0.f;
    }
    s = warp_sum(s);
    const float m2 = fmaxf(m, s), a = expf(m - m2), b = expf(s - m2);
    m = m2;
    l = l * a + b;
#pragma unroll
    for (int i = 0; i < RN; ++i) o[i] = o[i] * a + b * v[i];
  }
  if (lane == 0) { sm[w] = m; sl[w] = l; }
#pragma unroll
  for (int i = 0; i < RN; ++i)
    if (i * 32 + lane < p.D) sh[w * p.D + i * 32 + lane] = o[i];
  __syncthreads();
  float mm = -INFINITY;
  for (int i = 0; i < kWnWarps; ++i) mm = fmaxf(mm, sm[i]);
  T* out = static_cast<T*>(p.out) + (static_cast<int64_t>(row) * p.H + h) * p.D;
  for (int c = threadIdx.x; c < p.D; c += kWnWarps * 32) {
    float acc = 0.f, ll = 0.f;
    for (int i = 0; i < kWnWarps; ++i) {
      const float f = sm[i] == -INFINITY ? 0.f : expf(sm[i] - mm);
      acc += f * sh[i * p.D + c];
      ll += f * sl[i];
    }
    out[c] = from_f<T>(ll > 0.f ? acc / ll : 0.f);
  }
}

template <class T>
static int run_window(const WindowParams& p, cudaStream_t st) {
  const dim3 grid(p.H, p.R);
  const int smem = kWnWarps * p.D * 4;
  if (p.D <= 64) mix_window_row_kernel<T, 2><<<grid, kWnWarps * 32, smem, st>>>(p);
  else if (p.D <= 128) mix_window_row_kernel<T, 4><<<grid, kWnWarps * 32, smem, st>>>(p);
  else if (p.D <= 256) mix_window_row_kernel<T, 8><<<grid, kWnWarps * 32, smem, st>>>(p);
  else mix_window_row_kernel<T, 32><<<grid, kWnWarps * 32, smem, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

// the same without a window: separate key and value widths, and a sink in the denominator
template <class T, int RK, int RV>
__global__ void __launch_bounds__(kWnWarps * 32) mix_sink_row_kernel(SinkParams p) {
  extern __shared__ float sh[];                   // [kWnWarps][V]
  __shared__ float sm[kWnWarps], sl[kWnWarps];
  const int h = blockIdx.x, row = blockIdx.y, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G);
  const T* qr = static_cast<const T*>(p.q) + (static_cast<int64_t>(row) * p.H + h) * p.D;
  float q[RK], o[RV];
#pragma unroll
  for (int i = 0; i < RK; ++i) {
    const int c = i * 32 + lane;
    q[i] = c < p.D ? to_f<T>(qr[c]) * p.scale : 0.f;
  }
#pragma unroll
  for (int i = 0; i < RV; ++i) o[i] = 0.f;
  const int len = p.kv_len[row];
  const int32_t* bt = p.table + static_cast<int64_t>(p.seq_of ? p.seq_of[row] : row) * p.ld_table;
  const T* kp = static_cast<const T*>(p.k_pool);
  const T* vp = static_cast<const T*>(p.v_pool);
  float m = -INFINITY, l = 0.f;
  for (int j = w; j < len; j += kWnWarps) {
    const int64_t at = (static_cast<int64_t>(bt[j / 16]) * p.G + g) * 16 + j % 16;
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < RK; ++i) {
      const int c = i * 32 + lane;
      s += c < p.D ? q[i] * to_f<T>(kp[at * p.D + c]) : 0.f;
    }
    s = warp_sum(s);
    const float m2 = fmaxf(m, s), a = expf(m - m2), b = expf(s - m2);
    m = m2;
    l = l * a + b;
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      const int c = i * 32 + lane;
      o[i] = o[i] * a + b * (c < p.V ? to_f<T>(vp[at * p.V + c]) : 0.f);
    }
  }
  if (lane == 0) { sm[w] = m; sl[w] = l; }
#pragma unroll
  for (int i = 0; i < RV; ++i)
    if (i * 32 + lane < p.V) sh[w * p.V + i * 32 + lane] = o[i];
  __syncthreads();
  float mm = -INFINITY;
  for (int i = 0; i < kWnWarps; ++i) mm = fmaxf(mm, sm[i]);
  if (p.sink && len > 0) mm = fmaxf(mm, p.sink[h]);
  T* out = static_cast<T*>(p.out) + (static_cast<int64_t>(row) * p.H + h) * p.V;
  for (int c = threadIdx.x; c < p.V; c += kWnWarps * 32) {
    float acc = 0.f, ll = p.sink && len > 0 ? expf(p.sink[h] - mm) : 0.f;
    for (int i = 0; i < kWnWarps; ++i) {
      const float f = sm[i] == -INFINITY ? 0.f : expf(sm[i] - mm);
      acc += f * sh[i * p.V + c];
      ll += f * sl[i];
    }
    out[c] = from_f<T>(ll > 0.f ? acc / ll : 0.f);
  }
}

template <class T>
static int run_sink(const SinkParams& p, cudaStream_t st) {
  const dim3 grid(p.H, p.R);
  const int smem = kWnWarps * p.V * 4;            // at most 16 KB
  const int w = p.D > p.V ? p.D : p.V;
  if (w <= 64) mix_sink_row_kernel<T, 2, 2><<<grid, kWnWarps * 32, smem, st>>>(p);
  else if (w <= 128) mix_sink_row_kernel<T, 4, 4><<<grid, kWnWarps * 32, smem, st>>>(p);
  else mix_sink_row_kernel<T, 8, 16><<<grid, kWnWarps * 32, smem, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_sink(const SinkParams* p, int dtype, cudaStream_t st) {
  if (p->R <= 0) return 0;
  if (p->R > 65535 || p->D < 1 || p->D > 256 || p->V < 1 || p->V > 512 || p->G < 1 || p->H % p->G) return -251;
  return dtype == 0 ? run_sink<__nv_bfloat16>(*p, st) : run_sink<float>(*p, st);
}

extern "C" int prl_mix_window(const WindowParams* p, int dtype, cudaStream_t st) {
  if (p->R <= 0) return 0;
  if (p->R > 65535 || p->D > 1024 || p->D < 1 || p->G < 1 || p->H % p->G || p->window < 1) return -250;
  return dtype == 0 ? run_window<__nv_bfloat16>(*p, st) : run_window<float>(*p, st);
}
