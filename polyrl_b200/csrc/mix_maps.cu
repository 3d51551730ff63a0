// polyrl_b200 — differential attention beside the tensor-core kernels: rows (bias, norm per head and map, rotation, cache write) and
// paged attention of any width, bf16 or fp32.  The row kernels also serve attention with one map per head whose values are rotated like keys
// (outputs are turned back by mix_turn_back_kernel).
//
// A head has two softmax maps over the same values; the output is  (a1 - lambda a2) / sqrt(mean^2 + eps) * keep.  The cache holds
// [map 1 | map 2] keys of a head in one row.  bf16 rows of the padded widths take attn_fwd.cu (prompt portions) and decode_attn.cu
// (single tokens); both end in the same combination.
#include "mixers.cuh"

namespace prl {

__device__ __forceinline__ void map_angles(int64_t pos, const double* __restrict__ freq, int n, float* cs, float* sn) {
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    double a = static_cast<double>(pos) * freq[i];
    a -= 6.283185307179586 * rint(a * 0.15915494309189535);
    sincosf(static_cast<float>(a), &sn[i], &cs[i]);
  }
}

struct MapRows {
  const void* p;                // T [R, ldp]: [queries H x maps x dim | keys G x maps x dim | values G x V]
  int64_t ldp;
  const float *bias, *wq, *wk;  // wq, wk: null = ones
  const double *freq, *vfreq;   // [rd / 2], [V / 2] (null: values are not rotated)
  const int64_t *pos, *kvslot;
  void *q, *kp, *vp, *k_pool, *v_pool;      // q [R, maps * H, qw]; packed kp / vp may be null
  int H, G, D, V, rd, qw, kw, vw, maps;
  float eps;
};

// LANES lanes own a (head, map) vector, eight entries each: LANES * 8 >= kw, entries beyond D are zero; D, V, rd / 2 (V / 2 where values are
// rotated) multiples of 8
template <class T, int LANES>
__global__ void __launch_bounds__(256) mix_map_rows_kernel(MapRows a) {
  __shared__ float cs[256], sn[256], vcs[256], vsn[256];
  const int64_t t = blockIdx.x;
  const int n = a.rd / 2, nq = a.maps * a.H, nk = a.maps * a.G, lane = threadIdx.x % LANES;
  const T* row = static_cast<const T*>(a.p) + t * a.ldp;
  map_angles(a.pos[t], a.freq, n, cs, sn);
  if (a.vfreq) map_angles(a.pos[t], a.vfreq, a.V / 2, vcs, vsn);
  __syncthreads();
  const int64_t slot = a.kvslot[t], page = slot / 16, off = slot % 16;
  const int c = lane * 8;
  for (int v0 = 0; v0 < nq + nk; v0 += 256 / LANES) {              // uniform over the CTA: the shuffles below stay inside a vector
    const int v = v0 + threadIdx.x / LANES;
    const bool on = v < nq + nk, key = v >= nq, in = on && c < a.D;
    float y[8] = {};
    if (in) {
      float b[8];
      ld_vec<T, 8>(row + v * a.D + c, y);
      ld_vec<float, 8>(a.bias + v * a.D + c, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] += b[i];
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += y[i] * y[i];
#pragma unroll
    for (int o = LANES / 2; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float r = rsqrtf(ss / a.D + a.eps);
    if (in && a.wq) {
      float w[8];
      ld_vec<float, 8>((key ? a.wk : a.wq) + c, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] *= r * w[i];
    } else if (in) {
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] *= r;
    }
    const bool first = c < n, second = !first && c < 2 * n;        // the halves of the rotated part
    const int other = first ? lane + n / 8 : (second ? lane - n / 8 : lane);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float z = __shfl_sync(0xffffffffu, y[i], other, LANES);
      if (first) y[i] = y[i] * cs[c + i] - z * sn[c + i];
      else if (second) y[i] = y[i] * cs[c - n + i] + z * sn[c - n + i];
    }
    if (!on || c >= a.kw) continue;
    if (!key) {
      T* q = static_cast<T*>(a.q) + (t * nq + v) * a.qw;
      if (a.qw == a.kw) {
        st_vec<T, 8>(q + c, y);
      } else {                                                     // the map's half of a row that both maps share
        const float zero[8] = {};
        st_vec<T, 8>(q + (v & 1) * a.kw + c, y);
        st_vec<T, 8>(q + (1 - (v & 1)) * a.kw + c, zero);
      }
    } else {
      const int g = (v - nq) / a.maps, col = (v - nq) % a.maps * a.kw + c;
      st_vec<T, 8>(static_cast<T*>(a.k_pool) + ((page * a.G + g) * 16 + off) * a.maps * a.kw + col, y);
      if (a.kp) st_vec<T, 8>(static_cast<T*>(a.kp) + (t * a.G + g) * a.maps * a.kw + col, y);
    }
  }
  const int vu = a.vw / 8, v_at = (nq + nk) * a.D;
  for (int u = threadIdx.x; u < a.G * vu; u += 256) {
    const int g = u / vu, x = (u % vu) * 8;
    float y[8] = {};
    if (x < a.V) {
      float b[8];
      ld_vec<T, 8>(row + v_at + g * a.V + x, y);
      ld_vec<float, 8>(a.bias + v_at + g * a.V + x, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] += b[i];
      if (a.vfreq) {
        const int half = a.V / 2, m = x < half ? x : x - half;     // pair of the first entry; its other half lies half a row away
        const int o = v_at + g * a.V + (x < half ? x + half : m);
        float z[8];
        ld_vec<T, 8>(row + o, z);
        ld_vec<float, 8>(a.bias + o, b);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = y[i] * vcs[m + i] + (x < half ? -1.f : 1.f) * (z[i] + b[i]) * vsn[m + i];
      }
    }
    st_vec<T, 8>(static_cast<T*>(a.v_pool) + ((page * a.G + g) * 16 + off) * a.vw + x, y);
    if (a.vp) st_vec<T, 8>(static_cast<T*>(a.vp) + (t * a.G + g) * a.vw + x, y);
  }
}

// any sizes (D <= 256): a warp per vector
template <class T>
__global__ void __launch_bounds__(256) mix_map_rows_any_kernel(MapRows a) {
  __shared__ float cs[256], sn[256], vcs[256], vsn[256], buf[8][256];
  const int64_t t = blockIdx.x;
  const int n = a.rd / 2, nq = a.maps * a.H, nk = a.maps * a.G, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* row = static_cast<const T*>(a.p) + t * a.ldp;
  map_angles(a.pos[t], a.freq, n, cs, sn);
  if (a.vfreq) map_angles(a.pos[t], a.vfreq, a.V / 2, vcs, vsn);
  __syncthreads();
  const int64_t slot = a.kvslot[t], page = slot / 16, off = slot % 16;
  float* y = buf[warp];
  for (int v = warp; v < nq + nk; v += 8) {
    const bool key = v >= nq;
    const float* w = key ? a.wk : a.wq;
    float ss = 0.f;
    for (int c = lane; c < a.D; c += 32) {
      y[c] = to_f<T>(row[v * a.D + c]) + a.bias[v * a.D + c];
      ss += y[c] * y[c];
    }
    const float r = rsqrtf(warp_sum(ss) / a.D + a.eps);
    __syncwarp();
    const int g = (v - nq) / a.maps, m = key ? (v - nq) % a.maps : v % a.maps;
    auto weight = [&](int c) { return w ? w[c] : 1.f; };
    T* q = static_cast<T*>(a.q) + (t * nq + v) * a.qw;
    for (int c = lane; c < a.kw; c += 32) {
      float z = 0.f;
      if (c < a.D) {
        z = y[c] * r * weight(c);
        if (c < n) z = z * cs[c] - y[c + n] * r * weight(c + n) * sn[c];
        else if (c < 2 * n) z = z * cs[c - n] + y[c - n] * r * weight(c - n) * sn[c - n];
      }
      if (!key) {
        if (a.qw == a.kw) {
          q[c] = from_f<T>(z);
        } else {
          q[m * a.kw + c] = from_f<T>(z);
          q[(1 - m) * a.kw + c] = from_f<T>(0.f);
        }
      } else {
        const int col = m * a.kw + c;
        static_cast<T*>(a.k_pool)[((page * a.G + g) * 16 + off) * a.maps * a.kw + col] = from_f<T>(z);
        if (a.kp) static_cast<T*>(a.kp)[(t * a.G + g) * a.maps * a.kw + col] = from_f<T>(z);
      }
    }
    __syncwarp();
  }
  const int v_at = (nq + nk) * a.D;
  for (int u = threadIdx.x; u < a.G * a.vw; u += 256) {
    const int g = u / a.vw, x = u % a.vw;
    auto value = [&](int c) { return to_f<T>(row[v_at + g * a.V + c]) + a.bias[v_at + g * a.V + c]; };
    float f = x < a.V ? value(x) : 0.f;
    if (a.vfreq && x < a.V) {
      const int half = a.V / 2, i = x < half ? x : x - half;
      f = f * vcs[i] + (x < half ? -value(x + half) : value(i)) * vsn[i];
    }
    const T z = from_f<T>(f);
    static_cast<T*>(a.v_pool)[((page * a.G + g) * 16 + off) * a.vw + x] = z;
    if (a.vp) static_cast<T*>(a.vp)[(t * a.G + g) * a.vw + x] = z;
  }
}

// o [R, H, vw]: entries (m, m + V / 2) of every head turned by -pos * vfreq[m], times scale * sigmoid(gate) -> out [R, H * V]
template <class T, int VEC>
__global__ void __launch_bounds__(256) mix_turn_back_kernel(const T* __restrict__ o, const T* __restrict__ gate, int64_t ldg, const double* __restrict__ vfreq,
                                                            const int64_t* __restrict__ pos, float scale, T* __restrict__ out, int64_t ldo, int H, int V, int vw) {
  __shared__ float cs[256], sn[256];
  const int64_t t = blockIdx.x;
  const int half = V / 2, units = half / VEC;
  map_angles(pos[t], vfreq, half, cs, sn);
  __syncthreads();
  for (int e = threadIdx.x; e < H * units; e += 256) {
    const int h = e / units, m = (e % units) * VEC;
    const T* src = o + (t * H + h) * vw + m;
    float u[VEC], v[VEC], g[VEC], f[VEC];
    ld_vec<T, VEC>(src, u);
    ld_vec<T, VEC>(src + half, v);
    ld_vec<T, VEC>(gate + t * ldg + h * V + m, g);
    ld_vec<T, VEC>(gate + t * ldg + h * V + half + m, f);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float c = cs[m + i], s = sn[m + i], a = u[i], b = v[i];
      u[i] = (a * c + b * s) * (scale * sigmoid_t<T>(g[i]));
      v[i] = (b * c - a * s) * (scale * sigmoid_t<T>(f[i]));
    }
    st_vec<T, VEC>(out + t * ldo + h * V + m, u);
    st_vec<T, VEC>(out + t * ldo + h * V + half + m, v);
  }
}

// one CTA per (head, row): a key per warp and step for both maps, fp32 throughout; RK >= D / 32, RV >= V / 32
constexpr int kMpWarps = 8;
template <class T, int RK, int RV>
__global__ void __launch_bounds__(kMpWarps * 32) mix_map_attention_kernel(MapParams p) {
  extern __shared__ float sh[];                   // [2][kMpWarps][V]
  __shared__ float sm[2][kMpWarps], sl[2][kMpWarps], red[kMpWarps];
  const int h = blockIdx.x, row = blockIdx.y, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = h / (p.H / p.G);
  const T* qr = static_cast<const T*>(p.q) + (static_cast<int64_t>(row) * p.H + h) * 2 * p.qw;
  float q[2][RK], o[2][RV], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int k = 0; k < 2; ++k) {
#pragma unroll
    for (int i = 0; i < RK; ++i) {
      const int c = i * 32 + lane;
      q[k][i] = c < p.D ? to_f<T>(qr[k * p.qw + k * (p.qw - p.kw) + c]) * p.scale : 0.f;
    }
#pragma unroll
    for (int i = 0; i < RV; ++i) o[k][i] = 0.f;
  }
  const int len = p.kv_len[row];
  const int32_t* bt = p.table + static_cast<int64_t>(p.seq_of ? p.seq_of[row] : row) * p.ld_table;
  const T* kp = static_cast<const T*>(p.k_pool);
  const T* vp = static_cast<const T*>(p.v_pool);
  for (int j = max(0, len - p.window) + w; j < len; j += kMpWarps) {
    const int64_t at = (static_cast<int64_t>(bt[j / 16]) * p.G + g) * 16 + j % 16;
    float v[RV];
#pragma unroll
    for (int i = 0; i < RV; ++i) {
      const int c = i * 32 + lane;
      v[i] = c < p.V ? to_f<T>(vp[at * p.vw + c]) : 0.f;
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < RK; ++i) {
        const int c = i * 32 + lane;
        s += c < p.D ? q[k][i] * to_f<T>(kp[(at * 2 + k) * p.kw + c]) : 0.f;
      }
      s = warp_sum(s);
      const float m2 = fmaxf(m[k], s), a = expf(m[k] - m2), b = expf(s - m2);
      m[k] = m2;
      l[k] = l[k] * a + b;
#pragma unroll
      for (int i = 0; i < RV; ++i) o[k][i] = o[k][i] * a + b * v[i];
    }
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    if (lane == 0) { sm[k][w] = m[k]; sl[k][w] = l[k]; }
#pragma unroll
    for (int i = 0; i < RV; ++i)
      if (i * 32 + lane < p.V) sh[(k * kMpWarps + w) * p.V + i * 32 + lane] = o[k][i];
  }
  __syncthreads();
  const float lam = p.lam[0];
  float y[2], ss = 0.f;                           // V <= 512: at most two values per thread
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int c = threadIdx.x + e * kMpWarps * 32;
    y[e] = 0.f;
    if (c < p.V) {
      float a[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        float mm = -INFINITY, acc = 0.f, ll = 0.f;
        for (int i = 0; i < kMpWarps; ++i) mm = fmaxf(mm, sm[k][i]);
        for (int i = 0; i < kMpWarps; ++i) {
          const float f = sm[k][i] == -INFINITY ? 0.f : expf(sm[k][i] - mm);
          acc += f * sh[(k * kMpWarps + i) * p.V + c];
          ll += f * sl[k][i];
        }
        a[k] = ll > 0.f ? acc / ll : 0.f;
      }
      y[e] = a[0] - lam * a[1];
      ss += y[e] * y[e];
    }
  }
  const float f = rsqrtf(block_sum<kMpWarps>(ss, red) / p.V + p.eps) * p.keep;
  T* out = static_cast<T*>(p.out) + (static_cast<int64_t>(row) * p.H + h) * p.V;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int c = threadIdx.x + e * kMpWarps * 32;
    if (c < p.V) out[c] = from_f<T>(y[e] * f);
  }
}

template <class T>
static int run_maps(const MapParams& p, cudaStream_t st) {
  const dim3 grid(p.H, p.R);
  const int smem = 2 * kMpWarps * p.V * 4;        // at most 32 KB
  if (p.D <= 32 && p.V <= 64) mix_map_attention_kernel<T, 1, 2><<<grid, kMpWarps * 32, smem, st>>>(p);
  else if (p.D <= 64 && p.V <= 128) mix_map_attention_kernel<T, 2, 4><<<grid, kMpWarps * 32, smem, st>>>(p);
  else if (p.D <= 128 && p.V <= 256) mix_map_attention_kernel<T, 4, 8><<<grid, kMpWarps * 32, smem, st>>>(p);
  else mix_map_attention_kernel<T, 8, 16><<<grid, kMpWarps * 32, smem, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

template <class T>
static int run_rows(const MapRows& a, int rows, cudaStream_t st) {
  bool vec = a.D % 8 == 0 && a.V % (a.vfreq ? 16 : 8) == 0 && a.vw % 8 == 0 && a.rd % 16 == 0 && a.ldp % 8 == 0;
  for (const void* q : {a.p, static_cast<const void*>(a.bias), static_cast<const void*>(a.wq), static_cast<const void*>(a.wk), static_cast<const void*>(a.q),
                        static_cast<const void*>(a.kp), static_cast<const void*>(a.vp), static_cast<const void*>(a.k_pool), static_cast<const void*>(a.v_pool)})
    vec = vec && al16(q);
  if (vec && a.kw == 32) mix_map_rows_kernel<T, 4><<<rows, 256, 0, st>>>(a);
  else if (vec && a.kw == 64) mix_map_rows_kernel<T, 8><<<rows, 256, 0, st>>>(a);
  else if (vec && a.kw == 128) mix_map_rows_kernel<T, 16><<<rows, 256, 0, st>>>(a);
  else if (vec && a.kw == 192) mix_map_rows_kernel<T, 32><<<rows, 256, 0, st>>>(a);
  else mix_map_rows_any_kernel<T><<<rows, 256, 0, st>>>(a);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_map_rows(const void* p, int64_t ldp, const float* bias, const float* wq, const float* wk, const double* freq, const int64_t* pos,
                                const int64_t* kvslot, void* q, void* kp, void* vp, void* k_pool, void* v_pool, int rows, int H, int G, int D, int V, int rd,
                                int qw, int kw, int vw, float eps, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (D < 1 || D > 256 || rd > D || rd % 2 || kw < D || vw < V || H % G || (qw != kw && qw != 2 * kw)) return -280;
  const MapRows a{p, ldp, bias, wq, wk, freq, nullptr, pos, kvslot, q, kp, vp, k_pool, v_pool, H, G, D, V, rd, qw, kw, vw, 2, eps};
  return dtype == 0 ? run_rows<__nv_bfloat16>(a, rows, st) : run_rows<float>(a, rows, st);
}

// one map per head, norms without weights, values rotated over all of V
extern "C" int prl_mix_turn_rows(const void* p, int64_t ldp, const float* bias, const double* freq, const double* vfreq, const int64_t* pos,
                                 const int64_t* kvslot, void* q, void* kp, void* vp, void* k_pool, void* v_pool, int rows, int H, int G, int D, int V, int rd, int kw,
                                 int vw, float eps, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (D < 1 || D > 256 || V < 2 || V > 512 || V % 2 || rd > D || rd % 2 || kw < D || vw < V || H % G) return -282;
  const MapRows a{p, ldp, bias, nullptr, nullptr, freq, vfreq, pos, kvslot, q, kp, vp, k_pool, v_pool, H, G, D, V, rd, kw, kw, vw, 1, eps};
  return dtype == 0 ? run_rows<__nv_bfloat16>(a, rows, st) : run_rows<float>(a, rows, st);
}

extern "C" int prl_mix_turn_back(const void* o, const void* gate, int64_t ldg, const double* vfreq, const int64_t* pos, float scale, void* out, int64_t ldo,
                                 int rows, int H, int V, int vw, int dtype, cudaStream_t st) {
  if (rows <= 0) return 0;
  if (V < 2 || V > 512 || V % 2 || vw < V) return -283;
  const bool vec = V % 16 == 0 && vw % 8 == 0 && ldg % 8 == 0 && ldo % 8 == 0 && al16(o) && al16(gate) && al16(out);
  MIX_DISPATCH(vec, (mix_turn_back_kernel<T, VEC><<<rows, 256, 0, st>>>(static_cast<const T*>(o), static_cast<const T*>(gate), ldg, vfreq, pos, scale,
                                                                       static_cast<T*>(out), ldo, H, V, vw)));
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

extern "C" int prl_mix_map_attention(const MapParams* p, int dtype, cudaStream_t st) {
  if (p->R <= 0) return 0;
  if (p->R > 65535 || p->D < 1 || p->D > 256 || p->V < 1 || p->V > 512 || p->G < 1 || p->H % p->G || p->window < 1) return -281;
  return dtype == 0 ? run_maps<__nv_bfloat16>(*p, st) : run_maps<float>(*p, st);
}
