// polyrl_b200 — paged latent attention in the absorbed (multi-query) form, with an optional per-head sink.
//
// The cache holds ONE row per token and layer: [latent r | rotated shared key rd].  Query row (t, head) is
// [q_lat r | q_rot rd] (key up-projection folded into q_lat), so   score = q . row * scale,   out = softmax . row[:r],
// where the sink adds exp(sink_h) to the softmax denominator and nothing else.
//   * mix_latent_tc_kernel   decode: 16 or 32 heads x 32 keys per step on the tensor cores, cp.async double buffering
//                            over pages, split over the keys with a merge kernel
//   * mix_latent_row_kernel  any size, bf16 or fp32: one CTA per (row, head), fp32 throughout
#include "mixers.cuh"

namespace prl {

constexpr int kLtPage = 16;
constexpr int kLtKeys = 32;
constexpr int kLtWarps = 4;

// ------------------------------------------------------------------------------------------ any size
template <class T, int RN>
__global__ void __launch_bounds__(kLtWarps * 32) mix_latent_row_kernel(LatentParams p) {
  extern __shared__ float sh[];
  const int D = p.r + p.rd;
  float* sq = sh;                                 // [D]
  float* so = sh + D;                             // [kLtWarps][r]
  __shared__ float sm[kLtWarps], sl[kLtWarps];
  const int h = blockIdx.x, row = blockIdx.y, w = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* ql = static_cast<const T*>(p.q_lat) + (static_cast<int64_t>(h) * p.R + row) * p.r;
  const T* qr = static_cast<const T*>(p.q) + row * p.ldq + static_cast<int64_t>(h) * p.dq + p.d;
  for (int i = threadIdx.x; i < D; i += kLtWarps * 32) sq[i] = (i < p.r ? to_f<T>(ql[i]) : to_f<T>(qr[i - p.r])) * p.scale;
  __syncthreads();
  const int len = p.kv_len[row];
  const int32_t* bt = p.table + static_cast<int64_t>(p.seq_of ? p.seq_of[row] : row) * p.ld_table;
  const T* pool = static_cast<const T*>(p.pool);
  float m = -INFINITY, l = 0.f, o[RN];
#pragma unroll
  for (int i = 0; i < RN; ++i) o[i] = 0.f;
  for (int j = w; j < len; j += kLtWarps) {
    const T* kr = pool + (static_cast<int64_t>(bt[j / kLtPage]) * kLtPage + j % kLtPage) * D;
    float kv[RN], dot = 0.f;
#pragma unroll
    for (int i = 0; i < RN; ++i) {
      const int c = i * 32 + lane;
      kv[i] = c < p.r ? to_f<T>(kr[c]) : 0.f;
      if (c < p.r) dot += sq[c] * kv[i];
    }
    for (int c = p.r + lane; c < D; c += 32) dot += sq[c] * to_f<T>(kr[c]);
    dot = warp_sum(dot);
    const float m2 = fmaxf(m, dot);
    const float a = expf(m - m2), e = expf(dot - m2);
    l = l * a + e;
#pragma unroll
    for (int i = 0; i < RN; ++i) o[i] = o[i] * a + e * kv[i];
    m = m2;
  }
  if (lane == 0) { sm[w] = m; sl[w] = l; }
#pragma unroll
  for (int i = 0; i < RN; ++i)
    if (i * 32 + lane < p.r) so[w * p.r + i * 32 + lane] = o[i];
  __syncthreads();
  float mm = p.sink ? p.sink[h] : -INFINITY;
#pragma unroll
  for (int i = 0; i < kLtWarps; ++i) mm = fmaxf(mm, sm[i]);
  float ll = p.sink ? expf(p.sink[h] - mm) : 0.f, f[kLtWarps];
#pragma unroll
  for (int i = 0; i < kLtWarps; ++i) {
    f[i] = sm[i] == -INFINITY ? 0.f : expf(sm[i] - mm);
    ll += sl[i] * f[i];
  }
  const float inv = ll > 0.f ? 1.f / ll : 0.f;
  T* out = static_cast<T*>(p.out) + (static_cast<int64_t>(h) * p.R + row) * p.r;
  for (int c = threadIdx.x; c < p.r; c += kLtWarps * 32) {
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < kLtWarps; ++i) acc += so[i * p.r + c] * f[i];
    out[c] = from_f<T>(acc * inv);
  }
}

// ------------------------------------------------------------------------------------------ decode, bf16
__device__ __forceinline__ void lt_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lt_ldsm(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void lt_ldsm_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}

// MT row tiles of 16 heads per CTA, 4 * MT warps: warp w scores keys [8 (w % 4), +8) for row tile w / 4 and owns NTW output column
// tiles (8 wide) of every row tile.  r <= 32 * MT * NTW, r a multiple of 16, r + rd a multiple of 8.
template <int NTW, int MT>
__global__ void __launch_bounds__(128 * MT) mix_latent_tc_kernel(LatentParams p) {
  constexpr int NW = 4 * MT, HT = 16 * MT;
  extern __shared__ __align__(128) uint8_t raw[];
  const int D = p.r + p.rd, Dp = (D + 31) / 32 * 32, LD = Dp + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(raw);       // [HT][LD]
  __nv_bfloat16* sK = sQ + HT * LD;                                // [2][32][LD]
  __nv_bfloat16* sP = sK + 2 * kLtKeys * LD;                       // [HT][40]
  __shared__ float s_m[4][HT], s_l[4][HT];
  const int h0 = blockIdx.x * HT, row = blockIdx.y, split = blockIdx.z;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31, gq = lane >> 2, qd = lane & 3;
  const int wn = w & 3, wm = w >> 2;
  const int hn = min(HT, p.H - h0);
  const int len = p.kv_len[row];
  const int tiles = (len + kLtKeys - 1) / kLtKeys, per = (tiles + p.splits - 1) / p.splits;
  const int tb = split * per, te = min(tiles, tb + per);
  const int32_t* bt = p.table + static_cast<int64_t>(p.seq_of ? p.seq_of[row] : row) * p.ld_table;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(p.pool);

  // rows w, w + NW, ... of a tile per warp: one page number for each, neighbouring lanes on neighbouring 16-byte pieces
  int64_t src[kLtKeys / NW];
  auto pages = [&](int tile) {
#pragma unroll
    for (int i = 0; i < kLtKeys / NW; ++i) {
      const int key = tile * kLtKeys + w + i * NW;
      src[i] = key < len ? (static_cast<int64_t>(bt[key / kLtPage]) * kLtPage + key % kLtPage) * D : -1;
    }
  };
  auto load = [&](int buf) {
#pragma unroll
    for (int i = 0; i < kLtKeys / NW; ++i) {
      __nv_bfloat16* dst = sK + (buf * kLtKeys + w + i * NW) * LD;
      for (int c = lane * 8; c < Dp; c += 256) {
        const bool ok = src[i] >= 0 && c < D;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + c)), "l"(pool + (ok ? src[i] + c : 0)), "r"(ok ? 16 : 0) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (tb < te) {
    pages(tb);
    load(0);
    if (tb + 1 < te) pages(tb + 1);
  }
  for (int h = w; h < HT; h += NW) {
    for (int c = lane; c < Dp; c += 32) {
      __nv_bfloat16 v = __float2bfloat16(0.f);
      if (h < hn && c < D)
        v = c < p.r ? static_cast<const __nv_bfloat16*>(p.q_lat)[(static_cast<int64_t>(h0 + h) * p.R + row) * p.r + c]
                    : static_cast<const __nv_bfloat16*>(p.q)[row * p.ldq + static_cast<int64_t>(h0 + h) * p.dq + p.d + c - p.r];
      sQ[h * LD + c] = v;
    }
  }
  float o[MT][NTW][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int i = 0; i < NTW; ++i) o[a][i][0] = o[a][i][1] = o[a][i][2] = o[a][i][3] = 0.f;
  float m[MT][2], l0 = 0.f, l1 = 0.f;                              // maxima of every row pair; sums of this warp's own row tile and keys
#pragma unroll
  for (int a = 0; a < MT; ++a) m[a][0] = m[a][1] = -INFINITY;
  for (int t = tb; t < te; ++t) {
    const int buf = (t - tb) & 1;
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                                               // tile t is in; everyone is done with the other buffer
    if (t + 1 < te) {
      load(buf ^ 1);
      if (t + 2 < te) pages(t + 2);
    }
    const __nv_bfloat16* kt = sK + buf * kLtKeys * LD;
    float sa[4] = {0.f, 0.f, 0.f, 0.f}, sb[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 3
    for (int k = 0; k < Dp; k += 32) {
      uint32_t a[4], b[4];
      lt_ldsm(b, &kt[(wn * 8 + (lane & 7)) * LD + k + (lane >> 3) * 8]);
      lt_ldsm(a, &sQ[(wm * 16 + (lane & 15)) * LD + k + (lane >> 4) * 8]);
      lt_mma(sa, a, b[0], b[1]);
      lt_ldsm(a, &sQ[(wm * 16 + (lane & 15)) * LD + k + 16 + (lane >> 4) * 8]);
      lt_mma(sb, a, b[2], b[3]);
    }
    float x[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = t * kLtKeys + wn * 8 + 2 * qd + (e & 1);
      x[e] = key < len ? (sa[e] + sb[e]) * p.scale : -INFINITY;
    }
    float c0 = fmaxf(x[0], x[1]), c1 = fmaxf(x[2], x[3]);
    c0 = fmaxf(c0, __shfl_xor_sync(0xffffffffu, c0, 1));
    c0 = fmaxf(c0, __shfl_xor_sync(0xffffffffu, c0, 2));
    c1 = fmaxf(c1, __shfl_xor_sync(0xffffffffu, c1, 1));
    c1 = fmaxf(c1, __shfl_xor_sync(0xffffffffu, c1, 2));
    if (qd == 0) { s_m[wn][wm * 16 + gq] = c0; s_m[wn][wm * 16 + gq + 8] = c1; }
    __syncthreads();
    float own0 = 0.f, own1 = 0.f, al0 = 1.f, al1 = 1.f;            // this warp's row tile
#pragma unroll
    for (int a = 0; a < MT; ++a) {
      float n0 = m[a][0], n1 = m[a][1];
#pragma unroll
      for (int i = 0; i < 4; ++i) { n0 = fmaxf(n0, s_m[i][a * 16 + gq]); n1 = fmaxf(n1, s_m[i][a * 16 + gq + 8]); }
      const float a0 = __expf(m[a][0] - n0), a1 = __expf(m[a][1] - n1);        // n is finite: a tile holds at least one key
      m[a][0] = n0; m[a][1] = n1;
      if (a == wm) { own0 = n0; own1 = n1; al0 = a0; al1 = a1; }
#pragma unroll
      for (int i = 0; i < NTW; ++i) { o[a][i][0] *= a0; o[a][i][1] *= a0; o[a][i][2] *= a1; o[a][i][3] *= a1; }
    }
    const float p0 = __expf(x[0] - own0), p1 = __expf(x[1] - own0), p2 = __expf(x[2] - own1), p3 = __expf(x[3] - own1);
    l0 = l0 * al0 + p0 + p1;
    l1 = l1 * al1 + p2 + p3;
    *reinterpret_cast<uint32_t*>(&sP[(wm * 16 + gq) * 40 + wn * 8 + 2 * qd]) = pack_bf16(p0, p1);
    *reinterpret_cast<uint32_t*>(&sP[(wm * 16 + gq + 8) * 40 + wn * 8 + 2 * qd]) = pack_bf16(p2, p3);
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kLtKeys; k += 16) {
      uint32_t a[MT][4], b[4];
#pragma unroll
      for (int i = 0; i < MT; ++i) lt_ldsm(a[i], &sP[(i * 16 + (lane & 15)) * 40 + k + (lane >> 4) * 8]);
#pragma unroll
      for (int i = 0; i < NTW; i += 2) {
        const int col = (w * NTW + i) * 8;
        if (col < p.r) {
          lt_ldsm_t(b, &kt[(k + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + col + (lane >> 4) * 8]);
#pragma unroll
          for (int j = 0; j < MT; ++j) {
            lt_mma(o[j][i], a[j], b[0], b[1]);
            lt_mma(o[j][i + 1], a[j], b[2], b[3]);
          }
        }
      }
    }
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if (qd == 0) { s_l[wn][wm * 16 + gq] = l0; s_l[wn][wm * 16 + gq + 8] = l1; }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2 * MT; ++e) {
    const int hr = gq + 8 * e, h = h0 + hr;
    if (hr >= hn) continue;
    const float l = s_l[0][hr] + s_l[1][hr] + s_l[2][hr] + s_l[3][hr], mx = m[e >> 1][e & 1];
    const int64_t base = static_cast<int64_t>(h) * p.R + row;
    if (p.splits == 1) {
      const float snk = p.sink ? p.sink[h] : -INFINITY, mm = fmaxf(mx, snk);
      const float f = mx == -INFINITY ? 0.f : expf(mx - mm);
      const float den = l * f + (p.sink ? expf(snk - mm) : 0.f), g = den > 0.f ? f / den : 0.f;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + base * p.r;
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        const int c = (w * NTW + i) * 8 + 2 * qd;
        if (c < p.r) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[e >> 1][i][2 * (e & 1)] * g, o[e >> 1][i][2 * (e & 1) + 1] * g);
      }
    } else {
      float* dst = p.part + (base * p.splits + split) * p.r;
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        const int c = (w * NTW + i) * 8 + 2 * qd;
        if (c < p.r) *reinterpret_cast<float2*>(dst + c) = make_float2(o[e >> 1][i][2 * (e & 1)], o[e >> 1][i][2 * (e & 1) + 1]);
      }
      if (w == 0 && qd == 0) {
        float* ml = p.part + static_cast<int64_t>(p.H) * p.R * p.splits * p.r + (base * p.splits + split) * 2;
        ml[0] = mx;
        ml[1] = l;
      }
    }
  }
}

__global__ void __launch_bounds__(128) mix_latent_merge_kernel(LatentParams p) {
  const int h = blockIdx.x, row = blockIdx.y;
  const int64_t base = static_cast<int64_t>(h) * p.R + row;
  const float* ml = p.part + static_cast<int64_t>(p.H) * p.R * p.splits * p.r + base * p.splits * 2;
  float mm = p.sink ? p.sink[h] : -INFINITY;
  for (int s = 0; s < p.splits; ++s) mm = fmaxf(mm, ml[2 * s]);
  float den = p.sink ? expf(p.sink[h] - mm) : 0.f;
  for (int s = 0; s < p.splits; ++s) den += ml[2 * s] == -INFINITY ? 0.f : ml[2 * s + 1] * expf(ml[2 * s] - mm);
  const float inv = den > 0.f ? 1.f / den : 0.f;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + base * p.r;
  for (int c = threadIdx.x; c < p.r; c += 128) {
    float acc = 0.f;
    for (int s = 0; s < p.splits; ++s)
      if (ml[2 * s] != -INFINITY) acc += p.part[(base * p.splits + s) * p.r + c] * expf(ml[2 * s] - mm);
    dst[c] = __float2bfloat16(acc * inv);
  }
}

template <int NTW, int MT>
static int run_tc(const LatentParams& p, cudaStream_t st) {
  const int LD = (p.r + p.rd + 31) / 32 * 32 + 8;
  const int smem = (16 * MT + 2 * kLtKeys) * LD * 2 + 16 * MT * 40 * 2;
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_latent_tc_kernel<NTW, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024));
    attr = true;
  }
  if (smem > 160 * 1024) return -232;
  mix_latent_tc_kernel<NTW, MT><<<dim3((p.H + 16 * MT - 1) / (16 * MT), p.R, p.splits), 128 * MT, smem, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  if (p.splits > 1) {
    mix_latent_merge_kernel<<<dim3(p.H, p.R), 128, 0, st>>>(p);
    PRL_CUDA_CHECK(cudaGetLastError());
  }
  return 0;
}
template <class T, int RN>
static int run_row(const LatentParams& p, cudaStream_t st) {
  const int smem = (p.r + p.rd + kLtWarps * p.r) * 4;
  if (smem > 48 * 1024) return -233;
  mix_latent_row_kernel<T, RN><<<dim3(p.H, p.R), kLtWarps * 32, smem, st>>>(p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}
template <class T>
static int pick_row(const LatentParams& p, cudaStream_t st) {
  if (p.r <= 64) return run_row<T, 2>(p, st);
  if (p.r <= 128) return run_row<T, 4>(p, st);
  if (p.r <= 256) return run_row<T, 8>(p, st);
  if (p.r <= 512) return run_row<T, 16>(p, st);
  if (p.r <= 1024) return run_row<T, 32>(p, st);
  return -234;
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_latent_tc_ok(int r, int rd) { return r % 16 == 0 && r <= 512 && (r + rd) % 8 == 0 && rd <= 128; }

// tc: use the tensor-core kernel (bf16, sizes accepted by prl_mix_latent_tc_ok); otherwise one CTA per (row, head)
extern "C" int prl_mix_latent(const LatentParams* p, int tc, int dtype, cudaStream_t st) {
  if (p->R <= 0) return 0;
  if (p->R > 65535 || p->splits < 1 || p->splits > 65535) return -230;
  if (!tc) return dtype == 0 ? pick_row<__nv_bfloat16>(*p, st) : pick_row<float>(*p, st);
  if (dtype != 0 || !prl_mix_latent_tc_ok(p->r, p->rd)) return -231;
  if (p->H > 16) {                  // two row tiles share every key load
    if (p->r <= 128) return run_tc<2, 2>(*p, st);
    if (p->r <= 256) return run_tc<4, 2>(*p, st);
    return run_tc<8, 2>(*p, st);
  }
  if (p->r <= 64) return run_tc<2, 1>(*p, st);
  if (p->r <= 128) return run_tc<4, 1>(*p, st);
  if (p->r <= 256) return run_tc<8, 1>(*p, st);
  return run_tc<16, 1>(*p, st);
}
