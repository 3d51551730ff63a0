// polyrl_b200 — gated delta rule over prompt portions on tcgen05 / TMEM (bf16 activations, 64 tokens per chunk).
//
// The recurrence is kDelta of mix_scan.cu.  With L_t the running sum of log keep inside a chunk, S_0 the state ahead of it and k', q' the
// unit vectors, the writes u_t of the chunk solve a unit lower triangular system:
//     u_t + sum_{s < t} A_ts u_s = r_t,     A_ts = beta_t e^(L_t - L_s) k'_t . k'_s,     r_t = beta_t (v_t - e^(L_t) S_0^T k'_t)
//     y_t = e^(L_t) S_0^T q'_t + sum_{s <= t} P_ts u_s,                                   P_ts = e^(L_t - L_s) q'_t . k'_s
//     S   = e^(L_C) S_0 + sum_s e^(L_C - L_s) k'_s u_s^T
// All exponents are <= 0.  The norms enter as fp32 factors of rows and columns, so q and k stay the bf16 operands they are.
//
// mix_delta_prep_kernel   one CTA per (chunk, key head), everything that does not depend on the state: the scores of [Q; K] against K in one
//                         128 x 64 product, then per value head T = (I + A)^-1 diag(beta) by forward substitution in fp32 (thread = column)
//                         and P.  T and P go to the workspace as bf16 pairs hi + lo, laid out as the swizzled tiles the next kernel copies.
// mix_delta_chunk_kernel  one CTA per (span, head, 128 value columns) marching over its chunks, all products transposed so that the value
//                         columns are the 128 rows (TMEM lane = value column) and the tokens or state rows the columns:
//                             carried = S_0^T [K | Q]^T     U^T = R^T T^T     own = U^T P^T     delta = (weighted U)^T K
//                         The fp32 state lives in registers, thread (value column, half) owning half of the state rows, and is restaged as the
//                         hi + lo operand once per chunk.  A chunk's outputs are written while the next chunk's first product runs.
// Operands that are not bf16 by nature (S, R, U, T, P) enter the products as bf16 pairs hi + lo.
// Every wait is bounded: on a timeout the CTA raises *err, stops computing, frees its TMEM and returns.
#include "mix_tc.cuh"

namespace prl {

constexpr int kDc = 64;                        // tokens per chunk
constexpr int kDcTile = 64 * 128;              // bytes of a 64 x 64 bf16 tile
constexpr int kDcWork = 4 * kDcTile;           // workspace of one (chunk, head): T hi, T lo, P hi, P lo
constexpr int kDcGates = 3 * kDc + 4;          // floats: carry of a key row, weight in the final state, carry of a query row, keep
constexpr int kDpThreads = 128, kDcThreads = 256;
constexpr int kDpLd = 68;                      // row pitch of A in floats

__device__ __forceinline__ int delta_chunk_base(const int32_t* cu, int s) { return cu[s] / kDc + s; }     // workspace rows of a span start here

// column c of (I + A)^-1, rows S0.. (rows above are zero): x_t = [t == c] - sum_{s < t} A_ts x_s
template <int S0>
__device__ __forceinline__ void delta_solve(const float* A, int c, float (&x)[kDc]) {
#pragma unroll
  for (int t = 0; t < kDc; ++t) {
    if (t < S0) { x[t] = 0.f; continue; }
    float a0 = t == c ? 1.f : 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
#pragma unroll
    for (int s = S0; s < t; s += 4) {                                  // (A is zero on and above the diagonal)
      const float4 a = *reinterpret_cast<const float4*>(A + t * kDpLd + s);
      a0 -= a.x * x[s];
      if (s + 1 < t) a1 -= a.y * x[s + 1];
      if (s + 2 < t) a2 -= a.z * x[s + 2];
      if (s + 3 < t) a3 -= a.w * x[s + 3];
    }
    x[t] = (a0 + a1) + (a2 + a3);
  }
}

template <int NB>
__global__ void __launch_bounds__(kDpThreads) mix_delta_prep_kernel(ScanParams p, uint8_t* work, float* gates, int32_t* err) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* tile = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));   // NB chunks of [64 Q rows; 64 K rows]
  float* sA = reinterpret_cast<float*>(tile + NB * 2 * kDcTile);       // [2][64][kDpLd]
  __shared__ float s_L[2][kDc], s_beta[2][kDc], s_rq[kDc], s_rk[kDc];
  __shared__ int s_span;
  __shared__ uint64_t bar;
  __shared__ uint32_t s_tmem;
  const int b = blockIdx.x, kh = blockIdx.y, r = threadIdx.x, w = r >> 5, lane = r & 31;
  if (r == 0) {                                                        // the span whose workspace rows hold b
    int lo = 0, hi = p.spans - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (delta_chunk_base(p.cu, mid) <= b) lo = mid; else hi = mid - 1;
    }
    s_span = lo;
    mbar_init(&bar, 1);
    fence_barrier_init();
  }
  __syncthreads();
  const int s = s_span, c0 = (b - delta_chunk_base(p.cu, s)) * kDc, nv = min(kDc, p.cu[s + 1] - p.cu[s] - c0);
  if (nv <= 0) return;
  const int64_t t0 = p.cu[s] + c0;
  const int N = p.N;
  {
    const __nv_bfloat16* gQ = static_cast<const __nv_bfloat16*>(p.q) + t0 * p.ldq + static_cast<int64_t>(kh) * N;
    const __nv_bfloat16* gK = static_cast<const __nv_bfloat16*>(p.k) + t0 * p.ldk + static_cast<int64_t>(kh) * N;
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      tc_load_rows<kDc, kDpThreads>(tile + i * 2 * kDcTile, gQ, p.ldq, nv, i * 64, N);
      tc_load_rows<kDc, kDpThreads>(tile + i * 2 * kDcTile + kDcTile, gK, p.ldk, nv, i * 64, N);
    }
    tc_cp_commit();
  }
  if (w == 0) { tmem_alloc(&s_tmem, 64); tmem_relinquish(); }
  tc_cp_wait<0>();
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s_tmem;
  if (r == 0) {
    constexpr uint32_t id = umma_idesc(128, kDc, 1, 1);
#pragma unroll
    for (int kk = 0; kk < NB * 4; ++kk) {
      const uint8_t* ch = tile + (kk >> 2) * 2 * kDcTile;
      umma_bf16_ss(tmem, umma_desc_sw128_kmajor(ch) + 2 * (kk & 3), umma_desc_sw128_kmajor(ch + kDcTile) + 2 * (kk & 3), id, kk != 0);
    }
    umma_commit(&bar);
  }
  __syncwarp();
  {                                                                    // 1 / |row|
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < NB * 8; ++u) {
      const uint4 q = tc_ld16(tile + (u >> 3) * 2 * kDcTile, r, u & 7);
      const float2 a = unpack_bf16(q.x), c = unpack_bf16(q.y), d = unpack_bf16(q.z), e = unpack_bf16(q.w);
      ss += a.x * a.x + a.y * a.y + c.x * c.x + c.y * c.y + d.x * d.x + d.y * d.y + e.x * e.x + e.y * e.y;
    }
    const float rn = rsqrtf(ss + kUnitEps);
    if (r < kDc) s_rq[r] = rn * p.qscale; else s_rk[r - kDc] = rn;
  }
  const bool ok = tc_wait(&bar, 0);
  tc_fence_after();
  float raw[kDc];                                                      // row r of [Q; K] K^T
  {
    const uint32_t base = tmem + (static_cast<uint32_t>(w * 32) << 16);
    __syncwarp();
    tmem_ld_32x32(base, reinterpret_cast<uint32_t(&)[32]>(raw[0]));
    tmem_ld_32x32(base + 32, reinterpret_cast<uint32_t(&)[32]>(raw[32]));
    tmem_ld_wait();
  }
  tc_fence_before();
  __syncthreads();
  if (w == 0) { tc_fence_after(); tmem_dealloc(tmem, 64); }
  if (!ok) {
    if (r == 0) atomicExch(err, 1);
    return;                                                            // (what the chunk kernel reads is then arbitrary; the flag says so)
  }

  for (int h0 = 0; h0 < p.rep; h0 += 2) {
    const int pair = min(2, p.rep - h0);
    if (w < pair) {                                                    // running log2 of keep, and beta: two tokens per lane
      const int h = kh * p.rep + h0 + w;
      const float a_neg = -expf(p.a_log[h]) * 1.4426950408889634f, bias = p.b0 ? p.b0[h] : 0.f;
      float l[2], be[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        const bool in = t < nv;
        l[e] = in ? a_neg * softplus_f(p.g0[(t0 + t) * p.ldg + h] + bias) : 0.f;
        be[e] = in ? sigmoid_f(p.g1[(t0 + t) * p.ldg + h]) : 0.f;
      }
      float run = l[0] + l[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += x;
      }
      s_L[w][2 * lane + 1] = run;
      s_L[w][2 * lane] = run - l[1];
      s_beta[w][2 * lane] = be[0];
      s_beta[w][2 * lane + 1] = be[1];
    }
    __syncthreads();
    const int t = r & 63;
    for (int j = 0; j < pair; ++j) {
      const float Lt = s_L[j][t];
      if (r < kDc) {                                                   // P, row t
        uint8_t* dst = work + (static_cast<int64_t>(b) * p.H + kh * p.rep + h0 + j) * kDcWork + 2 * kDcTile;
        const float rq = s_rq[t];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int c = u * 8 + 2 * e;
            const float x = c <= t ? raw[c] * (rq * s_rk[c]) * fast_exp2(Lt - s_L[j][c]) : 0.f;
            const float y = c + 1 <= t ? raw[c + 1] * (rq * s_rk[c + 1]) * fast_exp2(Lt - s_L[j][c + 1]) : 0.f;
            tc_split(x, y, hi[e], lo[e]);
          }
          tc_st16(dst, t, u, hi);
          tc_st16(dst + kDcTile, t, u, lo);
        }
      } else {                                                         // A, row t
        float* row = sA + (j * kDc + t) * kDpLd;
        const float f = s_beta[j][t] * s_rk[t];
#pragma unroll
        for (int c = 0; c < kDc; c += 4) {
          float x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = c + e < t ? raw[c + e] * (f * s_rk[c + e]) * fast_exp2(Lt - s_L[j][c + e]) : 0.f;
          *reinterpret_cast<float4*>(row + c) = make_float4(x[0], x[1], x[2], x[3]);
        }
      }
    }
    __syncthreads();
    const int j = r >> 6;
    if (j < pair) {
      const int64_t item = static_cast<int64_t>(b) * p.H + kh * p.rep + h0 + j;
      const float Lt = s_L[j][t], end = s_L[j][kDc - 1], et = fast_exp2(Lt), rk = s_rk[t];
      float* gt = gates + item * kDcGates;
      gt[t] = et * rk;
      gt[kDc + t] = fast_exp2(end - Lt) * rk;
      gt[2 * kDc + t] = et * s_rq[t];
      if (t < 4) gt[3 * kDc + t] = fast_exp2(end);
      float x[kDc];
      if (t < 32) delta_solve<0>(sA + j * kDc * kDpLd, t, x); else delta_solve<32>(sA + j * kDc * kDpLd, t, x);
      const float be = s_beta[j][t];
      uint8_t* dst = work + item * kDcWork;
      const int unit = t >> 3, sub = (t & 7) * 2;
#pragma unroll
      for (int i = 0; i < kDc; ++i) {
        const float y = x[i] * be;
        const __nv_bfloat16 hi = __float2bfloat16(y), lo = __float2bfloat16(y - __bfloat162float(hi));
        const int at = i * 128 + ((unit ^ (i & 7)) << 4) + sub;
        *reinterpret_cast<__nv_bfloat16*>(dst + at) = hi;
        *reinterpret_cast<__nv_bfloat16*>(dst + kDcTile + at) = lo;
      }
    }
    __syncthreads();
  }
}

template <int NB>
struct DeltaTc {
  static constexpr int NT = NB * kDcTile;                    // 64 tokens x N
  static constexpr int ST = NB * 2 * kDcTile;                // 128 value columns x N
  static constexpr int OFF_K = 2 * ST;                       // two buffers (S: hi, lo ahead of it)
  static constexpr int OFF_Q = OFF_K + 2 * NT;
  static constexpr int OFF_V = OFF_Q + NT;                   // 64 tokens x 128 value columns, plain rows
  static constexpr int OFF_T = OFF_V + 2 * kDcTile;          // hi, lo
  static constexpr int OFF_P = OFF_T + 2 * kDcTile;
  static constexpr int OFF_R = OFF_P + 2 * kDcTile;          // R, then U: 128 x 64 hi, lo
  static constexpr int OFF_W = OFF_R + 4 * kDcTile;          // weighted U: hi, lo
  static constexpr int OFF_F = OFF_W + 4 * kDcTile;
};
struct DeltaShared {                                         // behind the tiles
  float ck[2][kDc], wgt[2][kDc], cq[3][kDc];                 // (a chunk's query carries are read while the chunk after the next one loads)
  float keep[2][4];
  uint64_t bar[5];
  uint32_t tmem;
};

template <int NB>
__global__ void __launch_bounds__(kDcThreads, 1)
mix_delta_chunk_kernel(ScanParams p, const uint8_t* work, const float* gates, int32_t* err) {
  using Cfg = DeltaTc<NB>;
  constexpr int OWN = NB * 32;                               // state rows per thread
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *sS = smem, *sQ = smem + Cfg::OFF_Q, *sV = smem + Cfg::OFF_V, *sT = smem + Cfg::OFF_T, *sP = smem + Cfg::OFF_P, *sR = smem + Cfg::OFF_R,
          *sW = smem + Cfg::OFF_W;
  DeltaShared& sm = *reinterpret_cast<DeltaShared*>(smem + Cfg::OFF_F);
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * 128;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31, quad = w & 3, g = w >> 2, r = quad * 32 + lane;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int N = p.N, V = p.V, vn = min(128, V - v0);
  const __nv_bfloat16* gQ = static_cast<const __nv_bfloat16*>(p.q) + static_cast<int64_t>(t0) * p.ldq + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gK = static_cast<const __nv_bfloat16*>(p.k) + static_cast<int64_t>(t0) * p.ldk + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gV = static_cast<const __nv_bfloat16*>(p.v) + static_cast<int64_t>(t0) * p.ldv + static_cast<int64_t>(h) * V + v0;
  __nv_bfloat16* gO = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(t0) * p.ldo + static_cast<int64_t>(h) * V + v0 + r;
  float* gS = p.S + (p.slot[s] * p.H + h) * static_cast<int64_t>(N) * V + v0 + r;
  const int64_t item0 = static_cast<int64_t>(delta_chunk_base(p.cu, s)) * p.H + h;
  const int chunks = (len + kDc - 1) / kDc;

  auto load_k = [&](int ci) {                                // keys and gates of a chunk
    const int nv = min(kDc, len - ci * kDc);
#pragma unroll
    for (int i = 0; i < NB; ++i)
      tc_load_rows<kDc, kDcThreads>(smem + Cfg::OFF_K + (ci & 1) * Cfg::NT + i * kDcTile, gK + static_cast<int64_t>(ci) * kDc * p.ldk, p.ldk, nv, i * 64, N);
    const float* gt = gates + (item0 + static_cast<int64_t>(ci) * p.H) * kDcGates;
    if (tid < 16) tc_cp16(&sm.ck[ci & 1][tid * 4], gt + tid * 4, true);
    else if (tid < 32) tc_cp16(&sm.wgt[ci & 1][(tid - 16) * 4], gt + kDc + (tid - 16) * 4, true);
    else if (tid < 48) tc_cp16(&sm.cq[ci % 3][(tid - 32) * 4], gt + 2 * kDc + (tid - 32) * 4, true);
    else if (tid == 48) tc_cp16(sm.keep[ci & 1], gt + 3 * kDc, true);
  };
  auto load_q = [&](int ci) {
    const int nv = min(kDc, len - ci * kDc);
#pragma unroll
    for (int i = 0; i < NB; ++i) tc_load_rows<kDc, kDcThreads>(sQ + i * kDcTile, gQ + static_cast<int64_t>(ci) * kDc * p.ldq, p.ldq, nv, i * 64, N);
  };
  auto load_v = [&](int ci) {
    const int nv = min(kDc, len - ci * kDc);
    const __nv_bfloat16* src = gV + static_cast<int64_t>(ci) * kDc * p.ldv;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = tid + i * kDcThreads, t = idx >> 4, c = (idx & 15) * 8;
      const bool ok = t < nv && c < vn;
      tc_cp16(sV + t * 256 + c * 2, src + (ok ? static_cast<int64_t>(t) * p.ldv + c : 0), ok);
    }
  };
  auto load_pair = [&](uint8_t* dst, int ci, int which) {    // 0: T, 1: P
    const uint8_t* src = work + (item0 + static_cast<int64_t>(ci) * p.H) * kDcWork + which * 2 * kDcTile;
#pragma unroll
    for (int i = 0; i < 4; ++i) tc_cp16(dst + (tid + i * kDcThreads) * 16, src + (tid + i * kDcThreads) * 16, true);
  };

  load_k(0);
  load_q(0);
  load_v(0);
  tc_cp_commit();
  load_pair(sT, 0, 0);
  tc_cp_commit();
  if (tid == 0) {
    for (int i = 0; i < 5; ++i) mbar_init(&sm.bar[i], 1);
    fence_barrier_init();
  }
  if (w == 0) { tmem_alloc(&sm.tmem, 512); tmem_relinquish(); }

  float S[OWN];                                              // state rows g * OWN + i of value column r
#pragma unroll
  for (int i = 0; i < OWN; ++i) {
    const int n = g * OWN + i;
    S[i] = (!fresh && n < N && r < vn) ? gS[static_cast<int64_t>(n) * V] : 0.f;
  }
  auto stage_state = [&]() {
#pragma unroll
    for (int u = 0; u < OWN / 8; ++u) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) tc_split(S[u * 8 + 2 * e], S[u * 8 + 2 * e + 1], hi[e], lo[e]);
      const int n = g * OWN + u * 8;
      tc_st16(sS + (n >> 6) * 2 * kDcTile, r, (n & 63) >> 3, hi);
      tc_st16(sS + Cfg::ST + (n >> 6) * 2 * kDcTile, r, (n & 63) >> 3, lo);
    }
  };
  bool have_state = !fresh, ok = true;
  if (have_state) stage_state();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem, tK = tmem, tQ = tmem + 64, tU = tmem + 192, tO = tmem + 256, tD = tmem + 320;
  const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
  constexpr uint32_t idKK = umma_idesc(128, kDc, 1, 1);
  constexpr uint32_t idKM = umma_idesc_major(128, NB * 64, 1, 1, 0, 1);

  // y of chunk ci: columns are its tokens, this thread's half
  auto write_out = [&](int ci, bool carried) {
    uint32_t a[32], b[32];
    __syncwarp();
    tmem_ld_32x32(tO + lanes + g * 32, a);
    if (carried) tmem_ld_32x32(tQ + (ci & 1) * 64 + lanes + g * 32, b);
    tmem_ld_wait();
    const int nv = min(kDc, len - ci * kDc) - g * 32;
    const float* cq = sm.cq[ci % 3] + g * 32;
    __nv_bfloat16* dst = gO + (static_cast<int64_t>(ci) * kDc + g * 32) * p.ldo;
    if (r < vn) {
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float y = __uint_as_float(a[i]) + (carried ? cq[i] * __uint_as_float(b[i]) : 0.f);
        if (i < nv) dst[i * p.ldo] = __float2bfloat16(y);
      }
    }
  };
  // 32 values of row r as hi + lo, columns g * 32 ...
  auto stage_half = [&](uint8_t* tile, const float (&x)[32]) {
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) tc_split(x[u * 8 + 2 * e], x[u * 8 + 2 * e + 1], hi[e], lo[e]);
      tc_st16(tile, r, g * 4 + u, hi);
      tc_st16(tile + 2 * kDcTile, r, g * 4 + u, lo);
    }
  };
  // D[128 x 64] = (A hi + A lo) (B hi + B lo)^T over 64, without lo lo; both K-major
  auto mma_pairs = [&](uint32_t d, const uint8_t* a, const uint8_t* b) {
#pragma unroll
    for (int c = 0; c < 3; ++c)
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        umma_bf16_ss(d, umma_desc_sw128_kmajor(a + (c == 1 ? 2 * kDcTile : 0)) + 2 * kk, umma_desc_sw128_kmajor(b + (c == 2 ? kDcTile : 0)) + 2 * kk, idKK,
                     (c | kk) != 0);
  };
  bool carried_prev = false;

  for (int ci = 0; ci < chunks; ++ci) {
    const uint32_t ph = ci & 1;
    const bool more = ci + 1 < chunks;
    const uint8_t* sK = smem + Cfg::OFF_K + (ci & 1) * Cfg::NT;
    tc_cp_wait<1>();                                         // keys, gates, queries and values; T may still be on its way
    fence_proxy_async();
    tc_fence_before();
    if (__syncthreads_or(!ok)) {
      if (tid == 0) atomicExch(err, 1);
      ok = false;
      break;
    }
    if (tid == 0) {
      tc_fence_after();
      if (have_state) {
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < NB * 4; ++kk)
            umma_bf16_ss(tK, umma_desc_sw128_kmajor(sS + hl * Cfg::ST + (kk >> 2) * 2 * kDcTile) + 2 * (kk & 3),
                         umma_desc_sw128_kmajor(sK + (kk >> 2) * kDcTile) + 2 * (kk & 3), idKK, (hl | kk) != 0);
      }
      umma_commit(&sm.bar[0]);
      if (have_state) {
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < NB * 4; ++kk)
            umma_bf16_ss(tQ + (ci & 1) * 64, umma_desc_sw128_kmajor(sS + hl * Cfg::ST + (kk >> 2) * 2 * kDcTile) + 2 * (kk & 3),
                         umma_desc_sw128_kmajor(sQ + (kk >> 2) * kDcTile) + 2 * (kk & 3), idKK, (hl | kk) != 0);
      }
      umma_commit(&sm.bar[1]);
    }
    __syncwarp();
    if (more) load_k(ci + 1);
    tc_cp_commit();
    if (ci > 0) {
      ok = tc_wait(&sm.bar[4], ph ^ 1) && ok;
      tc_fence_after();
      write_out(ci - 1, carried_prev);
    }
    load_pair(sP, ci, 1);                                    // (its reader, the own part of the previous chunk, is done)
    tc_cp_commit();
    carried_prev = have_state;
    ok = tc_wait(&sm.bar[0], ph) && ok;
    tc_fence_after();
    {                                                        // R = v - carry_t S_0^T k_t  (T holds beta)
      float x[32];
      uint32_t d[32];
      if (have_state) {
        __syncwarp();
        tmem_ld_32x32(tK + lanes + g * 32, d);
        tmem_ld_wait();
      }
      const float* ck = sm.ck[ci & 1] + g * 32;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float v = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sV + (g * 32 + i) * 256 + r * 2));
        x[i] = have_state ? v - ck[i] * __uint_as_float(d[i]) : v;
      }
      stage_half(sR, x);
    }
    tc_cp_wait<2>();                                         // T
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
      mma_pairs(tU, sR, sT);
      umma_commit(&sm.bar[2]);
    }
    __syncwarp();
    ok = tc_wait(&sm.bar[1], ph) && ok;
    if (more) load_q(ci + 1);
    tc_cp_commit();
    if (more) load_v(ci + 1);
    tc_cp_commit();
    ok = tc_wait(&sm.bar[2], ph) && ok;
    tc_fence_after();
    {                                                        // U, and U weighted by its part in the final state
      uint32_t d[32];
      __syncwarp();
      tmem_ld_32x32(tU + lanes + g * 32, d);
      tmem_ld_wait();
      float x[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] = __uint_as_float(d[i]);
      stage_half(sR, x);
      const float* wg = sm.wgt[ci & 1] + g * 32;
#pragma unroll
      for (int i = 0; i < 32; ++i) x[i] *= wg[i];
      stage_half(sW, x);
    }
    tc_cp_wait<2>();                                         // P
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
#pragma unroll
      for (int hl = 0; hl < 2; ++hl)
#pragma unroll
        for (int kk = 0; kk < 4; ++kk)
          umma_bf16_ss(tD, umma_desc_sw128_kmajor(sW + hl * 2 * kDcTile) + 2 * kk, umma_desc_sw128_mnmajor(sK, kDcTile) + kk * 128, idKM, (hl | kk) != 0);
      umma_commit(&sm.bar[3]);
      mma_pairs(tO, sR, sP);
      umma_commit(&sm.bar[4]);
    }
    __syncwarp();
    if (more) load_pair(sT, ci + 1, 0);
    tc_cp_commit();
    const float keep = sm.keep[ci & 1][0];
    ok = tc_wait(&sm.bar[3], ph) && ok;
    tc_fence_after();
#pragma unroll
    for (int c = 0; c < OWN; c += 32) {
      uint32_t d[32];
      __syncwarp();
      tmem_ld_32x32(tD + lanes + g * OWN + c, d);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) S[c + i] = keep * S[c + i] + __uint_as_float(d[i]);
    }
    have_state = true;
    if (more) stage_state();
  }
  tc_cp_wait<0>();
  ok = ok && tc_wait(&sm.bar[4], (chunks - 1) & 1);
  if (__syncthreads_or(!ok)) {
    if (tid == 0) atomicExch(err, 1);
  } else {
    tc_fence_after();
    write_out(chunks - 1, carried_prev);
    if (r < vn) {
#pragma unroll
      for (int i = 0; i < OWN; ++i)
        if (g * OWN + i < N) gS[static_cast<int64_t>(g * OWN + i) * V] = S[i];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (w == 0) { tc_fence_after(); tmem_dealloc(sm.tmem, 512); }
}

template <int NB>
static int run_delta(const ScanParams& p, int total_chunks, uint8_t* work, float* gates, int32_t* err, cudaStream_t st) {
  constexpr int smem1 = NB * 2 * kDcTile + 2 * kDc * kDpLd * 4 + 1024, smem2 = DeltaTc<NB>::OFF_F + static_cast<int>(sizeof(DeltaShared)) + 1024;
  static_assert(smem2 <= 232448, "shared memory");
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_delta_prep_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem1));
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_delta_chunk_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2));
    attr = true;
  }
  mix_delta_prep_kernel<NB><<<dim3(total_chunks, p.H / p.rep), kDpThreads, smem1, st>>>(p, work, gates, err);
  PRL_CUDA_CHECK(cudaGetLastError());
  mix_delta_chunk_kernel<NB><<<dim3((p.V + 127) / 128, p.H, p.spans), kDcThreads, smem2, st>>>(p, work, gates, err);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

// 16-byte aligned rows of q, k and v; head sizes multiples of 8, at most 128 state rows
extern "C" int prl_mix_delta_ok(const void* q, int64_t ldq, const void* k, int64_t ldk, const void* v, int64_t ldv, int N, int V) {
  auto al = [](const void* x, int64_t ld) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0 && ld % 8 == 0; };
  return N % 8 == 0 && V % 8 == 0 && N <= 128 && al(q, ldq) && al(k, ldk) && al(v, ldv);
}
extern "C" int64_t prl_mix_delta_chunks(int64_t tokens, int64_t spans) { return tokens / kDc + spans; }
extern "C" int prl_mix_delta_work_bytes() { return kDcWork; }
extern "C" int prl_mix_delta_gate_floats() { return kDcGates; }
// chunks: prl_mix_delta_chunks; work: chunks * H * work_bytes, gates: chunks * H * gate_floats, both 16-byte aligned; *err becomes 1 when
// a wait inside a kernel timed out
extern "C" int prl_mix_delta(const ScanParams* p, int64_t chunks, void* work, float* gates, int32_t* err, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || chunks > 0x7fffffff || !prl_mix_delta_ok(p->q, p->ldq, p->k, p->ldk, p->v, p->ldv, p->N, p->V)) return -260;
  uint8_t* wk = static_cast<uint8_t*>(work);
  return p->N <= 64 ? run_delta<1>(*p, static_cast<int>(chunks), wk, gates, err, st) : run_delta<2>(*p, static_cast<int>(chunks), wk, gates, err, st);
}
