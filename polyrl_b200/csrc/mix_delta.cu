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
//                         128 x 64 product, then per value head T = (I + A)^-1 diag(beta) by substitution in fp32 (thread = column)
//                         and P.  T and P go to the workspace as bf16 pairs hi + lo, laid out as the swizzled tiles the next kernel copies.
// mix_delta_chunk_kernel  one CTA per (span, head, 128 value columns) marching over its chunks, all products transposed so that the value
//                         columns are the 128 rows (TMEM lane = value column) and the tokens or state rows the columns:
//                             carried = S_0^T [K | Q]^T     U^T = R^T T^T     own = U^T P^T     delta = (weighted U)^T K
//                         The left operands (state, R, U) are staged from registers into TMEM, the right ones lie in shared memory.  The fp32
//                         state lives in registers, thread (value column, half) owning half of the state rows, and is restaged once per chunk.
//                         Warps 0-7 do that arithmetic; warp 8 issues the products of the chain and the loads (a chunk ahead), warp 9 the own part
//                         and the stores.  A chunk's outputs are written while the next chunk's U is computed.
// Operands that are not bf16 by nature (S, R, U, T, P) enter the products as bf16 pairs hi + lo.
// Every wait is bounded: on a timeout the CTA raises *err, runs out its chunks without waiting, loading or multiplying, frees its TMEM and returns.
#include "mix_tc.cuh"

namespace prl {

constexpr int kDc = 64;                        // tokens per chunk
constexpr int kDcTile = 64 * 128;              // bytes of a 64 x 64 bf16 tile
constexpr int kDcWork = 4 * kDcTile;           // workspace of one (chunk, head): T hi, T lo, P hi, P lo
constexpr int kDcGates = 3 * kDc + 4;          // floats: carry of a key row, weight in the final state, carry of a query row, keep
constexpr int kDpThreads = 128, kDcThreads = 384;
constexpr int kDpLd = 68;                      // row pitch of A in floats

__device__ __forceinline__ int delta_chunk_base(const int32_t* cu, int s) { return cu[s] / kDc + s; }     // workspace rows of a span start here

// column c of X = (I + A)^-1, 16 rows at a time: what the rows ahead of a block say about it, then the block itself.  buf holds A transposed
// (A_ts at row s, column t > s) and takes X below its diagonal (x_t at row t, column c < t).  Rolled: every instruction runs once per CTA
// otherwise, and the instruction cache is what it waits for.  Rows below `from` are known to be zero.
__device__ __forceinline__ float delta_x(const float* buf, int t, int c) { return t > c ? buf[t * kDpLd + c] : (t == c ? 1.f : 0.f); }
__device__ __forceinline__ void delta_solve(float* buf, int c, int from) {
#pragma unroll 1
  for (int t0 = from; t0 < kDc; t0 += 16) {
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) x[i] = t0 + i == c ? 1.f : 0.f;
#pragma unroll 4
    for (int s = from; s < t0; ++s) {
      const float xs = delta_x(buf, s, c);
#pragma unroll
      for (int i = 0; i < 16; i += 4) {
        const float4 a = *reinterpret_cast<const float4*>(buf + s * kDpLd + t0 + i);
        x[i] -= a.x * xs; x[i + 1] -= a.y * xs; x[i + 2] -= a.z * xs; x[i + 3] -= a.w * xs;
      }
    }
#pragma unroll
    for (int s = 0; s < 15; ++s) {
#pragma unroll
      for (int i = (s + 1) & ~3; i < 16; i += 4) {
        const float4 a = *reinterpret_cast<const float4*>(buf + (t0 + s) * kDpLd + t0 + i);
        if (i > s) x[i] -= a.x * x[s];
        if (i + 1 > s) x[i + 1] -= a.y * x[s];
        if (i + 2 > s) x[i + 2] -= a.z * x[s];
        x[i + 3] -= a.w * x[s];
      }
    }
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (t0 + i > c) buf[(t0 + i) * kDpLd + c] = x[i];
  }
}

template <int NB>
__global__ void __launch_bounds__(kDpThreads, 3) mix_delta_prep_kernel(ScanParams p, uint8_t* work, float* gates, int32_t* err) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* tile = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));   // NB chunks of [64 Q rows; 64 K rows],
  float* sA = reinterpret_cast<float*>(tile + 4 * kDcTile);            // later P of two heads; [2][64][kDpLd], later T of two heads
  __shared__ alignas(16) float s_L[2][kDc], s_beta[2][kDc], s_rq[kDc], s_rk[kDc];
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
  auto run_gates = [&](int h0) {                                       // warp w: running log2 of keep, and beta, of a head; two tokens per lane
    if (w >= min(2, p.rep - h0)) return;
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
  };
  run_gates(0);
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
  if (__syncthreads_or(!ok)) {
    if (r == 0) atomicExch(err, 1);
    if (w == 0) tmem_dealloc(tmem, 64);
    return;                                                            // (what the chunk kernel reads is then arbitrary; the flag says so)
  }

  for (int h0 = 0; h0 < p.rep; h0 += 2) {
    const int pair = min(2, p.rep - h0);
    if (h0 > 0) run_gates(h0);
    __syncthreads();
    const int t = r & 63;
    const int64_t item = static_cast<int64_t>(b) * p.H + kh * p.rep + h0;
    // 16 raw scores of the thread's row at a time (rolled, as the substitution is): row t of P, or of A into its transposed place
#pragma unroll 1
    for (int c0 = 0; c0 <= (w & 1) * 32 + 31; c0 += 16) {
      uint32_t raw[16];
      __syncwarp();
      tmem_ld_32x16(tmem + (static_cast<uint32_t>(w * 32) << 16) + c0, raw);
      tmem_ld_wait();
#pragma unroll 1
      for (int j = 0; j < pair; ++j) {
        const float Lt = s_L[j][t], f = r < kDc ? s_rq[t] : s_beta[j][t] * s_rk[t];
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; i += 4) {
          const float4 k = *reinterpret_cast<const float4*>(&s_rk[c0 + i]), l = *reinterpret_cast<const float4*>(&s_L[j][c0 + i]);
          x[i] = __uint_as_float(raw[i]) * (f * k.x) * fast_exp2(Lt - l.x);
          x[i + 1] = __uint_as_float(raw[i + 1]) * (f * k.y) * fast_exp2(Lt - l.y);
          x[i + 2] = __uint_as_float(raw[i + 2]) * (f * k.z) * fast_exp2(Lt - l.z);
          x[i + 3] = __uint_as_float(raw[i + 3]) * (f * k.w) * fast_exp2(Lt - l.w);
        }
        if (r < kDc) {
          uint8_t* dst = tile + j * 2 * kDcTile;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int e = 0; e < 8; ++e) x[u * 8 + e] = c0 + u * 8 + e <= t ? x[u * 8 + e] : 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) tc_split(x[u * 8 + 2 * e], x[u * 8 + 2 * e + 1], hi[e], lo[e]);
            tc_st16(dst, t, c0 / 8 + u, hi);
            tc_st16(dst + kDcTile, t, c0 / 8 + u, lo);
          }
        } else {
          float* col = sA + (j * kDc + c0) * kDpLd + t;
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (c0 + i < t) col[i * kDpLd] = x[i];
        }
      }
    }
    if (r < 32) {                                                      // above the diagonal block
      const uint32_t zero[4] = {0, 0, 0, 0};
      for (int j = 0; j < 2 * pair; ++j)
#pragma unroll
        for (int u = 4; u < 8; ++u) tc_st16(tile + j * kDcTile, t, u, zero);
    }
    __syncthreads();
    const int j = r >> 6;
    float x[kDc];
    if (j < pair) {
      const float Lt = s_L[j][t], end = s_L[j][kDc - 1], et = fast_exp2(Lt), rk = s_rk[t];
      float* gt = gates + (item + j) * kDcGates;
      gt[t] = et * rk;
      gt[kDc + t] = fast_exp2(end - Lt) * rk;
      gt[2 * kDc + t] = et * s_rq[t];
      if (t < 4) gt[3 * kDc + t] = fast_exp2(end);
      float* buf = sA + j * kDc * kDpLd;
      delta_solve(buf, t, t & 32);
#pragma unroll
      for (int i = 0; i < kDc; ++i) x[i] = delta_x(buf, i, t);
    }
    __syncthreads();
    if (j < pair) {                                                    // T over A, column t
      const float be = s_beta[j][t];
      uint8_t* dst = reinterpret_cast<uint8_t*>(sA + j * kDc * kDpLd);
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
    fence_proxy_async();
    __syncthreads();
    if (r == 0) {
      for (int i = 0; i < pair; ++i) {
        bulk_store(work + (item + i) * kDcWork, sA + i * kDc * kDpLd, 2 * kDcTile);
        bulk_store(work + (item + i) * kDcWork + 2 * kDcTile, tile + i * 2 * kDcTile, 2 * kDcTile);
      }
      tma_store_commit();
      if (h0 + 2 < p.rep) tma_store_wait_read<0>(); else tma_store_wait<0>();
    }
    tc_fence_before();
    __syncthreads();
  }
  if (w == 0) { tc_fence_after(); tmem_dealloc(tmem, 64); }
}

template <int NB>
struct DeltaTc {
  static constexpr int NT = NB * kDcTile;                    // 64 tokens x N
  static constexpr int VT = 2 * kDcTile;                     // 64 tokens x 128 value columns, plain rows
  static constexpr int OFF_Q = 2 * NT;                       // everything but the outputs in two buffers
  static constexpr int OFF_V = 4 * NT;
  static constexpr int OFF_W = OFF_V + 2 * VT;               // T hi, T lo, P hi, P lo
  static constexpr int OFF_O = OFF_W + 2 * kDcWork;
  static constexpr int OFF_F = OFF_O + VT;
  static constexpr uint32_t LOAD = 2 * NT + VT + kDcWork + kDcGates * 4;        // bytes of a chunk
};
struct DeltaShared {                                         // behind the tiles
  float gates[3][kDcGates];                                  // (a chunk's query carries are read while the chunk after the next one loads)
  uint64_t carried, writes, delta, own, full[2];             // products done: S_0^T K, U, the state's increment, U P; a chunk has arrived
  uint32_t tmem;
  int fail;
};
static_assert(kDcGates * 4 % 16 == 0, "copied in 16-byte units");
// warps 0-7 hand over to warp 8 (state, R, weighted U) and warp 9 (U, outputs); at state and outputs they wait too, which keeps all in one chunk
enum : int { kBarState = 1, kBarR, kBarW, kBarU, kBarOut };
constexpr int kDcHandoff = 288;
// 12 warps x 168 registers at launch = 8 x 216 + 4 x 72
constexpr int kDcRegsMath = 216, kDcRegsIo = 72;
static_assert(8 * kDcRegsMath + 4 * kDcRegsIo <= 12 * 168, "register split");

__device__ __forceinline__ void delta_arrive(int id) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "n"(kDcHandoff) : "memory"); }
__device__ __forceinline__ void delta_sync(int id) { asm volatile("bar.sync %0, %1;" ::"r"(id), "n"(kDcHandoff) : "memory"); }
__device__ __forceinline__ void delta_wait(DeltaShared& sm, uint64_t* bar, uint32_t parity) {
  if (*reinterpret_cast<volatile int*>(&sm.fail)) return;
  if (!tc_wait(bar, parity)) *reinterpret_cast<volatile int*>(&sm.fail) = 1;
}
// C values of a row as bf16 pairs: hi + lo
template <int C>
__device__ __forceinline__ void delta_stage(uint32_t hi_at, uint32_t lo_at, const float* x) {
#pragma unroll
  for (int c = 0; c < C; c += 32) {
    uint32_t hi[16], lo[16];
#pragma unroll
    for (int e = 0; e < 16; ++e) tc_split(x[c + 2 * e], x[c + 2 * e + 1], hi[e], lo[e]);
    tmem_st_32x16(hi_at + c / 2, hi);
    tmem_st_32x16(lo_at + c / 2, lo);
  }
}

template <int NB>
__global__ void __launch_bounds__(kDcThreads, 1)
mix_delta_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmO,
                       ScanParams p, const uint8_t* work, const float* gates, int32_t* err) {
  using Cfg = DeltaTc<NB>;
  constexpr int OWN = NB * 32;                               // state rows per thread
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sO = smem + Cfg::OFF_O;
  DeltaShared& sm = *reinterpret_cast<DeltaShared*>(smem + Cfg::OFF_F);
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * 128;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int N = p.N, V = p.V, vn = min(128, V - v0);
  const int chunks = (len + kDc - 1) / kDc;
  if (tid == 0) {
    mbar_init(&sm.carried, 1);
    mbar_init(&sm.writes, 1);
    mbar_init(&sm.delta, 1);
    mbar_init(&sm.own, 1);
    mbar_init(&sm.full[0], 1);
    mbar_init(&sm.full[1], 1);
    sm.fail = 0;
    fence_barrier_init();
  }
  if (w == 8) { tmem_alloc(&sm.tmem, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // TMEM columns.  State operand of half g: hi at tS + g * OWN, lo behind it; the state's increment uses the same columns once the operand is
  // spent, row by row where the thread that reads it stages its next operand.  U overwrites R, and its accumulator that of the carried keys.
  const uint32_t tS = sm.tmem, tR = tS + 128, tW = tS + 192, tK = tS + 256, tQ = tS + 320, tO = tS + 448;

  if (w >= 8) {
    // ================================ products, loads, stores ================================
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kDcRegsIo));
    constexpr uint32_t idKK = umma_idesc(128, kDc, 1, 1);
    // D [128 x 64] = (A hi + A lo) (B hi + B lo)^T over the chunk's tokens, without lo lo
    auto mma_pairs = [&](uint32_t d, const uint8_t* b) {
      const uint64_t desc = umma_desc_sw128_kmajor(b);
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        umma_bf16_ts(d, tR + kk * 8, desc + 2 * kk, idKK, kk != 0);
        umma_bf16_ts(d, tR + 32 + kk * 8, desc + 2 * kk, idKK, 1);
        umma_bf16_ts(d, tR + kk * 8, desc + (kDcTile >> 4) + 2 * kk, idKK, 1);
      }
    };
    if (w == 9) {
      __nv_bfloat16* gO = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(t0) * p.ldo + static_cast<int64_t>(h) * V + v0;
      auto store = [&](int ci) {
        if (*reinterpret_cast<volatile int*>(&sm.fail)) return;
        const int nv = len - ci * kDc;
        if (nv >= kDc) {
          if (lane == 0) tma_store_3d(&tmO, sO, v0, h, t0 + ci * kDc);
        } else {                                             // a row at a time: the next rows are another span's
          for (int t = lane; t < nv; t += 32) bulk_store(gO + (static_cast<int64_t>(ci) * kDc + t) * p.ldo, sO + t * 256, vn * 2);
        }
        tma_store_commit();
      };
      for (int ci = 0; ci < chunks; ++ci) {
        if (ci > 0) {
          delta_sync(kBarOut);
          store(ci - 1);
        }
        delta_sync(kBarU);
        tma_store_wait_read<0>();                            // (`own` also tells that sO is free)
        __syncwarp();
        if (lane == 0 && !*reinterpret_cast<volatile int*>(&sm.fail)) {
          tc_fence_after();
          mma_pairs(tO, smem + Cfg::OFF_W + (ci & 1) * kDcWork + 2 * kDcTile);
          umma_commit(&sm.own);
        }
        __syncwarp();
      }
      delta_sync(kBarOut);
      store(chunks - 1);
      tma_store_wait<0>();
    } else if (w == 8) {
    constexpr uint32_t idKM = umma_idesc_major(128, NB * 64, 1, 1, 0, 1);
    const int64_t item0 = static_cast<int64_t>(delta_chunk_base(p.cu, s)) * p.H + h;
    auto load = [&](int ci) {
      const int bf = ci & 1, t = t0 + ci * kDc;
      const int64_t item = item0 + static_cast<int64_t>(ci) * p.H;
      uint64_t* bar = &sm.full[bf];
      mbar_expect_tx(bar, Cfg::LOAD);
#pragma unroll
      for (int c = 0; c < NB; ++c) tma_load_3d(&tmK, bar, smem + bf * Cfg::NT + c * kDcTile, c * 64, h / p.rep, t);
#pragma unroll
      for (int c = 0; c < NB; ++c) tma_load_3d(&tmQ, bar, smem + Cfg::OFF_Q + bf * Cfg::NT + c * kDcTile, c * 64, h / p.rep, t);
      tma_load_3d(&tmV, bar, smem + Cfg::OFF_V + bf * Cfg::VT, v0, h, t);
      bulk_load(bar, smem + Cfg::OFF_W + bf * kDcWork, work + item * kDcWork, kDcWork);
      bulk_load(bar, sm.gates[ci % 3], gates + item * kDcGates, kDcGates * 4);
    };
    // D [128 x 64] = S_0^T X^T, X = keys or queries of the chunk
    auto mma_state = [&](uint32_t d, const uint8_t* x) {
      const uint64_t desc = umma_desc_sw128_kmajor(x);
#pragma unroll
      for (int kk = 0; kk < NB * 4; ++kk) {
        const uint32_t a = tS + (kk * 16 / OWN) * OWN + (kk * 16 % OWN) / 2;
        const uint64_t b = desc + (kk >> 2) * (kDcTile >> 4) + 2 * (kk & 3);
        umma_bf16_ts(d, a, b, idKK, kk != 0);
        umma_bf16_ts(d, a + OWN / 2, b, idKK, 1);
      }
    };
    int loaded = 0;
    if (lane == 0) {
      tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
      load(0);
      loaded = 1;
    }
    for (int ci = 0; ci < chunks; ++ci) {
      const uint32_t ph = ci & 1, fph = (ci >> 1) & 1;
      uint8_t *sK = smem + ph * Cfg::NT, *sT = smem + Cfg::OFF_W + ph * kDcWork;
      if (lane == 0) delta_wait(sm, &sm.full[ph], fph);
      __syncwarp();
      const int nv = len - ci * kDc;
      if (nv < kDc) {                                        // the tile's last rows are another span's tokens
        for (int i = lane; i < (kDc - nv) * 8 * NB; i += 32) {
          const int row = nv + i / (8 * NB), at = (i % (8 * NB) / 8) * kDcTile + row * 128 + (i % 8) * 16;
          *reinterpret_cast<uint4*>(sK + at) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(sK + Cfg::OFF_Q + at) = make_uint4(0, 0, 0, 0);
        }
        fence_proxy_async();
      }
      __syncwarp();
      delta_sync(kBarState);
      const bool run = !*reinterpret_cast<volatile int*>(&sm.fail);
      if (lane == 0 && run) {
        tc_fence_after();
        const bool have_state = ci > 0 || !fresh;
        if (have_state) mma_state(tK, sK);
        umma_commit(&sm.carried);
        if (have_state) mma_state(tQ + ph * 64, sK + Cfg::OFF_Q);
        if (ci > 0) delta_wait(sm, &sm.own, ph ^ 1);        // the last reader of the buffers that fill next
        if (ci + 1 < chunks) { load(ci + 1); ++loaded; }
      }
      __syncwarp();
      delta_sync(kBarR);
      if (lane == 0 && run) {
        tc_fence_after();
        mma_pairs(tK, sT);
        umma_commit(&sm.writes);
      }
      __syncwarp();
      delta_sync(kBarW);
      if (lane == 0 && run) {
        tc_fence_after();
        const uint64_t desc = umma_desc_sw128_mnmajor(sK, kDcTile);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
          umma_bf16_ts(tS, tW + kk * 8, desc + kk * 128, idKM, kk != 0);
          umma_bf16_ts(tS, tW + 32 + kk * 8, desc + kk * 128, idKM, 1);
        }
        umma_commit(&sm.delta);
      }
      __syncwarp();
    }
    delta_sync(kBarState);                                   // (after the last chunk: every wait of the others is over)
    if (*reinterpret_cast<volatile int*>(&sm.fail) && lane == 0) {
      atomicExch(err, 1);                                    // copies in flight end before the shared memory is given up
      if (loaded > 0) tc_wait(&sm.full[0], ((loaded + 1) / 2 - 1) & 1);
      if (loaded > 1) tc_wait(&sm.full[1], (loaded / 2 - 1) & 1);
    }
    __syncwarp();
    }
  } else {
    // ================================ warps 0-7: state, R, U and outputs ================================
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kDcRegsMath));
    const int quad = w & 3, g = w >> 2, r = quad * 32 + lane;          // value column, half of the state rows or tokens
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    float* gS = p.S + (p.slot[s] * p.H + h) * static_cast<int64_t>(N) * V + v0 + r;
    float S[OWN];                                            // state rows g * OWN + i
#pragma unroll
    for (int i = 0; i < OWN; ++i) {
      const int n = g * OWN + i;
      S[i] = (!fresh && n < N && r < vn) ? gS[static_cast<int64_t>(n) * V] : 0.f;
    }
    auto stage_state = [&]() { delta_stage<OWN>(tS + lanes + g * OWN, tS + lanes + g * OWN + OWN / 2, S); };
    bool have_state = !fresh, carried_prev = false;
    if (have_state) stage_state();
    auto stage_out = [&](int ci, bool carried) {             // y of chunk ci, this thread's half of its tokens
      uint32_t a[32], b[32];
      __syncwarp();
      tmem_ld_32x32(tO + lanes + g * 32, a);
      if (carried) tmem_ld_32x32(tQ + (ci & 1) * 64 + lanes + g * 32, b);
      tmem_ld_wait();
      const float* cq = sm.gates[ci % 3] + 2 * kDc + g * 32;
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(sO) + g * 32 * 128 + r;
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        const float4 c = *reinterpret_cast<const float4*>(cq + i);
        const float cc[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          dst[(i + e) * 128] = __float2bfloat16(__uint_as_float(a[i + e]) + (carried ? cc[e] * __uint_as_float(b[i + e]) : 0.f));
      }
    };

    for (int ci = 0; ci < chunks; ++ci) {
      const uint32_t ph = ci & 1, fph = (ci >> 1) & 1;
      const float* gt = sm.gates[ci % 3];
      tmem_st_wait();
      tc_fence_before();
      delta_sync(kBarState);
      if (ci > 0) {
        delta_wait(sm, &sm.own, ph ^ 1);
      }
      delta_wait(sm, &sm.full[ph], fph);
      {                                                      // R = v - carry_t S_0^T k_t  (T holds beta)
        float x[32];
        uint32_t d[32];
        const uint8_t* vv = smem + Cfg::OFF_V + ph * Cfg::VT + g * 32 * 256 + r * 2;
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(vv + i * 256));
        delta_wait(sm, &sm.carried, ph);
        tc_fence_after();
        if (have_state) {
          __syncwarp();
          tmem_ld_32x32(tK + lanes + g * 32, d);
          tmem_ld_wait();
        }
        if (have_state) {
          const float* ck = gt + g * 32;
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 c = *reinterpret_cast<const float4*>(ck + i);
            x[i] -= c.x * __uint_as_float(d[i]); x[i + 1] -= c.y * __uint_as_float(d[i + 1]);
            x[i + 2] -= c.z * __uint_as_float(d[i + 2]); x[i + 3] -= c.w * __uint_as_float(d[i + 3]);
          }
        }
        const int nv = len - ci * kDc - g * 32;
        if (nv < 32) {                                       // rows of another span
#pragma unroll
          for (int i = 0; i < 32; ++i) x[i] = i < nv ? x[i] : 0.f;
        }
        __syncwarp();
        delta_stage<32>(tR + lanes + g * 16, tR + lanes + 32 + g * 16, x);
      }
      tmem_st_wait();
      tc_fence_before();
      delta_arrive(kBarR);
      if (ci > 0) {                                          // while U is computed
        stage_out(ci - 1, carried_prev);
        tc_fence_before();
        fence_proxy_async();
        delta_sync(kBarOut);
      }
      carried_prev = have_state;
      delta_wait(sm, &sm.writes, ph);
      tc_fence_after();
      {                                                      // U, weighted by its part in the final state and as it is
        uint32_t d[32];
        __syncwarp();
        tmem_ld_32x32(tK + lanes + g * 32, d);
        tmem_ld_wait();
        float x[32];
        const float* wg = gt + kDc + g * 32;
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float4 c = *reinterpret_cast<const float4*>(wg + i);
          x[i] = __uint_as_float(d[i]) * c.x; x[i + 1] = __uint_as_float(d[i + 1]) * c.y;
          x[i + 2] = __uint_as_float(d[i + 2]) * c.z; x[i + 3] = __uint_as_float(d[i + 3]) * c.w;
        }
        delta_stage<32>(tW + lanes + g * 16, tW + lanes + 32 + g * 16, x);
        tmem_st_wait();
        tc_fence_before();
        delta_arrive(kBarW);
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = __uint_as_float(d[i]);
        delta_stage<32>(tR + lanes + g * 16, tR + lanes + 32 + g * 16, x);
      }
      tmem_st_wait();
      tc_fence_before();
      delta_arrive(kBarU);
      const float keep = gt[3 * kDc];
      delta_wait(sm, &sm.delta, ph);
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < OWN; c += 32) {
        uint32_t d[32];
        __syncwarp();
        tmem_ld_32x32(tS + lanes + g * OWN + c, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) S[c + i] = keep * S[c + i] + __uint_as_float(d[i]);
      }
      have_state = true;
      if (ci + 1 < chunks) stage_state();
    }
    tmem_st_wait();
    delta_wait(sm, &sm.own, (chunks - 1) & 1);
    tc_fence_after();
    stage_out(chunks - 1, carried_prev);
    fence_proxy_async();
    delta_sync(kBarOut);
    delta_sync(kBarState);
    if (!*reinterpret_cast<volatile int*>(&sm.fail) && r < vn) {
      int64_t ld = V;
      asm volatile("" : "+l"(gS), "+l"(ld));                 // (addresses are computed again, not kept across the loop)
      float* dst = gS + g * OWN * ld;
#pragma unroll
      for (int i = 0; i < OWN; ++i, dst += ld)
        if (g * OWN + i < N) *dst = S[i];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (w == 8) { tc_fence_after(); tmem_dealloc(sm.tmem, 512); }
}

template <int NB>
static int run_delta(const ScanParams& p, int64_t tokens, int total_chunks, uint8_t* work, float* gates, int32_t* err, cudaStream_t st) {
  constexpr int smem1 = 4 * kDcTile + 2 * kDc * kDpLd * 4 + 1024, smem2 = DeltaTc<NB>::OFF_F + static_cast<int>(sizeof(DeltaShared)) + 1024;
  static_assert(smem2 <= 232448, "shared memory");
  CUtensorMap tmQ, tmK, tmV, tmO;
  const int G = p.H / p.rep;
  if (tc_tokens_tmap(&tmQ, p.q, tokens, G, p.N, p.ldq, kDc, 64, true) || tc_tokens_tmap(&tmK, p.k, tokens, G, p.N, p.ldk, kDc, 64, true) ||
      tc_tokens_tmap(&tmV, p.v, tokens, p.H, p.V, p.ldv, kDc, 128, false) || tc_tokens_tmap(&tmO, p.out, tokens, p.H, p.V, p.ldo, kDc, 128, false))
    return -261;
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_delta_prep_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem1));
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_delta_chunk_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2));
    attr = true;
  }
  mix_delta_prep_kernel<NB><<<dim3(total_chunks, G), kDpThreads, smem1, st>>>(p, work, gates, err);
  PRL_CUDA_CHECK(cudaGetLastError());
  mix_delta_chunk_kernel<NB><<<dim3((p.V + 127) / 128, p.H, p.spans), kDcThreads, smem2, st>>>(tmQ, tmK, tmV, tmO, p, work, gates, err);
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
// tokens: rows of q, k and v; chunks: prl_mix_delta_chunks; work: chunks * H * work_bytes, gates: chunks * H * gate_floats, both 16-byte aligned; *err becomes 1 when
// a wait inside a kernel timed out
extern "C" int prl_mix_delta(const ScanParams* p, int64_t tokens, int64_t chunks, void* work, float* gates, int32_t* err, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || chunks > 0x7fffffff || !prl_mix_delta_ok(p->q, p->ldq, p->k, p->ldk, p->v, p->ldv, p->N, p->V)) return -260;
  uint8_t* wk = static_cast<uint8_t*>(work);
  return p->N <= 64 ? run_delta<1>(*p, tokens, static_cast<int>(chunks), wk, gates, err, st) : run_delta<2>(*p, tokens, static_cast<int>(chunks), wk, gates, err, st);
}
