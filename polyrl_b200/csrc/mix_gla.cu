// polyrl_b200 — gated linear attention (a decay for every key channel) over prompt portions on tcgen05 / TMEM (bf16, 64 tokens per chunk).
//
// The recurrence is kGla of mix_scan.cu.  With G_t the running sum of log keep inside a chunk (a vector over the channels), S_0 the state ahead
// of it and C its last token:
//     y_t = S_0^T (q_t e^G_t) + sum_{s <= t} P_ts v_s,      P_ts = sum_n q_tn k_sn e^(G_tn - G_sn)
//     S   = diag(e^G_C) S_0 + sum_s (k_s e^(G_C - G_s)) v_s^T
// The decays act inside the sum over channels, so P is no product of q and k; taken apart at the chunk's start, e^(-G_s) may overflow.
//
// mix_gla_prep_kernel   one CTA per (chunk, head), everything that does not depend on the state.  Blocks of 16 tokens: q relative to its own
//                       block's start, k relative to its own block's end, the blocks between them as a factor per channel, so that every factor is
//                       <= 1; for pairs inside a block the factor is e^(-block's decay), and a block that decays by more than 2^-100 in some channel is
//                       computed pair by pair instead.  P by fp32 FMAs.  Leaves q e^G, k e^(G_C - G) and P as bf16 pairs hi + lo, laid out as
//                       the swizzled tiles the next kernel copies, and e^G_C.
// mix_gla_chunk_kernel  one CTA per (span, head, 128 value columns) marching over its chunks, transposed so that the value columns are the 128 rows
//                       (TMEM lane = value column):  Y^T = V^T P^T + S_0^T (q e^G)^T,   D^T = V^T (k e^(G_C - G)),   S = diag(e^G_C) S_0 + D.
//                       V^T P^T and D do not wait for the state: they run while the state ahead of the chunk is still being made.  The fp32 state
//                       lives in registers, thread (value column, half) owning half of the state rows, and is staged into TMEM as a pair
//                       hi + lo once per chunk.  Warps 0-7 do that and the outputs; warp 8 issues the products, warp 9 the stores, warp 10 the loads.
// Every wait is bounded: on a timeout the CTA raises *err, runs out its chunks without waiting, loading or multiplying, frees its TMEM and returns.
#include "mix_tc.cuh"

namespace prl {

constexpr int kGc = 64, kGb = 16;              // tokens per chunk, per block
constexpr int kGTile = 64 * 128;               // bytes of a 64 x 64 bf16 tile
constexpr float kGFar = 100.f;                 // log2 of the strongest decay over a block that the factored form takes
template <int NB>
struct GlaWork {                               // bytes of a (chunk, head): q hi, q lo, k hi, k lo (NB tiles each), P hi, P lo
  static constexpr int K = 2 * NB * kGTile, P = 4 * NB * kGTile, SIZE = (4 * NB + 2) * kGTile;
};

__device__ __forceinline__ int gla_chunk_base(const int32_t* cu, int s) { return cu[s] / kGc + s; }      // workspace rows of a span start here

template <int NB>
__global__ void __launch_bounds__(NB * 128, NB == 2 ? 2 : 4) mix_gla_prep_kernel(ScanParams p, uint8_t* work, float* keep) {
  constexpr int THREADS = NB * 128, N = NB * 64, LD = N + 4, SLOTS = THREADS / 16, PLD = kGc + 4;
  extern __shared__ float sh[];
  float *sq = sh, *sk = sq + kGc * LD;         // q relative to its block's start, k relative to its block's end
  float* sf = sk + kGc * LD;                   // factors between blocks: [4] own block, [3] (2, 0), (3, 1), (3, 0)
  float* st = sf + 7 * N;                      // [4] decay of a block, log2
  float* sp = NB == 2 ? sh : st + 4 * N;       // P; NB = 2: over q, once that is read
  __shared__ int s_span, s_far[4];
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
  if (tid == 0) {                                                      // the span whose workspace rows hold b
    int lo = 0, hi = p.spans - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (gla_chunk_base(p.cu, mid) <= b) lo = mid; else hi = mid - 1;
    }
    s_span = lo;
  }
  if (tid < 4) s_far[tid] = 0;
  __syncthreads();
  const int s = s_span, c0 = (b - gla_chunk_base(p.cu, s)) * kGc, nv = min(kGc, p.cu[s + 1] - p.cu[s] - c0);
  if (nv <= 0) return;
  const int64_t t0 = p.cu[s] + c0, item = static_cast<int64_t>(b) * p.H + h;
  uint8_t* out = work + item * GlaWork<NB>::SIZE;
  // thread: 16 tokens of block J, two neighbouring channels
  const int J = w / NB, half = w % NB, c = half * 64 + 2 * lane;
  const bool on = c < p.N;                                             // (N is even)
  float l[kGb][2];                                                     // log2 of keep, summed from the block's start
  uint32_t q[kGb], k[kGb];
  auto load = [&]() {
    const float bx = on && p.b0 ? p.b0[h * p.N + c] : 0.f, by = on && p.b0 ? p.b0[h * p.N + c + 1] : 0.f;
    const float* gz = p.g0 + static_cast<int64_t>(h) * p.N + c;
    const __nv_bfloat16 *gq = static_cast<const __nv_bfloat16*>(p.q) + static_cast<int64_t>(h / p.rep) * p.N + c,
                        *gk = static_cast<const __nv_bfloat16*>(p.k) + static_cast<int64_t>(h / p.rep) * p.N + c;
    const float f = 1.4426950408889634f / p.cap;
#pragma unroll
    for (int i = 0; i < kGb; ++i) {
      const int t = J * kGb + i;
      const bool in = on && t < nv;
      const int64_t row = t0 + (in ? t : 0);
      const float2 z = in ? *reinterpret_cast<const float2*>(gz + row * p.ldg) : make_float2(0.f, 0.f);
      l[i][0] = z.x + bx;
      l[i][1] = z.y + by;
      q[i] = in ? *reinterpret_cast<const uint32_t*>(gq + row * p.ldq) : 0u;
      k[i] = in ? *reinterpret_cast<const uint32_t*>(gk + row * p.ldk) : 0u;
    }
    float run[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < kGb; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (on && J * kGb + i < nv) run[e] -= softplus_series(-l[i][e]) * f;       // log2 of sigmoid^(1 / tau)
        l[i][e] = run[e];
      }
  };
  load();
  const float T[2] = {l[kGb - 1][0], l[kGb - 1][1]};
  *reinterpret_cast<float2*>(st + J * N + c) = make_float2(T[0], T[1]);
  if (fminf(T[0], T[1]) < -kGFar) s_far[J] = 1;
  __syncthreads();
  float before[2], behind[2];                                          // e^ of the blocks ahead of, behind this one
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    float t[4], lo = 0.f, hi = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) t[j] = st[j * N + c + e];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j < J) lo += t[j];
      if (j > J) hi += t[j];
    }
    before[e] = fast_exp2(lo);
    behind[e] = fast_exp2(hi);
    sf[J * N + c + e] = fast_exp2(fminf(-T[e], kGFar));                // (a far block does not use its own)
    if (J == 0) {
      sf[4 * N + c + e] = fast_exp2(t[1]);
      sf[5 * N + c + e] = fast_exp2(t[2]);
      sf[6 * N + c + e] = fast_exp2(t[1] + t[2]);
      keep[item * N + c + e] = fast_exp2((t[0] + t[1]) + (t[2] + t[3]));
    }
  }
#pragma unroll
  for (int i = 0; i < kGb; ++i) {
    const int t = J * kGb + i;
    const float2 a = unpack_bf16(q[i]), e = unpack_bf16(k[i]);
    const float qx = a.x * (p.qscale * fast_exp2(l[i][0])), qy = a.y * (p.qscale * fast_exp2(l[i][1]));
    const float kx = e.x * fast_exp2(T[0] - l[i][0]), ky = e.y * fast_exp2(T[1] - l[i][1]);
    *reinterpret_cast<float2*>(sq + t * LD + c) = make_float2(qx, qy);
    *reinterpret_cast<float2*>(sk + t * LD + c) = make_float2(kx, ky);
    uint8_t* dst = out + half * kGTile + t * 128 + (((lane >> 2) ^ (t & 7)) << 4) + (lane & 3) * 4;
    uint32_t hi, lo;
    tc_split(qx * before[0], qy * before[1], hi, lo);
    *reinterpret_cast<uint32_t*>(dst) = hi;
    *reinterpret_cast<uint32_t*>(dst + NB * kGTile) = lo;
    tc_split(kx * behind[0], ky * behind[1], hi, lo);
    *reinterpret_cast<uint32_t*>(dst + GlaWork<NB>::K) = hi;
    *reinterpret_cast<uint32_t*>(dst + GlaWork<NB>::K + NB * kGTile) = lo;
  }
  __syncthreads();
  // P: 16 threads per pair of blocks, four rows and four columns each, a quarter of a block apart
  const int slot = tid >> 4, ti = (tid >> 2) & 3, tj = tid & 3;
  constexpr int ITER = (10 + SLOTS - 1) / SLOTS;
  float acc[ITER][4][4];
  auto row_block = [](int pr) { return pr < 4 ? pr : pr == 4 ? 2 : pr <= 6 ? 3 : pr - 6; };               // (0,0) .. (3,3), (2,0), (3,1), (3,0),
  auto col_block = [](int pr) { return pr < 4 ? pr : pr == 4 ? 0 : pr == 5 ? 1 : pr == 6 ? 0 : pr - 7; };  // (1,0), (2,1), (3,2)
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int pr = slot + it * SLOTS;
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y) acc[it][x][y] = 0.f;
    if (pr >= 10) continue;
    const float *rq = sq + (row_block(pr) * kGb + ti) * LD, *rk = sk + (col_block(pr) * kGb + tj) * LD, *rf = sf + pr * N;
#pragma unroll 1
    for (int n = 0; n < N; n += 4) {
      float4 a[4], e[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        a[x] = *reinterpret_cast<const float4*>(rq + x * 4 * LD + n);
        e[x] = *reinterpret_cast<const float4*>(rk + x * 4 * LD + n);
      }
      if (pr < 7) {
        const float4 f = *reinterpret_cast<const float4*>(rf + n);
#pragma unroll
        for (int x = 0; x < 4; ++x) { a[x].x *= f.x; a[x].y *= f.y; a[x].z *= f.z; a[x].w *= f.w; }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[it][x][y] += (a[x].x * e[y].x + a[x].y * e[y].y) + (a[x].z * e[y].z + a[x].w * e[y].w);
    }
  }
  __syncthreads();
  if (s_far[0] | s_far[1] | s_far[2] | s_far[3]) {                     // pair by pair: q, k and the running sums themselves
    if (s_far[J]) {
      load();
#pragma unroll
      for (int i = 0; i < kGb; ++i) {
        const int t = J * kGb + i;
        *reinterpret_cast<float2*>(sq + t * LD + c) = make_float2(l[i][0], l[i][1]);
        *reinterpret_cast<uint2*>(sk + t * LD + c) = make_uint2((q[i] & 0xffffu) | k[i] << 16, q[i] >> 16 | (k[i] & 0xffff0000u));
      }
    }
    __syncthreads();
    if (slot < 4 && s_far[slot]) {
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) {
          const int i = slot * kGb + ti + 4 * x, j = slot * kGb + tj + 4 * y;
          float sum = 0.f;
          if (j <= i) {
            for (int n = 0; n < N; ++n) {
              const float a = unpack_bf16(reinterpret_cast<const uint32_t*>(sk)[i * LD + n]).x, e = unpack_bf16(reinterpret_cast<const uint32_t*>(sk)[j * LD + n]).y;
              sum += a * e * fast_exp2(sq[i * LD + n] - sq[j * LD + n]);
            }
          }
          acc[0][x][y] = sum * p.qscale;
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int pr = slot + it * SLOTS;
    if (pr < 10) {
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) sp[(row_block(pr) * kGb + ti + 4 * x) * PLD + col_block(pr) * kGb + tj + 4 * y] = acc[it][x][y];
    }
  }
  __syncthreads();
  for (int r = w; r < kGc; r += THREADS / 32) {
    const float2 x = *reinterpret_cast<const float2*>(sp + r * PLD + 2 * lane);
    uint32_t hi, lo;
    tc_split(2 * lane <= r ? x.x : 0.f, 2 * lane + 1 <= r ? x.y : 0.f, hi, lo);
    uint8_t* dst = out + GlaWork<NB>::P + r * 128 + (((lane >> 2) ^ (r & 7)) << 4) + (lane & 3) * 4;
    *reinterpret_cast<uint32_t*>(dst) = hi;
    *reinterpret_cast<uint32_t*>(dst + kGTile) = lo;
  }
}

template <int NB>
struct GlaTc {
  static constexpr int VT = 2 * kGTile;                      // 64 tokens x 128 value columns
  static constexpr int STAGE = GlaWork<NB>::SIZE + VT;       // the workspace of a chunk, then V
  static constexpr int OFF_O = 2 * STAGE;                    // outputs, plain rows
  static constexpr int OFF_F = OFF_O + VT;
};
template <int NB>
struct GlaShared {                                           // behind the tiles
  float keep[3][NB * 64];                                    // (a chunk's keeps are read while the chunk after the next one loads)
  uint64_t full[2], delta[2], own[2], taken[2], stored;      // chunk arrived; products done: D, Y; Y read by the threads; its rows are on their way
  uint32_t tmem;
  int fail;
};
enum : int { kBarGlaState = 1, kBarGlaOut = 2 };             // warps 0-7 hand over to warp 8 (state) and warp 9 (outputs)
constexpr int kGlaHandoff = 288, kGlaThreads = 352;

__device__ __forceinline__ void gla_arrive(int id) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "n"(kGlaHandoff) : "memory"); }
__device__ __forceinline__ void gla_sync(int id) { asm volatile("bar.sync %0, %1;" ::"r"(id), "n"(kGlaHandoff) : "memory"); }
template <class Sm>
__device__ __forceinline__ bool gla_failed(Sm& sm) { return *reinterpret_cast<volatile int*>(&sm.fail) != 0; }
template <class Sm>
__device__ __forceinline__ void gla_wait(Sm& sm, uint64_t* bar, uint32_t parity) {
  if (gla_failed(sm)) return;
  if (!tc_wait(bar, parity)) *reinterpret_cast<volatile int*>(&sm.fail) = 1;
}

template <int NB>
__global__ void __launch_bounds__(kGlaThreads, 1)
mix_gla_chunk_kernel(const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmO, ScanParams p, const uint8_t* work, const float* keep, int32_t* err) {
  using Cfg = GlaTc<NB>;
  constexpr int OWN = NB * 32, NN = NB * 64;                 // state rows per thread, of the operand
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sO = smem + Cfg::OFF_O;
  GlaShared<NB>& sm = *reinterpret_cast<GlaShared<NB>*>(smem + Cfg::OFF_F);
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * 128;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int N = p.N, V = p.V, vn = min(128, V - v0);
  const int chunks = (len + kGc - 1) / kGc;
  if (tid == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sm.full[i], 1);
      mbar_init(&sm.delta[i], 1);
      mbar_init(&sm.own[i], 1);
      mbar_init(&sm.taken[i], 256);
    }
    mbar_init(&sm.stored, 1);
    sm.fail = 0;
    fence_barrier_init();
  }
  if (w == 8) { tmem_alloc(&sm.tmem, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // TMEM columns: state operand (of half g: hi at tS + g * OWN, lo behind it), outputs of two chunks, increments of two chunks
  const uint32_t tS = sm.tmem, tO = tS + 128, tD = tS + 256;

  if (w == 8) {
    // ================================ products ================================
    constexpr uint32_t idO = umma_idesc_major(128, kGc, 1, 1, 1, 0), idS = umma_idesc(128, kGc, 1, 1), idD = umma_idesc_major(128, NN, 1, 1, 1, 1);
    for (int ci = 0; ci < chunks; ++ci) {
      const int bf = ci & 1;
      uint8_t *sW = smem + bf * Cfg::STAGE, *sV = sW + GlaWork<NB>::SIZE;
      if (lane == 0) {
        gla_wait(sm, &sm.full[bf], (ci >> 1) & 1);
        if (ci >= 2) gla_wait(sm, &sm.taken[bf], ((ci >> 1) & 1) ^ 1);
      }
      __syncwarp();
      const int nv = len - ci * kGc;
      if (nv < kGc) {                                        // the tile's last rows are another span's values
        for (int i = lane; i < (kGc - nv) * 16; i += 32)
          *reinterpret_cast<uint4*>(sV + (i & 15) / 8 * kGTile + (nv + i / 16) * 128 + (i & 7) * 16) = make_uint4(0, 0, 0, 0);
        fence_proxy_async();
      }
      __syncwarp();
      if (lane == 0 && !gla_failed(sm)) {
        tc_fence_after();
        const uint64_t dv = umma_desc_sw128_mnmajor(sV, kGTile);
        const uint64_t dp = umma_desc_sw128_kmajor(sW + GlaWork<NB>::P), dk = umma_desc_sw128_mnmajor(sW + GlaWork<NB>::K, kGTile);
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_bf16_ss(tD + bf * 128, dv + kk * 128, dk + hl * (NB * kGTile >> 4) + kk * 128, idD, (hl | kk) != 0);
        umma_commit(&sm.delta[bf]);
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_bf16_ss(tO + bf * kGc, dv + kk * 128, dp + hl * (kGTile >> 4) + 2 * kk, idO, (hl | kk) != 0);
      }
      __syncwarp();
      gla_sync(kBarGlaState);
      if (lane == 0 && !gla_failed(sm)) {
        tc_fence_after();
        if (ci > 0 || !fresh) {
          const uint64_t dq = umma_desc_sw128_kmajor(sW);
#pragma unroll
          for (int kk = 0; kk < NB * 4; ++kk) {
            const uint32_t a = tS + (kk * 16 / OWN) * OWN + (kk * 16 % OWN) / 2;
            const uint64_t b = dq + (kk >> 2) * (kGTile >> 4) + 2 * (kk & 3);
            umma_bf16_ts(tO + bf * kGc, a, b, idS, 1);
            umma_bf16_ts(tO + bf * kGc, a + OWN / 2, b, idS, 1);
            umma_bf16_ts(tO + bf * kGc, a, b + (NB * kGTile >> 4), idS, 1);
          }
        }
        umma_commit(&sm.own[bf]);
      }
      __syncwarp();
    }
  } else if (w == 9) {
    // ================================ stores ================================
    __nv_bfloat16* gO = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(t0) * p.ldo + static_cast<int64_t>(h) * V + v0;
    for (int ci = 0; ci < chunks; ++ci) {
      gla_sync(kBarGlaOut);
      const int nv = len - ci * kGc;
      if (!gla_failed(sm)) {
        if (nv >= kGc) {
          if (lane == 0) tma_store_3d(&tmO, sO, v0, h, t0 + ci * kGc);
        } else {                                             // a row at a time: the next rows are another span's
          for (int t = lane; t < nv; t += 32) bulk_store(gO + (static_cast<int64_t>(ci) * kGc + t) * p.ldo, sO + t * 256, vn * 2);
        }
        tma_store_commit();
        tma_store_wait_read<0>();
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&sm.stored);
    }
    tma_store_wait<0>();
  } else if (w == 10) {
    // ================================ loads ================================
    if (lane == 0) {
      const int64_t item0 = static_cast<int64_t>(gla_chunk_base(p.cu, s)) * p.H + h;
      tma_prefetch_desc(&tmV);
      int loaded = 0;
      for (int ci = 0; ci < chunks; ++ci) {
        const int bf = ci & 1, t = t0 + ci * kGc;
        const int64_t item = item0 + static_cast<int64_t>(ci) * p.H;
        uint8_t* sW = smem + bf * Cfg::STAGE;
        if (ci >= 2) gla_wait(sm, &sm.own[bf], ((ci >> 1) & 1) ^ 1);     // the last reader of the buffer
        if (gla_failed(sm)) break;
        uint64_t* bar = &sm.full[bf];
        mbar_expect_tx(bar, Cfg::STAGE + NN * 4);
        tma_load_3d(&tmV, bar, sW + GlaWork<NB>::SIZE, v0, h, t);
        tma_load_3d(&tmV, bar, sW + GlaWork<NB>::SIZE + kGTile, v0 + 64, h, t);
        bulk_load(bar, sm.keep[ci % 3], keep + item * NN, NN * 4);
        bulk_load(bar, sW, work + item * GlaWork<NB>::SIZE, GlaWork<NB>::SIZE);
        loaded = ci + 1;
      }
      if (gla_failed(sm)) {                                  // copies in flight end before the shared memory is given up
        if (loaded > 0) tc_wait(&sm.full[0], ((loaded + 1) / 2 - 1) & 1);
        if (loaded > 1) tc_wait(&sm.full[1], (loaded / 2 - 1) & 1);
      }
    }
    __syncwarp();
  } else {
    // ================================ warps 0-7: state and outputs ================================
    const int quad = w & 3, g = w >> 2, r = quad * 32 + lane;          // value column, half of the state rows or tokens
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    float* gS = p.S + (p.slot[s] * p.H + h) * static_cast<int64_t>(N) * V + v0 + r;
    float S[OWN];                                            // state rows g * OWN + i
#pragma unroll
    for (int i = 0; i < OWN; ++i) {
      const int n = g * OWN + i;
      S[i] = (!fresh && n < N && r < vn) ? gS[static_cast<int64_t>(n) * V] : 0.f;
    }
    auto stage_state = [&]() {
#pragma unroll
      for (int c = 0; c < OWN; c += 32) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) tc_split(S[c + 2 * e], S[c + 2 * e + 1], hi[e], lo[e]);
        __syncwarp();
        tmem_st_32x16(tS + lanes + g * OWN + c / 2, hi);
        tmem_st_32x16(tS + lanes + g * OWN + OWN / 2 + c / 2, lo);
      }
      tmem_st_wait();
    };
    if (!fresh) stage_state();
    tc_fence_before();
    gla_arrive(kBarGlaState);
    for (int ci = 0; ci < chunks; ++ci) {
      const int bf = ci & 1;
      const uint32_t ph = (ci >> 1) & 1;
      gla_wait(sm, &sm.full[bf], ph);                        // (its keeps)
      gla_wait(sm, &sm.delta[bf], ph);
      tc_fence_after();
      const float* kp = sm.keep[ci % 3] + g * OWN;
#pragma unroll
      for (int c = 0; c < OWN; c += 32) {
        uint32_t d[32];
        __syncwarp();
        tmem_ld_32x32(tD + bf * 128 + lanes + g * OWN + c, d);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          const float4 f = *reinterpret_cast<const float4*>(kp + c + i);
          S[c + i] = f.x * S[c + i] + __uint_as_float(d[i]);
          S[c + i + 1] = f.y * S[c + i + 1] + __uint_as_float(d[i + 1]);
          S[c + i + 2] = f.z * S[c + i + 2] + __uint_as_float(d[i + 2]);
          S[c + i + 3] = f.w * S[c + i + 3] + __uint_as_float(d[i + 3]);
        }
      }
      gla_wait(sm, &sm.own[bf], ph);                         // the operand's last reader; Y is complete
      tc_fence_after();
      if (ci + 1 < chunks) {
        stage_state();
        tc_fence_before();
        gla_arrive(kBarGlaState);
      }
      uint32_t y[32];
      __syncwarp();
      tmem_ld_32x32(tO + bf * kGc + lanes + g * 32, y);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&sm.taken[bf]);
      if (ci > 0) gla_wait(sm, &sm.stored, (ci & 1) ^ 1);
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(sO) + g * 32 * 128 + r;
#pragma unroll
      for (int i = 0; i < 32; ++i) dst[i * 128] = __float2bfloat16(__uint_as_float(y[i]));
      fence_proxy_async();
      gla_arrive(kBarGlaOut);
    }
    if (!gla_failed(sm) && r < vn) {
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
  if (tid == 0 && gla_failed(sm)) atomicExch(err, 1);
  if (w == 8) { tc_fence_after(); tmem_dealloc(sm.tmem, 512); }
}

template <int NB>
static int run_gla(const ScanParams& p, int64_t tokens, int total_chunks, uint8_t* work, float* keep, int32_t* err, cudaStream_t st) {
  constexpr int N = NB * 64, smem1 = (2 * kGc * (N + 4) + 11 * N + (NB == 2 ? 0 : kGc * (kGc + 4))) * 4;
  constexpr int smem2 = GlaTc<NB>::OFF_F + static_cast<int>(sizeof(GlaShared<NB>)) + 1024;
  static_assert(smem2 <= 232448, "shared memory");
  CUtensorMap tmV, tmO;
  if (tc_tokens_tmap(&tmV, p.v, tokens, p.H, p.V, p.ldv, kGc, 64, true) || tc_tokens_tmap(&tmO, p.out, tokens, p.H, p.V, p.ldo, kGc, 128, false)) return -311;
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_gla_prep_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem1));
    PRL_CUDA_CHECK(cudaFuncSetAttribute(mix_gla_chunk_kernel<NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2));
    attr = true;
  }
  mix_gla_prep_kernel<NB><<<dim3(total_chunks, p.H), NB * 128, smem1, st>>>(p, work, keep);
  PRL_CUDA_CHECK(cudaGetLastError());
  mix_gla_chunk_kernel<NB><<<dim3((p.V + 127) / 128, p.H, p.spans), kGlaThreads, smem2, st>>>(tmV, tmO, p, work, keep, err);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

// at most 128 state rows, an even number; neighbouring channels of q, k and the gates in one aligned word; 16-byte aligned rows of v, heads of 8 columns
extern "C" int prl_mix_gla_ok(const ScanParams* p) {
  auto al = [](const void* x, int bytes) { return (reinterpret_cast<uintptr_t>(x) & (bytes - 1)) == 0; };
  return p->N % 2 == 0 && p->N <= 128 && p->V % 8 == 0 && al(p->q, 4) && al(p->k, 4) && p->ldq % 2 == 0 && p->ldk % 2 == 0 && al(p->g0, 8) && p->ldg % 2 == 0 &&
         al(p->v, 16) && p->ldv % 8 == 0 && al(p->out, 16) && p->ldo % 8 == 0 && p->qscale != 0.f;
}
extern "C" int64_t prl_mix_gla_chunks(int64_t tokens, int64_t spans) { return tokens / kGc + spans; }
extern "C" int64_t prl_mix_gla_work_bytes(int N) { return N <= 64 ? GlaWork<1>::SIZE : GlaWork<2>::SIZE; }
extern "C" int64_t prl_mix_gla_keep_floats(int N) { return N <= 64 ? 64 : 128; }
// tokens: rows of q, k and v; chunks: prl_mix_gla_chunks; work: chunks * H * work_bytes, keep: chunks * H * keep_floats, both 16-byte aligned; *err becomes 1
// when a wait inside a kernel timed out
extern "C" int prl_mix_gla(const ScanParams* p, int64_t tokens, int64_t chunks, void* work, float* keep, int32_t* err, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || chunks > 0x7fffffff || !prl_mix_gla_ok(p)) return -310;
  uint8_t* wk = static_cast<uint8_t*>(work);
  return p->N <= 64 ? run_gla<1>(*p, tokens, static_cast<int>(chunks), wk, keep, err, st) : run_gla<2>(*p, tokens, static_cast<int>(chunks), wk, keep, err, st);
}
