// polyrl_b200 — gated linear recurrences over prompt portions on tcgen05 / TMEM (bf16 activations, 128 tokens per chunk).
//
// Same algebra and the same exactness choices as mix_chunk.cu (bf16 pairs hi + lo for weighted scores, weighted values and
// the state as an operand; the state itself in fp32).  One CTA = one (span, head, 64 value columns) marching over its chunks:
//     scores  = Q K^T                     both K-major
//     carried = Q S_0                     S_0 as an MN-major B operand (rows = state rows)
//     own     = (weight . scores) V       scores written K-major by the threads, V MN-major
//     delta   = K^T (weighted V)          K read MN-major from the very tile the scores read K-major
// Accumulators live in TMEM (thread = TMEM lane = token or state row); the fp32 state lives in registers, thread (row, half)
// owning 32 columns per 128 state rows, and is restaged as the hi + lo operand once per chunk.  All tiles are 128-row x
// 64-column 128B-swizzled chunks filled by cp.async (zero beyond the span, the head size and the value columns).
//
// Shared memory: NB chunks of 64 state columns.  NB = 2 (N <= 128) keeps Q, the scores and two K tiles side by side, so every
// load of the next chunk is in flight during this one; NB = 4 (N <= 256) overlays the scores on Q.
// Every wait is bounded: on a timeout the CTA raises *err, stops computing, frees its TMEM and returns.
#include "mix_tc.cuh"

namespace prl {

constexpr int kTcC = 128;               // tokens per chunk
constexpr int kTcThreads = 256;
constexpr int kTcTile = 128 * 128;      // bytes of a 128 x 64 bf16 chunk

template <int NB>
struct ChunkTc {
  static constexpr int MB = NB / 2;                                   // 128-row blocks of the state
  static constexpr int KBUF = NB == 2 ? 2 : 1;
  static constexpr int QB = NB * kTcTile;
  static constexpr int P_BYTES = 4 * kTcTile;                         // scores: hi (2 chunks) + lo (2 chunks)
  static constexpr int OFF_K = QB + (NB == 2 ? P_BYTES : 0);
  static constexpr int OFF_P = NB == 2 ? QB : 0;
  static constexpr int OFF_V = OFF_K + KBUF * QB;
  static constexpr int OFF_S = OFF_V + kTcTile;                       // hi: MB tiles, lo: MB tiles
  static constexpr int OFF_F = OFF_S + 2 * MB * kTcTile;
  static constexpr int SMEM = OFF_F + 11264 + 1024;
};

struct alignas(16) TcGates {                       // weights of one chunk
  float row[kTcC], col[kTcC], mul[kTcC], carry[kTcC], wgt[kTcC], flo[kTcC];
  float keep;
};
static_assert(sizeof(TcGates) % 16 == 0, "both copies are read as float4");
struct TcShared {                        // behind the tiles
  TcGates gate[2];
  float den[2][kTcC], deni[2][kTcC], half[2][kTcC];
  float n[256];
  float m;
  uint64_t bar[4];
  uint32_t tmem;
};

// one 128 x 64 chunk: rows [0, nv) x columns [c0, c0 + 64) of src (columns below n), zero elsewhere
__device__ __forceinline__ void tc_load(uint8_t* dst, const __nv_bfloat16* src, int64_t ld, int nv, int c0, int n) {
  tc_load_rows<128, kTcThreads>(dst, src, ld, nv, c0, n);
}

// raw gate values of the lane's four tokens (4 lane, ...) of a chunk
struct TcRaw { float a[4], b[4]; };
template <int MODE>
__device__ __forceinline__ void tc_raw(TcRaw& g, const ScanParams& p, int64_t t0, int nv, int h, int lane) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int t = 4 * lane + e;
    const bool ok = t < nv;
    g.a[e] = ok && MODE != kDecay ? p.g0[(t0 + t) * p.ldg + h] : 0.f;
    g.b[e] = (ok && MODE == kMlstm) ? p.g1[(t0 + t) * p.ldg + h] : 0.f;
  }
}
// one warp: weights of the chunk.  weight(t, s) = 2^(row_t + col_s) mul_s (qscale folded into row), carry: carried-in factor with
// qscale, wgt: weight of a token in the chunk's final state
template <int MODE>
__device__ __forceinline__ void tc_gates(TcGates& sm, float& m_run, const TcRaw& g, const ScanParams& p, int nv, int h, float b0, float b1, float a_neg, int lane) {
  constexpr float kL2e = 1.4426950408889634f;
  const float lq = log2f(p.qscale);
  float la[4], ad[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const bool ok = 4 * lane + e < nv;
    if (MODE == kDecay) {
      ad[e] = ok ? 1.f : 0.f;
      la[e] = ok ? p.a_log[h] : 0.f;
    } else if (MODE == kSsd) {
      ad[e] = ok ? softplus_f(g.a[e] + b0) : 0.f;
      la[e] = a_neg * ad[e];
    } else {
      ad[e] = ok ? softcap_f(g.a[e] + b0, p.cap) : -INFINITY;
      la[e] = ok ? logsigmoid_f(softcap_f(g.b[e] + b1, p.cap)) : 0.f;
    }
    if (e) la[e] += la[e - 1];
  }
  float run = la[3];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += x;
  }
  const float before = __shfl_up_sync(0xffffffffu, run, 1);
  const float end = __shfl_sync(0xffffffffu, run, 31);
#pragma unroll
  for (int e = 0; e < 4; ++e) la[e] += lane ? before : 0.f;
  if (MODE != kMlstm) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = 4 * lane + e;
      sm.row[t] = la[e] * kL2e + lq;
      sm.col[t] = -la[e] * kL2e;
      sm.mul[t] = ad[e];
      sm.carry[t] = expf(la[e]) * p.qscale;
      sm.wgt[t] = expf(end - la[e]) * ad[e];
    }
    if (lane == 0) sm.keep = expf(end);
  } else {
    float mx[4], gg[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      gg[e] = ad[e] - la[e];
      mx[e] = e ? fmaxf(mx[e - 1], gg[e]) : gg[e];
    }
    float rm = mx[3];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, rm, o);
      if (lane >= o) rm = fmaxf(rm, x);
    }
    const float m0 = m_run;
    const float pm = __shfl_up_sync(0xffffffffu, rm, 1);
    const float base = lane ? fmaxf(pm, m0) : m0;
    const float m_end = fmaxf(__shfl_sync(0xffffffffu, rm, 31), m0);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = 4 * lane + e;
      const float M = fmaxf(mx[e], base);
      sm.row[t] = -M * kL2e + lq;
      sm.col[t] = gg[e] * kL2e;
      sm.mul[t] = 1.f;
      sm.carry[t] = expf(m0 - M) * p.qscale;
      sm.wgt[t] = expf(gg[e] - m_end);
      sm.flo[t] = expf(-(la[e] + M));
    }
    __syncwarp();
    if (lane == 0) { sm.keep = expf(m0 - m_end); m_run = end + m_end; }
  }
}

template <int MODE, int NB>
__global__ void __launch_bounds__(kTcThreads, 1)
mix_chunk_tc_kernel(ScanParams p, int32_t* err) {
  using Cfg = ChunkTc<NB>;
  constexpr int MB = Cfg::MB, QB = Cfg::QB;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *sQ = smem, *sV = smem + Cfg::OFF_V, *sP = smem + Cfg::OFF_P, *sS = smem + Cfg::OFF_S;
  TcShared& sm = *reinterpret_cast<TcShared*>(smem + Cfg::OFF_F);
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * 64;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31;
  const int quad = w & 3, g = w >> 2, r = quad * 32 + lane;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int64_t slot = p.slot[s];
  const int N = p.N, V = p.V, vn = min(64, V - v0);
  const __nv_bfloat16* gQ = static_cast<const __nv_bfloat16*>(p.q) + static_cast<int64_t>(t0) * p.ldq + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gK = static_cast<const __nv_bfloat16*>(p.k) + static_cast<int64_t>(t0) * p.ldk + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gV = static_cast<const __nv_bfloat16*>(p.v) + static_cast<int64_t>(t0) * p.ldv + static_cast<int64_t>(h) * V + v0;
  __nv_bfloat16* gO = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(t0) * p.ldo + static_cast<int64_t>(h) * V + v0;
  float* gS = p.S + (slot * p.H + h) * static_cast<int64_t>(N) * V + v0;
  const float b0 = p.b0 ? p.b0[h] : 0.f, b1 = p.b1 ? p.b1[h] : 0.f;
  const float a_neg = MODE == kSsd ? -expf(p.a_log[h]) : 0.f;
  const float skip = (MODE == kSsd && p.d_skip) ? p.d_skip[h] : 0.f;

  auto load_q = [&](int c, int lo, int hi) {
    const int nv = min(kTcC, len - c);
    for (int i = lo; i < hi; ++i) tc_load(sQ + i * kTcTile, gQ + static_cast<int64_t>(c) * p.ldq, p.ldq, nv, i * 64, N);
  };
  auto load_k = [&](int c, int buf) {
    const int nv = min(kTcC, len - c);
    for (int i = 0; i < NB; ++i) tc_load(smem + Cfg::OFF_K + buf * QB + i * kTcTile, gK + static_cast<int64_t>(c) * p.ldk, p.ldk, nv, i * 64, N);
  };
  auto load_v = [&](int c) { tc_load(sV, gV + static_cast<int64_t>(c) * p.ldv, p.ldv, min(kTcC, len - c), 0, vn); };

  load_q(0, 0, NB);
  load_k(0, 0);
  load_v(0);
  TcRaw raw;
  if (w == 4) tc_raw<MODE>(raw, p, t0, min(kTcC, len), h, lane);
  if (tid == 0) {
    for (int i = 0; i < 4; ++i) mbar_init(&sm.bar[i], 1);
    fence_barrier_init();
  }
  if (w == 0) { tmem_alloc(&sm.tmem, 512); tmem_relinquish(); }

  // fp32 state: rows mb * 128 + r, columns g * 32 + c
  float S[MB][32];
#pragma unroll
  for (int mb = 0; mb < MB; ++mb) {
    const int n = mb * 128 + r;
#pragma unroll
    for (int c = 0; c < 32; c += 4) {
      float4 q = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && n < N && g * 32 + c < vn) q = *reinterpret_cast<const float4*>(gS + static_cast<int64_t>(n) * V + g * 32 + c);
      S[mb][c] = q.x; S[mb][c + 1] = q.y; S[mb][c + 2] = q.z; S[mb][c + 3] = q.w;
    }
  }
  auto stage_state = [&]() {
#pragma unroll
    for (int mb = 0; mb < MB; ++mb)
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) tc_split(S[mb][u * 8 + 2 * e], S[mb][u * 8 + 2 * e + 1], hi[e], lo[e]);
        tc_st16(sS + mb * kTcTile, r, g * 4 + u, hi);
        tc_st16(sS + (MB + mb) * kTcTile, r, g * 4 + u, lo);
      }
  };
  bool have_state = !fresh;
  if (have_state) stage_state();
  if (MODE == kMlstm) {
    const int64_t hb = slot * p.H + h;
    sm.n[tid] = (!fresh && tid < N) ? p.nst[hb * N + tid] : 0.f;
  }
  if (w == 4) {          // rows 0..31, columns 64..127 of the scores: the warp whose share lies above the diagonal runs the gates, a chunk ahead
    if (MODE == kMlstm && lane == 0) sm.m = fresh ? 0.f : p.mst[slot * p.H + h];
    __syncwarp();
    tc_gates<MODE>(sm.gate[0], sm.m, raw, p, min(kTcC, len), h, b0, b1, a_neg, lane);
    if (len > kTcC) tc_raw<MODE>(raw, p, t0 + kTcC, min(kTcC, len - kTcC), h, lane);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sm.tmem, tS = tmem, tI = tmem + 128, tP = tmem + 192, tD = tmem + 256;
  const uint32_t lane_base = static_cast<uint32_t>(quad * 32) << 16;
  constexpr uint32_t idKK = umma_idesc(128, 128, 1, 1);                         // scores: A, B K-major
  constexpr uint32_t idKM = umma_idesc_major(128, 64, 1, 1, 0, 1);              // A K-major, B MN-major
  constexpr uint32_t idMM = umma_idesc_major(128, 64, 1, 1, 1, 1);              // A, B MN-major
  bool ok = true;
  const int chunks = (len + kTcC - 1) / kTcC;

  for (int ci = 0; ci < chunks; ++ci) {
    const int c0 = ci * kTcC, nv = min(kTcC, len - c0);
    const uint32_t ph = ci & 1;
    const bool more = ci + 1 < chunks;
    const TcGates& gt = sm.gate[ci & 1];
    const uint8_t* sK = smem + Cfg::OFF_K + (Cfg::KBUF == 2 ? (ci & 1) : 0) * QB;
    asm volatile("cp.async.wait_all;" ::: "memory");
    fence_proxy_async();
    __syncthreads();                                                             // tiles and staged state are in place
    if (tid == 0) {
      tc_fence_after();
#pragma unroll
      for (int kk = 0; kk < NB * 4; ++kk)
        umma_bf16_ss(tS, umma_desc_sw128_kmajor(sQ + (kk >> 2) * kTcTile) + 2 * (kk & 3), umma_desc_sw128_kmajor(sK + (kk >> 2) * kTcTile) + 2 * (kk & 3),
                     idKK, kk != 0);
      umma_commit(&sm.bar[0]);
      if (have_state) {
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < NB * 4; ++kk)
            umma_bf16_ss(tI, umma_desc_sw128_kmajor(sQ + (kk >> 2) * kTcTile) + 2 * (kk & 3),
                         umma_desc_sw128_mnmajor(sS + hl * MB * kTcTile, kTcTile) + kk * 128, idKM, (hl | kk) != 0);
      }
      umma_commit(&sm.bar[1]);
    }
    __syncwarp();          // the issuing lane first: its warp must not sit in a wait for products that are not issued yet
    if (Cfg::KBUF == 2 && more) load_k(c0 + kTcC, (ci + 1) & 1);                 // (its last reader finished with the previous chunk)
    if (MODE == kMlstm) {                                                        // n_0 . q_t, half of the columns per thread
      float d0 = 0.f, d1 = 0.f;
      if (have_state) {
#pragma unroll 4
        for (int u = 0; u < NB * 4; ++u) {
          const int uu = g * NB * 4 + u;                                         // 16-byte unit of the row
          const uint4 q = tc_ld16(sQ + (uu >> 3) * kTcTile, r, uu & 7);
          const float* nn = sm.n + uu * 8;
          const float2 a = unpack_bf16(q.x), b = unpack_bf16(q.y), c = unpack_bf16(q.z), d = unpack_bf16(q.w);
          d0 += a.x * nn[0] + a.y * nn[1] + b.x * nn[2] + b.y * nn[3];
          d1 += c.x * nn[4] + c.y * nn[5] + d.x * nn[6] + d.y * nn[7];
        }
      }
      sm.deni[g][r] = d0 + d1;
    }
    if (MODE == kMlstm) __syncthreads();                                         // (the scores may overlay the Q that was just read)
    ok = tc_wait(&sm.bar[0], ph) && ok;
    if (NB == 4) ok = tc_wait(&sm.bar[1], ph) && ok;                             // the scores overlay Q
    tc_fence_after();
    if (w == 4 && more) {
      const int c1 = c0 + kTcC;
      tc_gates<MODE>(sm.gate[(ci + 1) & 1], sm.m, raw, p, min(kTcC, len - c1), h, b0, b1, a_neg, lane);
      if (len > c1 + kTcC) tc_raw<MODE>(raw, p, t0 + c1 + kTcC, min(kTcC, len - c1 - kTcC), h, lane);
    }
    // ---- weighted scores of row r, columns [64 g, +64)
    {
      const float row = gt.row[r];
      float den = 0.f;
#pragma unroll
      for (int c = 0; c < 64; c += 32) {
        uint32_t hi[16], lo[16];
        const int cb = g * 64 + c;
        if (cb <= quad * 32 + 31) {                                              // some column of this block is at or below the diagonal
          uint32_t v[32];
          __syncwarp();
          tmem_ld_32x32(tS + lane_base + cb, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 cc = *reinterpret_cast<const float4*>(&gt.col[cb + i]);
            float x[4] = {__uint_as_float(v[i]) * fast_exp2(row + cc.x), __uint_as_float(v[i + 1]) * fast_exp2(row + cc.y),
                          __uint_as_float(v[i + 2]) * fast_exp2(row + cc.z), __uint_as_float(v[i + 3]) * fast_exp2(row + cc.w)};
            if (MODE == kSsd) {
              const float4 mm = *reinterpret_cast<const float4*>(&gt.mul[cb + i]);
              x[0] *= mm.x; x[1] *= mm.y; x[2] *= mm.z; x[3] *= mm.w;
            }
            if (cb + 31 > quad * 32) {                                           // block on the diagonal
#pragma unroll
              for (int e = 0; e < 4; ++e) x[e] = cb + i + e <= r ? x[e] : 0.f;
            }
            if (MODE == kMlstm) den += (x[0] + x[1]) + (x[2] + x[3]);
            tc_split(x[0], x[1], hi[i / 2], lo[i / 2]);
            tc_split(x[2], x[3], hi[i / 2 + 1], lo[i / 2 + 1]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i) hi[i] = lo[i] = 0u;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const uint32_t a[4] = {hi[4 * u], hi[4 * u + 1], hi[4 * u + 2], hi[4 * u + 3]}, b[4] = {lo[4 * u], lo[4 * u + 1], lo[4 * u + 2], lo[4 * u + 3]};
          tc_st16(sP + g * kTcTile, r, c / 8 + u, a);
          tc_st16(sP + (2 + g) * kTcTile, r, c / 8 + u, b);
        }
      }
      if (MODE == kMlstm) sm.den[g][r] = den;
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
#pragma unroll
      for (int hl = 0; hl < 2; ++hl)
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          umma_bf16_ss(tP, umma_desc_sw128_kmajor(sP + (2 * hl + (kk >> 2)) * kTcTile) + 2 * (kk & 3), umma_desc_sw128_mnmajor(sV, kTcTile) + kk * 128,
                       idKM, (hl | kk) != 0);
      umma_commit(&sm.bar[2]);
    }
    __syncwarp();
    const float keep = gt.keep, wgt = gt.wgt[r];
    if (MODE == kMlstm) {                                                        // n = keep n + sum_s w_s k_s: two state rows, half of the tokens
      float a0 = 0.f, a1 = 0.f;
      const int np = tid & 127, half = tid >> 7, n = 2 * np;
      if (n < NB * 64) {
        const uint8_t* kt = sK + (n >> 6) * kTcTile;
        const int u = (n >> 3) & 7, off = (n & 7) * 2;
#pragma unroll 8
        for (int t = half * 64; t < half * 64 + 64; ++t) {
          const float2 x = unpack_bf16(*reinterpret_cast<const uint32_t*>(kt + t * 128 + ((u ^ (t & 7)) << 4) + off));
          a0 += gt.wgt[t] * x.x;
          a1 += gt.wgt[t] * x.y;
        }
      }
      if (half == 1) { sm.half[0][np] = a0; sm.half[1][np] = a1; }
      __syncthreads();
      if (half == 0) {
        sm.n[n] = keep * sm.n[n] + a0 + sm.half[0][np];
        sm.n[n + 1] = keep * sm.n[n + 1] + a1 + sm.half[1][np];
      }
    }
    if (NB == 2) {
      ok = tc_wait(&sm.bar[1], ph) && ok;
      if (more) load_q(c0 + kTcC, 0, NB);                                        // Q's last reader (the carried part) is done
    }
    ok = tc_wait(&sm.bar[2], ph) && ok;
    tc_fence_after();
    // ---- weighted values of token r, columns [32 g, +32): over the scores, which the tensor core has read
    uint4 vraw[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      vraw[u] = tc_ld16(sV, r, g * 4 + u);
      const uint32_t q[4] = {vraw[u].x, vraw[u].y, vraw[u].z, vraw[u].w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 x = unpack_bf16(q[e]);
        tc_split(wgt * x.x, wgt * x.y, hi[e], lo[e]);
      }
      tc_st16(sP, r, g * 4 + u, hi);
      tc_st16(sP + kTcTile, r, g * 4 + u, lo);
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
#pragma unroll
      for (int mb = 0; mb < MB; ++mb)
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            umma_bf16_ss(tD + mb * 64, umma_desc_sw128_mnmajor(sK + mb * 2 * kTcTile, kTcTile) + kk * 128,
                         umma_desc_sw128_mnmajor(sP + hl * kTcTile, kTcTile) + kk * 128, idMM, (hl | kk) != 0);
      umma_commit(&sm.bar[3]);
    }
    __syncwarp();
    if (more) {
      load_v(c0 + kTcC);
      if (NB == 4) load_q(c0 + kTcC, 2, 4);                                      // (the weighted values cover Q's first two chunks only)
    }
    // ---- outputs of token r, columns [32 g, +32)
    {
      uint32_t a[32], b[32];
      __syncwarp();
      tmem_ld_32x32(tP + lane_base + g * 32, a);
      if (have_state) tmem_ld_32x32(tI + lane_base + g * 32, b);
      tmem_ld_wait();
      const float carry = have_state ? gt.carry[r] : 0.f;
      float inv = 1.f;
      if (MODE == kMlstm) {
        const float den = sm.den[0][r] + sm.den[1][r] + carry * (sm.deni[0][r] + sm.deni[1][r]);
        inv = 1.f / (fmaxf(fabsf(den), gt.flo[r]) + 1e-6f);
      }
      if (r < nv) {
        __nv_bfloat16* dst = gO + static_cast<int64_t>(c0 + r) * p.ldo + g * 32;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const uint32_t q[4] = {vraw[u].x, vraw[u].y, vraw[u].z, vraw[u].w};
          uint32_t o[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = u * 8 + 2 * e;
            float y0 = __uint_as_float(a[i]), y1 = __uint_as_float(a[i + 1]);
            if (have_state) {
              y0 += carry * __uint_as_float(b[i]);
              y1 += carry * __uint_as_float(b[i + 1]);
            }
            if (MODE == kSsd) {
              const float2 x = unpack_bf16(q[e]);
              y0 += skip * x.x;
              y1 += skip * x.y;
            } else if (MODE == kMlstm) {
              y0 *= inv;
              y1 *= inv;
            }
            o[e] = pack_bf16(y0, y1);
          }
          if (g * 32 + u * 8 < vn) *reinterpret_cast<uint4*>(dst + u * 8) = make_uint4(o[0], o[1], o[2], o[3]);
        }
      }
    }
    ok = tc_wait(&sm.bar[3], ph) && ok;
    tc_fence_after();
    if (more && NB == 4) {
      load_k(c0 + kTcC, 0);
      load_q(c0 + kTcC, 0, 2);
    }
    // ---- S = keep S + delta
#pragma unroll
    for (int mb = 0; mb < MB; ++mb) {
      uint32_t d[32];
      __syncwarp();
      tmem_ld_32x32(tD + mb * 64 + lane_base + g * 32, d);
      tmem_ld_wait();
#pragma unroll
      for (int c = 0; c < 32; ++c) S[mb][c] = keep * S[mb][c] + __uint_as_float(d[c]);
    }
    have_state = true;
    if (more) stage_state();
    tc_fence_before();
    if (__syncthreads_or(!ok)) {
      if (tid == 0) atomicExch(err, 1);
      ok = false;
      break;
    }
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  if (ok) {
#pragma unroll
    for (int mb = 0; mb < MB; ++mb) {
      const int n = mb * 128 + r;
#pragma unroll
      for (int c = 0; c < 32; c += 4)
        if (n < N && g * 32 + c < vn)
          *reinterpret_cast<float4*>(gS + static_cast<int64_t>(n) * V + g * 32 + c) = make_float4(S[mb][c], S[mb][c + 1], S[mb][c + 2], S[mb][c + 3]);
    }
  }
  if (MODE == kMlstm) {
    if (last_tile(p.counter + s * p.H + h, gridDim.x)) {
      const int64_t hb = slot * p.H + h;
      if (tid < N) p.nst[hb * N + tid] = sm.n[tid];
      if (tid == 0) p.mst[hb] = sm.m;
    }
  }
  __syncthreads();
  if (w == 0) { tc_fence_after(); tmem_dealloc(sm.tmem, 512); }
}

template <int MODE, int NB>
static int run_tc(const ScanParams& p, int32_t* err, cudaStream_t st) {
  auto kern = mix_chunk_tc_kernel<MODE, NB>;
  constexpr int smem = ChunkTc<NB>::SMEM;
  static_assert(smem <= 232448 && sizeof(TcShared) <= 11264, "shared memory");
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr = true;
  }
  kern<<<dim3((p.V + 63) / 64, p.H, p.spans), kTcThreads, smem, st>>>(p, err);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

}  // namespace prl

using namespace prl;

// 16-byte aligned rows of q, k, v, out and state; head sizes multiples of 8
extern "C" int prl_mix_chunk_tc_ok(const ScanParams* p) {
  auto al = [](const void* q, int64_t ld) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0 && ld % 8 == 0; };
  return p->N % 8 == 0 && p->V % 8 == 0 && p->N <= 256 && al(p->q, p->ldq) && al(p->k, p->ldk) && al(p->v, p->ldv) && al(p->out, p->ldo) && al(p->S, 0) &&
         p->qscale > 0.f;
}
// *err becomes 1 when a wait inside the kernel timed out
extern "C" int prl_mix_chunk_tc(const ScanParams* p, int mode, int32_t* err, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || !prl_mix_chunk_tc_ok(p)) return -240;
  if (mode != kSsd && mode != kMlstm && mode != kDecay) return -241;
  if (mode == kDecay) return p->N <= 128 ? run_tc<kDecay, 2>(*p, err, st) : run_tc<kDecay, 4>(*p, err, st);
  if (p->N <= 128) return mode == kSsd ? run_tc<kSsd, 2>(*p, err, st) : run_tc<kMlstm, 2>(*p, err, st);
  return mode == kSsd ? run_tc<kSsd, 4>(*p, err, st) : run_tc<kMlstm, 4>(*p, err, st);
}
