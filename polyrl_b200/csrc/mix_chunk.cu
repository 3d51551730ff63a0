// polyrl_b200 — gated linear recurrences over prompt portions, chunk-parallel on the tensor cores (bf16 activations).
//
// Same recurrences as mix_scan.cu, 64 tokens at a time.  With La the running sum of log keep inside the chunk,
//     kSsd    weight(t, s) = exp(La_t - La_s) dt_s,       carry-in factor exp(La_t);  kDecay the same with dt = 1
//     kMlstm  F = running sum of f,  g_s = i_s - F_s,  M_t = max(m_0, max_{s <= t} g_s),  m_t = F_t + M_t:
//             weight(t, s) = exp(g_s - M_t),               carry-in factor exp(m_0 - M_t)
// so that  y_t = sum_{s <= t} weight(t, s) (q_t . k_s) v_s + carry_t S_0^T q_t  and the state after the chunk is
// S = carry_C S_0 + sum_s weight(C, s) k_s v_s^T.  All exponents are <= 0.
//
// One CTA = one (span, head, VT value columns) marching over its chunks; the fp32 state stays in the accumulator
// registers of the update product from the first chunk to the last.  Operands that are not bf16 by nature (the weighted
// scores, the weighted values and the state as an operand) enter the products as a bf16 pair hi + lo, so the recurrence
// keeps about 16 bits of them and the state itself all 32.
#include "mixers.cuh"

namespace prl {

constexpr int kCh = 64;                 // tokens per chunk
constexpr int kChThreads = 256;

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
// x = hi + lo with both parts bf16; two neighbours packed
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  const float2 h = unpack_bf16(hi);
  lo = pack_bf16(a - h.x, b - h.y);
}

template <int NT, int VT>
struct ChunkSmem {
  static constexpr int LDN = NT + 8, LDV = VT + 8, LDP = kCh + 8;
  static constexpr int LDX = LDP > LDV ? LDP : LDV;
  __nv_bfloat16 q[kCh * LDN], k[kCh * LDN], v[kCh * LDV];
  __nv_bfloat16 sh[NT * LDV], sl[NT * LDV];        // state as operand
  __nv_bfloat16 xh[kCh * LDX], xl[kCh * LDX];      // weighted scores, then weighted values
  float row[kCh], col[kCh], mul[kCh], carry[kCh], wgt[kCh], den[2][kCh], deni[kCh], flo[kCh];
  float n[NT];
  float keep, m;
};

// rows [0, nv) x cols [0, n) of a bf16 matrix -> shared memory, the rest of the 64 x W tile zero
template <int W, int LD>
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t ld, int nv, int n, bool vec) {
  if (vec) {
    for (int i = threadIdx.x; i < kCh * (W / 8); i += kChThreads) {
      const int r = i / (W / 8), c = (i % (W / 8)) * 8;
      const bool ok = r < nv && c < n;                  // n is a multiple of 8 here
      const uint32_t d = smem_u32(dst + r * LD + c);
      const void* g = src + (ok ? static_cast<int64_t>(r) * ld + c : 0);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(g), "r"(ok ? 16 : 0) : "memory");
    }
  } else {
    for (int i = threadIdx.x; i < kCh * W; i += kChThreads) {
      const int r = i / W, c = i % W;
      dst[r * LD + c] = (r < nv && c < n) ? src[static_cast<int64_t>(r) * ld + c] : __float2bfloat16(0.f);
    }
  }
}

template <int MODE, int NT, int VT>
__global__ void __launch_bounds__(kChThreads)
mix_chunk_kernel(ScanParams p, int vec) {
  using Sm = ChunkSmem<NT, VT>;
  constexpr int LDN = Sm::LDN, LDV = Sm::LDV, LDX = Sm::LDX;
  constexpr int MT = NT / 16;                         // 16-row tiles of the state
  constexpr int SM = MT >= 8 ? MT / 8 : 1;            // state row tiles of a warp
  constexpr int SN = MT >= 8 ? VT / 8 : VT / 8 / (8 / MT);   // state column tiles of a warp
  constexpr int ON = VT / 16;                         // output column tiles of a warp
  static_assert(SN % 2 == 0 && ON % 2 == 0, "column tiles are consumed in pairs");
  extern __shared__ __align__(128) uint8_t raw[];
  Sm& sm = *reinterpret_cast<Sm*>(raw);
  const int h = blockIdx.y, s = blockIdx.z, v0 = blockIdx.x * VT;
  const int tid = threadIdx.x, w = tid >> 5, lane = tid & 31, gq = lane >> 2, qd = lane & 3;
  const int t0 = p.cu[s], len = p.cu[s + 1] - t0;
  if (len <= 0) return;
  const bool fresh = p.start[s] == 0;
  const int64_t slot = p.slot[s];
  const int N = p.N, V = p.V, vn = min(VT, V - v0);
  const __nv_bfloat16* gQ = static_cast<const __nv_bfloat16*>(p.q) + static_cast<int64_t>(t0) * p.ldq + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gK = static_cast<const __nv_bfloat16*>(p.k) + static_cast<int64_t>(t0) * p.ldk + static_cast<int64_t>(h / p.rep) * N;
  const __nv_bfloat16* gV = static_cast<const __nv_bfloat16*>(p.v) + static_cast<int64_t>(t0) * p.ldv + static_cast<int64_t>(h) * V + v0;
  __nv_bfloat16* gO = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(t0) * p.ldo + static_cast<int64_t>(h) * V + v0;
  float* gS = p.S + (slot * p.H + h) * static_cast<int64_t>(N) * V + v0;
  const float b0 = p.b0 ? p.b0[h] : 0.f, b1 = p.b1 ? p.b1[h] : 0.f;
  const float a_neg = MODE == kSsd ? -expf(p.a_log[h]) : 0.f;
  const float skip = (MODE == kSsd && p.d_skip) ? p.d_skip[h] : 0.f;

  const int sn0 = MT >= 8 ? 0 : (w / MT) * SN;        // first state column tile of this warp
  const int om = w & 3, on0 = (w >> 2) * ON;          // output row tile, first output column tile
  float S[SM][SN][4];
#pragma unroll
  for (int i = 0; i < SM; ++i)
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = ((MT >= 8 ? w + 8 * i : w % MT) * 16) + gq + (e >> 1) * 8, c = (sn0 + j) * 8 + 2 * qd + (e & 1);
        S[i][j][e] = (!fresh && n < N && c < vn) ? gS[static_cast<int64_t>(n) * V + c] : 0.f;
      }
  auto stage_state = [&]() {
#pragma unroll
    for (int i = 0; i < SM; ++i)
#pragma unroll
      for (int j = 0; j < SN; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int n = ((MT >= 8 ? w + 8 * i : w % MT) * 16) + gq + e * 8, c = (sn0 + j) * 8 + 2 * qd;
          uint32_t hi, lo;
          split2(S[i][j][2 * e], S[i][j][2 * e + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(&sm.sh[n * LDV + c]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.sl[n * LDV + c]) = lo;
        }
  };
  stage_state();
  if (MODE == kMlstm) {
    const int64_t hb = slot * p.H + h;
    for (int n = tid; n < NT; n += kChThreads) sm.n[n] = (!fresh && n < N) ? p.nst[hb * N + n] : 0.f;
    if (tid == 0) sm.m = fresh ? 0.f : p.mst[hb];
  }
  bool have_state = !fresh;

  for (int c0 = 0; c0 < len; c0 += kCh) {
    const int nv = min(kCh, len - c0);
    load_tile<NT, LDN>(sm.q, gQ + static_cast<int64_t>(c0) * p.ldq, p.ldq, nv, N, vec);
    load_tile<NT, LDN>(sm.k, gK + static_cast<int64_t>(c0) * p.ldk, p.ldk, nv, N, vec);
    load_tile<VT, LDV>(sm.v, gV + static_cast<int64_t>(c0) * p.ldv, p.ldv, nv, vn, vec);
    // ---- gates of the chunk: warp 0, two tokens per lane
    if (w == 0) {
      float la[2], ad[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = lane + 32 * e;
        la[e] = 0.f;
        ad[e] = MODE == kMlstm ? -INFINITY : 0.f;
        if (t < nv) {
          const int64_t r = static_cast<int64_t>(t0 + c0 + t) * p.ldg + h;
          if (MODE == kDecay) {
            ad[e] = 1.f;
            la[e] = p.a_log[h];
          } else if (MODE == kSsd) {
            ad[e] = softplus_f(p.g0[r] + b0);
            la[e] = a_neg * ad[e];
          } else {
            ad[e] = softcap_f(p.g0[r] + b0, p.cap);
            la[e] = logsigmoid_f(softcap_f(p.g1[r] + b1, p.cap));
          }
        }
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x0 = __shfl_up_sync(0xffffffffu, la[0], o), x1 = __shfl_up_sync(0xffffffffu, la[1], o);
        if (lane >= o) { la[0] += x0; la[1] += x1; }
      }
      la[1] += __shfl_sync(0xffffffffu, la[0], 31);
      const float la_end = __shfl_sync(0xffffffffu, la[1], 31);
      if (MODE != kMlstm) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = lane + 32 * e;
          sm.row[t] = la[e];
          sm.col[t] = -la[e];
          sm.mul[t] = ad[e];
          sm.carry[t] = expf(la[e]);
          sm.wgt[t] = expf(la_end - la[e]) * ad[e];
        }
        if (lane == 0) sm.keep = expf(la_end);
      } else {
        float g[2] = {ad[0] - la[0], ad[1] - la[1]}, mx[2] = {g[0], g[1]};
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float x0 = __shfl_up_sync(0xffffffffu, mx[0], o), x1 = __shfl_up_sync(0xffffffffu, mx[1], o);
          if (lane >= o) { mx[0] = fmaxf(mx[0], x0); mx[1] = fmaxf(mx[1], x1); }
        }
        const float m0 = sm.m;
        mx[0] = fmaxf(mx[0], m0);
        mx[1] = fmaxf(mx[1], __shfl_sync(0xffffffffu, mx[0], 31));
        const float m_end = __shfl_sync(0xffffffffu, mx[1], 31);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = lane + 32 * e;
          sm.row[t] = -mx[e];
          sm.col[t] = g[e];
          sm.mul[t] = 1.f;
          sm.carry[t] = expf(m0 - mx[e]);
          sm.wgt[t] = expf(g[e] - m_end);
          sm.flo[t] = expf(-(la[e] + mx[e]));
        }
        __syncwarp();
        if (lane == 0) { sm.keep = expf(m0 - m_end); sm.m = la_end + m_end; }
      }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();

    // ---- scores of row tile om, columns [32 (w >> 2), +32); tiles above the diagonal are never read
    const int pc0 = (w >> 2) * 32;
    float den0 = 0.f, den1 = 0.f;
    if (pc0 <= om * 16 + 15) {
      float acc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < NT; kk += 16) {
        uint32_t a[4], b[4];
        ldsm4(a, &sm.q[(om * 16 + (lane & 15)) * LDN + kk + (lane >> 4) * 8]);
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          ldsm4(b, &sm.k[(pc0 + j * 8 + (lane & 7) + ((lane >> 4) << 3)) * LDN + kk + ((lane >> 3) & 1) * 8]);
          mma_bf16(acc[j], a, b[0], b[1]);
          mma_bf16(acc[j + 1], a, b[2], b[3]);
        }
      }
      const int r0 = om * 16 + gq, r1 = r0 + 8;
      const float ra = sm.row[r0], rb = sm.row[r1];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float x[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = pc0 + j * 8 + 2 * qd + (e & 1), r = (e >> 1) ? r1 : r0;
          x[e] = c <= r ? acc[j][e] * p.qscale * (expf(((e >> 1) ? rb : ra) + sm.col[c]) * sm.mul[c]) : 0.f;
        }
        den0 += x[0] + x[1];
        den1 += x[2] + x[3];
        uint32_t hi, lo;
        const int c = pc0 + j * 8 + 2 * qd;
        split2(x[0], x[1], hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.xh[r0 * LDX + c]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.xl[r0 * LDX + c]) = lo;
        split2(x[2], x[3], hi, lo);
        *reinterpret_cast<uint32_t*>(&sm.xh[r1 * LDX + c]) = hi;
        *reinterpret_cast<uint32_t*>(&sm.xl[r1 * LDX + c]) = lo;
      }
    }
    if (MODE == kMlstm) {
      den0 += __shfl_xor_sync(0xffffffffu, den0, 1);
      den0 += __shfl_xor_sync(0xffffffffu, den0, 2);
      den1 += __shfl_xor_sync(0xffffffffu, den1, 1);
      den1 += __shfl_xor_sync(0xffffffffu, den1, 2);
      if (qd == 0) { sm.den[w >> 2][om * 16 + gq] = den0; sm.den[w >> 2][om * 16 + gq + 8] = den1; }
      // n_0 . q_t: four threads per row
      float d = 0.f;
      const int r = tid >> 2;
      for (int n = tid & 3; n < N; n += 4) d += __bfloat162float(sm.q[r * LDN + n]) * sm.n[n];
      d += __shfl_xor_sync(0xffffffffu, d, 1);
      d += __shfl_xor_sync(0xffffffffu, d, 2);
      if ((tid & 3) == 0) sm.deni[r] = d * p.qscale;
    }
    // ---- carried-in part: q S_0
    float o[ON][4];
#pragma unroll
    for (int j = 0; j < ON; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    if (have_state) {
#pragma unroll 2
      for (int kk = 0; kk < NT; kk += 16) {
        uint32_t a[4], b[4];
        ldsm4(a, &sm.q[(om * 16 + (lane & 15)) * LDN + kk + (lane >> 4) * 8]);
#pragma unroll
        for (int j = 0; j < ON; j += 2) {
          const int off = (kk + (lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (on0 + j) * 8 + (lane >> 4) * 8;
          ldsm4_t(b, &sm.sh[off]);
          mma_bf16(o[j], a, b[0], b[1]);
          mma_bf16(o[j + 1], a, b[2], b[3]);
          ldsm4_t(b, &sm.sl[off]);
          mma_bf16(o[j], a, b[0], b[1]);
          mma_bf16(o[j + 1], a, b[2], b[3]);
        }
      }
      const float ca = sm.carry[om * 16 + gq] * p.qscale, cb = sm.carry[om * 16 + gq + 8] * p.qscale;
#pragma unroll
      for (int j = 0; j < ON; ++j) { o[j][0] *= ca; o[j][1] *= ca; o[j][2] *= cb; o[j][3] *= cb; }
    }
    __syncthreads();
    // ---- own part: weighted scores times values (key tiles up to the diagonal)
    for (int kt = 0; kt <= om; ++kt) {
      uint32_t ah[4], al[4], b[4];
      ldsm4(ah, &sm.xh[(om * 16 + (lane & 15)) * LDX + kt * 16 + (lane >> 4) * 8]);
      ldsm4(al, &sm.xl[(om * 16 + (lane & 15)) * LDX + kt * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int j = 0; j < ON; j += 2) {
        ldsm4_t(b, &sm.v[(kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDV + (on0 + j) * 8 + (lane >> 4) * 8]);
        mma_bf16(o[j], ah, b[0], b[1]);
        mma_bf16(o[j + 1], ah, b[2], b[3]);
        mma_bf16(o[j], al, b[0], b[1]);
        mma_bf16(o[j + 1], al, b[2], b[3]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = om * 16 + gq + 8 * e;
      if (r < nv) {
        float inv = 1.f;
        if (MODE == kMlstm) {
          const float den = sm.den[0][r] + (r >= 32 ? sm.den[1][r] : 0.f) + (have_state ? sm.carry[r] * sm.deni[r] : 0.f);
          inv = 1.f / (fmaxf(fabsf(den), sm.flo[r]) + 1e-6f);
        }
        __nv_bfloat16* dst = gO + static_cast<int64_t>(c0 + r) * p.ldo;
#pragma unroll
        for (int j = 0; j < ON; ++j) {
          const int c = (on0 + j) * 8 + 2 * qd;
          float y0 = o[j][2 * e] * inv, y1 = o[j][2 * e + 1] * inv;
          if (MODE == kSsd) {
            y0 += skip * __bfloat162float(sm.v[r * LDV + c]);
            y1 += skip * __bfloat162float(sm.v[r * LDV + c + 1]);
          }
          if (vec) {
            if (c < vn) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(y0, y1);
          } else {
            if (c < vn) dst[c] = __float2bfloat16(y0);
            if (c + 1 < vn) dst[c + 1] = __float2bfloat16(y1);
          }
        }
      }
    }
    __syncthreads();
    // ---- weighted values, normaliser
    for (int i = tid; i < kCh * (VT / 2); i += kChThreads) {
      const int r = i / (VT / 2), c = (i % (VT / 2)) * 2;
      const float g = sm.wgt[r];
      const float2 x = unpack_bf16(*reinterpret_cast<const uint32_t*>(&sm.v[r * LDV + c]));
      uint32_t hi, lo;
      split2(g * x.x, g * x.y, hi, lo);
      *reinterpret_cast<uint32_t*>(&sm.xh[r * LDX + c]) = hi;
      *reinterpret_cast<uint32_t*>(&sm.xl[r * LDX + c]) = lo;
    }
    const float keep = sm.keep;
    if (MODE == kMlstm) {
      for (int n = tid; n < NT; n += kChThreads) {
        float acc = keep * sm.n[n];
#pragma unroll 8
        for (int r = 0; r < kCh; ++r) acc += sm.wgt[r] * __bfloat162float(sm.k[r * LDN + n]);
        sm.n[n] = acc;
      }
    }
    __syncthreads();
    // ---- S = keep S + K^T (weighted V)
#pragma unroll
    for (int i = 0; i < SM; ++i) {
      const int mrow = (MT >= 8 ? w + 8 * i : w % MT) * 16;
#pragma unroll
      for (int j = 0; j < SN; ++j) { S[i][j][0] *= keep; S[i][j][1] *= keep; S[i][j][2] *= keep; S[i][j][3] *= keep; }
#pragma unroll
      for (int kt = 0; kt < kCh / 16; ++kt) {
        uint32_t a[4], b[4];
        ldsm4_t(a, &sm.k[(kt * 16 + (lane & 7) + (lane >> 4) * 8) * LDN + mrow + ((lane >> 3) & 1) * 8]);
#pragma unroll
        for (int j = 0; j < SN; j += 2) {
          const int off = (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LDX + (sn0 + j) * 8 + (lane >> 4) * 8;
          ldsm4_t(b, &sm.xh[off]);
          mma_bf16(S[i][j], a, b[0], b[1]);
          mma_bf16(S[i][j + 1], a, b[2], b[3]);
          ldsm4_t(b, &sm.xl[off]);
          mma_bf16(S[i][j], a, b[0], b[1]);
          mma_bf16(S[i][j + 1], a, b[2], b[3]);
        }
      }
    }
    have_state = true;
    if (c0 + kCh < len) stage_state();
    __syncthreads();
  }

#pragma unroll
  for (int i = 0; i < SM; ++i)
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = ((MT >= 8 ? w + 8 * i : w % MT) * 16) + gq + (e >> 1) * 8, c = (sn0 + j) * 8 + 2 * qd + (e & 1);
        if (n < N && c < vn) gS[static_cast<int64_t>(n) * V + c] = S[i][j][e];
      }
  if (MODE == kMlstm) {
    if (last_tile(p.counter + s * p.H + h, gridDim.x)) {
      const int64_t hb = slot * p.H + h;
      for (int n = tid; n < N; n += kChThreads) p.nst[hb * N + n] = sm.n[n];
      if (tid == 0) p.mst[hb] = sm.m;
    }
  }
}

template <int MODE, int NT, int VT>
static int run_chunk(const ScanParams& p, cudaStream_t st) {
  auto kern = mix_chunk_kernel<MODE, NT, VT>;
  constexpr int smem = sizeof(ChunkSmem<NT, VT>);
  static_assert(smem <= 232448, "shared memory");
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    attr = true;
  }
  auto al = [](const void* q, int64_t ld) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0 && ld % 8 == 0; };
  const int vec = al(p.q, p.ldq) && al(p.k, p.ldk) && al(p.v, p.ldv) && al(p.out, p.ldo) && p.N % 8 == 0 && p.V % 8 == 0;
  dim3 grid((p.V + VT - 1) / VT, p.H, p.spans);
  kern<<<grid, kChThreads, smem, st>>>(p, vec);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

template <int MODE>
static int pick_chunk(const ScanParams& p, cudaStream_t st) {
  if (p.V <= 32) {
    if (p.N <= 64) return run_chunk<MODE, 64, 32>(p, st);
    if (p.N <= 128) return run_chunk<MODE, 128, 32>(p, st);
    return run_chunk<MODE, 256, 32>(p, st);
  }
  if (p.N <= 64) return run_chunk<MODE, 64, 64>(p, st);
  if (p.N <= 128) return run_chunk<MODE, 128, 64>(p, st);
  return run_chunk<MODE, 256, 64>(p, st);
}

}  // namespace prl

using namespace prl;

extern "C" int prl_mix_chunk_supported(int N) { return N <= 256; }

extern "C" int prl_mix_chunk(const ScanParams* p, int mode, cudaStream_t st) {
  if (p->spans <= 0) return 0;
  if (p->spans > 65535 || p->H > 65535 || p->N > 256) return -210;
  if (mode != kSsd && mode != kMlstm && mode != kDecay) return -211;
  return mode == kSsd ? pick_chunk<kSsd>(*p, st) : mode == kDecay ? pick_chunk<kDecay>(*p, st) : pick_chunk<kMlstm>(*p, st);
}
