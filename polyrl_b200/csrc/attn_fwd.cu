// polyrl_b200 — varlen causal flash-attention FORWARD on tcgen05 / TMEM / TMA (query / key width 64, 128 or 192, value width 64 or 128, GQA,
// one or two softmax maps per head).
//
// Replaces the flash-attn 2 library call (mma.sync) the reference reaches through
// 3rdparty/verl/verl/models/transformers/monkey_patch.py:49-117 (`_flash_attention_forward`) for training,
// old-log-prob and prefill (incl. prefill behind a cached prefix: bottom-right aligned causal mask).
//
// One CTA = one (128-row query tile of one sequence, one query head), 192 threads:
//   warp 0   TMA producer: Q tile once, then K/V tiles (128 keys) through a 2-stage ring
//   warp 1   MMA issuer:   S_j = Q K_j^T (8 x tcgen05.mma 128x128x16, both operands K-major) into one of two TMEM
//                          S buffers — S_{j+1} is issued BEFORE waiting for P_j, so the tensor core works on the next
//                          scores while the softmax warps are busy — then  PV_j = P_j V_j  with P_j from shared
//                          memory and V_j consumed as an MN-major B operand (no transpose of V anywhere)
//   warps 2-9  softmax:    two warpgroups; group g owns columns [64g, 64g+64) of every query row (thread = TMEM lane):
//                          two passes over its 64 scores in TMEM (max — exchanged with the other group through shared
//                          memory and one 256-thread named barrier — then exp2 / sum), P_j written as bf16 into the
//                          128B-swizzled K-major layout the MMA reads, running output half kept in 64 fp32 registers:
//                          O = O * alpha + PV_j  (PV_j read back from TMEM).  exp2 is ex2.approx.
// DK = 192 (latent attention expanded to heads: 128 + 64 rotary) keeps both K stages and drops to one V stage, which is
// reloaded while the next scores and their softmax run.  An optional per-head sink adds exp(sink_h) to the softmax
// denominator in the epilogue.
// With two P stages (two maps per head) PV_j is read back after P_(j+1) has been written: the product runs while the softmax
// warps work on the next scores.
// Two maps per head (differential attention): the CTA runs the loop twice over the same values, keeps the first map's output in
// TMEM (fp32) and writes  (a1 - lambda a2) / sqrt(mean^2 + eps) * keep.  Keys of width 32 lie pairwise in rows of 64 (both maps read
// the same row, the queries are zero outside their half).
// A sliding window with kept first tokens (query i sees key j if i - j < window or j < keep_first) skips the key tiles between the
// kept ones and the window of the tile's first query.
// Epilogue: O / l -> bf16 (16-byte stores), log-sum-exp per (head, token) for the backward pass.
#include "common.cuh"

namespace prl {

constexpr int kAfThreads = 320;          // warp0 TMA, warp1 MMA, warps 2-5 + 6-9: two softmax warpgroups
constexpr int kAfBM = 128, kAfBN = 128;
constexpr int kAfTile = 128 * 128 * 2;              // 32 KB: one 128 x 128 bf16 operand tile (2 chunks of 64 columns)
template <int DK, int DV, int MAPS>
struct AfCfg {
  static constexpr int QKT = 128 * DK * 2;            // Q or K tile: DK / 64 chunks of 128 rows x 64 columns
  static constexpr int VT = 128 * DV * 2;             // V tile
  static constexpr int VST = DK * MAPS + DV <= 256 ? 2 : 1;       // V stages
  static constexpr int BASE = (MAPS + 2) * QKT /*Q, K x 2*/ + VST * VT /*V*/ + 1024 + 256;
  static constexpr int PST = MAPS == 2 && BASE + 2 * kAfTile <= 220 * 1024 ? 2 : 1;        // P stages
  static constexpr int SMEM = BASE + PST * kAfTile;
};

struct AttnFwdParams {
  __nv_bfloat16* o;            // [Tq, ldo]
  float* lse;                  // [nq, Tq]
  const int32_t* cu_q;         // [B+1]
  const int32_t* cu_k;         // [B+1]
  int64_t ldo;
  int B, nq, nkv, Tq;          // nq: output heads (q holds MAPS of each)
  float scale_log2;            // sm_scale * log2(e)
  float sm_scale;
  int causal;
  int window, keep_first;      // window: 0x7fffffff when every earlier key is seen
  const float* sink;           // [nq] or null: natural-log sink of the softmax denominator
  const float* lam;            // two maps: [1] weight of the second
  float keep, eps;             // two maps: factor behind the norm, and what is added under its root
  int dv_out, shared_row;      // two maps: values of a head that are written (<= DV); both maps' keys in one row
  long long* dbg;              // optional timeline buffer (kernel experiments)
};

template <int DK, int kAfD, int MAPS>
__global__ void __launch_bounds__(kAfThreads, 1)
attn_fwd_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                const __grid_constant__ CUtensorMap tmV, AttnFwdParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  using Cfg = AfCfg<DK, kAfD, MAPS>;
  constexpr int QKT = Cfg::QKT, VST = Cfg::VST, VT = Cfg::VT, OW = kAfD / 2, PST = Cfg::PST;
  uint8_t* sK = smem + MAPS * QKT;                    // [2 stages]
  uint8_t* sV = smem + (MAPS + 2) * QKT;              // [VST stages]
  uint8_t* sP = sV + VST * VT;
  uint64_t* bars = reinterpret_cast<uint64_t*>(sP + PST * kAfTile);
  uint64_t* q_full = bars;            // 1
  uint64_t* k_full = bars + 1;        // [2]
  uint64_t* v_full = bars + 3;        // [2]
  uint64_t* k_empty = bars + 5;       // [2]
  uint64_t* s_full = bars + 7;        // [2]
  uint64_t* s_empty = bars + 9;       // [2]  (128 arrivals)
  uint64_t* p_full0 = bars + 11;      // 256 arrivals; P stage 1: bars + 16
  uint64_t* o_full = bars + 12;       // 1
  uint64_t* o_empty = bars + 13;      // 128 arrivals
  uint64_t* v_empty = bars + 14;      // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);
  auto p_full = [&](int j) { return PST == 2 && (j & 1) ? bars + 16 : p_full0; };
  auto p_phase = [&](int j) { return static_cast<uint32_t>(PST == 2 ? (j >> 1) & 1 : j & 1); };
  __shared__ int s_seq, s_q0;
  __shared__ float s_mx[2][2][128];             // [tile parity][warpgroup][row]: half-row maxima
  __shared__ float s_sum[MAPS][2][128];         // half-row sums

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y;
  const int hk = h / (p.nq / p.nkv);

  // ---- which (sequence, query tile) is this CTA?  tiles are numbered sequence by sequence
  if (threadIdx.x == 0) {
    int t = blockIdx.x, seq = -1, q0 = 0;
    for (int b = 0; b < p.B; ++b) {
      const int lq = p.cu_q[b + 1] - p.cu_q[b];
      const int nt = (lq + kAfBM - 1) / kAfBM;
      if (t < nt) { seq = b; q0 = t * kAfBM; break; }
      t -= nt;
    }
    s_seq = seq; s_q0 = q0;
  }
  __syncthreads();
  const int seq = s_seq;
  if (seq < 0) return;                                 // grid is an upper bound on the tile count
  const int q0 = s_q0;
  const int qs = p.cu_q[seq], lq = p.cu_q[seq + 1] - qs;
  const int ks = p.cu_k[seq], lk = p.cu_k[seq + 1] - ks;
  const int off = lk - lq;                             // bottom-right aligned causal mask (prefix-cached prefill: lk > lq)
  int kv_end = lk;
  if (p.causal) kv_end = min(lk, q0 + kAfBM + off);    // keys beyond the last row's diagonal are never needed
  // key tiles in use: those of the kept first keys, then those from the window of this tile's first query on
  const int w_tile = max(0, q0 + off - p.window + 1) / kAfBN;
  const int kept_tiles = min((p.keep_first + kAfBN - 1) / kAfBN, w_tile), gap = w_tile - kept_tiles;
  const int nt = max(1, (kv_end + kAfBN - 1) / kAfBN - gap);
  auto tile_of = [&](int j) { return j < kept_tiles ? j : j + gap; };

  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1); mbar_init(&v_full[i], 1); mbar_init(&k_empty[i], 1); mbar_init(&v_empty[i], 1);
      mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], 256);
    }
    mbar_init(p_full0, 256); mbar_init(bars + 16, 256); mbar_init(o_full, 1); mbar_init(o_empty, 256);
    fence_barrier_init();
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tS0 = tmem_base, tO = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      mbar_expect_tx(q_full, MAPS * QKT);
#pragma unroll
      for (int c = 0; c < MAPS * DK / 64; ++c) tma_load_2d(&tmQ, q_full, sQ + c * 16384, h * MAPS * DK + c * 64, qs + q0);
      for (int j = 0; j < MAPS * nt; ++j) {               // two maps: the key tiles of the first, then those of the second
        const int s = j & 1, map = MAPS == 2 && j >= nt ? 1 : 0, key0 = ks + tile_of(j - map * nt) * kAfBN;
        const int kcol = (MAPS == 1 || p.shared_row ? hk : hk * MAPS + map) * DK;
        const uint32_t ph = (j >> 1) & 1;
        const int sv = j % VST;
        mbar_wait(&k_empty[s], ph ^ 1);
        mbar_expect_tx(&k_full[s], QKT);
#pragma unroll
        for (int c = 0; c < DK / 64; ++c) tma_load_2d(&tmK, &k_full[s], sK + s * QKT + c * 16384, kcol + c * 64, key0);
        mbar_wait(&v_empty[sv], ((j / VST) & 1) ^ 1);
        mbar_expect_tx(&v_full[sv], VT);
#pragma unroll
        for (int c = 0; c < kAfD / 64; ++c) tma_load_2d(&tmV, &v_full[sv], sV + sv * VT + c * 16384, hk * kAfD + c * 64, key0);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idS = umma_idesc(128, 128, 1, 1);
      constexpr uint32_t idO = umma_idesc_major(128, kAfD, 1, 1, 0, 1);     // B = V consumed MN-major
      auto issue_s = [&](int j) {
        const int s = j & 1;
        mbar_wait(&k_full[s], (j >> 1) & 1);
        mbar_wait(&s_empty[s], ((j >> 1) & 1) ^ 1);
        tc_fence_after();
        const uint8_t* q = sQ + (MAPS == 2 && j >= nt ? QKT : 0);
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t da = umma_desc_sw128_kmajor(q + (kk >> 2) * 16384) + 2 * (kk & 3);
          const uint64_t db = umma_desc_sw128_kmajor(sK + s * QKT + (kk >> 2) * 16384) + 2 * (kk & 3);
          umma_bf16_ss(tS0 + s * 128, da, db, idS, kk != 0);
        }
        umma_commit(&s_full[s]);
      };
      mbar_wait(q_full, 0);
      issue_s(0);
      for (int j = 0; j < MAPS * nt; ++j) {
        const int s = j & 1;
        if (j + 1 < MAPS * nt) issue_s(j + 1);
        mbar_wait(p_full(j), p_phase(j));
        const int sv = j % VST;
        mbar_wait(&v_full[sv], (j / VST) & 1);
        mbar_wait(o_empty, (j & 1) ^ 1);
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t da = umma_desc_sw128_kmajor(sP + (PST == 2 ? (j & 1) * kAfTile : 0) + (kk >> 2) * 16384) + 2 * (kk & 3);
          const uint64_t db = umma_desc_sw128_mnmajor(sV + sv * VT, 16384) + kk * 128;
          umma_bf16_ss(tO, da, db, idO, kk != 0);
        }
        umma_commit(o_full);
        umma_commit(&k_empty[s]);
        umma_commit(&v_empty[sv]);
      }
    }
  } else {
    // two softmax warpgroups: group g owns score columns [64g, 64g+64) and its half of the output columns of every row
    const int g = (warp - 2) >> 2;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;                       // query row inside the tile == TMEM lane
    const uint32_t lane_base = static_cast<uint32_t>(quad * 32) << 16;
    const int qrow = q0 + r;                              // position inside the sequence's queries
    const int kmax = p.causal ? qrow + off : lk - 1;      // last key this row may attend to
    float m_run = -INFINITY, l_run = 0.f;
    const int klo = qrow + off - p.window;                // keys up to here are behind the window (unless kept)
    float O[OW];
#pragma unroll
    for (int i = 0; i < OW; ++i) O[i] = 0.f;
    const uint32_t sP0_u32 = smem_u32(sP) + g * 16384 + r * 128;
    const bool rec = p.dbg != nullptr && blockIdx.x == gridDim.x / 2 && blockIdx.y == 0 && threadIdx.x == 64;
    long long* dbg = p.dbg;
    if (rec) dbg[0] = clock64();
    auto store = [&](__nv_bfloat16* dst, float f) {
#pragma unroll
      for (int c = 0; c < OW; c += 8) {
        int4 ov;
        ov.x = pack_bf16(O[c] * f, O[c + 1] * f); ov.y = pack_bf16(O[c + 2] * f, O[c + 3] * f);
        ov.z = pack_bf16(O[c + 4] * f, O[c + 5] * f); ov.w = pack_bf16(O[c + 6] * f, O[c + 7] * f);
        st_v4(dst + c, ov);
      }
    };
    // own half of O = O * alpha + P V of key tile j
    auto take = [&](int j, float alpha) {
      mbar_wait(o_full, j & 1);
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < OW; c += 32) {
        uint32_t v[32];
        __syncwarp();
        tmem_ld_32x32(tO + lane_base + g * OW + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) O[c + i] = O[c + i] * alpha + __uint_as_float(v[i]);
      }
      tc_fence_before();
      mbar_arrive(o_empty);
    };
    for (int map = 0; map < MAPS; ++map) {
    float alpha_before = 0.f;
    for (int j = map * nt; j < (map + 1) * nt; ++j) {
      const int s = j & 1;
      mbar_wait(&s_full[s], (j >> 1) & 1);
      tc_fence_after();
      if (rec && j < 30) dbg[1 + 5 * j] = clock64();
      const uint32_t tS = tS0 + s * 128 + lane_base + g * 64;
      const int base = tile_of(j - map * nt) * kAfBN, col0 = base + g * 64;
      const bool need_mask = (base + kAfBN - 1 > kmax) || (base + kAfBN > lk) || base <= klo;
      auto seen = [&](int col) { return col <= kmax && col < lk && (col > klo || col < p.keep_first); };
      // pass 1: max over this thread's 64 scores, then exchange with the other warpgroup's half of the row
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 64; c += 32) {
        uint32_t v[32];
        __syncwarp();
        tmem_ld_32x32(tS + c, v);
        tmem_ld_wait();
        if (need_mask) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int col = col0 + c + i;
            mx = fmaxf(mx, seen(col) ? __uint_as_float(v[i]) : -INFINITY);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(v[i]));
        }
      }
      s_mx[j & 1][g][r] = mx;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      mx = fmaxf(mx, s_mx[j & 1][g ^ 1][r]);
      if (rec && j < 30) dbg[2 + 5 * j] = clock64();
      const float m_new = fmaxf(m_run, mx);
      const float m_use = (m_new == -INFINITY) ? 0.f : m_new;
      const float alpha = (m_run == -INFINITY) ? 0.f : fast_exp2((m_run - m_use) * p.scale_log2);
      const float mb = m_use * p.scale_log2;
      const uint32_t sP_u32 = sP0_u32 + (PST == 2 ? (j & 1) * kAfTile : 0);       // (PV_(j-2) has been taken: its P may be overwritten)
      // pass 2: probabilities -> bf16 P in shared memory (K-major, 128B swizzle), partial row sum
      float lsum = 0.f;
#pragma unroll
      for (int c = 0; c < 64; c += 32) {
        uint32_t v[32];
        __syncwarp();
        tmem_ld_32x32(tS + c, v);
        tmem_ld_wait();
        float pv[32];
        if (need_mask) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int col = col0 + c + i;
            pv[i] = fast_exp2(seen(col) ? __uint_as_float(v[i]) * p.scale_log2 - mb : -INFINITY);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) pv[i] = fast_exp2(__uint_as_float(v[i]) * p.scale_log2 - mb);
        }
        float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;          // four independent chains
#pragma unroll
        for (int i = 0; i < 32; i += 4) { s0 += pv[i]; s1 += pv[i + 1]; s2 += pv[i + 2]; s3 += pv[i + 3]; }
        lsum += (s0 + s1) + (s2 + s3);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int u = (c >> 3) + q;                               // 16-byte unit inside this group's 128-byte row
          const uint32_t p0 = pack_bf16(pv[8 * q + 0], pv[8 * q + 1]), p1 = pack_bf16(pv[8 * q + 2], pv[8 * q + 3]);
          const uint32_t p2 = pack_bf16(pv[8 * q + 4], pv[8 * q + 5]), p3 = pack_bf16(pv[8 * q + 6], pv[8 * q + 7]);
          asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(sP_u32 + ((u ^ (r & 7)) << 4)), "r"(p0), "r"(p1),
                       "r"(p2), "r"(p3)
                       : "memory");
        }
      }
      if (rec && j < 30) dbg[3 + 5 * j] = clock64();
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(p_full(j));
      mbar_arrive(&s_empty[s]);
      l_run = l_run * alpha + lsum;
      m_run = m_new;
      if (rec && j < 30) dbg[4 + 5 * j] = clock64();
      if constexpr (PST == 2) {
        if (j > map * nt) take(j - 1, alpha_before);
        alpha_before = alpha;
      } else {
        take(j, alpha);
      }
      if (rec && j < 30) dbg[5 + 5 * j] = clock64();
    }
    if constexpr (PST == 2) take((map + 1) * nt - 1, alpha_before);
    // total row sum = the two groups' partial sums (same running max on both sides)
    s_sum[map][g][r] = l_run;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    float l_tot = l_run + s_sum[map][g ^ 1][r];
    if (p.sink != nullptr && m_run != -INFINITY) l_tot += fast_exp2(p.sink[h] * 1.4426950408889634f - m_run * p.scale_log2);
    const float inv = l_tot > 0.f ? 1.f / l_tot : 0.f;
    if constexpr (MAPS == 1) {
      if (qrow < lq) {
        store(p.o + static_cast<int64_t>(qs + qrow) * p.ldo + h * kAfD + g * OW, inv);
        if (p.lse && g == 0)
          p.lse[static_cast<int64_t>(h) * p.Tq + qs + qrow] = (m_run == -INFINITY) ? -INFINITY : m_run * p.sm_scale + __logf(l_tot);
      }
    } else {
      const uint32_t t_first = tO + 128 + lane_base + g * OW;          // the first map's output
      if (map == 0) {
#pragma unroll
        for (int c = 0; c < OW; c += 16) {
          uint32_t v[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) { v[i] = __float_as_uint(O[c + i] * inv); O[c + i] = 0.f; }
          __syncwarp();
          tmem_st_32x16(t_first + c, v);
        }
        tmem_st_wait();
        m_run = -INFINITY;
        l_run = 0.f;
      } else {
        const float lam = p.lam[0];
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < OW; c += 32) {
          uint32_t v[32];
          __syncwarp();
          tmem_ld_32x32(t_first + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            O[c + i] = __uint_as_float(v[i]) - lam * (O[c + i] * inv);
            ss += O[c + i] * O[c + i];
          }
        }
        s_sum[0][g][r] = ss;                     // (the first map's sums were read before this map's last barrier)
        asm volatile("bar.sync 1, 256;" ::: "memory");
        ss += s_sum[0][g ^ 1][r];
        const float f = rsqrtf(ss / p.dv_out + p.eps) * p.keep;
        if (qrow < lq) {
          const int n = p.dv_out - g * OW;       // values of this half
          __nv_bfloat16* dst = p.o + static_cast<int64_t>(qs + qrow) * p.ldo + h * p.dv_out + g * OW;
          if (n >= OW && p.dv_out % 8 == 0 && p.ldo % 8 == 0) {
            store(dst, f);
          } else {
#pragma unroll
            for (int c = 0; c < OW; ++c)
              if (c < n) dst[c] = __float2bfloat16(O[c] * f);
          }
        }
      }
    }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, 512); }
}

using EncodeTiledFn4 = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                    const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                    CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static EncodeTiledFn4 af_encode_fn() {
  static EncodeTiledFn4 fn = nullptr;
  if (!fn) {
    void* q = nullptr;
    cudaDriverEntryPointQueryResult qr;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &q, cudaEnableDefault, &qr) != cudaSuccess || !q) return nullptr;
    fn = reinterpret_cast<EncodeTiledFn4>(q);
  }
  return fn;
}
// rows x cols bf16 matrix with row pitch ld_bytes; box = 64 columns (128 B) x box_rows rows, 128B swizzle
int af_tmap(CUtensorMap* m, const void* ptr, uint64_t rows, uint64_t cols, uint64_t ld_bytes, uint32_t box_rows) {
  ensure_thread_ctx();
  auto fn = af_encode_fn();
  if (!fn) return -1;
  cuuint64_t gdim[2] = {cols, rows};
  cuuint64_t gstride[1] = {ld_bytes};
  cuuint32_t box[2] = {64, box_rows};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), gdim, gstride, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -static_cast<int>(r);
}

}  // namespace prl

using namespace prl;

template <int DK, int DV, int MAPS>
static int run_attn_fwd(const void* q, const void* k, const void* v, const AttnFwdParams& p, int Tk, int64_t ldq, int64_t ldk, int64_t ldv,
                        int max_tiles, cudaStream_t stream) {
  using Cfg = AfCfg<DK, DV, MAPS>;
  CUtensorMap tmQ, tmK, tmV;
  if (af_tmap(&tmQ, q, p.Tq, static_cast<uint64_t>(p.nq) * MAPS * DK, ldq * 2, kAfBM)) return -111;
  if (af_tmap(&tmK, k, Tk, static_cast<uint64_t>(p.nkv) * (MAPS == 2 && !p.shared_row ? 2 : 1) * DK, ldk * 2, kAfBN)) return -112;
  if (af_tmap(&tmV, v, Tk, static_cast<uint64_t>(p.nkv) * DV, ldv * 2, kAfBN)) return -113;
  static bool attr = false;
  if (!attr) {
    PRL_CUDA_CHECK(cudaFuncSetAttribute(attn_fwd_kernel<DK, DV, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM));
    attr = true;
  }
  attn_fwd_kernel<DK, DV, MAPS><<<dim3(max_tiles, p.nq), kAfThreads, Cfg::SMEM, stream>>>(tmQ, tmK, tmV, p);
  PRL_CUDA_CHECK(cudaGetLastError());
  return 0;
}

// q:[Tq, nq*dk] (pitch ldq), k:[Tk, nkv*dk], v:[Tk, nkv*dv] (pitches ldk/ldv), o:[Tq, nq*dv] (pitch ldo); pitches in ELEMENTS;
// dk, dv = 64 or 128; dk = 192 (dv = 128).  window > 0 (causal only): query i sees keys j <= i with i - j < window or j < keep_first.  cu_q / cu_k: int32 [B+1] device arrays.  max_tiles: upper bound on sum_b ceil(lq_b / 128) (e.g. Tq/128 + B).
// sink: fp32 [nq] or null.
extern "C" int prl_attn_fwd(const void* q, const void* k, const void* v, void* o, float* lse, const int32_t* cu_q,
                            const int32_t* cu_k, int B, int Tq, int Tk, int nq, int nkv, int dk, int dv, int64_t ldq, int64_t ldk, int64_t ldv,
                            int64_t ldo, float sm_scale, int causal, int max_tiles, const float* sink, int window, int keep_first, long long* dbg,
                            cudaStream_t stream) {
  if (Tq <= 0 || B <= 0) return 0;
  if (nq % nkv != 0) return -110;
  AttnFwdParams p{};
  p.o = static_cast<__nv_bfloat16*>(o);
  p.lse = lse;
  p.cu_q = cu_q; p.cu_k = cu_k;
  p.ldo = ldo; p.B = B; p.nq = nq; p.nkv = nkv; p.Tq = Tq;
  p.sm_scale = sm_scale;
  p.scale_log2 = sm_scale * 1.4426950408889634f;
  p.causal = causal;
  if (window > 0 && !causal) return -115;
  p.window = window > 0 ? window : 0x7fffffff;
  p.keep_first = window > 0 ? keep_first : 0;
  p.sink = sink;
  p.dbg = dbg;
  if (dk == 64 && dv == 64) return run_attn_fwd<64, 64, 1>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 64 && dv == 128) return run_attn_fwd<64, 128, 1>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 128 && dv == 64) return run_attn_fwd<128, 64, 1>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 128 && dv == 128) return run_attn_fwd<128, 128, 1>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 192 && dv == 128) return run_attn_fwd<192, 128, 1>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  return -114;
}

// differential attention, causal: q:[Tq, nq*2*dk], k:[Tk, nkv*2*dk] — or [Tk, nkv*64] when shared_row (dk = 64: both maps' keys of width 32 in one row) —
// v:[Tk, nkv*dv], o:[Tq, nq*dv_out], all contiguous; dk, dv = 64 or 128
extern "C" int prl_map_attn_fwd(const void* q, const void* k, const void* v, void* o, const int32_t* cu_q, const int32_t* cu_k, int B, int Tq, int Tk, int nq,
                                int nkv, int dk, int dv, int dv_out, int shared_row, float sm_scale, int window, const float* lam, float keep, float eps,
                                int max_tiles, cudaStream_t stream) {
  if (Tq <= 0 || B <= 0) return 0;
  if (nq % nkv != 0 || dv_out < 1 || dv_out > dv || window < 1 || (shared_row && dk != 64)) return -110;
  AttnFwdParams p{};
  p.o = static_cast<__nv_bfloat16*>(o);
  p.cu_q = cu_q; p.cu_k = cu_k;
  p.ldo = static_cast<int64_t>(nq) * dv_out; p.B = B; p.nq = nq; p.nkv = nkv; p.Tq = Tq;
  p.sm_scale = sm_scale;
  p.scale_log2 = sm_scale * 1.4426950408889634f;
  p.causal = 1;
  p.window = window;
  p.lam = lam; p.keep = keep; p.eps = eps; p.dv_out = dv_out; p.shared_row = shared_row;
  const int64_t ldq = static_cast<int64_t>(nq) * 2 * dk, ldk = static_cast<int64_t>(nkv) * (shared_row ? 1 : 2) * dk, ldv = static_cast<int64_t>(nkv) * dv;
  if (dk == 64 && dv == 64) return run_attn_fwd<64, 64, 2>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 64 && dv == 128) return run_attn_fwd<64, 128, 2>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 128 && dv == 64) return run_attn_fwd<128, 64, 2>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  if (dk == 128 && dv == 128) return run_attn_fwd<128, 128, 2>(q, k, v, p, Tk, ldq, ldk, ldv, max_tiles, stream);
  return -114;
}
