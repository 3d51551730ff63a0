// polyrl_b200 — launch parameters of the sequence-mixer kernels (plain pointers; shared by kernels and bindings).
#pragma once
#include <cstdint>

namespace prl {

struct ScanParams {
  const void *q, *k, *v;        // T; row pitches in elements; head h of q / k starts at (h / rep) * N, of v at h * V
  int64_t ldq, ldk, ldv;
  int rep;
  const float *g0, *g1;         // raw gate projections [tokens, ldg], one column per head (kGla: per head and state row; kDecay: none)
  int64_t ldg;
  const float *b0, *b1;         // their biases [H] (kGla [H, N])
  const float *a_log, *d_skip;  // kSsd, kDelta (a_log only), kDecay (a_log: log of the decay) [H]
  float qscale, cap;            // q is multiplied by qscale; cap bounds the kMlstm gates, is the kGla exponent's denominator
  int raw;                      // kDecay, one token per span: q, k and v are still to be silu-activated
  void* out;                    // T [tokens, ldo], head h at h * V
  int64_t ldo;
  float* S;                     // [slots, H, N, V]
  float* nst;                   // kMlstm [slots, H, N]
  float* mst;                   // kMlstm [slots, H]
  const int32_t* cu;            // [spans + 1]
  const int32_t* start;         // [spans]
  const int64_t* slot;          // [spans]
  int32_t* counter;             // [>= spans * H], zero between launches
  int H, N, V, spans;
};

struct WindowParams {
  const void* q;                // T [R, H, D]
  const void *k_pool, *v_pool;  // T [blocks, G, 16, D]
  const int32_t* table;         // [spans, ld_table] page numbers
  int64_t ld_table;
  const int32_t* seq_of;        // [R] span of a row (null: row r is span r)
  const int32_t* kv_len;        // [R] keys up to the row's own; 0 = idle row
  void* out;                    // T [R, H, D]
  int R, H, G, D, window, keep_first;
  float scale;
};

// paged attention with a sink, any widths (mix_window.cu)
struct SinkParams {
  const void* q;                // T [R, H, D]
  const void *k_pool, *v_pool;  // T [blocks, G, 16, D], [blocks, G, 16, V]
  const int32_t* table;
  int64_t ld_table;
  const int32_t* seq_of;
  const int32_t* kv_len;
  const float* sink;            // [H] or null
  void* out;                    // T [R, H, V]
  int R, H, G, D, V;
  float scale;
};

// selective scan (mix_selective.cu)
struct SelectiveParams {
  const void *x, *z, *b, *c;    // T [tokens, C] and [tokens, N]; row pitches in elements
  int64_t ldx, ldz, ldb, ldc;
  const float* dt;              // [tokens, C] step sizes ahead of their bias
  int64_t ldd;
  const float *dt_bias, *d_skip;        // [C]
  const float* a_neg;           // [C, N] -exp(A_log)
  void* out;                    // T [tokens, ldo]
  int64_t ldo;
  float* S;                     // [slots, C, N]
  const int32_t* cu;
  const int32_t* start;
  const int64_t* slot;
  int C, N, spans;
};

// residual streams (mix_streams.cu): the end of a sublayer and the beginning of the next
struct StreamsParams {
  const float* x_in;            // row r, stream s at r * row_in + s * stream_in (stream_in 0: all streams equal)
  int64_t row_in, stream_in;
  float* x_out;                 // row r, stream s at r * row_out + s * W; null after the last sublayer
  int64_t row_out;
  const int64_t* ids;           // embedding form: x_out = scale * emb[ids], one stream, and nothing is added
  const void* emb;              // T
  float scale;
  const void* y;                // T [R, ldy] or null
  int64_t ldy;
  const float* bias;            // [W] or null
  const void* rows;             // T [., W] routed rows (null: none), row pos[r * top + j] belongs to row r with weight[r * top + j] (null: 1)
  const int32_t* pos;
  const float* weight;
  int top;
  const float *mix, *out;       // [S, S] (from, to), [S]
  const float* win;             // [S] or null (ones): what the next sublayer reads
  float* sum;                   // [R, W] or null: that row itself
  const float* w_next;          // [W] — [1] when w_scalar — or null: no h
  int w_scalar;
  void* h;                      // T [R, W]
  int R, W, S;
  float eps;
};

// a parallel block's end (mix_block.cu): X = x + s1 y1 + s2 (y2 + routed rows),  x' = average over depth,  h = norm(x') w_next,  convolution
struct BlockParams {
  float* past;                  // results of the layers [., R, W], `stride` elements apart
  int64_t stride;
  int n;                        // results so far beside the embedding output; the new one is number n + 1 (without averages: number 0)
  const int64_t* ids;           // embedding form: past[0] = emb[ids] and nothing is added
  const void* emb;              // T
  const void *y1, *y2;          // T [R, ld]; y2 may be null
  int64_t ld1, ld2;
  const void* rows;             // T [., W] routed rows (null: none), row pos[r * top + j] belongs to row r
  const int32_t* pos;
  int top;
  const float *s1, *s2;         // [W] or null
  const float *a_prev, *a_cur;  // coefficients [n + 1] of x and [n + 2] of x' (null: x = past[0]; x' = X)
  const float* w_next;          // [W] or null: no h
  float* x_out;                 // [R, W] or null
  void *h, *h2;                 // T [R, W]; h2 is the second convolution's
  const float *c1, *c2;         // single-token rows: convolutions [taps, W] (null: h is the norm itself), row r is span r
  void* state;                  // T [slots, taps - 1, W]
  const int32_t* start;
  const int64_t* slot;
  int taps, R, W, center;
  float eps;
};

// differential attention, paged, any width (mix_maps.cu)
struct MapParams {
  const void* q;                // T [R, H, 2, qw]; the data of map m starts at column m * (qw - kw) unless qw == kw
  const void *k_pool, *v_pool;  // T [blocks, G, 16, 2 kw], [blocks, G, 16, vw]
  const int32_t* table;
  int64_t ld_table;
  const int32_t* seq_of;
  const int32_t* kv_len;
  const float* lam;             // [1]
  void* out;                    // T [R, H * V]
  int R, H, G, D, V, qw, kw, vw, window;
  float scale, keep, eps;       // keep: factor behind the norm
};

struct LatentParams {
  const void* q_lat;            // T [H, R, r] contiguous
  const void* q;                // T [R, ldq]; rotated part of head h at h * dq + d
  int64_t ldq;
  int dq, d;
  const void* pool;             // T [blocks * 16, r + rd]
  const int32_t* table;         // [spans, ld_table] page numbers
  int64_t ld_table;
  const int32_t* seq_of;        // [R] span of a row (null: row r is span r)
  const int32_t* kv_len;        // [R] keys the row sees (its own included); 0 = idle row
  const float* sink;            // [H] or null
  void* out;                    // T [H, R, r]
  float* part;                  // split workspace: o [H, R, splits, r] then (m, l) [H, R, splits, 2]
  int H, R, r, rd, splits;
  float scale;
};

}  // namespace prl
