// polyrl_b200 — launch parameters of the sequence-mixer kernels (plain pointers; shared by kernels and bindings).
#pragma once
#include <cstdint>

namespace prl {

struct ScanParams {
  const void *q, *k, *v;        // T; row pitches in elements; head h of q / k starts at (h / rep) * N, of v at h * V
  int64_t ldq, ldk, ldv;
  int rep;
  const float *g0, *g1;         // raw gate projections [tokens, ldg], one column per head
  int64_t ldg;
  const float *b0, *b1;         // their biases [H]
  const float *a_log, *d_skip;  // kSsd, kDelta (a_log only) [H]
  float qscale, cap;            // q is multiplied by qscale; cap bounds the kMlstm gates
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
