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
