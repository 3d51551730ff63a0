// polyrl_b200 — pieces of the tcgen05 recurrence kernels: bounded barrier waits, 128B-swizzled bf16 tiles, hi + lo bf16 pairs, tensor maps.
#pragma once
#include "mixers.cuh"

namespace prl {

__device__ __forceinline__ bool tc_wait(uint64_t* bar, uint32_t parity) {
  if (mbar_try_wait(bar, parity)) return true;
  const long long t0 = clock64();
  while (!mbar_try_wait(bar, parity)) {
    if (clock64() - t0 > 4000000000ll) return false;                  // about two seconds
  }
  return true;
}
__device__ __forceinline__ void tc_cp16(void* dst, const void* src, bool ok) {      // 16 bytes, zeros when not ok (src stays a valid address)
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void tc_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void tc_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }
// one ROWS x 64 tile: rows [0, nv) x columns [c0, c0 + 64) of src (columns below n), zero elsewhere
template <int ROWS, int THREADS>
__device__ __forceinline__ void tc_load_rows(uint8_t* dst, const __nv_bfloat16* src, int64_t ld, int nv, int c0, int n) {
#pragma unroll
  for (int i = 0; i < ROWS * 8 / THREADS; ++i) {
    const int idx = threadIdx.x + i * THREADS, r = idx >> 3, u = idx & 7, c = c0 + u * 8;
    const bool ok = r < nv && c < n;
    tc_cp16(dst + r * 128 + ((u ^ (r & 7)) << 4), src + (ok ? static_cast<int64_t>(r) * ld + c : 0), ok);
  }
}
__device__ __forceinline__ uint4 tc_ld16(const uint8_t* tile, int r, int u) {
  return *reinterpret_cast<const uint4*>(tile + r * 128 + ((u ^ (r & 7)) << 4));
}
__device__ __forceinline__ void tc_st16(uint8_t* tile, int r, int u, const uint32_t (&q)[4]) {
  *reinterpret_cast<uint4*>(tile + r * 128 + ((u ^ (r & 7)) << 4)) = make_uint4(q[0], q[1], q[2], q[3]);
}
__device__ __forceinline__ void tc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  const float2 h = unpack_bf16(hi);
  lo = pack_bf16(a - h.x, b - h.y);
}

using TcEncodeFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
// rows [tokens, heads * width] of pitch ld -> boxes of `rows` tokens x 1 head x box columns, zeros beyond the head's width
inline int tc_tokens_tmap(CUtensorMap* m, const void* ptr, int64_t tokens, int heads, int width, int64_t ld, int rows, int box, bool swizzle) {
  ensure_thread_ctx();
  static TcEncodeFn fn = nullptr;
  if (!fn) {
    void* q = nullptr;
    cudaDriverEntryPointQueryResult qr;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &q, cudaEnableDefault, &qr) != cudaSuccess || !q) return -1;
    fn = reinterpret_cast<TcEncodeFn>(q);
  }
  const cuuint64_t dim[3] = {static_cast<cuuint64_t>(width), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(tokens)};
  const cuuint64_t stride[2] = {static_cast<cuuint64_t>(width) * 2, static_cast<cuuint64_t>(ld) * 2};
  const cuuint32_t bx[3] = {static_cast<cuuint32_t>(box), 1, static_cast<cuuint32_t>(rows)}, one[3] = {1, 1, 1};
  const CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dim, stride, bx, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
                        swizzle ? CU_TENSOR_MAP_SWIZZLE_128B : CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : -static_cast<int>(r);
}

}  // namespace prl
