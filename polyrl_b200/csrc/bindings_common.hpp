// polyrl_b200 — what the binding translation units share.
#pragma once
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <cstdint>
#include <string>
#include <vector>

namespace {

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

inline void check(int rc, const char* what) {
  TORCH_CHECK(rc == 0, "polyrl_b200 kernel '", what, "' failed with code ", rc);
}
#define CHECK_BF16(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kBFloat16, #t " must be a CUDA bf16 tensor")
#define CHECK_F32(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kFloat, #t " must be a CUDA fp32 tensor")
#define CHECK_LASTDIM(t) TORCH_CHECK((t).stride(-1) == 1, #t " must be contiguous in the last dim")

}  // namespace
