// Argument checks shared by the binding files.
#pragma once
#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>
#include <torch/extension.h>

#include "gemm.h"

namespace mb_bind {

inline cudaStream_t cur_stream() { return c10::cuda::getCurrentCUDAStream().stream(); }

#define CHECK_BF16(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kBFloat16 && (t).is_contiguous(), #t " must be a contiguous bf16 CUDA tensor")
#define CHECK_F32(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kFloat && (t).is_contiguous(), #t " must be a contiguous fp32 CUDA tensor")
#define CHECK_I32(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kInt && (t).is_contiguous(), #t " must be a contiguous int32 CUDA tensor")

template <typename T>
T* opt_ptr(const c10::optional<at::Tensor>& t) {
  return t.has_value() ? static_cast<T*>(t->data_ptr()) : nullptr;
}

inline void check_bf16_2d(const at::Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kBFloat16, name, " must be bf16");
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1, name, " must be 2-D with a contiguous inner dimension");
}

inline int* status_ptr(const c10::optional<at::Tensor>& status) {
  if (!status.has_value()) return nullptr;
  TORCH_CHECK(status->is_cuda() && status->scalar_type() == at::kInt, "status must be an int32 CUDA tensor");
  return status->data_ptr<int>();
}

inline mb::GemmOperand operand(const at::Tensor& t, bool mn_major) {
  mb::GemmOperand o;
  o.ptr = t.data_ptr();
  o.rows = t.size(0);
  o.cols = t.size(1);
  o.ld = t.stride(0);
  o.mn_major = mn_major;
  return o;
}

inline void fill_out(mb::GemmProblem& p, const at::Tensor& c) {
  TORCH_CHECK(c.is_cuda() && (c.scalar_type() == at::kBFloat16 || c.scalar_type() == at::kFloat),
              "output must be a bf16 or fp32 CUDA tensor");
  TORCH_CHECK(c.stride(-1) == 1, "output must have a contiguous inner dimension");
  p.c = c.data_ptr();
  p.out_fp32 = c.scalar_type() == at::kFloat;
}

}  // namespace mb_bind
