// Tensor checks shared by the torch bindings.
#pragma once
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

namespace {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

void chk(const Tensor& t, c10::ScalarType dt, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == dt, name, " has dtype ", t.scalar_type(), ", expected ", dt);
}
void chk_c(const Tensor& t, c10::ScalarType dt, const char* name) {
  chk(t, dt, name);
  TORCH_CHECK(t.is_contiguous(), name, " must be contiguous");
}
const void* cptr(const OptTensor& t) { return t.has_value() ? t->data_ptr() : nullptr; }
void* mptr(OptTensor& t) { return t.has_value() ? t->data_ptr() : nullptr; }
int* status_ptr(const OptTensor& s) {
  if (!s.has_value()) return nullptr;
  chk_c(*s, torch::kInt32, "status");
  return s->data_ptr<int>();
}

constexpr auto BF16 = torch::kBFloat16;
constexpr auto F32 = torch::kFloat32;
constexpr auto I32 = torch::kInt32;
constexpr auto U8 = torch::kUInt8;

}  // namespace
