// Argument checks that the binding files share.
#pragma once

#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <cstdint>

namespace {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

[[maybe_unused]] void check_rc(int rc, const char* what) { TORCH_CHECK(rc == 0, what, " failed with code ", rc); }
[[maybe_unused]] cudaStream_t stream_of(const Tensor& t) { return at::cuda::getCurrentCUDAStream(t.get_device()).stream(); }
[[maybe_unused]] unsigned* status_word(const Tensor& status) {
  TORCH_CHECK(status.is_cuda() && status.scalar_type() == at::kInt && status.numel() >= 1, "status must be a CUDA int32 tensor");
  return reinterpret_cast<unsigned*>(status.data_ptr<int>());
}
// 1: fp32, 0: bf16
[[maybe_unused]] int elem(const Tensor& t) {
  TORCH_CHECK(t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16, "element type must be bfloat16 or float32");
  return t.scalar_type() == at::kFloat ? 1 : 0;
}
[[maybe_unused]] void need(const Tensor& t, at::ScalarType dtype, int64_t min_numel, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == dtype, what, ": contiguous CUDA tensor of the right type expected");
  TORCH_CHECK(t.numel() >= min_numel, what, ": too few elements (", t.numel(), " of ", min_numel, ")");
}
[[maybe_unused]] const int* ints(const Tensor& t, int64_t n, const char* what) {
  need(t, at::kInt, n, what);
  return t.data_ptr<int>();
}
[[maybe_unused]] float* floats(const Tensor& t, int64_t n, const char* what) {
  need(t, at::kFloat, n, what);
  return t.data_ptr<float>();
}
[[maybe_unused]] void* data(const Tensor& t, at::ScalarType dtype, int64_t n, const char* what) {
  need(t, dtype, n, what);
  return t.data_ptr();
}
[[maybe_unused]] int i32(int64_t v) {
  TORCH_CHECK(v >= INT32_MIN && v <= INT32_MAX, "value does not fit 32 bits");
  return static_cast<int>(v);
}

// A 2-D view [rows, cols] of unit inner stride, rows `ld` elements apart.
[[maybe_unused]] void* view2(const Tensor& t, at::ScalarType dtype, int64_t rows, int64_t cols, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == dtype && t.dim() == 2 && t.size(0) == rows && t.size(1) == cols && (t.stride(1) == 1 || cols == 1),
              what, ": CUDA view [", rows, ", ", cols, "] of the right type with unit inner stride expected");
  return t.data_ptr();
}

}  // namespace
