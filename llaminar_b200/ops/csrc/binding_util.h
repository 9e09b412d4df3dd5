// Checks and conversions shared by the small Python bindings.  Every tensor is checked on the host before a launch.
#pragma once
#include <ATen/cuda/CUDAContext.h>
#include <torch/extension.h>

namespace llm_binding {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

inline cudaStream_t stream() { return at::cuda::getCurrentCUDAStream().stream(); }

inline void check(cudaError_t e, const char* what) { TORCH_CHECK(e == cudaSuccess, what, ": ", cudaGetErrorString(e)); }

inline bool is_f32(const Tensor& t, const char* name) {
    TORCH_CHECK(t.is_cuda(), name, " must be on the GPU");
    TORCH_CHECK(t.scalar_type() == torch::kFloat32 || t.scalar_type() == torch::kBFloat16, name, " must be float32 or bfloat16");
    return t.scalar_type() == torch::kFloat32;
}
inline void want(const Tensor& t, torch::ScalarType st, const char* name) {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == st && t.is_contiguous(), name, " must be a contiguous ", st, " CUDA tensor");
}
inline void want_like(const Tensor& t, bool f32, const char* name) {
    TORCH_CHECK(is_f32(t, name) == f32, name, " has the wrong element type");
}
inline const int* ints(const Tensor& t, const char* name) {
    want(t, torch::kInt32, name);
    return t.data_ptr<int>();
}
inline const float* floats(const Tensor& t, int64_t n, const char* name) {
    want(t, torch::kFloat32, name);
    TORCH_CHECK(t.numel() == n, name, " must hold ", n, " values");
    return t.data_ptr<float>();
}
inline const float2* angle_ptr(const Tensor& t, int64_t rows) {
    want(t, torch::kFloat32, "angles");
    TORCH_CHECK(t.dim() == 3 && t.size(0) >= rows && t.size(2) == 2, "angles must be [rows, dims/2, 2]");
    return reinterpret_cast<const float2*>(t.data_ptr<float>());
}

}  // namespace llm_binding
