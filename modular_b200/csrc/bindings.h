// What the binding files share: error translation, the current stream, the process-wide error word.
#pragma once
#include <torch/extension.h>
#include <cuda_runtime.h>

namespace mb {
namespace bind {

cudaStream_t cur_stream();
void check_rc(int rc, const char* what);          // throws on anything but MB_OK
void need_cuda(const torch::Tensor& t, const char* name);
const void* optptr(const c10::optional<torch::Tensor>& t);
int* error_flag();
int num_sms();

}  // namespace bind

void bind_layers(pybind11::module_& m);           // bindings_layers.cpp

}  // namespace mb
