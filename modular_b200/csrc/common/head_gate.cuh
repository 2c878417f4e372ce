// Output gate of attention heads, applied where a kernel normalises its output: gate_mult * sigmoid(gate[token, head]).
#pragma once
#include "api.h"
#include "scalar.cuh"

namespace mb {

struct HeadGate {
  const void* g = nullptr;
  int ld = 0;
  float mult = 1.f;
  HeadGate() = default;
  explicit HeadGate(const MbAttnOptions* o) {
    if (o != nullptr && o->gate != nullptr) { g = o->gate; ld = o->ld_gate; mult = o->gate_mult; }
  }
  // the factor on head `head` of token row `t`
  template <typename T>
  __device__ __forceinline__ float of(long long t, int head) const {
    if (g == nullptr) return 1.f;
    return mult * sigmoidf(ldf(static_cast<const T*>(g) + t * ld + head));
  }
  __device__ __forceinline__ float operator()(long long t, int head) const { return of<__nv_bfloat16>(t, head); }
};

}  // namespace mb
