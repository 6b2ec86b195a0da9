// Scalar functions that projections apply to their F32 accumulators.
#pragma once

#include "common.cuh"
#include "ops_internal.hpp"

namespace evob {

__device__ __forceinline__ float soft_cap(const float x, const float cap) { return cap > 0.0F ? cap * tanhf(x / cap) : x; }
// The same for epilogues of BF16 products: tanh through one exponential (absolute error a few 1e-7 of the cap).
__device__ __forceinline__ float fast_soft_cap(const float x, const float cap) {
  if (!(cap > 0.0F)) return x;
  const float e = __expf(fminf(__fdividef(2.0F * x, cap), 80.0F));
  return fmaf(-2.0F * cap, __fdividef(1.0F, e + 1.0F), cap);
}

// max(gate, 0) up, and g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u = up clamped to +-limit.  (the
// quotient is good to two units in the last place; beyond its range the value is 0)
__device__ __forceinline__ float relu_gate(const float gate, const float up) { return fmaxf(gate, 0.0F) * up; }
template <bool kFast = false>
__device__ __forceinline__ float clamped_gate(const float limit, const float gate, const float up) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  const float e = kFast ? __expf(-1.702F * g) : expf(-1.702F * g);
  return __fdividef(g, 1.0F + e) * (u + 1.0F);
}
__device__ __forceinline__ float gated_value(const int mode, const float limit, const float gate, const float up) {
  return mode == kGateRelu ? relu_gate(gate, up) : clamped_gate(limit, gate, up);
}

}  // namespace evob
