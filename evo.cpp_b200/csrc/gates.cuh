// Scalar functions that projections apply to their F32 accumulators.
#pragma once

#include "common.cuh"
#include "ops_internal.hpp"

namespace evob {

__device__ __forceinline__ float soft_cap(const float x, const float cap) { return cap > 0.0F ? cap * tanhf(x / cap) : x; }

// kGateRelu: max(gate, 0) up.  kGateClamped: g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u = up
// clamped to +-limit.  (the quotient is good to two units in the last place; beyond its range the value is 0)
__device__ __forceinline__ float gated_value(const int mode, const float limit, const float gate, const float up) {
  if (mode == kGateRelu) return fmaxf(gate, 0.0F) * up;
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g, 1.0F + expf(-1.702F * g)) * (u + 1.0F);
}

}  // namespace evob
