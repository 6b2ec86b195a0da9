// Device helpers of the decoder kernels: the two storage types of activations and the scalar functions of
// the gates, evaluated in F32.
#pragma once

#include "common.cuh"
#include "decoder_ops.hpp"

namespace evob {

__device__ __forceinline__ float to_float(const bf16 v) { return bf2f(v); }
__device__ __forceinline__ float to_float(const float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_float(const float v);
template <>
__device__ __forceinline__ bf16 from_float<bf16>(const float v) { return f2bf(v); }
template <>
__device__ __forceinline__ float from_float<float>(const float v) { return v; }

// kCount consecutive elements of an aligned row as F32, through 16-byte accesses where they fit.
template <int kCount>
__device__ __forceinline__ void load_floats(const float *const p, float (&v)[kCount]) {
  static_assert(kCount % 4 == 0, "whole 16-byte words");
#pragma unroll
  for (int i = 0; i < kCount / 4; ++i) {
    const float4 w = reinterpret_cast<const float4 *>(p)[i];
    v[4 * i] = w.x;
    v[4 * i + 1] = w.y;
    v[4 * i + 2] = w.z;
    v[4 * i + 3] = w.w;
  }
}
template <int kCount>
__device__ __forceinline__ void load_floats(const bf16 *const p, float (&v)[kCount]) {
  static_assert(kCount % 8 == 0, "whole 16-byte words");
#pragma unroll
  for (int i = 0; i < kCount / 8; ++i) {
    Bf16x8 w;
    w.raw = reinterpret_cast<const uint4 *>(p)[i];
#pragma unroll
    for (int j = 0; j < 8; ++j) v[8 * i + j] = w.get(j);
  }
}
__device__ __forceinline__ void store_floats(float *const p, const float (&v)[8]) {
  reinterpret_cast<float4 *>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4 *>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store_floats(bf16 *const p, const float (&v)[8]) {
  *reinterpret_cast<uint4 *>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]),
                                             pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}

// Four consecutive elements.
__device__ __forceinline__ void load_quad(const float *const p, float (&v)[4]) {
  const float4 w = *reinterpret_cast<const float4 *>(p);
  v[0] = w.x, v[1] = w.y, v[2] = w.z, v[3] = w.w;
}
__device__ __forceinline__ void load_quad(const bf16 *const p, float (&v)[4]) {
  const uint2 w = *reinterpret_cast<const uint2 *>(p);
  v[0] = __uint_as_float(w.x << 16U), v[1] = __uint_as_float(w.x & 0xffff0000U);
  v[2] = __uint_as_float(w.y << 16U), v[3] = __uint_as_float(w.y & 0xffff0000U);
}
__device__ __forceinline__ void store_quad(float *const p, const float (&v)[4]) {
  *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_quad(bf16 *const p, const float (&v)[4]) {
  *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}

__device__ __forceinline__ float sigmoid_f32(const float x) { return 1.0F / (1.0F + expf(-x)); }
// (the quotient is good to two units in the last place and wants a divisor below 2^126)
__device__ __forceinline__ float silu_f32(const float x) { return __fdividef(x, 1.0F + expf(-fmaxf(x, -80.0F))); }
// ln(1 + e^x) without overflow or cancellation
__device__ __forceinline__ float softplus_f32(const float x) { return fmaxf(x, 0.0F) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int offset = 16; offset > 0; offset /= 2) v += __shfl_xor_sync(0xffffffffU, v, offset);
  return v;
}

// Sum over the CTA, returned to every thread.  `scratch` holds one float per warp and is free again after
// the call's second barrier.
template <int kThreads>
__device__ __forceinline__ float block_sum(float v, float *const scratch) {
  v = warp_sum(v);
  if (threadIdx.x % 32 == 0) scratch[threadIdx.x / 32] = v;
  __syncthreads();
  float total = 0.0F;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) total += scratch[w];
  __syncthreads();
  return total;
}

inline bool aligned16(const void *const p) { return (reinterpret_cast<std::uintptr_t>(p) & 15U) == 0; }

}  // namespace evob
