// Shared pieces of the weight loaders: the expected tensor of a design, and the cursor that lays the
// tensors of a stage out in its device slab.
#pragma once

#include <cuda_runtime.h>

#include <cstring>
#include <deque>
#include <string>
#include <vector>

#include "../common.cuh"
#include "model.hpp"

namespace evob {

constexpr std::size_t kWeightAlign = 256;
inline std::size_t weight_aligned(const std::size_t bytes) {
  return (bytes + kWeightAlign - 1) / kWeightAlign * kWeightAlign;
}

struct ExpectedTensor {
  std::string name;
  TensorType type;
  std::vector<std::size_t> shape;
};

inline int lookup_tensor(const ModelFile &file, const ExpectedTensor &e, const TensorView **out) {
  const TensorView *tensor = file.find(e.name);
  if (tensor == nullptr) return fail(kModelFormat, "required tensor is missing: " + e.name);
  if (tensor->type != e.type || tensor->shape != e.shape)
    return fail(kModelFormat, "tensor has an unexpected dtype or shape: " + e.name);
  *out = tensor;
  return kOk;
}

// Elements of a BF16 tensor widened to F32 (the mapping need not be aligned).
inline std::vector<float> widened(const TensorView &t) {
  std::vector<float> values(t.elements());
  for (std::size_t i = 0; i < values.size(); ++i) {
    std::uint16_t raw;
    std::memcpy(&raw, t.data + 2 * i, 2);
    const std::uint32_t bits = static_cast<std::uint32_t>(raw) << 16U;
    std::memcpy(&values[i], &bits, 4);
  }
  return values;
}

// Cursor over a stage slab: a dry run measures it, the second pass copies.
struct WeightUploader {
  unsigned char *base = nullptr;
  std::size_t offset = 0;
  cudaStream_t stream = nullptr;
  bool dry_run = true;
  std::deque<std::vector<float>> staged;  // host values that copies in flight still read

  void *place(const std::size_t bytes) {
    void *p = dry_run ? nullptr : base + offset;
    offset += weight_aligned(bytes);
    return p;
  }
  int copy(void *dst, const void *src, const std::size_t bytes) {
    if (dry_run || bytes == 0) return kOk;
    if (cudaMemcpyAsync(dst, src, bytes, cudaMemcpyHostToDevice, stream) != cudaSuccess)
      return fail(kCuda, "weight upload failed");
    return kOk;
  }
  // `rows` rows of row_bytes, source_pitch apart, to rows `pitch` apart.
  int copy_rows(void *dst, const std::size_t pitch, const void *src, const std::size_t source_pitch,
                const std::size_t row_bytes, const std::size_t rows) {
    if (dry_run || rows == 0 || row_bytes == 0) return kOk;
    if (cudaMemcpy2DAsync(dst, pitch, src, source_pitch, row_bytes, rows, cudaMemcpyHostToDevice, stream) != cudaSuccess)
      return fail(kCuda, "weight upload failed");
    return kOk;
  }
  // A piece of the slab filled with zeros.
  int zeros(const std::size_t bytes, unsigned char **out) {
    *out = static_cast<unsigned char *>(place(bytes));
    if (!dry_run && cudaMemsetAsync(*out, 0, bytes, stream) != cudaSuccess) return fail(kCuda, "weight upload failed");
    return kOk;
  }
  int tensor(const TensorView &t, const void **out) {
    void *dst = place(t.bytes);
    *out = dst;
    return copy(dst, t.data, t.bytes);
  }
  int floats(std::vector<float> values, const float **out) {
    const std::size_t bytes = values.size() * sizeof(float);
    void *dst = place(bytes);
    *out = static_cast<const float *>(dst);
    if (dry_run) return kOk;
    staged.push_back(std::move(values));
    return copy(dst, staged.back().data(), bytes);
  }
};

}  // namespace evob
