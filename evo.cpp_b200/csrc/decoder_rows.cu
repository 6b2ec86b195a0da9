// Row operators of the decoder graph: embedding with learned positions, the norm of the F32 residual
// stream, the normalised polynomial activation, and the F32 projection of the F32 profile.
#include "decoder_types.cuh"
#include "ops_internal.hpp"

namespace evob {
namespace {

constexpr int kThreads = 256;
constexpr int kCached = 4;  // groups of eight elements a thread keeps between the two sweeps over its row

// One row as groups of eight: thread t owns groups t, t + kThreads, ...  The first kCached of them stay in
// registers between the statistics and the output sweep (rows of up to 8,192 elements read memory once).
template <typename Load, typename Store>
__device__ __forceinline__ void two_sweeps(const int groups, const Load &load, const Store &store,
                                           float *const scratch, const float inverse_width, const float epsilon) {
  float cached[kCached][8];
  float square = 0.0F;
#pragma unroll
  for (int c = 0; c < kCached; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) {
      load(group, cached[c]);
#pragma unroll
      for (int i = 0; i < 8; ++i) square = fmaf(cached[c][i], cached[c][i], square);
    }
  }
  for (int group = threadIdx.x + kCached * kThreads; group < groups; group += kThreads) {
    float v[8];
    load(group, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) square = fmaf(v[i], v[i], square);
  }
  const float total = block_sum<kThreads>(square, scratch);
  const float factor = 1.0F / sqrtf(total * inverse_width + epsilon);
#pragma unroll
  for (int c = 0; c < kCached; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) store(group, cached[c], factor);
  }
  for (int group = threadIdx.x + kCached * kThreads; group < groups; group += kThreads) {
    float v[8];
    load(group, v);
    store(group, v, factor);
  }
}

// kVector: width % 8 == 0 and 16-byte aligned rows.  Otherwise groups of eight with a ragged last one.
template <typename T, bool kVector>
__device__ __forceinline__ void load_group(const T *const row, const int group, const int width, float (&v)[8]) {
  if constexpr (kVector) {
    load_floats<8>(row + 8 * group, v);
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = 8 * group + i < width ? to_float(row[8 * group + i]) : 0.0F;
  }
}
template <typename T, bool kVector>
__device__ __forceinline__ void store_group(T *const row, const int group, const int width, const float (&v)[8]) {
  if constexpr (kVector) {
    store_floats(row + 8 * group, v);
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (8 * group + i < width) row[8 * group + i] = from_float<T>(v[i]);
  }
}

template <bool kVector>
__global__ void __launch_bounds__(kThreads)
embed_positions_kernel(const std::uint32_t *__restrict__ tokens, const bf16 *__restrict__ table,
                       const bf16 *__restrict__ positions, const float *__restrict__ gain, const int width,
                       const std::uint32_t vocabulary, const int position, const int *__restrict__ dynamic_position,
                       const float epsilon, float *__restrict__ output, int *const error_word) {
  __shared__ float scratch[kThreads / 32];
  const std::size_t row = blockIdx.x;
  const std::uint32_t token = tokens[row];
  float *const out = output + row * width;
  if (token >= vocabulary) {
    for (int i = threadIdx.x; i < width; i += kThreads) out[i] = 0.0F;
    if (threadIdx.x == 0) atomicOr(error_word, 2);
    return;
  }
  const std::size_t at = (dynamic_position != nullptr ? *dynamic_position : position) + row;
  const bf16 *const word = table + static_cast<std::size_t>(token) * width;
  const bf16 *const place = positions + at * width;
  two_sweeps(
      (width + 7) / 8,
      [&](const int group, float (&v)[8]) {
        float p[8];
        load_group<bf16, kVector>(word, group, width, v);
        load_group<bf16, kVector>(place, group, width, p);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] += p[i];
      },
      [&](const int group, const float (&v)[8], const float factor) {
        float g[8], y[8];
        load_group<float, kVector>(gain, group, width, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = v[i] * factor * g[i];
        store_group<float, kVector>(out, group, width, y);
      },
      scratch, 1.0F / static_cast<float>(width), epsilon);
}

template <typename T, bool kVector>
__global__ void __launch_bounds__(kThreads)
rms_norm_residual_kernel(const float *__restrict__ input, const float *__restrict__ gain, const int width,
                         const float epsilon, T *__restrict__ output) {
  __shared__ float scratch[kThreads / 32];
  const float *const x = input + static_cast<std::size_t>(blockIdx.x) * width;
  T *const out = output + static_cast<std::size_t>(blockIdx.x) * width;
  two_sweeps(
      (width + 7) / 8, [&](const int group, float (&v)[8]) { load_group<float, kVector>(x, group, width, v); },
      [&](const int group, const float (&v)[8], const float factor) {
        float g[8], y[8];
        load_group<float, kVector>(gain, group, width, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = v[i] * factor * g[i];
        store_group<T, kVector>(out, group, width, y);
      },
      scratch, 1.0F / static_cast<float>(width), epsilon);
}

template <typename T, bool kVector>
__global__ void __launch_bounds__(kThreads)
poly_norm_kernel(const T *input, const float *__restrict__ coefficients, const int width, const float epsilon,
                 T *output) {
  __shared__ float scratch[kThreads / 32];
  const T *const z = input + static_cast<std::size_t>(blockIdx.x) * width;
  T *const out = output + static_cast<std::size_t>(blockIdx.x) * width;
  const int groups = (width + 7) / 8;
  constexpr int kKept = kCached;
  float cached[kKept][8];
  float second = 0.0F, fourth = 0.0F, sixth = 0.0F;  // sums of z^2, z^4, z^6
  const auto add = [&](const float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float s = v[i] * v[i];
      second += s;
      fourth = fmaf(s, s, fourth);
      sixth = fmaf(s * s, s, sixth);
    }
  };
#pragma unroll
  for (int c = 0; c < kKept; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) {
      load_group<T, kVector>(z, group, width, cached[c]);
      add(cached[c]);
    }
  }
  for (int group = threadIdx.x + kKept * kThreads; group < groups; group += kThreads) {
    float v[8];
    load_group<T, kVector>(z, group, width, v);
    add(v);
  }
  const float inverse_width = 1.0F / static_cast<float>(width);
  second = block_sum<kThreads>(second, scratch);
  fourth = block_sum<kThreads>(fourth, scratch);
  sixth = block_sum<kThreads>(sixth, scratch);
  const float a = coefficients[0] * rsqrtf(second * inverse_width + epsilon);
  const float b = coefficients[1] * rsqrtf(fourth * inverse_width + epsilon);
  const float c3 = coefficients[2] * rsqrtf(sixth * inverse_width + epsilon);
  const float e = coefficients[3];
  const auto emit = [&](const int group, const float (&v)[8]) {
    float y[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = fmaf(fmaf(fmaf(c3, v[i], b), v[i], a), v[i], e);
    store_group<T, kVector>(out, group, width, y);
  };
#pragma unroll
  for (int c = 0; c < kKept; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) emit(group, cached[c]);
  }
  for (int group = threadIdx.x + kKept * kThreads; group < groups; group += kThreads) {
    float v[8];
    load_group<T, kVector>(z, group, width, v);
    emit(group, v);
  }
}

__global__ void __launch_bounds__(kThreads)
distance_bias_kernel(const float *__restrict__ r1, const float *__restrict__ r2, const int distances,
                     float *__restrict__ table) {
  const int head = blockIdx.y;
  for (int d = blockIdx.x * kThreads + threadIdx.x; d < distances; d += gridDim.x * kThreads)
    table[static_cast<std::size_t>(head) * distances + d] = r1[head] * logf(fmaf(r2[head], static_cast<float>(d), 1.0F));
}

// 64 x 64 output tile, 16 inputs per step, 4 x 4 products per thread; plain F32 multiply-adds, every step's 16
// products summed on their own before they join the running sum.
__global__ void __launch_bounds__(256)
linear_f32_kernel(const float *__restrict__ input, const bf16 *__restrict__ weight, float *__restrict__ output,
                  const int rows, const int out_features, const int in_features, const bool accumulate) {
  __shared__ float x_tile[16][68];
  __shared__ float w_tile[16][68];
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < in_features; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i / 16, k = i % 16;
      const bool inside = k0 + k < in_features;
      x_tile[k][r] = m0 + r < rows && inside ? input[static_cast<std::size_t>(m0 + r) * in_features + k0 + k] : 0.0F;
      w_tile[k][r] =
          n0 + r < out_features && inside ? bf2f(weight[static_cast<std::size_t>(n0 + r) * in_features + k0 + k]) : 0.0F;
    }
    __syncthreads();
    float step[4][4] = {};
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 x = *reinterpret_cast<const float4 *>(&x_tile[k][ty * 4]);
      const float4 w = *reinterpret_cast<const float4 *>(&w_tile[k][tx * 4]);
      const float xs[4] = {x.x, x.y, x.z, x.w}, ws[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) step[i][j] = fmaf(xs[i], ws[j], step[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += step[i][j];
    __syncthreads();
  }
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j) {
      const int row = m0 + ty * 4 + i, col = n0 + tx * 4 + j;
      if (row >= rows || col >= out_features) continue;
      float *const out = output + static_cast<std::size_t>(row) * out_features + col;
      *out = accumulate ? *out + acc[i][j] : acc[i][j];
    }
}

// Few rows: a warp per (row, output).
__global__ void __launch_bounds__(256)
linear_f32_rows_kernel(const float *__restrict__ input, const bf16 *__restrict__ weight, float *__restrict__ output,
                       const int out_features, const int in_features, const bool accumulate) {
  const int column = blockIdx.x * 8 + threadIdx.x / 32, lane = threadIdx.x % 32;
  if (column >= out_features) return;
  const float *const x = input + static_cast<std::size_t>(blockIdx.y) * in_features;
  const bf16 *const w = weight + static_cast<std::size_t>(column) * in_features;
  float sum = 0.0F;
  for (int k = lane; k < in_features; k += 32) sum = fmaf(x[k], bf2f(w[k]), sum);
  sum = warp_sum(sum);
  float *const out = output + static_cast<std::size_t>(blockIdx.y) * out_features + column;
  if (lane == 0) *out = accumulate ? *out + sum : sum;
}

bool row_vector_ok(const std::size_t width, const void *a, const void *b, const void *c) {
  return width % 8 == 0 && aligned16(a) && aligned16(b) && aligned16(c);
}

}  // namespace

int embed_positions(const std::uint32_t *tokens, const void *table, const void *positions, const float *gain,
                    const std::size_t rows, const std::size_t width, const std::size_t vocabulary,
                    const std::size_t position, const float epsilon, float *output, cudaStream_t stream,
                    const int *dynamic_position) {
  if (tokens == nullptr || table == nullptr || positions == nullptr || gain == nullptr || output == nullptr ||
      width == 0 || width > 0x7fffff00U || rows > 0x7fffffffU || position > 0x7fffffffU)
    return fail(kInvalidArgument, "embedding arguments are invalid");
  if (rows == 0) return kOk;
  int status = kOk;
  int *const error = device_error_word(&status);
  if (error == nullptr) return status;
  const bool vector = row_vector_ok(width, table, positions, output) && aligned16(gain);
  const auto kernel = vector ? embed_positions_kernel<true> : embed_positions_kernel<false>;
  kernel<<<static_cast<unsigned int>(rows), kThreads, 0, stream>>>(
      tokens, static_cast<const bf16 *>(table), static_cast<const bf16 *>(positions), gain, static_cast<int>(width),
      static_cast<std::uint32_t>(vocabulary), static_cast<int>(position), dynamic_position, epsilon, output, error);
  return check_launch("embedding kernel with positions");
}

int rms_norm_residual(const float *input, const float *gain, const std::size_t rows, const std::size_t width,
                      const float epsilon, void *output, const Activation type, cudaStream_t stream) {
  if (input == nullptr || gain == nullptr || output == nullptr || width == 0 || width > 0x7fffff00U ||
      rows > 0x7fffffffU)
    return fail(kInvalidArgument, "residual norm arguments are invalid");
  if (rows == 0) return kOk;
  const bool vector = row_vector_ok(width, input, gain, output);
  const unsigned int grid = static_cast<unsigned int>(rows);
  const int w = static_cast<int>(width);
  if (type == Activation::kBf16) {
    const auto kernel = vector ? rms_norm_residual_kernel<bf16, true> : rms_norm_residual_kernel<bf16, false>;
    kernel<<<grid, kThreads, 0, stream>>>(input, gain, w, epsilon, static_cast<bf16 *>(output));
  } else {
    const auto kernel = vector ? rms_norm_residual_kernel<float, true> : rms_norm_residual_kernel<float, false>;
    kernel<<<grid, kThreads, 0, stream>>>(input, gain, w, epsilon, static_cast<float *>(output));
  }
  return check_launch("residual norm kernel");
}

int poly_norm(const void *input, const float *coefficients, const std::size_t rows, const std::size_t width,
              const float epsilon, void *output, const Activation type, cudaStream_t stream) {
  if (input == nullptr || coefficients == nullptr || output == nullptr || width == 0 || width > 0x7fffff00U ||
      rows > 0x7fffffffU)
    return fail(kInvalidArgument, "polynomial activation arguments are invalid");
  if (rows == 0) return kOk;
  const bool vector = row_vector_ok(width, input, output, nullptr);
  const unsigned int grid = static_cast<unsigned int>(rows);
  const int w = static_cast<int>(width);
  if (type == Activation::kBf16) {
    const auto kernel = vector ? poly_norm_kernel<bf16, true> : poly_norm_kernel<bf16, false>;
    kernel<<<grid, kThreads, 0, stream>>>(static_cast<const bf16 *>(input), coefficients, w, epsilon,
                                          static_cast<bf16 *>(output));
  } else {
    const auto kernel = vector ? poly_norm_kernel<float, true> : poly_norm_kernel<float, false>;
    kernel<<<grid, kThreads, 0, stream>>>(static_cast<const float *>(input), coefficients, w, epsilon,
                                          static_cast<float *>(output));
  }
  return check_launch("polynomial activation kernel");
}

int distance_bias_table(const float *r1, const float *r2, const std::size_t heads, const std::size_t distances,
                        float *table, cudaStream_t stream) {
  if (r1 == nullptr || r2 == nullptr || table == nullptr || heads == 0 || heads > 65535 || distances == 0 ||
      distances > 0x7fffff00U)
    return fail(kInvalidArgument, "distance bias arguments are invalid");
  const dim3 grid(ceil_div_u(distances, kThreads) > 64 ? 64 : ceil_div_u(distances, kThreads),
                  static_cast<unsigned int>(heads));
  distance_bias_kernel<<<grid, kThreads, 0, stream>>>(r1, r2, static_cast<int>(distances), table);
  return check_launch("distance bias kernel");
}

int linear_f32(const float *input, const void *weight, const std::size_t rows, const std::size_t in_features,
               const std::size_t out_features, float *output, const bool accumulate, cudaStream_t stream) {
  if (input == nullptr || weight == nullptr || output == nullptr || in_features == 0 || out_features == 0 ||
      in_features > 0x7fffff00U || out_features > 0x7fffff00U || rows > 64 * 65535U)
    return fail(kInvalidArgument, "F32 linear arguments are invalid");
  if (rows == 0) return kOk;
  if (rows <= 16) {
    const dim3 grid(ceil_div_u(out_features, 8), static_cast<unsigned int>(rows));
    linear_f32_rows_kernel<<<grid, 256, 0, stream>>>(input, static_cast<const bf16 *>(weight), output,
                                                     static_cast<int>(out_features), static_cast<int>(in_features),
                                                     accumulate);
    return check_launch("F32 linear kernel (few rows)");
  }
  const dim3 grid(ceil_div_u(out_features, 64), ceil_div_u(rows, 64));
  linear_f32_kernel<<<grid, 256, 0, stream>>>(input, static_cast<const bf16 *>(weight), output, static_cast<int>(rows),
                                              static_cast<int>(out_features), static_cast<int>(in_features),
                                              accumulate);
  return check_launch("F32 linear kernel");
}

}  // namespace evob
