// Row operators of the decoder graph: embeddings (with and without learned positions), the norms of the F32
// residual stream and of what is added to it, the activations of the feed-forwards, and the F32 projection of
// the F32 profile.
#include "decoder_types.cuh"
#include "gates.cuh"
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

template <typename T, bool kVector>
__global__ void __launch_bounds__(kThreads)
embed_rows_kernel(const std::uint32_t *__restrict__ tokens, const bf16 *__restrict__ table, const int width,
                  const std::uint32_t vocabulary, float *__restrict__ stream_rows, T *__restrict__ copy,
                  int *const error_word) {
  const std::size_t row = blockIdx.x;
  const std::uint32_t token = tokens[row];
  const bool known = token < vocabulary;
  if (!known && threadIdx.x == 0) atomicOr(error_word, 2);
  const bf16 *const word = table + static_cast<std::size_t>(known ? token : 0U) * width;
  for (int group = threadIdx.x; group < (width + 7) / 8; group += kThreads) {
    float v[8];
    load_group<bf16, kVector>(word, group, width, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = known ? v[i] : 0.0F;
    store_group<float, kVector>(stream_rows + row * width, group, width, v);
    if (copy != nullptr) store_group<T, kVector>(copy + row * width, group, width, v);
  }
}

struct LayerNormParams {
  const int *slots;
  int parts;
  const float *gain;
  float *residual;
  int width;
  float epsilon;
};

// Mean and variance from the row itself (two sweeps over registers), one read and one write of the residual.  A
// thread keeps kKeep groups of eight elements between the sweeps.
template <typename In, typename Out, bool kVector, int kKeep>
__global__ void __launch_bounds__(kThreads)
layer_norm_kernel(const In *__restrict__ input, Out *__restrict__ output, const LayerNormParams p) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float scratch[kThreads / 32];
  const std::size_t row = blockIdx.x;
  const int groups = (p.width + 7) / 8;
  const float inverse_width = 1.0F / static_cast<float>(p.width);
  const auto load = [&](const int group, float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = 0.0F;
    for (int k = 0; k < p.parts; ++k) {
      const std::size_t pair = row * p.parts + k;
      const std::size_t at = p.slots != nullptr ? static_cast<std::size_t>(p.slots[pair]) : pair;
      float w[8];
      load_group<In, kVector>(input + at * p.width, group, p.width, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] += w[i];
    }
  };
  const auto live = [&](const int group, const int i) { return kVector || 8 * group + i < p.width; };
  float cached[kKeep][8], old[kKeep][8];
  float sum = 0.0F;
#pragma unroll
  for (int c = 0; c < kKeep; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) {
      load(group, cached[c]);
      if (p.residual != nullptr) load_group<float, kVector>(p.residual + row * p.width, group, p.width, old[c]);
#pragma unroll
      for (int i = 0; i < 8; ++i) sum += cached[c][i];
    }
  }
  for (int group = threadIdx.x + kKeep * kThreads; group < groups; group += kThreads) {
    float v[8];
    load(group, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) sum += v[i];
  }
  const float mean = block_sum<kThreads>(sum, scratch) * inverse_width;
  float square = 0.0F;
  const auto deviate = [&](const int group, const float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float d = live(group, i) ? v[i] - mean : 0.0F;
      square = fmaf(d, d, square);
    }
  };
#pragma unroll
  for (int c = 0; c < kKeep; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) deviate(group, cached[c]);
  }
  for (int group = threadIdx.x + kKeep * kThreads; group < groups; group += kThreads) {
    float v[8];
    load(group, v);
    deviate(group, v);
  }
  const float factor = 1.0F / sqrtf(block_sum<kThreads>(square, scratch) * inverse_width + p.epsilon);
  const auto emit = [&](const int group, const float (&v)[8], const float (&before)[8]) {
    float g[8], y[8];
    load_group<float, kVector>(p.gain, group, p.width, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = (v[i] - mean) * factor * g[i];
    if (p.residual != nullptr) {
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] += before[i];
      store_group<float, kVector>(p.residual + row * p.width, group, p.width, y);
    }
    if (output != nullptr) store_group<Out, kVector>(output + row * p.width, group, p.width, y);
  };
#pragma unroll
  for (int c = 0; c < kKeep; ++c) {
    const int group = threadIdx.x + c * kThreads;
    if (group < groups) emit(group, cached[c], old[c]);
  }
  for (int group = threadIdx.x + kKeep * kThreads; group < groups; group += kThreads) {
    float v[8], before[8] = {};
    load(group, v);
    if (p.residual != nullptr) load_group<float, kVector>(p.residual + row * p.width, group, p.width, before);
    emit(group, v, before);
  }
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
convert_kernel(const float *__restrict__ input, T *__restrict__ output, const std::size_t elements) {
  const std::size_t stride = static_cast<std::size_t>(gridDim.x) * kThreads;
  for (std::size_t i = static_cast<std::size_t>(blockIdx.x) * kThreads + threadIdx.x; i < elements; i += stride)
    output[i] = from_float<T>(input[i]);
}

// One row of one 128-column block of the output per iteration.
template <typename T>
__global__ void __launch_bounds__(128)
gated_activation_kernel(const float *__restrict__ input, T *__restrict__ output, const int gate, const float limit,
                        const std::size_t rows, const int inner, const int *__restrict__ tile_count, const int tile_rows) {
  std::size_t live = rows;
  if (tile_count != nullptr) {
    const std::size_t used = static_cast<std::size_t>(*tile_count) * tile_rows;
    live = used < rows ? used : rows;
  }
  const int block = blockIdx.y, column = block * 128 + static_cast<int>(threadIdx.x);
  for (std::size_t row = blockIdx.x; row < live; row += gridDim.x) {
    const float *const pair = input + row * 2 * inner + 256 * block + threadIdx.x;
    output[row * inner + column] = from_float<T>(gated_value(gate, limit, pair[0], pair[128]));
  }
}

struct F32Params {
  const bf16 *weight;
  float *output;
  int rows, out_features, in_features, accumulate;
  float alpha, softcap;
  const float *row_scale, *bias;
  const int *row_group;
  int row_fanout;
  const int *tile_group, *tile_count;
  int tile_rows;
};

__device__ __forceinline__ void store_f32_result(const F32Params &p, const std::size_t row, const int column,
                                                 const float product) {
  float *const out = p.output + row * p.out_features + column;
  float value = product * (p.row_scale != nullptr ? p.alpha * p.row_scale[row] : p.alpha);
  if (p.accumulate != 0) value += *out;
  if (p.bias != nullptr) value += p.bias[column];
  *out = soft_cap(value, p.softcap);
}

// 64 x 64 output tile, 16 inputs per step, 4 x 4 products per thread; plain F32 multiply-adds, every step's 16
// products summed on their own before they join the running sum.
template <typename T>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const T *__restrict__ input, const F32Params p) {
  __shared__ float x_tile[16][68];
  __shared__ float w_tile[16][68];
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const bf16 *weight = p.weight;
  if (p.tile_group != nullptr) {
    const int tile = m0 / p.tile_rows;
    if (tile >= *p.tile_count) return;
    weight += static_cast<std::size_t>(p.tile_group[tile]) * p.out_features * p.in_features;
  }
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.in_features; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i / 16, k = i % 16;
      const bool inside = k0 + k < p.in_features;
      x_tile[k][r] =
          m0 + r < p.rows && inside ? to_float(input[static_cast<std::size_t>(m0 + r) * p.in_features + k0 + k]) : 0.0F;
      w_tile[k][r] = n0 + r < p.out_features && inside
                         ? bf2f(weight[static_cast<std::size_t>(n0 + r) * p.in_features + k0 + k])
                         : 0.0F;
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
      if (row < p.rows && col < p.out_features) store_f32_result(p, static_cast<std::size_t>(row), col, acc[i][j]);
    }
}

// Few rows: a warp per (row, output).
template <typename T>
__global__ void __launch_bounds__(256)
linear_f32_rows_kernel(const T *__restrict__ input, const F32Params p) {
  const int column = blockIdx.x * 8 + threadIdx.x / 32, lane = threadIdx.x % 32;
  if (column >= p.out_features) return;
  const std::size_t row = blockIdx.y;
  const T *const x = input + row / p.row_fanout * p.in_features;
  const std::size_t group = p.row_group != nullptr ? static_cast<std::size_t>(p.row_group[row]) : 0;
  const bf16 *const w = p.weight + (group * p.out_features + column) * p.in_features;
  float sum = 0.0F;
  for (int k = lane; k < p.in_features; k += 32) sum = fmaf(to_float(x[k]), bf2f(w[k]), sum);
  sum = warp_sum(sum);
  if (lane == 0) store_f32_result(p, row, column, sum);
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

int embed_rows(const std::uint32_t *tokens, const void *table, const std::size_t rows, const std::size_t width,
               const std::size_t vocabulary, float *stream_rows, void *copy, const Activation type, cudaStream_t stream) {
  if (tokens == nullptr || table == nullptr || stream_rows == nullptr || width == 0 || width > 0x7fffff00U ||
      rows > 0x7fffffffU)
    return fail(kInvalidArgument, "embedding arguments are invalid");
  if (rows == 0) return kOk;
  int status = kOk;
  int *const error = device_error_word(&status);
  if (error == nullptr) return status;
  const bool vector = row_vector_ok(width, table, stream_rows, copy);
  const auto launch = [&](auto tag) {
    using T = decltype(tag);
    const auto kernel = vector ? embed_rows_kernel<T, true> : embed_rows_kernel<T, false>;
    kernel<<<static_cast<unsigned int>(rows), kThreads, 0, stream>>>(tokens, static_cast<const bf16 *>(table),
                                                                     static_cast<int>(width),
                                                                     static_cast<std::uint32_t>(vocabulary), stream_rows,
                                                                     static_cast<T *>(copy), error);
  };
  if (type == Activation::kBf16) launch(bf16{});
  else launch(float{});
  return check_launch("embedding kernel of the residual stream");
}

int layer_norm(const LayerNormArgs &a, cudaStream_t stream) {
  if (a.input == nullptr || a.gain == nullptr || (a.residual == nullptr && a.output == nullptr) || a.parts == 0 ||
      a.parts > 0x7fffffffU || a.width == 0 || a.width > 0x7fffff00U || a.rows > 0x7fffffffU)
    return fail(kInvalidArgument, "layer norm arguments are invalid");
  if (a.rows == 0) return kOk;
  const bool vector = row_vector_ok(a.width, a.input, a.gain, a.output) && aligned16(a.residual);
  LayerNormParams p{};
  p.slots = a.slots;
  p.parts = static_cast<int>(a.parts);
  p.gain = a.gain;
  p.residual = a.residual;
  p.width = static_cast<int>(a.width);
  p.epsilon = a.epsilon;
  const auto launch = [&](auto in_tag, auto out_tag) {
    using In = decltype(in_tag);
    using Out = decltype(out_tag);
    const auto kernel = !vector                      ? layer_norm_kernel<In, Out, false, kCached>
                        : a.width <= 8 * kThreads  ? layer_norm_kernel<In, Out, true, 1>
                        : a.width <= 16 * kThreads ? layer_norm_kernel<In, Out, true, 2>
                                                   : layer_norm_kernel<In, Out, true, kCached>;
    kernel<<<static_cast<unsigned int>(a.rows), kThreads, 0, stream>>>(static_cast<const In *>(a.input),
                                                                       static_cast<Out *>(a.output), p);
  };
  if (a.input_type == Activation::kBf16) {
    if (a.output_type == Activation::kBf16) launch(bf16{}, bf16{});
    else launch(bf16{}, float{});
  } else {
    if (a.output_type == Activation::kBf16) launch(float{}, bf16{});
    else launch(float{}, float{});
  }
  return check_launch("layer norm kernel");
}

int convert_rows(const float *input, const std::size_t elements, void *output, const Activation type, cudaStream_t stream) {
  if (input == nullptr || output == nullptr) return fail(kInvalidArgument, "conversion arguments are invalid");
  if (elements == 0) return kOk;
  const std::size_t blocks = (elements + kThreads - 1) / kThreads;
  const unsigned int grid = static_cast<unsigned int>(blocks < 8 * kSmCount ? blocks : 8 * kSmCount);
  if (type == Activation::kBf16)
    convert_kernel<<<grid, kThreads, 0, stream>>>(input, static_cast<bf16 *>(output), elements);
  else
    convert_kernel<<<grid, kThreads, 0, stream>>>(input, static_cast<float *>(output), elements);
  return check_launch("conversion kernel");
}

int gated_activation(const float *input, const int gate, const float limit, const std::size_t rows,
                     const std::size_t inner, void *output, const Activation type, const int *tile_count,
                     const std::size_t tile_rows, cudaStream_t stream) {
  if (input == nullptr || output == nullptr || (gate != kGateRelu && gate != kGateClamped) || inner == 0 || inner % 128 != 0 ||
      inner / 128 > 65535 || inner > 0x3fffff00U || tile_rows > 0x7fffffffU)
    return fail(kInvalidArgument, "gated activation arguments are invalid");
  if (rows == 0) return kOk;
  const dim3 grid(static_cast<unsigned int>(rows < 65536 ? rows : 65536), static_cast<unsigned int>(inner / 128));
  if (type == Activation::kBf16)
    gated_activation_kernel<<<grid, 128, 0, stream>>>(input, static_cast<bf16 *>(output), gate, limit, rows,
                                                      static_cast<int>(inner), tile_count, static_cast<int>(tile_rows));
  else
    gated_activation_kernel<<<grid, 128, 0, stream>>>(input, static_cast<float *>(output), gate, limit, rows,
                                                      static_cast<int>(inner), tile_count, static_cast<int>(tile_rows));
  return check_launch("gated activation kernel");
}

int linear_f32(const LinearF32Args &a, cudaStream_t stream) {
  if (a.input == nullptr || a.weight == nullptr || a.output == nullptr || a.in_features == 0 || a.out_features == 0 ||
      a.in_features > 0x7fffff00U || a.out_features > 0x7fffff00U || a.rows > 64 * 65535U || a.row_fanout == 0 ||
      (a.tile_group != nullptr && (a.tile_count == nullptr || a.tile_rows % 64 != 0 || a.row_group != nullptr)) ||
      (a.row_group != nullptr && a.rows > 65535U))
    return fail(kInvalidArgument, "F32 linear arguments are invalid");
  if (a.rows == 0) return kOk;
  F32Params p{};
  p.weight = static_cast<const bf16 *>(a.weight);
  p.output = a.output;
  p.rows = static_cast<int>(a.rows);
  p.out_features = static_cast<int>(a.out_features);
  p.in_features = static_cast<int>(a.in_features);
  p.accumulate = a.accumulate ? 1 : 0;
  p.alpha = a.alpha;
  p.softcap = a.softcap;
  p.row_scale = a.row_scale;
  p.bias = a.bias;
  p.row_group = a.row_group;
  p.row_fanout = static_cast<int>(a.row_fanout);
  p.tile_group = a.tile_group;
  p.tile_count = a.tile_count;
  p.tile_rows = static_cast<int>(a.tile_rows);
  const auto launch = [&](auto tag) {
    using T = decltype(tag);
    const T *const input = static_cast<const T *>(a.input);
    if (a.row_group != nullptr || (a.rows <= 16 && a.tile_group == nullptr)) {
      const dim3 grid(ceil_div_u(a.out_features, 8), static_cast<unsigned int>(a.rows));
      linear_f32_rows_kernel<T><<<grid, 256, 0, stream>>>(input, p);
      return check_launch("F32 linear kernel (few rows)");
    }
    const dim3 grid(ceil_div_u(a.out_features, 64), ceil_div_u(a.rows, 64));
    linear_f32_kernel<T><<<grid, 256, 0, stream>>>(input, p);
    return check_launch("F32 linear kernel");
  };
  return a.input_type == Activation::kBf16 ? launch(bf16{}) : launch(float{});
}

int linear_f32(const float *input, const void *weight, const std::size_t rows, const std::size_t in_features,
               const std::size_t out_features, float *output, const bool accumulate, cudaStream_t stream) {
  LinearF32Args a;
  a.input = input;
  a.weight = weight;
  a.rows = rows;
  a.in_features = in_features;
  a.out_features = out_features;
  a.output = output;
  a.accumulate = accumulate;
  return linear_f32(a, stream);
}

}  // namespace evob
