// The two recurrences of recurrent_mixers.cu over prompts in chunks of 16 tokens on the tensor cores.
//
// Within a chunk the recurrences are linear in the state S in front of it, so with K, Q, V the chunk's rows
//   gated linear attention:  O = S^T Q~^T + V X,          S' = diag(L) S + K~^T V
//     Q~_t = (a_0 .. a_t) q_t, K~_s = (a_{s+1} .. a_15) k_s, L = a_0 .. a_15 per channel,
//     X_st = sum_d q_td (a_{s+1} .. a_t)_d k_sd for s <= t
//   gated delta rule:        R = beta (V - G S^T K^T),     O = G S^T Q^T + R XM,   S' = G_15 S + K^T (R XW)
//     G_t = g_0 .. g_t, D_ts = g_{s+1} .. g_t, A_ts = beta_t D_ts (k_s.k_t) below the diagonal,
//     N = (I + A)^-1, XW_st = D_15,t N_ts, XM_st = sum_r D_tr (k_r.q_t) N_rs
// (tokens in rows of K, Q, columns of O, R; decay products only, no quotients, so extreme decays stay finite).
// A first kernel prepares Q~, K~ and the 16 x 16 matrices for all chunks at once; the second walks the chunks
// of one head and 16 value columns per CTA.  Its eight warps split the key channels: each keeps S^T for its
// channels as MMA accumulators and uses them in place as the A operand of the next chunk (the contraction
// may run over the channels in any order, so the accumulator layout is a valid operand layout).
//
// F32 operands go through the TF32 pipe as sums of two parts, x = big + small with big rounded to TF32, and
// x y = big big + big small + small big: 22 bits of every operand take part, accumulated in F32.  The F32
// profile does not use this file.
#include "decoder_types.cuh"
#include "ops_internal.hpp"
#include "recurrent_chunks.hpp"

namespace evob {
namespace {

constexpr int kChunk = 16, kColumns = 16, kWarps = 8, kThreads = 32 * kWarps;
constexpr int kMatrixStride = 20;                       // floats between rows of a 16 x 16 matrix
constexpr int kMatrix = kChunk * kMatrixStride;
// per chunk and head: XW | XM | beta | beta G | G (delta), X (linear)
constexpr int kDeltaFloats = 2 * kMatrix + 3 * kChunk, kLinearFloats = kMatrix;

std::size_t up(const std::size_t n, const std::size_t m) { return (n + m - 1) / m * m; }

// ---------------------------------------------------------------- delta: preparation
struct DeltaParams {
  std::size_t stride;
  int rows, heads, kv_heads, dim, value_dim, head_stride, taps, channels;
  int key_column, value_column, beta_column, decay_column;
  int fresh;
};

constexpr int kPrepThreads = 256;
// Floats between rows of keys or queries in shared memory: whole 16-byte words, four banks from row to row.
__host__ __device__ constexpr int pair_stride(const int dim) { return (dim + 31) / 32 * 32 + 4; }

// 16 tokens of one channel of the convolution with SiLU, handed to emit(token, value).
template <int kTaps, typename T, typename Emit>
__device__ __forceinline__ void convolve_chunk(const T *const projection, const DeltaParams &p, const T *const history,
                                               const float *const conv, const int row0, const int column,
                                               const Emit &emit) {
  const int n = p.taps;
  float taps[kTaps], window[kTaps];  // right-aligned: the last entry meets the current token
#pragma unroll
  for (int j = 0; j < kTaps; ++j) {
    const int tap = j - (kTaps - n);
    taps[j] = tap >= 0 ? conv[static_cast<std::size_t>(column) * n + tap] : 0.0F;
  }
  float next[kChunk];
  if (row0 >= kTaps - 1 && row0 + kChunk <= p.rows) {
    const T *const source = projection + static_cast<std::size_t>(row0) * p.stride + column;
    T raw[kTaps - 1 + kChunk];
#pragma unroll
    for (int i = 0; i < kTaps - 1 + kChunk; ++i)
      raw[i] = source[(static_cast<long long>(i) - (kTaps - 1)) * static_cast<long long>(p.stride)];
    window[0] = 0.0F;
#pragma unroll
    for (int j = 1; j < kTaps; ++j) window[j] = to_float(raw[j - 1]);
#pragma unroll
    for (int t = 0; t < kChunk; ++t) next[t] = to_float(raw[kTaps - 1 + t]);
  } else {
    const auto input = [&](const int row) -> float {
      if (row >= p.rows) return 0.0F;
      if (row >= 0) return to_float(projection[static_cast<std::size_t>(row) * p.stride + column]);
      if (p.fresh != 0 || row + n - 1 < 0) return 0.0F;
      return to_float(history[static_cast<std::size_t>(row + n - 1) * p.channels + column]);
    };
#pragma unroll
    for (int j = 0; j < kTaps; ++j) window[j] = j == 0 ? 0.0F : input(row0 - kTaps + j);
#pragma unroll
    for (int t = 0; t < kChunk; ++t) next[t] = input(row0 + t);
  }
#pragma unroll
  for (int t = 0; t < kChunk; ++t) {
#pragma unroll
    for (int j = 0; j + 1 < kTaps; ++j) window[j] = window[j + 1];
    window[kTaps - 1] = next[t];
    float sum = 0.0F;
#pragma unroll
    for (int j = 0; j < kTaps; ++j) sum = fmaf(taps[j], window[j], sum);
    emit(t, row0 + t < p.rows ? silu_f32(sum) : 0.0F);
  }
}

template <int kTaps, typename T>
__global__ void __launch_bounds__(kPrepThreads, 2)
delta_chunks_kernel(const T *__restrict__ projection, const T *__restrict__ history, const float *__restrict__ conv,
                    const float *__restrict__ decay_rate, const float *__restrict__ decay_shift,
                    float *__restrict__ queries, float *__restrict__ keys, T *__restrict__ values,
                    float *__restrict__ matrices, const DeltaParams p) {
  extern __shared__ __align__(16) float smem[];  // per slot of heads two 16 x 16 matrices, then keys and queries [16][pair_stride]
  const int stride = pair_stride(p.dim);
  float *const heads_base = smem;
  float *const ks = heads_base + kPrepThreads / kChunk * 2 * kChunk * kMatrixStride, *const qs = ks + kChunk * stride;
  __shared__ float kk[kChunk][kChunk + 1], kq[kChunk][kChunk + 1];  // [t][s]
  __shared__ float part[4][2][kChunk][kChunk];
  const int chunk = blockIdx.x, g = blockIdx.y, row0 = chunk * kChunk;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int group = p.heads / p.kv_heads;
  const int total = 2 * p.dim + group * p.value_dim;
  for (int i = threadIdx.x; i < 2 * kChunk * (stride - p.dim); i += kPrepThreads)  // padding behind the channels
    ks[i / (stride - p.dim) * stride + p.dim + i % (stride - p.dim)] = 0.0F;
  for (int c = threadIdx.x; c < total; c += kPrepThreads) {
    if (c < 2 * p.dim) {
      const bool is_key = c < p.dim;
      const int d = is_key ? c : c - p.dim;
      float *const target = (is_key ? ks : qs) + d;
      convolve_chunk<kTaps>(projection, p, history, conv, row0, (is_key ? p.key_column : 0) + g * p.dim + d,
                            [&](const int t, const float v) { target[t * stride] = v; });
    } else {
      const int channel = g * group * p.value_dim + c - 2 * p.dim;
      T *const target = values + static_cast<std::size_t>(row0) * p.heads * p.value_dim + channel;
      convolve_chunk<kTaps>(projection, p, history, conv, row0, p.value_column + channel, [&](const int t, const float v) {
        if (row0 + t < p.rows) target[static_cast<std::size_t>(t) * p.heads * p.value_dim] = from_float<T>(v);
      });
    }
  }
  __syncthreads();
  for (int item = warp; item < 2 * kChunk; item += kPrepThreads / 32) {  // unit vectors
    const bool is_key = item < kChunk;
    const int t = item % kChunk;
    float *const row = (is_key ? ks : qs) + t * stride;
    float square = 0.0F;
    for (int d = lane; d < p.dim; d += 32) square = fmaf(row[d], row[d], square);
    square = warp_sum(square);
    float factor = 1.0F / sqrtf(square + 1e-6F);
    if (!is_key) factor *= 1.0F / sqrtf(static_cast<float>(p.dim));
    float *const out = (is_key ? keys : queries) + (static_cast<std::size_t>(row0 + t) * p.kv_heads + g) * p.head_stride;
    for (int d = lane; d < p.head_stride; d += 32) {
      const float v = d < p.dim ? row[d] * factor : 0.0F;
      if (d < p.dim) row[d] = v;
      out[d] = v;
    }
  }
  __syncthreads();
  // inner products: a quarter of the channels of 2 x 2 (t, s) pairs per thread, rows eight apart so that the
  // 16-byte reads of a warp spread over the banks
  {
    const int quarter = threadIdx.x / 64, pair = threadIdx.x % 64, t = pair / 8, s = pair % 8;
    float a[2][2] = {}, b[2][2] = {};
    const int words = stride / 4;
    for (int word = quarter; word < words; word += 4) {
      float k[2][4], kt[2][4], q[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        load_floats<4>(ks + (s + 8 * i) * stride + 4 * word, k[i]);
        load_floats<4>(ks + (t + 8 * i) * stride + 4 * word, kt[i]);
        load_floats<4>(qs + (t + 8 * i) * stride + 4 * word, q[i]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int l = 0; l < 2; ++l)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            a[i][l] = fmaf(kt[i][e], k[l][e], a[i][l]);
            b[i][l] = fmaf(q[i][e], k[l][e], b[i][l]);
          }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int l = 0; l < 2; ++l) {
        part[quarter][0][t + 8 * i][s + 8 * l] = a[i][l];
        part[quarter][1][t + 8 * i][s + 8 * l] = b[i][l];
      }
  }
  __syncthreads();
  {
    const int t = threadIdx.x / kChunk, s = threadIdx.x % kChunk;
    kk[t][s] = (part[0][0][t][s] + part[1][0][t][s]) + (part[2][0][t][s] + part[3][0][t][s]);
    kq[t][s] = (part[0][1][t][s] + part[1][1][t][s]) + (part[2][1][t][s] + part[3][1][t][s]);
  }
  __syncthreads();
  // heads that share the key, two per warp: thread j of sixteen owns column j of the inverse
  const int j = lane % kChunk, slot = threadIdx.x / kChunk;
  constexpr int kSlots = kPrepThreads / kChunk;
  float *const below = heads_base + slot * (2 * kChunk * kMatrixStride);  // A [t][s], rows of whole 16-byte words
  float *const reads = below + kChunk * kMatrixStride;                    // D (k.q) [t][s]
  for (int first = 0; first + 2 * warp < group; first += kSlots) {
    const int local = first + slot, head = g * group + local;
    const bool live = local < group;
    float gate = 1.0F, beta = 0.0F;  // of token j
    if (live && row0 + j < p.rows) {
      const T *const source = projection + static_cast<std::size_t>(row0 + j) * p.stride;
      beta = sigmoid_f32(to_float(source[p.beta_column + head]));
      gate = expf(decay_rate[head] * softplus_f32(to_float(source[p.decay_column + head]) + decay_shift[head]));
    }
    float product = 1.0F, cumulative = 1.0F;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      const float g_t = __shfl_sync(0xffffffffU, gate, t, kChunk), beta_t = __shfl_sync(0xffffffffU, beta, t, kChunk);
      if (t > j) product *= g_t;      // D_tj
      if (t <= j) cumulative *= g_t;  // G_j
      below[t * kMatrixStride + j] = t > j ? beta_t * product * kk[t][j] : 0.0F;
      reads[t * kMatrixStride + j] = t >= j ? product * kq[t][j] : 0.0F;
    }
    const float last_decay = product;  // D_15,j
    __syncwarp();
    const auto row_of = [](const float *const matrix, const int t, float (&v)[kChunk]) {
      load_floats<kChunk>(matrix + t * kMatrixStride, v);
    };
    float column[kChunk];  // N_tj
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      float row[kChunk], x[2] = {t == j ? 1.0F : 0.0F, 0.0F};
      row_of(below, t, row);
#pragma unroll
      for (int s = 0; s < t; ++s) x[s % 2] = fmaf(-row[s], column[s], x[s % 2]);
      column[t] = x[0] + x[1];
    }
    float *const out = matrices + (static_cast<std::size_t>(chunk) * p.heads + head) * kDeltaFloats;
    float updates[kChunk], readouts[kChunk];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      updates[t] = __shfl_sync(0xffffffffU, last_decay, t, kChunk) * column[t];  // D_15,t N_tj
      float row[kChunk], x[2] = {0.0F, 0.0F};
      row_of(reads, t, row);
#pragma unroll
      for (int r = 0; r <= t; ++r) x[r % 2] = fmaf(row[r], column[r], x[r % 2]);
      readouts[t] = x[0] + x[1];
    }
    if (live) {
#pragma unroll
      for (int t = 0; t < kChunk; t += 4) {
        *reinterpret_cast<float4 *>(out + j * kMatrixStride + t) = make_float4(updates[t], updates[t + 1], updates[t + 2], updates[t + 3]);
        *reinterpret_cast<float4 *>(out + kMatrix + j * kMatrixStride + t) =
            make_float4(readouts[t], readouts[t + 1], readouts[t + 2], readouts[t + 3]);
      }
      *reinterpret_cast<float4 *>(out + j * kMatrixStride + kChunk) = make_float4(0.0F, 0.0F, 0.0F, 0.0F);
      *reinterpret_cast<float4 *>(out + kMatrix + j * kMatrixStride + kChunk) = make_float4(0.0F, 0.0F, 0.0F, 0.0F);
      out[2 * kMatrix + j] = beta;
      out[2 * kMatrix + kChunk + j] = beta * cumulative;
      out[2 * kMatrix + 2 * kChunk + j] = cumulative;
    }
    __syncwarp();
  }
}

// ---------------------------------------------------------------- linear: preparation
// Sums sixteen values over the warp; lane l is left with the sum of value l / 2.
__device__ __forceinline__ float reduce_scatter16(const float (&v)[16], const int lane) {
  float a[8], b[4], c[2];
  const bool b4 = (lane & 16) != 0, b3 = (lane & 8) != 0, b2 = (lane & 4) != 0, b1 = (lane & 2) != 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) a[i] = (b4 ? v[i + 8] : v[i]) + __shfl_xor_sync(0xffffffffU, b4 ? v[i] : v[i + 8], 16);
#pragma unroll
  for (int i = 0; i < 4; ++i) b[i] = (b3 ? a[i + 4] : a[i]) + __shfl_xor_sync(0xffffffffU, b3 ? a[i] : a[i + 4], 8);
#pragma unroll
  for (int i = 0; i < 2; ++i) c[i] = (b2 ? b[i + 2] : b[i]) + __shfl_xor_sync(0xffffffffU, b2 ? b[i] : b[i + 2], 4);
  const float d = (b1 ? c[1] : c[0]) + __shfl_xor_sync(0xffffffffU, b1 ? c[0] : c[1], 2);
  return d + __shfl_xor_sync(0xffffffffU, d, 1);
}

// A thread per key channel (blockDim = dim rounded up to warps).
template <typename T>
__global__ void __launch_bounds__(256)
linear_chunks_kernel(const T *__restrict__ projection, const std::size_t stride, const int key_column,
                     const int bottleneck_column, const float *__restrict__ weight, const float *__restrict__ bias,
                     const int rank, const float inverse_tau, const int rows, const int heads, const int dim,
                     const int head_stride, float *__restrict__ queries, float *__restrict__ keys,
                     float *__restrict__ last, float *__restrict__ matrices) {
  extern __shared__ float bottleneck[];  // [16][rank]
  __shared__ float parts[8][kChunk][kChunk];
  const int chunk = blockIdx.x, head = blockIdx.y, row0 = chunk * kChunk, d = threadIdx.x;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, warps = blockDim.x / 32;
  for (int i = threadIdx.x; i < kChunk * rank; i += blockDim.x) {
    const int t = i / rank, k = i % rank;
    bottleneck[i] = row0 + t < rows ? to_float(projection[static_cast<std::size_t>(row0 + t) * stride + bottleneck_column + k]) : 0.0F;
  }
  __syncthreads();
  const int channel = head * dim + d, channels = heads * dim;
  const bool inside = d < dim;
  float a[kChunk], q[kChunk], k[kChunk];
  if (inside && row0 + kChunk <= rows) {
    const T *const source = projection + static_cast<std::size_t>(row0) * stride + channel;
    T raw_q[kChunk], raw_k[kChunk];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      raw_q[t] = source[t * stride];
      raw_k[t] = source[t * stride + key_column];
    }
    const float offset = bias[channel];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      a[t] = offset;
      q[t] = to_float(raw_q[t]);
      k[t] = to_float(raw_k[t]);
    }
  } else
#pragma unroll
  for (int t = 0; t < kChunk; ++t) {
    a[t] = inside ? bias[channel] : 0.0F;
    const bool live = inside && row0 + t < rows;
    const T *const source = projection + static_cast<std::size_t>(row0 + t) * stride + channel;
    q[t] = live ? to_float(source[0]) : 0.0F;
    k[t] = live ? to_float(source[key_column]) : 0.0F;
  }
  if (inside)
    for (int r = 0; r < rank; ++r) {
      const float w = weight[static_cast<std::size_t>(r) * channels + channel];
#pragma unroll
      for (int t = 0; t < kChunk; ++t) a[t] = fmaf(w, bottleneck[t * rank + r], a[t]);
    }
  const float scale = 1.0F / sqrtf(static_cast<float>(dim));
#pragma unroll
  for (int t = 0; t < kChunk; ++t) {
    // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
    a[t] = inside && row0 + t < rows ? expf(-softplus_f32(-a[t]) * inverse_tau) : 1.0F;
    q[t] *= scale;
  }
  float carried[kChunk];  // k_s times the decays up to the current token
#pragma unroll
  for (int t = 0; t < kChunk; ++t) {
    float products[kChunk];
#pragma unroll
    for (int s = 0; s < kChunk; ++s) {
      if (s < t) carried[s] *= a[t];
      if (s == t) carried[s] = k[s];
      products[s] = s <= t ? q[t] * carried[s] : 0.0F;
    }
    const float sum = reduce_scatter16(products, lane);
    if ((lane & 1) == 0) parts[warp][t][lane / 2] = sum;
  }
  if (d < head_stride) {
    float forward = 1.0F;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      forward *= a[t];
      const std::size_t at = (static_cast<std::size_t>(row0 + t) * heads + head) * head_stride + d;
      queries[at] = forward * q[t];
      keys[at] = carried[t];  // decayed to the end of the chunk
    }
    last[(static_cast<std::size_t>(chunk) * heads + head) * head_stride + d] = forward;
  }
  __syncthreads();
  float *const out = matrices + (static_cast<std::size_t>(chunk) * heads + head) * kLinearFloats;
  for (int i = threadIdx.x; i < kMatrix; i += blockDim.x) {
    const int s = i / kMatrixStride, t = i % kMatrixStride;
    float sum = 0.0F;
    if (t < kChunk)
      for (int w = 0; w < warps; ++w) sum += parts[w][t][s];
    out[i] = sum;
  }
}

// ---------------------------------------------------------------- the walk over the chunks
struct Split {
  std::uint32_t big, small;
};
// big: x rounded to TF32 (10 mantissa bits, halves away from zero), small: the exact rest
__device__ __forceinline__ Split split(const float x) {
  Split s;
  s.big = (__float_as_uint(x) + 0x1000U) & 0xffffe000U;
  s.small = __float_as_uint(x - __uint_as_float(s.big));
  return s;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const std::uint32_t (&a)[4], const std::uint32_t b0,
                                         const std::uint32_t b1) {
  asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// An accumulator tile (rows g, g + 8; columns 2t, 2t + 1) as an A operand whose contraction index t is column
// 2t and t + 4 column 2t + 1.
struct Operand {
  std::uint32_t big[4], small[4];
};
__device__ __forceinline__ Operand operand_of(const float (&c)[4]) {
  Operand a;
  const float order[4] = {c[0], c[2], c[1], c[3]};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const Split s = split(order[i]);
    a.big[i] = s.big;
    a.small[i] = s.small;
  }
  return a;
}
// Main and correction sums in separate accumulators: shorter chains of dependent MMAs.
struct Sum {
  float main[4] = {}, first[4] = {}, second[4] = {};
  __device__ __forceinline__ float get(const int i) const { return main[i] + (first[i] + second[i]); }
};
__device__ __forceinline__ void mma_f32(Sum &d, const Operand &a, const float b0, const float b1) {
  const Split x = split(b0), y = split(b1);
  mma_tf32(d.first, a.small, x.big, y.big);
  mma_tf32(d.second, a.big, x.small, y.small);
  mma_tf32(d.main, a.big, x.big, y.big);
}

struct WalkParams {
  int rows, heads, kv_heads, dim, value_dim, head_stride;
  std::size_t value_stride;
  int fresh;
};

__device__ __forceinline__ void copy16(float *const dst, const float *const src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<std::uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src)
               : "memory");
}

template <bool kDelta, int kTiles>
struct WalkLayout {
  static constexpr int kWidth = kTiles * 8 * kWarps;  // key channels, eight per tile and warp
  static constexpr int kRow = kWidth + 8;         // floats: the 64-bit operand reads hit every bank once
  static constexpr int kValueStride = 20;
  static constexpr int kKeys = 0, kQueries = kChunk * kRow, kLast = 2 * kChunk * kRow;
  static constexpr int kMatrices = kLast + (kDelta ? 0 : kWidth);
  static constexpr int kValues = kMatrices + (kDelta ? kDeltaFloats : kLinearFloats);
  static constexpr int kBuffer = kValues + kChunk * kValueStride;
  static constexpr int kParts = 2 * kBuffer;      // [warp][product][lane] float4
  static constexpr int kRight = kParts + kWarps * (kDelta ? 4 : 2) * 32 * 4;  // delta: R, two halves of 32 float4
  static constexpr int kFloats = kRight + (kDelta ? 2 * 32 * 4 : 0);
};

template <bool kDelta, int kTiles, typename T>
__global__ void __launch_bounds__(kThreads)
chunk_walk_kernel(const float *__restrict__ queries, const float *__restrict__ keys, const float *__restrict__ last,
                  const float *__restrict__ matrices, const T *__restrict__ values, float *__restrict__ state,
                  float *__restrict__ output, const WalkParams p) {
  using L = WalkLayout<kDelta, kTiles>;
  constexpr int kProducts = kDelta ? 4 : 2;
  extern __shared__ __align__(16) float smem[];
  const int head = blockIdx.y, column0 = blockIdx.x * kColumns;
  const int key_head = kDelta ? head / (p.heads / p.kv_heads) : head;
  const int key_heads = kDelta ? p.kv_heads : p.heads;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, g = lane / 4, t = lane % 4;
  const int chunks = (p.rows + kChunk - 1) / kChunk;
  const int channel0 = warp * kTiles * 8;

  for (int i = threadIdx.x; i < L::kFloats; i += kThreads) smem[i] = 0.0F;  // channels past dim stay zero
  __syncthreads();
  const auto fetch = [&](const int chunk) {
    float *const b = smem + (chunk & 1) * L::kBuffer;
    const int words = p.head_stride / 4;
    constexpr int kWords = L::kWidth / 4;
#pragma unroll
    for (int i = 0; i < kChunk * kWords / kThreads; ++i) {
      const int row = (i * kThreads + threadIdx.x) / kWords, word = (i * kThreads + threadIdx.x) % kWords;
      if (word >= words) continue;
      const std::size_t source = (static_cast<std::size_t>(chunk * kChunk + row) * key_heads + key_head) * p.head_stride + word * 4;
      copy16(b + L::kKeys + row * L::kRow + word * 4, keys + source);
      copy16(b + L::kQueries + row * L::kRow + word * 4, queries + source);
    }
    if constexpr (!kDelta)
      for (int i = threadIdx.x; i < words; i += kThreads)
        copy16(b + L::kLast + 4 * i, last + (static_cast<std::size_t>(chunk) * p.heads + head) * p.head_stride + 4 * i);
    constexpr int kFloats = kDelta ? kDeltaFloats : kLinearFloats;
    for (int i = threadIdx.x; i < kFloats / 4; i += kThreads)
      copy16(b + L::kMatrices + 4 * i, matrices + (static_cast<std::size_t>(chunk) * p.heads + head) * kFloats + 4 * i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  T staged;  // widened only when they are stored: the loads stay in flight until then
  static_assert(kThreads == kChunk * kColumns, "one value of the chunk per thread");
  const auto load_values = [&](const int chunk) {
    const int row = chunk * kChunk + threadIdx.x / kColumns, c = column0 + threadIdx.x % kColumns;
    staged = row < p.rows && c < p.value_dim ? values[static_cast<std::size_t>(row) * p.value_stride + head * p.value_dim + c]
                                             : from_float<T>(0.0F);
  };

  float S[kTiles][4];  // S^T: rows = value columns g, g + 8; columns = channels channel0 + 8 tile + 2t, + 1
#pragma unroll
  for (int n = 0; n < kTiles; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = channel0 + 8 * n + 2 * t + (i & 1), column = column0 + g + (i & 2) * 4;
      S[n][i] = p.fresh == 0 && d < p.dim && column < p.value_dim
                    ? state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column]
                    : 0.0F;
    }
  fetch(0);
  load_values(0);
  float4 *const parts = reinterpret_cast<float4 *>(smem + L::kParts);
  for (int chunk = 0; chunk < chunks; ++chunk) {
    float *const b = smem + (chunk & 1) * L::kBuffer;
    b[L::kValues + threadIdx.x / kColumns * L::kValueStride + threadIdx.x % kColumns] = to_float(staged);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the chunk is here, and everybody is done with the one before
    // this warp's channels of S^T K^T and S^T Q^T, two halves of eight tokens each
    Sum products[kProducts];
#pragma unroll
    for (int n = 0; n < kTiles; ++n) {
      const Operand a = operand_of(S[n]);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int at = (8 * half + g) * L::kRow + channel0 + 8 * n + 2 * t;
        const float2 q = *reinterpret_cast<const float2 *>(b + L::kQueries + at);
        mma_f32(products[half], a, q.x, q.y);
        if constexpr (kDelta) {
          const float2 k = *reinterpret_cast<const float2 *>(b + L::kKeys + at);
          mma_f32(products[2 + half], a, k.x, k.y);
        }
      }
    }
    const float *const m = b + L::kMatrices;
#pragma unroll
    for (int i = 0; i < kProducts; ++i)
      parts[(warp * kProducts + i) * 32 + lane] = make_float4(products[i].get(0), products[i].get(1), products[i].get(2), products[i].get(3));
    if (chunk + 1 < chunks) {
      fetch(chunk + 1);
      load_values(chunk + 1);
    }
    const auto gathered = [&](const int product, float (&sum)[4]) {
      float4 total = parts[product * 32 + lane];
#pragma unroll
      for (int w = 1; w < kWarps; ++w) {
        const float4 v = parts[(w * kProducts + product) * 32 + lane];
        total.x += v.x, total.y += v.y, total.z += v.z, total.w += v.w;
      }
      sum[0] = total.x, sum[1] = total.y, sum[2] = total.z, sum[3] = total.w;
    };
    const float *const beta = m + 2 * kMatrix, *const beta_g = beta + kChunk, *const cumulative = beta_g + kChunk;
    Operand right[2], update[2];  // the right-hand side, and what is added to the state, by token half
    // in the accumulator layout, [column][token]: the values, for the delta rule corrected
    float R[2][4];
    if constexpr (kDelta) {
      __syncthreads();
      // one element per thread: (token half, lane, accumulator register)
      const int half = threadIdx.x / 128, at = threadIdx.x % 128, i = at % 4;
      const int token = 8 * half + 2 * (at / 4 % 4) + (i & 1), column = at / 16 + (i & 2) * 4;
      const float *const held = smem + L::kParts + (2 + half) * 128 + at;
      float sum[2] = {0.0F, 0.0F};
#pragma unroll
      for (int w = 0; w < kWarps; ++w) sum[w % 2] += held[w * kProducts * 128];
      smem[L::kRight + threadIdx.x] =
          fmaf(-beta_g[token], sum[0] + sum[1], beta[token] * b[L::kValues + token * L::kValueStride + column]);
      __syncthreads();
#pragma unroll
      for (int half = 0; half < 2; ++half) load_floats<4>(smem + L::kRight + half * 128 + lane * 4, R[half]);
    } else {
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          R[half][i] = b[L::kValues + (8 * half + 2 * t + (i & 1)) * L::kValueStride + g + (i & 2) * 4];
    }
    right[0] = operand_of(R[0]);
    right[1] = operand_of(R[1]);
    if constexpr (kDelta) {
#pragma unroll
      for (int out = 0; out < 2; ++out) {
        Sum u;
#pragma unroll
        for (int half = 0; half <= out; ++half) {  // later tokens do not reach earlier ones
          const float *const x = m + (8 * half + 2 * t) * kMatrixStride + 8 * out + g;
          mma_f32(u, right[half], x[0], x[kMatrixStride]);
        }
        const float sums[4] = {u.get(0), u.get(1), u.get(2), u.get(3)};
        update[out] = operand_of(sums);
      }
    } else {
      update[0] = right[0];
      update[1] = right[1];
    }
#pragma unroll
    for (int n = 0; n < kTiles; ++n) {
      if constexpr (kDelta) {
        const float decay = cumulative[kChunk - 1];
#pragma unroll
        for (int i = 0; i < 4; ++i) S[n][i] *= decay;
      } else {
        const float2 decay = *reinterpret_cast<const float2 *>(b + L::kLast + channel0 + 8 * n + 2 * t);
        S[n][0] *= decay.x, S[n][1] *= decay.y, S[n][2] *= decay.x, S[n][3] *= decay.y;
      }
      Sum added;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const float *const k = b + L::kKeys + (8 * half + 2 * t) * L::kRow + channel0 + 8 * n + g;
        mma_f32(added, update[half], k[0], k[L::kRow]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) S[n][i] += added.get(i);
    }
    if constexpr (!kDelta) __syncthreads();
    if (warp < 2) {  // outputs of token half `warp`
      float o[4];
      gathered(warp, o);
      const float *const x = m + (kDelta ? kMatrix : 0) + 2 * t * kMatrixStride + 8 * warp + g;
      Sum inside;
      mma_f32(inside, right[0], x[0], x[kMatrixStride]);
      if (warp == 1) mma_f32(inside, right[1], x[8 * kMatrixStride], x[9 * kMatrixStride]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int token = 8 * warp + 2 * t + (i & 1), row = chunk * kChunk + token, column = column0 + g + (i & 2) * 4;
        if (row < p.rows && column < p.value_dim)
          output[(static_cast<std::size_t>(row) * p.heads + head) * p.value_dim + column] =
              kDelta ? fmaf(o[i], cumulative[token], inside.get(i)) : o[i] + inside.get(i);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < kTiles; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = channel0 + 8 * n + 2 * t + (i & 1), column = column0 + g + (i & 2) * 4;
      if (d < p.dim && column < p.value_dim) state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column] = S[n][i];
    }
}

template <bool kDelta, int kTiles>
int launch_walk(const float *queries, const float *keys, const float *last, const float *matrices, const bf16 *values,
                float *state, float *output, const WalkParams &p, cudaStream_t stream) {
  constexpr std::size_t bytes = WalkLayout<kDelta, kTiles>::kFloats * sizeof(float);
  if (cudaFuncSetAttribute(chunk_walk_kernel<kDelta, kTiles, bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           static_cast<int>(bytes)) != cudaSuccess)
    return fail(kCuda, "cannot raise the recurrence shared-memory limit");
  const dim3 grid(ceil_div_u(p.value_dim, kColumns), static_cast<unsigned int>(p.heads));
  chunk_walk_kernel<kDelta, kTiles, bf16><<<grid, kThreads, bytes, stream>>>(queries, keys, last, matrices, values, state,
                                                                            output, p);
  return check_launch(kDelta ? "gated delta rule chunk kernel" : "gated linear attention chunk kernel");
}

template <bool kDelta>
int dispatch_walk(const float *queries, const float *keys, const float *last, const float *matrices, const bf16 *values,
                  float *state, float *output, const WalkParams &p, cudaStream_t stream) {
  if (p.dim <= 64) return launch_walk<kDelta, 1>(queries, keys, last, matrices, values, state, output, p, stream);
  if (p.dim <= 128) return launch_walk<kDelta, 2>(queries, keys, last, matrices, values, state, output, p, stream);
  return launch_walk<kDelta, 4>(queries, keys, last, matrices, values, state, output, p, stream);
}

struct Layout {
  std::size_t rows, head_stride, query, key, last, value, matrices, output, bytes;
};
Layout layout_of(const bool delta, const std::size_t rows, const std::size_t heads, const std::size_t kv_heads,
                 const std::size_t dim, const std::size_t value_dim) {
  Layout l{};
  l.rows = up(rows, kChunk);
  l.head_stride = up(dim, 4);
  const std::size_t key_heads = delta ? kv_heads : heads, chunks = l.rows / kChunk;
  std::size_t cursor = 0;
  const auto take = [&cursor](const std::size_t bytes) {
    const std::size_t at = cursor;
    cursor += up(bytes, 256);
    return at;
  };
  l.query = take(l.rows * key_heads * l.head_stride * 4);
  l.key = take(l.rows * key_heads * l.head_stride * 4);
  l.last = take(delta ? 0 : chunks * heads * l.head_stride * 4);
  l.value = take(delta ? rows * heads * value_dim * 2 : 0);
  l.matrices = take(chunks * heads * (delta ? kDeltaFloats : kLinearFloats) * 4);
  l.output = take(rows * heads * value_dim * 4);
  l.bytes = cursor;
  return l;
}

}  // namespace

bool recurrent_chunks_applicable(const RecurrentArgs &a) {
  return a.type == Activation::kBf16 && a.rows >= 2 * kChunk && (!a.delta || a.conv_taps <= 8);
}

std::size_t recurrent_chunks_workspace(const bool delta, const std::size_t rows, const std::size_t heads,
                                       const std::size_t kv_heads, const std::size_t dim, const std::size_t value_dim) {
  return layout_of(delta, rows, heads, kv_heads, dim, value_dim).bytes;
}

int recurrent_chunks(const RecurrentArgs &a, float **output, cudaStream_t stream) {
  const Layout l = layout_of(a.delta, a.rows, a.heads, a.kv_heads, a.dim, a.value_dim);
  unsigned char *const base = static_cast<unsigned char *>(a.workspace);
  const auto floats = [base](const std::size_t at) { return reinterpret_cast<float *>(base + at); };
  const bf16 *const projection = static_cast<const bf16 *>(a.projection);
  *output = floats(l.output);
  WalkParams w{};
  w.rows = static_cast<int>(a.rows);
  w.heads = static_cast<int>(a.heads);
  w.kv_heads = static_cast<int>(a.kv_heads);
  w.dim = static_cast<int>(a.dim);
  w.value_dim = static_cast<int>(a.value_dim);
  w.head_stride = static_cast<int>(l.head_stride);
  w.fresh = a.fresh ? 1 : 0;
  const unsigned int chunks = static_cast<unsigned int>(l.rows / kChunk);
  int status;
  if (a.delta) {
    DeltaParams p{};
    p.stride = a.stride;
    p.rows = w.rows;
    p.heads = w.heads;
    p.kv_heads = w.kv_heads;
    p.dim = w.dim;
    p.value_dim = w.value_dim;
    p.head_stride = w.head_stride;
    p.taps = static_cast<int>(a.conv_taps);
    p.channels = static_cast<int>(a.gate_column);
    p.key_column = static_cast<int>(a.key_column);
    p.value_column = static_cast<int>(a.value_column);
    p.beta_column = static_cast<int>(a.beta_column);
    p.decay_column = static_cast<int>(a.decay_column);
    p.fresh = w.fresh;
    const std::size_t bytes = (2 * kChunk * pair_stride(static_cast<int>(a.dim)) + kPrepThreads / kChunk * 2 * kChunk * kMatrixStride) * sizeof(float);
    bf16 *const values = reinterpret_cast<bf16 *>(base + l.value);
    const auto kernel = a.conv_taps <= 4 ? delta_chunks_kernel<4, bf16> : delta_chunks_kernel<8, bf16>;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) != cudaSuccess)
      return fail(kCuda, "cannot raise the delta preparation shared-memory limit");
    kernel<<<dim3(chunks, static_cast<unsigned int>(a.kv_heads)), kPrepThreads, bytes, stream>>>(
        projection, static_cast<const bf16 *>(a.conv_history), a.conv, a.decay_rate, a.decay_shift, floats(l.query),
        floats(l.key), values, floats(l.matrices), p);
    if ((status = check_launch("delta chunk preparation kernel")) != kOk) return status;
    w.value_stride = a.heads * a.value_dim;
    return dispatch_walk<true>(floats(l.query), floats(l.key), nullptr, floats(l.matrices), values, a.state, *output, w,
                               stream);
  }
  const unsigned int threads = static_cast<unsigned int>(up(a.dim, 32));
  linear_chunks_kernel<bf16><<<dim3(chunks, static_cast<unsigned int>(a.heads)), threads,
                               kChunk * a.decay_rank * sizeof(float), stream>>>(
      projection, a.stride, static_cast<int>(a.key_column), static_cast<int>(a.beta_column), a.decay_weight, a.decay_bias,
      static_cast<int>(a.decay_rank), 1.0F / a.tau, w.rows, w.heads, w.dim, w.head_stride, floats(l.query), floats(l.key),
      floats(l.last), floats(l.matrices));
  if ((status = check_launch("linear attention chunk preparation kernel")) != kOk) return status;
  w.value_stride = a.stride;
  return dispatch_walk<false>(floats(l.query), floats(l.key), floats(l.last), floats(l.matrices),
                              projection + a.value_column, a.state, *output, w, stream);
}

}  // namespace evob
