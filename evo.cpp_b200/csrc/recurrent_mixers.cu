// Mixers with a matrix state per head: gated linear attention (a decay per key channel) and the gated
// delta rule (a scalar decay per head, values corrected by what the state already holds for the key).
// Everything that enters the recurrences is F32.
//
// One token (cached decode) is one launch: decode_kernel.  BF16 prompt portions of 32 rows and more take the
// tensor-core form (recurrent_chunks.cu); shorter ones, and the F32 profile, run in three launches:
//   1. preparation: per token the decays and the queries / keys the recurrence reads (F32), for the delta
//      rule also the short convolutions, the unit vectors, the step sizes, and the scalars of the blocked
//      form below;
//   2. the recurrence: columns of the state (one per value channel) never mix, so a CTA owns 16 of them and
//      a warp four; the warp's lanes divide the key channels between them (2, 4 or 8 each, so that one
//      shared-memory read of a key serves four columns) and the state stays in registers as packed pairs.
//      Tokens stream through a double-buffered shared-memory tile; sums over the channels are shuffle
//      exchanges that leave every lane with one column and one token;
//   3. the output norm and gate, row-wise.
//
// Blocked delta rule.  Four tokens at a time, with S the state in front of the block, G_t = g_0 .. g_t and
// D_ts = g_{s+1} .. g_t the decay products inside it:
//   u_t = beta_t (v_t - G_t S^T k_t - sum_{s<t} D_ts (k_s.k_t) u_s)
//   o_t = G_t S^T q_t + sum_{s<=t} D_ts (k_s.q_t) u_s
//   S'  = G_3 S + sum_s D_3s k_s u_s^T
// so the eight products with S are taken at once and summed over the lanes together; the scalars
// depend on the head only and come from the preparation.
#include <cooperative_groups.h>

#include "decoder_types.cuh"
#include "ops_internal.hpp"
#include "recurrent_chunks.hpp"

namespace evob {
namespace {
namespace cg = cooperative_groups;

constexpr int kBlock = 4;              // tokens per block of the delta rule
constexpr int kTile = 16;              // tokens per shared-memory tile
constexpr int kColumns = 16;           // state columns per CTA
constexpr int kRecurrenceThreads = 128;
constexpr int kScalars = 40;           // of a block and head, see enum below
// b_t = beta_t | b_t G_t | b_t D_ts (k_s.k_t) (1,0)(2,0)(2,1)(3,0)(3,1)(3,2) pad pad | G_t | D_3s | D_ts (k_s.q_t) [4][4]
enum Scalar : int { kBeta = 0, kBetaG = 4, kPair = 8, kG = 16, kTail = 20, kRead = 24 };

__host__ __device__ constexpr std::size_t round_up(const std::size_t n, const std::size_t m) { return (n + m - 1) / m * m; }

struct Workspace {
  std::size_t rows, head_stride;  // padded token count, floats per head row of queries and keys
  std::size_t query, key, alpha, value, scalars, output, bytes;
};

Workspace workspace_layout(const bool delta, const std::size_t rows, const std::size_t heads,
                           const std::size_t kv_heads, const std::size_t dim, const std::size_t value_dim,
                           const Activation type) {
  Workspace w{};
  w.rows = round_up(rows, kTile);
  w.head_stride = round_up(dim, 4);
  const std::size_t key_heads = delta ? kv_heads : heads;
  std::size_t cursor = 0;
  const auto take = [&cursor](const std::size_t bytes) {
    const std::size_t at = cursor;
    cursor += round_up(bytes, 256);
    return at;
  };
  w.query = take(w.rows * key_heads * w.head_stride * 4);
  w.key = take(w.rows * key_heads * w.head_stride * 4);
  w.alpha = take(delta ? 0 : w.rows * key_heads * w.head_stride * 4);
  w.value = take(delta ? rows * heads * value_dim * activation_bytes(type) : 0);
  w.scalars = take(delta ? w.rows / kBlock * heads * kScalars * 4 : 0);
  w.output = take(rows * heads * value_dim * 4);
  w.bytes = cursor;
  return w;
}

// ---------------------------------------------------------------- delta: preparation
struct DeltaPrepParams {
  std::size_t stride;
  int rows, padded_rows, heads, kv_heads, dim, value_dim, head_stride, taps, channels;
  int key_column, value_column, beta_column, decay_column;
  int fresh;
};

// Channel `column` of the convolution at row r: rows in front of the portion come from the history.
template <typename T>
__device__ __forceinline__ float conv_silu(const T *const projection, const std::size_t stride, const T *const history,
                                           const int channels, const float *const taps, const int n, const bool fresh,
                                           const int r, const int column) {
  float sum = 0.0F;
  for (int j = 0; j < n; ++j) {
    const int source = r - (n - 1) + j;
    float x = 0.0F;
    if (source >= 0) x = to_float(projection[static_cast<std::size_t>(source) * stride + column]);
    else if (!fresh) x = to_float(history[static_cast<std::size_t>(source + n - 1) * channels + column]);
    sum = fmaf(taps[static_cast<std::size_t>(column) * n + j], x, sum);
  }
  return silu_f32(sum);
}

template <typename T>
__global__ void __launch_bounds__(128)
delta_prepare_kernel(const T *__restrict__ projection, const T *__restrict__ history, const float *__restrict__ conv,
                     const float *__restrict__ decay_rate, const float *__restrict__ decay_shift,
                     float *__restrict__ queries, float *__restrict__ keys, T *__restrict__ values,
                     float *__restrict__ scalars, const DeltaPrepParams p) {
  extern __shared__ float prep_smem[];  // [2][kBlock][dim]: keys, queries
  __shared__ float pair_kk[kBlock][kBlock], pair_kq[kBlock][kBlock];
  float *const ks = prep_smem, *const qs = prep_smem + kBlock * p.dim;
  const int block = blockIdx.x, g = blockIdx.y;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int group = p.heads / p.kv_heads;
  const int r = block * kBlock + warp;  // this warp's token
  for (int which = 0; which < 2; ++which) {
    float *const shared = (which == 0 ? ks : qs) + warp * p.dim;
    const int column0 = (which == 0 ? p.key_column : 0) + g * p.dim;
    float v[kDecoderMaxHeadDim / 32];
    float square = 0.0F;
#pragma unroll
    for (int i = 0; i < static_cast<int>(kDecoderMaxHeadDim) / 32; ++i) {
      const int d = lane + 32 * i;
      v[i] = d < p.dim && r < p.rows ? conv_silu(projection, p.stride, history, p.channels, conv, p.taps, p.fresh != 0, r,
                                                 column0 + d)
                                     : 0.0F;
      square = fmaf(v[i], v[i], square);
    }
    square = warp_sum(square);
    float factor = 1.0F / sqrtf(square + 1e-6F);
    if (which == 1) factor *= 1.0F / sqrtf(static_cast<float>(p.dim));
    float *const out = (which == 0 ? keys : queries) +
                       (static_cast<std::size_t>(r) * p.kv_heads + g) * p.head_stride;
#pragma unroll
    for (int i = 0; i < static_cast<int>(kDecoderMaxHeadDim) / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < p.dim) shared[d] = v[i] * factor;
      if (d < p.head_stride) out[d] = d < p.dim ? v[i] * factor : 0.0F;
    }
  }
  // values of the heads that share this key
  for (int c = threadIdx.x; c < group * p.value_dim; c += 128) {
    const int channel = g * group * p.value_dim + c;
    for (int t = 0; t < kBlock; ++t) {
      const int row = block * kBlock + t;
      if (row < p.rows)
        values[static_cast<std::size_t>(row) * p.heads * p.value_dim + channel] = from_float<T>(
            conv_silu(projection, p.stride, history, p.channels, conv, p.taps, p.fresh != 0, row, p.value_column + channel));
    }
  }
  __syncthreads();
  // the block's inner products: warp t takes token t against tokens 0 .. t
  for (int s = 0; s <= warp; ++s) {
    float kk = 0.0F, kq = 0.0F;
    for (int d = lane; d < p.dim; d += 32) {
      kk = fmaf(ks[s * p.dim + d], ks[warp * p.dim + d], kk);
      kq = fmaf(ks[s * p.dim + d], qs[warp * p.dim + d], kq);
    }
    kk = warp_sum(kk);
    kq = warp_sum(kq);
    if (lane == 0) {
      pair_kk[warp][s] = kk;
      pair_kq[warp][s] = kq;
    }
  }
  __syncthreads();
  for (int local = threadIdx.x; local < group; local += 128) {
    const int head = g * group + local;
    float beta[kBlock], gate[kBlock];
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      const int row = block * kBlock + t;
      beta[t] = 0.0F;
      gate[t] = 1.0F;
      if (row < p.rows) {
        const T *const source = projection + static_cast<std::size_t>(row) * p.stride;
        beta[t] = sigmoid_f32(to_float(source[p.beta_column + head]));
        gate[t] = expf(decay_rate[head] * softplus_f32(to_float(source[p.decay_column + head]) + decay_shift[head]));
      }
    }
    float *const out = scalars + (static_cast<std::size_t>(block) * p.heads + head) * kScalars;
    float cumulative = 1.0F;
    float decay[kBlock][kBlock];  // D_ts
    int pair = 0;
#pragma unroll
    for (int t = 0; t < kBlock; ++t) {
      cumulative *= gate[t];
      out[kBeta + t] = beta[t];
      out[kBetaG + t] = beta[t] * cumulative;
      out[kG + t] = cumulative;
      decay[t][t] = 1.0F;
#pragma unroll
      for (int s = t - 1; s >= 0; --s) decay[t][s] = decay[t - 1][s] * gate[t];
#pragma unroll
      for (int s = 0; s < kBlock; ++s) {
        out[kRead + 4 * t + s] = s <= t ? decay[t][s] * pair_kq[t][s] : 0.0F;
        if (s < t) out[kPair + pair++] = beta[t] * decay[t][s] * pair_kk[t][s];
      }
    }
    out[kPair + 6] = out[kPair + 7] = 0.0F;
#pragma unroll
    for (int s = 0; s < kBlock; ++s) out[kTail + s] = decay[kBlock - 1][s];
  }
}

// The last taps - 1 rows of [history | portion] become the history of the next portion.
template <typename T>
__global__ void __launch_bounds__(256)
conv_history_kernel(const T *__restrict__ projection, const std::size_t stride, T *const history, const int channels,
                    const int kept, const int rows, const bool fresh) {
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= channels) return;
  for (int i = 0; i < kept; ++i) {  // ascending: entry i reads entry i + rows, which is not written yet
    const int source = rows - kept + i;
    T value = from_float<T>(0.0F);
    if (source >= 0) value = projection[static_cast<std::size_t>(source) * stride + c];
    else if (!fresh) value = history[static_cast<std::size_t>(source + kept) * channels + c];
    history[static_cast<std::size_t>(i) * channels + c] = value;
  }
}

// ---------------------------------------------------------------- linear: preparation
constexpr int kPrepTokens = 16;
constexpr std::size_t kMaxDecayRank = 512;  // bottleneck rows of a preparation step in shared memory

template <typename T>
__global__ void __launch_bounds__(128)
linear_prepare_kernel(const T *__restrict__ projection, const std::size_t stride, const int key_column,
                      const int bottleneck_column, const float *__restrict__ weight, const float *__restrict__ bias,
                      const int rank, const float inverse_tau, const int rows, const int heads, const int dim,
                      const int head_stride, float *__restrict__ queries, float *__restrict__ keys,
                      float *__restrict__ alpha) {
  extern __shared__ float bottleneck[];  // [kPrepTokens][rank]
  const int row0 = blockIdx.x * kPrepTokens;
  for (int i = threadIdx.x; i < kPrepTokens * rank; i += 128) {
    const int t = i / rank, k = i % rank;
    bottleneck[i] =
        row0 + t < rows ? to_float(projection[static_cast<std::size_t>(row0 + t) * stride + bottleneck_column + k]) : 0.0F;
  }
  __syncthreads();
  const int slot = blockIdx.y * 128 + threadIdx.x;  // channel of the padded [heads, head_stride] row
  if (slot >= heads * head_stride) return;
  const int head = slot / head_stride, d = slot % head_stride, channels = heads * dim, channel = head * dim + d;
  const bool inside = d < dim;
  float z[kPrepTokens];
#pragma unroll
  for (int t = 0; t < kPrepTokens; ++t) z[t] = inside ? bias[channel] : 0.0F;
  if (inside) {
    for (int k = 0; k < rank; ++k) {
      const float w = weight[static_cast<std::size_t>(k) * channels + channel];
#pragma unroll
      for (int t = 0; t < kPrepTokens; ++t) z[t] = fmaf(w, bottleneck[t * rank + k], z[t]);
    }
  }
  const float scale = 1.0F / sqrtf(static_cast<float>(dim));
#pragma unroll
  for (int t = 0; t < kPrepTokens; ++t) {
    const std::size_t row = row0 + t, at = row * heads * head_stride + slot;
    const bool live = inside && row < static_cast<std::size_t>(rows);
    const T *const source = projection + row * stride;
    // sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
    alpha[at] = live ? expf(-softplus_f32(-z[t]) * inverse_tau) : 1.0F;
    queries[at] = live ? to_float(source[channel]) * scale : 0.0F;
    keys[at] = live ? to_float(source[key_column + channel]) : 0.0F;
  }
}

// ---------------------------------------------------------------- recurrence
struct RecurrenceParams {
  int rows, heads, kv_heads, dim, value_dim, head_stride;
  std::size_t value_stride;  // elements between rows of the value tensor
  int fresh;
};

__device__ __forceinline__ void copy16(float *const dst, const float *const src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<std::uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src)
               : "memory");
}

// Packed F32 pairs: one instruction for two multiply-adds.
using Pair = unsigned long long;
__device__ __forceinline__ Pair pair_of(const float low, const float high) {
  Pair d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(low), "f"(high));
  return d;
}
__device__ __forceinline__ float low_of(const Pair v) { return __uint_as_float(static_cast<unsigned int>(v)); }
__device__ __forceinline__ float high_of(const Pair v) { return __uint_as_float(static_cast<unsigned int>(v >> 32)); }
__device__ __forceinline__ Pair fma2(const Pair a, const Pair b, const Pair c) {
  Pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ Pair mul2(const Pair a, const Pair b) {
  Pair d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// A lane's key channels in a shared-memory row: kElements = 2 -> 2 lane + i, otherwise runs of four, run r at
// 128 r + 4 lane.
template <int kElements>
__device__ __forceinline__ int channel_of(const int lane, const int e) {
  if constexpr (kElements == 2) return 2 * lane + e;
  else return 128 * (e / 4) + 4 * lane + e % 4;
}
template <int kElements>
__device__ __forceinline__ void load_pairs(const float *const row, const int lane, Pair (&v)[kElements / 2]) {
  if constexpr (kElements == 2) {
    v[0] = *reinterpret_cast<const Pair *>(row + 2 * lane);
  } else {
#pragma unroll
    for (int r = 0; r < kElements / 4; ++r) {
      const ulonglong2 w = *reinterpret_cast<const ulonglong2 *>(row + 128 * r + 4 * lane);
      v[2 * r] = w.x;
      v[2 * r + 1] = w.y;
    }
  }
}

// Sums of a warp's 4 columns x 4 tokens over its 32 lanes.  The first two exchanges leave a lane with the
// column of its upper two bits, partly summed (over 4 of the 32 lanes).
__device__ __forceinline__ void scatter_columns(const float (&v)[4][kBlock], const int lane, float (&own)[kBlock]) {
  const bool upper = (lane & 16) != 0, odd = (lane & 8) != 0;
  float half[2][kBlock];
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int t = 0; t < kBlock; ++t)
      half[c][t] = (upper ? v[c + 2][t] : v[c][t]) + __shfl_xor_sync(0xffffffffU, upper ? v[c][t] : v[c + 2][t], 16);
#pragma unroll
  for (int t = 0; t < kBlock; ++t)
    own[t] = (odd ? half[1][t] : half[0][t]) + __shfl_xor_sync(0xffffffffU, odd ? half[0][t] : half[1][t], 8);
}
// ... and this leaves the sum of token 2 * bit 2 + bit 1 in the lane.
__device__ __forceinline__ float scatter_tokens(const float (&own)[kBlock], const int lane) {
  const bool upper = (lane & 4) != 0, odd = (lane & 2) != 0;
  const float a = (upper ? own[2] : own[0]) + __shfl_xor_sync(0xffffffffU, upper ? own[0] : own[2], 4);
  const float b = (upper ? own[3] : own[1]) + __shfl_xor_sync(0xffffffffU, upper ? own[1] : own[3], 4);
  const float c = (odd ? b : a) + __shfl_xor_sync(0xffffffffU, odd ? a : b, 2);
  return c + __shfl_xor_sync(0xffffffffU, c, 1);
}

template <bool kDelta, int kElements, typename T>
__global__ void __launch_bounds__(kRecurrenceThreads)
recurrence_kernel(const float *__restrict__ queries, const float *__restrict__ keys, const float *__restrict__ alpha,
                  const T *__restrict__ values, const float *__restrict__ scalars, float *__restrict__ state,
                  float *__restrict__ output, const RecurrenceParams p) {
  constexpr int kWidth = kElements * 32;
  constexpr int kPairs = kElements / 2;
  constexpr int kVectors = kDelta ? 2 : 3;  // keys, queries (, decays)
  constexpr int kScalarFloats = kDelta ? kTile / kBlock * kScalars : 0;
  constexpr int kBuffer = kVectors * kTile * kWidth + kScalarFloats + kTile * kColumns;
  extern __shared__ __align__(16) float smem[];
  const int head = blockIdx.y, column0 = blockIdx.x * kColumns;
  const int key_head = kDelta ? head / (p.heads / p.kv_heads) : head;
  const int key_heads = kDelta ? p.kv_heads : p.heads;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int own_column = column0 + warp * 4 + lane / 8;  // the column whose sums this lane ends up with
  const bool own_live = own_column < p.value_dim;
  const int own_token = 2 * ((lane >> 2) & 1) + ((lane >> 1) & 1);
  const int tiles = (p.rows + kTile - 1) / kTile;

  for (int i = threadIdx.x; i < 2 * kBuffer; i += kRecurrenceThreads) smem[i] = 0.0F;  // channels past dim stay zero
  __syncthreads();
  const auto buffer = [&](const int tile) { return smem + (tile & 1) * kBuffer; };
  // asynchronous part of a tile: rows of queries, keys, decays and the block scalars
  const auto fetch = [&](const int tile) {
    float *const b = buffer(tile);
    const int words = p.head_stride / 4;
    for (int i = threadIdx.x; i < kTile * words; i += kRecurrenceThreads) {
      const int t = i / words, word = i % words;
      const std::size_t source = (static_cast<std::size_t>(tile * kTile + t) * key_heads + key_head) * p.head_stride + word * 4;
      float *const dst = b + t * kWidth + word * 4;
      copy16(dst, keys + source);
      copy16(dst + kTile * kWidth, queries + source);
      if constexpr (!kDelta) copy16(dst + 2 * kTile * kWidth, alpha + source);
    }
    if constexpr (kDelta) {
      constexpr int kWords = kScalars / 4;
      for (int i = threadIdx.x; i < kTile / kBlock * kWords; i += kRecurrenceThreads) {
        const int block = i / kWords, word = i % kWords;
        copy16(b + kVectors * kTile * kWidth + block * kScalars + word * 4,
               scalars + (static_cast<std::size_t>(tile * (kTile / kBlock) + block) * p.heads + head) * kScalars + word * 4);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // values go through registers: kTile x kColumns of them, two per thread
  constexpr int kValuesPerThread = kTile * kColumns / kRecurrenceThreads;
  T staged[kValuesPerThread];  // widened only when they are stored: the loads stay in flight until then
  const auto load_values = [&](const int tile) {
#pragma unroll
    for (int i = 0; i < kValuesPerThread; ++i) {
      const int index = i * kRecurrenceThreads + threadIdx.x, row = tile * kTile + index / kColumns, c = column0 + index % kColumns;
      staged[i] = row < p.rows && c < p.value_dim
                      ? values[static_cast<std::size_t>(row) * p.value_stride + head * p.value_dim + c]
                      : from_float<T>(0.0F);
    }
  };
  const auto store_values = [&](const int tile) {
    float *const b = buffer(tile) + kVectors * kTile * kWidth + kScalarFloats;
#pragma unroll
    for (int i = 0; i < kValuesPerThread; ++i) b[i * kRecurrenceThreads + threadIdx.x] = to_float(staged[i]);
  };

  Pair S[4][kPairs];  // [column of the warp][channel pair]
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int e = 0; e < kPairs; ++e) {
      float v[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int d = channel_of<kElements>(lane, 2 * e + i), column = column0 + warp * 4 + c;
        v[i] = p.fresh == 0 && d < p.dim && column < p.value_dim
                   ? state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column]
                   : 0.0F;
      }
      S[c][e] = pair_of(v[0], v[1]);
    }
  fetch(0);
  load_values(0);
  for (int tile = 0; tile < tiles; ++tile) {
    store_values(tile);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // the tile is here, and nobody reads the other buffer any more
    if (tile + 1 < tiles) {
      fetch(tile + 1);
      load_values(tile + 1);
    }
    const float *const b = buffer(tile);
    const float *const value_tile = b + kVectors * kTile * kWidth + kScalarFloats + warp * 4;
    // (rows past the last token are neutral: no key, no step, no decay)
#pragma unroll
    for (int block = 0; block < kTile / kBlock; ++block) {
      const float *const base = b + block * kBlock * kWidth;
      float o;
      if constexpr (kDelta) {
        const float *const c = b + kVectors * kTile * kWidth + block * kScalars;
        Pair k[kBlock][kPairs];
        float held[4][kBlock], read[4][kBlock];  // this lane's share of S^T k_t and S^T q_t
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
          Pair q[kPairs];
          load_pairs<kElements>(base + t * kWidth, lane, k[t]);
          load_pairs<kElements>(base + (kTile + t) * kWidth, lane, q);
#pragma unroll
          for (int column = 0; column < 4; ++column) {
            Pair dk = mul2(S[column][0], k[t][0]), dq = mul2(S[column][0], q[0]);
#pragma unroll
            for (int e = 1; e < kPairs; ++e) {
              dk = fma2(S[column][e], k[t][e], dk);
              dq = fma2(S[column][e], q[e], dq);
            }
            held[column][t] = low_of(dk) + high_of(dk);
            read[column][t] = low_of(dq) + high_of(dq);
          }
        }
        float h[kBlock], r[kBlock];
        scatter_columns(held, lane, h);
        scatter_columns(read, lane, r);
#pragma unroll
        for (int offset = 4; offset > 0; offset /= 2)
#pragma unroll
          for (int t = 0; t < kBlock; ++t) h[t] += __shfl_xor_sync(0xffffffffU, h[t], offset);
        const float read_sum = scatter_tokens(r, lane);
        const float4 beta = *reinterpret_cast<const float4 *>(c + kBeta);
        const float4 beta_g = *reinterpret_cast<const float4 *>(c + kBetaG);
        const float4 pair_a = *reinterpret_cast<const float4 *>(c + kPair);
        const float4 pair_b = *reinterpret_cast<const float4 *>(c + kPair + 4);
        const float4 tail = *reinterpret_cast<const float4 *>(c + kTail);
        const float *const v = value_tile + block * kBlock * kColumns + lane / 8;
        const float u0 = fmaf(-beta_g.x, h[0], beta.x * v[0]);
        const float u1 = fmaf(-pair_a.x, u0, fmaf(-beta_g.y, h[1], beta.y * v[kColumns]));
        const float u2 = fmaf(-pair_a.z, u1, fmaf(-pair_a.y, u0, fmaf(-beta_g.z, h[2], beta.z * v[2 * kColumns])));
        const float u3 = fmaf(-pair_b.y, u2, fmaf(-pair_b.x, u1, fmaf(-pair_a.w, u0, fmaf(-beta_g.w, h[3], beta.w * v[3 * kColumns]))));
        const float4 w = *reinterpret_cast<const float4 *>(c + kRead + 4 * own_token);
        o = fmaf(w.w, u3, fmaf(w.z, u2, fmaf(w.y, u1, fmaf(w.x, u0, c[kG + own_token] * read_sum))));
        // what the block adds to the columns: every lane needs all four
        const float added[kBlock] = {tail.x * u0, tail.y * u1, tail.z * u2, u3};
        const float g = c[kG + kBlock - 1];
        const Pair gg = pair_of(g, g);
#pragma unroll
        for (int column = 0; column < 4; ++column) {
          Pair a[kBlock];
#pragma unroll
          for (int t = 0; t < kBlock; ++t) {
            const float x = __shfl_sync(0xffffffffU, added[t], 8 * column);
            a[t] = pair_of(x, x);
          }
#pragma unroll
          for (int e = 0; e < kPairs; ++e)
            S[column][e] = fma2(k[3][e], a[3], fma2(k[2][e], a[2], fma2(k[1][e], a[1], fma2(k[0][e], a[0], mul2(gg, S[column][e])))));
        }
      } else {
        float read[4][kBlock];
        // the block's operands are requested up front: one warp per scheduler has nothing else to hide them
        Pair k[kBlock][kPairs], q[kBlock][kPairs], a[kBlock][kPairs];
        float4 v[kBlock];
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
          load_pairs<kElements>(base + t * kWidth, lane, k[t]);
          load_pairs<kElements>(base + (2 * kTile + t) * kWidth, lane, a[t]);
          v[t] = *reinterpret_cast<const float4 *>(value_tile + (block * kBlock + t) * kColumns);
          load_pairs<kElements>(base + (kTile + t) * kWidth, lane, q[t]);
        }
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
          const float vs[4] = {v[t].x, v[t].y, v[t].z, v[t].w};
#pragma unroll
          for (int column = 0; column < 4; ++column) {
            const Pair vv = pair_of(vs[column], vs[column]);
            Pair dq = 0ULL;
#pragma unroll
            for (int e = 0; e < kPairs; ++e) {
              S[column][e] = fma2(k[t][e], vv, mul2(a[t][e], S[column][e]));
              dq = e == 0 ? mul2(S[column][e], q[t][e]) : fma2(S[column][e], q[t][e], dq);
            }
            read[column][t] = low_of(dq) + high_of(dq);
          }
        }
        float r[kBlock];
        scatter_columns(read, lane, r);
        o = scatter_tokens(r, lane);
      }
      const int row = tile * kTile + block * kBlock + own_token;
      if ((lane & 1) == 0 && own_live && row < p.rows)
        output[(static_cast<std::size_t>(row) * p.heads + head) * p.value_dim + own_column] = o;
    }
  }
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int e = 0; e < kElements; ++e) {
      const int d = channel_of<kElements>(lane, e), column = column0 + warp * 4 + c;
      if (d < p.dim && column < p.value_dim)
        state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column] =
            e % 2 == 0 ? low_of(S[c][e / 2]) : high_of(S[c][e / 2]);
    }
}

// ---------------------------------------------------------------- output norm and gate
template <typename T>
__global__ void __launch_bounds__(256)
norm_gate_kernel(const float *__restrict__ input, const float *__restrict__ gain, const T *__restrict__ gate,
                 const std::size_t gate_stride, const int rows, const int heads, const int value_dim,
                 const float epsilon, T *__restrict__ output) {
  const std::size_t item = static_cast<std::size_t>(blockIdx.x) * 8 + threadIdx.x / 32;
  const int lane = threadIdx.x % 32;
  if (item >= static_cast<std::size_t>(rows) * heads) return;
  const std::size_t row = item / heads, head = item % heads;
  const float *const o = input + item * value_dim;
  const T *const g = gate + row * gate_stride + head * value_dim;
  T *const out = output + item * value_dim;
  constexpr int kKept = 8;
  float v[kKept], square = 0.0F;
#pragma unroll
  for (int i = 0; i < kKept; ++i) {
    const int d = lane + 32 * i;
    v[i] = d < value_dim ? o[d] : 0.0F;
    square = fmaf(v[i], v[i], square);
  }
  for (int d = lane + 32 * kKept; d < value_dim; d += 32) square = fmaf(o[d], o[d], square);
  square = warp_sum(square);
  const float factor = 1.0F / sqrtf(square / static_cast<float>(value_dim) + epsilon);
#pragma unroll
  for (int i = 0; i < kKept; ++i) {
    const int d = lane + 32 * i;
    if (d < value_dim) out[d] = from_float<T>(v[i] * factor * gain[d] * silu_f32(to_float(g[d])));
  }
  for (int d = lane + 32 * kKept; d < value_dim; d += 32)
    out[d] = from_float<T>(o[d] * factor * gain[d] * silu_f32(to_float(g[d])));
}

// The same for value sizes that are multiples of four up to 512: a lane owns runs of four.
template <int kQuads, typename T>
__global__ void __launch_bounds__(256)
norm_gate_quads_kernel(const float *__restrict__ input, const float *__restrict__ gain, const T *__restrict__ gate,
                       const std::size_t gate_stride, const int rows, const int heads, const int value_dim,
                       const float epsilon, T *__restrict__ output) {
  const std::size_t item = static_cast<std::size_t>(blockIdx.x) * 8 + threadIdx.x / 32;
  const int lane = threadIdx.x % 32;
  if (item >= static_cast<std::size_t>(rows) * heads) return;
  const std::size_t row = item / heads, head = item % heads;
  const float *const o = input + item * value_dim;
  const T *const g = gate + row * gate_stride + head * value_dim;
  float v[kQuads][4] = {}, z[kQuads][4] = {}, square = 0.0F;
#pragma unroll
  for (int i = 0; i < kQuads; ++i) {
    const int d = 4 * (lane + 32 * i);
    if (d < value_dim) {
      load_quad(o + d, v[i]);
      load_quad(g + d, z[i]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) square = fmaf(v[i][e], v[i][e], square);
  }
  const float factor = rsqrtf(warp_sum(square) / static_cast<float>(value_dim) + epsilon);
#pragma unroll
  for (int i = 0; i < kQuads; ++i) {
    const int d = 4 * (lane + 32 * i);
    if (d >= value_dim) continue;
    float w[4], y[4];
    load_quad(gain + d, w);
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = v[i][e] * factor * w[e] * silu_f32(z[i][e]);
    store_quad(output + item * value_dim + d, y);
  }
}

// ---------------------------------------------------------------- one token
// A cluster of CTAs per key head: each owns a slice of the value columns of the heads that share the key, keeps
// its part of the state in registers between the read-out and the update (a warp per set of channels, a lane
// per column), and the output norm's sums meet in distributed shared memory.
constexpr int kDecodeRanks = 8, kDecodeThreads = 256, kDecodeWarps = kDecodeThreads / 32;
constexpr int kDecodeMaxGroup = 64;  // heads per key head

struct DecodeParams {
  int heads, kv_heads, dim, value_dim, taps, channels, rank;
  int key_column, value_column, gate_column, beta_column, decay_column;
  float inverse_tau, epsilon;
  int fresh;
};

template <bool kDelta, typename T>
__global__ void __launch_bounds__(kDecodeThreads)
decode_kernel(const T *__restrict__ projection, T *const history, const float *__restrict__ conv,
              const float *__restrict__ decay_rate, const float *__restrict__ decay_shift,
              const float *__restrict__ decay_weight, const float *__restrict__ decay_bias,
              const float *__restrict__ gain, float *const state, T *__restrict__ output, const DecodeParams p) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float key[kDecoderMaxHeadDim], query[kDecoderMaxHeadDim], alpha[kDecoderMaxHeadDim];
  __shared__ float partial[2][kDecodeWarps][32], scratch[kDecodeWarps];
  __shared__ float squares[kDecodeMaxGroup];  // this CTA's part of every head's sum of squares
  extern __shared__ float outputs[];          // this CTA's columns
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = static_cast<int>(cluster.block_rank()), g = blockIdx.y;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int group = kDelta ? p.heads / p.kv_heads : 1;
  const int columns = group * p.value_dim, share = (columns + kDecodeRanks - 1) / kDecodeRanks;
  const int begin = rank * share, count = max(0, min(columns, begin + share) - begin);
  const auto convolved = [&](const int column) {
    return conv_silu(projection, 0, history, p.channels, conv, p.taps, p.fresh != 0, 0, column);
  };
  float k = 0.0F, q = 0.0F;
  const int d = threadIdx.x;  // kDecodeThreads == kDecoderMaxHeadDim: a thread per key channel
  if (d < p.dim) {
    if constexpr (kDelta) {
      k = convolved(p.key_column + g * p.dim + d);
      q = convolved(g * p.dim + d);
    } else {
      const int channel = g * p.dim + d;
      k = to_float(projection[p.key_column + channel]);
      q = to_float(projection[channel]);
      float z = decay_bias[channel];
      for (int r = 0; r < p.rank; ++r)
        z = fmaf(decay_weight[static_cast<std::size_t>(r) * p.heads * p.dim + channel], to_float(projection[p.beta_column + r]), z);
      alpha[d] = expf(-softplus_f32(-z) * p.inverse_tau);
    }
  }
  const float inverse_root = 1.0F / sqrtf(static_cast<float>(p.dim));
  if constexpr (kDelta) {
    k *= 1.0F / sqrtf(block_sum<kDecodeThreads>(k * k, scratch) + 1e-6F);
    q *= 1.0F / sqrtf(block_sum<kDecodeThreads>(q * q, scratch) + 1e-6F);
  }
  q *= inverse_root;
  if (d < p.dim) {
    key[d] = k;
    query[d] = q;
  }
  const float key_query = block_sum<kDecodeThreads>(k * q, scratch);  // (its barriers also publish key and query)
  constexpr int kHeld = static_cast<int>(kDecoderMaxHeadDim) / kDecodeWarps;
  for (int c0 = 0; c0 < count; c0 += 32) {
    const int c = begin + c0 + lane;
    const bool live = c0 + lane < count;
    const int head = g * group + (live ? c / p.value_dim : 0), column = live ? c % p.value_dim : 0;
    float *const cells = state + static_cast<std::size_t>(head) * p.dim * p.value_dim + column;
    float v = 0.0F, beta = 0.0F, decay = 1.0F;
    if (live) {
      if constexpr (kDelta) {
        v = convolved(p.value_column + head * p.value_dim + column);
        v = to_float(from_float<T>(v));  // the prompt's kernels keep convolved values in the activation type
        beta = sigmoid_f32(to_float(projection[p.beta_column + head]));
        decay = expf(decay_rate[head] * softplus_f32(to_float(projection[p.decay_column + head]) + decay_shift[head]));
      } else {
        v = to_float(projection[p.value_column + head * p.value_dim + column]);
      }
    }
    float held[kHeld], with_key = 0.0F, with_query = 0.0F;
#pragma unroll
    for (int i = 0; i < kHeld; ++i) {
      const int row = warp + kDecodeWarps * i;
      held[i] = live && row < p.dim && p.fresh == 0 ? cells[static_cast<std::size_t>(row) * p.value_dim] : 0.0F;
    }
#pragma unroll
    for (int i = 0; i < kHeld; ++i) {
      const int row = warp + kDecodeWarps * i;
      if (row < p.dim) {
        if constexpr (kDelta) {
          held[i] *= decay;
          with_key = fmaf(held[i], key[row], with_key);
        } else {
          held[i] = fmaf(key[row], v, alpha[row] * held[i]);
        }
        with_query = fmaf(held[i], query[row], with_query);
      }
    }
    partial[0][warp][lane] = with_key;
    partial[1][warp][lane] = with_query;
    __syncthreads();
    with_key = with_query = 0.0F;
#pragma unroll
    for (int w = 0; w < kDecodeWarps; ++w) {
      with_key += partial[0][w][lane];
      with_query += partial[1][w][lane];
    }
    const float u = kDelta ? beta * (v - with_key) : 0.0F;
    const float o = kDelta ? fmaf(u, key_query, with_query) : with_query;
#pragma unroll
    for (int i = 0; i < kHeld; ++i) {
      const int row = warp + kDecodeWarps * i;
      if (live && row < p.dim)
        cells[static_cast<std::size_t>(row) * p.value_dim] = kDelta ? fmaf(key[row], u, held[i]) : held[i];
    }
    if (warp == 0 && live) outputs[c0 + lane] = o;
    __syncthreads();
  }
  for (int local = 0; local < group; ++local) {
    const int from = max(local * p.value_dim, begin) - begin, to = min((local + 1) * p.value_dim, begin + count) - begin;
    float square = 0.0F;
    if (from < to) {  // the same for every thread
      for (int c = from + threadIdx.x; c < to; c += kDecodeThreads) square = fmaf(outputs[c], outputs[c], square);
      square = block_sum<kDecodeThreads>(square, scratch);
    }
    if (threadIdx.x == 0) squares[local] = square;
  }
  cluster.sync();  // every part of the norms is there, and every CTA has read the history of the shared channels
  for (int c = threadIdx.x; c < count; c += kDecodeThreads) {
    const int local = (begin + c) / p.value_dim, column = (begin + c) % p.value_dim, head = g * group + local;
    float total = 0.0F;
    for (int r = 0; r < kDecodeRanks; ++r) total += cluster.map_shared_rank(squares, r)[local];
    const float factor = 1.0F / sqrtf(total / static_cast<float>(p.value_dim) + p.epsilon);
    const int at = head * p.value_dim + column;
    output[at] = from_float<T>(outputs[c] * factor * gain[column] * silu_f32(to_float(projection[p.gate_column + at])));
  }
  if constexpr (kDelta) {
    const auto advance = [&](const int column) {
      for (int i = 0; i + 1 < p.taps; ++i)
        history[static_cast<std::size_t>(i) * p.channels + column] =
            i + 2 < p.taps ? (p.fresh == 0 ? history[static_cast<std::size_t>(i + 1) * p.channels + column] : from_float<T>(0.0F))
                           : projection[column];
    };
    for (int c = threadIdx.x; c < count; c += kDecodeThreads) advance(p.value_column + g * columns + begin + c);
    if (rank == 0 && d < p.dim) {
      advance(g * p.dim + d);
      advance(p.key_column + g * p.dim + d);
    }
  }
  cluster.sync();  // remote shared memory stays alive until everybody has read it
}

template <bool kDelta, typename T>
int launch_decode(const RecurrentArgs &a, cudaStream_t stream) {
  DecodeParams p{};
  p.heads = static_cast<int>(a.heads);
  p.kv_heads = static_cast<int>(a.kv_heads);
  p.dim = static_cast<int>(a.dim);
  p.value_dim = static_cast<int>(a.value_dim);
  p.taps = static_cast<int>(a.conv_taps);
  p.channels = static_cast<int>(a.gate_column);
  p.rank = static_cast<int>(a.decay_rank);
  p.key_column = static_cast<int>(a.key_column);
  p.value_column = static_cast<int>(a.value_column);
  p.gate_column = static_cast<int>(a.gate_column);
  p.beta_column = static_cast<int>(a.beta_column);
  p.decay_column = static_cast<int>(a.decay_column);
  p.inverse_tau = 1.0F / a.tau;
  p.epsilon = a.epsilon;
  p.fresh = a.fresh ? 1 : 0;
  cudaLaunchAttribute attribute{};
  attribute.id = cudaLaunchAttributeClusterDimension;
  attribute.val.clusterDim.x = kDecodeRanks;
  attribute.val.clusterDim.y = attribute.val.clusterDim.z = 1;
  cudaLaunchConfig_t config{};
  config.gridDim = dim3(kDecodeRanks, static_cast<unsigned int>(kDelta ? a.kv_heads : a.heads));
  config.blockDim = dim3(kDecodeThreads);
  const std::size_t columns = (kDelta ? a.heads / a.kv_heads : 1) * a.value_dim;
  config.dynamicSmemBytes = (columns + kDecodeRanks - 1) / kDecodeRanks * sizeof(float);
  config.stream = stream;
  config.attrs = &attribute;
  config.numAttrs = 1;
  if (cudaLaunchKernelEx(&config, decode_kernel<kDelta, T>, static_cast<const T *>(a.projection),
                         static_cast<T *>(a.conv_history), a.conv, a.decay_rate, a.decay_shift, a.decay_weight,
                         a.decay_bias, a.output_norm, a.state, static_cast<T *>(a.output), p) != cudaSuccess)
    return fail(kCuda, std::string("cannot launch the recurrent decode kernel: ") +
                           cudaGetErrorString(cudaGetLastError()));
  return check_launch("recurrent decode kernel");
}

template <bool kDelta, int kElements, typename T>
int launch_recurrence(const float *queries, const float *keys, const float *alpha, const T *values,
                      const float *scalars, float *state, float *output, const RecurrenceParams &p,
                      cudaStream_t stream) {
  constexpr std::size_t kBuffer = (kDelta ? 2 : 3) * kTile * kElements * 32 + (kDelta ? kTile / kBlock * kScalars : 0) + kTile * kColumns;
  constexpr std::size_t bytes = 2 * kBuffer * sizeof(float);
  if (cudaFuncSetAttribute(recurrence_kernel<kDelta, kElements, T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           static_cast<int>(bytes)) != cudaSuccess)
    return fail(kCuda, "cannot raise the recurrence shared-memory limit");
  const dim3 grid(ceil_div_u(p.value_dim, kColumns), static_cast<unsigned int>(p.heads));
  recurrence_kernel<kDelta, kElements, T><<<grid, kRecurrenceThreads, bytes, stream>>>(queries, keys, alpha, values,
                                                                                       scalars, state, output, p);
  return check_launch(kDelta ? "gated delta rule kernel" : "gated linear attention kernel");
}

template <bool kDelta, typename T>
int dispatch_recurrence(const float *queries, const float *keys, const float *alpha, const T *values,
                        const float *scalars, float *state, float *output, const RecurrenceParams &p,
                        cudaStream_t stream) {
  if (p.dim <= 64) return launch_recurrence<kDelta, 2, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
  if (p.dim <= 128) return launch_recurrence<kDelta, 4, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
  return launch_recurrence<kDelta, 8, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
}

template <typename T>
int advance_history(const RecurrentArgs &a, cudaStream_t stream) {
  if (!a.delta || a.conv_taps <= 1) return kOk;
  conv_history_kernel<T><<<ceil_div_u(a.gate_column, 256), 256, 0, stream>>>(
      static_cast<const T *>(a.projection), a.stride, static_cast<T *>(a.conv_history), static_cast<int>(a.gate_column),
      static_cast<int>(a.conv_taps) - 1, static_cast<int>(a.rows), a.fresh);
  return check_launch("convolution history kernel");
}

template <typename T>
int norm_gate(const RecurrentArgs &a, const float *input, cudaStream_t stream) {
  const T *const gate = static_cast<const T *>(a.projection) + a.gate_column;
  const bool quads = a.value_dim % 4 == 0 && a.value_dim <= 512 && a.stride % 8 == 0 && a.gate_column % 8 == 0 &&
                     aligned16(a.projection) && aligned16(a.output) && aligned16(a.output_norm);
  const auto kernel = !quads ? norm_gate_kernel<T>
                      : a.value_dim <= 128 ? norm_gate_quads_kernel<1, T>
                      : a.value_dim <= 256 ? norm_gate_quads_kernel<2, T> : norm_gate_quads_kernel<4, T>;
  kernel<<<ceil_div_u(a.rows * a.heads, 8), 256, 0, stream>>>(
      input, a.output_norm, gate, a.stride, static_cast<int>(a.rows), static_cast<int>(a.heads),
      static_cast<int>(a.value_dim), a.epsilon, static_cast<T *>(a.output));
  return check_launch("output norm and gate kernel");
}

int run_chunks(const RecurrentArgs &a, cudaStream_t stream) {
  float *output = nullptr;
  int status = recurrent_chunks(a, &output, stream);
  if (status == kOk) status = advance_history<bf16>(a, stream);
  return status == kOk ? norm_gate<bf16>(a, output, stream) : status;
}

template <typename T>
int run(const RecurrentArgs &a, cudaStream_t stream) {
  const Workspace w = workspace_layout(a.delta, a.rows, a.heads, a.kv_heads, a.dim, a.value_dim, a.type);
  unsigned char *const base = static_cast<unsigned char *>(a.workspace);
  float *const queries = reinterpret_cast<float *>(base + w.query), *const keys = reinterpret_cast<float *>(base + w.key);
  float *const output = reinterpret_cast<float *>(base + w.output);
  const T *const projection = static_cast<const T *>(a.projection);
  RecurrenceParams p{};
  p.rows = static_cast<int>(a.rows);
  p.heads = static_cast<int>(a.heads);
  p.kv_heads = static_cast<int>(a.kv_heads);
  p.dim = static_cast<int>(a.dim);
  p.value_dim = static_cast<int>(a.value_dim);
  p.head_stride = static_cast<int>(w.head_stride);
  p.fresh = a.fresh ? 1 : 0;
  int status;
  if (a.delta) {
    DeltaPrepParams d{};
    d.stride = a.stride;
    d.rows = p.rows;
    d.padded_rows = static_cast<int>(w.rows);
    d.heads = p.heads;
    d.kv_heads = p.kv_heads;
    d.dim = p.dim;
    d.value_dim = p.value_dim;
    d.head_stride = p.head_stride;
    d.taps = static_cast<int>(a.conv_taps);
    d.channels = static_cast<int>(a.gate_column);
    d.key_column = static_cast<int>(a.key_column);
    d.value_column = static_cast<int>(a.value_column);
    d.beta_column = static_cast<int>(a.beta_column);
    d.decay_column = static_cast<int>(a.decay_column);
    d.fresh = p.fresh;
    float *const scalars = reinterpret_cast<float *>(base + w.scalars);
    T *const values = reinterpret_cast<T *>(base + w.value);
    const dim3 grid(static_cast<unsigned int>(w.rows / kBlock), static_cast<unsigned int>(a.kv_heads));
    delta_prepare_kernel<T><<<grid, 128, 2 * kBlock * a.dim * sizeof(float), stream>>>(
        projection, static_cast<const T *>(a.conv_history), a.conv, a.decay_rate, a.decay_shift, queries, keys, values,
        scalars, d);
    if ((status = check_launch("delta preparation kernel")) != kOk) return status;
    if ((status = advance_history<T>(a, stream)) != kOk) return status;
    p.value_stride = a.heads * a.value_dim;
    status = dispatch_recurrence<true, T>(queries, keys, nullptr, values, scalars, a.state, output, p, stream);
  } else {
    float *const alpha = reinterpret_cast<float *>(base + w.alpha);
    const dim3 grid(static_cast<unsigned int>(w.rows / kPrepTokens), ceil_div_u(a.heads * w.head_stride, 128));
    linear_prepare_kernel<T><<<grid, 128, kPrepTokens * a.decay_rank * sizeof(float), stream>>>(
        projection, a.stride, static_cast<int>(a.key_column), static_cast<int>(a.beta_column), a.decay_weight,
        a.decay_bias, static_cast<int>(a.decay_rank), 1.0F / a.tau, p.rows, p.heads, p.dim, p.head_stride, queries, keys,
        alpha);
    if ((status = check_launch("linear attention preparation kernel")) != kOk) return status;
    p.value_stride = a.stride;
    status = dispatch_recurrence<false, T>(queries, keys, alpha, projection + a.value_column, nullptr, a.state, output, p,
                                           stream);
  }
  if (status != kOk) return status;
  return norm_gate<T>(a, output, stream);
}

}  // namespace

std::size_t recurrent_workspace_bytes(const bool delta, const std::size_t rows, const std::size_t heads,
                                      const std::size_t kv_heads, const std::size_t dim, const std::size_t value_dim,
                                      const Activation type) {
  const std::size_t blocks = workspace_layout(delta, rows, heads, kv_heads, dim, value_dim, type).bytes;
  const std::size_t chunks = recurrent_chunks_workspace(delta, rows, heads, kv_heads, dim, value_dim);
  return blocks > chunks ? blocks : chunks;
}

int recurrent_mixer(const RecurrentArgs &a, cudaStream_t stream) {
  if (a.projection == nullptr || a.output_norm == nullptr || a.state == nullptr || a.workspace == nullptr ||
      a.output == nullptr || a.heads == 0 || a.heads > 65535 || a.kv_heads == 0 || a.heads % a.kv_heads != 0 ||
      a.dim == 0 || a.dim > kDecoderMaxHeadDim || a.value_dim == 0 || a.rows > 0x3fffffffU || a.stride > 0x7fffff00U ||
      !aligned16(a.workspace))
    return fail(kInvalidArgument, "recurrent mixer arguments are invalid");
  if (a.delta && (a.conv == nullptr || a.conv_taps == 0 || (a.conv_taps > 1 && a.conv_history == nullptr) ||
                  a.decay_rate == nullptr || a.decay_shift == nullptr))
    return fail(kInvalidArgument, "delta mixer arguments are invalid");
  if (!a.delta && (a.decay_weight == nullptr || a.decay_bias == nullptr || a.decay_rank == 0 ||
                   !(a.tau > 0.0F)))
    return fail(kInvalidArgument, "linear attention arguments are invalid");
  if (!a.delta && a.decay_rank > kMaxDecayRank)
    return fail(kUnsupported, "decay bottlenecks wider than " + std::to_string(kMaxDecayRank) + " are not supported");
  if (a.rows == 0) return kOk;
  const std::size_t decode_columns = (a.delta ? a.heads / a.kv_heads : 1) * a.value_dim;
  if (a.rows == 1 && (!a.delta || a.heads / a.kv_heads <= static_cast<std::size_t>(kDecodeMaxGroup)) &&
      decode_columns <= 8192 * static_cast<std::size_t>(kDecodeRanks)) {
    if (a.type == Activation::kBf16) return a.delta ? launch_decode<true, bf16>(a, stream) : launch_decode<false, bf16>(a, stream);
    return a.delta ? launch_decode<true, float>(a, stream) : launch_decode<false, float>(a, stream);
  }
  if (recurrent_chunks_applicable(a)) return run_chunks(a, stream);
  return a.type == Activation::kBf16 ? run<bf16>(a, stream) : run<float>(a, stream);
}

}  // namespace evob
