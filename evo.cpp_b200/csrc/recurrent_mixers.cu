// Mixers with a matrix state per head: gated linear attention (a decay per key channel) and the gated
// delta rule (a scalar decay per head, values corrected by what the state already holds for the key).
// Everything that enters the recurrences is F32.
//
// A prompt portion runs in three launches:
//   1. preparation: per token the decays and the queries / keys the recurrence reads (F32), for the delta
//      rule also the short convolutions, the unit vectors, the step sizes, and the scalars of the blocked
//      form below;
//   2. the recurrence: columns of the state (one per value channel) never mix, so a CTA owns 16 of them;
//      eight lanes share a column, each with kElements key channels of it in registers, and the tokens
//      stream through a double-buffered shared-memory tile;
//   3. the output norm and gate, row-wise.
//
// Blocked delta rule.  Four tokens at a time, with S the state in front of the block, G_t = g_0 .. g_t and
// D_ts = g_{s+1} .. g_t the decay products inside it:
//   u_t = beta_t (v_t - G_t S^T k_t - sum_{s<t} D_ts (k_s.k_t) u_s)
//   o_t = G_t S^T q_t + sum_{s<=t} D_ts (k_s.q_t) u_s
//   S'  = G_3 S + sum_s D_3s k_s u_s^T
// so the eight products with S are taken at once and reduced over the lanes together; the scalars
// depend on the head only and come from the preparation.
#include "decoder_types.cuh"
#include "ops_internal.hpp"

namespace evob {
namespace {

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

// Sums four values over the eight lanes of a column; lane p is left with the sum of value
// 2 * bit2(p) + bit1(p).
__device__ __forceinline__ float reduce_scatter4(const float (&v)[4], const int part) {
  const bool high = (part & 4) != 0, odd = (part & 2) != 0;
  float a = high ? v[2] : v[0], b = high ? v[3] : v[1];
  a += __shfl_xor_sync(0xffffffffU, high ? v[0] : v[2], 4);
  b += __shfl_xor_sync(0xffffffffU, high ? v[1] : v[3], 4);
  float c = odd ? b : a;
  c += __shfl_xor_sync(0xffffffffU, odd ? a : b, 2);
  return c + __shfl_xor_sync(0xffffffffU, c, 1);
}

template <bool kDelta, int kElements, typename T>
__global__ void __launch_bounds__(kRecurrenceThreads)
recurrence_kernel(const float *__restrict__ queries, const float *__restrict__ keys, const float *__restrict__ alpha,
                  const T *__restrict__ values, const float *__restrict__ scalars, float *__restrict__ state,
                  float *__restrict__ output, const RecurrenceParams p) {
  constexpr int kWidth = kElements * 8;
  constexpr int kVectors = kDelta ? 2 : 3;  // keys, queries (, decays)
  constexpr int kScalarFloats = kDelta ? kTile / kBlock * kScalars : 0;
  constexpr int kBuffer = kVectors * kTile * kWidth + kScalarFloats + kTile * kColumns;
  extern __shared__ __align__(16) float smem[];
  const int head = blockIdx.y, column0 = blockIdx.x * kColumns;
  const int key_head = kDelta ? head / (p.heads / p.kv_heads) : head;
  const int key_heads = kDelta ? p.kv_heads : p.heads;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32, part = lane % 8;
  const int local = warp * 4 + lane / 8, column = column0 + local;  // this thread's state column
  const bool live = column < p.value_dim;
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
  float staged[kValuesPerThread];
  const auto load_values = [&](const int tile) {
#pragma unroll
    for (int i = 0; i < kValuesPerThread; ++i) {
      const int index = i * kRecurrenceThreads + threadIdx.x, row = tile * kTile + index / kColumns, c = column0 + index % kColumns;
      staged[i] = row < p.rows && c < p.value_dim
                      ? to_float(values[static_cast<std::size_t>(row) * p.value_stride + head * p.value_dim + c])
                      : 0.0F;
    }
  };
  const auto store_values = [&](const int tile) {
    float *const b = buffer(tile) + kVectors * kTile * kWidth + kScalarFloats;
#pragma unroll
    for (int i = 0; i < kValuesPerThread; ++i) b[i * kRecurrenceThreads + threadIdx.x] = staged[i];
  };

  float S[kElements];
#pragma unroll
  for (int e = 0; e < kElements; ++e) {
    const int d = (e / 4 * 8 + part) * 4 + e % 4;
    S[e] = p.fresh == 0 && live && d < p.dim
               ? state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column]
               : 0.0F;
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
    const float *const value_tile = b + kVectors * kTile * kWidth + kScalarFloats + local;
    const float *const lane_base = b + part * 4;
    const int blocks = min(kTile, p.rows - tile * kTile + kBlock - 1) / kBlock;
    for (int block = 0; block < blocks; ++block) {
      const float *const base = lane_base + block * kBlock * kWidth;
      float read[kBlock];  // S^T q_t
      if constexpr (kDelta) {
        const float *const c = b + kVectors * kTile * kWidth + block * kScalars;
        float k[kBlock][kElements], held[kBlock];  // S^T k_t
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
          float dk[2] = {0.0F, 0.0F}, dq[2] = {0.0F, 0.0F};
#pragma unroll
          for (int e = 0; e < kElements; e += 4) {
            const float4 kv = *reinterpret_cast<const float4 *>(base + t * kWidth + e * 8);
            const float4 qv = *reinterpret_cast<const float4 *>(base + (kTile + t) * kWidth + e * 8);
            k[t][e] = kv.x, k[t][e + 1] = kv.y, k[t][e + 2] = kv.z, k[t][e + 3] = kv.w;
            dk[0] = fmaf(S[e], kv.x, dk[0]);
            dk[1] = fmaf(S[e + 1], kv.y, dk[1]);
            dk[0] = fmaf(S[e + 2], kv.z, dk[0]);
            dk[1] = fmaf(S[e + 3], kv.w, dk[1]);
            dq[0] = fmaf(S[e], qv.x, dq[0]);
            dq[1] = fmaf(S[e + 1], qv.y, dq[1]);
            dq[0] = fmaf(S[e + 2], qv.z, dq[0]);
            dq[1] = fmaf(S[e + 3], qv.w, dq[1]);
          }
          held[t] = dk[0] + dk[1];
          read[t] = dq[0] + dq[1];
        }
        const float mine = reduce_scatter4(held, part);
        const float read_sum = reduce_scatter4(read, part);
#pragma unroll
        for (int t = 0; t < kBlock; ++t) held[t] = __shfl_sync(0xffffffffU, mine, (lane & 24) + 2 * t);
        const float4 beta = *reinterpret_cast<const float4 *>(c + kBeta);
        const float4 beta_g = *reinterpret_cast<const float4 *>(c + kBetaG);
        const float4 pair_a = *reinterpret_cast<const float4 *>(c + kPair);
        const float4 pair_b = *reinterpret_cast<const float4 *>(c + kPair + 4);
        const float4 tail = *reinterpret_cast<const float4 *>(c + kTail);
        const float *const v = value_tile + block * kBlock * kColumns;
        const float u0 = fmaf(-beta_g.x, held[0], beta.x * v[0]);
        const float u1 = fmaf(-pair_a.x, u0, fmaf(-beta_g.y, held[1], beta.y * v[kColumns]));
        const float u2 = fmaf(-pair_a.z, u1, fmaf(-pair_a.y, u0, fmaf(-beta_g.z, held[2], beta.z * v[2 * kColumns])));
        const float u3 = fmaf(-pair_b.y, u2, fmaf(-pair_b.x, u1, fmaf(-pair_a.w, u0, fmaf(-beta_g.w, held[3], beta.w * v[3 * kColumns]))));
        const int t = 2 * ((part >> 2) & 1) + ((part >> 1) & 1);
        const float4 r = *reinterpret_cast<const float4 *>(c + kRead + 4 * t);
        const float o = fmaf(r.w, u3, fmaf(r.z, u2, fmaf(r.y, u1, fmaf(r.x, u0, c[kG + t] * read_sum))));
        const int row = tile * kTile + block * kBlock + t;
        if ((part & 1) == 0 && live && row < p.rows)
          output[(static_cast<std::size_t>(row) * p.heads + head) * p.value_dim + column] = o;
        const float g = c[kG + kBlock - 1];
        const float w0 = tail.x * u0, w1 = tail.y * u1, w2 = tail.z * u2;
#pragma unroll
        for (int e = 0; e < kElements; ++e)
          S[e] = fmaf(k[3][e], u3, fmaf(k[2][e], w2, fmaf(k[1][e], w1, fmaf(k[0][e], w0, g * S[e]))));
      } else {
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
          const float v = value_tile[(block * kBlock + t) * kColumns];
          float dq[2] = {0.0F, 0.0F};
#pragma unroll
          for (int e = 0; e < kElements; e += 4) {
            const float4 kv = *reinterpret_cast<const float4 *>(base + t * kWidth + e * 8);
            const float4 qv = *reinterpret_cast<const float4 *>(base + (kTile + t) * kWidth + e * 8);
            const float4 av = *reinterpret_cast<const float4 *>(base + (2 * kTile + t) * kWidth + e * 8);
            S[e] = fmaf(kv.x, v, av.x * S[e]);
            S[e + 1] = fmaf(kv.y, v, av.y * S[e + 1]);
            S[e + 2] = fmaf(kv.z, v, av.z * S[e + 2]);
            S[e + 3] = fmaf(kv.w, v, av.w * S[e + 3]);
            dq[0] = fmaf(S[e], qv.x, dq[0]);
            dq[1] = fmaf(S[e + 1], qv.y, dq[1]);
            dq[0] = fmaf(S[e + 2], qv.z, dq[0]);
            dq[1] = fmaf(S[e + 3], qv.w, dq[1]);
          }
          read[t] = dq[0] + dq[1];
        }
        const float o = reduce_scatter4(read, part);
        const int row = tile * kTile + block * kBlock + 2 * ((part >> 2) & 1) + ((part >> 1) & 1);
        if ((part & 1) == 0 && live && row < p.rows)
          output[(static_cast<std::size_t>(row) * p.heads + head) * p.value_dim + column] = o;
      }
    }
  }
#pragma unroll
  for (int e = 0; e < kElements; ++e) {
    const int d = (e / 4 * 8 + part) * 4 + e % 4;
    if (live && d < p.dim) state[(static_cast<std::size_t>(head) * p.dim + d) * p.value_dim + column] = S[e];
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

template <bool kDelta, int kElements, typename T>
int launch_recurrence(const float *queries, const float *keys, const float *alpha, const T *values,
                      const float *scalars, float *state, float *output, const RecurrenceParams &p,
                      cudaStream_t stream) {
  constexpr std::size_t kBuffer = (kDelta ? 2 : 3) * kTile * kElements * 8 + (kDelta ? kTile / kBlock * kScalars : 0) + kTile * kColumns;
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
  if (p.dim <= 32) return launch_recurrence<kDelta, 4, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
  if (p.dim <= 64) return launch_recurrence<kDelta, 8, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
  if (p.dim <= 128) return launch_recurrence<kDelta, 16, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
  return launch_recurrence<kDelta, 32, T>(queries, keys, alpha, values, scalars, state, output, p, stream);
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
    if (a.conv_taps > 1) {
      conv_history_kernel<T><<<ceil_div_u(a.gate_column, 256), 256, 0, stream>>>(
          projection, a.stride, static_cast<T *>(a.conv_history), d.channels, d.taps - 1, p.rows, a.fresh);
      if ((status = check_launch("convolution history kernel")) != kOk) return status;
    }
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
  norm_gate_kernel<T><<<ceil_div_u(a.rows * a.heads, 8), 256, 0, stream>>>(
      output, a.output_norm, projection + a.gate_column, a.stride, p.rows, p.heads, p.value_dim, a.epsilon,
      static_cast<T *>(a.output));
  return check_launch("output norm and gate kernel");
}

}  // namespace

std::size_t recurrent_workspace_bytes(const bool delta, const std::size_t rows, const std::size_t heads,
                                      const std::size_t kv_heads, const std::size_t dim, const std::size_t value_dim,
                                      const Activation type) {
  return workspace_layout(delta, rows, heads, kv_heads, dim, value_dim, type).bytes;
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
  if (!a.delta && (a.decay_weight == nullptr || a.decay_bias == nullptr || a.decay_rank == 0 || a.decay_rank > 2048 ||
                   !(a.tau > 0.0F)))
    return fail(kInvalidArgument, "linear attention arguments are invalid");
  if (a.rows == 0) return kOk;
  return a.type == Activation::kBf16 ? run<bf16>(a, stream) : run<float>(a, stream);
}

}  // namespace evob
