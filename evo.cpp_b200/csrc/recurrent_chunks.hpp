// Tensor-core form of the recurrences for BF16 prompts (recurrent_chunks.cu), used by recurrent_mixer.
#pragma once

#include "decoder_ops.hpp"

namespace evob {

bool recurrent_chunks_applicable(const RecurrentArgs &args);
std::size_t recurrent_chunks_workspace(bool delta, std::size_t rows, std::size_t heads, std::size_t kv_heads,
                                       std::size_t dim, std::size_t value_dim);
// Prepares and runs the recurrence; *output is the F32 [rows, heads, value_dim] result inside the workspace.
// The convolution's history is read, not advanced.
int recurrent_chunks(const RecurrentArgs &args, float **output, cudaStream_t stream);

}  // namespace evob
