// The gated delta rule with one decay a head over long prompt portions, a chunk of tokens at a time (delta_chunk.cu).
#pragma once

#include "common.cuh"

namespace mi {

constexpr int DELTA_CHUNK_TOKENS = 64;
constexpr int DELTA_CHUNK_MAX_DIM = 128;      // key channels a head

struct DeltaChunkArgs {
  const float* qn; const float* kn;           // [tokens, kv_heads * dim] unit queries (times dim^-1/2) and keys
  const float* lg; const float* beta;         // [tokens, heads] logarithms of the decays, write strengths
  float* raw;                                 // [tokens, heads * vdim]: the values in, the read-outs out
  float* state; long long state_stride;       // [slot][heads][dim][vdim]
  const int* q_start; const int* q_len; const int* seq_slot;
  int items, heads, kv_heads, dim, vdim;
  int min_tokens;                             // items of fewer new tokens are left alone
};

// Floats of scratch for a step of T tokens in `items` items (some slabs of chunks at a time share it).
long long delta_chunk_scratch_floats(int T, int items, int heads, int dim, int vdim);
int delta_chunk_slabs(int T, int items, int heads);      // three launches each
int delta_chunk_run(const DeltaChunkArgs& a, int T, float* scratch, cudaStream_t stream);

}  // namespace mi
