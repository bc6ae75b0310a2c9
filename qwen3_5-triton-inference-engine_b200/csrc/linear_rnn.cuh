// Shared declarations of the forget-gated outer-product recurrence's kernels (linear_rnn.cu, linear_rnn_chunk.cu).
#pragma once
#include "b200_attn.h"
#include "common.cuh"

namespace b200 {

struct OuterRnnParams {
  const void* qfv;         // [rows, stride] E: [q heads*dim | f heads*dim | v heads*vdim]
  int64_t stride;
  const float* lower;      // [heads*dim]
  const float* bias;       // [heads*dim]
  float* state;            // [slots, heads, dim, vdim]
  const int32_t* cu;
  const int32_t* slots;
  const int32_t* start;
  float* o;                // [rows, heads*vdim] fp32, before the head norm
  int heads, dim, vdim;    // padded sizes
  // chunked form with the head norm inside (out != NULL)
  const float* norm;
  void* out;
  int true_vdim;
  float eps;
  // chunked form over segments of `segment` tokens (a multiple of 16), at most `segments` per sequence (1: none)
  int segment, segments;
  float* seg_state;        // [sequences, segments, heads, dim, vdim]
  float* seg_decay;        // [sequences, segments, heads, dim]
};

bool outer_rnn_chunk_supports(int dim, int vdim);
int outer_rnn_chunk_launch(const OuterRnnParams& p, int n, cudaStream_t st);

}  // namespace b200
