// Shared declarations of the outer-product recurrences' kernels (linear_rnn.cu, linear_rnn_chunk.cu, ssd.cu):
//   S_t = diag(f_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// per head, S [dim, vdim] in fp32.  The kinds differ in where f, k, q and v come from and in what happens to o:
//   FORGET  HGRN2: f = l + (1 - l) sigmoid(f' + bias), k = 1 - f, q = silu(q'); head norm
//   KEYED   gated linear attention: f = sigmoid(z + bias)^(1 / tau), k as projected, q = q' * scale; head norm, times silu(gate)
//   SSD     state space: f = exp(-exp(A) dt) for all rows, dt = softplus(dt' + bias), k = dt * B, q = C, v = x; plus D x.
//           B and C belong to groups of heads.
#pragma once
#include "b200_attn.h"
#include "elem.cuh"

namespace b200 {

enum RnnKind { RNN_FORGET, RNN_KEYED, RNN_SSD };

struct OuterRnnParams {
  const void* x;           // [rows, stride] E with the columns below
  int64_t stride;
  int q_off, k_off, v_off; // first columns of q, of k (FORGET: f') and of v; head h takes q, k at (h / per_group) * dim
  int per_group;
  float* state;            // [slots, heads, dim, vdim]
  const int32_t* cu;
  const int32_t* slots;
  const int32_t* start;
  float* o;                // [rows, heads*vdim] fp32: o before the head norm (prefill), or y (SSD decode)
  int heads, dim, vdim;    // padded sizes
  const float* lower;      // FORGET [heads*dim]
  const float* bias;       // FORGET, KEYED [heads*dim], SSD [heads] (dt)
  // KEYED: z of a prefill (fp32 [rows, z_stride]); in the decode step z = w_low . low, per row and channel
  const float* z;
  int64_t z_stride;
  const void* low;         // [rows, stride] E: `rank` columns
  const void* w_low;       // [heads*dim, rank] E
  int rank;
  float q_scale, inv_tau;
  // SSD
  const void* dt;          // [rows, dt_stride] E, one column per head
  int64_t dt_stride;
  const float *a_log, *skip;   // [heads]
  // SSD decode: x holds the raw inputs [x | B | C] of a causal convolution; ring [slots, taps, channels] fp32 keeps the last ones
  float* ring;
  const float *taps_w, *taps_b;  // [taps, channels] (first row: the current token's weight), [channels]
  int taps, channels;
  // head norm and gate
  const float* norm;       // [vdim]
  const void* gate;        // [rows, gate_stride] E or NULL
  int64_t gate_stride, out_stride;
  void* out;               // [rows, out_stride] E
  int true_vdim;
  float eps;
  // chunked forms over segments of `segment` tokens, at most `segments` per sequence (1: none)
  int segment, segments;
  float* seg_state;        // [sequences, segments, heads, dim, vdim]
  float* seg_decay;        // [sequences, segments, heads, dim]
  // decode step
  const int64_t *pos, *active;
  int lanes_per_row, overlap;
};

bool outer_rnn_chunk_supports(int dim, int vdim);
int outer_rnn_chunk_launch(const OuterRnnParams& p, RnnKind kind, int n, cudaStream_t st);   // FORGET, KEYED
void outer_rnn_fold_launch(const OuterRnnParams& p, int n, cudaStream_t st);
int outer_rnn_serial_launch(const OuterRnnParams& p, RnnKind kind, bool f32, int n, cudaStream_t st);
int outer_rnn_decode_launch(OuterRnnParams p, RnnKind kind, bool f32, int batch, const char* name, cudaStream_t st);

// softplus without a branch on the size of u; fp32 accuracy also where it is tiny
__device__ __forceinline__ float softplus_f(float u) { return fmaxf(u, 0.f) + log1pf(expf(-fabsf(u))); }

// sigmoid(z)^(1 / tau) = exp(-softplus(-z) / tau)
template <typename E>
__device__ __forceinline__ float sigmoid_root(float z, float inv_tau) {
  if constexpr (sizeof(E) == 4) return expf(-softplus_f(-z) * inv_tau);
  else return __expf(-(fmaxf(-z, 0.f) + __logf(1.0f + __expf(-fabsf(z)))) * inv_tau);
}

}  // namespace b200
