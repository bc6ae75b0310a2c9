// Shared declarations of the attention kernels of hybrid stacks over paged rows: latent attention (latent.cu) and windowed
// attention with grouped heads (window.cu), on common tensor-core kernels (latent_decode.cu, latent_prefill_umma.cu).
#pragma once
#include "b200_attn.h"
#include "elem.cuh"

namespace b200 {

constexpr int LATENT_MAX_SPLITS = 64;

// (u, v) -> (u cos - v sin, v cos + u sin); a = (cos, sin), both already times the rotation's amplitude
__device__ __forceinline__ void rotate_pair(float& u, float& v, const float2& a) {
  const float r = __fmaf_rn(u, a.x, -__fmul_rn(v, a.y));
  v = __fmaf_rn(v, a.x, __fmul_rn(u, a.y));
  u = r;
}

struct LatentPrefillParams {
  const void* q;         // [tokens, heads, dim + rot] E, rotated
  const void* kv;        // [keys, heads*dim | heads*vdim] E: expanded keys and values
  const void* ctx;       // [keys, rank + rot] E: packed cache rows (the rotated part is read from here)
  void* out;             // [tokens, heads, vdim] E
  const int32_t *cu_q, *cu_k, *q_pos0, *k_pos0;
  int heads, dim, rot, vdim, rank, window;
  float scale;
};

// Decode attention over paged rows: a row serves `group` query heads; its first `key` elements score, the `rank` ones from
// v_off on are summed.  Latent attention: one row per token, key = the whole row, v_off = 0.  Grouped heads: a row
// [key | value] per key/value head.
struct RowDecodeParams {
  const void* q;         // [batch, q_stride] E: heads of `key` elements
  int64_t q_stride;
  const void* cache;     // [pages, kv_heads, PAGE, pitch] E
  const int32_t* table;
  int64_t table_stride;
  const int64_t *pos, *active;
  float2* ml;            // [batch, heads, splits] (row maximum, sum)
  float* o;              // [batch, heads, splits, rank]
  int heads, kv_heads, group, key, v_off, rank, pitch, window, splits, overlap;
  float scale;
  int* err;
};
int row_decode_launch(const RowDecodeParams& p, int64_t num_pages, int batch, const char* name, cudaStream_t st);
int row_decode_simple_launch(const RowDecodeParams& p, int batch, bool f32, const char* name, cudaStream_t st);

// Merge of the key ranges: out[b, h, :] = sum_s w_s o_s (* sigmoid(gate) * scale when a gate is given).
struct RowMergeParams {
  const float2* ml;
  const float* o;
  const void* gate;      // [batch, gate_stride] E or NULL
  int64_t gate_stride;
  void* out;             // [batch, out_stride] E
  int64_t out_stride;
  int heads, rank, splits, overlap;
  float scale;
};
int row_merge_launch(const RowMergeParams& p, int batch, bool f32, const char* name, cudaStream_t st);

// Prefill attention of packed portions on tcgen05 (latent_prefill_umma.cu): keys and values as strided matrices
struct RowPrefillOperands {
  const void *q, *k, *r, *v;          // r: the part of the keys that all heads share, or NULL
  int64_t q_stride, k_stride, k_head, r_stride, v_stride, v_head;   // elements: rows, and from one key/value head to the next
  const void* gate;                   // [tokens, gate_stride] or NULL
  int64_t gate_stride, out_stride;
  void* out;
  const int32_t *cu_q, *cu_k, *q_pos0, *k_pos0;
  int batch, max_q, tokens, keys, heads, group, dim, true_dim, rot, true_rot, vdim, window;
  float scale, out_scale;
};
int row_prefill_launch(const RowPrefillOperands& a, const char* name, cudaStream_t st);
// ... and its form for pairs of heads that share keys and values (window_pair_umma.cu)
bool row_prefill_pairs(const RowPrefillOperands& a);
int row_prefill_pair_launch(const RowPrefillOperands& a, const char* name, cudaStream_t st);

struct LatentAbsorbParams {
  const void *q, *w;     // [batch, heads, dim + rot], [heads, dim, rank]
  const int64_t* pos;
  const float2* angles;
  void* out;             // [batch, heads, rank + rot]
  int batch, heads, dim, rot, rot_pairs, rank, overlap;
};

struct LatentValueParams {
  const void* w;         // [heads, vdim, rank]
  void* merged;          // [batch, heads, rank] E
  void* out;             // [batch, heads, vdim]
  int batch, heads, rank, vdim, overlap;
};

// Positions [lo, hi) of split `split` of slot b: the visible range (window, causal, the new token included) cut at page
// borders into `splits` nearly equal runs of pages.  Empty for an idle slot.
__device__ __forceinline__ void latent_split_range(const RowDecodeParams& p, int b, int split, int& lo, int& hi) {
  lo = hi = 0;
  if (p.active && p.active[b] == 0) return;
  const int pos = static_cast<int>(p.pos[b]);
  const int first = max(0, pos - p.window + 1);
  const int page0 = first / PAGE, pages = pos / PAGE - page0 + 1;
  const int per = (pages + p.splits - 1) / p.splits;
  const int a = split * per;
  if (a >= pages) return;
  lo = max(first, (page0 + a) * PAGE);
  hi = min(pos + 1, (page0 + min(a + per, pages)) * PAGE);
}

// ------------------------------------------------------------------------------- attention on CUDA cores, any shape
constexpr int LS_TILE = 64;
constexpr int LS_MAX_COLS = 1024;  // value columns: 8 per thread

// One query row against keys [0, n): scores of a 64-key tile by warps, then every thread owns columns of the sum.
// key(j, c) / rkey(j, c) / val(j, c) return fp32 elements.
template <typename KeyDot, typename Val>
__device__ __forceinline__ void simple_attend(int j_lo, int j_hi, int cols, float scale, KeyDot dot, Val val, float* ps,
                                              float& m_out, float& l_out, float (&acc)[LS_MAX_COLS / 128]) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float m = -INFINITY, l = 0.f;
#pragma unroll
  for (int i = 0; i < LS_MAX_COLS / 128; ++i) acc[i] = 0.f;
  for (int j0 = j_lo; j0 < j_hi; j0 += LS_TILE) {
    const int n = min(LS_TILE, j_hi - j0);
    for (int j = warp; j < n; j += 4) {
      const float s = warp_sum(dot(j0 + j, lane)) * scale;
      if (lane == 0) ps[j] = s;
    }
    __syncthreads();
    float tile_max = -INFINITY;
    for (int j = lane; j < n; j += 32) tile_max = fmaxf(tile_max, ps[j]);
    tile_max = warp_max(tile_max);
    const float m_new = fmaxf(m, tile_max);
    const float alpha = expf(m - m_new);
    float part = 0.f;
    for (int j = lane; j < n; j += 32) part += expf(ps[j] - m_new);
    l = l * alpha + warp_sum(part);
    m = m_new;
#pragma unroll
    for (int i = 0; i < LS_MAX_COLS / 128; ++i) acc[i] *= alpha;
    for (int j = 0; j < n; ++j) {
      const float w = expf(ps[j] - m_new);
#pragma unroll
      for (int i = 0; i < LS_MAX_COLS / 128; ++i)
        if (tid + i * 128 < cols) acc[i] = fmaf(w, val(j0 + j, tid + i * 128), acc[i]);
    }
    __syncthreads();
  }
  m_out = m;
  l_out = l;
}

}  // namespace b200
