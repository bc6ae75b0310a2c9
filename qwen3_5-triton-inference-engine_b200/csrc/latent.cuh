// Shared declarations of the latent-attention kernels (latent.cu, latent_decode.cu, latent_prefill_umma.cu).
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

struct LatentDecodeParams {
  const void* q;         // [batch, heads, rank + rot] E
  const void* cache;     // [pages, PAGE, rank + rot] E
  const int32_t* table;
  int64_t table_stride;
  const int64_t *pos, *active;
  float2* ml;            // [batch, heads, splits] (row maximum, sum)
  float* o;              // [batch, heads, splits, rank]
  int heads, rank, rot, window, splits, overlap;
  float scale;
  int* err;
};

struct LatentAbsorbParams {
  const void *q, *w;     // [batch, heads, dim + rot], [heads, dim, rank]
  const int64_t* pos;
  const float2* angles;
  void* out;             // [batch, heads, rank + rot]
  int batch, heads, dim, rot, rot_pairs, rank, overlap;
};

struct LatentValueParams {
  const float2* ml;
  const float* o;
  const void* w;         // [heads, vdim, rank]
  void* merged;          // [batch, heads, rank] E
  void* out;             // [batch, heads, vdim]
  int batch, heads, rank, vdim, splits, overlap;
};

// Positions [lo, hi) of split `split` of slot b: the visible range (window, causal, the new token included) cut at page
// borders into `splits` nearly equal runs of pages.  Empty for an idle slot.
__device__ __forceinline__ void latent_split_range(const LatentDecodeParams& p, int b, int split, int& lo, int& hi) {
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

}  // namespace b200
