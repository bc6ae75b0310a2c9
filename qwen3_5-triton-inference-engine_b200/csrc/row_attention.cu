// Attention of one token per slot over paged rows (latent.cuh, RowDecodeParams): the CUDA-core form for any shape and
// element type, and the merge of the key ranges that both forms leave.  The tensor-core form is in latent_decode.cu.
#include "latent.cuh"

namespace b200 {

template <typename E>
__global__ void __launch_bounds__(128) row_decode_simple_kernel(const __grid_constant__ RowDecodeParams p) {
  __shared__ float ps[LS_TILE];
  const int split = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  int lo, hi;
  latent_split_range(p, b, split, lo, hi);
  const int64_t part = (static_cast<int64_t>(b) * p.heads + h) * p.splits + split;
  if (lo >= hi) {
    if (threadIdx.x == 0) p.ml[part] = make_float2(-INFINITY, 0.f);
    return;
  }
  const int g = h / p.group;
  const E* q = static_cast<const E*>(p.q) + b * p.q_stride + static_cast<int64_t>(h) * p.key;
  const E* cache = static_cast<const E*>(p.cache);
  const int32_t* table = p.table + b * p.table_stride;
  auto row = [&](int j) { return cache + ((static_cast<int64_t>(table[j / PAGE]) * p.kv_heads + g) * PAGE + j % PAGE) * p.pitch; };
  float m, l, acc[LS_MAX_COLS / 128];
  simple_attend(
      lo, hi, p.rank, p.scale,
      [&](int j, int lane) {
        const E* k = row(j);
        float s = 0.f;
        for (int c = lane; c < p.key; c += 32) s = fmaf(load1(q + c), load1(k + c), s);
        return s;
      },
      [&](int j, int c) { return load1(row(j) + p.v_off + c); }, ps, m, l, acc);
  if (threadIdx.x == 0) p.ml[part] = make_float2(m, l);
#pragma unroll
  for (int c = 0; c < LS_MAX_COLS / 128; ++c)
    if (threadIdx.x + c * 128 < p.rank) p.o[part * p.rank + threadIdx.x + c * 128] = acc[c];
}

// out[b, h, :] = sum_s w_s o_s with w_s = exp(m_s - m) / sum exp(m_s - m) l_s; an idle slot gives zeros.
// grid (heads, batch)
template <typename E>
__global__ void __launch_bounds__(128) row_merge_kernel(const __grid_constant__ RowMergeParams p) {
  __shared__ float weight[LATENT_MAX_SPLITS];
  const int64_t bh = static_cast<int64_t>(blockIdx.y) * p.heads + blockIdx.x;
  const int tid = threadIdx.x;
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  if (tid < 32) {
    constexpr int N = LATENT_MAX_SPLITS / 32;
    float2 a[N];
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      a[i] = tid + i * 32 < p.splits ? p.ml[bh * p.splits + tid + i * 32] : make_float2(-INFINITY, 0.f);
      m = fmaxf(m, a[i].x);
    }
    m = warp_max(m);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      a[i].x = a[i].y > 0.f ? expf(a[i].x - m) : 0.f;
      l += a[i].x * a[i].y;
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (tid + i * 32 < p.splits) weight[tid + i * 32] = a[i].x * inv;
  }
  __syncthreads();
  for (int c = tid * 4; c < p.rank; c += 512) {
    const float* o = p.o + bh * p.splits * p.rank + c;
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int U = 8;
    for (int s0 = 0; s0 < p.splits; s0 += U) {
      float4 v[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (s0 + u < p.splits) v[u] = load4(o + static_cast<int64_t>(s0 + u) * p.rank);
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (s0 + u < p.splits && weight[s0 + u] != 0.f) {  // an empty range left its part of the workspace unwritten
          const float w = weight[s0 + u];
          sum.x = fmaf(w, v[u].x, sum.x), sum.y = fmaf(w, v[u].y, sum.y);
          sum.z = fmaf(w, v[u].z, sum.z), sum.w = fmaf(w, v[u].w, sum.w);
        }
    }
    if (p.gate) {
      const float4 g = load4(static_cast<const E*>(p.gate) + blockIdx.y * p.gate_stride + blockIdx.x * p.rank + c);
      sum.x *= sigmoid_f<E>(g.x) * p.scale, sum.y *= sigmoid_f<E>(g.y) * p.scale;
      sum.z *= sigmoid_f<E>(g.z) * p.scale, sum.w *= sigmoid_f<E>(g.w) * p.scale;
    }
    store4(static_cast<E*>(p.out) + blockIdx.y * p.out_stride + blockIdx.x * p.rank + c, sum);
  }
}

int row_decode_simple_launch(const RowDecodeParams& p, int batch, bool f32, const char* name, cudaStream_t st) {
  B200_REQUIRE(p.rank > 0 && p.rank <= LS_MAX_COLS && p.window > 0 && p.splits > 0 && p.splits <= LATENT_MAX_SPLITS &&
                   p.heads <= 65535 && batch <= 65535,
               "%s: at most %d value columns and %d splits", name, LS_MAX_COLS, LATENT_MAX_SPLITS);
  const dim3 grid(p.splits, p.heads, batch);
  const bool early = (p.overlap & OVERLAP_START) != 0;
  const cudaError_t e = f32 ? launch_pdl(early, row_decode_simple_kernel<float>, grid, dim3(128), 0, st, p)
                            : launch_pdl(early, row_decode_simple_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, p);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "%s: %s", name, cudaGetErrorString(e));
  return check_launch(name);
}

int row_merge_launch(const RowMergeParams& p, int batch, bool f32, const char* name, cudaStream_t st) {
  B200_REQUIRE(p.rank > 0 && p.rank % 4 == 0 && p.gate_stride % 4 == 0 && p.out_stride % 4 == 0 && p.splits > 0 &&
                   p.splits <= LATENT_MAX_SPLITS && batch <= 65535,
               "%s: columns and strides must be multiples of 4, at most %d splits", name, LATENT_MAX_SPLITS);
  B200_REQUIRE(aligned16(p.o) && aligned16(p.out) && aligned16(p.gate), "%s: unaligned tensor", name);
  const dim3 grid(p.heads, batch);
  const bool early = (p.overlap & OVERLAP_START) != 0;
  const cudaError_t e = f32 ? launch_pdl(early, row_merge_kernel<float>, grid, dim3(128), 0, st, p)
                            : launch_pdl(early, row_merge_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, p);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "%s: %s", name, cudaGetErrorString(e));
  return check_launch(name);
}

}  // namespace b200
