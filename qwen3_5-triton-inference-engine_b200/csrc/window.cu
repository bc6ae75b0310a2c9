// Windowed attention with grouped query heads around its projections: biases, rotation of halves, paged rows [key | value] per
// key/value head, the gate on the heads' outputs.  Keys and values may have different sizes.
//   b200_window_prep      biases, rotation of q (in place) and k, rows to the pages and to the packed keys of a prefill
//   b200_window_prefill   packed portions: tcgen05 (latent_prefill_umma.cu), or CUDA cores for fp32 and wide heads (here)
//   b200_window_decode    one token per slot over the pages (latent_decode.cu, row_attention.cu)
//   b200_window_merge     merge of the key ranges, gate (row_attention.cu)
#include <type_traits>

#include "latent.cuh"

namespace b200 {

struct WindowPrepParams {
  void* x;                  // [rows, stride] E: [q | k | v | ...]
  int64_t stride;
  const float* bias;        // [q | k | v]
  const void* pos;
  int pos_is_int64;
  const int32_t* slot;
  const int64_t* active;
  const int32_t* table;
  int64_t table_stride;
  const float2* angles;     // [positions, pairs]
  void* cache;              // [pages, kv_heads, PAGE, pitch] E
  void* ctx;                // [keys, kv_heads, pitch] E or NULL
  const int32_t* ctx_row;
  int heads, kv_heads, dim, pairs, vdim, pitch, overlap;
};

template <typename E, int W>
__device__ __forceinline__ void load_w(const E* p, float (&f)[W]) {
  if constexpr (W == 8) load8(p, f);
  else f[0] = load1(p);
}
template <typename E>
struct Raw1 {
  E v;
  __device__ __forceinline__ void load(const E* p) { v = *p; }
  __device__ __forceinline__ void get(float (&f)[1]) const { f[0] = load1(&v); }
};
template <typename E, int W>
using RawW = std::conditional_t<W == 8, Raw8<E>, Raw1<E>>;
template <typename E, int W>
__device__ __forceinline__ void store_w(E* p, const float (&f)[W]) {
  if constexpr (W == 8) store8(p, f);
  else store1(p, f[0]);
}

// One CTA per ROWS rows.  An item is W consecutive elements that stay as they are, or W rotated pairs; W = 8 when the halves
// and what lies behind them start on groups of 8.  An item's biases are loaded once for all rows, and its elements of all rows
// before the first is used.
template <typename E, int W, int ROWS>
__global__ void __launch_bounds__(256) window_prep_kernel(const __grid_constant__ WindowPrepParams p, int rows) {
  __shared__ int64_t row_pos[ROWS], row_at[ROWS], row_ctx[ROWS];   // position; row of key/value head 0 in the cache (-1: none) and in ctx
  const int row0 = blockIdx.x * ROWS, count = min(ROWS, rows - row0);
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  E* const x0 = static_cast<E*>(p.x) + row0 * p.stride;
  E* const cache = static_cast<E*>(p.cache);
  E* const ctx = static_cast<E*>(p.ctx);
  const int n = p.pairs, ri = n / W, qi = ri + (p.dim - 2 * n) / W, vi = p.vdim / W;
  const int qk_items = (p.heads + p.kv_heads) * qi, total = qk_items + p.kv_heads * vi;
  bool first = true;
  for (int i = threadIdx.x; i < total || first; i += blockDim.x) {
    // source column, column in a cache row, key/value head (negative: a query), rotated or not
    int src = 0, dst = 0, g = 0;
    bool rotated = false;
    if (i < qk_items) {
      const int h = i / qi, j = i - h * qi;
      rotated = j < ri;
      dst = rotated ? j * W : 2 * n + (j - ri) * W;
      src = h * p.dim + dst;
      g = h - p.heads;
    } else if (i < total) {
      const int e = i - qk_items;
      g = e / vi;
      const int c = (e - g * vi) * W;
      src = (p.heads + p.kv_heads) * p.dim + g * p.vdim + c;
      dst = p.dim + c;
    }
    float bu[W], bv[W];
    RawW<E, W> ru[ROWS], rv[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const E* from = x0 + min(r, count - 1) * p.stride + src;
      ru[r].load(from);
      if (rotated) rv[r].load(from + n);
    }
    load_w<float, W>(p.bias + src, bu);
    if (rotated) load_w<float, W>(p.bias + src + n, bv);
    if (first) {                 // where the rows go, looked up while their elements are on the way
      first = false;
      if (threadIdx.x < count) {
        const int row = row0 + threadIdx.x, slot = p.slot ? p.slot[row] : row;
        const int64_t pos = p.pos_is_int64 ? static_cast<const int64_t*>(p.pos)[row] : static_cast<int64_t>(static_cast<const int32_t*>(p.pos)[row]);
        row_pos[threadIdx.x] = pos;
        row_at[threadIdx.x] = p.active && p.active[slot] == 0
                                  ? -1 : static_cast<int64_t>(p.table[slot * p.table_stride + pos / PAGE]) * p.kv_heads * PAGE + pos % PAGE;
        row_ctx[threadIdx.x] = p.ctx ? static_cast<int64_t>(p.ctx_row[row]) * p.kv_heads : 0;
      }
      __syncthreads();
      if (i >= total) break;
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      if (r >= count) break;
      float u[W], v[W];
      ru[r].get(u);
#pragma unroll
      for (int k = 0; k < W; ++k) u[k] += bu[k];
      if (rotated) {
        const float2* at = p.angles + row_pos[r] * n + dst;
        float a[2 * W];                      // (cos, sin) of the W pairs
        if constexpr (W == 8) {
#pragma unroll
          for (int k = 0; k < W / 2; ++k) reinterpret_cast<float4*>(a)[k] = reinterpret_cast<const float4*>(at)[k];
        } else {
          a[0] = at->x, a[1] = at->y;
        }
        rv[r].get(v);
#pragma unroll
        for (int k = 0; k < W; ++k) {
          v[k] += bv[k];
          rotate_pair(u[k], v[k], make_float2(a[2 * k], a[2 * k + 1]));
        }
      }
      auto put = [&](E* to) {
        store_w<E, W>(to, u);
        if (rotated) store_w<E, W>(to + n, v);
      };
      if (g < 0) {
        put(x0 + r * p.stride + src);
      } else {
        if (row_at[r] >= 0) put(cache + (row_at[r] + g * PAGE) * p.pitch + dst);
        if (ctx) put(ctx + (row_ctx[r] + g) * p.pitch + dst);
      }
    }
  }
}

struct WindowPrefillParams {
  const void *q, *ctx, *gate;
  int64_t q_stride, gate_stride, out_stride;
  void* out;
  const int32_t *cu_q, *cu_k, *q_pos0, *k_pos0;
  int kv_heads, group, dim, vdim, pitch, window;
  float scale, out_scale;
};

// any shape, fp32 arithmetic: one CTA per (query, head)
template <typename E>
__global__ void __launch_bounds__(128) window_prefill_simple_kernel(const __grid_constant__ WindowPrefillParams p) {
  __shared__ float ps[LS_TILE];
  const int seq = blockIdx.z, h = blockIdx.y, i = blockIdx.x;
  const int q0 = p.cu_q[seq], len = p.cu_q[seq + 1] - q0;
  if (i >= len) return;
  const int pos = p.q_pos0[seq] + i, lo = max(p.k_pos0[seq], pos - p.window + 1);
  const E* q = static_cast<const E*>(p.q) + (q0 + i) * p.q_stride + h * p.dim;
  // row of position 0 of this key/value head
  const E* keys = static_cast<const E*>(p.ctx) + (static_cast<int64_t>(p.cu_k[seq] - p.k_pos0[seq]) * p.kv_heads + h / p.group) * p.pitch;
  const int64_t step = static_cast<int64_t>(p.kv_heads) * p.pitch;
  float m, l, acc[LS_MAX_COLS / 128];
  simple_attend(
      lo, pos + 1, p.vdim, p.scale,
      [&](int j, int lane) {
        const E* k = keys + j * step;
        float s = 0.f;
        for (int c = lane; c < p.dim; c += 32) s = fmaf(load1(q + c), load1(k + c), s);
        return s;
      },
      [&](int j, int c) { return load1(keys + j * step + p.dim + c); }, ps, m, l, acc);
  E* out = static_cast<E*>(p.out) + (q0 + i) * p.out_stride + h * p.vdim;
  const E* gate = static_cast<const E*>(p.gate) + (q0 + i) * p.gate_stride + h * p.vdim;
#pragma unroll
  for (int c = 0; c < LS_MAX_COLS / 128; ++c) {
    const int col = threadIdx.x + c * 128;
    if (col < p.vdim) store1(out + col, acc[c] / l * (p.gate ? sigmoid_f<E>(load1(gate + col)) * p.out_scale : 1.f));
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_window_prep(void* x, int64_t stride, const float* bias, const void* pos, int32_t pos_is_int64,
                                const int32_t* slot, const int64_t* active, const int32_t* block_table, int64_t table_stride,
                                const float* angles, void* cache, void* ctx, const int32_t* ctx_row, int32_t rows,
                                int32_t heads, int32_t kv_heads, int32_t dim, int32_t rot_pairs, int32_t vdim, int32_t pitch,
                                int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && dim % 32 == 0 && vdim > 0 && vdim % 64 == 0 &&
                   pitch % 64 == 0 && pitch >= dim + vdim && rot_pairs >= 0 && 2 * rot_pairs <= dim && stride % 8 == 0,
               "window_prep: keys must be a multiple of 32, values and rows of 64, rotated pairs inside the keys");
  B200_REQUIRE(aligned16(x) && aligned16(bias) && aligned16(cache) && aligned16(ctx) && aligned16(angles) && (!ctx || ctx_row), "window_prep: unaligned tensor");
  const WindowPrepParams p = {x, stride, bias, pos, pos_is_int64, slot, active, block_table, table_stride,
                              reinterpret_cast<const float2*>(angles), cache, ctx, ctx_row, heads, kv_heads, dim, rot_pairs, vdim,
                              pitch, overlap};
  const int w = rot_pairs % 8 == 0 ? 8 : 1;
  const int items = ((heads + kv_heads) * (dim - rot_pairs) + kv_heads * vdim) / w;
  const dim3 block(items >= 256 ? 256 : (items + 31) / 32 * 32);
  const bool early = (overlap & OVERLAP_START) != 0;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (f32) e = w == 8 ? launch_pdl(early, window_prep_kernel<float, 8, 1>, dim3(rows), block, 0, st, p, rows)
                      : launch_pdl(early, window_prep_kernel<float, 1, 1>, dim3(rows), block, 0, st, p, rows);
  else if (w == 8 && rows >= GLUE_WIDE_ROWS) e = launch_pdl(early, window_prep_kernel<__nv_bfloat16, 8, 4>, dim3((rows + 3) / 4), block, 0, st, p, rows);
  else e = w == 8 ? launch_pdl(early, window_prep_kernel<__nv_bfloat16, 8, 1>, dim3(rows), block, 0, st, p, rows)
                  : launch_pdl(early, window_prep_kernel<__nv_bfloat16, 1, 1>, dim3(rows), block, 0, st, p, rows);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "window_prep: %s", cudaGetErrorString(e));
  return check_launch("window_prep");
}

extern "C" int b200_window_prefill(const void* q, int64_t q_stride, const void* ctx, const void* gate, int64_t gate_stride,
                                   void* out, int64_t out_stride, const int32_t* cu_q, const int32_t* cu_k,
                                   const int32_t* q_pos0, const int32_t* k_pos0, int32_t batch, int32_t max_q, int32_t tokens,
                                   int32_t keys, int32_t heads, int32_t kv_heads, int32_t dim, int32_t true_dim, int32_t vdim,
                                   int32_t pitch, int32_t window, float scale, float out_scale, int32_t simple, int32_t f32,
                                   b200_stream_t stream) {
  if (batch <= 0 || max_q <= 0) return OK;
  B200_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && dim % 32 == 0 && vdim > 0 && vdim % 64 == 0 &&
                   pitch % 64 == 0 && pitch >= dim + vdim && q_stride % 8 == 0,
               "window_prefill: keys must be a multiple of 32, values and rows of 64");
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (!f32 && !simple) {
    RowPrefillOperands a = {};
    const int64_t row = static_cast<int64_t>(kv_heads) * pitch;
    a.q = q, a.q_stride = q_stride;
    a.k = ctx, a.k_stride = row, a.k_head = pitch;
    a.v = static_cast<const __nv_bfloat16*>(ctx) + dim, a.v_stride = row, a.v_head = pitch;
    a.gate = gate, a.gate_stride = gate_stride, a.out = out, a.out_stride = out_stride;
    a.cu_q = cu_q, a.cu_k = cu_k, a.q_pos0 = q_pos0, a.k_pos0 = k_pos0;
    a.batch = batch, a.max_q = max_q, a.tokens = tokens, a.keys = keys, a.heads = heads, a.group = heads / kv_heads;
    a.dim = dim, a.true_dim = true_dim, a.vdim = vdim, a.window = window, a.scale = scale, a.out_scale = out_scale;
    return row_prefill_launch(a, "window_prefill", st);
  }
  B200_REQUIRE(vdim <= LS_MAX_COLS && heads <= 65535 && batch <= 65535 && window > 0,
               "window_prefill: values at most %d, heads and batch at most 65535, window positive", LS_MAX_COLS);
  const WindowPrefillParams p = {q, ctx, gate, q_stride, gate_stride, out_stride, out, cu_q, cu_k, q_pos0, k_pos0,
                                 kv_heads, heads / kv_heads, dim, vdim, pitch, window, scale, out_scale};
  const dim3 grid(max_q, heads, batch);
  if (f32) window_prefill_simple_kernel<float><<<grid, 128, 0, st>>>(p);
  else window_prefill_simple_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(p);
  return check_launch("window_prefill");
}

extern "C" int b200_window_decode(const void* q, int64_t q_stride, const void* cache, int64_t num_pages,
                                  const int32_t* block_table, int64_t table_stride, const int64_t* pos, const int64_t* active,
                                  float* ml, float* o, int32_t batch, int32_t heads, int32_t kv_heads, int32_t dim,
                                  int32_t vdim, int32_t pitch, int32_t window, int32_t splits, float scale, int32_t simple,
                                  int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 && pitch >= dim + vdim,
               "window_decode: heads must be a multiple of the key/value heads, rows must hold key and value");
  const RowDecodeParams p = {q, q_stride, cache, block_table, table_stride, pos, active, reinterpret_cast<float2*>(ml), o, heads,
                             kv_heads, heads / kv_heads, dim, dim, vdim, pitch, window, splits, overlap, scale, nullptr};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 || simple ? row_decode_simple_launch(p, batch, f32 != 0, "window_decode", st)
                       : row_decode_launch(p, num_pages, batch, "window_decode", st);
}

extern "C" int b200_window_merge(const float* ml, const float* o, const void* gate, int64_t gate_stride, void* out,
                                 int64_t out_stride, int32_t batch, int32_t heads, int32_t vdim, int32_t splits,
                                 float out_scale, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  const RowMergeParams p = {reinterpret_cast<const float2*>(ml), o, gate, gate_stride, out, out_stride, heads, vdim, splits, overlap, out_scale};
  return row_merge_launch(p, batch, f32 != 0, "window_merge", reinterpret_cast<cudaStream_t>(stream));
}
