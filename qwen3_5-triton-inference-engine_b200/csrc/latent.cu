// Latent attention around its projections: a low-rank query, one cached latent c and one rotated key part per token that
// all heads share, per-head up-projections W_uk / W_uv, an optional sliding window.
//   b200_latent_prep       RMS norm of the query latent; RMS norm of the key/value latent and interleaved rotation of the
//                          shared key part, both written to the paged cache (rows [latent | rotated part])
//   b200_rope_interleaved  rotation of the queries' rotated part in place (prefill)
//   b200_latent_gather     cache rows of a range of positions per sequence into a packed buffer (prefill context)
//   b200_latent_prefill_simple   attention over expanded keys/values, any shape, bf16 or fp32 (CUDA cores)
//   b200_latent_absorb     decode: q' = [W_uk^T q_unrotated | rotated part], so that scores need the cache rows only
//   b200_latent_decode_simple    decode over the paged rows, split over key ranges, any shape (CUDA cores)
//   b200_latent_value      decode: merges the splits and applies W_uv
// The tensor-core forms live in latent_decode.cu and latent_prefill_umma.cu.
// Padded layout (the weight loader's): kv_rank, rot_dim, dim, vdim and q_rank are rounded up to multiples of 64 with
// zero rows / columns, a cache row is [latent | rotated part] with both parts padded.  Norms divide by the true widths.
// Scores, softmax, angles (a float64-made table of cos / sin) and norms are fp32.
#include "latent.cuh"

namespace b200 {

// ---------------------------------------------------------------------------------------------------------- prep
struct LatentPrepParams {
  const void* fused;        // [rows, stride] E: [query latent q_rank | kv latent rank | rotated part rot] (last two optional)
  int64_t stride;
  const float* q_weight;    // [q_rank]
  const float* kv_weight;   // [rank]
  const void* pos;          // int64 [slots] or int32 [rows]
  int pos_is_int64;
  const int32_t* slot;      // [rows] or NULL (row = slot)
  const int64_t* active;    // [slots] or NULL
  const int32_t* table;     // page table
  int64_t table_stride;
  const float2* angles;     // [positions, rot_pairs]
  void* cache;              // [pages, PAGE, rank + rot] E or NULL
  void* cq;                 // [rows, q_rank] E
  int q_rank, true_q_rank, rank, true_rank, rot, rot_pairs, overlap;
  float eps;
};

template <typename E>
__global__ void __launch_bounds__(128) latent_prep_kernel(const __grid_constant__ LatentPrepParams p) {
  __shared__ float red[64];
  const int row = blockIdx.x, tid = threadIdx.x;
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  const E* x = static_cast<const E*>(p.fused) + row * p.stride;
  const E* kv = x + p.q_rank;
  float sq[2] = {0.f, 0.f};
  for (int c = tid * 4; c < p.q_rank; c += 512) {
    const float4 v = load4(x + c);
    sq[0] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const bool own = p.cache != nullptr;
  if (own)
    for (int c = tid * 4; c < p.rank; c += 512) {
      const float4 v = load4(kv + c);
      sq[1] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  block_sum<2>(sq, red);
  const float qs = 1.0f / sqrtf(sq[0] / static_cast<float>(p.true_q_rank) + p.eps);
  E* cq = static_cast<E*>(p.cq) + static_cast<int64_t>(row) * p.q_rank;
  for (int c = tid * 4; c < p.q_rank; c += 512) {
    const float4 v = load4(x + c), w = load4(p.q_weight + c);
    store4(cq + c, make_float4(v.x * qs * w.x, v.y * qs * w.y, v.z * qs * w.z, v.w * qs * w.w));
  }
  if (!own) return;
  const int slot = p.slot ? p.slot[row] : row;
  if (p.active && p.active[slot] == 0) return;
  const int64_t pos = p.pos_is_int64 ? static_cast<const int64_t*>(p.pos)[row]
                                     : static_cast<int64_t>(static_cast<const int32_t*>(p.pos)[row]);
  const int64_t page = p.table[slot * p.table_stride + pos / PAGE];
  E* out = static_cast<E*>(p.cache) + (page * PAGE + pos % PAGE) * (p.rank + p.rot);
  const float ks = 1.0f / sqrtf(sq[1] / static_cast<float>(p.true_rank) + p.eps);
  for (int c = tid * 4; c < p.rank; c += 512) {
    const float4 v = load4(kv + c), w = load4(p.kv_weight + c);
    store4(out + c, make_float4(v.x * ks * w.x, v.y * ks * w.y, v.z * ks * w.z, v.w * ks * w.w));
  }
  const E* kr = kv + p.rank;
  for (int i = tid; i < p.rot / 2; i += 128) {
    float u = load1(kr + 2 * i), v = load1(kr + 2 * i + 1);
    if (i < p.rot_pairs) rotate_pair(u, v, p.angles[pos * p.rot_pairs + i]);
    store1(out + p.rank + 2 * i, u);
    store1(out + p.rank + 2 * i + 1, v);
  }
}

// ---------------------------------------------------------------------------------------------------------- rotation
// x [rows, heads, head_stride]: the pairs from offset `off` on
template <typename E>
__global__ void __launch_bounds__(256) rope_interleaved_kernel(E* x, int64_t row_stride, int head_stride, int off, int heads,
                                                               int pairs, const int32_t* pos, const float2* angles) {
  const int row = blockIdx.x;
  const float2* a = angles + static_cast<int64_t>(pos[row]) * pairs;
  for (int i = threadIdx.x; i < heads * pairs; i += 256) {
    const int h = i / pairs, j = i % pairs;
    E* q = x + row * row_stride + static_cast<int64_t>(h) * head_stride + off + 2 * j;
    float u = load1(q), v = load1(q + 1);
    rotate_pair(u, v, a[j]);
    store1(q, u);
    store1(q + 1, v);
  }
}

// ------------------------------------------------------------------------------------------------------------ gather
// out[cu_k[s] + i] = cache row of position k_pos0[s] + i of sequence s; grid (16-row groups, sequences)
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* cache, uint4* out, const int32_t* table,
                                                            int64_t table_stride, const int32_t* slots, const int32_t* cu_k,
                                                            const int32_t* k_pos0, int row_vecs) {
  const int seq = blockIdx.y, row0 = cu_k[seq], len = cu_k[seq + 1] - row0, base = k_pos0[seq];
  const int32_t* t = table + slots[seq] * table_stride;
  const int r_lo = blockIdx.x * 16, r_hi = min(r_lo + 16, len);
  for (int i = r_lo * row_vecs + threadIdx.x; i < r_hi * row_vecs; i += 256) {
    const int r = i / row_vecs, c = i % row_vecs, pos = base + r;
    out[static_cast<int64_t>(row0 + r) * row_vecs + c] =
        cache[(static_cast<int64_t>(t[pos / PAGE]) * PAGE + pos % PAGE) * row_vecs + c];
  }
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

template <typename E>
__global__ void __launch_bounds__(128) latent_prefill_simple_kernel(const __grid_constant__ LatentPrefillParams p) {
  __shared__ float ps[LS_TILE];
  const int seq = blockIdx.z, h = blockIdx.y, i = blockIdx.x;
  const int q0 = p.cu_q[seq], len = p.cu_q[seq + 1] - q0;
  if (i >= len) return;
  const int pos = p.q_pos0[seq] + i;
  const int k_row0 = p.cu_k[seq] - p.k_pos0[seq];  // packed row of position 0
  const int lo = max(p.k_pos0[seq], pos - p.window + 1);
  const E* q = static_cast<const E*>(p.q) + (static_cast<int64_t>(q0 + i) * p.heads + h) * (p.dim + p.rot);
  const E* kv = static_cast<const E*>(p.kv);
  const E* ctx = static_cast<const E*>(p.ctx);
  const int64_t kv_stride = static_cast<int64_t>(p.heads) * (p.dim + p.vdim);
  float m, l, acc[LS_MAX_COLS / 128];
  simple_attend(
      lo, pos + 1, p.vdim, p.scale,
      [&](int j, int lane) {
        const E* k = kv + (k_row0 + j) * kv_stride + static_cast<int64_t>(h) * p.dim;
        const E* kr = ctx + static_cast<int64_t>(k_row0 + j) * (p.rank + p.rot) + p.rank;
        float s = 0.f;
        for (int c = lane; c < p.dim; c += 32) s = fmaf(load1(q + c), load1(k + c), s);
        for (int c = lane; c < p.rot; c += 32) s = fmaf(load1(q + p.dim + c), load1(kr + c), s);
        return s;
      },
      [&](int j, int c) {
        return load1(kv + (k_row0 + j) * kv_stride + static_cast<int64_t>(p.heads) * p.dim + static_cast<int64_t>(h) * p.vdim + c);
      },
      ps, m, l, acc);
  E* out = static_cast<E*>(p.out) + (static_cast<int64_t>(q0 + i) * p.heads + h) * p.vdim;
#pragma unroll
  for (int c = 0; c < LS_MAX_COLS / 128; ++c)
    if (threadIdx.x + c * 128 < p.vdim) store1(out + threadIdx.x + c * 128, acc[c] / l);
}

template <typename E>
__global__ void __launch_bounds__(128) latent_decode_simple_kernel(const __grid_constant__ LatentDecodeParams p) {
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
  const int pitch = p.rank + p.rot;
  const E* q = static_cast<const E*>(p.q) + (static_cast<int64_t>(b) * p.heads + h) * pitch;
  const E* cache = static_cast<const E*>(p.cache);
  const int32_t* table = p.table + b * p.table_stride;
  auto row = [&](int j) { return cache + (static_cast<int64_t>(table[j / PAGE]) * PAGE + j % PAGE) * pitch; };
  float m, l, acc[LS_MAX_COLS / 128];
  simple_attend(
      lo, hi, p.rank, p.scale,
      [&](int j, int lane) {
        const E* k = row(j);
        float s = 0.f;
        for (int c = lane; c < pitch; c += 32) s = fmaf(load1(q + c), load1(k + c), s);
        return s;
      },
      [&](int j, int c) { return load1(row(j) + c); }, ps, m, l, acc);
  if (threadIdx.x == 0) p.ml[part] = make_float2(m, l);
#pragma unroll
  for (int c = 0; c < LS_MAX_COLS / 128; ++c)
    if (threadIdx.x + c * 128 < p.rank) p.o[part * p.rank + threadIdx.x + c * 128] = acc[c];
}

// ------------------------------------------------------------------------------------------------ decode: q' = W_uk^T q
// grid (heads, rank / 64, ceil(batch / 16)); 128 threads.  The CTAs of the first rank block also rotate.
template <typename E>
__device__ __forceinline__ void absorb_rotated_part(const LatentAbsorbParams& p, int h, int b0) {
  const int width = p.dim + p.rot, pitch = p.rank + p.rot;
  for (int i = threadIdx.x; i < 16 * (p.rot / 2); i += 128) {
    const int b = b0 + i / (p.rot / 2), j = i % (p.rot / 2);
    if (b >= p.batch) break;
    const E* q = static_cast<const E*>(p.q) + (static_cast<int64_t>(b) * p.heads + h) * width + p.dim + 2 * j;
    float u = load1(q), v = load1(q + 1);
    if (j < p.rot_pairs) rotate_pair(u, v, p.angles[p.pos[b] * p.rot_pairs + j]);
    E* o = static_cast<E*>(p.out) + (static_cast<int64_t>(b) * p.heads + h) * pitch + p.rank + 2 * j;
    store1(o, u);
    store1(o + 1, v);
  }
}

__global__ void __launch_bounds__(128) latent_absorb_f32_kernel(const __grid_constant__ LatentAbsorbParams p) {
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16;
  const int width = p.dim + p.rot, pitch = p.rank + p.rot;
  const float* w = static_cast<const float*>(p.w) + static_cast<int64_t>(h) * p.dim * p.rank + n0;
  for (int i = threadIdx.x; i < 16 * 64; i += 128) {
    const int b = b0 + i / 64, n = i % 64;
    if (b >= p.batch) break;
    const float* q = static_cast<const float*>(p.q) + (static_cast<int64_t>(b) * p.heads + h) * width;
    float s = 0.f;
    for (int k = 0; k < p.dim; ++k) s = fmaf(q[k], w[static_cast<int64_t>(k) * p.rank + n], s);
    static_cast<float*>(p.out)[(static_cast<int64_t>(b) * p.heads + h) * pitch + n0 + n] = s;
  }
  if (blockIdx.y == 0) absorb_rotated_part<float>(p, h, b0);
}

// bf16: one m16 tile of slots, W tile [64 k][64 n] at a time in shared memory, a warp per 16 columns
constexpr int LA_PITCH = 144;  // bytes of a 64-element row plus 16: ldmatrix rows fall into different banks
__global__ void __launch_bounds__(128) latent_absorb_bf16_kernel(const __grid_constant__ LatentAbsorbParams p) {
  __shared__ __align__(16) uint8_t ws[2][64 * LA_PITCH];
  __shared__ __align__(16) uint8_t qs[2][16 * LA_PITCH];
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int width = p.dim + p.rot, pitch = p.rank + p.rot, steps = p.dim / 64;
  const uint8_t* w = reinterpret_cast<const uint8_t*>(static_cast<const __nv_bfloat16*>(p.w) +
                                                      static_cast<int64_t>(h) * p.dim * p.rank + n0);
  uint4 wr[4];
  auto fetch_w = [&](int s) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (tid + i * 128) >> 3, c = tid & 7;
      wr[i] = *reinterpret_cast<const uint4*>(w + (static_cast<int64_t>(s * 64 + r) * p.rank + c * 8) * 2);
    }
  };
  fetch_w(0);  // a weight: may be read before the predecessor has finished
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  for (int s = 0; s < steps; ++s) {
    uint8_t *wb = ws[s & 1], *qb = qs[s & 1];
    {
      const int r = tid >> 3, c = tid & 7, b = b0 + r;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (b < p.batch)
        v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q) +
                                            (static_cast<int64_t>(b) * p.heads + h) * width + s * 64 + c * 8);
      *reinterpret_cast<uint4*>(qb + r * LA_PITCH + c * 16) = v;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) *reinterpret_cast<uint4*>(wb + ((tid + i * 128) >> 3) * LA_PITCH + (tid & 7) * 16) = wr[i];
    __syncthreads();  // two buffers: a warp may still read the other one
    if (s + 1 < steps) fetch_w(s + 1);
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[4], bm[4];
      ldmatrix_x4(a, smem_u32(qb) + (lane & 15) * LA_PITCH + ks * 32 + (lane >> 4) * 16);
      // k rows x n columns, transposed on the way in: matrices (k 0-7, n 0-7), (k 8-15, n 0-7), (k 0-7, n 8-15), ...
      ldmatrix_x4_trans(bm, smem_u32(wb) + (ks * 16 + (lane & 15)) * LA_PITCH + warp * 32 + (lane >> 4) * 16);
      mma_bf16_16816(acc[0], a, bm[0], bm[1]);
      mma_bf16_16816(acc[1], a, bm[2], bm[3]);
    }
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int b = b0 + (lane >> 2) + half * 8;
      if (b < p.batch)
        *reinterpret_cast<uint32_t*>(out + (static_cast<int64_t>(b) * p.heads + h) * pitch + n0 + warp * 16 + t * 8 + (lane & 3) * 2) =
            pack_bf16(acc[t][half * 2], acc[t][half * 2 + 1]);
    }
  if (blockIdx.y == 0) absorb_rotated_part<__nv_bfloat16>(p, h, b0);
}

// --------------------------------------------------------------------------------------- decode: merge splits, W_uv
// grid (heads, vdim / 64, ceil(batch / 16)).  Merged latents of up to 16 slots go to shared memory (E), then W_uv.
template <typename E>
__global__ void __launch_bounds__(128) latent_value_kernel(const __grid_constant__ LatentValueParams p) {
  extern __shared__ __align__(16) uint8_t lv_smem[];
  __shared__ float weight[16][LATENT_MAX_SPLITS];
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pitch = p.rank * static_cast<int>(sizeof(E)) + 16;  // bytes of a merged row
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  for (int r = warp; r < 16; r += 4) {
    const int b = b0 + r;
    float m = -INFINITY;
    const float2* ml = p.ml + (static_cast<int64_t>(b) * p.heads + h) * p.splits;
    if (b < p.batch)
      for (int s = lane; s < p.splits; s += 32) m = fmaxf(m, ml[s].x);
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < p.splits; s += 32) {
      const float2 a = b < p.batch ? ml[s] : make_float2(-INFINITY, 0.f);
      const float e = a.y > 0.f ? expf(a.x - m) : 0.f;
      weight[r][s] = e;
      l += e * a.y;
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    for (int s = lane; s < p.splits; s += 32) weight[r][s] *= inv;
  }
  __syncthreads();
  const int quads = p.rank / 4;
  for (int i = tid; i < 16 * quads; i += 128) {
    const int r = i / quads, c = (i % quads) * 4, b = b0 + r;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (b < p.batch) {
      const float* o = p.o + ((static_cast<int64_t>(b) * p.heads + h) * p.splits) * p.rank + c;
#pragma unroll 4
      for (int s = 0; s < p.splits; ++s) {
        const float w = weight[r][s];
        if (w != 0.f) {
          const float4 v = load4(o + static_cast<int64_t>(s) * p.rank);
          a.x = fmaf(w, v.x, a.x), a.y = fmaf(w, v.y, a.y), a.z = fmaf(w, v.z, a.z), a.w = fmaf(w, v.w, a.w);
        }
      }
    }
    store4(reinterpret_cast<E*>(lv_smem + r * pitch) + c, a);
  }
  __syncthreads();
  const E* w = static_cast<const E*>(p.w) + (static_cast<int64_t>(h) * p.vdim + n0) * p.rank;
  E* out = static_cast<E*>(p.out);
  if constexpr (sizeof(E) == 2) {
    // a warp per 16 value columns; the B operand comes straight from W_uv rows (K contiguous): lane (n = lane / 4,
    // k pair = lane % 4) loads its own 32-bit words
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const uint32_t* w0 = reinterpret_cast<const uint32_t*>(w + static_cast<int64_t>(warp * 16 + (lane >> 2)) * p.rank) + (lane & 3);
    const uint32_t* w1 = w0 + static_cast<int64_t>(8) * p.rank / 2;
#pragma unroll 8
    for (int ks = 0; ks < p.rank / 16; ++ks) {
      uint32_t a[4];
      ldmatrix_x4(a, smem_u32(lv_smem) + (lane & 15) * pitch + ks * 32 + (lane >> 4) * 16);
      mma_bf16_16816(acc[0], a, w0[ks * 8], w0[ks * 8 + 4]);
      mma_bf16_16816(acc[1], a, w1[ks * 8], w1[ks * 8 + 4]);
    }
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int b = b0 + (lane >> 2) + half * 8;
        if (b < p.batch)
          *reinterpret_cast<uint32_t*>(out + (static_cast<int64_t>(b) * p.heads + h) * p.vdim + n0 + warp * 16 + t * 8 + (lane & 3) * 2) =
              pack_bf16(acc[t][half * 2], acc[t][half * 2 + 1]);
      }
  } else {
    for (int i = tid; i < 16 * 64; i += 128) {
      const int r = i / 64, n = i % 64, b = b0 + r;
      if (b >= p.batch) break;
      const float* x = reinterpret_cast<const float*>(lv_smem + r * pitch);
      float s = 0.f;
      for (int k = 0; k < p.rank; ++k) s = fmaf(x[k], w[static_cast<int64_t>(n) * p.rank + k], s);
      out[(static_cast<int64_t>(b) * p.heads + h) * p.vdim + n0 + n] = s;
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_prep(const void* fused, int64_t stride, const float* q_weight, const float* kv_weight,
                                const void* pos, int32_t pos_is_int64, const int32_t* slot, const int64_t* active,
                                const int32_t* block_table, int64_t table_stride, const float* angles, void* cache, void* cq,
                                int32_t rows, int32_t q_rank, int32_t true_q_rank, int32_t rank, int32_t true_rank,
                                int32_t rot, int32_t rot_pairs, float eps, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(q_rank > 0 && q_rank % 4 == 0 && rank % 4 == 0 && rot % 2 == 0 && stride % 4 == 0 && rot_pairs * 2 <= rot,
               "latent_prep: widths must be multiples of 4 and cover the rotated pairs");
  B200_REQUIRE(aligned16(fused) && aligned16(cq) && aligned16(cache), "latent_prep: unaligned tensor");
  LatentPrepParams p = {fused, stride, q_weight, kv_weight, pos, pos_is_int64, slot, active, block_table, table_stride,
                        reinterpret_cast<const float2*>(angles), cache, cq, q_rank, true_q_rank, rank, true_rank, rot,
                        rot_pairs, overlap, eps};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool early = (overlap & OVERLAP_START) != 0;
  const cudaError_t e = f32 ? launch_pdl(early, latent_prep_kernel<float>, dim3(rows), dim3(128), 0, st, p)
                            : launch_pdl(early, latent_prep_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, st, p);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_prep: %s", cudaGetErrorString(e));
  return check_launch("latent_prep");
}

extern "C" int b200_rope_interleaved(void* x, int64_t row_stride, int32_t head_stride, int32_t offset, int32_t heads,
                                     int32_t pairs, const int32_t* pos, const float* angles, int32_t rows, int32_t f32,
                                     b200_stream_t stream) {
  if (rows <= 0 || pairs <= 0) return OK;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32)
    rope_interleaved_kernel<float><<<rows, 256, 0, st>>>(static_cast<float*>(x), row_stride, head_stride, offset, heads, pairs,
                                                         pos, reinterpret_cast<const float2*>(angles));
  else
    rope_interleaved_kernel<__nv_bfloat16><<<rows, 256, 0, st>>>(static_cast<__nv_bfloat16*>(x), row_stride, head_stride, offset,
                                                                 heads, pairs, pos, reinterpret_cast<const float2*>(angles));
  return check_launch("rope_interleaved");
}

extern "C" int b200_latent_gather(const void* cache, void* out, const int32_t* block_table, int64_t table_stride,
                                  const int32_t* slots, const int32_t* cu_k, const int32_t* k_pos0, int32_t batch,
                                  int32_t max_keys, int32_t row_bytes, b200_stream_t stream) {
  if (batch <= 0 || max_keys <= 0) return OK;
  B200_REQUIRE(row_bytes % 16 == 0 && aligned16(cache) && aligned16(out) && batch <= 65535, "latent_gather: unaligned rows");
  latent_gather_kernel<<<dim3((max_keys + 15) / 16, batch), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), static_cast<uint4*>(out), block_table, table_stride, slots, cu_k, k_pos0, row_bytes / 16);
  return check_launch("latent_gather");
}

extern "C" int b200_latent_prefill_simple(const void* q, const void* kv, const void* ctx, void* out, const int32_t* cu_q,
                                          const int32_t* cu_k, const int32_t* q_pos0, const int32_t* k_pos0, int32_t batch,
                                          int32_t max_q, int32_t heads, int32_t dim, int32_t rot, int32_t vdim, int32_t rank,
                                          int32_t window, float scale, int32_t f32, b200_stream_t stream) {
  if (batch <= 0 || max_q <= 0) return OK;
  B200_REQUIRE(vdim > 0 && vdim <= LS_MAX_COLS && heads > 0 && heads <= 65535 && batch <= 65535 && window > 0,
               "latent_prefill_simple: vdim at most %d, heads and batch at most 65535, window positive", LS_MAX_COLS);
  LatentPrefillParams p = {q, kv, ctx, out, cu_q, cu_k, q_pos0, k_pos0, heads, dim, rot, vdim, rank, window, scale};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(max_q, heads, batch);
  if (f32) latent_prefill_simple_kernel<float><<<grid, 128, 0, st>>>(p);
  else latent_prefill_simple_kernel<__nv_bfloat16><<<grid, 128, 0, st>>>(p);
  return check_launch("latent_prefill_simple");
}

extern "C" int b200_latent_absorb(const void* q, const void* w_uk, const int64_t* pos, const float* angles, void* out,
                                  int32_t batch, int32_t heads, int32_t dim, int32_t rot, int32_t rot_pairs, int32_t rank,
                                  int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(dim % 64 == 0 && rank % 64 == 0 && rot % 2 == 0 && rot_pairs * 2 <= rot && (batch + 15) / 16 <= 65535,
               "latent_absorb: dim and rank must be multiples of 64");
  B200_REQUIRE(aligned16(q) && aligned16(w_uk) && aligned16(out), "latent_absorb: unaligned tensor");
  LatentAbsorbParams p = {q, w_uk, pos, reinterpret_cast<const float2*>(angles), out, batch, heads, dim, rot, rot_pairs, rank, overlap};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(heads, rank / 64, (batch + 15) / 16);
  if (f32) latent_absorb_f32_kernel<<<grid, 128, 0, st>>>(p);
  else {
    const cudaError_t e = launch_pdl((overlap & OVERLAP_START) != 0, latent_absorb_bf16_kernel, grid, dim3(128), 0, st, p);
    if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_absorb: %s", cudaGetErrorString(e));
  }
  return check_launch("latent_absorb");
}

extern "C" int b200_latent_decode_simple(const void* q, const void* cache, const int32_t* block_table, int64_t table_stride,
                                         const int64_t* pos, const int64_t* active, float* ml, float* o, int32_t batch,
                                         int32_t heads, int32_t rank, int32_t rot, int32_t window, int32_t splits, float scale,
                                         int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(rank > 0 && rank <= LS_MAX_COLS && window > 0 && splits > 0 && splits <= LATENT_MAX_SPLITS && heads <= 65535 &&
                   batch <= 65535,
               "latent_decode_simple: rank at most %d, splits at most %d", LS_MAX_COLS, LATENT_MAX_SPLITS);
  LatentDecodeParams p = {q, cache, block_table, table_stride, pos, active, reinterpret_cast<float2*>(ml), o,
                          heads, rank, rot, window, splits, overlap, scale, nullptr};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(splits, heads, batch);
  const bool early = (overlap & OVERLAP_START) != 0;
  const cudaError_t e = f32 ? launch_pdl(early, latent_decode_simple_kernel<float>, grid, dim3(128), 0, st, p)
                            : launch_pdl(early, latent_decode_simple_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, p);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_decode_simple: %s", cudaGetErrorString(e));
  return check_launch("latent_decode_simple");
}

extern "C" int b200_latent_value(const float* ml, const float* o, const void* w_uv, void* out, int32_t batch, int32_t heads,
                                 int32_t rank, int32_t vdim, int32_t splits, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(rank % 64 == 0 && rank <= LS_MAX_COLS && vdim % 64 == 0 && splits > 0 && splits <= LATENT_MAX_SPLITS,
               "latent_value: rank and vdim must be multiples of 64, rank at most %d, splits at most %d", LS_MAX_COLS,
               LATENT_MAX_SPLITS);
  LatentValueParams p = {reinterpret_cast<const float2*>(ml), o, w_uv, out, batch, heads, rank, vdim, splits, overlap};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(heads, vdim / 64, (batch + 15) / 16);
  const int smem = 16 * (rank * (f32 ? 4 : 2) + 16);
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    constexpr int most = 16 * (LS_MAX_COLS * 4 + 16);
    if (cudaFuncSetAttribute(latent_value_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess ||
        cudaFuncSetAttribute(latent_value_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess)
      return fail(ERR_RUNTIME, "latent_value: cannot raise dynamic shared memory");
    configured[dev] = true;
  }
  const bool early = (overlap & OVERLAP_START) != 0;
  const cudaError_t e = f32 ? launch_pdl(early, latent_value_kernel<float>, grid, dim3(128), smem, st, p)
                            : launch_pdl(early, latent_value_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, p);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_value: %s", cudaGetErrorString(e));
  return check_launch("latent_value");
}
