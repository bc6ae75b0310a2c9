// Latent attention around its projections: a low-rank query, one cached latent c and one rotated key part per token that
// all heads share, per-head up-projections W_uk / W_uv, an optional sliding window.
//   b200_latent_prep       RMS norm of the query latent; RMS norm of the key/value latent and interleaved rotation of the
//                          shared key part, both written to the paged cache (rows [latent | rotated part])
//   b200_rope_interleaved  rotation of the queries' rotated part in place (prefill)
//   b200_latent_gather     cache rows of a range of positions per sequence into a packed buffer (prefill context)
//   b200_latent_prefill_simple   attention over expanded keys/values, any shape, bf16 or fp32 (CUDA cores)
//   b200_latent_absorb     decode: q' = [W_uk^T q_unrotated | rotated part], so that scores need the cache rows only
//   b200_latent_decode_simple    decode over the paged rows, split over key ranges, any shape (row_attention.cu)
//   b200_latent_value      decode: merges the splits (row_attention.cu), then applies W_uv (two launches)
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

// One CTA per row; a thread holds up to V groups of 8 elements of the row [query latent | kv latent | rotated part] in
// registers: one pass over memory, one block reduction for both norms.
template <typename E, int V>
__global__ void __launch_bounds__(256) latent_prep_kernel(const __grid_constant__ LatentPrepParams p) {
  __shared__ float red[64];
  const int row = blockIdx.x, tid = threadIdx.x;
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  const E* x = static_cast<const E*>(p.fused) + row * p.stride;
  const bool own = p.cache != nullptr;
  const int nq = p.q_rank / 8, nk = nq + p.rank / 8, total = own ? nk + p.rot / 8 : nq;
  float f[V][8], sq[2] = {0.f, 0.f};
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = tid + v * blockDim.x;
    if (i < total) load8(x + i * 8, f[v]);
    if (i < nk && i < total) {
      float part = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) part = fmaf(f[v][j], f[v][j], part);
      sq[i < nq ? 0 : 1] += part;
    }
  }
  const int slot = own && p.slot ? p.slot[row] : row;
  const bool write = own && !(p.active && p.active[slot] == 0);
  int64_t pos = 0;
  E* out = nullptr;
  if (write) {
    pos = p.pos_is_int64 ? static_cast<const int64_t*>(p.pos)[row] : static_cast<int64_t>(static_cast<const int32_t*>(p.pos)[row]);
    const int64_t page = p.table[slot * p.table_stride + pos / PAGE];
    out = static_cast<E*>(p.cache) + (page * PAGE + pos % PAGE) * (p.rank + p.rot);
  }
  block_sum<2>(sq, red);
  const float qs = 1.0f / sqrtf(sq[0] / static_cast<float>(p.true_q_rank) + p.eps);
  const float ks = 1.0f / sqrtf(sq[1] / static_cast<float>(p.true_rank) + p.eps);
  E* cq = static_cast<E*>(p.cq) + static_cast<int64_t>(row) * p.q_rank;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = tid + v * blockDim.x;
    if (i < nq) {
      float w[8];
      load8(p.q_weight + i * 8, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[v][j] *= qs * w[j];
      store8(cq + i * 8, f[v]);
    } else if (i < total && write) {
      if (i < nk) {
        float w[8];
        load8(p.kv_weight + (i - nq) * 8, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[v][j] *= ks * w[j];
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int pair = (i - nk) * 4 + j;
          if (pair < p.rot_pairs) rotate_pair(f[v][2 * j], f[v][2 * j + 1], p.angles[pos * p.rot_pairs + pair]);
        }
      }
      store8(out + (i - nq) * 8, f[v]);
    }
  }
}

// Prompt-sized batches: one warp per row, eight rows per CTA, no block barrier; the same arithmetic.
template <typename E, int V>
__global__ void __launch_bounds__(256) latent_prep_rows_kernel(const __grid_constant__ LatentPrepParams p, int rows) {
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const E* x = static_cast<const E*>(p.fused) + row * p.stride;
  const bool own = p.cache != nullptr;
  const int nq = p.q_rank / 8, nk = nq + p.rank / 8, total = own ? nk + p.rot / 8 : nq;
  const int slot = own && p.slot ? p.slot[row] : row;
  const int64_t pos = !own ? 0 : p.pos_is_int64 ? static_cast<const int64_t*>(p.pos)[row]
                                                : static_cast<int64_t>(static_cast<const int32_t*>(p.pos)[row]);
  uint4 raw[V][sizeof(E) / 2];
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = lane + v * 32;
    if (i < total) {
#pragma unroll
      for (int k = 0; k < static_cast<int>(sizeof(E) / 2); ++k) raw[v][k] = reinterpret_cast<const uint4*>(x + i * 8)[k];
    }
  }
  const bool write = own && !(p.active && p.active[slot] == 0);
  E* out = nullptr;
  if (write) out = static_cast<E*>(p.cache) + (static_cast<int64_t>(p.table[slot * p.table_stride + pos / PAGE]) * PAGE + pos % PAGE) * (p.rank + p.rot);
  auto unpack = [&](int v, float (&f)[8]) { load8(reinterpret_cast<const E*>(&raw[v][0]), f); };
  float sq0 = 0.f, sq1 = 0.f;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = lane + v * 32;
    if (i < nk && i < total) {
      float f[8], part = 0.f;
      unpack(v, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) part = fmaf(f[j], f[j], part);
      if (i < nq) sq0 += part;
      else sq1 += part;
    }
  }
  const float qs = 1.0f / sqrtf(warp_sum(sq0) / static_cast<float>(p.true_q_rank) + p.eps);
  const float ks = 1.0f / sqrtf(warp_sum(sq1) / static_cast<float>(p.true_rank) + p.eps);
  E* cq = static_cast<E*>(p.cq) + static_cast<int64_t>(row) * p.q_rank;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int i = lane + v * 32;
    if (i >= total || (i >= nq && !write)) continue;
    float f[8], w[8];
    unpack(v, f);
    if (i < nk) {
      const float s = i < nq ? qs : ks;
      load8(i < nq ? p.q_weight + i * 8 : p.kv_weight + (i - nq) * 8, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= s * w[j];
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int pair = (i - nk) * 4 + j;
        if (pair < p.rot_pairs) rotate_pair(f[2 * j], f[2 * j + 1], p.angles[pos * p.rot_pairs + pair]);
      }
    }
    store8(i < nq ? cq + i * 8 : out + (i - nq) * 8, f);
  }
}

// ---------------------------------------------------------------------------------------------------------- rotation
// x [rows, heads, head_stride]: the pairs from offset `off` on, four per thread; the parts are padded to multiples of 8
template <typename E>
__global__ void __launch_bounds__(256) rope_interleaved_kernel(E* x, int64_t row_stride, int head_stride, int off, int heads,
                                                               int pairs, const int32_t* pos, const float2* angles, int rows) {
  const int quads = (pairs + 3) / 4, per_row = heads * quads;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  const int64_t row = i / per_row;
  if (row >= rows) return;
  const int r = static_cast<int>(i - row * per_row), h = r / quads, j = (r - h * quads) * 4;
  E* q = x + row * row_stride + static_cast<int64_t>(h) * head_stride + off + 2 * j;
  const float2* a = angles + static_cast<int64_t>(pos[row]) * pairs + j;
  float f[8];
  load8(q, f);
#pragma unroll
  for (int k = 0; k < 4; ++k)
    if (j + k < pairs) rotate_pair(f[2 * k], f[2 * k + 1], a[k]);
  store8(q, f);
}

// ------------------------------------------------------------------------------------------------------------ gather
// out[cu_k[s] + i] = cache rows (one per key/value head) of position k_pos0[s] + i of sequence s; grid (16-row groups,
// sequences)
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* cache, uint4* out, const int32_t* table,
                                                            int64_t table_stride, const int32_t* slots, const int32_t* cu_k,
                                                            const int32_t* k_pos0, int kv_heads, int row_vecs) {
  const int seq = blockIdx.y, row0 = cu_k[seq], len = cu_k[seq + 1] - row0, base = k_pos0[seq];
  const int32_t* t = table + slots[seq] * table_stride;
  const int r_lo = blockIdx.x * 16, r_hi = min(r_lo + 16, len);
  const int token_vecs = kv_heads * row_vecs;
  for (int i = r_lo * token_vecs + threadIdx.x; i < r_hi * token_vecs; i += 256) {
    const int r = i / token_vecs, gc = i - r * token_vecs, g = gc / row_vecs, pos = base + r;
    out[static_cast<int64_t>(row0 + r) * token_vecs + gc] =
        cache[((static_cast<int64_t>(t[pos / PAGE]) * kv_heads + g) * PAGE + pos % PAGE) * row_vecs + gc - g * row_vecs];
  }
}

// ------------------------------------------------------------------------------- attention on CUDA cores, any shape
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

// bf16 products of up to 16 slots with a head's own matrix: out[b, h, n] = sum_k x[b, h, k] W_h[k, n], a CTA per
// (head, 64 columns, 16 slots), a warp per 16 columns.  The whole [K x 64] slice of W is requested at once (cp.async,
// before the predecessor has finished), the slots' rows after it: one memory round trip.
// K_ROWS: W_h is stored [K, N] (absorb), else [N, K] (value).
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
constexpr int HG_PITCH = 144;                              // bytes of a 64-element row plus 16
constexpr int HG_STEP = (64 + 16) * HG_PITCH;              // bytes of one 64-wide step of K: W tile, then the slots' tile

template <bool K_ROWS>
__device__ __forceinline__ void head_gemm(const __nv_bfloat16* w, int ldw, const __nv_bfloat16* x, int64_t x_stride, int slots,
                                          int steps, int n0, bool trigger, uint8_t* smem, float (&acc)[2][4]) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int s = 0; s < steps; ++s)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (tid + i * 128) >> 3, c = tid & 7;
      const __nv_bfloat16* src = K_ROWS ? w + static_cast<int64_t>(s * 64 + r) * ldw + n0 + c * 8
                                        : w + static_cast<int64_t>(n0 + r) * ldw + s * 64 + c * 8;
      cp_async16(smem + s * HG_STEP + r * HG_PITCH + c * 16, src);
    }
  if (trigger) pdl_trigger();
  pdl_wait();
  for (int s = 0; s < steps; ++s) {
    const int r = tid >> 3, c = tid & 7;
    uint8_t* dst = smem + s * HG_STEP + (64 + r) * HG_PITCH + c * 16;
    if (r < slots) cp_async16(dst, x + r * x_stride + s * 64 + c * 8);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  for (int s = 0; s < steps; ++s) {
    const uint32_t wb = smem_u32(smem + s * HG_STEP), xb = wb + 64 * HG_PITCH;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t a[4], bm[4];
      ldmatrix_x4(a, xb + (lane & 15) * HG_PITCH + ks * 32 + (lane >> 4) * 16);
      // matrices (k 0-7, n 0-7), (k 8-15, n 0-7), (k 0-7, n 8-15), (k 8-15, n 8-15)
      if (K_ROWS) ldmatrix_x4_trans(bm, wb + (ks * 16 + (lane & 15)) * HG_PITCH + warp * 32 + (lane >> 4) * 16);
      else ldmatrix_x4(bm, wb + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * HG_PITCH + ks * 32 + ((lane >> 3) & 1) * 16);
      mma_bf16_16816(acc[0], a, bm[0], bm[1]);
      mma_bf16_16816(acc[1], a, bm[2], bm[3]);
    }
  }
}
__device__ __forceinline__ void head_gemm_store(const float (&acc)[2][4], __nv_bfloat16* out, int64_t stride, int slots) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = (lane >> 2) + half * 8;
      if (r < slots)
        *reinterpret_cast<uint32_t*>(out + r * stride + warp * 16 + t * 8 + (lane & 3) * 2) = pack_bf16(acc[t][half * 2], acc[t][half * 2 + 1]);
    }
}

__global__ void __launch_bounds__(128) latent_absorb_bf16_kernel(const __grid_constant__ LatentAbsorbParams p) {
  extern __shared__ __align__(16) uint8_t hg_smem[];
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16, slots = min(16, p.batch - b0);
  const int width = p.dim + p.rot, pitch = p.rank + p.rot;
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  head_gemm<true>(static_cast<const __nv_bfloat16*>(p.w) + static_cast<int64_t>(h) * p.dim * p.rank, p.rank,
                  static_cast<const __nv_bfloat16*>(p.q) + (static_cast<int64_t>(b0) * p.heads + h) * width,
                  static_cast<int64_t>(p.heads) * width, slots, p.dim / 64, n0, (p.overlap & OVERLAP_TRIGGER) != 0, hg_smem, acc);
  head_gemm_store(acc, static_cast<__nv_bfloat16*>(p.out) + (static_cast<int64_t>(b0) * p.heads + h) * pitch + n0,
                  static_cast<int64_t>(p.heads) * pitch, slots);
  if (blockIdx.y == 0) absorb_rotated_part<__nv_bfloat16>(p, h, b0);
}

// --------------------------------------------------------------------------------------- decode: merge splits, W_uv
__global__ void __launch_bounds__(128) latent_value_bf16_kernel(const __grid_constant__ LatentValueParams p) {
  extern __shared__ __align__(16) uint8_t hg_smem[];
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16, slots = min(16, p.batch - b0);
  float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
  head_gemm<false>(static_cast<const __nv_bfloat16*>(p.w) + static_cast<int64_t>(h) * p.vdim * p.rank, p.rank,
                   static_cast<const __nv_bfloat16*>(p.merged) + (static_cast<int64_t>(b0) * p.heads + h) * p.rank,
                   static_cast<int64_t>(p.heads) * p.rank, slots, p.rank / 64, n0, (p.overlap & OVERLAP_TRIGGER) != 0, hg_smem, acc);
  head_gemm_store(acc, static_cast<__nv_bfloat16*>(p.out) + (static_cast<int64_t>(b0) * p.heads + h) * p.vdim + n0,
                  static_cast<int64_t>(p.heads) * p.vdim, slots);
}
__global__ void __launch_bounds__(128) latent_value_f32_kernel(const __grid_constant__ LatentValueParams p) {
  const int h = blockIdx.x, n0 = blockIdx.y * 64, b0 = blockIdx.z * 16;
  for (int i = threadIdx.x; i < 16 * 64; i += 128) {
    const int b = b0 + i / 64, n = n0 + i % 64;
    if (b >= p.batch) break;
    const float* x = static_cast<const float*>(p.merged) + (static_cast<int64_t>(b) * p.heads + h) * p.rank;
    const float* w = static_cast<const float*>(p.w) + (static_cast<int64_t>(h) * p.vdim + n) * p.rank;
    float s = 0.f;
    for (int k = 0; k < p.rank; ++k) s = fmaf(x[k], w[k], s);
    static_cast<float*>(p.out)[(static_cast<int64_t>(b) * p.heads + h) * p.vdim + n] = s;
  }
}

static bool head_gemm_configure(const void* kernel, int which) {
  static bool configured[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64 || configured[which][dev]) return true;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 16 * HG_STEP) != cudaSuccess) return false;
  configured[which][dev] = true;
  return true;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_prep(const void* fused, int64_t stride, const float* q_weight, const float* kv_weight,
                                const void* pos, int32_t pos_is_int64, const int32_t* slot, const int64_t* active,
                                const int32_t* block_table, int64_t table_stride, const float* angles, void* cache, void* cq,
                                int32_t rows, int32_t q_rank, int32_t true_q_rank, int32_t rank, int32_t true_rank,
                                int32_t rot, int32_t rot_pairs, float eps, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(q_rank > 0 && q_rank % 8 == 0 && rank % 8 == 0 && rot % 8 == 0 && stride % 8 == 0 && rot_pairs * 2 <= rot,
               "latent_prep: widths must be multiples of 8 and cover the rotated pairs");
  B200_REQUIRE(aligned16(fused) && aligned16(cq) && aligned16(cache) && aligned16(q_weight) && aligned16(kv_weight),
               "latent_prep: unaligned tensor");
  LatentPrepParams p = {fused, stride, q_weight, kv_weight, pos, pos_is_int64, slot, active, block_table, table_stride,
                        reinterpret_cast<const float2*>(angles), cache, cq, q_rank, true_q_rank, rank, true_rank, rot,
                        rot_pairs, overlap, eps};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const bool early = (overlap & OVERLAP_START) != 0;
  const int vecs = (q_rank + (cache ? rank + rot : 0)) / 8;
  int v = 1;
  while (v < 4 && vecs > 256 * v) v *= 2;
  B200_REQUIRE(vecs <= 1024, "latent_prep: at most 8192 elements per row (got %d)", vecs * 8);
  const dim3 block(((vecs + v - 1) / v + 31) / 32 * 32);
  cudaError_t e;
  if (!f32 && rows >= GLUE_WIDE_ROWS && vecs <= 256) {
    const unsigned grid = (rows + 7) / 8;
    if (vecs <= 64) latent_prep_rows_kernel<__nv_bfloat16, 2><<<grid, 256, 0, st>>>(p, rows);
    else if (vecs <= 128) latent_prep_rows_kernel<__nv_bfloat16, 4><<<grid, 256, 0, st>>>(p, rows);
    else if (vecs <= 192) latent_prep_rows_kernel<__nv_bfloat16, 6><<<grid, 256, 0, st>>>(p, rows);
    else latent_prep_rows_kernel<__nv_bfloat16, 8><<<grid, 256, 0, st>>>(p, rows);
    return check_launch("latent_prep");
  }
  if (f32) {
    e = v == 1 ? launch_pdl(early, latent_prep_kernel<float, 1>, dim3(rows), block, 0, st, p)
        : v == 2 ? launch_pdl(early, latent_prep_kernel<float, 2>, dim3(rows), block, 0, st, p)
                 : launch_pdl(early, latent_prep_kernel<float, 4>, dim3(rows), block, 0, st, p);
  } else {
    e = v == 1 ? launch_pdl(early, latent_prep_kernel<__nv_bfloat16, 1>, dim3(rows), block, 0, st, p)
        : v == 2 ? launch_pdl(early, latent_prep_kernel<__nv_bfloat16, 2>, dim3(rows), block, 0, st, p)
                 : launch_pdl(early, latent_prep_kernel<__nv_bfloat16, 4>, dim3(rows), block, 0, st, p);
  }
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_prep: %s", cudaGetErrorString(e));
  return check_launch("latent_prep");
}

extern "C" int b200_rope_interleaved(void* x, int64_t row_stride, int32_t head_stride, int32_t offset, int32_t heads,
                                     int32_t pairs, const int32_t* pos, const float* angles, int32_t rows, int32_t f32,
                                     b200_stream_t stream) {
  if (rows <= 0 || pairs <= 0) return OK;
  B200_REQUIRE(row_stride % 8 == 0 && head_stride % 8 == 0 && offset % 8 == 0 && aligned16(x) && offset + (2 * pairs + 7) / 8 * 8 <= head_stride,
               "rope_interleaved: the rotated part must start and end on groups of 8 elements");
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int64_t items = static_cast<int64_t>(rows) * heads * ((pairs + 3) / 4);
  const unsigned grid = static_cast<unsigned>((items + 255) / 256);
  const float2* a = reinterpret_cast<const float2*>(angles);
  if (f32) rope_interleaved_kernel<float><<<grid, 256, 0, st>>>(static_cast<float*>(x), row_stride, head_stride, offset, heads, pairs, pos, a, rows);
  else rope_interleaved_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(static_cast<__nv_bfloat16*>(x), row_stride, head_stride, offset, heads, pairs, pos, a, rows);
  return check_launch("rope_interleaved");
}

extern "C" int b200_latent_gather(const void* cache, void* out, const int32_t* block_table, int64_t table_stride,
                                  const int32_t* slots, const int32_t* cu_k, const int32_t* k_pos0, int32_t batch,
                                  int32_t max_keys, int32_t kv_heads, int32_t row_bytes, b200_stream_t stream) {
  if (batch <= 0 || max_keys <= 0) return OK;
  B200_REQUIRE(row_bytes % 16 == 0 && aligned16(cache) && aligned16(out) && batch <= 65535 && kv_heads > 0, "latent_gather: unaligned rows");
  latent_gather_kernel<<<dim3((max_keys + 15) / 16, batch), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), static_cast<uint4*>(out), block_table, table_stride, slots, cu_k, k_pos0,
      kv_heads, row_bytes / 16);
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
  B200_REQUIRE(dim % 64 == 0 && dim <= 1024 && rank % 64 == 0 && rot % 2 == 0 && rot_pairs * 2 <= rot && (batch + 15) / 16 <= 65535,
               "latent_absorb: dim (at most 1024) and rank must be multiples of 64");
  B200_REQUIRE(aligned16(q) && aligned16(w_uk) && aligned16(out), "latent_absorb: unaligned tensor");
  LatentAbsorbParams p = {q, w_uk, pos, reinterpret_cast<const float2*>(angles), out, batch, heads, dim, rot, rot_pairs, rank, overlap};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(heads, rank / 64, (batch + 15) / 16);
  if (f32) latent_absorb_f32_kernel<<<grid, 128, 0, st>>>(p);
  else {
    if (!head_gemm_configure(reinterpret_cast<const void*>(latent_absorb_bf16_kernel), 0))
      return fail(ERR_RUNTIME, "latent_absorb: cannot raise dynamic shared memory");
    const cudaError_t e = launch_pdl((overlap & OVERLAP_START) != 0, latent_absorb_bf16_kernel, grid, dim3(128), dim / 64 * HG_STEP, st, p);
    if (e != cudaSuccess) return fail(ERR_LAUNCH, "latent_absorb: %s", cudaGetErrorString(e));
  }
  return check_launch("latent_absorb");
}

extern "C" int b200_latent_decode_simple(const void* q, const void* cache, const int32_t* block_table, int64_t table_stride,
                                         const int64_t* pos, const int64_t* active, float* ml, float* o, int32_t batch,
                                         int32_t heads, int32_t rank, int32_t rot, int32_t window, int32_t splits, float scale,
                                         int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  const RowDecodeParams p = {q, static_cast<int64_t>(heads) * (rank + rot), cache, block_table, table_stride, pos, active,
                             reinterpret_cast<float2*>(ml), o, heads, 1, heads, rank + rot, 0, rank, rank + rot, window, splits,
                             overlap, scale, nullptr};
  return row_decode_simple_launch(p, batch, f32 != 0, "latent_decode_simple", reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int b200_latent_value(const float* ml, const float* o, const void* w_uv, void* merged, void* out, int32_t batch,
                                 int32_t heads, int32_t rank, int32_t vdim, int32_t splits, int32_t f32, int32_t overlap,
                                 b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(rank % 64 == 0 && rank <= LS_MAX_COLS && vdim % 64 == 0 && splits > 0 && splits <= LATENT_MAX_SPLITS && batch <= 65535,
               "latent_value: rank and vdim must be multiples of 64, rank at most %d, splits at most %d", LS_MAX_COLS,
               LATENT_MAX_SPLITS);
  B200_REQUIRE(aligned16(o) && aligned16(w_uv) && aligned16(merged) && aligned16(out), "latent_value: unaligned tensor");
  const LatentValueParams p = {w_uv, merged, out, batch, heads, rank, vdim, overlap};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(heads, vdim / 64, (batch + 15) / 16);
  // the product behind the merge: in bf16 it starts early and waits, in fp32 it is launched plainly
  const int merge_overlap = f32 ? overlap & ~OVERLAP_TRIGGER : overlap | OVERLAP_TRIGGER;
  const RowMergeParams merge = {reinterpret_cast<const float2*>(ml), o, nullptr, 0, merged, static_cast<int64_t>(heads) * rank,
                                heads, rank, splits, merge_overlap, 1.f};
  const int rc = row_merge_launch(merge, batch, f32 != 0, "latent_value", st);
  if (rc != OK) return rc;
  if (f32) {
    latent_value_f32_kernel<<<grid, 128, 0, st>>>(p);
    return check_launch("latent_value");
  }
  if (!head_gemm_configure(reinterpret_cast<const void*>(latent_value_bf16_kernel), 1))
    return fail(ERR_RUNTIME, "latent_value: cannot raise dynamic shared memory");
  if (launch_pdl(true, latent_value_bf16_kernel, grid, dim3(128), rank / 64 * HG_STEP, st, p) != cudaSuccess)
    return fail(ERR_LAUNCH, "latent_value: %s", cudaGetErrorString(cudaGetLastError()));
  return check_launch("latent_value");
}
