// Decode attention over paged rows on the tensor cores (latent.cuh, RowDecodeParams): the heads that share a row are one MMA
// M tile of 16, so a row is read once per 16 heads.  Latent attention: all heads share the rows [latent | rotated key part]
// and sum their first `rank` elements.  Grouped heads: rows [key | value] per key/value head.
//
// One CTA = (key range of a slot, block of up to 16 heads of one key/value head).  A producer warp brings 32-token tiles (two 16-token pages, one
// tensor-map TMA box each, 128-byte swizzle, no multicast) through a ring of mbarrier-tracked stages; eight warps work on
// a tile together:
//     S[16 x 32]    = q . keys^T      a warp takes 16 tokens and every fourth 32-wide step of the key part
//     P             = exp2(S - m)     half a warp per head row, two tokens per lane; online maximum and sum in fp32
//     O[16 x rank] += P . values      a warp owns rank / 8 columns; accumulators stay in registers
// The kernel is bound by HBM (at most 2 * 16 FLOP per byte), far below what 16-row tiles reach on tcgen05 (M = 128), so
// mma.sync carries the products, as in the paged decode kernels.  Key ranges leave (max, sum, unnormalised O) in fp32;
// row_merge_kernel merges them.  Rows of a tile outside the visible range are zeroed in shared memory before they are used:
// whatever a page held for an earlier owner cannot reach the sums.  Every wait is bounded.
#include <mutex>

#include "latent.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int LD_WARPS = 8;                      // consumers; one more warp produces
constexpr int LD_THREADS = (LD_WARPS + 1) * 32;
constexpr int LD_TOK = 32;
constexpr int LD_MAX_STAGES = 6;
constexpr int LD_S_PITCH = 36;                   // floats per score row
constexpr int LD_P_PITCH = 40;                   // bf16 per probability row (80 bytes: ldmatrix rows in different banks)
constexpr int LD_SMEM_LIMIT = 216 * 1024;         // dynamic; 11 KiB more are static
constexpr int LD_SMEM_PAIR = 102 * 1024;          // ... when two CTAs share an SM

// NT: value columns per warp / 8 that the accumulators hold (rank <= 64 * NT)
template <int NT>
__global__ void __launch_bounds__(LD_THREADS, NT <= 8 ? 2 : 1)
row_decode_kernel(const __grid_constant__ RowDecodeParams p, const __grid_constant__ CUtensorMap map_rows, int stages) {
  extern __shared__ __align__(1024) uint8_t ld_smem_raw[];
  __shared__ uint64_t full[LD_MAX_STAGES], empty[LD_MAX_STAGES];
  __shared__ float ss[4][16][LD_S_PITCH];            // partial scores of the four quarters of a row
  __shared__ __align__(16) __nv_bfloat16 ps[16][LD_P_PITCH];
  __shared__ float alphas[16];
  const int blocks = (p.group + 15) / 16, split = blockIdx.x, g = blockIdx.y / blocks, hb = blockIdx.y % blocks, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row_bytes = p.pitch * 2, tile_bytes = LD_TOK * row_bytes, page_bytes = PAGE * row_bytes;
  const int q_pitch = p.key * 2 + 16;
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(ld_smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* qs = ring + stages * tile_bytes;
  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], LD_WARPS);
    }
    mbar_fence_init();
  }
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  int lo, hi;
  latent_split_range(p, b, split, lo, hi);
  const int heads_here = min(16, p.group - hb * 16), head0 = g * p.group + hb * 16;
  const int64_t part0 = (static_cast<int64_t>(b) * p.heads + head0) * p.splits + split;
  if (lo >= hi) {
    if (tid < heads_here) p.ml[part0 + static_cast<int64_t>(tid) * p.splits] = make_float2(-INFINITY, 0.f);
    return;
  }
  const int page0 = lo / PAGE, pages = (hi + PAGE - 1) / PAGE - page0, tiles = (pages + 1) / 2;
  __syncthreads();  // barriers initialised
  if (warp == LD_WARPS) {
    const int32_t* table = p.table + b * p.table_stride + page0;
    bool ok = true;
    for (int t = 0; t < tiles && ok; ++t) {
      const int s = t % stages;
      if (t >= stages) ok = mbar_wait_bounded(&empty[s], (t / stages - 1) & 1);
      if (!ok) break;
      if (lane == 0) {
        const int n = min(2, pages - 2 * t);
        mbar_expect_tx(&full[s], n * page_bytes);
        for (int i = 0; i < n; ++i)
          tma_load_3d(ring + s * tile_bytes + i * page_bytes, &map_rows, 0, (table[2 * t + i] * p.kv_heads + g) * PAGE, 0, &full[s]);
      }
      __syncwarp();
    }
    if (!ok && lane == 0) atomicExch(p.err, 1);
    return;
  }
  // q rows of the head block (rows past the last head are zero)
  {
    const uint4* q = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q) + b * p.q_stride + static_cast<int64_t>(head0) * p.key);
    const int vecs = p.key / 8;
    for (int i = tid; i < 16 * vecs; i += LD_WARPS * 32) {
      const int r = i / vecs, c = i % vecs;
      *reinterpret_cast<uint4*>(qs + r * q_pitch + c * 16) = r < heads_here ? q[r * vecs + c] : make_uint4(0, 0, 0, 0);
    }
  }
  named_barrier(1, LD_WARPS * 32);
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;   // of head row sm_row: the maximum, and this lane's part of the sum
  const int sm_row = warp * 2 + (lane >> 4), sm_tok = (lane & 15) * 2;
  const float scale_log2 = p.scale * 1.4426950408889634f;
  const int tg = warp & 1, kq = warp >> 1;
  const int units = p.key / 32;
  const int nt = p.rank / 64, col0 = warp * nt * 8;
  const int v_chunk = (p.v_off + col0) / 8, last_chunk = p.pitch / 8 - 1;
  const uint32_t a_base = smem_u32(qs) + (lane & 15) * q_pitch + (lane >> 4) * 16;
  const int s_row = lane & 7;   // rows s_row and s_row + 8 of page tg
  const uint32_t s_off = tg * page_bytes + s_row * 128;
  bool ok = true;
  for (int t = 0; t < tiles; ++t) {
    const int s = t % stages;
    uint8_t* tile = ring + s * tile_bytes;
    const uint32_t tile_a = smem_u32(tile);
    const int tok0 = (page0 + 2 * t) * PAGE;  // position of the tile's first row
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&full[s], (t / stages) & 1));  // uniform in the warp
    const bool ragged = tok0 < lo || tok0 + LD_TOK > hi;
    if (ragged) {
      for (int r = warp; r < LD_TOK; r += LD_WARPS)
        if (tok0 + r < lo || tok0 + r >= hi)
          for (int c = lane; c < row_bytes / 16; c += 32)
            *reinterpret_cast<uint4*>(tile + (r / PAGE) * page_bytes + (c >> 3) * (PAGE * 128) + (r % PAGE) * 128 + (c & 7) * 16) =
                make_uint4(0, 0, 0, 0);
      named_barrier(1, LD_WARPS * 32);
    }
    // ---- scores
    if (ok) {
      float c[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 3
      for (int u = kq; u < units; u += 4) {
        uint32_t a0[4], a1[4], b0[4], b1[4];
        const int chunk = u * 4 + (lane >> 3);
        const uint32_t at = tile_a + s_off + (chunk >> 3) * (PAGE * 128) + (((chunk & 7) ^ s_row) << 4);
        ldmatrix_x4(a0, a_base + u * 64);
        ldmatrix_x4(b0, at);
        ldmatrix_x4(b1, at + 8 * 128);
        ldmatrix_x4(a1, a_base + u * 64 + 32);
        mma_bf16_16816(c[0], a0, b0[0], b0[1]);
        mma_bf16_16816(c[1], a0, b1[0], b1[1]);
        mma_bf16_16816(c[0], a1, b0[2], b0[3]);
        mma_bf16_16816(c[1], a1, b1[2], b1[3]);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int col = tg * 16 + i * 8 + (lane & 3) * 2, r = lane >> 2;
        *reinterpret_cast<float2*>(&ss[kq][r][col]) = make_float2(c[i][0], c[i][1]);
        *reinterpret_cast<float2*>(&ss[kq][r + 8][col]) = make_float2(c[i][2], c[i][3]);
      }
    }
    named_barrier(1, LD_WARPS * 32);
    // ---- softmax: half a warp per head row, two tokens per lane
    {
      float2 a = make_float2(0.f, 0.f);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 part = *reinterpret_cast<const float2*>(&ss[k][sm_row][sm_tok]);
        a.x += part.x, a.y += part.y;
      }
      const int at = tok0 + sm_tok;
      const float x0 = at >= lo && at < hi ? a.x * scale_log2 : -INFINITY;
      const float x1 = at + 1 >= lo && at + 1 < hi ? a.y * scale_log2 : -INFINITY;
      float mx = fmaxf(x0, x1);
#pragma unroll
      for (int bit = 8; bit >= 1; bit >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, bit));
      const float m_new = fmaxf(m_run, mx);               // a tile holds at least one visible token
      const float alpha = ex2_fast(m_run - m_new);
      const float p0 = ex2_fast(x0 - m_new), p1 = ex2_fast(x1 - m_new);
      l_run = fmaf(l_run, alpha, p0 + p1);
      m_run = m_new;
      *reinterpret_cast<uint32_t*>(&ps[sm_row][sm_tok]) = pack_bf16(p0, p1);
      if ((lane & 15) == 0) alphas[sm_row] = alpha;
    }
    named_barrier(1, LD_WARPS * 32);
    // ---- O: this warp's columns
    if (ok) {
      const float al0 = alphas[lane >> 2], al1 = alphas[(lane >> 2) + 8];
      if (__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) {
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          acc[i][0] *= al0, acc[i][1] *= al0;
          acc[i][2] *= al1, acc[i][3] *= al1;
        }
      }
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        if (ks * PAGE >= hi - tok0) break;               // the second page of the last tile may be missing
        uint32_t a[4];
        ldmatrix_x4(a, smem_u32(&ps[lane & 15][ks * 16 + (lane >> 4) * 8]));
        const uint32_t v_row = tile_a + ks * page_bytes + (lane & 15) * 128;
#pragma unroll
        for (int i = 0; i < NT; i += 2) {
          if (i < nt) {
            uint32_t bm[4];
            const int chunk = min(v_chunk + i + (lane >> 4), last_chunk);  // an odd last pair's second half is not used
            ldmatrix_x4_trans(bm, v_row + (chunk >> 3) * (PAGE * 128) + (((chunk & 7) ^ (lane & 7)) << 4));
            mma_bf16_16816(acc[i], a, bm[0], bm[1]);
            if (NT > 1 && i + 1 < nt) mma_bf16_16816(acc[i + 1 < NT ? i + 1 : i], a, bm[2], bm[3]);
          }
        }
      }
    }
    if (ragged) fence_proxy_async();  // the zeroed rows before the next copy into this stage
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
  }
  if (!ok) {
    if (lane == 0) atomicExch(p.err, 1);
    return;
  }
#pragma unroll
  for (int bit = 8; bit >= 1; bit >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, bit);
  // maxima are kept in the log2 domain; the merge works with natural exponentials
  if ((lane & 15) == 0 && sm_row < heads_here)
    p.ml[part0 + static_cast<int64_t>(sm_row) * p.splits] = make_float2(m_run * 0.6931471805599453f, l_run);
#pragma unroll
  for (int i = 0; i < NT; ++i)
    if (i < nt) {
      const int r = lane >> 2, c = col0 + i * 8 + (lane & 3) * 2;
      float* o = p.o + part0 * p.rank + c;
      const int64_t step = static_cast<int64_t>(p.splits) * p.rank;
      if (r < heads_here) *reinterpret_cast<float2*>(o + r * step) = make_float2(acc[i][0], acc[i][1]);
      if (r + 8 < heads_here) *reinterpret_cast<float2*>(o + (r + 8) * step) = make_float2(acc[i][2], acc[i][3]);
    }
}

// One encoded map per cache (base, rows, row width); a handful per engine.
static bool row_map(CUtensorMap* out, const void* base, int64_t rows, int pitch) {
  struct Entry {
    const void* base;
    int64_t rows;
    int pitch;
    CUtensorMap map;
  };
  static std::mutex lock;
  static Entry entries[64];
  static int used = 0, next = 0;
  std::lock_guard<std::mutex> guard(lock);
  for (int i = 0; i < used; ++i)
    if (entries[i].base == base && entries[i].rows == rows && entries[i].pitch == pitch) {
      *out = entries[i].map;
      return true;
    }
  Entry e = {base, rows, pitch, {}};
  if (!encode_tile_map(&e.map, base, static_cast<uint64_t>(rows), pitch, static_cast<uint64_t>(pitch) * 2, PAGE, pitch / 64)) return false;
  const int at = used < 64 ? used++ : next++ % 64;
  entries[at] = e;
  *out = e.map;
  return true;
}

template <int NT>
static int launch_row_decode(const RowDecodeParams& p, const CUtensorMap& map, int batch, int stages, int smem,
                                cudaStream_t st) {
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(row_decode_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, LD_SMEM_LIMIT) != cudaSuccess)
      return fail(ERR_RUNTIME, "row_decode: cannot raise dynamic shared memory to %d", LD_SMEM_LIMIT);
    configured[dev] = true;
  }
  const dim3 grid(p.splits, p.kv_heads * ((p.group + 15) / 16), batch);
  if (launch_pdl((p.overlap & OVERLAP_START) != 0, row_decode_kernel<NT>, grid, dim3(LD_THREADS), smem, st, p, map, stages) != cudaSuccess)
    return fail(ERR_LAUNCH, "row_decode: %s", cudaGetErrorString(cudaGetLastError()));
  return check_launch("row_decode");
}

int row_decode_launch(const RowDecodeParams& in, int64_t num_pages, int batch, const char* name, cudaStream_t st) {
  B200_REQUIRE(in.key > 0 && in.key % 32 == 0 && in.rank > 0 && in.rank % 64 == 0 && in.rank <= 1024 && in.pitch % 64 == 0 &&
                   in.v_off % 8 == 0 && in.key <= in.pitch && in.v_off + in.rank <= in.pitch && in.q_stride % 8 == 0,
               "%s: keys must be a multiple of 32, values and rows of 64, at most 1024 value columns (got %d, %d, %d)", name, in.key,
               in.rank, in.pitch);
  B200_REQUIRE(in.window > 0 && in.splits > 0 && in.splits <= LATENT_MAX_SPLITS && batch <= 65535 && in.scale > 0.f && num_pages > 0 &&
                   in.kv_heads > 0 && in.heads == in.kv_heads * in.group && num_pages * in.kv_heads * PAGE < (1ll << 31),
               "%s: window, scale and splits (at most %d) must be positive, heads a multiple of the key/value heads", name,
               LATENT_MAX_SPLITS);
  B200_REQUIRE(aligned16(in.q) && aligned16(in.cache) && aligned16(in.o), "%s: unaligned tensor", name);
  RowDecodeParams p = in;
  const int tile = LD_TOK * p.pitch * 2, q_bytes = 16 * (p.key * 2 + 16) + 1024;  // incl. alignment of the ring
  int stages = p.rank <= 512 ? (LD_SMEM_PAIR - q_bytes) / tile : 0;   // two CTAs on an SM cover each other's latencies
  if (stages < 2) stages = (LD_SMEM_LIMIT - q_bytes) / tile;
  if (stages > LD_MAX_STAGES) stages = LD_MAX_STAGES;
  B200_REQUIRE(stages >= 2, "%s: rows of %d elements do not fit", name, p.pitch);
  p.err = wait_timeout_flag();
  if (!p.err) return fail(ERR_RUNTIME, "%s: no error flag", name);
  CUtensorMap map;
  if (!row_map(&map, p.cache, num_pages * p.kv_heads * PAGE, p.pitch)) return fail(ERR_RUNTIME, "%s: cannot encode the cache's tensor map", name);
  const int smem = stages * tile + q_bytes;
  if (p.rank <= 128) return launch_row_decode<2>(p, map, batch, stages, smem, st);
  if (p.rank <= 512) return launch_row_decode<8>(p, map, batch, stages, smem, st);
  return launch_row_decode<16>(p, map, batch, stages, smem, st);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_decode(const void* q, const void* cache, int64_t num_pages, const int32_t* block_table,
                                  int64_t table_stride, const int64_t* pos, const int64_t* active, float* ml, float* o,
                                  int32_t batch, int32_t heads, int32_t rank, int32_t rot, int32_t window, int32_t splits,
                                  float scale, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(rank > 0 && rank % 64 == 0 && rot >= 0 && rot % 64 == 0 && heads > 0,
               "latent_decode: rank and rot must be multiples of 64 (got %d, %d)", rank, rot);
  const RowDecodeParams p = {q, static_cast<int64_t>(heads) * (rank + rot), cache, block_table, table_stride, pos, active,
                             reinterpret_cast<float2*>(ml), o, heads, 1, heads, rank + rot, 0, rank, rank + rot, window, splits,
                             overlap, scale, nullptr};
  return row_decode_launch(p, num_pages, batch, "latent_decode", reinterpret_cast<cudaStream_t>(stream));
}
