// Windowed causal attention of packed prompt portions on tcgen05 (bf16, accumulators in TMEM), over expanded latents or over
// the keys and values of grouped heads.
//
// One CTA = 128 query tokens of one head of one sequence.  Latent keys are [expanded part of the head | rotated part shared
// by all heads]: two TMA boxes per 128-key tile land side by side as the column blocks of one K-major operand, so the shared
// part is never copied per head.  Grouped heads: `group` query heads read the same key/value head, keys are one box; a key
// size that is no multiple of 64 brings columns of its neighbour along, which no product reads.  The epilogue may multiply
// by sigmoid(gate) and a constant.  Per tile:
//     S[128 x 128]   = Q . K^T            tcgen05.mma, both operands in shared memory, two S buffers in TMEM
//     P              = exp2(S*scale - m)  two softmax threads per row, TMEM -> registers -> TMEM (bf16 over S)
//     O[128 x vdim] += P . V              tcgen05.mma, P from TMEM, V as an MN-major operand
// Tiles run from the first key the block's first query sees to the last query's own key; rows mask their window's and
// the diagonal's edge.  K and V are double-buffered where shared memory allows.  Roles: warps 0-7 softmax and epilogue,
// warp 8 issues MMAs, warps 9 / 10 load K (and Q) / V.  The running maximum may lag by 2^8 before O is rescaled.
// Scores, maxima and sums are fp32.  Every wait is bounded; on expiry the error flag is set and the CTA drains.
#include "latent.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int LP_TILE = 128;
constexpr int LP_SOFTMAX_THREADS = 256;
constexpr int LP_THREADS = 352;
constexpr int LP_BLOCK_BYTES = LP_TILE * 128;      // one 64-column block of 128 rows
constexpr uint32_t LP_TMEM_COLS = 512;             // S0 [0,128) S1 [128,256) O [256, 256 + vdim)
constexpr float LP_TAU = 8.0f;
constexpr int LP_SMEM_LIMIT = 220 * 1024;

struct LatentUmmaParams {
  __nv_bfloat16* out;
  const __nv_bfloat16* gate;      // [tokens, gate_stride] or NULL
  int64_t out_stride, gate_stride;
  float out_scale;
  const int32_t *cu_q, *cu_k, *q_pos0, *k_pos0;
  int group, vdim, dim_blocks, rot_blocks, dim_steps, rot_steps, window, k_stages, v_stages;
  float scale_log2;
  int* err;
};

__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_v,
                      const __grid_constant__ LatentUmmaParams p) {
  extern __shared__ __align__(1024) uint8_t lp_smem_raw[];
  __shared__ uint64_t bar_q, bar_k[2], bar_v[2], bar_s[2], bar_p[2], bar_pv[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float xm[2][2][128];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qb = gridDim.x - 1 - blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / p.group;
  const int q_row0 = p.cu_q[b], len = p.cu_q[b + 1] - q_row0;
  const int q0 = qb * LP_TILE;
  if (q0 >= len) return;
  const int k_first = p.k_pos0[b];
  const int pos0 = p.q_pos0[b] + q0, pos_last = p.q_pos0[b] + min(q0 + LP_TILE, len) - 1;
  const int key0 = max(k_first, pos0 - p.window + 1);          // position of the first tile's first key
  const int n_tiles = (pos_last - key0) / LP_TILE + 1;
  const int k_row0 = p.cu_k[b] + key0 - k_first;               // its packed row

  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lp_smem_raw) + 1023) & ~uintptr_t(1023));
  const int k_blocks = p.dim_blocks + p.rot_blocks, v_blocks = p.vdim / 64;
  const int k_bytes = k_blocks * LP_BLOCK_BYTES, v_bytes = v_blocks * LP_BLOCK_BYTES;
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + k_bytes;
  uint8_t* v_s = k_s + p.k_stages * k_bytes;

  if (warp == 0) tmem_alloc(&tmem_slot, LP_TMEM_COLS);
  if (tid == 0) {
    mbar_init(&bar_q, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar_k[i], 1);
      mbar_init(&bar_v[i], 1);
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], LP_SOFTMAX_THREADS);
      mbar_init(&bar_pv[i], 1);
    }
    mbar_fence_init();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot, tmem_o = tmem + 2 * LP_TILE;

  if (warp == 9) {
    if (lane == 0) {
      bool ok = true;
      mbar_expect_tx(&bar_q, k_bytes);
      tma_load_4d(q_s, &map_q, 0, q_row0 + q0, 0, h, &bar_q);
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j % p.k_stages, i = j - p.k_stages;
        if (i >= 0) ok = mbar_wait_bounded(&bar_s[i & 1], (i >> 1) & 1);  // S of the tile that used this stage is done
        if (!ok) break;
        mbar_expect_tx(&bar_k[st], k_bytes);
        tma_load_4d(k_s + st * k_bytes, &map_k, 0, k_row0 + j * LP_TILE, 0, g, &bar_k[st]);
        if (p.rot_blocks > 0) tma_load_3d(k_s + st * k_bytes + p.dim_blocks * LP_BLOCK_BYTES, &map_r, 0, k_row0 + j * LP_TILE, 0, &bar_k[st]);
      }
      if (!ok) atomicExch(p.err, 1);
    }
  } else if (warp == 10) {
    if (lane == 0) {
      bool ok = true;
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j % p.v_stages, i = j - p.v_stages;
        if (i >= 0) ok = mbar_wait_bounded(&bar_pv[i & 1], (i >> 1) & 1);
        if (!ok) break;
        mbar_expect_tx(&bar_v[st], v_bytes);
        tma_load_4d(v_s + st * v_bytes, &map_v, 0, k_row0 + j * LP_TILE, 0, g, &bar_v[st]);
      }
      if (!ok) atomicExch(p.err, 1);
    }
  } else if (warp == 8) {
    const bool leader = lane == 0;
    const uint32_t idesc_s = idesc_bf16_f32(128, LP_TILE, false, false);
    const uint32_t idesc_o = idesc_bf16_f32(128, p.vdim, false, true);
    const uint32_t q_addr = smem_u32(q_s), k_addr = smem_u32(k_s), v_addr = smem_u32(v_s);
    bool ok = mbar_wait_bounded(&bar_q, 0);
    auto issue_pv = [&](int j) {
      const int st = j % p.v_stages;
      ok = ok && mbar_wait_bounded(&bar_p[j & 1], (j >> 1) & 1);
      ok = ok && mbar_wait_bounded(&bar_v[st], (j / p.v_stages) & 1);
      if (!ok) return;
      tc_fence_after_sync();
#pragma unroll
      for (int kt = 0; kt < LP_TILE / 16; ++kt)
        umma_ts_leader(tmem_o, tmem + (j & 1) * LP_TILE + kt * 8,
                       smem_desc_sw128(v_addr + st * v_bytes + kt * 2048, LP_BLOCK_BYTES, 1024), idesc_o, j > 0 || kt > 0, leader);
      umma_commit_leader(&bar_pv[j & 1], leader);
    };
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int s = j & 1, st = j % p.k_stages;
      ok = mbar_wait_bounded(&bar_k[st], (j / p.k_stages) & 1);
      if (ok && j >= 2) ok = mbar_wait_bounded(&bar_pv[s], ((j - 2) >> 1) & 1);  // P of tile j-2 has been consumed
      if (!ok) break;
      tc_fence_after_sync();
      const uint32_t k_st = k_addr + st * k_bytes;
      for (int ks = 0; ks < p.dim_steps; ++ks) {
        const uint32_t o = (ks >> 2) * LP_BLOCK_BYTES + (ks & 3) * 32;
        umma_ss_leader(tmem + s * LP_TILE, smem_desc_sw128(q_addr + o, 16, 1024), smem_desc_sw128(k_st + o, 16, 1024), idesc_s,
                       ks > 0, leader);
      }
      for (int ks = 0; ks < p.rot_steps; ++ks) {
        const uint32_t o = (p.dim_blocks + (ks >> 2)) * LP_BLOCK_BYTES + (ks & 3) * 32;
        umma_ss_leader(tmem + s * LP_TILE, smem_desc_sw128(q_addr + o, 16, 1024), smem_desc_sw128(k_st + o, 16, 1024), idesc_s,
                       true, leader);
      }
      umma_commit_leader(&bar_s[s], leader);
      if (j >= 1) issue_pv(j - 1);
    }
    if (ok) issue_pv(n_tiles - 1);
    if (!ok && leader) atomicExch(p.err, 1);
  } else {
    const int row = 32 * (warp & 3) + lane, half = warp >> 2;
    const int pos = min(pos0 + row, pos_last);             // rows behind the end repeat the last query and are not stored
    const int col_lo = pos - p.window + 1 - key0, col_hi = pos - key0;  // visible columns over all tiles (col_lo may be < 0)
    const uint32_t lane_base = static_cast<uint32_t>(32 * (warp & 3)) << 16;
    const int pair_bar = 1 + (warp & 3);
    const float sc = p.scale_log2;
    float m_ref = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int s = j & 1;
      // `ok` stays uniform in the warp: what follows are warp-wide operations
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_s[s], (j >> 1) & 1));
      uint32_t r0[32], r1[32];
      float m_half = -INFINITY;
      if (ok) {
        tc_fence_after_sync();
        tmem_ld32(tmem + lane_base + s * LP_TILE + half * 64, r0);
        tmem_ld32(tmem + lane_base + s * LP_TILE + half * 64 + 32, r1);
        tmem_ld_wait();
        const int lo = col_lo - j * LP_TILE - half * 64, hi = col_hi - j * LP_TILE - half * 64;
        if (lo > 0 || hi < 63) {
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            if (c < lo || c > hi) r0[c] = 0xff800000u;
            if (c + 32 < lo || c + 32 > hi) r1[c] = 0xff800000u;
          }
        }
        float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
        for (int c = 0; c < 32; c += 2) {
          mx0 = fmaxf(mx0, __uint_as_float(r0[c]));
          mx1 = fmaxf(mx1, __uint_as_float(r0[c + 1]));
          mx2 = fmaxf(mx2, __uint_as_float(r1[c]));
          mx3 = fmaxf(mx3, __uint_as_float(r1[c + 1]));
        }
        m_half = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
      }
      xm[s][half][row] = m_half;
      named_barrier(pair_bar, 64);
      if (ok) {
        // the first tile starts at the block's first visible key, at most 127 columns in front of any row's own window:
        // every row sees at least one of its columns, so m_ref is finite from here on
        const float m_new = fmaxf(m_ref, fmaxf(m_half, xm[s][half ^ 1][row]) * sc);
        if (j == 0) {
          m_ref = m_new;
        } else {
          const bool need = (m_new - m_ref) > LP_TAU;
          if (__any_sync(0xffffffffu, need)) {
            ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_pv[(j - 1) & 1], ((j - 1) >> 1) & 1));  // O at rest
            tc_fence_after_sync();
            const float alpha = need ? ex2_fast(m_ref - m_new) : 1.f;
#pragma unroll 1
            for (int c0 = 0; c0 < p.vdim / 2; c0 += 32) {
              uint32_t o[32];
              tmem_ld32(tmem_o + lane_base + half * (p.vdim / 2) + c0, o);
              tmem_ld_wait();
#pragma unroll
              for (int c = 0; c < 32; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
              tmem_st32(tmem_o + lane_base + half * (p.vdim / 2) + c0, o);
            }
            tmem_st_wait();
            l_run *= alpha;
            if (need) m_ref = m_new;
          }
        }
        float sum0 = 0.f, sum1 = 0.f;
        const float neg_m = -m_ref;
        uint32_t w[32];
#pragma unroll
        for (int c = 0; c < 32; ++c) {
          const float x0 = ex2_fast(fmaf(__uint_as_float(c < 16 ? r0[2 * c] : r1[2 * c - 32]), sc, neg_m));
          const float x1 = ex2_fast(fmaf(__uint_as_float(c < 16 ? r0[2 * c + 1] : r1[2 * c - 31]), sc, neg_m));
          sum0 += x0;
          sum1 += x1;
          w[c] = pack_bf16(x0, x1);
        }
        l_run += sum0 + sum1;
        tmem_st32(tmem + lane_base + s * LP_TILE + half * 32, w);
        tmem_st_wait();
      }
      tc_fence_before_sync();
      mbar_arrive(&bar_p[s]);
    }
    // ---- epilogue: O / l -> bf16 -> staged over Q and K (no copy or product is in flight any more) -> global
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_pv[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1));
    float* xl = &xm[n_tiles & 1][0][0];
    xl[half * 128 + row] = l_run;
    named_barrier(pair_bar, 64);
    const int out_pitch = p.vdim * 2 + 16;
    if (ok) {
      tc_fence_after_sync();
      const float inv_l = 1.f / (l_run + xl[(half ^ 1) * 128 + row]);
      uint8_t* orow = smem + row * out_pitch + half * p.vdim;
#pragma unroll 1
      for (int c0 = 0; c0 < p.vdim / 2; c0 += 32) {
        uint32_t o[32];
        tmem_ld32(tmem_o + lane_base + half * (p.vdim / 2) + c0, o);
        tmem_ld_wait();
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint32_t w[4];
#pragma unroll
          for (int k = 0; k < 4; ++k)
            w[k] = pack_bf16(__uint_as_float(o[g * 8 + k * 2]) * inv_l, __uint_as_float(o[g * 8 + k * 2 + 1]) * inv_l);
          *reinterpret_cast<uint4*>(orow + (c0 + g * 8) * 2) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    } else {
      atomicExch(p.err, 1);
    }
    named_barrier(9, LP_SOFTMAX_THREADS);
    if (ok) {
      const int vecs = p.vdim / 8, col = h * p.vdim;
      constexpr int U = 8;                             // rows' parts per thread whose gates are requested together
      for (int i0 = tid; i0 < LP_TILE * vecs; i0 += U * LP_SOFTMAX_THREADS) {
        uint4 z[U];
        if (p.gate) {
#pragma unroll
          for (int u = 0; u < U; ++u) {
            const int i = i0 + u * LP_SOFTMAX_THREADS, r = i / vecs;
            if (r < LP_TILE && q0 + r < len)
              z[u] = *reinterpret_cast<const uint4*>(p.gate + static_cast<int64_t>(q_row0 + q0 + r) * p.gate_stride + col + (i - r * vecs) * 8);
          }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int i = i0 + u * LP_SOFTMAX_THREADS, r = i / vecs, c = i - r * vecs;
          if (r >= LP_TILE || q0 + r >= len) continue;
          uint4 o = *reinterpret_cast<const uint4*>(smem + r * out_pitch + c * 16);
          if (p.gate) {
            float f[8], g8[8];
            load8(reinterpret_cast<const __nv_bfloat16*>(&o), f);
            load8(reinterpret_cast<const __nv_bfloat16*>(&z[u]), g8);
#pragma unroll
            for (int k = 0; k < 8; ++k) f[k] *= sigmoid_f<__nv_bfloat16>(g8[k]) * p.out_scale;
            store8(reinterpret_cast<__nv_bfloat16*>(&o), f);
          }
          *reinterpret_cast<uint4*>(p.out + static_cast<int64_t>(q_row0 + q0 + r) * p.out_stride + col + c * 8) = o;
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, LP_TMEM_COLS);
}

int row_prefill_launch(const RowPrefillOperands& a, const char* name, cudaStream_t st) {
  B200_REQUIRE(a.dim > 0 && a.rot % 64 == 0 && a.vdim > 0 && a.vdim % 64 == 0 && a.dim + a.rot <= 256 && a.vdim <= 256 &&
                   (a.rot == 0 || a.dim % 64 == 0),
               "%s: keys and values of at most 256, in multiples of 64 (got %d, %d, %d)", name, a.dim, a.rot, a.vdim);
  B200_REQUIRE(a.true_dim > 0 && a.true_dim <= a.dim && a.true_rot <= a.rot && a.window > 0 && a.scale > 0.f && a.tokens > 0 && a.keys > 0,
               "%s: bad true sizes, window or scale", name);
  B200_REQUIRE(a.heads > 0 && a.heads <= 65535 && a.batch <= 65535 && a.group > 0 && a.heads % a.group == 0,
               "%s: at most 65535 heads and sequences", name);
  B200_REQUIRE(aligned16(a.q) && aligned16(a.k) && aligned16(a.r) && aligned16(a.v) && aligned16(a.out) && aligned16(a.gate) &&
                   a.out_stride % 8 == 0 && a.gate_stride % 8 == 0,
               "%s: unaligned tensor", name);
  const int dim_blocks = (a.dim + 63) / 64, rot_blocks = a.rot / 64, kv_heads = a.heads / a.group;
  const int head_width = a.dim + a.rot;
  B200_REQUIRE(a.q_stride >= static_cast<int64_t>(a.heads - 1) * head_width + (dim_blocks + rot_blocks) * 64,
               "%s: rows of q end inside the last head's column blocks", name);
  if (row_prefill_pairs(a)) return row_prefill_pair_launch(a, name, st);
  CUtensorMap map_q, map_k, map_r = {}, map_v;
  if (!encode_head_map(&map_q, a.q, a.tokens, a.q_stride, dim_blocks + rot_blocks, head_width, a.heads, LP_TILE) ||
      !encode_head_map(&map_k, a.k, a.keys, a.k_stride, dim_blocks, a.k_head, kv_heads, LP_TILE) ||
      !encode_head_map(&map_v, a.v, a.keys, a.v_stride, a.vdim / 64, a.v_head, kv_heads, LP_TILE))
    return fail(ERR_RUNTIME, "%s: cannot encode a tensor map", name);
  if (rot_blocks > 0) {
    const uint64_t dims[3] = {64, static_cast<uint64_t>(a.keys), static_cast<uint64_t>(rot_blocks)};
    const uint64_t strides[2] = {static_cast<uint64_t>(a.r_stride) * 2, 128};
    const uint32_t box[3] = {64, LP_TILE, static_cast<uint32_t>(rot_blocks)};
    if (!encode_map_bf16_sw128(&map_r, a.r, 3, dims, strides, box))
      return fail(ERR_RUNTIME, "%s: cannot encode the shared part's tensor map", name);
  }
  LatentUmmaParams p = {};
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.gate = static_cast<const __nv_bfloat16*>(a.gate);
  p.out_stride = a.out_stride, p.gate_stride = a.gate_stride, p.out_scale = a.out_scale;
  p.cu_q = a.cu_q, p.cu_k = a.cu_k, p.q_pos0 = a.q_pos0, p.k_pos0 = a.k_pos0;
  p.group = a.group, p.vdim = a.vdim, p.dim_blocks = dim_blocks, p.rot_blocks = rot_blocks;
  p.dim_steps = (a.true_dim + 15) / 16, p.rot_steps = (a.true_rot + 15) / 16;
  p.window = a.window;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.err = wait_timeout_flag();
  if (!p.err) return fail(ERR_RUNTIME, "%s: no error flag", name);
  const int k_bytes = (dim_blocks + rot_blocks) * LP_BLOCK_BYTES, v_bytes = a.vdim / 64 * LP_BLOCK_BYTES;
  p.k_stages = 2, p.v_stages = 2;
  auto smem_for = [&] { return k_bytes * (1 + p.k_stages) + v_bytes * p.v_stages + 1024; };
  if (smem_for() > LP_SMEM_LIMIT) p.v_stages = 1;
  if (smem_for() > LP_SMEM_LIMIT) p.k_stages = 1;
  int smem = smem_for();
  // the epilogue stages rows of vdim * 2 + 16 bytes over the operands
  if (smem < LP_TILE * (a.vdim * 2 + 16) + 1024) smem = LP_TILE * (a.vdim * 2 + 16) + 1024;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LP_SMEM_LIMIT) != cudaSuccess)
      return fail(ERR_RUNTIME, "%s: cannot raise dynamic shared memory to %d", name, LP_SMEM_LIMIT);
    configured[dev] = true;
  }
  latent_prefill_kernel<<<dim3((a.max_q + LP_TILE - 1) / LP_TILE, a.heads, a.batch), LP_THREADS, smem, st>>>(map_q, map_k, map_r,
                                                                                                            map_v, p);
  return check_launch(name);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_prefill(const void* q, const void* kv, const void* ctx, void* out, const int32_t* cu_q,
                                   const int32_t* cu_k, const int32_t* q_pos0, const int32_t* k_pos0, int32_t batch,
                                   int32_t max_q, int32_t tokens, int32_t keys, int32_t heads, int32_t dim, int32_t true_dim,
                                   int32_t rot, int32_t true_rot, int32_t vdim, int32_t rank, int32_t window, float scale,
                                   b200_stream_t stream) {
  if (batch <= 0 || max_q <= 0) return OK;
  B200_REQUIRE(dim > 0 && dim % 64 == 0 && rot > 0 && rank % 64 == 0 && true_rot > 0, "latent_prefill: sizes must be multiples of 64");
  const int64_t kv_row = static_cast<int64_t>(heads) * (dim + vdim), ctx_row = rank + rot;
  RowPrefillOperands a = {};
  a.q = q, a.q_stride = static_cast<int64_t>(heads) * (dim + rot);
  a.k = kv, a.k_stride = kv_row, a.k_head = dim;
  a.r = static_cast<const __nv_bfloat16*>(ctx) + rank, a.r_stride = ctx_row;
  a.v = static_cast<const __nv_bfloat16*>(kv) + static_cast<int64_t>(heads) * dim, a.v_stride = kv_row, a.v_head = vdim;
  a.out = out, a.out_stride = static_cast<int64_t>(heads) * vdim;
  a.cu_q = cu_q, a.cu_k = cu_k, a.q_pos0 = q_pos0, a.k_pos0 = k_pos0;
  a.batch = batch, a.max_q = max_q, a.tokens = tokens, a.keys = keys, a.heads = heads, a.group = 1;
  a.dim = dim, a.true_dim = true_dim, a.rot = rot, a.true_rot = true_rot, a.vdim = vdim, a.window = window;
  a.scale = scale, a.out_scale = 1.f;
  return row_prefill_launch(a, "latent_prefill", reinterpret_cast<cudaStream_t>(stream));
}
