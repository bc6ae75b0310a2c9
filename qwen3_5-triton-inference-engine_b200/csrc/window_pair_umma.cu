// Windowed causal attention of packed prompt portions for grouped heads of up to 128 + 128 dimensions, on tcgen05.
//
// Like latent_prefill_umma.cu, but a CTA works on 128 query tokens of TWO query heads that share a key/value head.  One head's
// softmax runs while the tensor cores work on the other's products, and a key tile is brought in once for both.  Per head h
// and tile of 128 keys:
//     S_h[128 x 128]   = Q_h . K^T           tcgen05.mma, both operands in shared memory
//     P_h              = exp2(S_h*scale - m) two softmax threads per row, TMEM -> registers -> TMEM (bf16 over S_h)
//     O_h[128 x vdim] += P_h . V             tcgen05.mma, P from TMEM, V as an MN-major operand
// TMEM is full with S and O of both heads, so S_h of the next tile is issued once P_h has been consumed; the other head's
// chain fills that time.  Roles: warps 0-7 / 8-15 softmax and epilogue of head 0 / 1, warp 16 issues MMAs, warps 17 / 18 load
// K (and Q) / V, double-buffered.  The running maximum may lag by 2^8 before O is rescaled.  Scores, maxima and sums are
// fp32.  The epilogue may multiply by sigmoid(gate) and a constant.  Every wait is bounded; on expiry the error flag is set
// and the CTA drains.
#include "latent.cuh"
#include "umma.cuh"

namespace b200 {

constexpr int WP_TILE = 128;
constexpr int WP_SOFTMAX_THREADS = 512;          // 256 per head
constexpr int WP_THREADS = 608;
constexpr int WP_BLOCK_BYTES = WP_TILE * 128;      // one 64-column block of 128 rows
constexpr uint32_t WP_TMEM_COLS = 512;             // S0 [0,128) S1 [128,256) O0 [256,384) O1 [384,512)
constexpr float WP_TAU = 8.0f;

struct WindowPairParams {
  __nv_bfloat16* out;
  const __nv_bfloat16* gate;
  int64_t out_stride, gate_stride;
  float out_scale;
  const int32_t *cu_q, *cu_k, *q_pos0, *k_pos0;
  int group, vdim, blocks, steps, window;          // column blocks and 16-wide steps of a key
  float scale_log2;
  int* err;
};

__global__ void __launch_bounds__(WP_THREADS, 1)
window_pair_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                   const __grid_constant__ CUtensorMap map_v, const __grid_constant__ WindowPairParams p) {
  extern __shared__ __align__(1024) uint8_t wp_smem_raw[];
  __shared__ uint64_t bar_q, bar_k[2], bar_v[2], free_k[2], free_v[2], bar_s[2], bar_p[2], bar_pv[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float xm[2][2][2][WP_TILE];             // [buffer][head][half][row]: what the two threads of a row tell each other
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qb = gridDim.x - 1 - blockIdx.x, h0 = blockIdx.y * 2, b = blockIdx.z, g = h0 / p.group;
  const int q_row0 = p.cu_q[b], len = p.cu_q[b + 1] - q_row0;
  const int q0 = qb * WP_TILE;
  if (q0 >= len) return;
  const int k_first = p.k_pos0[b];
  const int pos0 = p.q_pos0[b] + q0, pos_last = p.q_pos0[b] + min(q0 + WP_TILE, len) - 1;
  const int key0 = max(k_first, pos0 - p.window + 1);          // position of the first tile's first key
  const int n_tiles = (pos_last - key0) / WP_TILE + 1;
  const int k_row0 = p.cu_k[b] + key0 - k_first;               // its packed row

  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(wp_smem_raw) + 1023) & ~uintptr_t(1023));
  const int k_bytes = p.blocks * WP_BLOCK_BYTES, v_bytes = p.vdim / 64 * WP_BLOCK_BYTES;
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + 2 * k_bytes;
  uint8_t* v_s = k_s + 2 * k_bytes;

  if (warp == 0) tmem_alloc(&tmem_slot, WP_TMEM_COLS);
  if (tid == 17 * 32) {           // the thread that loads keys: queries and the first keys are under way before anything else
    prefetch_tensormap(&map_v);
    mbar_init(&bar_q, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar_k[i], 1);
      mbar_init(&bar_v[i], 1);
      mbar_init(&free_k[i], 1);
      mbar_init(&free_v[i], 1);
      mbar_init(&bar_s[i], 1);
      mbar_init(&bar_p[i], WP_SOFTMAX_THREADS / 2);
      mbar_init(&bar_pv[i], 1);
    }
    mbar_fence_init();
    mbar_expect_tx(&bar_k[0], k_bytes);
    tma_load_4d(k_s, &map_k, 0, k_row0, 0, g, &bar_k[0]);
    mbar_expect_tx(&bar_q, 2 * k_bytes);
    tma_load_4d(q_s, &map_q, 0, q_row0 + q0, 0, h0, &bar_q);
    tma_load_4d(q_s + k_bytes, &map_q, 0, q_row0 + q0, 0, h0 + 1, &bar_q);
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_slot;

  if (warp == 17) {
    if (lane == 0) {
      bool ok = true;
      for (int j = 1; j < n_tiles; ++j) {
        const int st = j & 1;
        if (j >= 2) ok = mbar_wait_bounded(&free_k[st], ((j - 2) >> 1) & 1);
        if (!ok) break;
        mbar_expect_tx(&bar_k[st], k_bytes);
        tma_load_4d(k_s + st * k_bytes, &map_k, 0, k_row0 + j * WP_TILE, 0, g, &bar_k[st]);
      }
      if (!ok) atomicExch(p.err, 1);
    }
  } else if (warp == 18) {
    if (lane == 0) {
      bool ok = true;
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j & 1;
        if (j >= 2) ok = mbar_wait_bounded(&free_v[st], ((j - 2) >> 1) & 1);
        if (!ok) break;
        mbar_expect_tx(&bar_v[st], v_bytes);
        tma_load_4d(v_s + st * v_bytes, &map_v, 0, k_row0 + j * WP_TILE, 0, g, &bar_v[st]);
      }
      if (!ok) atomicExch(p.err, 1);
    }
  } else if (warp == 16) {
    const bool leader = lane == 0;
    const uint32_t idesc_s = idesc_bf16_f32(128, WP_TILE, false, false);
    const uint32_t idesc_o = idesc_bf16_f32(128, p.vdim, false, true);
    const uint32_t q_addr = smem_u32(q_s), k_addr = smem_u32(k_s), v_addr = smem_u32(v_s);
    auto issue_s = [&](int h, int j) {
      const uint32_t q_h = q_addr + h * k_bytes, k_st = k_addr + (j & 1) * k_bytes;
      for (int ks = 0; ks < p.steps; ++ks) {
        const uint32_t o = (ks >> 2) * WP_BLOCK_BYTES + (ks & 3) * 32;
        umma_ss_leader(tmem + h * WP_TILE, smem_desc_sw128(q_h + o, 16, 1024), smem_desc_sw128(k_st + o, 16, 1024), idesc_s, ks > 0, leader);
      }
      umma_commit_leader(&bar_s[h], leader);
      if (h == 1) umma_commit_leader(&free_k[j & 1], leader);   // a commit covers everything issued before it
    };
    bool ok = mbar_wait_bounded(&bar_q, 0) && mbar_wait_bounded(&bar_k[0], 0);
    if (ok) {
      tc_fence_after_sync();
      issue_s(0, 0);
      issue_s(1, 0);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j & 1, next = (j + 1) & 1;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        ok = ok && mbar_wait_bounded(&bar_p[h], j & 1);
        if (h == 0) ok = ok && mbar_wait_bounded(&bar_v[st], (j >> 1) & 1);
        if (!ok) break;
        tc_fence_after_sync();
#pragma unroll
        for (int kt = 0; kt < WP_TILE / 16; ++kt)
          umma_ts_leader(tmem + 256 + h * 128, tmem + h * WP_TILE + kt * 8, smem_desc_sw128(v_addr + st * v_bytes + kt * 2048, WP_BLOCK_BYTES, 1024),
                         idesc_o, j > 0 || kt > 0, leader);
        umma_commit_leader(&bar_pv[h], leader);
        if (h == 1) umma_commit_leader(&free_v[st], leader);
        if (j + 1 < n_tiles) {
          if (h == 0) ok = ok && mbar_wait_bounded(&bar_k[next], ((j + 1) >> 1) & 1);
          ok = ok && mbar_wait_bounded(&bar_pv[h], j & 1);        // P has been consumed: S may be written again
          if (!ok) break;
          tc_fence_after_sync();
          issue_s(h, j + 1);
        }
      }
    }
    if (!ok && leader) atomicExch(p.err, 1);
  } else {
    const int h = warp >> 3, half = (warp >> 2) & 1, row = 32 * (warp & 3) + lane;
    const int pos = min(pos0 + row, pos_last);             // rows behind the end repeat the last query and are not stored
    const int col_lo = pos - p.window + 1 - key0, col_hi = pos - key0;  // visible columns over all tiles (col_lo may be < 0)
    const uint32_t lane_base = static_cast<uint32_t>(32 * (warp & 3)) << 16;
    const uint32_t s_addr = tmem + lane_base + h * WP_TILE, o_addr = tmem + lane_base + 256 + h * 128 + half * (p.vdim / 2);
    const int pair_bar = 1 + h * 4 + (warp & 3);           // the two warps that share rows
    const float sc = p.scale_log2;
    float m_ref = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      // `ok` stays uniform in the warp: what follows are warp-wide operations
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_s[h], j & 1));
      uint32_t r0[32], r1[32];
      float m_half = -INFINITY;
      if (ok) {
        tc_fence_after_sync();
        tmem_ld32(s_addr + half * 64, r0);
        tmem_ld32(s_addr + half * 64 + 32, r1);
        tmem_ld_wait();
        const int lo = col_lo - j * WP_TILE - half * 64, hi = col_hi - j * WP_TILE - half * 64;
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
      xm[j & 1][h][half][row] = m_half;
      named_barrier(pair_bar, 64);
      if (ok) {
        // the first tile starts at the block's first visible key, at most 127 columns in front of any row's own window:
        // every row sees at least one of its columns, so m_ref is finite from here on
        const float m_new = fmaxf(m_ref, fmaxf(m_half, xm[j & 1][h][half ^ 1][row]) * sc);
        if (j == 0) {
          m_ref = m_new;
        } else {
          const bool need = (m_new - m_ref) > WP_TAU;
          if (__any_sync(0xffffffffu, need)) {             // O is at rest: S of this tile was issued behind the last product
            const float alpha = need ? ex2_fast(m_ref - m_new) : 1.f;
            l_run *= alpha;
            if (need) m_ref = m_new;
#pragma unroll 1
            for (int c0 = 0; c0 < p.vdim / 2; c0 += 16) {
              uint32_t o[16];
              tmem_ld16(o_addr + c0, o);
              tmem_ld_wait();
#pragma unroll
              for (int c = 0; c < 16; ++c) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha);
              tmem_st16(o_addr + c0, o);
            }
          }
        }
        const F2 neg_m = f2(-m_ref, -m_ref), sc2 = f2(sc, sc);
        F2 sum[2] = {f2(0.f, 0.f), f2(0.f, 0.f)};
        // packed in place: a pair lands on a register whose score has been used
        auto pack = [&](uint32_t a, uint32_t b, int c) {
          const float2 x = unf2(fma2(f2(__uint_as_float(a), __uint_as_float(b)), sc2, neg_m));
          const float x0 = ex2_fast(x.x), x1 = ex2_fast(x.y);
          sum[c & 1] = add2(sum[c & 1], f2(x0, x1));
          return pack_bf16(x0, x1);
        };
#pragma unroll
        for (int c = 0; c < 16; ++c) r0[c] = pack(r0[2 * c], r0[2 * c + 1], c);
#pragma unroll
        for (int c = 0; c < 16; ++c) r0[16 + c] = pack(r1[2 * c], r1[2 * c + 1], c);
        const float2 total = unf2(add2(sum[0], sum[1]));
        l_run += total.x + total.y;
        tmem_st32(s_addr + half * 32, r0);
        tmem_st_wait();
      }
      tc_fence_before_sync();
      mbar_arrive(&bar_p[h]);
    }
    // ---- epilogue: O / l -> bf16 -> staged over the operands once both heads are done with them -> global.  The gates are
    // requested in front of the last product.
    const int vecs = p.vdim / 8, col = (h0 + h) * p.vdim, me = tid & 255;
    constexpr int U = 8;                                     // 16-byte pieces per thread at 128 value columns
    uint4 z[U];
    if (p.gate) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = me + u * 256, r = i / vecs;
        if (r < WP_TILE && q0 + r < len)
          z[u] = *reinterpret_cast<const uint4*>(p.gate + static_cast<int64_t>(q_row0 + q0 + r) * p.gate_stride + col + (i - r * vecs) * 8);
      }
    }
    float* xl = &xm[n_tiles & 1][h][0][0];
    xl[half * WP_TILE + row] = l_run;
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_pv[h], (n_tiles - 1) & 1));
    if (!ok && lane == 0) atomicExch(p.err, 1);
    named_barrier(9, WP_SOFTMAX_THREADS);
    const int out_pitch = p.vdim * 2 + 16;
    uint8_t* stage = smem + h * WP_TILE * out_pitch;
    if (ok) {
      tc_fence_after_sync();
      const float inv_l = 1.f / (l_run + xl[(half ^ 1) * WP_TILE + row]);
      uint8_t* orow = stage + row * out_pitch + half * p.vdim;
#pragma unroll 1
      for (int c0 = 0; c0 < p.vdim / 2; c0 += 16) {
        uint32_t o[16];
        tmem_ld16(o_addr + c0, o);
        tmem_ld_wait();
#pragma unroll
        for (int k8 = 0; k8 < 2; ++k8) {
          uint32_t w[4];
#pragma unroll
          for (int k = 0; k < 4; ++k)
            w[k] = pack_bf16(__uint_as_float(o[k8 * 8 + k * 2]) * inv_l, __uint_as_float(o[k8 * 8 + k * 2 + 1]) * inv_l);
          *reinterpret_cast<uint4*>(orow + (c0 + k8 * 8) * 2) = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
    named_barrier(10 + h, WP_SOFTMAX_THREADS / 2);
    if (ok) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = me + u * 256, r = i / vecs, c = i - r * vecs;
        if (r >= WP_TILE || q0 + r >= len) continue;
        uint4 o = *reinterpret_cast<const uint4*>(stage + r * out_pitch + c * 16);
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
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, WP_TMEM_COLS);
}

bool row_prefill_pairs(const RowPrefillOperands& a) { return a.group % 2 == 0 && a.rot == 0 && a.dim <= 128 && a.vdim <= 128; }

// `a` has passed row_prefill_launch's checks
int row_prefill_pair_launch(const RowPrefillOperands& a, const char* name, cudaStream_t st) {
  const int blocks = (a.dim + 63) / 64, kv_heads = a.heads / a.group;
  CUtensorMap map_q, map_k, map_v;
  if (!encode_head_map(&map_q, a.q, a.tokens, a.q_stride, blocks, a.dim, a.heads, WP_TILE) ||
      !encode_head_map(&map_k, a.k, a.keys, a.k_stride, blocks, a.k_head, kv_heads, WP_TILE) ||
      !encode_head_map(&map_v, a.v, a.keys, a.v_stride, a.vdim / 64, a.v_head, kv_heads, WP_TILE))
    return fail(ERR_RUNTIME, "%s: cannot encode a tensor map", name);
  WindowPairParams p = {};
  p.out = static_cast<__nv_bfloat16*>(a.out);
  p.gate = static_cast<const __nv_bfloat16*>(a.gate);
  p.out_stride = a.out_stride, p.gate_stride = a.gate_stride, p.out_scale = a.out_scale;
  p.cu_q = a.cu_q, p.cu_k = a.cu_k, p.q_pos0 = a.q_pos0, p.k_pos0 = a.k_pos0;
  p.group = a.group, p.vdim = a.vdim, p.blocks = blocks, p.steps = (a.true_dim + 15) / 16, p.window = a.window;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.err = wait_timeout_flag();
  if (!p.err) return fail(ERR_RUNTIME, "%s: no error flag", name);
  constexpr int limit = (4 * 2 + 2 * 2) * WP_BLOCK_BYTES + 1024;
  const int operands = (4 * blocks + 2 * (a.vdim / 64)) * WP_BLOCK_BYTES, staging = 2 * WP_TILE * (a.vdim * 2 + 16);
  const int smem = (operands > staging ? operands : staging) + 1024;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(window_pair_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, limit) != cudaSuccess)
      return fail(ERR_RUNTIME, "%s: cannot raise dynamic shared memory to %d", name, limit);
    configured[dev] = true;
  }
  window_pair_kernel<<<dim3((a.max_q + WP_TILE - 1) / WP_TILE, a.heads / 2, a.batch), WP_THREADS, smem, st>>>(map_q, map_k, map_v, p);
  return check_launch(name);
}

}  // namespace b200
