// Prefill of the outer-product recurrences with a decay per key channel (linear_rnn.cuh, FORGET and KEYED) in chunks of 16
// tokens on the tensor cores, for bf16 activations and head sizes up to 128:
//     S_t = diag(f_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out = rms(o) * w (* silu(gate)) per head
// With B_t = f_1 .. f_t and R_s = f_(s+1) .. f_16 inside a chunk (products of numbers <= 1: they can only shrink, no
// quotient of them is ever formed):
//     o_t    = S_0^T (q_t B_t) + sum_(s<=t) A_ts v_s,     A_ts = sum_d q_td k_sd f_(s+1)d .. f_td
//     S_16^T = S_0^T diag(B_16) + V^T (K R),              FORGET: k = 1 - f
// One CTA = one head of one sequence (and up to 128 value columns).  Per chunk:
//   gates   activations, decays and biases of the chunk's raw rows (brought in by cp.async a chunk ahead) -> shared fp32
//   decays  running products forward (q B) and backward (K R) per channel, by half of the warps; A on the CUDA cores in
//           fp32, half a warp per key token with the decayed key carried in registers from query to query
//   mma     a warp owns 16 value columns of S^T as fp32 accumulators of m16n8k16; the same registers, split into bf16
//           high and low parts, are the B operand of (q B) S: no state leaves the registers between chunks.
// fp32 operands are carried as bf16 pairs (hi hi + hi lo + lo hi: relative error 2^-16); v is bf16 as it comes.
// When a CTA holds the whole head (vdim <= 128) the head norm is applied in place, else o goes to scratch in fp32.
//
// Few heads and long sequences leave most SMs idle, so sequences may be cut into segments: a first launch leaves every
// segment's state from zero and its channels' total decay, a small kernel turns those into the state each segment starts
// from (S <- diag(decay) S + local, in order), and the main launch runs all segments at once.
#include "elem.cuh"
#include "linear_rnn.cuh"

namespace b200 {

constexpr int OC_C = 16;             // tokens per chunk
constexpr int OC_WARPS = 8;
constexpr int OC_THREADS = OC_WARPS * 32;
constexpr int OC_VCOLS = 16 * OC_WARPS;
constexpr int OC_VP = OC_VCOLS + 8;  // bf16 pitch of the value rows

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
__device__ __forceinline__ void split_store(__nv_bfloat16* hi, __nv_bfloat16* lo, float x) {
  const __nv_bfloat16 h = __float2bfloat16_rn(x);
  *hi = h;
  *lo = __float2bfloat16_rn(x - __bfloat162float(h));
}
// 16 bytes global -> shared without registers; nothing is read (zeros are written) when `on` is false
__device__ __forceinline__ void cp_async16_or_zero(void* dst, const void* src, bool on) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

template <int D, bool KEYED>
struct ChunkSmem {
  static constexpr int FP = D + 4;   // fp32 row pitch
  static constexpr int BP = D + 8;   // bf16 row pitch: ldmatrix rows in different banks
  float fs[OC_C * FP], qs[OC_C * FP];
  __nv_bfloat16 qh[OC_C * BP], ql[OC_C * BP], kh[OC_C * BP], kl[OC_C * BP];
  __nv_bfloat16 raw[2][OC_C * D];    // the next chunk's q and f' (KEYED: k) rows as they come
  float ks[KEYED ? OC_C * FP : 4], zs[KEYED ? OC_C * D : 4];   // keys; the next chunk's z rows
  __nv_bfloat16 vs[2][OC_C * OC_VP];
  float am[OC_C][OC_C + 2];
  float bc[D], total[D];
  float ssq[OC_WARPS][OC_C];
};

// D: channels incl. padding (32, 64 or 128).  LOCAL: only the state from zero and the total decay of every segment.
// grid (vdim / 128, heads, sequences * segments)
template <int D, bool LOCAL, bool KEYED>
__global__ void __launch_bounds__(OC_THREADS, 2) outer_rnn_chunk_kernel(const __grid_constant__ OuterRnnParams p) {
  using Smem = ChunkSmem<D, KEYED>;
  constexpr int FP = Smem::FP, BP = Smem::BP;
  constexpr int ROW_VECS = D / 8, V_VECS = OC_VCOLS / 8;
  extern __shared__ __align__(16) uint8_t oc_smem[];
  Smem& sm = *reinterpret_cast<Smem*>(oc_smem);
  const int seq = blockIdx.z / p.segments, seg = blockIdx.z % p.segments, head = blockIdx.y, col0 = blockIdx.x * OC_VCOLS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int all = p.cu[seq + 1] - p.cu[seq], seg0 = seg * p.segment;
  const int row0 = p.cu[seq] + seg0, len = min(all - seg0, p.segment);
  if (len <= 0 || (LOCAL && seg0 + len == all)) return;  // nothing follows a sequence's last segment
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(p.x) + static_cast<int64_t>(row0) * p.stride;
  auto fetch = [&](int t0, int buf) {
    for (int i = tid; i < OC_C * ROW_VECS; i += OC_THREADS) {
      const int t = i / ROW_VECS, c = (i % ROW_VECS) * 8;
      const bool on = t0 + t < len && c < p.dim;
      const __nv_bfloat16* r = base + static_cast<int64_t>(on ? t0 + t : 0) * p.stride + head * p.dim + (on ? c : 0);
      if (!LOCAL) cp_async16_or_zero(&sm.raw[0][t * D + c], r + p.q_off, on);
      cp_async16_or_zero(&sm.raw[1][t * D + c], r + p.k_off, on);
    }
    if constexpr (KEYED) {
      for (int i = tid; i < OC_C * (D / 4); i += OC_THREADS) {
        const int t = i / (D / 4), c = (i % (D / 4)) * 4;
        const bool on = t0 + t < len && c < p.dim;
        cp_async16_or_zero(&sm.zs[t * D + c], p.z + static_cast<int64_t>(row0 + (on ? t0 + t : 0)) * p.z_stride + head * p.dim + (on ? c : 0), on);
      }
    }
    const int t = tid / V_VECS, c = (tid % V_VECS) * 8;
    const bool on = t0 + t < len && col0 + c < p.vdim;
    cp_async16_or_zero(&sm.vs[buf][t * OC_VP + c],
                       base + static_cast<int64_t>(on ? t0 + t : 0) * p.stride + p.v_off + head * p.vdim + (on ? col0 + c : 0), on);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  // gate phase: channels ch, ch + 1 of every (2 * OC_THREADS / D)-th token
  constexpr int GROUPS = 2 * OC_THREADS / D;
  const int ch = (tid % (D / 2)) * 2, grp = tid / (D / 2);
  float low0 = 0.f, low1 = 0.f, fb0 = 0.f, fb1 = 0.f;
  if (ch < p.dim) {
    if (!KEYED) low0 = p.lower[head * p.dim + ch], low1 = p.lower[head * p.dim + ch + 1];
    fb0 = p.bias[head * p.dim + ch], fb1 = p.bias[head * p.dim + ch + 1];
  }
  for (int i = tid; i < OC_C * (OC_C + 2); i += OC_THREADS) (&sm.am[0][0])[i] = 0.f;  // A above the diagonal stays zero
  if (LOCAL && tid < D) sm.total[tid] = 1.f;
  // S^T: value column 16 * warp + lane / 4 (+ 8), channels 8 n + (lane % 4) * 2 (+ 1)
  float S[D / 8][4];
  const int64_t head_elems = static_cast<int64_t>(p.dim) * p.vdim;
  float* slot_state = p.state + (static_cast<int64_t>(p.slots[seq]) * p.heads + head) * head_elems;
  float* seg_state = p.seg_state + (static_cast<int64_t>(blockIdx.z) * p.heads + head) * head_elems;
  const float* from = p.segments > 1 ? seg_state : slot_state;
  const bool carry = !LOCAL && (p.segments > 1 || p.start[seq] > 0);
  const int my_col = col0 + warp * 16 + (lane >> 2);
#pragma unroll
  for (int n = 0; n < D / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      S[n][j] = carry && d < p.dim && c < p.vdim ? from[static_cast<int64_t>(d) * p.vdim + c] : 0.f;
    }
  const int out_col = col0 + warp * 16 + (lane & 3) * 2;
  const bool fused_norm = p.out != nullptr, warp_on = col0 + warp * 16 < p.vdim;
  float w0 = 0.f, w1 = 0.f, w2 = 0.f, w3 = 0.f;  // head-norm weights of this lane's output columns
  if (!LOCAL && fused_norm && out_col < p.vdim) {
    w0 = p.norm[out_col], w1 = p.norm[out_col + 1];
    if (out_col + 8 < p.vdim) w2 = p.norm[out_col + 8], w3 = p.norm[out_col + 9];
  }
  for (int t0 = 0, buf = 0; t0 < len; t0 += OC_C, buf ^= 1) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // the chunk's rows are here; everybody is done with the previous chunk
    // ---- gates
    for (int t = grp; t < OC_C; t += GROUPS) {
      float2 q = make_float2(0.f, 0.f), f = make_float2(1.f, 1.f), k = q;   // padding keeps the state and reads nothing
      if (ch < p.dim && t0 + t < len) {
        const uint32_t rf = *reinterpret_cast<const uint32_t*>(&sm.raw[1][t * D + ch]);
        if constexpr (KEYED) {
          const float2 z = *reinterpret_cast<const float2*>(&sm.zs[t * D + ch]);
          f = make_float2(sigmoid_root<__nv_bfloat16>(z.x + fb0, p.inv_tau), sigmoid_root<__nv_bfloat16>(z.y + fb1, p.inv_tau));
          k = make_float2(bf16_lo(rf), bf16_hi(rf));
        } else {
          f = make_float2(low0 + (1.0f - low0) * sigmoid_f<__nv_bfloat16>(bf16_lo(rf) + fb0),
                          low1 + (1.0f - low1) * sigmoid_f<__nv_bfloat16>(bf16_hi(rf) + fb1));
        }
        if (!LOCAL) {
          const uint32_t rq = *reinterpret_cast<const uint32_t*>(&sm.raw[0][t * D + ch]);
          if constexpr (KEYED) q = make_float2(bf16_lo(rq) * p.q_scale, bf16_hi(rq) * p.q_scale);
          else q = make_float2(silu_f<__nv_bfloat16>(bf16_lo(rq)), silu_f<__nv_bfloat16>(bf16_hi(rq)));
        }
      }
      if constexpr (KEYED) *reinterpret_cast<float2*>(&sm.ks[t * FP + ch]) = k;
      *reinterpret_cast<float2*>(&sm.fs[t * FP + ch]) = f;
      if (!LOCAL) *reinterpret_cast<float2*>(&sm.qs[t * FP + ch]) = q;
    }
    __syncthreads();
    if (t0 + OC_C < len) fetch(t0 + OC_C, buf ^ 1);
    // ---- decays, by the warps with the fewest pairs below: backward (K R), then forward (q B) of a channel
    if (LOCAL || warp >= OC_WARPS / 2) {
      for (int c = LOCAL ? tid : tid - OC_THREADS / 2; c < D; c += LOCAL ? OC_THREADS : OC_THREADS / 2) {
        float f[OC_C], run = 1.f;
#pragma unroll
        for (int t = 0; t < OC_C; ++t) f[t] = sm.fs[t * FP + c];
#pragma unroll
        for (int t = OC_C - 1; t >= 0; --t) {
          split_store(&sm.kh[t * BP + c], &sm.kl[t * BP + c], (KEYED ? sm.ks[t * FP + c] : 1.0f - f[t]) * run);
          run *= f[t];
        }
        sm.bc[c] = run;
        if (LOCAL) {
          sm.total[c] *= run;
        } else {
          run = 1.f;
#pragma unroll
          for (int t = 0; t < OC_C; ++t) {
            run *= f[t];
            split_store(&sm.qh[t * BP + c], &sm.ql[t * BP + c], sm.qs[t * FP + c] * run);
          }
        }
      }
    }
    // ---- A: key token s per half warp, a lane every 16th group of channels
    if (!LOCAL) {
      constexpr int LC = D / 16;                       // channels per lane
      constexpr int W = LC >= 4 ? 4 : LC;              // ... in groups of W
      const int s = 2 * warp + (lane >> 4), hl = lane & 15;
      float g[LC];
      auto row = [&](const float* src, int t, float (&x)[LC]) {
#pragma unroll
        for (int k = 0; k < LC / W; ++k)
          if constexpr (W == 4) {
            const float4 a = *reinterpret_cast<const float4*>(src + t * FP + k * 64 + hl * 4);
            x[k * 4] = a.x, x[k * 4 + 1] = a.y, x[k * 4 + 2] = a.z, x[k * 4 + 3] = a.w;
          } else {
            const float2 a = *reinterpret_cast<const float2*>(src + t * FP + hl * 2);
            x[0] = a.x, x[1] = a.y;
          }
      };
      row(KEYED ? sm.ks : sm.fs, s, g);
      if (!KEYED) {
#pragma unroll
        for (int c = 0; c < LC; ++c) g[c] = 1.0f - g[c];
      }
#pragma unroll 4
      for (int t = 2 * warp; t < OC_C; ++t) {
        float f[LC], q[LC];
        row(sm.fs, t, f);
        row(sm.qs, t, q);
        float a0 = 0.f, a1 = 0.f;
#pragma unroll
        for (int c = 0; c < LC; c += 2) {
          g[c] *= t > s ? f[c] : 1.f;
          g[c + 1] *= t > s ? f[c + 1] : 1.f;
          a0 = fmaf(q[c], g[c], a0);
          a1 = fmaf(q[c + 1], g[c + 1], a1);
        }
        a0 += a1;
#pragma unroll
        for (int bit = 8; bit >= 1; bit >>= 1) a0 += __shfl_xor_sync(0xffffffffu, a0, bit);
        if (hl == 0 && t >= s) sm.am[t][s] = a0;
      }
    }
    __syncthreads();
    // ---- products
    float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    if (warp_on) {
      uint32_t vm[4];   // the chunk's values of this warp's columns: matrices (k 0-7, c 0-7), (k 0-7, c 8-15), (k 8-15, ...)
      ldmatrix_x4_trans(vm, smem_u32(&sm.vs[buf][((lane & 7) + (lane >> 4) * 8) * OC_VP + warp * 16 + ((lane >> 3) & 1) * 8]));
      const uint32_t a_off = ((lane & 15) * BP + (lane >> 4) * 8) * 2;
      if (!LOCAL) {
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          uint32_t ah[4], al[4];
          ldmatrix_x4(ah, smem_u32(sm.qh) + a_off + ks * 32);
          ldmatrix_x4(al, smem_u32(sm.ql) + a_off + ks * 32);
#pragma unroll
          for (int n = 0; n < 2; ++n) {               // value columns 0-7 and 8-15 of the warp
            uint32_t h0, l0, h1, l1;
            split_pair(S[2 * ks][2 * n], S[2 * ks][2 * n + 1], h0, l0);
            split_pair(S[2 * ks + 1][2 * n], S[2 * ks + 1][2 * n + 1], h1, l1);
            mma_bf16_16816(o[n], ah, h0, h1);
            mma_bf16_16816(o[n], ah, l0, l1);
            mma_bf16_16816(o[n], al, h0, h1);
          }
        }
        uint32_t xh[4], xl[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 x = *reinterpret_cast<const float2*>(&sm.am[(lane >> 2) + (i & 1) * 8][(lane & 3) * 2 + (i >> 1) * 8]);
          split_pair(x.x, x.y, xh[i], xl[i]);
        }
        mma_bf16_16816(o[0], xh, vm[0], vm[2]);
        mma_bf16_16816(o[0], xl, vm[0], vm[2]);
        mma_bf16_16816(o[1], xh, vm[1], vm[3]);
        mma_bf16_16816(o[1], xl, vm[1], vm[3]);
      }
      // S^T <- S^T diag(B) + V^T (K R)
#pragma unroll
      for (int n = 0; n < D / 8; n += 2) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, smem_u32(sm.kh) + a_off + n * 16);
        ldmatrix_x4_trans(bl, smem_u32(sm.kl) + a_off + n * 16);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float2 d = *reinterpret_cast<const float2*>(&sm.bc[(n + i) * 8 + (lane & 3) * 2]);
          S[n + i][0] *= d.x, S[n + i][1] *= d.y, S[n + i][2] *= d.x, S[n + i][3] *= d.y;
          mma_bf16_16816(S[n + i], vm, bh[2 * i], bh[2 * i + 1]);
          mma_bf16_16816(S[n + i], vm, bl[2 * i], bl[2 * i + 1]);
        }
      }
    }
    if (LOCAL) continue;
    // ---- output rows lane / 4 and + 8, columns out_col (+ 1), + 8 (+ 9)
    const int t_lo = t0 + (lane >> 2), t_hi = t_lo + 8;
    if (fused_norm) {
      float s_lo = o[0][0] * o[0][0] + o[0][1] * o[0][1] + o[1][0] * o[1][0] + o[1][1] * o[1][1];
      float s_hi = o[0][2] * o[0][2] + o[0][3] * o[0][3] + o[1][2] * o[1][2] + o[1][3] * o[1][3];
#pragma unroll
      for (int bit = 1; bit <= 2; bit <<= 1) {
        s_lo += __shfl_xor_sync(0xffffffffu, s_lo, bit);
        s_hi += __shfl_xor_sync(0xffffffffu, s_hi, bit);
      }
      if ((lane & 3) == 0) {
        sm.ssq[warp][lane >> 2] = s_lo;
        sm.ssq[warp][(lane >> 2) + 8] = s_hi;
      }
      __syncthreads();
      s_lo = s_hi = 0.f;
#pragma unroll
      for (int w = 0; w < OC_WARPS; ++w) {
        s_lo += sm.ssq[w][lane >> 2];
        s_hi += sm.ssq[w][(lane >> 2) + 8];
      }
      const float r_lo = 1.0f / sqrtf(s_lo / static_cast<float>(p.true_vdim) + p.eps);
      const float r_hi = 1.0f / sqrtf(s_hi / static_cast<float>(p.true_vdim) + p.eps);
      const int col = head * p.vdim + out_col;
      auto put = [&](int t, int c, float x, float y) {
        if (p.gate) {
          const uint32_t g = *reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(p.gate) + (row0 + t) * p.gate_stride + c);
          x *= silu_f<__nv_bfloat16>(bf16_lo(g)), y *= silu_f<__nv_bfloat16>(bf16_hi(g));
        }
        *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(p.out) + (row0 + t) * p.out_stride + c) = pack_bf16(x, y);
      };
      if (out_col < p.vdim) {
        if (t_lo < len) put(t_lo, col, o[0][0] * r_lo * w0, o[0][1] * r_lo * w1);
        if (t_hi < len) put(t_hi, col, o[0][2] * r_hi * w0, o[0][3] * r_hi * w1);
      }
      if (out_col + 8 < p.vdim) {
        if (t_lo < len) put(t_lo, col + 8, o[1][0] * r_lo * w2, o[1][1] * r_lo * w3);
        if (t_hi < len) put(t_hi, col + 8, o[1][2] * r_hi * w2, o[1][3] * r_hi * w3);
      }
    } else {
      const int64_t step = static_cast<int64_t>(p.heads) * p.vdim;
      float* out = p.o + static_cast<int64_t>(row0) * step + head * p.vdim + out_col;
#pragma unroll
      for (int n = 0; n < 2; ++n)
        if (out_col + n * 8 < p.vdim) {
          if (t_lo < len) *reinterpret_cast<float2*>(out + t_lo * step + n * 8) = make_float2(o[n][0], o[n][1]);
          if (t_hi < len) *reinterpret_cast<float2*>(out + t_hi * step + n * 8) = make_float2(o[n][2], o[n][3]);
        }
    }
  }
  if (!LOCAL && seg0 + len < all) return;              // only the last segment leaves the sequence's state behind
  float* to = LOCAL ? seg_state : slot_state;
#pragma unroll
  for (int n = 0; n < D / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      if (d < p.dim && c < p.vdim) to[static_cast<int64_t>(d) * p.vdim + c] = S[n][j];
    }
  if (LOCAL && blockIdx.x == 0) {
    __syncthreads();
    if (tid < p.dim) p.seg_decay[(static_cast<int64_t>(blockIdx.z) * p.heads + head) * p.dim + tid] = sm.total[tid];
  }
}

// Local states and decays of the segments -> the state every segment starts from, in place; four columns per thread.
// grid (dim * vdim / 1024, heads, sequences)
__global__ void __launch_bounds__(256) outer_rnn_fold_kernel(const __grid_constant__ OuterRnnParams p) {
  const int seq = blockIdx.z, head = blockIdx.y, e = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (e >= p.dim * p.vdim) return;
  const int d = e / p.vdim, all = p.cu[seq + 1] - p.cu[seq], used = (all + p.segment - 1) / p.segment;
  const int64_t head_elems = static_cast<int64_t>(p.dim) * p.vdim;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.start[seq] > 0) s = load4(p.state + (static_cast<int64_t>(p.slots[seq]) * p.heads + head) * head_elems + e);
  for (int i = 0; i < used; ++i) {
    const int64_t at = (static_cast<int64_t>(seq) * p.segments + i) * p.heads + head;
    float* x = p.seg_state + at * head_elems + e;
    float4 local = make_float4(0.f, 0.f, 0.f, 0.f);
    float f = 0.f;
    if (i + 1 < used) {
      local = load4(x);
      f = p.seg_decay[at * p.dim + d];
    }
    store4(x, s);
    s = make_float4(fmaf(f, s.x, local.x), fmaf(f, s.y, local.y), fmaf(f, s.z, local.z), fmaf(f, s.w, local.w));
  }
}

bool outer_rnn_chunk_supports(int dim, int vdim) { return dim <= 128 && dim % 8 == 0 && vdim % 8 == 0; }

void outer_rnn_fold_launch(const OuterRnnParams& p, int n, cudaStream_t st) {
  outer_rnn_fold_kernel<<<dim3((p.dim * p.vdim / 4 + 255) / 256, p.heads, n), 256, 0, st>>>(p);
}

template <int D, bool KEYED>
static int launch_chunks(const OuterRnnParams& p, int n, cudaStream_t st) {
  constexpr int smem = sizeof(ChunkSmem<D, KEYED>);
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(outer_rnn_chunk_kernel<D, false, KEYED>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
        cudaFuncSetAttribute(outer_rnn_chunk_kernel<D, true, KEYED>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return fail(ERR_RUNTIME, "outer_rnn: cannot raise dynamic shared memory to %d", smem);
    configured[dev] = true;
  }
  const dim3 grid((p.vdim + OC_VCOLS - 1) / OC_VCOLS, p.heads, n * p.segments);
  if (p.segments > 1) {
    outer_rnn_chunk_kernel<D, true, KEYED><<<grid, OC_THREADS, smem, st>>>(p);
    outer_rnn_fold_launch(p, n, st);
  }
  outer_rnn_chunk_kernel<D, false, KEYED><<<grid, OC_THREADS, smem, st>>>(p);
  return check_launch("outer_rnn (chunks)");
}

int outer_rnn_chunk_launch(const OuterRnnParams& p, RnnKind kind, int n, cudaStream_t st) {
  if (kind == RNN_KEYED) {
    if (p.dim <= 32) return launch_chunks<32, true>(p, n, st);
    if (p.dim <= 64) return launch_chunks<64, true>(p, n, st);
    return launch_chunks<128, true>(p, n, st);
  }
  if (p.dim <= 32) return launch_chunks<32, false>(p, n, st);
  if (p.dim <= 64) return launch_chunks<64, false>(p, n, st);
  return launch_chunks<128, false>(p, n, st);
}

}  // namespace b200
