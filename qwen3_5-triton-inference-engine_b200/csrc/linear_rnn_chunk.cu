// Prefill of the forget-gated outer-product recurrence (HGRN2 form, linear_rnn.cu) in chunks of 16 tokens on the tensor
// cores, for bf16 activations and head sizes up to 128:
//     S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T q_t,   out = rms(o) * w per head
// With B_t = f_1 .. f_t and R_s = f_(s+1) .. f_16 inside a chunk (products of numbers <= 1: they can only shrink, no
// quotient of them is ever formed):
//     o_t    = S_0^T (q_t B_t) + sum_(s<=t) A_ts v_s,     A_ts = sum_d q_td (1 - f_sd) f_(s+1)d .. f_td
//     S_16^T = S_0^T diag(B_16) + V^T (K R),              K = 1 - f
// One CTA = one head of one sequence (and up to 128 value columns).  Three phases per chunk:
//   gates   silu, forget gates and biases of the chunk's raw rows (fetched into registers a chunk ahead) -> shared fp32
//   decays  running products forward (q B) and backward (K R) per channel; A on the CUDA cores in fp32, a warp per key
//           token with the decayed key carried in registers from query to query
//   mma     a warp owns 16 value columns of S^T as fp32 accumulators of m16n8k16; the same registers, split into bf16
//           high and low parts, are the B operand of (q B) S: no state leaves the registers between chunks.
// fp32 operands are carried as bf16 pairs (hi hi + hi lo + lo hi: relative error 2^-16); v is bf16 as it comes.
// When a CTA holds the whole head (vdim <= 128) the head norm is applied in place, else o goes to scratch in fp32.
#include "elem.cuh"
#include "linear_rnn.cuh"

namespace b200 {

constexpr int OC_C = 16;             // tokens per chunk
constexpr int OC_WARPS = 8;
constexpr int OC_THREADS = OC_WARPS * 32;
constexpr int OC_VCOLS = 16 * OC_WARPS;

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}

// D: channels incl. padding (32, 64 or 128).  grid (vdim / 128, heads, sequences)
template <int D>
__global__ void __launch_bounds__(OC_THREADS, 2) outer_rnn_chunk_kernel(const __grid_constant__ OuterRnnParams p) {
  constexpr int FP = D + 4;                         // fp32 row pitch
  constexpr int BP = D + 8;                         // bf16 row pitch (elements): ldmatrix rows in different banks
  constexpr int VP = OC_VCOLS + 8;
  constexpr int LC = D / 32;                        // channels per lane in the A phase
  constexpr int GROUPS = OC_THREADS / (D / 2);      // token groups of the gate phase (two channels per thread)
  constexpr int GT = OC_C / GROUPS > 0 ? OC_C / GROUPS : 1;
  __shared__ __align__(16) float fs[OC_C * FP], qs[OC_C * FP];
  __shared__ __align__(16) __nv_bfloat16 qh[OC_C * BP], ql[OC_C * BP], kh[OC_C * BP], kl[OC_C * BP];
  __shared__ __align__(16) __nv_bfloat16 vs[OC_C * VP];
  __shared__ __align__(16) float am[OC_C][OC_C + 2];
  __shared__ __align__(8) float bc[D];
  __shared__ float ssq[OC_WARPS][OC_C];
  const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * OC_VCOLS;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row0 = p.cu[seq], len = p.cu[seq + 1] - row0;
  if (len <= 0) return;
  const int hd = p.heads * p.dim;
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(p.qfv) + static_cast<int64_t>(row0) * p.stride;
  // gate phase: channels ch, ch + 1 of tokens grp * GT ..
  const int ch = (tid % (D / 2)) * 2, grp = tid / (D / 2);
  const bool gate_on = grp * GT < OC_C, ch_on = ch < p.dim;
  float low0 = 0.f, low1 = 0.f, fb0 = 0.f, fb1 = 0.f;
  if (ch_on) {
    low0 = p.lower[head * p.dim + ch], low1 = p.lower[head * p.dim + ch + 1];
    fb0 = p.bias[head * p.dim + ch], fb1 = p.bias[head * p.dim + ch + 1];
  }
  uint32_t rq[GT], rf[GT];
  uint4 rv;
  const int v_tok = tid / (OC_VCOLS / 8), v_col = (tid % (OC_VCOLS / 8)) * 8;
  const bool v_on = col0 + v_col < p.vdim;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < GT; ++i) {
      const int t = t0 + grp * GT + i;
      rq[i] = rf[i] = 0u;
      if (gate_on && ch_on && t < len) {
        const __nv_bfloat16* r = base + static_cast<int64_t>(t) * p.stride + head * p.dim + ch;
        rq[i] = *reinterpret_cast<const uint32_t*>(r);
        rf[i] = *reinterpret_cast<const uint32_t*>(r + hd);
      }
    }
    rv = make_uint4(0, 0, 0, 0);
    if (v_on && t0 + v_tok < len)
      rv = *reinterpret_cast<const uint4*>(base + static_cast<int64_t>(t0 + v_tok) * p.stride + 2 * hd + head * p.vdim + col0 + v_col);
  };
  // S^T: value column 16 * warp + lane / 4 (+ 8), channels 8 n + (lane % 4) * 2 (+ 1)
  float S[D / 8][4];
  float* st = p.state + (static_cast<int64_t>(p.slots[seq]) * p.heads + head) * p.dim * p.vdim;
  const int my_col = col0 + warp * 16 + (lane >> 2);
  const bool carry = p.start[seq] > 0;
#pragma unroll
  for (int n = 0; n < D / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      S[n][j] = carry && d < p.dim && c < p.vdim ? st[static_cast<int64_t>(d) * p.vdim + c] : 0.f;
    }
  float w0 = 0.f, w1 = 0.f, w2 = 0.f, w3 = 0.f;  // head-norm weights of this lane's output columns
  const int out_col = col0 + warp * 16 + (lane & 3) * 2;
  const bool fused_norm = p.out != nullptr;
  if (fused_norm && out_col < p.vdim) {
    w0 = p.norm[out_col], w1 = p.norm[out_col + 1];
    if (out_col + 8 < p.vdim) w2 = p.norm[out_col + 8], w3 = p.norm[out_col + 9];
  }
  const bool warp_on = col0 + warp * 16 < p.vdim;
  fetch(0);
  for (int t0 = 0; t0 < len; t0 += OC_C) {
    // ---- gates
    if (gate_on) {
#pragma unroll
      for (int i = 0; i < GT; ++i) {
        const int t = grp * GT + i;
        float2 q = make_float2(0.f, 0.f), f = make_float2(1.f, 1.f);   // padding keeps the state and reads nothing
        if (ch_on && t0 + t < len) {
          q = make_float2(silu_f<__nv_bfloat16>(bf16_lo(rq[i])), silu_f<__nv_bfloat16>(bf16_hi(rq[i])));
          f = make_float2(low0 + (1.0f - low0) * sigmoid_f<__nv_bfloat16>(bf16_lo(rf[i]) + fb0),
                          low1 + (1.0f - low1) * sigmoid_f<__nv_bfloat16>(bf16_hi(rf[i]) + fb1));
        }
        *reinterpret_cast<float2*>(fs + t * FP + ch) = f;
        *reinterpret_cast<float2*>(qs + t * FP + ch) = q;
      }
    }
    *reinterpret_cast<uint4*>(vs + v_tok * VP + v_col) = rv;
    if (t0 + OC_C < len) fetch(t0 + OC_C);
    __syncthreads();
    // ---- decays: forward products by the first D threads of each 2 * D, backward ones by the others
    for (int i = tid; i < 2 * D; i += OC_THREADS) {
      const int c = i % D;
      float run = 1.f;
      if (i < D) {
#pragma unroll
        for (int t = 0; t < OC_C; ++t) {
          run *= fs[t * FP + c];
          const float x = qs[t * FP + c] * run;
          const __nv_bfloat16 h = __float2bfloat16_rn(x);
          qh[t * BP + c] = h;
          ql[t * BP + c] = __float2bfloat16_rn(x - __bfloat162float(h));
        }
        bc[c] = run;
      } else {
#pragma unroll
        for (int t = OC_C - 1; t >= 0; --t) {
          const float f = fs[t * FP + c];
          const float x = (1.0f - f) * run;
          const __nv_bfloat16 h = __float2bfloat16_rn(x);
          kh[t * BP + c] = h;
          kl[t * BP + c] = __float2bfloat16_rn(x - __bfloat162float(h));
          run *= f;
        }
      }
    }
    // ---- A: key tokens warp and 15 - warp (17 pairs together)
#pragma unroll
    for (int which = 0; which < 2; ++which) {
      const int s = which ? OC_C - 1 - warp : warp;
      float g[LC], a[OC_C];
#pragma unroll
      for (int c = 0; c < LC; ++c) g[c] = 1.0f - fs[s * FP + lane * LC + c];
#pragma unroll
      for (int t = 0; t < OC_C; ++t) {
        a[t] = 0.f;
        if (t >= s) {
#pragma unroll
          for (int c = 0; c < LC; ++c) {
            if (t > s) g[c] *= fs[t * FP + lane * LC + c];
            a[t] = fmaf(qs[t * FP + lane * LC + c], g[c], a[t]);
          }
        }
      }
#pragma unroll
      for (int half = 8, bit = 16; half >= 1; half >>= 1, bit >>= 1) {
        const bool upper = (lane & bit) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
          const float give = upper ? a[i] : a[i + half];
          const float keep = upper ? a[i + half] : a[i];
          a[i] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
        }
      }
      a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
      if ((lane & 1) == 0) am[lane >> 1][s] = a[0];
    }
    __syncthreads();
    // ---- products
    float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    uint32_t vm[4];   // the chunk's values of this warp's columns: matrices (k 0-7, c 0-7), (k 0-7, c 8-15), (k 8-15, ...)
    if (warp_on) {
      ldmatrix_x4_trans(vm, smem_u32(vs + ((lane & 7) + (lane >> 4) * 8) * VP + warp * 16 + ((lane >> 3) & 1) * 8));
      const uint32_t a_off = ((lane & 15) * BP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, smem_u32(qh) + a_off + ks * 32);
        ldmatrix_x4(al, smem_u32(ql) + a_off + ks * 32);
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
        const float2 x = *reinterpret_cast<const float2*>(&am[(lane >> 2) + (i & 1) * 8][(lane & 3) * 2 + (i >> 1) * 8]);
        split_pair(x.x, x.y, xh[i], xl[i]);
      }
      mma_bf16_16816(o[0], xh, vm[0], vm[2]);
      mma_bf16_16816(o[0], xl, vm[0], vm[2]);
      mma_bf16_16816(o[1], xh, vm[1], vm[3]);
      mma_bf16_16816(o[1], xl, vm[1], vm[3]);
      // S^T <- S^T diag(B) + V^T (K R)
      const uint32_t k_off = ((lane & 15) * BP + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int n = 0; n < D / 8; n += 2) {
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, smem_u32(kh) + k_off + n * 16);
        ldmatrix_x4_trans(bl, smem_u32(kl) + k_off + n * 16);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float2 d = *reinterpret_cast<const float2*>(bc + (n + i) * 8 + (lane & 3) * 2);
          S[n + i][0] *= d.x, S[n + i][1] *= d.y, S[n + i][2] *= d.x, S[n + i][3] *= d.y;
          mma_bf16_16816(S[n + i], vm, bh[2 * i], bh[2 * i + 1]);
          mma_bf16_16816(S[n + i], vm, bl[2 * i], bl[2 * i + 1]);
        }
      }
    }
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
        ssq[warp][lane >> 2] = s_lo;
        ssq[warp][(lane >> 2) + 8] = s_hi;
      }
      __syncthreads();
      s_lo = s_hi = 0.f;
#pragma unroll
      for (int w = 0; w < OC_WARPS; ++w) {
        s_lo += ssq[w][lane >> 2];
        s_hi += ssq[w][(lane >> 2) + 8];
      }
      const float r_lo = 1.0f / sqrtf(s_lo / static_cast<float>(p.true_vdim) + p.eps);
      const float r_hi = 1.0f / sqrtf(s_hi / static_cast<float>(p.true_vdim) + p.eps);
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(row0) * p.heads * p.vdim + head * p.vdim + out_col;
      const int64_t step = static_cast<int64_t>(p.heads) * p.vdim;
      if (out_col < p.vdim) {
        if (t_lo < len) *reinterpret_cast<uint32_t*>(out + t_lo * step) = pack_bf16(o[0][0] * r_lo * w0, o[0][1] * r_lo * w1);
        if (t_hi < len) *reinterpret_cast<uint32_t*>(out + t_hi * step) = pack_bf16(o[0][2] * r_hi * w0, o[0][3] * r_hi * w1);
      }
      if (out_col + 8 < p.vdim) {
        if (t_lo < len) *reinterpret_cast<uint32_t*>(out + t_lo * step + 8) = pack_bf16(o[1][0] * r_lo * w2, o[1][1] * r_lo * w3);
        if (t_hi < len) *reinterpret_cast<uint32_t*>(out + t_hi * step + 8) = pack_bf16(o[1][2] * r_hi * w2, o[1][3] * r_hi * w3);
      }
    } else {
      float* out = p.o + static_cast<int64_t>(row0) * p.heads * p.vdim + head * p.vdim + out_col;
      const int64_t step = static_cast<int64_t>(p.heads) * p.vdim;
#pragma unroll
      for (int n = 0; n < 2; ++n)
        if (out_col + n * 8 < p.vdim) {
          if (t_lo < len) *reinterpret_cast<float2*>(out + t_lo * step + n * 8) = make_float2(o[n][0], o[n][1]);
          if (t_hi < len) *reinterpret_cast<float2*>(out + t_hi * step + n * 8) = make_float2(o[n][2], o[n][3]);
        }
      __syncthreads();  // everybody has read this chunk's operands
    }
  }
#pragma unroll
  for (int n = 0; n < D / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      if (d < p.dim && c < p.vdim) st[static_cast<int64_t>(d) * p.vdim + c] = S[n][j];
    }
}

bool outer_rnn_chunk_supports(int dim, int vdim) { return dim <= 128 && dim % 2 == 0 && vdim % 8 == 0; }

int outer_rnn_chunk_launch(const OuterRnnParams& p, int n, cudaStream_t st) {
  const dim3 grid((p.vdim + OC_VCOLS - 1) / OC_VCOLS, p.heads, n);
  if (p.dim <= 32) outer_rnn_chunk_kernel<32><<<grid, OC_THREADS, 0, st>>>(p);
  else if (p.dim <= 64) outer_rnn_chunk_kernel<64><<<grid, OC_THREADS, 0, st>>>(p);
  else outer_rnn_chunk_kernel<128><<<grid, OC_THREADS, 0, st>>>(p);
  return check_launch("hgrn2_prefill (chunks)");
}

}  // namespace b200
