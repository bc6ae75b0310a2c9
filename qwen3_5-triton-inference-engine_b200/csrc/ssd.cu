// State-space mixer with one decay per head and token around its projections (linear_rnn.cuh, SSD): the causal convolution of
// its inputs, the recurrence
//     S_t = a_t S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   a_t = exp(-exp(A) dt_t)
// and the gated norm over groups of channels behind it.
//   b200_conv_prefill        any number of taps up to 16, bias, silu; reads and leaves a ring of raw inputs per slot
//   b200_ssd_prefill         bf16, up to 128 state rows: chunks of 32 tokens on the tensor cores (here); else token by token
//                            (linear_rnn.cu)
//   b200_ssd_decode          convolution and recurrence of one token per slot in one launch (linear_rnn.cu)
//   b200_gated_group_norm    y silu(z), RMS norm in equal parts of the channels, weight
//
// Chunked form.  With L_t = log a_1 + .. + log a_t inside a chunk (all <= 0) and E = the chunk's last token:
//     y_t  = exp(L_t) S_0^T C_t + sum_(s<=t) exp(L_t - L_s) dt_s (C_t . B_s) x_s + D x_t
//     S_E  = exp(L_E) S_0 + sum_s B_s (exp(L_E - L_s) dt_s x_s)^T
// One CTA = up to 128 value columns: part of a head, or several heads of a group, which share C B^T.  Per chunk:
//   decays   a warp per head scans the 32 tokens; meanwhile all warps compute C B^T (mma.sync, 16 x 8 tiles, fp32)
//   weights  the weighted 32 x 32 matrix per head and the weighted x, as bf16 pairs (hi + lo: relative error 2^-16)
//   mma      a warp owns 16 value columns of S^T as fp32 accumulators of m16n8k16; the same registers, split into pairs, are
//            the B operand of C S: no state leaves the registers between chunks.
// B, C and x are bf16 as the convolution leaves them.  Few heads and long sequences: segments side by side (state from zero
// and total decay of every segment, outer_rnn_fold_kernel, main pass).
#include "linear_rnn.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------------------ convolution
constexpr int CV_THREADS = 64;    // 8 channels each

struct ConvParams {
  const void* x;              // [rows, stride] E
  int64_t stride;
  const float *w, *bias;      // [T, channels] (first row: the current token's weight), [channels]
  float* ring;                // [slots, T, channels]: the input of position p at p % T
  const int32_t *cu, *slots, *start;
  void* out;                  // [rows, out_stride] E
  int64_t out_stride;
  int channels;
};

// A thread takes RUN tokens of 8 channels, BATCH of them requested at a time.
template <typename E, int T, int RUN, int BATCH>
__global__ void __launch_bounds__(CV_THREADS) conv_prefill_kernel(const __grid_constant__ ConvParams p) {
  const int seq = blockIdx.z, t0 = blockIdx.y * RUN, c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  pdl_trigger();                  // the launch behind (conv_state_kernel) waits for this one
  const int row0 = p.cu[seq], len = p.cu[seq + 1] - row0;
  if (t0 >= len || c >= p.channels) return;
  const int start = p.start[seq];
  const E* x = static_cast<const E*>(p.x) + static_cast<int64_t>(row0) * p.stride + c;
  const float* ring = p.ring + static_cast<int64_t>(p.slots[seq]) * T * p.channels + c;
  Raw8<E> raw[BATCH];
  auto request = [&](int i0) {
#pragma unroll
    for (int i = 0; i < BATCH; ++i) raw[i].load(x + static_cast<int64_t>(min(t0 + i0 + i, len - 1)) * p.stride);
  };
  request(0);
  float w[T][8], b[8], h[T][8];   // h[j]: the input j tokens back
#pragma unroll
  for (int j = 0; j < T; ++j) load8(p.w + static_cast<int64_t>(j) * p.channels + c, w[j]);
  load8(p.bias + c, b);
#pragma unroll
  for (int j = 1; j < T; ++j) {   // before the first step: one token nearer
    const int t = t0 - j;
    if (t >= 0) load8(x + t * p.stride, h[j - 1]);
    else if (start + t >= 0) load8(ring + static_cast<int64_t>((start + t) % T) * p.channels, h[j - 1]);
    else
#pragma unroll
      for (int k = 0; k < 8; ++k) h[j - 1][k] = 0.f;
  }
  E* out = static_cast<E*>(p.out) + static_cast<int64_t>(row0) * p.out_stride + c;
#pragma unroll 1
  for (int i0 = 0; i0 < RUN; i0 += BATCH) {
    if (i0 > 0) request(i0);
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const int t = t0 + i0 + i;
      if (t >= len) break;
#pragma unroll
      for (int j = T - 1; j > 0; --j)
#pragma unroll
        for (int k = 0; k < 8; ++k) h[j][k] = h[j - 1][k];
      raw[i].get(h[0]);
      float y[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        float acc = b[k];
#pragma unroll
        for (int j = 0; j < T; ++j) acc = fmaf(w[j][k], h[j][k], acc);
        y[k] = silu_f<E>(acc);
      }
      store8(out + t * p.out_stride, y);
    }
  }
}

// The last T inputs of every sequence's portion to its ring, after the launch above has read it.  grid (channels, T, sequences)
template <typename E, int T>
__global__ void __launch_bounds__(CV_THREADS) conv_state_kernel(const __grid_constant__ ConvParams p) {
  const int seq = blockIdx.z, c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  pdl_wait();
  const int row0 = p.cu[seq], len = p.cu[seq + 1] - row0, t = len - 1 - static_cast<int>(blockIdx.y);
  if (t < 0 || c >= p.channels) return;
  float f[8];
  load8(static_cast<const E*>(p.x) + (static_cast<int64_t>(row0) + t) * p.stride + c, f);
  store8(p.ring + (static_cast<int64_t>(p.slots[seq]) * T + (p.start[seq] + t) % T) * p.channels + c, f);
}

template <typename E, int T, int RUN, int BATCH>
static int launch_conv_run(const ConvParams& p, int batch, int max_len, cudaStream_t st) {
  const unsigned cols = (p.channels / 8 + CV_THREADS - 1) / CV_THREADS;
  B200_REQUIRE(max_len <= 65535 * RUN, "conv_prefill: sequences of at most %d tokens", 65535 * RUN);
  conv_prefill_kernel<E, T, RUN, BATCH><<<dim3(cols, (max_len + RUN - 1) / RUN, batch), CV_THREADS, 0, st>>>(p);
  if (launch_pdl(true, conv_state_kernel<E, T>, dim3(cols, T, batch), dim3(CV_THREADS), 0, st, p) != cudaSuccess)
    return fail(ERR_LAUNCH, "conv_prefill: %s", cudaGetErrorString(cudaGetLastError()));
  return check_launch("conv_prefill");
}

template <typename E, int T>
static int launch_conv(const ConvParams& p, int batch, int max_len, cudaStream_t st) {
  if constexpr (T == 4) {         // short runs when long ones leave SMs without enough requests in flight
    const int64_t warps = static_cast<int64_t>(p.channels / 256 + 1) * (max_len / 16 + 1) * batch;
    return warps < 16 * sm_count() ? launch_conv_run<E, T, 4, 4>(p, batch, max_len, st) : launch_conv_run<E, T, 16, 8>(p, batch, max_len, st);
  } else {
    return launch_conv_run<E, T, 16, 1>(p, batch, max_len, st);
  }
}

// ------------------------------------------------------------------------------------------------------ gated norm
struct GroupNormParams {
  const void* y;           // [rows, y_stride] Y: heads of vdim columns, the first true_vdim of each in use
  int64_t y_stride;
  const void* z;           // [rows, z_stride] E, same columns
  int64_t z_stride;
  const float* weight;     // [heads * vdim]
  void* out;               // [rows, out_stride] E
  int64_t out_stride;
  int64_t parts;           // rows * groups
  int groups, size, vdim, true_vdim, overlap;   // size: true channels per group
  float eps;
};

// The W = 8 forms take groups of whole 8-element vectors without padding, R vectors per thread in registers.  WARP: a warp per
// (row, group), 8 of them per CTA; else a CTA.  W = 1: any sizes, two passes over memory.
template <typename E, typename Y, int W, int R, bool WARP>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(const __grid_constant__ GroupNormParams p) {
  __shared__ float red[32];
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  const int64_t part = WARP ? static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5) : blockIdx.x;
  if (part >= p.parts) return;
  const int64_t row = part / p.groups;
  const int first = static_cast<int>(part - row * p.groups) * p.size;
  const Y* y = static_cast<const Y*>(p.y) + row * p.y_stride;
  const E* z = static_cast<const E*>(p.z) + row * p.z_stride;
  E* out = static_cast<E*>(p.out) + row * p.out_stride;
  const int lane = WARP ? threadIdx.x & 31 : threadIdx.x, step = WARP ? 32 : blockDim.x;
  float sq[1] = {0.f};
  if constexpr (W == 8) {
    float f[R][8];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = (lane + r * step) * 8;
      if (i < p.size) {
        float g[8];
        load8(y + first + i, f[r]);
        load8(z + first + i, g);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          f[r][k] *= silu_f<E>(g[k]);
          sq[0] = fmaf(f[r][k], f[r][k], sq[0]);
        }
      }
    }
    if constexpr (WARP) sq[0] = warp_sum(sq[0]);
    else block_sum<1>(sq, red);
    const float scale = 1.0f / sqrtf(sq[0] / static_cast<float>(p.size) + p.eps);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = (lane + r * step) * 8;
      if (i < p.size) {
        float w[8];
        load8(p.weight + first + i, w);
#pragma unroll
        for (int k = 0; k < 8; ++k) f[r][k] *= scale * w[k];
        store8(out + first + i, f[r]);
      }
    }
  } else {
    auto at = [&](int i) { return (i / p.true_vdim) * p.vdim + i % p.true_vdim; };
    for (int i = lane; i < p.size; i += step) {
      const int c = at(first + i);
      const float f = load1(y + c) * silu_f<E>(load1(z + c));
      sq[0] = fmaf(f, f, sq[0]);
    }
    block_sum<1>(sq, red);
    const float scale = 1.0f / sqrtf(sq[0] / static_cast<float>(p.size) + p.eps);
    for (int i = lane; i < p.size; i += step) {
      const int c = at(first + i);
      store1(out + c, load1(y + c) * silu_f<E>(load1(z + c)) * scale * p.weight[c]);
      if ((first + i) % p.true_vdim == p.true_vdim - 1)
        for (int k = 1; k <= p.vdim - p.true_vdim; ++k) store1(out + c + k, 0.f);   // the head's padding
    }
  }
}

template <typename E, typename Y>
static cudaError_t launch_group_norm(const GroupNormParams& p, cudaStream_t st) {
  const bool early = (p.overlap & OVERLAP_START) != 0;
  const dim3 block(256), each(static_cast<unsigned>(p.parts));
  if (p.vdim == p.true_vdim && p.size % 8 == 0 && p.size <= 8192) {
    const dim3 warps(static_cast<unsigned>((p.parts + 7) / 8));
    if (p.size <= 256 || (p.size <= 1024 && p.parts >= GLUE_WIDE_ROWS))
      return p.size <= 256 ? launch_pdl(early, gated_group_norm_kernel<E, Y, 8, 1, true>, warps, block, 0, st, p)
                           : launch_pdl(early, gated_group_norm_kernel<E, Y, 8, 4, true>, warps, block, 0, st, p);
    const dim3 fit(static_cast<unsigned>(p.size >= 2048 ? 256 : (p.size / 8 + 31) / 32 * 32));
    return p.size <= 2048 ? launch_pdl(early, gated_group_norm_kernel<E, Y, 8, 1, false>, each, fit, 0, st, p)
                          : launch_pdl(early, gated_group_norm_kernel<E, Y, 8, 4, false>, each, fit, 0, st, p);
  }
  return launch_pdl(early, gated_group_norm_kernel<E, Y, 1, 1, false>, each, block, 0, st, p);
}

// ---------------------------------------------------------------------------------------------------- chunked prefill
constexpr int SC_Q = 32;                 // tokens per chunk: one per lane of the scanning warp
constexpr int SC_WARPS = 8;
constexpr int SC_THREADS = SC_WARPS * 32;
constexpr int SC_COLS = 16 * SC_WARPS;   // value columns of a CTA
constexpr int SC_XP = SC_COLS + 8;       // pitches: ldmatrix rows in different banks
constexpr int SC_PP = SC_Q + 8;
constexpr int SC_HEADS = 4;              // most heads of a CTA

template <int N>
struct SsdSmem {
  static constexpr int NP = N + 8;
  __nv_bfloat16 c[2][SC_Q * NP], b[2][SC_Q * NP], x[2][SC_Q * SC_XP];
  __nv_bfloat16 xh[SC_Q * SC_XP], xl[SC_Q * SC_XP];              // weighted x
  __nv_bfloat16 ph[SC_HEADS][SC_Q * SC_PP], pl[SC_HEADS][SC_Q * SC_PP];
  float cum[SC_HEADS][SC_Q], dt[SC_HEADS][SC_Q], w[SC_HEADS][SC_Q], e[SC_HEADS][SC_Q];
};

__device__ __forceinline__ void sc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}
__device__ __forceinline__ void sc_copy16(void* dst, const void* src, bool on) {   // zeros when off
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

// N: state rows incl. padding.  LOCAL: only the state from zero and the total decay of every segment.
// grid (column blocks, heads / heads per CTA, sequences * segments)
template <int N, bool LOCAL>
__global__ void __launch_bounds__(SC_THREADS, 2) ssd_chunk_kernel(const __grid_constant__ OuterRnnParams p, int per_cta) {
  using Smem = SsdSmem<N>;
  constexpr int NP = Smem::NP, NV = N / 8, XV = SC_COLS / 8;
  extern __shared__ __align__(16) uint8_t sc_smem[];
  Smem& sm = *reinterpret_cast<Smem*>(sc_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seq = blockIdx.z / p.segments, seg = blockIdx.z % p.segments, head0 = blockIdx.y * per_cta, col0 = blockIdx.x * SC_COLS;
  const int all = p.cu[seq + 1] - p.cu[seq], seg0 = seg * p.segment;
  const int row0 = p.cu[seq] + seg0, len = min(all - seg0, p.segment);
  if (len <= 0 || (LOCAL && seg0 + len == all)) return;  // nothing follows a sequence's last segment
  const int cols = per_cta > 1 ? per_cta * p.vdim : min(SC_COLS, p.vdim - col0);
  const int lh = per_cta > 1 ? warp * 16 / p.vdim : 0, head = head0 + lh;
  const bool warp_on = warp * 16 < cols;
  const int head_col = per_cta > 1 ? warp * 16 - lh * p.vdim : col0 + warp * 16;   // this warp's first column in its head
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(p.x) + static_cast<int64_t>(row0) * p.stride;
  const int bc_col = (head0 / p.per_group) * p.dim, x_col = p.v_off + head0 * p.vdim + col0;
  auto fetch = [&](int t0, int buf) {
    for (int i = tid; i < SC_Q * NV; i += SC_THREADS) {
      const int t = i / NV, c = (i % NV) * 8;
      const bool on = t0 + t < len && c < p.dim;
      const __nv_bfloat16* r = base + static_cast<int64_t>(on ? t0 + t : 0) * p.stride + bc_col + (on ? c : 0);
      if (!LOCAL) sc_copy16(&sm.c[buf][t * NP + c], r + p.q_off, on);
      sc_copy16(&sm.b[buf][t * NP + c], r + p.k_off, on);
    }
    for (int i = tid; i < SC_Q * XV; i += SC_THREADS) {
      const int t = i / XV, c = (i % XV) * 8;
      const bool on = t0 + t < len && c < cols;
      sc_copy16(&sm.x[buf][t * SC_XP + c], base + static_cast<int64_t>(on ? t0 + t : 0) * p.stride + x_col + (on ? c : 0), on);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  // decay scan: warp w < per_cta works on head head0 + w, a lane per token; its raw step sizes come a chunk ahead
  const bool scans = warp < per_cta;
  float dt_bias = 0.f, rate = 0.f, dt_raw = 0.f, log_total = 0.f;
  const __nv_bfloat16* dt_col = static_cast<const __nv_bfloat16*>(p.dt) + static_cast<int64_t>(row0) * p.dt_stride + head0 + warp;
  if (scans) {
    dt_bias = p.bias[head0 + warp], rate = expf(p.a_log[head0 + warp]);
    if (lane < len) dt_raw = load1(dt_col + lane * p.dt_stride);
  }
  // S^T: value column lane / 4 (+ 8) of the warp, state rows 8 n + (lane % 4) * 2 (+ 1)
  float S[N / 8][4];
  const int64_t head_elems = static_cast<int64_t>(p.dim) * p.vdim;
  float* slot_state = p.state + (static_cast<int64_t>(p.slots[seq]) * p.heads + head) * head_elems;
  float* seg_state = p.seg_state + (static_cast<int64_t>(blockIdx.z) * p.heads + head) * head_elems;
  const float* from = p.segments > 1 ? seg_state : slot_state;
  const bool carry = !LOCAL && warp_on && (p.segments > 1 || p.start[seq] > 0);
  const int my_col = head_col + (lane >> 2);
#pragma unroll
  for (int n = 0; n < N / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      S[n][j] = carry && d < p.dim ? from[static_cast<int64_t>(d) * p.vdim + c] : 0.f;
    }
  const float skip = LOCAL ? 0.f : p.skip[min(head, p.heads - 1)];
  const int gm = warp & 1, gn = warp >> 1;             // this warp's 16 x 8 tile of C B^T
  const bool tile_on = !LOCAL && gn * 8 <= gm * 16 + 15;
  for (int t0 = 0, buf = 0; t0 < len; t0 += SC_Q, buf ^= 1) {
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // the chunk's rows are here; everybody is done with the previous chunk
    if (t0 + SC_Q < len) fetch(t0 + SC_Q, buf ^ 1);
    // ---- decays
    if (scans) {
      const float dt = t0 + lane < len ? softplus_f(dt_raw + dt_bias) : 0.f;
      if (t0 + SC_Q + lane < len) dt_raw = load1(dt_col + static_cast<int64_t>(t0 + SC_Q + lane) * p.dt_stride);
      float run = -rate * dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      const float total = __shfl_sync(0xffffffffu, run, 31);
      log_total += total;
      sm.cum[warp][lane] = run;
      sm.dt[warp][lane] = dt;
      sm.w[warp][lane] = expf(total - run) * dt;
      sm.e[warp][lane] = expf(run);
    }
    float g[4] = {0.f, 0.f, 0.f, 0.f};
    if (tile_on) {
#pragma unroll
      for (int k2 = 0; k2 < N / 32; ++k2) {
        uint32_t a0[4], a1[4], bk[4];
        const uint32_t a_at = smem_u32(&sm.c[buf][(gm * 16 + (lane & 15)) * NP + k2 * 32 + (lane >> 4) * 8]);
        ldmatrix_x4(a0, a_at);
        ldmatrix_x4(a1, a_at + 32);
        ldmatrix_x4(bk, smem_u32(&sm.b[buf][(gn * 8 + (lane & 7)) * NP + k2 * 32 + (lane >> 3) * 8]));
        mma_bf16_16816(g, a0, bk[0], bk[1]);
        mma_bf16_16816(g, a1, bk[2], bk[3]);
      }
    }
    __syncthreads();
    // ---- weights
    if (tile_on) {
      const int t = gm * 16 + (lane >> 2), s = gn * 8 + (lane & 3) * 2;
      for (int h = 0; h < per_cta; ++h) {
        const float c0 = sm.cum[h][s], c1 = sm.cum[h][s + 1], d0 = sm.dt[h][s], d1 = sm.dt[h][s + 1];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int tt = t + half * 8;
          const float ct = sm.cum[h][tt];
          const float p0 = s <= tt ? g[half * 2] * __expf(ct - c0) * d0 : 0.f;
          const float p1 = s + 1 <= tt ? g[half * 2 + 1] * __expf(ct - c1) * d1 : 0.f;
          uint32_t hi, lo;
          sc_split(p0, p1, hi, lo);
          *reinterpret_cast<uint32_t*>(&sm.ph[h][tt * SC_PP + s]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.pl[h][tt * SC_PP + s]) = lo;
        }
      }
    }
    for (int i = tid; i < SC_Q * XV; i += SC_THREADS) {
      const int t = i / XV, c = (i % XV) * 8;
      if (c >= cols) continue;
      const float w = sm.w[per_cta > 1 ? c / p.vdim : 0][t];
      float f[8];
      load8(&sm.x[buf][t * SC_XP + c], f);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) sc_split(f[2 * k] * w, f[2 * k + 1] * w, hi[k], lo[k]);
      *reinterpret_cast<uint4*>(&sm.xh[t * SC_XP + c]) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(&sm.xl[t * SC_XP + c]) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    __syncthreads();
    if (!warp_on) continue;
    // ---- products
    // matrices (tokens 0-7, columns 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15) of 16 tokens x this warp's 16 columns
    const int x_off = ((lane & 7) + (lane >> 4) * 8) * SC_XP + warp * 16 + ((lane >> 3) & 1) * 8;
    if (!LOCAL) {
      float o[2][2][4];
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < N / 16; ++ks) {
        uint32_t a0[4], a1[4];
        const uint32_t a_at = smem_u32(&sm.c[buf][(lane & 15) * NP + ks * 16 + (lane >> 4) * 8]);
        ldmatrix_x4(a0, a_at);
        ldmatrix_x4(a1, a_at + 16 * NP * 2);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          uint32_t h0, l0, h1, l1;
          sc_split(S[2 * ks][2 * n], S[2 * ks][2 * n + 1], h0, l0);
          sc_split(S[2 * ks + 1][2 * n], S[2 * ks + 1][2 * n + 1], h1, l1);
          mma_bf16_16816(o[0][n], a0, h0, h1);
          mma_bf16_16816(o[1][n], a1, h0, h1);
          mma_bf16_16816(o[0][n], a0, l0, l1);
          mma_bf16_16816(o[1][n], a1, l0, l1);
        }
      }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float e0 = sm.e[lh][m * 16 + (lane >> 2)], e1 = sm.e[lh][m * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int n = 0; n < 2; ++n) o[m][n][0] *= e0, o[m][n][1] *= e0, o[m][n][2] *= e1, o[m][n][3] *= e1;
      }
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        uint32_t vm[4];
        ldmatrix_x4_trans(vm, smem_u32(&sm.x[buf][ks * 16 * SC_XP + x_off]));
#pragma unroll
        for (int m = ks; m < 2; ++m) {
          uint32_t ah[4], al[4];
          const int at = (m * 16 + (lane & 15)) * SC_PP + ks * 16 + (lane >> 4) * 8;
          ldmatrix_x4(ah, smem_u32(&sm.ph[lh][at]));
          ldmatrix_x4(al, smem_u32(&sm.pl[lh][at]));
          mma_bf16_16816(o[m][0], ah, vm[0], vm[2]);
          mma_bf16_16816(o[m][1], ah, vm[1], vm[3]);
          mma_bf16_16816(o[m][0], al, vm[0], vm[2]);
          mma_bf16_16816(o[m][1], al, vm[1], vm[3]);
        }
      }
      __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + static_cast<int64_t>(row0 + t0) * p.out_stride + head * p.vdim +
                           head_col + (lane & 3) * 2;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = m * 16 + (lane >> 2) + half * 8;
          if (t0 + t >= len) continue;
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const uint32_t x = *reinterpret_cast<const uint32_t*>(&sm.x[buf][t * SC_XP + warp * 16 + n * 8 + (lane & 3) * 2]);
            *reinterpret_cast<uint32_t*>(out + t * p.out_stride + n * 8) =
                pack_bf16(fmaf(skip, bf16_lo(x), o[m][n][half * 2]), fmaf(skip, bf16_hi(x), o[m][n][half * 2 + 1]));
          }
        }
    }
    // S^T <- S^T exp(L_E) + (weighted x)^T B
    {
      const float keep = sm.e[lh][SC_Q - 1];
      uint32_t xh[2][4], xl[2][4];
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        ldmatrix_x4_trans(xh[ks], smem_u32(&sm.xh[ks * 16 * SC_XP + x_off]));
        ldmatrix_x4_trans(xl[ks], smem_u32(&sm.xl[ks * 16 * SC_XP + x_off]));
      }
#pragma unroll
      for (int n = 0; n < N / 8; n += 2) {
#pragma unroll
        for (int i = 0; i < 2; ++i) S[n + i][0] *= keep, S[n + i][1] *= keep, S[n + i][2] *= keep, S[n + i][3] *= keep;
#pragma unroll
        for (int ks = 0; ks < 2; ++ks) {
          uint32_t bt[4];
          ldmatrix_x4_trans(bt, smem_u32(&sm.b[buf][(ks * 16 + (lane & 15)) * NP + n * 8 + (lane >> 4) * 8]));
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16_16816(S[n + i], xh[ks], bt[2 * i], bt[2 * i + 1]);
            mma_bf16_16816(S[n + i], xl[ks], bt[2 * i], bt[2 * i + 1]);
          }
        }
      }
    }
  }
  if (LOCAL && scans && blockIdx.x == 0) {
    float* decay = p.seg_decay + (static_cast<int64_t>(blockIdx.z) * p.heads + head0 + warp) * p.dim;
    for (int d = lane; d < p.dim; d += 32) decay[d] = expf(log_total);
  }
  if ((!LOCAL && seg0 + len < all) || !warp_on) return;   // only the last segment leaves the sequence's state behind
  float* to = LOCAL ? seg_state : slot_state;
#pragma unroll
  for (int n = 0; n < N / 8; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = n * 8 + (lane & 3) * 2 + (j & 1), c = my_col + (j >> 1) * 8;
      if (d < p.dim) to[static_cast<int64_t>(d) * p.vdim + c] = S[n][j];
    }
}

template <int N>
static int launch_ssd(const OuterRnnParams& p, int n, cudaStream_t st) {
  constexpr int smem = sizeof(SsdSmem<N>);
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(ssd_chunk_kernel<N, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
        cudaFuncSetAttribute(ssd_chunk_kernel<N, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return fail(ERR_RUNTIME, "ssd_prefill: cannot raise dynamic shared memory to %d", smem);
    configured[dev] = true;
  }
  int per_cta = 1;
  while (per_cta < SC_HEADS && 2 * per_cta * p.vdim <= SC_COLS && p.per_group % (2 * per_cta) == 0) per_cta *= 2;
  const dim3 grid((p.vdim + SC_COLS - 1) / SC_COLS, p.heads / per_cta, n * p.segments);
  if (p.segments > 1) {
    ssd_chunk_kernel<N, true><<<grid, SC_THREADS, smem, st>>>(p, per_cta);
    outer_rnn_fold_launch(p, n, st);
  }
  ssd_chunk_kernel<N, false><<<grid, SC_THREADS, smem, st>>>(p, per_cta);
  return check_launch("ssd_prefill");
}

}  // namespace b200

using namespace b200;

extern "C" int b200_conv_prefill(const void* x, int64_t stride, const float* weight, const float* bias, float* ring,
                                 const int32_t* cu_seqlens, const int32_t* slots, const int32_t* start, void* out,
                                 int64_t out_stride, int32_t batch, int32_t max_len, int32_t channels, int32_t taps, int32_t f32,
                                 b200_stream_t stream) {
  if (batch <= 0 || max_len <= 0) return OK;
  B200_REQUIRE(channels > 0 && channels % 8 == 0 && stride % 8 == 0 && out_stride % 8 == 0 && batch <= 65535,
               "conv_prefill: channels and strides must be multiples of 8");
  B200_REQUIRE(taps == 4 || taps == 8 || taps == 16, "conv_prefill: 4, 8 or 16 taps (pad with zero weights), got %d", taps);
  B200_REQUIRE(aligned16(x) && aligned16(weight) && aligned16(bias) && aligned16(ring) && aligned16(out), "conv_prefill: unaligned tensor");
  const ConvParams p = {x, stride, weight, bias, ring, cu_seqlens, slots, start, out, out_stride, channels};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32) return taps == 4 ? launch_conv<float, 4>(p, batch, max_len, st) : taps == 8 ? launch_conv<float, 8>(p, batch, max_len, st)
                                                                                    : launch_conv<float, 16>(p, batch, max_len, st);
  return taps == 4 ? launch_conv<__nv_bfloat16, 4>(p, batch, max_len, st) : taps == 8 ? launch_conv<__nv_bfloat16, 8>(p, batch, max_len, st)
                                                                                      : launch_conv<__nv_bfloat16, 16>(p, batch, max_len, st);
}

extern "C" int32_t b200_ssd_chunked(int32_t dim, int32_t vdim) { return dim % 8 == 0 && dim <= 128 && vdim % 16 == 0; }

extern "C" int b200_ssd_prefill(const void* xbc, int64_t stride, const void* dt, int64_t dt_stride, const float* dt_bias,
                                const float* a_log, const float* skip, float* state, const int32_t* cu_seqlens,
                                const int32_t* slots, const int32_t* start, void* y, int32_t batch, int32_t heads,
                                int32_t groups, int32_t dim, int32_t vdim, int32_t f32, int32_t serial, int32_t segment,
                                int32_t segments, float* workspace, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && heads <= 65535 && static_cast<int64_t>(batch) * segments <= 65535,
               "ssd_prefill: heads must be a multiple of the groups, at most 65535 heads and segments");
  B200_REQUIRE(segment > 0 && segments > 0 && (segments == 1 || (segment % SC_Q == 0 && workspace && aligned16(workspace))),
               "ssd_prefill: segments must be multiples of %d tokens and have a workspace", SC_Q);
  B200_REQUIRE(dim > 0 && dim <= 256 && vdim > 0 && vdim % 4 == 0, "ssd_prefill: at most 256 state rows, vdim a multiple of 4");
  OuterRnnParams p = {};
  p.x = xbc, p.stride = stride, p.v_off = 0, p.k_off = heads * vdim, p.q_off = p.k_off + groups * dim, p.per_group = heads / groups;
  p.dt = dt, p.dt_stride = dt_stride, p.bias = dt_bias, p.a_log = a_log, p.skip = skip;
  p.state = state, p.cu = cu_seqlens, p.slots = slots, p.start = start, p.heads = heads, p.dim = dim, p.vdim = vdim;
  p.segment = segment, p.segments = segments, p.seg_state = workspace;
  p.seg_decay = workspace ? workspace + static_cast<int64_t>(batch) * segments * heads * dim * vdim : nullptr;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32 || serial || !b200_ssd_chunked(dim, vdim)) {
    p.o = static_cast<float*>(y);
    return outer_rnn_serial_launch(p, RNN_SSD, f32 != 0, batch, st);
  }
  B200_REQUIRE(aligned16(xbc) && aligned16(y) && stride % 8 == 0, "ssd_prefill: unaligned tensor");
  p.out = y, p.out_stride = static_cast<int64_t>(heads) * vdim;
  if (dim <= 32) return launch_ssd<32>(p, batch, st);
  if (dim <= 64) return launch_ssd<64>(p, batch, st);
  return launch_ssd<128>(p, batch, st);
}

extern "C" int b200_ssd_decode(const void* xbc, int64_t stride, const void* dt, int64_t dt_stride, const float* dt_bias,
                               const float* a_log, const float* skip, const float* conv_weight, const float* conv_bias,
                               float* ring, int32_t taps, float* state, const int64_t* pos, const int64_t* active, float* y,
                               int32_t batch, int32_t heads, int32_t groups, int32_t dim, int32_t vdim, int32_t f32,
                               int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && taps > 0, "ssd_decode: heads must be a multiple of the groups");
  OuterRnnParams p = {};
  p.x = xbc, p.stride = stride, p.v_off = 0, p.k_off = heads * vdim, p.q_off = p.k_off + groups * dim, p.per_group = heads / groups;
  p.dt = dt, p.dt_stride = dt_stride, p.bias = dt_bias, p.a_log = a_log, p.skip = skip;
  p.ring = ring, p.taps_w = conv_weight, p.taps_b = conv_bias, p.taps = taps, p.channels = heads * vdim + 2 * groups * dim;
  p.state = state, p.heads = heads, p.dim = dim, p.vdim = vdim, p.true_vdim = vdim, p.o = y;
  p.pos = pos, p.active = active, p.overlap = overlap;
  return outer_rnn_decode_launch(p, RNN_SSD, f32 != 0, batch, "ssd_decode", reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int b200_gated_group_norm(const void* y, int64_t y_stride, const void* z, int64_t z_stride, const float* weight,
                                     void* out, int64_t out_stride, int32_t rows, int32_t heads, int32_t vdim, int32_t true_vdim,
                                     int32_t groups, float eps, int32_t y_f32, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(heads > 0 && true_vdim > 0 && true_vdim <= vdim && groups > 0 && heads * true_vdim % groups == 0,
               "gated_group_norm: the channels must divide into equal groups");
  B200_REQUIRE(aligned16(y) && aligned16(z) && aligned16(weight) && aligned16(out) && y_stride % 8 == 0 && z_stride % 8 == 0 &&
                   out_stride % 8 == 0 && static_cast<int64_t>(rows) * groups < (1ll << 31),
               "gated_group_norm: unaligned tensor");
  const GroupNormParams p = {y, y_stride, z, z_stride, weight, out, out_stride, static_cast<int64_t>(rows) * groups,
                             groups, heads * true_vdim / groups, vdim, true_vdim, overlap, eps};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  B200_REQUIRE(y_f32 || !f32, "gated_group_norm: fp32 activations come with fp32 y");
  const cudaError_t e = f32     ? launch_group_norm<float, float>(p, st)
                        : y_f32 ? launch_group_norm<__nv_bfloat16, float>(p, st)
                                : launch_group_norm<__nv_bfloat16, __nv_bfloat16>(p, st);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "gated_group_norm: %s", cudaGetErrorString(e));
  return check_launch("gated_group_norm");
}
