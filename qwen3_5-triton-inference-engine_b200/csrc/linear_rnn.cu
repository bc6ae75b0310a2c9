// Recurrent mixers whose gates read only the current token, over packed batches (prefill) and one token per slot
// (decode).  States are fp32 and live in per-slot caches; a sequence whose first token sits at position 0 starts from
// zero whatever the slot held before.
//
//   minGRU (element-wise):  z = sigmoid(z' + zb), u = x' + xb, c = u >= 0 ? u + 1/2 : sigmoid(u)
//                           S_t = (1 - z) S_(t-1) + z c,   out = S_t * silu(g)
//     Prefill: a CTA walks a sequence in blocks of 64 tokens, its warps scan 8 tokens each in parallel.  Too few CTAs:
//     sequences are cut into segments; pass 1 reduces a segment to (product of 1 - z, state it leaves from zero), pass 2
//     folds the segments in front of its own.  HBM bound.
//   Outer-product recurrences (linear_rnn.cuh: HGRN2, gated linear attention, state space).
//     Prefill of bf16 activations runs in chunks on the tensor cores (linear_rnn_chunk.cu, ssd.cu).  The token-serial form
//     here is plain fp32, for fp32 activations and for heads wider than 128: a warp owns COLS state columns, a lane dim/32
//     rows of each as packed fp32 pairs (fma.rn.f32x2); 16 tokens of gates are staged in shared memory at a time, the next
//     16 are loaded while they are worked on.
#include "b200_attn.h"
#include "elem.cuh"
#include "linear_rnn.cuh"

namespace b200 {

// ------------------------------------------------------------------------------------------------------------ minGRU
struct MinGruParams {
  const void* zxg;          // [rows, stride] E: [z | x | g], each `width` wide
  int64_t stride;
  const float* bias;        // [z bias | x bias] 2 * width
  float* state;             // [slots, width]
  const int32_t* cu;        // [n + 1] packed rows of the sequences
  const int32_t* slots;     // [n]
  const int32_t* start;     // [n] position of each sequence's first packed token
  float2* ab;               // [n, segments + 1, width]: (product of 1 - z, state from zero) per segment; the last entry
                            // keeps the sequence's initial state
  void* out;                // [rows, width] E
  int width, segment, segments;
};

template <typename E>
__device__ __forceinline__ void mingru_gate(float z_raw, float u, float zb, float xb, float& keep, float& add) {
  const float z = sigmoid_f<E>(z_raw + zb);
  u += xb;
  const float cand = u >= 0.f ? u + 0.5f : sigmoid_f<E>(u);
  keep = 1.0f - z;
  add = z * cand;
}

__device__ __forceinline__ float2 load2(const __nv_bfloat16* q) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(q);
  return make_float2(bf16_lo(v), bf16_hi(v));
}
__device__ __forceinline__ float2 load2(const float* q) { return *reinterpret_cast<const float2*>(q); }

constexpr int MG_WARPS = 8, MG_RUN = 8;             // a warp's run of consecutive tokens
constexpr int MG_BLOCK = MG_WARPS * MG_RUN;         // tokens a CTA takes at a time
constexpr int MG_COLS = 64;                         // channels of a CTA, two per lane

// A CTA walks its segment in blocks of 64 tokens.  Every warp turns 8 of them into (keep, add) pairs in registers, leaves
// their product and sum in shared memory, folds the runs in front of its own and replays its run: inputs are read once.
// grid (width / 64, segments, sequences).  REDUCE: only the segment's (product, state from zero).
template <typename E, bool REDUCE>
__global__ void __launch_bounds__(MG_WARPS * 32, sizeof(E) == 2 ? 3 : 2) mingru_prefill_kernel(const __grid_constant__ MinGruParams p) {
  __shared__ float4 runs[2][MG_WARPS][32];
  const int seq = blockIdx.z, seg = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * MG_COLS + lane * 2;
  const int row0 = p.cu[seq], all = p.cu[seq + 1] - row0;
  const int s0 = seg * p.segment, s1 = min(s0 + p.segment, all);
  const bool last = s1 == all;
  if (s0 >= all || (REDUCE && last)) return;        // nobody folds a last segment
  const bool on = c < p.width;
  const int cc = on ? c : 0;
  const float2 zb = load2(p.bias + cc), xb = load2(p.bias + p.width + cc);
  float* state = p.state + static_cast<int64_t>(p.slots[seq]) * p.width + cc;
  float2* ab = p.ab + static_cast<int64_t>(seq) * (p.segments + 1) * p.width + cc;
  float2 carry = make_float2(0.f, 0.f);
  if (REDUCE || (s0 == 0 && last)) {
    if (!(REDUCE && s0 > 0) && p.start[seq] > 0) carry = load2(state);
    if (REDUCE && s0 == 0 && warp == 0 && on) *reinterpret_cast<float4*>(ab + static_cast<int64_t>(p.segments) * p.width) = make_float4(carry.x, 0.f, carry.y, 0.f);
    if (REDUCE) carry = make_float2(0.f, 0.f);
  } else {
    const float4 init = *reinterpret_cast<const float4*>(ab + static_cast<int64_t>(p.segments) * p.width);
    carry = make_float2(init.x, init.z);
#pragma unroll 8
    for (int i = 0; i < seg; ++i) {
      const float4 x = *reinterpret_cast<const float4*>(ab + static_cast<int64_t>(i) * p.width);
      carry.x = fmaf(x.x, carry.x, x.y);
      carry.y = fmaf(x.z, carry.y, x.w);
    }
  }
  float2 product = make_float2(1.f, 1.f);
  const E* base = static_cast<const E*>(p.zxg) + static_cast<int64_t>(row0) * p.stride + cc;
  for (int tb = s0, buf = 0; tb < s1; tb += MG_BLOCK, buf ^= 1) {
    const int t0 = tb + warp * MG_RUN;
    float2 keep[MG_RUN], add[MG_RUN], g[MG_RUN];
    const E *rz = base + static_cast<int64_t>(t0) * p.stride, *rx = rz + p.width, *rg = rx + p.width;
    const int stride = static_cast<int>(p.stride), lim = s1 - 1 - t0;
#pragma unroll
    for (int i = 0; i < MG_RUN; ++i) {
      const int off = min(i, lim) * stride;  // past the end: a row read again
      keep[i] = load2(rz + off);
      add[i] = load2(rx + off);
      if (!REDUCE) g[i] = load2(rg + off);
    }
    float4 run = make_float4(1.f, 0.f, 1.f, 0.f);
#pragma unroll
    for (int i = 0; i < MG_RUN; ++i) {
      float k0, b0, k1, b1;
      mingru_gate<E>(keep[i].x, add[i].x, zb.x, xb.x, k0, b0);
      mingru_gate<E>(keep[i].y, add[i].y, zb.y, xb.y, k1, b1);
      const bool in = i <= lim;
      keep[i] = in ? make_float2(k0, k1) : make_float2(1.f, 1.f);
      add[i] = in ? make_float2(b0, b1) : make_float2(0.f, 0.f);
      run.x *= keep[i].x, run.y = fmaf(keep[i].x, run.y, add[i].x);
      run.z *= keep[i].y, run.w = fmaf(keep[i].y, run.w, add[i].y);
    }
    runs[buf][warp][lane] = run;
    __syncthreads();  // two buffers: the next block's runs go to the other one
    float2 s = carry;
#pragma unroll
    for (int w = 0; w < MG_WARPS; ++w) {
      if (w == warp) s = carry;
      const float4 x = runs[buf][w][lane];
      carry.x = fmaf(x.x, carry.x, x.y);
      carry.y = fmaf(x.z, carry.y, x.w);
      if (REDUCE) product = make_float2(product.x * x.x, product.y * x.z);
    }
    if (!REDUCE && on) {
      E* const out = static_cast<E*>(p.out) + static_cast<int64_t>(row0 + t0) * p.width + c;
#pragma unroll
      for (int i = 0; i < MG_RUN; ++i) {
        s.x = fmaf(keep[i].x, s.x, add[i].x);
        s.y = fmaf(keep[i].y, s.y, add[i].y);
        if (i <= lim) {
          E* o = out + i * p.width;
          const float o0 = s.x * silu_f<E>(g[i].x), o1 = s.y * silu_f<E>(g[i].y);
          if constexpr (sizeof(E) == 2) *reinterpret_cast<uint32_t*>(o) = pack_bf16(o0, o1);
          else *reinterpret_cast<float2*>(o) = make_float2(o0, o1);
        }
      }
    }
  }
  if (warp != 0 || !on) return;
  if (REDUCE) *reinterpret_cast<float4*>(ab + static_cast<int64_t>(seg) * p.width) = make_float4(product.x, carry.x, product.y, carry.y);
  else if (last) *reinterpret_cast<float2*>(state) = carry;  // with several segments nobody else reads the slot in this launch
}

// one token per slot; thread = 4 channels
template <typename E>
__global__ void __launch_bounds__(128) mingru_decode_kernel(const E* zxg, int64_t stride, const float* bias, float* state,
                                                            const int64_t* pos, const int64_t* active, E* out, int width,
                                                            int overlap) {
  const int b = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  if (c >= width) return;
  const bool on = !active || active[b] != 0;
  const bool fresh = pos[b] == 0;
  const E* r = zxg + b * stride + c;
  const float4 z = load4(r), x = load4(r + width), g = load4(r + 2 * width);
  const float4 zb = load4(bias + c), xb = load4(bias + width + c);
  float* st = state + static_cast<int64_t>(b) * width + c;
  float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(st);
  float k, a;
  mingru_gate<E>(z.x, x.x, zb.x, xb.x, k, a), s.x = fmaf(k, s.x, a);
  mingru_gate<E>(z.y, x.y, zb.y, xb.y, k, a), s.y = fmaf(k, s.y, a);
  mingru_gate<E>(z.z, x.z, zb.z, xb.z, k, a), s.z = fmaf(k, s.z, a);
  mingru_gate<E>(z.w, x.w, zb.w, xb.w, k, a), s.w = fmaf(k, s.w, a);
  if (on) store4(st, s);
  store4(out + static_cast<int64_t>(b) * width + c,
         make_float4(s.x * silu_f<E>(g.x), s.y * silu_f<E>(g.y), s.z * silu_f<E>(g.z), s.w * silu_f<E>(g.w)));
}

// ------------------------------------------------------------------------------------------ outer-product recurrences
constexpr int OR_TB = 16;        // tokens staged at a time
constexpr int OR_WARPS = 4;
constexpr int OR_THREADS = OR_WARPS * 32;

// RP = row pairs per lane (dim = 64 * RP, or dim = 32 with RP = 1 and the second row of a pair absent -> dim is padded
// to a multiple of 64 by the caller of this template), COLS = columns per warp.
// grid (vdim / (4 * COLS), heads, sequences)
template <typename E, int RP, int COLS, RnnKind KIND>
__global__ void __launch_bounds__(OR_THREADS) outer_rnn_prefill_kernel(const __grid_constant__ OuterRnnParams p) {
  constexpr int DIM = 64 * RP;                       // rows incl. padding
  constexpr int CT = OR_WARPS * COLS;                // columns of the CTA
  constexpr int CPT = (DIM + OR_THREADS - 1) / OR_THREADS;  // gate channels per thread
  constexpr bool KEYS = KIND != RNN_FORGET;          // keys of their own
  extern __shared__ __align__(16) float or_smem[];
  float* fs = or_smem;                               // [2][TB][DIM]
  float* qs = fs + 2 * OR_TB * DIM;                  // [2][TB][DIM]
  float* ks = qs + 2 * OR_TB * DIM;                  // [2][TB][DIM] when KEYS
  float* vs = ks + (KEYS ? 2 * OR_TB * DIM : 0);     // [2][TB][CT][2]  every v twice: a ready-made pair
  float* os = vs + 2 * OR_TB * CT * 2;               // [TB][CT]
  const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * CT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row0 = p.cu[seq], len = p.cu[seq + 1] - row0;
  if (len <= 0) return;
  const E* base = static_cast<const E*>(p.x) + static_cast<int64_t>(row0) * p.stride;
  const int qk_col = (head / p.per_group) * p.dim, v_col = p.v_off + head * p.vdim;
  float low[CPT], fb[CPT], dt_b = 0.f, rate = 0.f, skip = 0.f;
#pragma unroll
  for (int i = 0; i < CPT; ++i) {
    const int ch = tid + i * OR_THREADS;
    low[i] = KIND == RNN_FORGET && ch < p.dim ? p.lower[head * p.dim + ch] : 0.f;
    fb[i] = KIND != RNN_SSD && ch < p.dim ? p.bias[head * p.dim + ch] : 0.f;
  }
  if (KIND == RNN_SSD) dt_b = p.bias[head], rate = expf(p.a_log[head]), skip = p.skip[head];
  // the raw rows of the next block travel in registers
  float rq[CPT][OR_TB], rf[CPT][OR_TB], rz[KIND == RNN_KEYED ? CPT : 1][OR_TB], rv[(OR_TB * CT + OR_THREADS - 1) / OR_THREADS];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < CPT; ++i) {
      const int ch = tid + i * OR_THREADS;
      if (ch < p.dim) {
#pragma unroll
        for (int t = 0; t < OR_TB; ++t)
          if (t0 + t < len) {
            const E* r = base + static_cast<int64_t>(t0 + t) * p.stride + qk_col + ch;
            rq[i][t] = load1(r + p.q_off);
            rf[i][t] = load1(r + p.k_off);
            if constexpr (KIND == RNN_KEYED) rz[i][t] = p.z[static_cast<int64_t>(row0 + t0 + t) * p.z_stride + head * p.dim + ch];
          }
      }
    }
    if constexpr (KIND == RNN_SSD) {
#pragma unroll
      for (int t = 0; t < OR_TB; ++t)
        if (t0 + t < len) rz[0][t] = load1(static_cast<const E*>(p.dt) + static_cast<int64_t>(row0 + t0 + t) * p.dt_stride + head);
    }
#pragma unroll
    for (int i = 0; i < (OR_TB * CT + OR_THREADS - 1) / OR_THREADS; ++i) {
      const int e = tid + i * OR_THREADS, t = e / CT, c = e % CT;
      rv[i] = 0.f;
      if (e < OR_TB * CT && t0 + t < len && col0 + c < p.vdim)
        rv[i] = load1(base + static_cast<int64_t>(t0 + t) * p.stride + v_col + col0 + c);
    }
  };
  auto stage = [&](int t0, int buf) {
#pragma unroll
    for (int t = 0; t < OR_TB; ++t) {
      const bool in = t0 + t < len;
      float dt = 0.f, decay = 1.f;
      if (KIND == RNN_SSD && in) {
        dt = softplus_f(rz[0][t] + dt_b);
        decay = expf(-rate * dt);
      }
#pragma unroll
      for (int i = 0; i < CPT; ++i) {
        const int ch = tid + i * OR_THREADS;
        if (ch < DIM) {
          float q = 0.f, f = 1.f, k = 0.f;           // padding rows and tokens: keep the state, read and add nothing
          if (ch < p.dim && in) {
            if constexpr (KIND == RNN_FORGET) {
              q = silu_f<E>(rq[i][t]);
              f = low[i] + (1.0f - low[i]) * sigmoid_f<E>(rf[i][t] + fb[i]);
            } else if constexpr (KIND == RNN_KEYED) {
              q = rq[i][t] * p.q_scale;
              k = rf[i][t];
              f = sigmoid_root<E>(rz[i][t] + fb[i], p.inv_tau);
            } else {
              q = rq[i][t];
              k = rf[i][t] * dt;
              f = decay;
            }
          }
          fs[(buf * OR_TB + t) * DIM + ch] = f;
          qs[(buf * OR_TB + t) * DIM + ch] = q;
          if (KEYS) ks[(buf * OR_TB + t) * DIM + ch] = k;
        }
      }
    }
#pragma unroll
    for (int i = 0; i < (OR_TB * CT + OR_THREADS - 1) / OR_THREADS; ++i) {
      const int e = tid + i * OR_THREADS;
      if (e < OR_TB * CT) *reinterpret_cast<float2*>(vs + (buf * OR_TB * CT + e) * 2) = make_float2(rv[i], rv[i]);
    }
  };
  // state: rows lane * 2 * RP + 2 * i (+1), columns col0 + warp * COLS + c
  F2 S[RP][COLS];
  float* st = p.state + (static_cast<int64_t>(p.slots[seq]) * p.heads + head) * p.dim * p.vdim;
  const bool carry = p.start[seq] > 0;
  const int my_col = col0 + warp * COLS;
#pragma unroll
  for (int i = 0; i < RP; ++i)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int r = lane * 2 * RP + 2 * i;
      float lo = 0.f, hi = 0.f;
      if (carry && my_col + c < p.vdim) {
        if (r < p.dim) lo = st[static_cast<int64_t>(r) * p.vdim + my_col + c];
        if (r + 1 < p.dim) hi = st[static_cast<int64_t>(r + 1) * p.vdim + my_col + c];
      }
      S[i][c] = f2(lo, hi);
    }
  fetch(0);
  stage(0, 0);
  __syncthreads();
  const int blocks = (len + OR_TB - 1) / OR_TB;
  for (int blk = 0; blk < blocks; ++blk) {
    const int t0 = blk * OR_TB, buf = blk & 1;
    if (blk + 1 < blocks) fetch(t0 + OR_TB);
    const int n = min(OR_TB, len - t0);
    const float* fsb = fs + buf * OR_TB * DIM + lane * 2 * RP;
    const float* qsb = qs + buf * OR_TB * DIM + lane * 2 * RP;
    const float* ksb = ks + buf * OR_TB * DIM + lane * 2 * RP;
    const float* vsb = vs + (buf * OR_TB * CT + warp * COLS) * 2;
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      F2 f[RP], q[RP], k[RP], v[COLS];
#pragma unroll
      for (int i = 0; i < RP; ++i) {
        const float2 a = *reinterpret_cast<const float2*>(fsb + t * DIM + 2 * i);
        const float2 b = *reinterpret_cast<const float2*>(qsb + t * DIM + 2 * i);
        f[i] = f2(a.x, a.y);
        q[i] = f2(b.x, b.y);
        if constexpr (KEYS) {
          const float2 c = *reinterpret_cast<const float2*>(ksb + t * DIM + 2 * i);
          k[i] = f2(c.x, c.y);
        } else {
          k[i] = f2(1.0f - a.x, 1.0f - a.y);
        }
      }
#pragma unroll
      for (int c = 0; c < COLS; c += 2) {
        const float4 w = *reinterpret_cast<const float4*>(vsb + (t * CT + c) * 2);
        v[c] = f2(w.x, w.y);
        v[c + 1] = f2(w.z, w.w);
      }
      float o[COLS];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        F2 acc = f2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < RP; ++i) {
          S[i][c] = fma2(f[i], S[i][c], mul2(k[i], v[c]));
          acc = fma2(q[i], S[i][c], acc);
        }
        const float2 a = unf2(acc);
        o[c] = a.x + a.y;
      }
      // sum over the 32 lanes, halving the number of columns a lane carries at each step
#pragma unroll
      for (int half = COLS / 2, bit = 16; half >= 1; half >>= 1, bit >>= 1) {
        const bool upper = (lane & bit) != 0;
#pragma unroll
        for (int c = 0; c < half; ++c) {
          const float give = upper ? o[c] : o[c + half];
          const float keep = upper ? o[c + half] : o[c];
          o[c] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
        }
      }
      constexpr int LOGC = COLS == 8 ? 3 : COLS == 4 ? 2 : 1;
#pragma unroll
      for (int bit = 16 >> LOGC; bit >= 1; bit >>= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], bit);
      // lane's column: its top LOGC bits select it, most significant first
      if ((lane & ((32 >> LOGC) - 1)) == 0) os[t * CT + warp * COLS + (lane >> (5 - LOGC))] = o[0];
    }
    if (blk + 1 < blocks) stage(t0 + OR_TB, buf ^ 1);
    __syncthreads();
    for (int e = tid; e < n * CT; e += OR_THREADS) {
      const int t = e / CT, c = e % CT;
      if (col0 + c < p.vdim) p.o[static_cast<int64_t>(row0 + t0 + t) * p.heads * p.vdim + head * p.vdim + col0 + c] =
            KIND == RNN_SSD ? fmaf(skip, vs[(buf * OR_TB * CT + e) * 2], os[e]) : os[e];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < RP; ++i)
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const int r = lane * 2 * RP + 2 * i;
      const float2 a = unf2(S[i][c]);
      if (my_col + c < p.vdim) {
        if (r < p.dim) st[static_cast<int64_t>(r) * p.vdim + my_col + c] = a.x;
        if (r + 1 < p.dim) st[static_cast<int64_t>(r + 1) * p.vdim + my_col + c] = a.y;
      }
    }
}

// out = o / sqrt(mean(o^2) + eps) * w (* silu(gate)) for rows (token, head); one warp per row
template <typename E>
__global__ void __launch_bounds__(256) head_rms_kernel(const __grid_constant__ OuterRnnParams p, int64_t rows) {
  const int64_t r = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= rows) return;
  const float* x = p.o + r * p.vdim;
  const int64_t token = r / p.heads;
  const int col = static_cast<int>(r - token * p.heads) * p.vdim;
  const E* gate = p.gate ? static_cast<const E*>(p.gate) + token * p.gate_stride + col : nullptr;
  E* out = static_cast<E*>(p.out) + token * p.out_stride + col;
  float sq = 0.f;
  for (int c = lane * 4; c < p.vdim; c += 128) {
    const float4 a = load4(x + c);
    sq += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
  }
  const float scale = 1.0f / sqrtf(warp_sum(sq) / static_cast<float>(p.true_vdim) + p.eps);
  for (int c = lane * 4; c < p.vdim; c += 128) {
    const float4 a = load4(x + c), w = load4(p.norm + c);
    float4 y = make_float4(a.x * scale * w.x, a.y * scale * w.y, a.z * scale * w.z, a.w * scale * w.w);
    if (gate) {
      const float4 g = load4(gate + c);
      y.x *= silu_f<E>(g.x), y.y *= silu_f<E>(g.y), y.z *= silu_f<E>(g.z), y.w *= silu_f<E>(g.w);
    }
    store4(out + c, y);
  }
}

// One token per slot, one CTA per (head, slot): state in, state out, head norm inside.  A warp walks rows, its lanes
// cover the columns four at a time (several rows at once when vdim < 128).  State space: the convolution of the head's
// inputs is inside; a ring of `taps` raw inputs per channel is written at pos % taps, which no CTA reads in this step.
constexpr int OD_WARPS = 8;
constexpr int OD_MAX_VDIM = 512;
template <typename E, RnnKind KIND>
__global__ void __launch_bounds__(OD_WARPS * 32) outer_rnn_decode_kernel(const __grid_constant__ OuterRnnParams p) {
  constexpr bool KEYS = KIND != RNN_FORGET;
  extern __shared__ __align__(16) float od_smem[];
  const int dim = p.dim, vdim = p.vdim, heads = p.heads;
  float* fs = od_smem;            // [dim]
  float* qs = fs + dim;           // [dim]
  float* ks = qs + dim;           // [dim] when KEYS
  float* vv = ks + (KEYS ? dim : 0);   // [vdim]
  float* part = vv + vdim;        // [OD_WARPS][vdim]
  __shared__ float red[32];
  const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  const bool on = !p.active || p.active[b] != 0;
  const int64_t pos = p.pos[b];
  const bool fresh = pos == 0;
  const E* row = static_cast<const E*>(p.x) + b * p.stride;
  const int qk_col = (head / p.per_group) * dim, v_col = p.v_off + head * vdim;
  if constexpr (KIND == RNN_SSD) {
    const float dt = softplus_f(load1(static_cast<const E*>(p.dt) + b * p.dt_stride + head) + p.bias[head]);
    const float decay = expf(-expf(p.a_log[head]) * dt);
    const int now = static_cast<int>(pos % p.taps), back = static_cast<int>(pos < p.taps - 1 ? pos : p.taps - 1);
    float* ring = p.ring + static_cast<int64_t>(b) * p.taps * p.channels;
    const bool first = head % p.per_group == 0;       // writes the group's inputs
    for (int i = tid; i < 2 * dim + vdim; i += OD_WARPS * 32) {
      const int c = i < dim ? p.q_off + qk_col + i : i < 2 * dim ? p.k_off + qk_col + i - dim : v_col + i - 2 * dim;
      const float raw = load1(row + c);
      float acc = fmaf(p.taps_w[c], raw, p.taps_b[c]);
      for (int j = 1; j <= back; ++j)
        acc = fmaf(p.taps_w[j * p.channels + c], ring[static_cast<int64_t>(now - j < 0 ? now - j + p.taps : now - j) * p.channels + c], acc);
      const float y = silu_f<E>(acc);
      if (i < dim) qs[i] = y, fs[i] = decay;
      else if (i < 2 * dim) ks[i - dim] = y * dt;
      else vv[i - 2 * dim] = y;
      if (on && (i >= 2 * dim || first)) ring[static_cast<int64_t>(now) * p.channels + c] = raw;
    }
  } else {
    for (int i = tid; i < dim; i += OD_WARPS * 32) {
      const int ch = head * dim + i;
      if constexpr (KIND == RNN_FORGET) {
        const float l = p.lower[ch];
        qs[i] = silu_f<E>(load1(row + p.q_off + ch));
        fs[i] = l + (1.0f - l) * sigmoid_f<E>(load1(row + p.k_off + ch) + p.bias[ch]);
      } else {
        float z = p.bias[ch];
        const E *w = static_cast<const E*>(p.w_low) + static_cast<int64_t>(ch) * p.rank, *a = static_cast<const E*>(p.low) + b * p.stride;
        for (int r = 0; r < p.rank; r += 4) {
          const float4 x = load4(a + r), y = load4(w + r);
          z = fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, z))));
        }
        qs[i] = load1(row + p.q_off + ch) * p.q_scale;
        ks[i] = load1(row + p.k_off + ch);
        fs[i] = sigmoid_root<E>(z, p.inv_tau);
      }
    }
    for (int i = tid; i < vdim; i += OD_WARPS * 32) vv[i] = load1(row + v_col + i);
  }
  __syncthreads();
  float* st = p.state + (static_cast<int64_t>(b) * heads + head) * dim * vdim;
  const int rows_at_once = 32 / p.lanes_per_row, sub = lane / p.lanes_per_row, cl = (lane % p.lanes_per_row) * 4;
  for (int c0 = 0; c0 < vdim; c0 += 128) {
    const int c = c0 + cl;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < vdim) {
      const float4 v = load4(vv + c);
      constexpr int U = 8;
      const int step = OD_WARPS * rows_at_once;
      for (int r0 = warp * rows_at_once + sub; r0 < dim; r0 += step * U) {
        float4 s[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * step;
          s[u] = (r < dim && !fresh) ? load4(st + static_cast<int64_t>(r) * vdim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int r = r0 + u * step;
          if (r < dim) {
            const float f = fs[r], k = KEYS ? ks[r] : 1.0f - f, q = qs[r];
            s[u].x = fmaf(f, s[u].x, k * v.x), s[u].y = fmaf(f, s[u].y, k * v.y);
            s[u].z = fmaf(f, s[u].z, k * v.z), s[u].w = fmaf(f, s[u].w, k * v.w);
            if (on) store4(st + static_cast<int64_t>(r) * vdim + c, s[u]);
            o.x = fmaf(q, s[u].x, o.x), o.y = fmaf(q, s[u].y, o.y);
            o.z = fmaf(q, s[u].z, o.z), o.w = fmaf(q, s[u].w, o.w);
          }
        }
      }
    }
    for (int bit = p.lanes_per_row; bit < 32; bit <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, bit), o.y += __shfl_xor_sync(0xffffffffu, o.y, bit);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, bit), o.w += __shfl_xor_sync(0xffffffffu, o.w, bit);
    }
    if (sub == 0 && c < vdim) store4(part + warp * vdim + c, o);
  }
  __syncthreads();
  float sum[OD_MAX_VDIM / (OD_WARPS * 32)], sq[1] = {0.f};
#pragma unroll
  for (int i = 0; i < OD_MAX_VDIM / (OD_WARPS * 32); ++i) {
    const int c = tid + i * OD_WARPS * 32;
    sum[i] = 0.f;
    if (c < vdim)
#pragma unroll
      for (int w = 0; w < OD_WARPS; ++w) sum[i] += part[w * vdim + c];
    sq[0] += sum[i] * sum[i];
  }
  if constexpr (KIND == RNN_SSD) {
#pragma unroll
    for (int i = 0; i < OD_MAX_VDIM / (OD_WARPS * 32); ++i) {
      const int c = tid + i * OD_WARPS * 32;
      if (c < vdim) p.o[(static_cast<int64_t>(b) * heads + head) * vdim + c] = fmaf(p.skip[head], vv[c], sum[i]);
    }
    return;
  }
  block_sum<1>(sq, red);
  const float scale = 1.0f / sqrtf(sq[0] / static_cast<float>(p.true_vdim) + p.eps);
#pragma unroll
  for (int i = 0; i < OD_MAX_VDIM / (OD_WARPS * 32); ++i) {
    const int c = tid + i * OD_WARPS * 32;
    if (c < vdim) {
      float y = sum[i] * scale * p.norm[c];
      if (p.gate) y *= silu_f<E>(load1(static_cast<const E*>(p.gate) + b * p.gate_stride + head * vdim + c));
      store1(static_cast<E*>(p.out) + b * p.out_stride + head * vdim + c, y);
    }
  }
}

template <typename E, int RP, int COLS, RnnKind KIND>
static int launch_outer_cols(const OuterRnnParams& p, int n, cudaStream_t st) {
  constexpr int DIM = 64 * RP, CT = OR_WARPS * COLS;
  constexpr int smem = ((KIND == RNN_FORGET ? 4 : 6) * OR_TB * DIM + 2 * OR_TB * CT * 2 + OR_TB * CT) * 4;
  static_assert(smem <= 200 * 1024, "staging must fit");
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (smem > 48 * 1024 && dev >= 0 && dev < 64 && !configured[dev]) {
    if (cudaFuncSetAttribute(outer_rnn_prefill_kernel<E, RP, COLS, KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
      return fail(ERR_RUNTIME, "outer_rnn: cannot raise dynamic shared memory to %d", smem);
    configured[dev] = true;
  }
  outer_rnn_prefill_kernel<E, RP, COLS, KIND><<<dim3((p.vdim + CT - 1) / CT, p.heads, n), OR_THREADS, smem, st>>>(p);
  return check_launch("outer_rnn (token by token)");
}

template <typename E, int RP, RnnKind KIND>
static int launch_outer(const OuterRnnParams& p, int n, cudaStream_t st) {
  // wide columns share the gates of a token among more state; narrow ones give more CTAs when there are few heads
  const int64_t wide = static_cast<int64_t>((p.vdim + 31) / 32) * p.heads * n;
  if constexpr (RP <= 2) {
    if (wide >= 2 * sm_count()) return launch_outer_cols<E, RP, 8, KIND>(p, n, st);
  }
  return launch_outer_cols<E, RP, 4, KIND>(p, n, st);
}

template <typename E, RnnKind KIND>
static int launch_outer_rows(const OuterRnnParams& p, int n, cudaStream_t st) {
  if (p.dim <= 64) return launch_outer<E, 1, KIND>(p, n, st);
  if (p.dim <= 128) return launch_outer<E, 2, KIND>(p, n, st);
  return launch_outer<E, 4, KIND>(p, n, st);
}

int outer_rnn_serial_launch(const OuterRnnParams& p, RnnKind kind, bool f32, int n, cudaStream_t st) {
  B200_REQUIRE(p.dim <= 256, "outer_rnn: at most 256 state rows (got %d)", p.dim);
  if (kind == RNN_FORGET) return f32 ? launch_outer_rows<float, RNN_FORGET>(p, n, st) : launch_outer_rows<__nv_bfloat16, RNN_FORGET>(p, n, st);
  if (kind == RNN_KEYED) return f32 ? launch_outer_rows<float, RNN_KEYED>(p, n, st) : launch_outer_rows<__nv_bfloat16, RNN_KEYED>(p, n, st);
  return f32 ? launch_outer_rows<float, RNN_SSD>(p, n, st) : launch_outer_rows<__nv_bfloat16, RNN_SSD>(p, n, st);
}

template <typename E, RnnKind KIND>
static cudaError_t launch_outer_decode(const OuterRnnParams& p, int batch, int smem, cudaStream_t st) {
  return launch_pdl((p.overlap & OVERLAP_START) != 0, outer_rnn_decode_kernel<E, KIND>, dim3(p.heads, batch), dim3(OD_WARPS * 32), smem, st, p);
}

int outer_rnn_decode_launch(OuterRnnParams p, RnnKind kind, bool f32, int batch, const char* name, cudaStream_t st) {
  B200_REQUIRE(p.dim > 0 && p.dim <= 1024 && p.vdim > 0 && p.vdim % 4 == 0 && p.vdim <= OD_MAX_VDIM && p.true_vdim <= p.vdim,
               "%s: dim at most 1024, vdim a multiple of 4 and at most %d (got %d, %d)", name, OD_MAX_VDIM, p.dim, p.vdim);
  B200_REQUIRE(p.heads > 0 && p.per_group > 0 && batch <= 65535 && aligned16(p.state), "%s: unaligned state or too many slots", name);
  p.lanes_per_row = 1;
  while (p.lanes_per_row < 32 && p.lanes_per_row * 4 < p.vdim) p.lanes_per_row <<= 1;
  const int smem = ((kind == RNN_FORGET ? 2 : 3) * p.dim + p.vdim + OD_WARPS * p.vdim) * 4 + 16;
  cudaError_t e;
  if (kind == RNN_FORGET) e = f32 ? launch_outer_decode<float, RNN_FORGET>(p, batch, smem, st) : launch_outer_decode<__nv_bfloat16, RNN_FORGET>(p, batch, smem, st);
  else if (kind == RNN_KEYED) e = f32 ? launch_outer_decode<float, RNN_KEYED>(p, batch, smem, st) : launch_outer_decode<__nv_bfloat16, RNN_KEYED>(p, batch, smem, st);
  else e = f32 ? launch_outer_decode<float, RNN_SSD>(p, batch, smem, st) : launch_outer_decode<__nv_bfloat16, RNN_SSD>(p, batch, smem, st);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "%s: %s", name, cudaGetErrorString(e));
  return check_launch(name);
}

// FORGET and KEYED, any length: chunks where the shape fits, else token by token; the head norm inside or behind
static int outer_rnn_prefill(OuterRnnParams p, RnnKind kind, bool f32, bool serial, int n, int tokens, cudaStream_t st) {
  float* const scratch = p.o;
  const bool chunked = !f32 && !serial && outer_rnn_chunk_supports(p.dim, p.vdim) && p.stride % 8 == 0 && p.q_off % 8 == 0 &&
                       p.k_off % 8 == 0 && p.v_off % 8 == 0 && p.z_stride % 4 == 0 && aligned16(p.x);
  void* const out = p.out;
  if (chunked && p.vdim <= 128) return outer_rnn_chunk_launch(p, kind, n, st);  // the head norm inside: one launch
  B200_REQUIRE(scratch, "outer_rnn: this shape needs a scratch tensor");
  p.out = nullptr;
  const int rc = chunked ? outer_rnn_chunk_launch(p, kind, n, st) : outer_rnn_serial_launch(p, kind, f32, n, st);
  if (rc != OK) return rc;
  p.out = out;
  const int64_t rows = static_cast<int64_t>(tokens) * p.heads;
  const unsigned grid = static_cast<unsigned>((rows + 7) / 8);
  if (f32) head_rms_kernel<float><<<grid, 256, 0, st>>>(p, rows);
  else head_rms_kernel<__nv_bfloat16><<<grid, 256, 0, st>>>(p, rows);
  return check_launch("outer_rnn (norm)");
}

}  // namespace b200

using namespace b200;

extern "C" int64_t b200_mingru_workspace_bytes(int32_t batch, int32_t segments, int32_t width) {
  return segments > 1 ? static_cast<int64_t>(batch) * (segments + 1) * width * 8 : 0;
}

extern "C" int b200_mingru_prefill(const void* zxg, int64_t stride, const float* bias, float* state, const int32_t* cu_seqlens,
                                   const int32_t* slots, const int32_t* start, void* workspace, void* out, int32_t batch,
                                   int32_t segment, int32_t segments, int32_t width, int32_t f32, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(width > 0 && width % 4 == 0 && stride % 4 == 0 && stride < (1 << 26) && segment > 0 && segments > 0 && batch <= 65535 && segments <= 65535,
               "mingru_prefill: width and stride must be multiples of 4, at most 65535 sequences and segments");
  B200_REQUIRE(aligned16(zxg) && aligned16(bias) && aligned16(state) && aligned16(out) && (segments == 1 || (workspace && aligned16(workspace))),
               "mingru_prefill: tensors must be 16-byte aligned, several segments need a workspace");
  MinGruParams p = {zxg, stride, bias, state, cu_seqlens, slots, start, static_cast<float2*>(workspace), out, width, segment, segments};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((width + MG_COLS - 1) / MG_COLS, segments, batch);
  if (f32) {
    if (segments > 1) mingru_prefill_kernel<float, true><<<grid, MG_WARPS * 32, 0, st>>>(p);
    mingru_prefill_kernel<float, false><<<grid, MG_WARPS * 32, 0, st>>>(p);
  } else {
    if (segments > 1) mingru_prefill_kernel<__nv_bfloat16, true><<<grid, MG_WARPS * 32, 0, st>>>(p);
    mingru_prefill_kernel<__nv_bfloat16, false><<<grid, MG_WARPS * 32, 0, st>>>(p);
  }
  return check_launch("mingru_prefill");
}

extern "C" int b200_mingru_decode(const void* zxg, int64_t stride, const float* bias, float* state, const int64_t* pos,
                                  const int64_t* active, void* out, int32_t batch, int32_t width, int32_t f32,
                                  int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(width > 0 && width % 4 == 0 && stride % 4 == 0 && batch <= 65535,
               "mingru_decode: width and stride must be multiples of 4, at most 65535 slots");
  B200_REQUIRE(aligned16(zxg) && aligned16(bias) && aligned16(state) && aligned16(out), "mingru_decode: unaligned tensor");
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((width / 4 + 127) / 128, batch);
  const bool early = (overlap & OVERLAP_START) != 0;
  const cudaError_t e =
      f32 ? launch_pdl(early, mingru_decode_kernel<float>, grid, dim3(128), 0, st, static_cast<const float*>(zxg), stride, bias,
                       state, pos, active, static_cast<float*>(out), width, overlap)
          : launch_pdl(early, mingru_decode_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, static_cast<const __nv_bfloat16*>(zxg),
                       stride, bias, state, pos, active, static_cast<__nv_bfloat16*>(out), width, overlap);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "mingru_decode: %s", cudaGetErrorString(e));
  return check_launch("mingru_decode");
}

extern "C" int64_t b200_hgrn2_workspace_bytes(int32_t batch, int32_t segments, int32_t heads, int32_t dim, int32_t vdim) {
  return static_cast<int64_t>(batch) * segments * heads * dim * (vdim + 1) * 4;
}

extern "C" int b200_hgrn2_prefill(const void* qfv, int64_t stride, const float* lower, const float* bias, const float* norm,
                                  float* state, const int32_t* cu_seqlens, const int32_t* slots, const int32_t* start,
                                  float* o_scratch, void* out, int32_t batch, int32_t tokens, int32_t heads, int32_t dim,
                                  int32_t vdim, int32_t true_vdim, float eps, int32_t f32, int32_t serial,
                                  int32_t segment, int32_t segments, float* workspace, b200_stream_t stream) {
  if (batch <= 0 || tokens <= 0) return OK;
  B200_REQUIRE(segment > 0 && segments > 0 && (segments == 1 || (segment % 16 == 0 && workspace && aligned16(workspace))),
               "hgrn2_prefill: segments must be multiples of 16 tokens and have a workspace");
  B200_REQUIRE(static_cast<int64_t>(batch) * segments <= 65535, "hgrn2_prefill: too many segments");
  B200_REQUIRE(dim > 0 && dim <= 256 && vdim > 0 && vdim % 4 == 0 && vdim <= OD_MAX_VDIM && true_vdim <= vdim,
               "hgrn2_prefill: dim at most 256, vdim a multiple of 4 and at most %d (got %d, %d)", OD_MAX_VDIM, dim, vdim);
  B200_REQUIRE(heads > 0 && heads <= 65535 && batch <= 65535, "hgrn2_prefill: at most 65535 heads and sequences");
  B200_REQUIRE(aligned16(o_scratch) && aligned16(out) && aligned16(norm), "hgrn2_prefill: unaligned tensor");
  OuterRnnParams p = {};
  p.x = qfv, p.stride = stride, p.q_off = 0, p.k_off = heads * dim, p.v_off = 2 * heads * dim, p.per_group = 1;
  p.lower = lower, p.bias = bias, p.state = state, p.cu = cu_seqlens, p.slots = slots, p.start = start, p.o = o_scratch;
  p.heads = heads, p.dim = dim, p.vdim = vdim, p.norm = norm, p.out = out, p.out_stride = static_cast<int64_t>(heads) * vdim;
  p.true_vdim = true_vdim, p.eps = eps, p.segment = segment, p.segments = segments, p.seg_state = workspace;
  p.seg_decay = workspace ? workspace + static_cast<int64_t>(batch) * segments * heads * dim * vdim : nullptr;
  return outer_rnn_prefill(p, RNN_FORGET, f32 != 0, serial != 0, batch, tokens, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int b200_hgrn2_decode(const void* qfv, int64_t stride, const float* lower, const float* bias, const float* norm,
                                 float* state, const int64_t* pos, const int64_t* active, void* out, int32_t batch,
                                 int32_t heads, int32_t dim, int32_t vdim, int32_t true_vdim, float eps, int32_t f32,
                                 int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  OuterRnnParams p = {};
  p.x = qfv, p.stride = stride, p.q_off = 0, p.k_off = heads * dim, p.v_off = 2 * heads * dim, p.per_group = 1;
  p.lower = lower, p.bias = bias, p.state = state, p.heads = heads, p.dim = dim, p.vdim = vdim, p.norm = norm;
  p.out = out, p.out_stride = static_cast<int64_t>(heads) * vdim, p.true_vdim = true_vdim, p.eps = eps;
  p.pos = pos, p.active = active, p.overlap = overlap;
  return outer_rnn_decode_launch(p, RNN_FORGET, f32 != 0, batch, "hgrn2_decode", reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int b200_gla_prefill(const void* qkv, int64_t stride, const float* z, int64_t z_stride, const float* bias,
                                const float* norm, const void* gate, int64_t gate_stride, float* state,
                                const int32_t* cu_seqlens, const int32_t* slots, const int32_t* start, float* o_scratch,
                                void* out, int64_t out_stride, int32_t batch, int32_t tokens, int32_t heads, int32_t dim,
                                int32_t vdim, int32_t true_vdim, float q_scale, float inv_tau, float eps, int32_t f32,
                                int32_t serial, int32_t segment, int32_t segments, float* workspace, b200_stream_t stream) {
  if (batch <= 0 || tokens <= 0) return OK;
  B200_REQUIRE(segment > 0 && segments > 0 && (segments == 1 || (segment % 16 == 0 && workspace && aligned16(workspace))),
               "gla_prefill: segments must be multiples of 16 tokens and have a workspace");
  B200_REQUIRE(dim > 0 && dim <= 256 && vdim > 0 && vdim % 4 == 0 && vdim <= OD_MAX_VDIM && true_vdim <= vdim,
               "gla_prefill: dim at most 256, vdim a multiple of 4 and at most %d (got %d, %d)", OD_MAX_VDIM, dim, vdim);
  B200_REQUIRE(heads > 0 && heads <= 65535 && static_cast<int64_t>(batch) * segments <= 65535, "gla_prefill: too many heads or segments");
  B200_REQUIRE(aligned16(z) && aligned16(gate) && aligned16(o_scratch) && aligned16(out) && aligned16(norm) &&
                   gate_stride % 8 == 0 && out_stride % 8 == 0,
               "gla_prefill: unaligned tensor");
  OuterRnnParams p = {};
  p.x = qkv, p.stride = stride, p.q_off = 0, p.k_off = heads * dim, p.v_off = 2 * heads * dim, p.per_group = 1;
  p.z = z, p.z_stride = z_stride, p.bias = bias, p.q_scale = q_scale, p.inv_tau = inv_tau;
  p.state = state, p.cu = cu_seqlens, p.slots = slots, p.start = start, p.o = o_scratch;
  p.heads = heads, p.dim = dim, p.vdim = vdim, p.norm = norm, p.gate = gate, p.gate_stride = gate_stride;
  p.out = out, p.out_stride = out_stride, p.true_vdim = true_vdim, p.eps = eps;
  p.segment = segment, p.segments = segments, p.seg_state = workspace;
  p.seg_decay = workspace ? workspace + static_cast<int64_t>(batch) * segments * heads * dim * vdim : nullptr;
  return outer_rnn_prefill(p, RNN_KEYED, f32 != 0, serial != 0, batch, tokens, reinterpret_cast<cudaStream_t>(stream));
}

extern "C" int b200_gla_decode(const void* qkv, int64_t stride, const void* low, const void* w_low, int32_t rank,
                               const float* bias, const float* norm, const void* gate, int64_t gate_stride, float* state,
                               const int64_t* pos, const int64_t* active, void* out, int64_t out_stride, int32_t batch,
                               int32_t heads, int32_t dim, int32_t vdim, int32_t true_vdim, float q_scale, float inv_tau,
                               float eps, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (batch <= 0) return OK;
  B200_REQUIRE(rank > 0 && rank % 4 == 0 && stride % 4 == 0 && aligned16(low) && aligned16(w_low),
               "gla_decode: the rank and the stride must be multiples of 4, tensors 16-byte aligned");
  OuterRnnParams p = {};
  p.x = qkv, p.stride = stride, p.q_off = 0, p.k_off = heads * dim, p.v_off = 2 * heads * dim, p.per_group = 1;
  p.low = low, p.w_low = w_low, p.rank = rank, p.bias = bias, p.q_scale = q_scale, p.inv_tau = inv_tau;
  p.state = state, p.heads = heads, p.dim = dim, p.vdim = vdim, p.norm = norm, p.gate = gate, p.gate_stride = gate_stride;
  p.out = out, p.out_stride = out_stride, p.true_vdim = true_vdim, p.eps = eps;
  p.pos = pos, p.active = active, p.overlap = overlap;
  return outer_rnn_decode_launch(p, RNN_KEYED, f32 != 0, batch, "gla_decode", reinterpret_cast<cudaStream_t>(stream));
}
