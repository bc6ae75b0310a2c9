// Hyper-connected residual streams: the step between two sublayers of a stack that keeps S copies of the residual, one
// launch for what would be a mix of the streams, the weighted return of the sublayer's output, the read-out of the next
// sublayer's input and its RMS norm with a single gain:
//     x_t <- sum_s mix[s, t] x_s + out[t] * y        (all streams from the old ones)
//     h   = (sum_s in[s] x_s) / sqrt(mean(.^2) + eps) * gain
// (gains: an optional vector over the width on top of the single gain; one stream with unit weights and a gain vector is
// the plain residual with an RMS norm).  Streams live in fp32 [rows, S, width]; y and h are bf16 or fp32 activations.  Without y the streams come from the
// embedding table (every stream equal to the token's row), or are only read.
// HBM / latency bound: one CTA per row, a thread owns 4 columns of every stream per step, all loads before the
// reduction.  Width is padded to a multiple of 4 with zero columns; the mean runs over the true width.
#include "b200_attn.h"
#include "elem.cuh"

namespace b200 {

constexpr int HC_MAX_WIDTH = 8192;
constexpr int HC_MAX_STREAMS = 16;

struct HyperParams {
  const void* ids;        // embedding form: token ids of the rows
  int ids_are_int64;
  const void* table;      // [vocab, width] E
  float* streams;         // [rows, S, width]
  const void* y;          // [parts][rows, width] E, summed, or NULL
  int parts;
  int64_t part_stride;
  const float* weights;   // [mix S*S | out S | in S | gain]
  const float* gains;     // [width] or NULL
  void* h;                // [rows, width] E
  int s, width, true_width, overlap;
  float eps;
};

// V: float4 groups a thread may own.  EXTRA: norm weights or several parts of y
template <typename E, int MAXS, int V, bool EXTRA>
__global__ void __launch_bounds__(512) hyper_connect_kernel(const __grid_constant__ HyperParams p) {
  __shared__ float wt[HC_MAX_STREAMS * HC_MAX_STREAMS + 2 * HC_MAX_STREAMS + 1];
  __shared__ float red[32];
  const int row = blockIdx.x, tid = threadIdx.x, s = p.s, width = p.width;
  for (int i = tid; i < s * s + 2 * s + 1; i += blockDim.x) wt[i] = p.weights[i];
  if (p.overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  __syncthreads();
  const float *mix = wt, *out = wt + s * s, *in = out + s;
  float* x = p.streams + static_cast<int64_t>(row) * s * width;
  float4 u[V], g[V];
  float sq[1] = {0.f};
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int c = (tid + v * blockDim.x) * 4;
    u[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    g[v] = make_float4(1.f, 1.f, 1.f, 1.f);
    if (c >= width) continue;
    if (EXTRA && p.gains) g[v] = load4(p.gains + c);
    if (p.ids) {
      const int64_t id = p.ids_are_int64 ? static_cast<const int64_t*>(p.ids)[row]
                                         : static_cast<int64_t>(static_cast<const int32_t*>(p.ids)[row]);
      const float4 e = load4(static_cast<const E*>(p.table) + id * width + c);
      float total = 0.f;
#pragma unroll
      for (int i = 0; i < MAXS; ++i)
        if (i < s) {
          store4(x + i * width + c, e);
          total += in[i];
        }
      u[v] = make_float4(total * e.x, total * e.y, total * e.z, total * e.w);
    } else {
      float4 old[MAXS];
#pragma unroll
      for (int i = 0; i < MAXS; ++i)
        if (i < s) old[i] = load4(x + i * width + c);
      if (p.y) {
        float4 y = load4(static_cast<const E*>(p.y) + static_cast<int64_t>(row) * width + c);
        if (EXTRA && p.parts > 1)
          for (int i = 1; i < p.parts; ++i) {
            const float4 more = load4(static_cast<const E*>(p.y) + i * p.part_stride + static_cast<int64_t>(row) * width + c);
            y.x += more.x, y.y += more.y, y.z += more.z, y.w += more.w;
          }
#pragma unroll
        for (int t = 0; t < MAXS; ++t)
          if (t < s) {
            const float o = out[t];
            float4 a = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
            for (int i = 0; i < MAXS; ++i)
              if (i < s) {
                const float m = mix[i * s + t];
                a.x = fmaf(m, old[i].x, a.x), a.y = fmaf(m, old[i].y, a.y);
                a.z = fmaf(m, old[i].z, a.z), a.w = fmaf(m, old[i].w, a.w);
              }
            store4(x + t * width + c, a);
            const float n = in[t];
            u[v].x = fmaf(n, a.x, u[v].x), u[v].y = fmaf(n, a.y, u[v].y);
            u[v].z = fmaf(n, a.z, u[v].z), u[v].w = fmaf(n, a.w, u[v].w);
          }
      } else {
#pragma unroll
        for (int i = 0; i < MAXS; ++i)
          if (i < s) {
            const float n = in[i];
            u[v].x = fmaf(n, old[i].x, u[v].x), u[v].y = fmaf(n, old[i].y, u[v].y);
            u[v].z = fmaf(n, old[i].z, u[v].z), u[v].w = fmaf(n, old[i].w, u[v].w);
          }
      }
    }
    sq[0] += u[v].x * u[v].x + u[v].y * u[v].y + u[v].z * u[v].z + u[v].w * u[v].w;
  }
  block_sum<1>(sq, red);
  const float scale = wt[s * s + 2 * s] / sqrtf(sq[0] / static_cast<float>(p.true_width) + p.eps);
  E* h = static_cast<E*>(p.h) + static_cast<int64_t>(row) * width;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int c = (tid + v * blockDim.x) * 4;
    if (c >= width) continue;
    store4(h + c, make_float4(u[v].x * scale * g[v].x, u[v].y * scale * g[v].y, u[v].z * scale * g[v].z, u[v].w * scale * g[v].w));
  }
}

template <typename E, int MAXS, bool EXTRA>
static cudaError_t launch_hyper_form(const HyperParams& p, int rows, cudaStream_t st) {
  const int quads = p.width / 4;
  const bool early = (p.overlap & OVERLAP_START) != 0;
  int threads = (quads + 31) / 32 * 32;
  if (threads <= 512) return launch_pdl(early, hyper_connect_kernel<E, MAXS, 1, EXTRA>, dim3(rows), dim3(threads), 0, st, p);
  threads = ((quads + 3) / 4 + 31) / 32 * 32;
  return launch_pdl(early, hyper_connect_kernel<E, MAXS, 4, EXTRA>, dim3(rows), dim3(threads), 0, st, p);
}

template <typename E, int MAXS>
static cudaError_t launch_hyper(const HyperParams& p, int rows, cudaStream_t st) {
  return p.gains || p.parts > 1 ? launch_hyper_form<E, MAXS, true>(p, rows, st) : launch_hyper_form<E, MAXS, false>(p, rows, st);
}

template <typename E>
static cudaError_t launch_hyper_e(const HyperParams& p, int rows, cudaStream_t st) {
  if (p.s == 1) return launch_hyper<E, 1>(p, rows, st);
  if (p.s == 2) return launch_hyper<E, 2>(p, rows, st);
  if (p.s <= 4) return launch_hyper<E, 4>(p, rows, st);
  return launch_hyper<E, HC_MAX_STREAMS>(p, rows, st);
}

// out[r, c] = act(x[r, c]) * x[r, up + c] over strided rows; act: silu or the tanh form of gelu.  A thread takes 8 columns
// of ROWS consecutive rows, all loads before the first use.
template <typename E>
__device__ __forceinline__ float gate_act(float z, int act) {
  if (act == B200_ACT_SILU) return silu_f<E>(z);
  // 0.5 z (1 + tanh(u)) = z * sigmoid(2 u)
  return z * sigmoid_f<E>(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
}

template <typename E, int ROWS>
__global__ void __launch_bounds__(128) gated_act_kernel(const E* x, int64_t stride, int up, E* out, int64_t out_stride, int rows,
                                                        int width, int act, int overlap) {
  if (overlap & OVERLAP_TRIGGER) pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= width) return;
  float g[ROWS][8], u[ROWS][8];
  const int64_t r0 = static_cast<int64_t>(blockIdx.y) * ROWS;
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const E* row = x + min(r0 + i, static_cast<int64_t>(rows) - 1) * stride + c;
    load8(row, g[i]);
    load8(row + up, u[i]);
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    if (r0 + i >= rows) break;
#pragma unroll
    for (int j = 0; j < 8; ++j) g[i][j] = gate_act<E>(g[i][j], act) * u[i][j];
    store8(out + (r0 + i) * out_stride + c, g[i]);
  }
}

// logits <- cap * tanh(logits / cap), columns behind `vocab` become -inf
__global__ void __launch_bounds__(256) softcap_kernel(float* logits, int64_t stride, int vocab, int width, float cap) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (c >= width) return;
  float* at = logits + static_cast<int64_t>(blockIdx.y) * stride + c;
  const float4 a = load4(at);
  float f[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) f[i] = c + i < vocab ? cap * tanhf(f[i] / cap) : -INFINITY;
  store4(at, make_float4(f[0], f[1], f[2], f[3]));
}

// out[r, c] = silu(gate_up[r, c]) * gate_up[r, width + c] for fp32 activations (the bf16 form is b200_swiglu)
__global__ void __launch_bounds__(256) swiglu_f32_kernel(const float* gate_up, int64_t stride, float* out, int width) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= width) return;
  const float* row = gate_up + blockIdx.y * stride;
  const float4 g = load4(row + c), u = load4(row + width + c);
  store4(out + static_cast<int64_t>(blockIdx.y) * width + c,
         make_float4(silu_f<float>(g.x) * u.x, silu_f<float>(g.y) * u.y, silu_f<float>(g.z) * u.z, silu_f<float>(g.w) * u.w));
}

}  // namespace b200

using namespace b200;

extern "C" int b200_hyper_connect(const void* ids, int32_t ids_are_int64, const void* table, float* streams, const void* y,
                                  int32_t y_parts, const float* weights, const float* gains, void* h, int32_t rows, int32_t num_streams, int32_t width,
                                  int32_t true_width, float eps, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(num_streams >= 1 && num_streams <= HC_MAX_STREAMS, "hyper_connect: 1 to %d streams (got %d)",
               HC_MAX_STREAMS, num_streams);
  B200_REQUIRE(width > 0 && width % 4 == 0 && width <= HC_MAX_WIDTH && true_width > 0 && true_width <= width,
               "hyper_connect: width must be a multiple of 4, at most %d, and cover the true width (got %d, %d)",
               HC_MAX_WIDTH, width, true_width);
  B200_REQUIRE(streams && weights && h && aligned16(streams) && aligned16(h) && aligned16(y) && aligned16(gains),
               "hyper_connect: NULL or unaligned tensor");
  B200_REQUIRE(!y || y_parts >= 1, "hyper_connect: y comes in at least one part");
  B200_REQUIRE(!ids || (table && aligned16(table) && !y), "hyper_connect: the embedding form takes a table, no y");
  HyperParams p = {ids, ids_are_int64, table, streams, y, y_parts, static_cast<int64_t>(rows) * width, weights, gains, h, num_streams, width, true_width, overlap, eps};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = f32 ? launch_hyper_e<float>(p, rows, st) : launch_hyper_e<__nv_bfloat16>(p, rows, st);
  if (e != cudaSuccess) return fail(ERR_LAUNCH, "hyper_connect: %s", cudaGetErrorString(e));
  return check_launch("hyper_connect");
}

extern "C" int b200_swiglu_f32(const float* gate_up, int64_t row_stride, float* out, int32_t rows, int32_t intermediate,
                               b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(intermediate > 0 && intermediate % 4 == 0 && row_stride % 4 == 0 && aligned16(gate_up) && aligned16(out),
               "swiglu_f32: width and stride must be multiples of 4, tensors 16-byte aligned");
  for (int r0 = 0; r0 < rows; r0 += 65535) {
    const int n = rows - r0 < 65535 ? rows - r0 : 65535;
    swiglu_f32_kernel<<<dim3((intermediate / 4 + 255) / 256, n), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
        gate_up + r0 * row_stride, row_stride, out + static_cast<int64_t>(r0) * intermediate, intermediate);
  }
  return check_launch("swiglu_f32");
}

extern "C" int b200_gated_act(const void* x, int64_t stride, int32_t up, void* out, int64_t out_stride, int32_t rows,
                              int32_t width, int32_t act, int32_t f32, int32_t overlap, b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(width > 0 && width % 8 == 0 && stride % 8 == 0 && up % 8 == 0 && out_stride % 8 == 0 && aligned16(x) && aligned16(out),
               "gated_act: width, offset and strides must be multiples of 8, tensors 16-byte aligned");
  B200_REQUIRE(act == B200_ACT_SILU || act == B200_ACT_GELU_TANH, "gated_act: unknown activation %d", act);
  const bool early = (overlap & OVERLAP_START) != 0;
  const int per = rows >= GLUE_WIDE_ROWS ? 4 : 1;
  const unsigned cols = (width / 8 + 127) / 128;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  for (int64_t r0 = 0; r0 < rows; r0 += 65535ll * per) {
    const int n = static_cast<int>(rows - r0 < 65535ll * per ? rows - r0 : 65535ll * per);
    const dim3 grid(cols, (n + per - 1) / per), block(128);
    cudaError_t e;
    if (f32) {
      const float* a = static_cast<const float*>(x) + r0 * stride;
      float* o = static_cast<float*>(out) + r0 * out_stride;
      e = per == 4 ? launch_pdl(early, gated_act_kernel<float, 4>, grid, block, 0, st, a, stride, up, o, out_stride, n, width, act, overlap)
                   : launch_pdl(early, gated_act_kernel<float, 1>, grid, block, 0, st, a, stride, up, o, out_stride, n, width, act, overlap);
    } else {
      const __nv_bfloat16* a = static_cast<const __nv_bfloat16*>(x) + r0 * stride;
      __nv_bfloat16* o = static_cast<__nv_bfloat16*>(out) + r0 * out_stride;
      e = per == 4 ? launch_pdl(early, gated_act_kernel<__nv_bfloat16, 4>, grid, block, 0, st, a, stride, up, o, out_stride, n, width, act, overlap)
                   : launch_pdl(early, gated_act_kernel<__nv_bfloat16, 1>, grid, block, 0, st, a, stride, up, o, out_stride, n, width, act, overlap);
    }
    if (e != cudaSuccess) return fail(ERR_LAUNCH, "gated_act: %s", cudaGetErrorString(e));
  }
  return check_launch("gated_act");
}

extern "C" int b200_softcap(float* logits, int64_t stride, int32_t rows, int32_t vocab, int32_t width, float cap,
                            b200_stream_t stream) {
  if (rows <= 0) return OK;
  B200_REQUIRE(width > 0 && width % 4 == 0 && stride % 4 == 0 && vocab > 0 && vocab <= width && cap > 0.f && aligned16(logits),
               "softcap: width and stride must be multiples of 4, the cap positive");
  for (int r0 = 0; r0 < rows; r0 += 65535) {
    const int n = rows - r0 < 65535 ? rows - r0 : 65535;
    softcap_kernel<<<dim3((width / 4 + 255) / 256, n), 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(
        logits + r0 * stride, stride, vocab, width, cap);
  }
  return check_launch("softcap");
}
