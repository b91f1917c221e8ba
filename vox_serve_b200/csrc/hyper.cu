// Hyper-connections: a residual stream kept as S parallel copies x_1 .. x_S (fp32 rows [T][S][W]) instead of one.
//
// A sublayer reads one weighted sum of the copies and its output y enters all of them:
//   u = sum_s in[s] x_s        y = sublayer(norm(u))        x_t <- sum_s mix[s][t] x_s + out[t] (y + bias)
// Between two sublayers all of that is element-wise along a row but for the norm, so ONE kernel per sublayer boundary writes
// the new copies, forms the next sublayer's u from them while they are in registers, norms it and hands it on: the copies move
// through memory once per sublayer.  Three more forms of the same kernel:
//   start        every copy begins as the row x0 (an embedding); nothing is mixed
//   end          no norm weight: the plain sum of the copies (in == nullptr: coefficients of one) leaves as the ordinary stream
//   single rows  steps in which every request brings one row: a causal convolution over time (h + conv(h), short_conv.cu's
//                arithmetic and state slots) runs on the normed row in the same launch, since a row's earlier inputs are all in
//                its request's slot
// Every value is an fp32 chain in a fixed order (streams ascending, then the sublayer's output), whatever else the step holds.
#include "../../include/vb_api.h"
#define VB_PDL_FAMILY 4
#include "common.cuh"

namespace vb {

constexpr int HY_MAX_STREAMS = 16, HY_MAX_KEEP = 3;      // taps of the fused convolution: at most HY_MAX_KEEP + 1

struct HyperParams {
  float* xs;              // [T][S][W]
  const float* x0;        // [T][W]: start form, or nullptr
  const float* y;         // [T][W] the sublayer's output (nullptr in the start form)
  const float* bias;      // [W] or nullptr
  const float* mix;       // [S][S], [from][to]
  const float* out_c;     // [S]
  const float* in_c;      // [S] of the next sublayer, or nullptr: ones
  const float* w;         // [W] norm weight of the next sublayer, or nullptr: u leaves un-normed
  void* h;                // [T][W] operand type, or nullptr
  float* h32;             // [T][W] fp32, or nullptr
  int T, W, S, keep_streams;
  float eps;
  const float* conv_w;    // [W][taps] (single rows), or nullptr
  float* conv_state;      // [slots][taps - 1][W]
  int taps;
  const int32_t* pos;     // [T]
  const int32_t* slots;   // [T]: row t is request t
};

template <typename T> __device__ __forceinline__ T hy_from_f(float v);
template <> __device__ __forceinline__ float hy_from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 hy_from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

template <int V> __device__ __forceinline__ void hy_load(const float* __restrict__ p, float (&v)[V]) {
  if constexpr (V == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else {
    v[0] = p[0];
  }
}
template <int V> __device__ __forceinline__ void hy_store(float* __restrict__ p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void hy_store_ct(float* __restrict__ p, const float (&v)[V]) { hy_store<V>(p, v); }
template <int V> __device__ __forceinline__ void hy_store_ct(__nv_bfloat16* __restrict__ p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
  else p[0] = __float2bfloat16_rn(v[0]);
}

// one row per CTA; SN: the number of copies when it is known at compile time, 0: p.S (at most HY_MAX_STREAMS); V: columns a
// thread handles at a time (4 where width and pointers allow 16-byte accesses)
template <typename OT, int SN, int V>
__global__ void __launch_bounds__(512) hyper_mix_norm_kernel(HyperParams p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int MS = SN > 0 ? SN : HY_MAX_STREAMS;
  const int S = SN > 0 ? SN : p.S, W = p.W;
  const bool conv = p.conv_w != nullptr;
  float* row = sm;                                  // [W] u
  float* hist = row + W;                            // [W] the convolution's earlier taps (single rows)
  float* coef = hist + (conv ? W : 0);              // [S][S] mix | [S] out | [S] in
  float* red = coef + S * (S + 2);                  // [16]
  for (int i = threadIdx.x; i < S * (S + 2); i += blockDim.x) {
    float c;
    if (i < S * S) c = p.mix ? p.mix[i] : 0.f;
    else if (i < S * S + S) c = p.out_c ? p.out_c[i - S * S] : 0.f;
    else c = p.in_c ? p.in_c[i - S * S - S] : 1.f;
    coef[i] = c;
  }
  __syncthreads();
  pdl_sync();
  const float* c_mix = coef;
  const float* c_out = coef + S * S;
  const float* c_in = c_out + S;
  const size_t t = blockIdx.x;
  float* xr = p.xs + t * S * W;
  const int K = p.taps - 1;
  int ps = 0;
  float* st = nullptr;
  if (conv) {
    ps = p.pos[t];
    st = p.conv_state + static_cast<size_t>(p.slots[t]) * K * W;
  }
  float q = 0.f;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float nx[MS][V], u[V];
    if (p.x0) {
      float e[V];
      hy_load<V>(p.x0 + t * W + c, e);
#pragma unroll
      for (int s = 0; s < MS; ++s)
        if (SN > 0 || s < S)
#pragma unroll
          for (int v = 0; v < V; ++v) nx[s][v] = e[v];
    } else {
      float x[MS][V], y[V], b[V];
#pragma unroll
      for (int s = 0; s < MS; ++s)
        if (SN > 0 || s < S) hy_load<V>(xr + static_cast<size_t>(s) * W + c, x[s]);
      hy_load<V>(p.y + t * W + c, y);
      if (p.bias) {
        hy_load<V>(p.bias + c, b);
#pragma unroll
        for (int v = 0; v < V; ++v) y[v] += b[v];
      }
#pragma unroll
      for (int d = 0; d < MS; ++d) {
        if (SN > 0 || d < S) {
#pragma unroll
          for (int v = 0; v < V; ++v) nx[d][v] = 0.f;
#pragma unroll
          for (int s = 0; s < MS; ++s)
            if (SN > 0 || s < S) {
              const float m = c_mix[s * S + d];
#pragma unroll
              for (int v = 0; v < V; ++v) nx[d][v] = fmaf(m, x[s][v], nx[d][v]);
            }
          const float o = c_out[d];
#pragma unroll
          for (int v = 0; v < V; ++v) nx[d][v] = fmaf(o, y[v], nx[d][v]);
        }
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) u[v] = 0.f;
#pragma unroll
    for (int s = 0; s < MS; ++s)
      if (SN > 0 || s < S) {
        const float a = c_in[s];
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = fmaf(a, nx[s][v], u[v]);
        if (p.keep_streams) hy_store<V>(xr + static_cast<size_t>(s) * W + c, nx[s]);
      }
    if (p.w == nullptr) {
      hy_store<V>(p.h32 + t * W + c, u);
      continue;
    }
#pragma unroll
    for (int v = 0; v < V; ++v) q = fmaf(u[v], u[v], q);
    hy_store<V>(row + c, u);
    if (conv) {
      // slot entry j holds the input of position ps - K + j; entries before position 0 count as zero, whatever they hold
      float old[HY_MAX_KEEP][V], acc[V];
#pragma unroll
      for (int v = 0; v < V; ++v) acc[v] = 0.f;
#pragma unroll
      for (int j = 0; j < HY_MAX_KEEP; ++j)
        if (j < K) {
          hy_load<V>(st + static_cast<size_t>(j) * W + c, old[j]);
          if (ps - K + j < 0)
#pragma unroll
            for (int v = 0; v < V; ++v) old[j][v] = 0.f;
        }
#pragma unroll
      for (int j = 0; j < HY_MAX_KEEP; ++j)
        if (j < K) {
#pragma unroll
          for (int v = 0; v < V; ++v) acc[v] = fmaf(p.conv_w[static_cast<size_t>(c + v) * p.taps + j], old[j][v], acc[v]);
          if (j > 0) hy_store<V>(st + static_cast<size_t>(j - 1) * W + c, old[j]);
        }
      hy_store<V>(hist + c, acc);
    }
  }
  if (p.w == nullptr) return;
  // (the block's sum of squares, added in the same order by every warp)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  q = warp_sum(q);
  if (lane == 0) red[warp] = q;
  __syncthreads();
  q = warp_sum(lane < nw ? red[lane] : 0.f);
  const float rs = 1.f / sqrtf(q / W + p.eps);
  OT* h = static_cast<OT*>(p.h);
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float v[V], w[V];
    hy_load<V>(row + c, v);
    hy_load<V>(p.w + c, w);
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = v[e] * rs * w[e];
    if (conv) {
      float a[V];
      hy_load<V>(hist + c, a);
      if (K > 0) hy_store<V>(st + static_cast<size_t>(K - 1) * W + c, v);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = fmaf(p.conv_w[static_cast<size_t>(c + e) * p.taps + K], v[e], a[e]) + v[e];
    }
    if (p.h32) hy_store<V>(p.h32 + t * W + c, v);
    if (h) hy_store_ct<V>(h + t * W + c, v);
  }
}

template <typename OT, int SN, int V>
static int launch_hyper_v(const HyperParams& p, int threads, size_t smem, cudaStream_t stream) {
  if (smem > 48 * 1024) VB_CHECK_CUDA(cudaFuncSetAttribute(hyper_mix_norm_kernel<OT, SN, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM));
  VB_LAUNCH_PDL((hyper_mix_norm_kernel<OT, SN, V>), p.T, threads, smem, stream, p);
  return 0;
}

template <typename OT, int SN>
static int launch_hyper(const HyperParams& p, bool vec, int threads, size_t smem, cudaStream_t stream) {
  return vec ? launch_hyper_v<OT, SN, 4>(p, threads, smem, stream) : launch_hyper_v<OT, SN, 1>(p, threads, smem, stream);
}

template <typename OT>
static int launch_hyper_streams(const HyperParams& p, bool vec, int threads, size_t smem, cudaStream_t stream) {
  switch (p.S) {
    case 1: return launch_hyper<OT, 1>(p, vec, threads, smem, stream);
    case 2: return launch_hyper<OT, 2>(p, vec, threads, smem, stream);
    case 3: return launch_hyper<OT, 3>(p, vec, threads, smem, stream);
    case 4: return launch_hyper<OT, 4>(p, vec, threads, smem, stream);
    default: return launch_hyper_v<OT, 0, 1>(p, threads, smem, stream);
  }
}

}  // namespace vb

using namespace vb;

extern "C" {

int vb_hyper_mix_norm(float* d_xs, int streams, const float* d_x0, const float* d_y, const float* d_bias, const float* d_mix,
                      const float* d_out_c, const float* d_in_c, const float* d_w, void* d_h, float* d_h32, int T, int width,
                      float eps, const float* d_conv_w, int taps, float* d_conv_state, const int32_t* d_pos,
                      const int32_t* d_slots, int keep_streams, int out_dtype, void* stream) {
  VB_CHECK_ARG(d_xs && streams >= 1 && streams <= HY_MAX_STREAMS && width > 0, "vb_hyper_mix_norm: %d streams (1..%d) of width %d",
               streams, HY_MAX_STREAMS, width);
  VB_CHECK_ARG(d_x0 || (d_y && d_mix && d_out_c), "vb_hyper_mix_norm: a sublayer's output needs its mixing coefficients");
  VB_CHECK_ARG(d_w ? (d_h || d_h32) : (d_h32 && !d_h && !d_conv_w), "vb_hyper_mix_norm: bad outputs");
  VB_CHECK_ARG(!d_conv_w || (taps >= 1 && taps <= HY_MAX_KEEP + 1 && d_pos && d_slots && (taps == 1 || d_conv_state)),
               "vb_hyper_mix_norm: convolution of %d taps (1..%d) needs positions, slots and their state", taps, HY_MAX_KEEP + 1);
  if (T <= 0) return 0;
  HyperParams p{d_xs, d_x0, d_y, d_bias, d_mix, d_out_c, d_in_c, d_w, d_h, d_h32, T, width, streams, keep_streams, eps,
                d_conv_w, d_conv_state, d_conv_w ? taps : 1, d_pos, d_slots};
  auto al16 = [](const void* q) { return q == nullptr || reinterpret_cast<uintptr_t>(q) % 16 == 0; };
  const bool vec = width % 4 == 0 && al16(d_xs) && al16(d_x0) && al16(d_y) && al16(d_bias) && al16(d_w) && al16(d_h) && al16(d_h32) &&
                   al16(d_conv_state);
  const size_t smem = (static_cast<size_t>(width) * (d_conv_w ? 2 : 1) + streams * (streams + 2) + 16) * sizeof(float);
  VB_CHECK_ARG(smem <= static_cast<size_t>(VB_MAX_DYN_SMEM), "vb_hyper_mix_norm: width %d too large", width);
  // few rows: more threads per row; many rows: CTAs of 256 threads, several per SM
  const int per = (width + (vec ? 4 : 1) - 1) / (vec ? 4 : 1);
  const int threads = min(T <= 148 ? 512 : 256, max(32, (per + 31) / 32 * 32));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return out_dtype == 1 ? launch_hyper_streams<float>(p, vec, threads, smem, s) : launch_hyper_streams<__nv_bfloat16>(p, vec, threads, smem, s);
}

}  // extern "C"
