// Element-wise gated recurrences over a per-request fp32 state slot, whose gates read only the current token.
//
// minGRU:
//   z_t = sigmoid(pz_t + bz)                       update gate
//   c_t = u + 1/2 (u >= 0), sigmoid(u) (u < 0)     candidate, u = px_t + bx   (positive and continuous at 0)
//   S_t = (1 - z_t) S_(t-1) + z_t c_t              per channel, S = 0 before a request's position 0
//   out_t = S_t * silu(pg_t)
//
// pz | px | pg are columns of the fp32 rows of a fused projection.  Everything here is fp32; only `out` takes the compute
// type (it feeds the output projection).  A slot's stored state is ignored when the request's first row of the step has
// position 0, so slots are handed out again without clearing.
//
//   vb_mingru        one thread per (request, channel) walks the request's rows in order: single-token rows and short portions
//   vb_mingru_tiled  prompt portions cut into pieces of rows: the recurrence S_t = a_t S_(t-1) + b_t composes as
//                    (A, B) = (prod a, local end state from zero), so pieces are summarised in parallel, a short scan over a
//                    request's pieces carries the state in, and the pieces then produce their rows in parallel.
//
// Real-gated linear recurrent unit (Griffin: De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for
// Efficient Language Models"):
//   r_t = sigmoid(R_b u_t + br),  i_t = sigmoid(I_b u_t + bi)     in every block b of neighbouring channels, R_b, I_b square
//   log a_t = -rate r_t (rate = c softplus(lam)),  S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,  out_t = S_t * gelu_tanh(y_t + by)
//   vb_rglru         one kernel forms the gates of all rows (block-diagonal products: tensor cores for bf16 matrices whose
//                    blocks are multiples of 16 channels, with u split into two bf16 terms so that a product keeps 16 bits of
//                    u's mantissa; fp32 FMAs otherwise) and finishes the rows of requests that bring one row; the others leave
//                    (a, sqrt(1 - a^2) i u) per channel, which a walk in order or the piecewise scan above turns into rows.
#include "../../include/vb_api.h"
#define VB_PDL_FAMILY 1
#include "common.cuh"

namespace vb {

struct MinGruParams {
  const float* proj;      // [T][ldp]
  int ldp, z_off, x_off, g_off;
  const float* bz;        // [width] or nullptr
  const float* bx;
  float* state;           // [slots][width]
  void* out;              // [T][width]
  const int32_t* qo_indptr;
  const int32_t* pos;
  const int32_t* slots;
  int B, width;
  int single_rows, multi_rows;      // which requests this launch serves: those bringing one row / several rows
  // tiled form
  const int32_t* tile_req;
  const int32_t* tile_row0;
  int n_tiles, tile_rows;
  float* scratch;         // [n_tiles * pieces per tile][2][width]: A, B of every piece; after the scan [..][0] is its carry-in
};

__device__ __forceinline__ float mg_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ void mg_gates(const float* __restrict__ row, const MinGruParams& p, int ch, float bz, float bx,
                                         float& z, float& c) {
  z = mg_sigmoid(row[p.z_off + ch] + bz);
  const float u = row[p.x_off + ch] + bx;
  c = u >= 0.f ? u + 0.5f : mg_sigmoid(u);
}
template <typename CT> __device__ __forceinline__ void mg_store(void* out, size_t i, float v);
template <> __device__ __forceinline__ void mg_store<float>(void* out, size_t i, float v) { static_cast<float*>(out)[i] = v; }
template <> __device__ __forceinline__ void mg_store<__nv_bfloat16>(void* out, size_t i, float v) {
  static_cast<__nv_bfloat16*>(out)[i] = __float2bfloat16_rn(v);
}

template <typename CT>
__global__ void __launch_bounds__(128) mingru_seq_kernel(MinGruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
  if (ch >= p.width) return;
  const int r0 = p.qo_indptr[b], r1 = p.qo_indptr[b + 1];
  const int n = r1 - r0;
  if (n <= 0 || (n == 1 && !p.single_rows) || (n > 1 && !p.multi_rows)) return;
  float* st = p.state + static_cast<size_t>(p.slots[b]) * p.width + ch;
  float S = p.pos[r0] == 0 ? 0.f : *st;
  const float bz = p.bz ? p.bz[ch] : 0.f, bx = p.bx ? p.bx[ch] : 0.f;
  for (int t = r0; t < r1; ++t) {
    const float* row = p.proj + static_cast<size_t>(t) * p.ldp;
    float z, c;
    mg_gates(row, p, ch, bz, bx, z, c);
    S = (1.f - z) * S + z * c;
    const float g = row[p.g_off + ch];
    mg_store<CT>(p.out, static_cast<size_t>(t) * p.width + ch, S * (g * mg_sigmoid(g)));
  }
  *st = S;
}

// Prompt portions.  A tile (tile_rows rows of one request, as the attention kernels use them) is cut into pieces of MG_ROWS
// rows; piece j of tile i is summary slot i * pieces_per_tile + j.  A thread owns one channel of one piece and first loads
// all of the piece's gate inputs (independent loads, all in flight), then runs the short dependent chain over them.
constexpr int MG_ROWS = 16;

// piece summaries: A = prod (1 - z_t), B = the piece's end state from a zero start
__global__ void __launch_bounds__(128) mingru_tile_sum_kernel(MinGruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, ppt = p.tile_rows / MG_ROWS;
  const int tile = blockIdx.y / ppt, piece = blockIdx.y - tile * ppt;
  if (ch >= p.width) return;
  const int b = p.tile_req[tile], r0 = p.tile_row0[tile] + piece * MG_ROWS;
  const int n = min(min(r0 + MG_ROWS, p.tile_row0[tile] + p.tile_rows), p.qo_indptr[b + 1]) - r0;
  float* s = p.scratch + static_cast<size_t>(blockIdx.y) * 2 * p.width;
  if (n <= 0) { s[ch] = 1.f; s[p.width + ch] = 0.f; return; }
  const float bz = p.bz ? p.bz[ch] : 0.f, bx = p.bx ? p.bx[ch] : 0.f;
  float pz[MG_ROWS], px[MG_ROWS];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    const float* row = p.proj + static_cast<size_t>(r0 + min(i, n - 1)) * p.ldp;
    pz[i] = row[p.z_off + ch];
    px[i] = row[p.x_off + ch];
  }
  float A = 1.f, Bv = 0.f;
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    if (i < n) {
      const float z = mg_sigmoid(pz[i] + bz), u = px[i] + bx;
      const float c = u >= 0.f ? u + 0.5f : mg_sigmoid(u);
      A *= 1.f - z;
      Bv = (1.f - z) * Bv + z * c;
    }
  }
  s[ch] = A;
  s[p.width + ch] = Bv;
}

// per (request, channel): walk the request's pieces in order, leave every piece's carry-in in its summary slot [0] and the
// request's end state in its slot
__global__ void __launch_bounds__(128) mingru_tile_scan_kernel(MinGruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
  if (ch >= p.width) return;
  const int r0 = p.qo_indptr[b], r1 = p.qo_indptr[b + 1];
  if (r1 - r0 <= 1) return;
  // the request's tiles are consecutive and in order; find the first (tiles are sorted by request)
  int lo = 0, hi = p.n_tiles;
  while (lo < hi) {
    const int mid = (lo + hi) >> 1;
    if (p.tile_req[mid] < b) lo = mid + 1; else hi = mid;
  }
  int last = lo;
  while (last < p.n_tiles && p.tile_req[last] == b) ++last;
  const int ppt = p.tile_rows / MG_ROWS;
  float* st = p.state + static_cast<size_t>(p.slots[b]) * p.width + ch;
  float S = p.pos[r0] == 0 ? 0.f : *st;
  float* s = p.scratch + static_cast<size_t>(lo) * ppt * 2 * p.width + ch;
  const int n = (last - lo) * ppt;
  // (the summaries do not depend on S: sixteen pieces' loads are issued before their chain runs)
  for (int i0 = 0; i0 < n; i0 += 16) {
    float A[16], Bv[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const bool ok = i0 + i < n;
      A[i] = ok ? s[static_cast<size_t>(i0 + i) * 2 * p.width] : 1.f;
      Bv[i] = ok ? s[static_cast<size_t>(i0 + i) * 2 * p.width + p.width] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      if (i0 + i < n) {
        s[static_cast<size_t>(i0 + i) * 2 * p.width] = S;
        S = A[i] * S + Bv[i];
      }
    }
  }
  *st = S;
}

template <typename CT>
__global__ void __launch_bounds__(128) mingru_tile_out_kernel(MinGruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, ppt = p.tile_rows / MG_ROWS;
  const int tile = blockIdx.y / ppt, piece = blockIdx.y - tile * ppt;
  if (ch >= p.width) return;
  const int b = p.tile_req[tile], r0 = p.tile_row0[tile] + piece * MG_ROWS;
  const int n = min(min(r0 + MG_ROWS, p.tile_row0[tile] + p.tile_rows), p.qo_indptr[b + 1]) - r0;
  if (n <= 0) return;
  const float bz = p.bz ? p.bz[ch] : 0.f, bx = p.bx ? p.bx[ch] : 0.f;
  float pz[MG_ROWS], px[MG_ROWS], pg[MG_ROWS];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    const float* row = p.proj + static_cast<size_t>(r0 + min(i, n - 1)) * p.ldp;
    pz[i] = row[p.z_off + ch];
    px[i] = row[p.x_off + ch];
    pg[i] = row[p.g_off + ch];
  }
  float S = p.scratch[static_cast<size_t>(blockIdx.y) * 2 * p.width + ch];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    if (i < n) {
      const float z = mg_sigmoid(pz[i] + bz), u = px[i] + bx;
      const float c = u >= 0.f ? u + 0.5f : mg_sigmoid(u);
      S = (1.f - z) * S + z * c;
      mg_store<CT>(p.out, static_cast<size_t>(r0 + i) * p.width + ch, S * (pg[i] * mg_sigmoid(pg[i])));
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------
// real-gated linear recurrent unit
// ------------------------------------------------------------------------------------------------------------------
struct RgLruParams {
  const float* u;         // [T][ld_u]: the recurrence's input
  int ld_u;
  const void* w;          // [blocks][2 * bs][bs]: the matrix of r, then that of i
  const float* bias;      // [blocks][2 * bs]
  const float* rate;      // [C]: c * softplus(lam)
  const float* y;         // [T][ld_y]: the other branch before its bias and gelu
  int ld_y;
  const float* y_bias;    // [C] or nullptr
  float* state;           // [slots][C]
  void* out;              // [T][ld_out]
  int ld_out;
  float* ab;              // [T][2][C]: a, then the scaled input, of the rows that this kernel does not finish
  const int32_t* qo_indptr;
  const int32_t* row_req;
  const int32_t* pos;
  const int32_t* slots;
  int T, B, C, bs;
  int n_tiles, tile_rows; // piecewise form
  const int32_t* tile_req;
  const int32_t* tile_row0;
  const float* scratch;   // [pieces][2][C]: carry-ins after the scan
};

__device__ __forceinline__ float gelu_tanh_f(float v) {
  return 0.5f * v * (1.f + tanhf(0.79788456080286536f * (v + 0.044715f * v * v * v)));
}

template <typename CT>
__device__ __forceinline__ void rg_out(const RgLruParams& p, int t, int ch, float S) {
  const float y = p.y[static_cast<size_t>(t) * p.ld_y + ch] + (p.y_bias ? p.y_bias[ch] : 0.f);
  mg_store<CT>(p.out, static_cast<size_t>(t) * p.ld_out + ch, S * gelu_tanh_f(y));
}

// gate pre-activations zr, zi of (row, channel) -> the decay and scaled input; a request's only row is finished here
template <typename CT>
__device__ __forceinline__ void rg_finish(const RgLruParams& p, int t, int ch, float zr, float zi) {
  const float la = -p.rate[ch] * mg_sigmoid(zr);
  const float a = expf(la);
  const float v = sqrtf(-expm1f(2.f * la)) * mg_sigmoid(zi) * p.u[static_cast<size_t>(t) * p.ld_u + ch];
  const int b = p.row_req[t];
  if (p.qo_indptr[b + 1] - p.qo_indptr[b] == 1) {
    float* st = p.state + static_cast<size_t>(p.slots[b]) * p.C + ch;
    const float S = fmaf(a, p.pos[t] == 0 ? 0.f : *st, v);
    *st = S;
    rg_out<CT>(p, t, ch, S);
  } else {
    float* o = p.ab + static_cast<size_t>(t) * 2 * p.C + ch;
    o[0] = a;
    o[p.C] = v;
  }
}

// any block size, fp32 FMAs in k order: CTA = 32 rows x 32 channels of one block (both gates)
constexpr int RG_R = 32, RG_CH = 32, RG_K = 32;

template <typename WT, typename CT>
__global__ void __launch_bounds__(256) rglru_gates_kernel(RgLruParams p) {
  __shared__ float Us[RG_R][RG_K + 1];
  __shared__ float Ws[2][RG_CH][RG_K + 1];
  pdl_sync();
  const int per = (p.bs + RG_CH - 1) / RG_CH, blk = blockIdx.x / per, c0 = (blockIdx.x - blk * per) * RG_CH;
  const int t0 = blockIdx.y * RG_R, tid = threadIdx.x, tx = tid & 31, ty = tid >> 5;
  const WT* W = static_cast<const WT*>(p.w) + static_cast<size_t>(blk) * 2 * p.bs * p.bs;
  float acc[2][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) acc[0][i] = acc[1][i] = 0.f;
  for (int k0 = 0; k0 < p.bs; k0 += RG_K) {
    const int k = k0 + tx;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = ty + 8 * i;
      Us[r][tx] = (t0 + r < p.T && k < p.bs) ? p.u[static_cast<size_t>(t0 + r) * p.ld_u + blk * p.bs + k] : 0.f;
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        float w = 0.f;
        if (c0 + r < p.bs && k < p.bs) {
          const WT v = W[static_cast<size_t>(g * p.bs + c0 + r) * p.bs + k];
          if constexpr (sizeof(WT) == 4) w = v;
          else w = __bfloat162float(v);
        }
        Ws[g][r][tx] = w;
      }
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < RG_K; ++kk) {
      const float wr = Ws[0][tx][kk], wi = Ws[1][tx][kk];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float u = Us[ty + 8 * i][kk];
        acc[0][i] = fmaf(u, wr, acc[0][i]);
        acc[1][i] = fmaf(u, wi, acc[1][i]);
      }
    }
    __syncthreads();
  }
  if (c0 + tx >= p.bs) return;
  const float* bias = p.bias + static_cast<size_t>(blk) * 2 * p.bs + c0 + tx;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty + 8 * i;
    if (t < p.T) rg_finish<CT>(p, t, blk * p.bs + c0 + tx, acc[0][i] + bias[0], acc[1][i] + bias[p.bs]);
  }
}

// bf16 matrices, blocks of a multiple of 16 channels: CTA = 64 rows x 32 channels of one block (64 gate columns: r, then i), 4
// warps x 16 rows, mma.sync m16n8k16 with fp32 accumulators over chunks of 64 inputs; u enters as two bf16 terms (its rounding
// and the remainder's).  The next chunk's loads are in flight while a chunk is multiplied.
constexpr int RM_R = 64, RM_CH = 32, RM_K = 64, RM_LD = RM_K + 8;

template <typename CT>
__global__ void __launch_bounds__(128) rglru_gates_mma_kernel(RgLruParams p) {
  __shared__ __align__(16) __nv_bfloat16 Uh[RM_R * RM_LD], Ul[RM_R * RM_LD], Ws[2 * RM_CH * RM_LD];
  const int per = (p.bs + RM_CH - 1) / RM_CH, blk = blockIdx.x / per, c0 = (blockIdx.x - blk * per) * RM_CH;
  const int t0 = blockIdx.y * RM_R, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const __nv_bfloat16* W = static_cast<const __nv_bfloat16*>(p.w) + static_cast<size_t>(blk) * 2 * p.bs * p.bs;
  const int ur = tid >> 4, uc = (tid & 15) * 4, wr = tid >> 3, wc = (tid & 7) * 8;
  float4 un[8];
  uint4 wn[4];
  auto fetch_w = [&](int k0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = wr + 16 * i, ch = c0 + (r & (RM_CH - 1));
      wn[i] = make_uint4(0u, 0u, 0u, 0u);
      if (ch < p.bs && k0 + wc < p.bs)
        wn[i] = *reinterpret_cast<const uint4*>(W + static_cast<size_t>((r >= RM_CH ? p.bs : 0) + ch) * p.bs + k0 + wc);
    }
  };
  auto fetch_u = [&](int k0) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = t0 + ur + 8 * i;
      un[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (t < p.T && k0 + uc < p.bs) un[i] = *reinterpret_cast<const float4*>(p.u + static_cast<size_t>(t) * p.ld_u + blk * p.bs + k0 + uc);
    }
  };
  fetch_w(0);                             // (weights: nothing that precedes this launch writes them)
  pdl_sync();
  fetch_u(0);
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
  const bool rows = t0 + warp * 16 < p.T;
  for (int k0 = 0; k0 < p.bs; k0 += RM_K) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float v[4] = {un[i].x, un[i].y, un[i].z, un[i].w};
      float hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        hi[e] = __bfloat162float(__float2bfloat16_rn(v[e]));
        lo[e] = v[e] - hi[e];
      }
      const int o = (ur + 8 * i) * RM_LD + uc;
      *reinterpret_cast<uint2*>(Uh + o) = make_uint2(pack_bf16(hi[0], hi[1]), pack_bf16(hi[2], hi[3]));
      *reinterpret_cast<uint2*>(Ul + o) = make_uint2(pack_bf16(lo[0], lo[1]), pack_bf16(lo[2], lo[3]));
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) *reinterpret_cast<uint4*>(Ws + (wr + 16 * i) * RM_LD + wc) = wn[i];
    __syncthreads();
    if (k0 + RM_K < p.bs) {
      fetch_w(k0 + RM_K);
      fetch_u(k0 + RM_K);
    }
    if (rows) {
#pragma unroll
      for (int kb = 0; kb < RM_K / 16; ++kb) {
        if (k0 + kb * 16 < p.bs) {
          const int ao = (warp * 16 + (lane & 15)) * RM_LD + kb * 16 + (lane >> 4) * 8;
          uint32_t ah[4], al[4];
          ldmatrix_x4(ah, smem_u32(Uh + ao));
          ldmatrix_x4(al, smem_u32(Ul + ao));
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            uint32_t bf[4];
            ldmatrix_x4(bf, smem_u32(Ws + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * RM_LD + kb * 16 + ((lane >> 3) & 1) * 8));
            mma_bf16_16816(acc[2 * np], ah, bf[0], bf[1]);
            mma_bf16_16816(acc[2 * np], al, bf[0], bf[1]);
            mma_bf16_16816(acc[2 * np + 1], ah, bf[2], bf[3]);
            mma_bf16_16816(acc[2 * np + 1], al, bf[2], bf[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  if (!rows) return;
  // as rg_finish, with all loads of a row's eight channels in flight before the first store
  const int lc = c0 + (lane & 3) * 2, gc = blk * p.bs + lc;
  const float* bias = p.bias + static_cast<size_t>(blk) * 2 * p.bs + lc;
  float rate[4][2], br[4][2], bi[4][2];
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = lc + n * 8 < p.bs;
      rate[n][e] = ok ? p.rate[gc + n * 8 + e] : 0.f;
      br[n][e] = ok ? bias[n * 8 + e] : 0.f;
      bi[n][e] = ok ? bias[p.bs + n * 8 + e] : 0.f;
    }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = t0 + warp * 16 + (lane >> 2) + 8 * half;
    if (t >= p.T) continue;
    const int b = p.row_req[t];
    const bool single = p.qo_indptr[b + 1] - p.qo_indptr[b] == 1, fresh = p.pos[t] == 0;
    float* st = p.state + static_cast<size_t>(p.slots[b]) * p.C + gc;
    const float* yr = p.y + static_cast<size_t>(t) * p.ld_y + gc;
    float2 u[4];
    float S[4][2], y[4][2];
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const bool ok = lc + n * 8 < p.bs;
      u[n] = ok ? *reinterpret_cast<const float2*>(p.u + static_cast<size_t>(t) * p.ld_u + gc + n * 8) : make_float2(0.f, 0.f);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        S[n][e] = ok && single && !fresh ? st[n * 8 + e] : 0.f;
        y[n][e] = ok && single ? yr[n * 8 + e] + (p.y_bias ? p.y_bias[gc + n * 8 + e] : 0.f) : 0.f;
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      if (lc + n * 8 >= p.bs) continue;
      float a[2], v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float la = -rate[n][e] * mg_sigmoid(acc[n][2 * half + e] + br[n][e]);
        a[e] = expf(la);
        v[e] = sqrtf(-expm1f(2.f * la)) * mg_sigmoid(acc[n + 4][2 * half + e] + bi[n][e]) * (e ? u[n].y : u[n].x);
      }
      if (single) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float s = fmaf(a[e], S[n][e], v[e]);
          st[n * 8 + e] = s;
          mg_store<CT>(p.out, static_cast<size_t>(t) * p.ld_out + gc + n * 8 + e, s * gelu_tanh_f(y[n][e]));
        }
      } else {
        float* o = p.ab + static_cast<size_t>(t) * 2 * p.C + gc + n * 8;
        *reinterpret_cast<float2*>(o) = make_float2(a[0], a[1]);
        *reinterpret_cast<float2*>(o + p.C) = make_float2(v[0], v[1]);
      }
    }
  }
}

// requests that bring several rows, in order: one thread per (request, channel)
template <typename CT>
__global__ void __launch_bounds__(128) rglru_walk_kernel(RgLruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
  if (ch >= p.C) return;
  const int r0 = p.qo_indptr[b], r1 = p.qo_indptr[b + 1];
  if (r1 - r0 < 2) return;
  float* st = p.state + static_cast<size_t>(p.slots[b]) * p.C + ch;
  float S = p.pos[r0] == 0 ? 0.f : *st;
  for (int t = r0; t < r1; ++t) {
    const float* ab = p.ab + static_cast<size_t>(t) * 2 * p.C + ch;
    S = fmaf(ab[0], S, ab[p.C]);
    rg_out<CT>(p, t, ch, S);
  }
  *st = S;
}

// the pieces' summaries (product of the decays, end state from zero); vb::mingru_tile_scan_kernel turns them into carry-ins
__global__ void __launch_bounds__(128) rglru_piece_sum_kernel(RgLruParams p, float* __restrict__ scratch) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, ppt = p.tile_rows / MG_ROWS;
  const int tile = blockIdx.y / ppt, piece = blockIdx.y - tile * ppt;
  if (ch >= p.C) return;
  const int r0 = p.tile_row0[tile] + piece * MG_ROWS;
  const int n = min(min(r0 + MG_ROWS, p.tile_row0[tile] + p.tile_rows), p.qo_indptr[p.tile_req[tile] + 1]) - r0;
  float* s = scratch + static_cast<size_t>(blockIdx.y) * 2 * p.C;
  if (n <= 0) { s[ch] = 1.f; s[p.C + ch] = 0.f; return; }
  float a[MG_ROWS], v[MG_ROWS];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    const float* ab = p.ab + static_cast<size_t>(r0 + min(i, n - 1)) * 2 * p.C + ch;
    a[i] = ab[0];
    v[i] = ab[p.C];
  }
  float A = 1.f, S = 0.f;
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i)
    if (i < n) { A *= a[i]; S = fmaf(a[i], S, v[i]); }
  s[ch] = A;
  s[p.C + ch] = S;
}

template <typename CT>
__global__ void __launch_bounds__(128) rglru_piece_out_kernel(RgLruParams p) {
  pdl_sync();
  const int ch = blockIdx.x * 128 + threadIdx.x, ppt = p.tile_rows / MG_ROWS;
  const int tile = blockIdx.y / ppt, piece = blockIdx.y - tile * ppt;
  if (ch >= p.C) return;
  const int r0 = p.tile_row0[tile] + piece * MG_ROWS;
  const int n = min(min(r0 + MG_ROWS, p.tile_row0[tile] + p.tile_rows), p.qo_indptr[p.tile_req[tile] + 1]) - r0;
  if (n <= 0) return;
  float a[MG_ROWS], v[MG_ROWS], y[MG_ROWS];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i) {
    const int t = r0 + min(i, n - 1);
    const float* ab = p.ab + static_cast<size_t>(t) * 2 * p.C + ch;
    a[i] = ab[0];
    v[i] = ab[p.C];
    y[i] = p.y[static_cast<size_t>(t) * p.ld_y + ch];
  }
  const float yb = p.y_bias ? p.y_bias[ch] : 0.f;
  float S = p.scratch[static_cast<size_t>(blockIdx.y) * 2 * p.C + ch];
#pragma unroll
  for (int i = 0; i < MG_ROWS; ++i)
    if (i < n) {
      S = fmaf(a[i], S, v[i]);
      mg_store<CT>(p.out, static_cast<size_t>(r0 + i) * p.ld_out + ch, S * gelu_tanh_f(y[i] + yb));
    }
}

}  // namespace vb

using namespace vb;
using bf16 = __nv_bfloat16;

extern "C" {

int vb_mingru(void* d_out, float* d_state, const float* d_proj, int ldp, int z_off, int x_off, int g_off, const float* d_bz,
              const float* d_bx, const int32_t* d_qo_indptr, const int32_t* d_pos, const int32_t* d_slots, int B, int width,
              int single_rows, int multi_rows, int out_dtype, void* stream) {
  VB_CHECK_ARG(d_out && d_state && d_proj && d_qo_indptr && d_pos && d_slots && width > 0, "vb_mingru: bad arguments");
  if (B <= 0) return 0;
  MinGruParams p{d_proj, ldp, z_off, x_off, g_off, d_bz, d_bx, d_state, d_out, d_qo_indptr, d_pos, d_slots, B, width,
                 single_rows, multi_rows, nullptr, nullptr, 0, 0, nullptr};
  dim3 grid((width + 127) / 128, B);
  if (out_dtype == 1) VB_LAUNCH_PDL(mingru_seq_kernel<float>, grid, 128, 0, stream, p);
  else VB_LAUNCH_PDL(mingru_seq_kernel<bf16>, grid, 128, 0, stream, p);
  return 0;
}

int vb_mingru_tiled(void* d_out, float* d_state, float* d_scratch, const float* d_proj, int ldp, int z_off, int x_off,
                    int g_off, const float* d_bz, const float* d_bx, const int32_t* d_qo_indptr, const int32_t* d_pos,
                    const int32_t* d_slots, const int32_t* d_tile_req, const int32_t* d_tile_row0, int n_tiles, int tile_rows,
                    int B, int width, int out_dtype, void* stream) {
  VB_CHECK_ARG(d_out && d_state && d_scratch && d_proj && d_qo_indptr && d_pos && d_slots && d_tile_req && d_tile_row0 &&
               width > 0 && tile_rows > 0 && tile_rows % MG_ROWS == 0, "vb_mingru_tiled: bad arguments (tile_rows a multiple of %d)",
               MG_ROWS);
  if (B <= 0 || n_tiles <= 0) return 0;
  MinGruParams p{d_proj, ldp, z_off, x_off, g_off, d_bz, d_bx, d_state, d_out, d_qo_indptr, d_pos, d_slots, B, width,
                 0, 1, d_tile_req, d_tile_row0, n_tiles, tile_rows, d_scratch};
  const int cx = (width + 127) / 128, pieces = n_tiles * (tile_rows / MG_ROWS);
  VB_LAUNCH_PDL(mingru_tile_sum_kernel, dim3(cx, pieces), 128, 0, stream, p);
  VB_LAUNCH_PDL(mingru_tile_scan_kernel, dim3(cx, B), 128, 0, stream, p);
  if (out_dtype == 1) VB_LAUNCH_PDL(mingru_tile_out_kernel<float>, dim3(cx, pieces), 128, 0, stream, p);
  else VB_LAUNCH_PDL(mingru_tile_out_kernel<bf16>, dim3(cx, pieces), 128, 0, stream, p);
  return 0;
}

int vb_rglru(void* d_out, int ld_out, float* d_state, float* d_ab, float* d_scratch, const float* d_u, int ld_u, const void* d_w,
             const float* d_bias, const float* d_rate, const float* d_y, int ld_y, const float* d_y_bias,
             const int32_t* d_qo_indptr, const int32_t* d_row_req, const int32_t* d_pos, const int32_t* d_slots,
             const int32_t* d_tile_req, const int32_t* d_tile_row0, int n_tiles, int tile_rows, int T, int B, int width,
             int blocks, int multi_rows, int w_dtype, int out_dtype, void* stream) {
  VB_CHECK_ARG(d_out && d_state && d_u && d_w && d_bias && d_rate && d_y && d_qo_indptr && d_row_req && d_pos && d_slots &&
               (!multi_rows || d_ab), "vb_rglru: null pointer");
  VB_CHECK_ARG(width > 0 && blocks > 0 && width % blocks == 0 && ld_u >= width && ld_y >= width && ld_out >= width,
               "vb_rglru: width %d in %d blocks", width, blocks);
  VB_CHECK_ARG(n_tiles <= 0 || (d_tile_req && d_tile_row0 && d_scratch && tile_rows > 0 && tile_rows % MG_ROWS == 0),
               "vb_rglru: the piecewise form needs tiles of a multiple of %d rows and scratch", MG_ROWS);
  if (T <= 0 || B <= 0) return 0;
  const int bs = width / blocks;
  RgLruParams p{d_u, ld_u, d_w, d_bias, d_rate, d_y, ld_y, d_y_bias, d_state, d_out, ld_out, d_ab, d_qo_indptr, d_row_req, d_pos,
                d_slots, T, B, width, bs, n_tiles, tile_rows, d_tile_req, d_tile_row0, d_scratch};
  const bool f32 = out_dtype == 1;
  const dim3 grid(blocks * ((bs + RG_CH - 1) / RG_CH), (T + RG_R - 1) / RG_R);
  if (w_dtype == 0 && bs % 16 == 0 && ld_u % 4 == 0 && reinterpret_cast<uintptr_t>(d_u) % 16 == 0 && reinterpret_cast<uintptr_t>(d_w) % 16 == 0) {
    const dim3 mgrid(blocks * ((bs + RM_CH - 1) / RM_CH), (T + RM_R - 1) / RM_R);
    if (f32) VB_LAUNCH_PDL(rglru_gates_mma_kernel<float>, mgrid, 128, 0, stream, p);
    else VB_LAUNCH_PDL(rglru_gates_mma_kernel<bf16>, mgrid, 128, 0, stream, p);
  } else if (w_dtype == 1) {
    if (f32) VB_LAUNCH_PDL((rglru_gates_kernel<float, float>), grid, 256, 0, stream, p);
    else VB_LAUNCH_PDL((rglru_gates_kernel<float, bf16>), grid, 256, 0, stream, p);
  } else {
    if (f32) VB_LAUNCH_PDL((rglru_gates_kernel<bf16, float>), grid, 256, 0, stream, p);
    else VB_LAUNCH_PDL((rglru_gates_kernel<bf16, bf16>), grid, 256, 0, stream, p);
  }
  if (!multi_rows) return 0;
  const int cx = (width + 127) / 128;
  if (n_tiles <= 0) {
    if (f32) VB_LAUNCH_PDL(rglru_walk_kernel<float>, dim3(cx, B), 128, 0, stream, p);
    else VB_LAUNCH_PDL(rglru_walk_kernel<bf16>, dim3(cx, B), 128, 0, stream, p);
    return 0;
  }
  const int pieces = n_tiles * (tile_rows / MG_ROWS);
  MinGruParams sp{};
  sp.state = d_state; sp.qo_indptr = d_qo_indptr; sp.pos = d_pos; sp.slots = d_slots; sp.B = B; sp.width = width;
  sp.tile_req = d_tile_req; sp.tile_row0 = d_tile_row0; sp.n_tiles = n_tiles; sp.tile_rows = tile_rows; sp.scratch = d_scratch;
  VB_LAUNCH_PDL(rglru_piece_sum_kernel, dim3(cx, pieces), 128, 0, stream, p, d_scratch);
  VB_LAUNCH_PDL(mingru_tile_scan_kernel, dim3(cx, B), 128, 0, stream, sp);
  if (f32) VB_LAUNCH_PDL(rglru_piece_out_kernel<float>, dim3(cx, pieces), 128, 0, stream, p);
  else VB_LAUNCH_PDL(rglru_piece_out_kernel<bf16>, dim3(cx, pieces), 128, 0, stream, p);
  return 0;
}

int vb_mingru_scratch_floats(int n_tiles, int tile_rows, int width) {
  return n_tiles * (tile_rows / MG_ROWS) * 2 * width;
}

}  // extern "C"
