// State-space duality (Mamba-2: Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through
// Structured State Space Duality"): per head h a state S [N][V] with one decay per token,
//   dt_t = softplus(dt_t + dt_bias_h),  a_t = exp(-exp(A_log_h) dt_t)
//   S_t = a_t S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D_h x_t,   out_t = y_t * silu(z_t)
// B and C [N] are shared by the heads of a group.  x | B | C are columns of rows that a short convolution has left in the
// compute type; dt, the decays, the state and every sum are fp32 (decay exponents are accumulated in double).  The state
// lives in an fp32 slot per live sequence; a request whose first new row has position 0 starts from zero, so slots are
// reused without clearing.
//
//   vb_ssd           requests whose number of new rows lies in a range, row by row over the slot: CTA = (request, head, block
//                    of value dims); one read and one write of the state per row.  Single decoded tokens; any sizes.
//   vb_ssd_tiled     prompt portions, 64-row tiles in parallel: local end states of all tiles, a scan over a request's tiles,
//                    then the rows of every tile:  Y = (C B^T .* exp(L_i - L_j) dt_j, j <= i) X + exp(L_i) C S_before,
//                    L the running sum of the log decays inside the tile.
//   vb_group_rmsnorm rows of channels in equal neighbourhoods, each divided by its own root mean square, times a weight.
#include "../../include/vb_api.h"
#define VB_PDL_FAMILY 1
#include "common.cuh"

namespace vb {

template <typename T> __device__ __forceinline__ float sd_to_f(T v);
template <> __device__ __forceinline__ float sd_to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float sd_to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float sd_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float sd_silu(float z) { return z / (1.f + expf(-z)); }
// two fp32 values as bf16 terms: the rounded values, and (lo) what the rounding left
__device__ __forceinline__ uint32_t sd_split(float a, float b, uint32_t& lo) {
  const __nv_bfloat16 ha = __float2bfloat16_rn(a), hb = __float2bfloat16_rn(b);
  lo = pack_bf16(a - __bfloat162float(ha), b - __bfloat162float(hb));
  return pack_bf16(__bfloat162float(ha), __bfloat162float(hb));
}


struct SsdParams {
  const void* xbc;        // [T][ld]: x [H * V] | B [G * N] | C [G * N]
  int ld;
  const float* dt;        // [T][ld_dt]
  int ld_dt;
  const float* dt_bias;   // [H]
  const float* A_log;     // [H]
  const float* D;         // [H]
  const float* z;         // [T][ld_z]
  int ld_z;
  float* state;           // [slots][H][N][V]
  float* out;             // [T][H * V]
  const int32_t* qo_indptr;
  const int32_t* pos;
  const int32_t* slots;
  int H, V, N, G, dvb;    // dvb: value dims per CTA
  int min_rows, max_rows; // requests with min_rows <= new rows <= max_rows are served
  // tiled form
  const int32_t* tile_req;
  const int32_t* tile_row0;
  float* scratch;         // [tiles][H][N][V]: local end states; fp32 form: then the states before the tiles
  __nv_bfloat16* before;  // tensor-core form: the states before the tiles as [tiles][H][2][N][V], rounded and the remainder
  float* tile_decay;      // [tiles][H]: the tile's whole decay
};

// VEC value dims per thread; threads = (value lane, group of state dims); the state dims are dealt round-robin to the groups
constexpr int SS_THREADS = 256, SS_MAXN = 8;

template <typename XT, int VEC>
__global__ void __launch_bounds__(SS_THREADS) ssd_step_kernel(SsdParams p) {
  extern __shared__ float smf[];
  pdl_sync();
  const int b = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * p.dvb;
  const int r0 = p.qo_indptr[b], n = p.qo_indptr[b + 1] - r0;
  if (n < p.min_rows || n > p.max_rows) return;
  const int N = p.N, V = p.V, g = h / (p.H / p.G), DV = min(p.dvb, V - e0);
  const int lanes = p.dvb / VEC, groups = SS_THREADS / lanes;
  float* bs = smf;              // [N] dt * B
  float* cs = bs + N;           // [N]
  float* red = cs + N;          // [groups][dvb]
  const int tid = threadIdx.x, e = (tid % lanes) * VEC, kg = tid / lanes;
  const bool act = e < DV && kg < groups;
  const XT* xbc = static_cast<const XT*>(p.xbc);
  float* S = p.state + (static_cast<size_t>(p.slots[b]) * p.H + h) * N * V + e0 + e;
  const float A = -expf(p.A_log[h]), dtb = p.dt_bias[h], D = p.D[h];
  for (int r = 0; r < n; ++r) {
    const size_t t = r0 + r;
    const XT* row = xbc + t * p.ld;
    const float dt = sd_softplus(p.dt[t * p.ld_dt + h] + dtb), a = expf(A * dt);
    const bool fresh = p.pos[t] == 0;
    __syncthreads();
    for (int k = tid; k < N; k += SS_THREADS) {
      bs[k] = dt * sd_to_f(row[p.H * V + g * N + k]);
      cs[k] = sd_to_f(row[p.H * V + p.G * N + g * N + k]);
    }
    __syncthreads();
    float y[VEC], x[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      y[j] = 0.f;
      x[j] = (act && e + j < DV) ? sd_to_f(row[h * V + e0 + e + j]) : 0.f;
    }
    if (act) {
      // SS_MAXN rows of the state in flight at a time
      for (int k0 = kg; k0 < N; k0 += groups * SS_MAXN) {
        float s[SS_MAXN][VEC];
#pragma unroll
        for (int i = 0; i < SS_MAXN; ++i) {
          const int k = k0 + i * groups;
          if (k < N && !fresh) {
            if constexpr (VEC == 4) {
              const float4 v = *reinterpret_cast<const float4*>(S + static_cast<size_t>(k) * V);
              s[i][0] = v.x; s[i][1] = v.y; s[i][2] = v.z; s[i][3] = v.w;
            } else {
              s[i][0] = S[static_cast<size_t>(k) * V];
            }
          } else {
#pragma unroll
            for (int j = 0; j < VEC; ++j) s[i][j] = 0.f;
          }
        }
#pragma unroll
        for (int i = 0; i < SS_MAXN; ++i) {
          const int k = k0 + i * groups;
          if (k < N) {
            const float bk = bs[k], ck = cs[k];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
              s[i][j] = fmaf(a, s[i][j], bk * x[j]);
              y[j] = fmaf(s[i][j], ck, y[j]);
            }
            if constexpr (VEC == 4) *reinterpret_cast<float4*>(S + static_cast<size_t>(k) * V) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
            else S[static_cast<size_t>(k) * V] = s[i][0];
          }
        }
      }
    }
    if (kg < groups) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) red[kg * p.dvb + e + j] = y[j];
    }
    __syncthreads();
    for (int v = tid; v < DV; v += SS_THREADS) {
      float o = 0.f;
      for (int q = 0; q < groups; ++q) o += red[q * p.dvb + v];
      o = fmaf(D, sd_to_f(row[h * V + e0 + v]), o);
      p.out[t * p.H * V + h * V + e0 + v] = o * sd_silu(p.z[t * p.ld_z + h * V + e0 + v]);
    }
  }
}

constexpr int SD_ROWS = 64;

// the tile's step sizes and running log decays (warp 0; lane l holds rows l and l + 32)
__device__ __forceinline__ void ssd_tile_decays(const SsdParams& p, int h, int row0, int L, float* dts, double* cum) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const double A = -static_cast<double>(expf(p.A_log[h]));
    double v[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = lane + 32 * u;
      const float dt = r < L ? sd_softplus(p.dt[static_cast<size_t>(row0 + r) * p.ld_dt + h] + p.dt_bias[h]) : 0.f;
      dts[r] = dt;
      v[u] = A * dt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double w = __shfl_up_sync(0xffffffffu, v[u], o);
        if (lane >= o) v[u] += w;
      }
    }
    const double first = __shfl_sync(0xffffffffu, v[0], 31);
    cum[lane] = v[0];
    cum[lane + 32] = first + v[1];
  }
  __syncthreads();
}

// local end state of a tile: U = sum_j exp(L_last - L_j) dt_j B_j x_j^T
template <typename XT>
__global__ void __launch_bounds__(256) ssd_tile_state_kernel(SsdParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float dts[SD_ROWS];
  __shared__ double cum[SD_ROWS];
  pdl_sync();
  const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * p.dvb, g = h / (p.H / p.G);
  const int row0 = p.tile_row0[tile], L = min(SD_ROWS, p.qo_indptr[p.tile_req[tile] + 1] - row0);
  const int N = p.N, V = p.V, DV = min(p.dvb, V - e0), np = N + 1, dvp = p.dvb + 1;
  float* Bs = smf;                    // [64][N + 1]
  float* Xs = Bs + SD_ROWS * np;      // [64][dvb + 1]
  const XT* xbc = static_cast<const XT*>(p.xbc) + static_cast<size_t>(row0) * p.ld;
  const int tid = threadIdx.x;
  ssd_tile_decays(p, h, row0, L, dts, cum);
  const double last = cum[L - 1];
  if (tid == 0 && blockIdx.z == 0) p.tile_decay[static_cast<size_t>(tile) * p.H + h] = static_cast<float>(exp(last));
  for (int i = tid; i < L * N; i += 256) {
    const int r = i / N, k = i - r * N;
    Bs[r * np + k] = sd_to_f(xbc[static_cast<size_t>(r) * p.ld + p.H * V + g * N + k]);
  }
  for (int i = tid; i < L * DV; i += 256) {
    const int r = i / DV, e = i - r * DV;
    Xs[r * dvp + e] = expf(static_cast<float>(last - cum[r])) * dts[r] * sd_to_f(xbc[static_cast<size_t>(r) * p.ld + h * V + e0 + e]);
  }
  __syncthreads();
  float* U = p.scratch + (static_cast<size_t>(tile) * p.H + h) * N * V;
  const int tx = tid & 15, ty = tid >> 4;
  for (int kb = 0; kb < N; kb += 128) {
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
    for (int j = 0; j < L; ++j) {
      float kv[8], vv[4];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int k = kb + ty + 16 * i;
        kv[i] = k < N ? Bs[j * np + k] : 0.f;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int ee = tx + 16 * e;
        vv[e] = ee < DV ? Xs[j * dvp + ee] : 0.f;
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = fmaf(kv[i], vv[e], acc[i][e]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int k = kb + ty + 16 * i;
      if (k >= N) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int ee = tx + 16 * e;
        if (ee < DV) U[static_cast<size_t>(k) * V + e0 + ee] = acc[i][e];
      }
    }
  }
}

// per request: scratch[tile] (or before[tile]) <- the state before the tile, the slot <- the state after the last one
__global__ void __launch_bounds__(256) ssd_tile_scan_kernel(SsdParams p) {
  pdl_sync();
  const int b = blockIdx.x, h = blockIdx.y;
  const int r0 = p.qo_indptr[b], n = p.qo_indptr[b + 1] - r0;
  if (n < 2) return;
  int first = 0;                          // tiles of the requests before this one
  for (int bb = 0; bb < b; ++bb) {
    const int nn = p.qo_indptr[bb + 1] - p.qo_indptr[bb];
    if (nn >= 2) first += (nn + SD_ROWS - 1) / SD_ROWS;
  }
  const int n_tiles = (n + SD_ROWS - 1) / SD_ROWS;
  const bool fresh = p.pos[r0] == 0;
  const size_t per = static_cast<size_t>(p.N) * p.V;
  float* S = p.state + (static_cast<size_t>(p.slots[b]) * p.H + h) * per;
  const float* dec = p.tile_decay + static_cast<size_t>(first) * p.H + h;
  float* sc = p.scratch + (static_cast<size_t>(first) * p.H + h) * per;
  if (per % 4 == 0 && ((reinterpret_cast<uintptr_t>(S) | reinterpret_cast<uintptr_t>(sc)) & 15) == 0) {
    // four neighbouring values per thread in 16-byte pieces (the grid covers them once)
    const size_t i = (static_cast<size_t>(blockIdx.z) * blockDim.x + threadIdx.x) * 4, step = static_cast<size_t>(p.H) * per;
    if (i >= per) return;
    float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(S + i);
    for (int c0 = 0; c0 < n_tiles; c0 += 8) {
      float4 uv[8];
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < n_tiles) uv[j] = *reinterpret_cast<const float4*>(sc + (c0 + j) * step + i);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (c0 + j < n_tiles) {
          if (p.before) {
            __nv_bfloat16* o = p.before + (static_cast<size_t>(first + c0 + j) * p.H + h) * 2 * per + i;
            uint2 hi, lo;
            hi.x = sd_split(s.x, s.y, lo.x);
            hi.y = sd_split(s.z, s.w, lo.y);
            *reinterpret_cast<uint2*>(o) = hi;
            *reinterpret_cast<uint2*>(o + per) = lo;
          } else {
            *reinterpret_cast<float4*>(sc + (c0 + j) * step + i) = s;
          }
          const float d = dec[static_cast<size_t>(c0 + j) * p.H];
          s.x = fmaf(d, s.x, uv[j].x); s.y = fmaf(d, s.y, uv[j].y); s.z = fmaf(d, s.z, uv[j].z); s.w = fmaf(d, s.w, uv[j].w);
        }
      }
    }
    *reinterpret_cast<float4*>(S + i) = s;
    return;
  }
  for (size_t i = blockIdx.z * blockDim.x + threadIdx.x; i < per; i += static_cast<size_t>(gridDim.z) * blockDim.x) {
    float s = fresh ? 0.f : S[i];
    for (int c0 = 0; c0 < n_tiles; c0 += 8) {          // eight independent loads in flight, then the serial update
      float uv[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) uv[j] = c0 + j < n_tiles ? sc[static_cast<size_t>(c0 + j) * p.H * per + i] : 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (c0 + j < n_tiles) {
          sc[static_cast<size_t>(c0 + j) * p.H * per + i] = s;
          s = fmaf(dec[static_cast<size_t>(c0 + j) * p.H], s, uv[j]);
        }
      }
    }
    S[i] = s;
  }
}

template <typename XT>
__global__ void __launch_bounds__(256) ssd_tile_out_kernel(SsdParams p) {
  extern __shared__ __align__(16) float smf[];
  __shared__ float dts[SD_ROWS];
  __shared__ double cum[SD_ROWS];
  pdl_sync();
  constexpr int C = SD_ROWS;
  const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * p.dvb, g = h / (p.H / p.G);
  const int row0 = p.tile_row0[tile], L = min(C, p.qo_indptr[p.tile_req[tile] + 1] - row0);
  const int N = p.N, V = p.V, DV = min(p.dvb, V - e0), np = N + 1, dvp = p.dvb;
  float* Cs = smf;                                // [64][N + 1]
  float* Bs = Cs + C * np;                        // [64][N + 1], then the weights [64][65]
  float* Ms = Bs;
  float* Xs = Bs + C * max(np, C + 1);            // [64][dvb]
  float* Ss = Xs + C * dvp;                       // [N][dvb]
  const XT* xbc = static_cast<const XT*>(p.xbc) + static_cast<size_t>(row0) * p.ld;
  const int tid = threadIdx.x;
  ssd_tile_decays(p, h, row0, L, dts, cum);
  const float* Sb = p.scratch + (static_cast<size_t>(tile) * p.H + h) * N * V;
  for (int i = tid; i < N * DV; i += 256) {
    const int k = i / DV, e = i - k * DV;
    Ss[k * dvp + e] = Sb[static_cast<size_t>(k) * V + e0 + e];
  }
  for (int i = tid; i < C * N; i += 256) {
    const int r = i / N, k = i - r * N;
    float bv = 0.f, cv = 0.f;
    if (r < L) {
      const XT* row = xbc + static_cast<size_t>(r) * p.ld + p.H * V + g * N + k;
      bv = sd_to_f(row[0]);
      cv = sd_to_f(row[p.G * N]);
    }
    Bs[r * np + k] = bv;
    Cs[r * np + k] = cv;
  }
  for (int i = tid; i < C * DV; i += 256) {
    const int r = i / DV, e = i - r * DV;
    Xs[r * dvp + e] = r < L ? sd_to_f(xbc[static_cast<size_t>(r) * p.ld + h * V + e0 + e]) : 0.f;
  }
  __syncthreads();
  // register tiles (16 x 16 threads): thread (ty, tx) owns rows ty + 16 i and columns tx + 16 j
  const int tx = tid & 15, ty = tid >> 4;
  {
    float a[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) a[i][j] = 0.f;
    for (int k = 0; k < N; ++k) {
      float cv[4], bv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) cv[i] = Cs[(ty + 16 * i) * np + k];
#pragma unroll
      for (int j = 0; j < 4; ++j) bv[j] = Bs[(tx + 16 * j) * np + k];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) a[i][j] = fmaf(cv[i], bv[j], a[i][j]);
    }
    __syncthreads();                              // the B tile is consumed: its place takes the weights
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = ty + 16 * i, c = tx + 16 * j;
        Ms[r * (C + 1) + c] = (c <= r && r < L) ? a[i][j] * expf(static_cast<float>(cum[r] - cum[c])) * dts[c] : 0.f;
      }
  }
  __syncthreads();
  float intra[4][4], inter[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) intra[i][e] = inter[i][e] = 0.f;
  const int jmax = min(L, ty + 49);               // the thread's last row is ty + 48: later rows weigh nothing
  for (int j = 0; j < jmax; ++j) {
    float mv[4], xv[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) mv[i] = Ms[(ty + 16 * i) * (C + 1) + j];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ee = tx + 16 * e;
      xv[e] = ee < DV ? Xs[j * dvp + ee] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) intra[i][e] = fmaf(mv[i], xv[e], intra[i][e]);
  }
  for (int k = 0; k < N; ++k) {
    float cv[4], sv[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) cv[i] = Cs[(ty + 16 * i) * np + k];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ee = tx + 16 * e;
      sv[e] = ee < DV ? Ss[k * dvp + ee] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) inter[i][e] = fmaf(cv[i], sv[e], inter[i][e]);
  }
  const float D = p.D[h];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty + 16 * i;
    if (r >= L) continue;
    const float da = expf(static_cast<float>(cum[r]));
    const size_t t = row0 + r;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ee = tx + 16 * e;
      if (ee >= DV) continue;
      const float y = fmaf(D, Xs[r * dvp + ee], fmaf(da, inter[i][e], intra[i][e]));
      p.out[t * p.H * V + h * V + e0 + ee] = y * sd_silu(p.z[t * p.ld_z + h * V + e0 + ee]);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------
// The tiles on the tensor cores (bf16 rows, N and V multiples of 16): CTA = (64-row tile, one or several heads of a group, up
// to 64 value dims), mma.sync m16n8k16 with fp32 accumulators.  B, C and x are bf16 as they stand; an fp32 operand (the
// decayed weights, the weighted x, the state) enters as two bf16 terms, its rounding and the remainder's, so that a product keeps
// 16 bits of its mantissa.
// ------------------------------------------------------------------------------------------------------------------
// rows [0, L) x n columns of bf16 (16-byte pieces) into smem [64][ld], zeros below
__device__ __forceinline__ void sd_stage(__nv_bfloat16* __restrict__ dst, int ld, const __nv_bfloat16* __restrict__ src, int ld_src, int n,
                                         int L) {
  const int v = n / 8;
  for (int i = threadIdx.x; i < SD_ROWS * v; i += 128) {
    const int r = i / v, c = (i - r * v) * 8;
    uint4 q = make_uint4(0u, 0u, 0u, 0u);
    if (r < L) q = *reinterpret_cast<const uint4*>(src + static_cast<size_t>(r) * ld_src + c);
    *reinterpret_cast<uint4*>(dst + r * ld + c) = q;
  }
}

__global__ void __launch_bounds__(128) ssd_tile_state_mma_kernel(SsdParams p, int hb) {
  extern __shared__ __align__(16) uint8_t sd_raw[];
  __shared__ float dts[SD_ROWS];
  __shared__ double cum[SD_ROWS];
  pdl_sync();
  const int tile = blockIdx.x, h0 = blockIdx.y * hb, e0 = blockIdx.z * p.dvb, g = h0 / (p.H / p.G);
  const int row0 = p.tile_row0[tile], L = min(SD_ROWS, p.qo_indptr[p.tile_req[tile] + 1] - row0);
  const int N = p.N, V = p.V, DV = min(p.dvb, V - e0), ldb = N + 8, ldx = p.dvb + 8;
  __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(sd_raw);       // [64][N + 8]
  __nv_bfloat16* Xh = Bs + SD_ROWS * ldb;                             // [64][dvb + 8] the weighted x, and its remainder
  __nv_bfloat16* Xl = Xh + SD_ROWS * ldx;
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(p.xbc) + static_cast<size_t>(row0) * p.ld;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, vb = DV / 8;
  sd_stage(Bs, ldb, xbc + p.H * V + g * N, p.ld, N, L);
  for (int h = h0; h < h0 + hb; ++h) {
    __syncthreads();                      // (the last head's x is consumed)
    ssd_tile_decays(p, h, row0, L, dts, cum);
    const double last = cum[L - 1];
    if (tid == 0 && blockIdx.z == 0) p.tile_decay[static_cast<size_t>(tile) * p.H + h] = static_cast<float>(exp(last));
    for (int i = tid; i < SD_ROWS * vb; i += 128) {
      const int r = i / vb, c = (i - r * vb) * 8;
      uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
      if (r < L) {
        const float w = expf(static_cast<float>(last - cum[r])) * dts[r];
        const uint4 q = *reinterpret_cast<const uint4*>(xbc + static_cast<size_t>(r) * p.ld + h * V + e0 + c);
        hi.x = sd_split(w * bf16_lo(q.x), w * bf16_hi(q.x), lo.x);
        hi.y = sd_split(w * bf16_lo(q.y), w * bf16_hi(q.y), lo.y);
        hi.z = sd_split(w * bf16_lo(q.z), w * bf16_hi(q.z), lo.z);
        hi.w = sd_split(w * bf16_lo(q.w), w * bf16_hi(q.w), lo.w);
      }
      *reinterpret_cast<uint4*>(Xh + r * ldx + c) = hi;
      *reinterpret_cast<uint4*>(Xl + r * ldx + c) = lo;
    }
    __syncthreads();
    float* U = p.scratch + (static_cast<size_t>(tile) * p.H + h) * N * V + e0;
    for (int m0 = warp * 16; m0 < N; m0 += 64) {
      float acc[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
      for (int kb = 0; kb < SD_ROWS / 16; ++kb) {
        uint32_t af[4];                   // B^T: the stored rows are k, transposed on the way into registers
        ldmatrix_x4_trans(af, smem_u32(Bs + (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ldb + m0 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          if (np * 16 < DV) {
            const int off = (kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * ldx + np * 16 + (lane >> 4) * 8;
            uint32_t bh[4], bl[4];
            ldmatrix_x4_trans(bh, smem_u32(Xh + off));
            ldmatrix_x4_trans(bl, smem_u32(Xl + off));
            mma_bf16_16816(acc[2 * np], af, bh[0], bh[1]);
            mma_bf16_16816(acc[2 * np], af, bl[0], bl[1]);
            mma_bf16_16816(acc[2 * np + 1], af, bh[2], bh[3]);
            mma_bf16_16816(acc[2 * np + 1], af, bl[2], bl[3]);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int c = n * 8 + (lane & 3) * 2;
        if (c < DV) {
          float* u = U + static_cast<size_t>(m0 + (lane >> 2)) * V + c;
          *reinterpret_cast<float2*>(u) = make_float2(acc[n][0], acc[n][1]);
          *reinterpret_cast<float2*>(u + static_cast<size_t>(8) * V) = make_float2(acc[n][2], acc[n][3]);
        }
      }
    }
  }
}

// 8 warps: warp w owns the 16 rows of w / 2 and one half of the value dims
__global__ void __launch_bounds__(256) ssd_tile_out_mma_kernel(SsdParams p) {
  extern __shared__ __align__(16) uint8_t sd_raw[];
  __shared__ float dts[SD_ROWS], cumf[SD_ROWS];
  __shared__ double cum[SD_ROWS];
  const int tile = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * p.dvb, g = h / (p.H / p.G);
  const int row0 = p.tile_row0[tile], L = min(SD_ROWS, p.qo_indptr[p.tile_req[tile] + 1] - row0);
  const int N = p.N, V = p.V, DV = min(p.dvb, V - e0), ldb = N + 8, ldx = p.dvb + 8, nkb = N / 16;
  __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(sd_raw);       // [64][N + 8]
  __nv_bfloat16* Bs = Cs + SD_ROWS * ldb;                             // [64][N + 8]
  __nv_bfloat16* Xs = Bs + SD_ROWS * ldb;                             // [64][dvb + 8]
  __nv_bfloat16* Sh = Xs + SD_ROWS * ldx;                             // [N][dvb + 8] the state before the tile, and its remainder
  __nv_bfloat16* Sl = Sh + N * ldx;
  const __nv_bfloat16* xbc = static_cast<const __nv_bfloat16*>(p.xbc) + static_cast<size_t>(row0) * p.ld;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // every copy is in flight before anything is waited for: B and C first (the scores need them), then x and the state
  auto copy = [&](__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, int ld_src, int n, int rows, int valid) {
    const int v = n / 8;
    for (int i = tid; i < rows * v; i += 256) {
      const int r = i / v, c = (i - r * v) * 8;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * ld + c)),
                   "l"(src + static_cast<size_t>(r < valid ? r : 0) * ld_src + c), "r"(r < valid ? 16u : 0u) : "memory");
    }
  };
  pdl_sync();
  copy(Bs, ldb, xbc + p.H * V + g * N, p.ld, N, SD_ROWS, L);
  copy(Cs, ldb, xbc + p.H * V + p.G * N + g * N, p.ld, N, SD_ROWS, L);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const __nv_bfloat16* Sb = p.before + (static_cast<size_t>(tile) * p.H + h) * 2 * N * V + e0;
  copy(Xs, ldx, xbc + h * V + e0, p.ld, DV, SD_ROWS, L);
  copy(Sh, ldx, Sb, V, DV, N, N);
  copy(Sl, ldx, Sb + static_cast<size_t>(N) * V, V, DV, N, N);
  asm volatile("cp.async.commit_group;" ::: "memory");
  ssd_tile_decays(p, h, row0, L, dts, cum);
  if (tid < SD_ROWS) cumf[tid] = static_cast<float>(cum[tid]);
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  // scores of the warp's 16 rows with the rows up to its last one
  const int rb = warp >> 1, v0 = (warp & 1) * 32;
  const __nv_bfloat16* Crow = Cs + (rb * 16 + (lane & 15)) * ldb + (lane >> 4) * 8;
  float sc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
  for (int kb = 0; kb < nkb; ++kb) {
    uint32_t af[4];
    ldmatrix_x4(af, smem_u32(Crow + kb * 16));
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np <= rb) {
        uint32_t bf[4];
        ldmatrix_x4(bf, smem_u32(Bs + (np * 16 + (lane >> 4) * 8 + (lane & 7)) * ldb + kb * 16 + ((lane >> 3) & 1) * 8));
        mma_bf16_16816(sc[2 * np], af, bf[0], bf[1]);
        mma_bf16_16816(sc[2 * np + 1], af, bf[2], bf[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (v0 >= DV) return;
  const int rA = rb * 16 + (lane >> 2), rB = rA + 8;
  float o[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  // what the state before the tile contributes
  for (int kb = 0; kb < nkb; ++kb) {
    uint32_t af[4];
    ldmatrix_x4(af, smem_u32(Crow + kb * 16));
#pragma unroll
    for (int np = 0; np < 2; ++np) {
      if (v0 + np * 16 < DV) {
        const int off = (kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * ldx + v0 + np * 16 + (lane >> 4) * 8;
        uint32_t bh[4], bl[4];
        ldmatrix_x4_trans(bh, smem_u32(Sh + off));
        ldmatrix_x4_trans(bl, smem_u32(Sl + off));
        mma_bf16_16816(o[2 * np], af, bh[0], bh[1]);
        mma_bf16_16816(o[2 * np + 1], af, bh[2], bh[3]);
        mma_bf16_16816(o[2 * np], af, bl[0], bl[1]);
        mma_bf16_16816(o[2 * np + 1], af, bl[2], bl[3]);
      }
    }
  }
  const float cA = cumf[rA], cB = cumf[rB], dA = expf(cA), dB = expf(cB);
#pragma unroll
  for (int n = 0; n < 4; ++n) { o[n][0] *= dA; o[n][1] *= dA; o[n][2] *= dB; o[n][3] *= dB; }
  // the tile's own rows
#pragma unroll
  for (int kb = 0; kb < SD_ROWS / 16; ++kb) {
    if (kb <= rb) {
      float m[2][4];
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = kb * 16 + u * 8 + (lane & 3) * 2 + (e & 1);
          const bool ok = j <= (e < 2 ? rA : rB);
          m[u][e] = ok ? sc[2 * kb + u][e] * expf((e < 2 ? cA : cB) - cumf[j]) * dts[j] : 0.f;
        }
      uint32_t ah[4], al[4];
      ah[0] = sd_split(m[0][0], m[0][1], al[0]);
      ah[1] = sd_split(m[0][2], m[0][3], al[1]);
      ah[2] = sd_split(m[1][0], m[1][1], al[2]);
      ah[3] = sd_split(m[1][2], m[1][3], al[3]);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        if (v0 + np * 16 < DV) {
          uint32_t xf[4];
          ldmatrix_x4_trans(xf, smem_u32(Xs + (kb * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * ldx + v0 + np * 16 + (lane >> 4) * 8));
          mma_bf16_16816(o[2 * np], ah, xf[0], xf[1]);
          mma_bf16_16816(o[2 * np + 1], ah, xf[2], xf[3]);
          mma_bf16_16816(o[2 * np], al, xf[0], xf[1]);
          mma_bf16_16816(o[2 * np + 1], al, xf[2], xf[3]);
        }
      }
    }
  }
  const float D = p.D[h];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = half ? rB : rA;
    if (r >= L) continue;
    const size_t t = row0 + r;
    const float* z = p.z + t * p.ld_z + h * V + e0;
    float* out = p.out + t * p.H * V + h * V + e0;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int c = v0 + n * 8 + (lane & 3) * 2;
      if (c < DV) {
        const uint32_t x = *reinterpret_cast<const uint32_t*>(Xs + r * ldx + c);
        const float y0 = fmaf(D, bf16_lo(x), o[n][2 * half]), y1 = fmaf(D, bf16_hi(x), o[n][2 * half + 1]);
        *reinterpret_cast<float2*>(out + c) = make_float2(y0 * sd_silu(z[c]), y1 * sd_silu(z[c + 1]));
      }
    }
  }
}

static size_t ssd_mma_smem1(int N, int dvb) { return (static_cast<size_t>(SD_ROWS) * (N + 8) + 2ull * SD_ROWS * (dvb + 8)) * 2; }
static size_t ssd_mma_smem3(int N, int dvb) {
  return (2ull * SD_ROWS * (N + 8) + static_cast<size_t>(SD_ROWS) * (dvb + 8) + 2ull * N * (dvb + 8)) * 2;
}

// one CTA per (row, neighbourhood of n channels)
template <typename OT>
__global__ void __launch_bounds__(256) group_rmsnorm_kernel(OT* __restrict__ out, const float* __restrict__ x,
                                                            const float* __restrict__ w, int C, int n, float eps) {
  __shared__ float red[8];
  pdl_sync();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c0 = blockIdx.y * n;
  const float* row = x + static_cast<size_t>(blockIdx.x) * C + c0;
  float q = 0.f;
  for (int i = threadIdx.x; i < n; i += 256) q = fmaf(row[i], row[i], q);
  q = warp_sum(q);
  if (lane == 0) red[warp] = q;
  __syncthreads();
  q = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) q += red[i];
  const float rs = 1.f / sqrtf(q / n + eps);
  OT* o = out + static_cast<size_t>(blockIdx.x) * C + c0;
  for (int i = threadIdx.x; i < n; i += 256) {
    const float v = row[i] * rs * w[c0 + i];
    if constexpr (sizeof(OT) == 4) o[i] = v;
    else o[i] = __float2bfloat16_rn(v);
  }
}

// one warp per (row, neighbourhood) in 16-byte pieces: n a multiple of 4, at most 1024
template <typename OT>
__global__ void __launch_bounds__(256) group_rmsnorm_warp_kernel(OT* __restrict__ out, const float* __restrict__ x,
                                                                 const float* __restrict__ w, int groups, int n, long long rows,
                                                                 float eps) {
  pdl_sync();
  const long long i = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (i >= rows) return;
  const int lane = threadIdx.x & 31, n4 = n >> 2;
  const float4* src = reinterpret_cast<const float4*>(x + i * n);
  const float4* wt = reinterpret_cast<const float4*>(w + (i % groups) * n);
  float4 v[8];
  float q = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (lane + 32 * j < n4) v[j] = src[lane + 32 * j];
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (lane + 32 * j < n4) {
      q = fmaf(v[j].x, v[j].x, q); q = fmaf(v[j].y, v[j].y, q); q = fmaf(v[j].z, v[j].z, q); q = fmaf(v[j].w, v[j].w, q);
    }
  const float rs = 1.f / sqrtf(warp_sum(q) / n + eps);
  OT* o = out + i * n;
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (lane + 32 * j < n4) {
      const int c = lane + 32 * j;
      const float4 ww = wt[c];
      const float a = v[j].x * rs * ww.x, b = v[j].y * rs * ww.y, d = v[j].z * rs * ww.z, e = v[j].w * rs * ww.w;
      if constexpr (sizeof(OT) == 4) reinterpret_cast<float4*>(o)[c] = make_float4(a, b, d, e);
      else reinterpret_cast<uint2*>(o)[c] = make_uint2(pack_bf16(a, b), pack_bf16(d, e));
    }
}

static int ssd_dvb(int V) {
  int d = 64;
  while (d > 4 && d / 2 >= V) d /= 2;            // the smallest power of two >= V between 4 and 64
  return d;
}
static size_t ssd_out_smem(int N, int dvb) {
  return (static_cast<size_t>(SD_ROWS) * (N + 1) + static_cast<size_t>(SD_ROWS) * ((N > SD_ROWS ? N : SD_ROWS) + 1) +
          static_cast<size_t>(SD_ROWS) * dvb + static_cast<size_t>(N) * dvb) * sizeof(float);
}

}  // namespace vb

using namespace vb;
using bf16 = __nv_bfloat16;

extern "C" {

int vb_ssd(float* d_out, float* d_state, const void* d_xbc, int ld, const float* d_dt, int ld_dt, const float* d_dt_bias,
           const float* d_A_log, const float* d_D, const float* d_z, int ld_z, const int32_t* d_qo_indptr, const int32_t* d_pos,
           const int32_t* d_slots, int B, int H, int V, int N, int G, int single_rows, int multi_rows, int x_dtype,
           void* stream) {
  VB_CHECK_ARG(d_out && d_state && d_xbc && d_dt && d_dt_bias && d_A_log && d_D && d_z && d_qo_indptr && d_pos && d_slots,
               "vb_ssd: null pointer");
  VB_CHECK_ARG(H > 0 && V > 0 && N > 0 && G > 0 && H % G == 0 && ld >= H * V + 2 * G * N, "vb_ssd: bad sizes H=%d V=%d N=%d G=%d", H, V, N, G);
  if (B <= 0 || (!single_rows && !multi_rows)) return 0;
  SsdParams p{};
  p.xbc = d_xbc; p.ld = ld; p.dt = d_dt; p.ld_dt = ld_dt; p.dt_bias = d_dt_bias; p.A_log = d_A_log; p.D = d_D; p.z = d_z; p.ld_z = ld_z;
  p.state = d_state; p.out = d_out; p.qo_indptr = d_qo_indptr; p.pos = d_pos; p.slots = d_slots;
  p.H = H; p.V = V; p.N = N; p.G = G; p.dvb = ssd_dvb(V);
  p.min_rows = single_rows ? 1 : 2;
  p.max_rows = multi_rows ? 1 << 30 : 1;
  const bool vec = V % 4 == 0 && reinterpret_cast<uintptr_t>(d_state) % 16 == 0;
  const int groups = SS_THREADS / (p.dvb / (vec ? 4 : 1));
  const size_t smem = (2 * static_cast<size_t>(N) + static_cast<size_t>(groups) * p.dvb) * sizeof(float);
  VB_CHECK_ARG(smem <= 48 * 1024, "vb_ssd: %d states per head", N);
  const dim3 grid(B, H, (V + p.dvb - 1) / p.dvb);
  if (x_dtype == 1) {
    if (vec) VB_LAUNCH_PDL((ssd_step_kernel<float, 4>), grid, SS_THREADS, smem, stream, p);
    else VB_LAUNCH_PDL((ssd_step_kernel<float, 1>), grid, SS_THREADS, smem, stream, p);
  } else {
    if (vec) VB_LAUNCH_PDL((ssd_step_kernel<bf16, 4>), grid, SS_THREADS, smem, stream, p);
    else VB_LAUNCH_PDL((ssd_step_kernel<bf16, 1>), grid, SS_THREADS, smem, stream, p);
  }
  return 0;
}

/* rows per tile of the tiled form, or 0 when these sizes do not fit its shared memory */
int vb_ssd_tile_rows(int V, int N) {
  return ssd_out_smem(N, ssd_dvb(V)) <= static_cast<size_t>(VB_MAX_DYN_SMEM) - 2048 ? SD_ROWS : 0;
}

long long vb_ssd_scratch_floats(int n_tiles, int H, int V, int N) {
  return static_cast<long long>(n_tiles) * H * (2ll * N * V + 1);
}

int vb_ssd_tiled(float* d_out, float* d_state, float* d_scratch, const void* d_xbc, int ld, const float* d_dt, int ld_dt,
                 const float* d_dt_bias, const float* d_A_log, const float* d_D, const float* d_z, int ld_z,
                 const int32_t* d_qo_indptr, const int32_t* d_pos, const int32_t* d_slots, const int32_t* d_tile_req,
                 const int32_t* d_tile_row0, int n_tiles, int B, int H, int V, int N, int G, int x_dtype, void* stream) {
  VB_CHECK_ARG(d_out && d_state && d_scratch && d_xbc && d_dt && d_dt_bias && d_A_log && d_D && d_z && d_qo_indptr && d_pos && d_slots &&
               d_tile_req && d_tile_row0, "vb_ssd_tiled: null pointer");
  VB_CHECK_ARG(H > 0 && V > 0 && N > 0 && G > 0 && H % G == 0 && ld >= H * V + 2 * G * N && vb_ssd_tile_rows(V, N) > 0,
               "vb_ssd_tiled: bad sizes H=%d V=%d N=%d G=%d", H, V, N, G);
  if (B <= 0 || n_tiles <= 0) return 0;
  SsdParams p{};
  p.xbc = d_xbc; p.ld = ld; p.dt = d_dt; p.ld_dt = ld_dt; p.dt_bias = d_dt_bias; p.A_log = d_A_log; p.D = d_D; p.z = d_z; p.ld_z = ld_z;
  p.state = d_state; p.out = d_out; p.qo_indptr = d_qo_indptr; p.pos = d_pos; p.slots = d_slots;
  p.H = H; p.V = V; p.N = N; p.G = G; p.dvb = ssd_dvb(V); p.min_rows = 2; p.max_rows = 1 << 30;
  p.tile_req = d_tile_req; p.tile_row0 = d_tile_row0; p.scratch = d_scratch;
  p.tile_decay = d_scratch + 2 * static_cast<size_t>(n_tiles) * H * N * V;
  const int zb = (V + p.dvb - 1) / p.dvb;
  const size_t per = static_cast<size_t>(N) * V;
  const size_t smem1 = static_cast<size_t>(SD_ROWS) * (N + 1 + p.dvb + 1) * sizeof(float), smem3 = ssd_out_smem(N, p.dvb);
  const dim3 grid(n_tiles, H, zb), scan_grid(B, H, static_cast<unsigned>((per + 1023) / 1024));
  if (x_dtype == 1) {
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_state_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_out_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_LAUNCH_PDL(ssd_tile_state_kernel<float>, grid, 256, smem1, stream, p);
    VB_LAUNCH_PDL(ssd_tile_scan_kernel, scan_grid, 256, 0, stream, p);
    VB_LAUNCH_PDL(ssd_tile_out_kernel<float>, grid, 256, smem3, stream, p);
  } else if (N % 16 == 0 && V % 16 == 0 && ld % 8 == 0 && ssd_mma_smem3(N, p.dvb) <= static_cast<size_t>(VB_MAX_DYN_SMEM) - 2048 &&
             ((reinterpret_cast<uintptr_t>(d_xbc) | reinterpret_cast<uintptr_t>(d_scratch) | reinterpret_cast<uintptr_t>(d_state)) & 15) == 0 &&
             reinterpret_cast<uintptr_t>(d_out) % 8 == 0) {
    // several heads of a group per CTA where that leaves two CTAs per SM
    int hb = 1;
    while (hb < 4 && (H / G) % (2 * hb) == 0 && n_tiles * (H / (2 * hb)) * zb >= 2 * 148) hb *= 2;
    p.before = reinterpret_cast<bf16*>(d_scratch + static_cast<size_t>(n_tiles) * H * N * V);
    const dim3 mgrid(n_tiles, H / hb, zb);
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_state_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_out_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_LAUNCH_PDL(ssd_tile_state_mma_kernel, mgrid, 128, ssd_mma_smem1(N, p.dvb), stream, p, hb);
    VB_LAUNCH_PDL(ssd_tile_scan_kernel, scan_grid, 256, 0, stream, p);
    VB_LAUNCH_PDL(ssd_tile_out_mma_kernel, grid, 256, ssd_mma_smem3(N, p.dvb), stream, p);
  } else {
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_state_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_CHECK_CUDA(cudaFuncSetAttribute(ssd_tile_out_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, VB_MAX_DYN_SMEM - 2048));
    VB_LAUNCH_PDL(ssd_tile_state_kernel<bf16>, grid, 256, smem1, stream, p);
    VB_LAUNCH_PDL(ssd_tile_scan_kernel, scan_grid, 256, 0, stream, p);
    VB_LAUNCH_PDL(ssd_tile_out_kernel<bf16>, grid, 256, smem3, stream, p);
  }
  return 0;
}

int vb_group_rmsnorm(void* d_out, const float* d_x, const float* d_w, int T, int C, int groups, float eps, int out_dtype,
                     void* stream) {
  VB_CHECK_ARG(d_out && d_x && d_w && C > 0 && groups > 0 && C % groups == 0, "vb_group_rmsnorm: %d channels in %d groups", C, groups);
  if (T <= 0) return 0;
  const dim3 grid(T, groups);
  const int n = C / groups;
  if (n % 4 == 0 && n <= 1024 && ((reinterpret_cast<uintptr_t>(d_x) | reinterpret_cast<uintptr_t>(d_w) | reinterpret_cast<uintptr_t>(d_out)) & 15) == 0) {
    const long long rows = static_cast<long long>(T) * groups;
    const unsigned blocks = static_cast<unsigned>((rows + 7) / 8);
    if (out_dtype == 1) VB_LAUNCH_PDL(group_rmsnorm_warp_kernel<float>, blocks, 256, 0, stream, static_cast<float*>(d_out), d_x, d_w, groups, n, rows, eps);
    else VB_LAUNCH_PDL(group_rmsnorm_warp_kernel<bf16>, blocks, 256, 0, stream, static_cast<bf16*>(d_out), d_x, d_w, groups, n, rows, eps);
    return 0;
  }
  if (out_dtype == 1) VB_LAUNCH_PDL(group_rmsnorm_kernel<float>, grid, 256, 0, stream, static_cast<float*>(d_out), d_x, d_w, C, C / groups, eps);
  else VB_LAUNCH_PDL(group_rmsnorm_kernel<bf16>, grid, 256, 0, stream, static_cast<bf16*>(d_out), d_x, d_w, C, C / groups, eps);
  return 0;
}

}  // extern "C"
