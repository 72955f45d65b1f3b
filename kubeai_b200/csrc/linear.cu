// Shape-agnostic linear layer: Y = act(X W^T + bias) for any T, N, K, in bf16 or fp32 storage with fp32 accumulation.
// Three uses share one kernel family (mixers.h LinearArgs): a plain projection, one projection per head inside wider
// rows (batch index = head), and expert-grouped rows (64-row tiles that each name their weight matrix).  It is the
// projection path of every shape the tcgen05 GEMMs (gemm2_tcgen05.cu: bf16, K % 8 == 0, bf16 output) do not take:
// fp32 models, fp32 outputs (router logits, decay pre-activations, latent queries), odd sizes, gathers.
//
// Kernels: a 64 x 64 x 32 shared-memory tile kernel (fp32 weights: FMA, k ascending; bf16 weights: mma.sync tensor-core
// products; either way one output element is accumulated in an order that does not depend on what else is in the batch), and
// two kernels for the few rows of a decode step: up to 16 rows of a bf16 matrix whose rows are whole 16-byte pieces go through
// mma.sync with the weights as the 16-row operand (every weight byte is loaded once, straight into fragments), anything else of
// up to 8 rows through one warp per output row.  Many rows against up to 64 columns take the fragment kernel with the operands
// exchanged.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdlib.h>

#include <algorithm>

#include "activations.cuh"
#include "mixers.h"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;
constexpr int BM = 64, BN = 64, BK = 32;

__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ float ld1(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void ld8(const float* p, float* o) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
}
__device__ __forceinline__ void ld8(const bf16* p, float* o) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    o[2 * i] = __uint_as_float(u[i] << 16);
    o[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
  }
}
// bias and activation of one output element (TY: the type it is rounded to)
template <typename TY>
__device__ __forceinline__ float finish(const LinearArgs& a, float v, int n) {
  if (a.bias) v += a.bias[n];
  if (a.act == LIN_RELU2) { v = fmaxf(v, 0.f); v = v * v; }
  else if (a.act == LIN_XIELU) v = sizeof(TY) == 2 ? xielu_fast(v, a.a_pos, a.a_neg) : xielu(v, a.a_pos, a.a_neg);
  return v;
}

template <typename TX, typename TW, typename TY>
__global__ void __launch_bounds__(256) linear_tile_kernel(LinearArgs a) {
  __shared__ float Xs[BM][BK + 1];
  __shared__ float Ws[BN][BK + 1];
  const int tid = threadIdx.x, lane = tid & 31, wrp = tid >> 5;
  const int row0 = blockIdx.y * BM, col0 = blockIdx.x * BN;
  const long long b = blockIdx.z;
  const TX* X = static_cast<const TX*>(a.X) + b * a.xbs;
  const TW* W = static_cast<const TW*>(a.W) + b * a.wbs;
  TY* Y = static_cast<TY*>(a.Y) + b * a.ybs;
  if (a.tile_group) {
    const int g = a.tile_group[blockIdx.y];
    if (g < 0) return;
    W += static_cast<long long>(g) * a.wbs;
  }
  // the 8 rows of X and of W this thread stages per k-tile (row = warp + 8 i, column = lane)
  long long xoff[8], woff[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int r = wrp + 8 * i;
    int t = row0 + r;
    if (t >= a.T) t = -1;
    else if (a.x_rows) t = a.x_rows[t];
    xoff[i] = t < 0 ? -1 : static_cast<long long>(t) * a.ldx;
    const int n = col0 + r;
    woff[i] = n < a.N ? static_cast<long long>(n) * a.ldw : -1;
  }
  const int ty = tid >> 4, tx = tid & 15;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < a.K; k0 += BK) {
    const int k = k0 + lane;
    const bool kin = k < a.K;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int r = wrp + 8 * i;
      Xs[r][lane] = (kin && xoff[i] >= 0) ? ld1(X + xoff[i] + k) : 0.f;
      Ws[r][lane] = (kin && woff[i] >= 0) ? ld1(W + woff[i] + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; ++kk) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { xv[i] = Xs[ty * 4 + i][kk]; wv[i] = Ws[tx * 4 + i][kk]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = row0 + ty * 4 + i;
    if (t >= a.T) continue;
    if (a.x_rows && a.x_rows[t] < 0) continue;
    const float rs = a.row_scale ? a.row_scale[t] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = col0 + tx * 4 + j;
      if (n < a.N) st1(Y + static_cast<long long>(t) * a.ldy + n, finish<TY>(a, a.row_scale ? acc[i][j] * rs : acc[i][j], n));
    }
  }
}

// bf16 weights: the same 64 x 64 x 32 tile with the products on the tensor cores (mma.sync m16n8k16, fp32 accumulators).
// X is staged as bf16 (an fp32 X is rounded here); 8 warps = 4 row blocks x 2 column halves, a warp owns 16 rows x 32 columns.
__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ bf16 to_bf16(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ bf16 to_bf16(bf16 v) { return v; }

// VEC: every row start and K are multiples of 8 elements and 16-byte aligned, so a thread stages one 8-element piece of X
// and one of W per k-tile with 16-byte loads (thread -> row tid / 4, columns 8 (tid % 4) ...).
template <typename TX, typename TY, bool VEC>
__global__ void __launch_bounds__(256) linear_tile_mma_kernel(LinearArgs a) {
  constexpr int LD = BK + 8;   // 80-byte rows: the 8 rows of a fragment fall into distinct banks
  __shared__ __align__(16) bf16 Xs[BM][LD];
  __shared__ __align__(16) bf16 Ws[BN][LD];
  const int tid = threadIdx.x, lane = tid & 31, wrp = tid >> 5;
  const int row0 = blockIdx.y * BM, col0 = blockIdx.x * BN;
  const long long b = blockIdx.z;
  const TX* X = static_cast<const TX*>(a.X) + b * a.xbs;
  const bf16* W = static_cast<const bf16*>(a.W) + b * a.wbs;
  TY* Y = static_cast<TY*>(a.Y) + b * a.ybs;
  if (a.tile_group) {
    const int g = a.tile_group[blockIdx.y];
    if (g < 0) return;
    W += static_cast<long long>(g) * a.wbs;
  }
  long long xoff[8], woff[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int r = wrp + 8 * i;
    int t = row0 + r;
    if (t >= a.T) t = -1;
    else if (a.x_rows) t = a.x_rows[t];
    xoff[i] = t < 0 ? -1 : static_cast<long long>(t) * a.ldx;
    const int n = col0 + r;
    woff[i] = n < a.N ? static_cast<long long>(n) * a.ldw : -1;
  }
  const int wm = wrp & 3, wn = wrp >> 2, g = lane >> 2, t4 = lane & 3;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const bf16 zero = __float2bfloat16_rn(0.f);
  // vector staging: this thread's row and column piece
  const int vr = tid >> 2, vc = (tid & 3) * 8;
  long long vx = -1, vw = -1;
  if (VEC) {
    int t = row0 + vr;
    if (t >= a.T) t = -1;
    else if (a.x_rows) t = a.x_rows[t];
    vx = t < 0 ? -1 : static_cast<long long>(t) * a.ldx;
    vw = col0 + vr < a.N ? static_cast<long long>(col0 + vr) * a.ldw : -1;
  }
  for (int k0 = 0; k0 < a.K; k0 += BK) {
    if (VEC) {
      const bool kin = k0 + vc < a.K;   // K is a multiple of 8: a piece is inside or outside as a whole
      uint4 xv = make_uint4(0, 0, 0, 0), wv = make_uint4(0, 0, 0, 0);
      if (kin && vw >= 0) wv = *reinterpret_cast<const uint4*>(W + vw + k0 + vc);
      if (kin && vx >= 0) {
        if constexpr (sizeof(TX) == 2) {
          xv = *reinterpret_cast<const uint4*>(X + vx + k0 + vc);
        } else {
          const float4 f0 = *reinterpret_cast<const float4*>(X + vx + k0 + vc), f1 = *reinterpret_cast<const float4*>(X + vx + k0 + vc + 4);
          __nv_bfloat162 p0 = __floats2bfloat162_rn(f0.x, f0.y), p1 = __floats2bfloat162_rn(f0.z, f0.w);
          __nv_bfloat162 p2 = __floats2bfloat162_rn(f1.x, f1.y), p3 = __floats2bfloat162_rn(f1.z, f1.w);
          xv = make_uint4(*reinterpret_cast<uint32_t*>(&p0), *reinterpret_cast<uint32_t*>(&p1), *reinterpret_cast<uint32_t*>(&p2), *reinterpret_cast<uint32_t*>(&p3));
        }
      }
      *reinterpret_cast<uint4*>(&Xs[vr][vc]) = xv;
      *reinterpret_cast<uint4*>(&Ws[vr][vc]) = wv;
    } else {
      const int k = k0 + lane;
      const bool kin = k < a.K;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = wrp + 8 * i;
        Xs[r][lane] = (kin && xoff[i] >= 0) ? to_bf16(X[xoff[i] + k]) : zero;
        Ws[r][lane] = (kin && woff[i] >= 0) ? W[woff[i] + k] : zero;
      }
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < BK; ks += 16) {
      uint32_t af[4];
      af[0] = *reinterpret_cast<const uint32_t*>(&Xs[16 * wm + g][ks + 2 * t4]);
      af[1] = *reinterpret_cast<const uint32_t*>(&Xs[16 * wm + g + 8][ks + 2 * t4]);
      af[2] = *reinterpret_cast<const uint32_t*>(&Xs[16 * wm + g][ks + 2 * t4 + 8]);
      af[3] = *reinterpret_cast<const uint32_t*>(&Xs[16 * wm + g + 8][ks + 2 * t4 + 8]);
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) {
        const int n = 32 * wn + 8 * nb + g;
        const uint32_t b0 = *reinterpret_cast<const uint32_t*>(&Ws[n][ks + 2 * t4]);
        const uint32_t b1 = *reinterpret_cast<const uint32_t*>(&Ws[n][ks + 2 * t4 + 8]);
        mma_16816(acc[nb], af, b0, b1);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = row0 + 16 * wm + g + 8 * half;
    if (t >= a.T) continue;
    if (a.x_rows && a.x_rows[t] < 0) continue;
    const float rs = a.row_scale ? a.row_scale[t] : 1.f;
#pragma unroll
    for (int nb = 0; nb < 4; ++nb)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int n = col0 + 32 * wn + 8 * nb + 2 * t4 + j;
        if (n < a.N) st1(Y + static_cast<long long>(t) * a.ldy + n, finish<TY>(a, a.row_scale ? acc[nb][2 * half + j] * rs : acc[nb][2 * half + j], n));
      }
  }
}

// T <= 8 rows: one warp per output column n streams W[n, :] once and keeps the T accumulators in registers.
template <typename TX, typename TW, typename TY, int VEC>
__global__ void __launch_bounds__(256) linear_rows_kernel(LinearArgs a) {
  const int lane = threadIdx.x & 31, wrp = threadIdx.x >> 5;
  const int n = blockIdx.x * 8 + wrp;
  if (n >= a.N) return;
  const long long b = blockIdx.z;
  const TX* X = static_cast<const TX*>(a.X) + b * a.xbs;
  const TW* w = static_cast<const TW*>(a.W) + b * a.wbs + static_cast<long long>(n) * a.ldw;
  TY* Y = static_cast<TY*>(a.Y) + b * a.ybs;
  float acc[8];
#pragma unroll
  for (int t = 0; t < 8; ++t) acc[t] = 0.f;
  for (int k = lane * VEC; k < a.K; k += 32 * VEC) {
    float wv[VEC];
    if constexpr (VEC == 8) ld8(w + k, wv); else wv[0] = ld1(w + k);
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      if (t < a.T) {
        float xv[VEC];
        const TX* xp = X + static_cast<long long>(t) * a.ldx + k;
        if constexpr (VEC == 8) ld8(xp, xv); else xv[0] = ld1(xp);
#pragma unroll
        for (int v = 0; v < VEC; ++v) acc[t] = fmaf(xv[v], wv[v], acc[t]);
      }
    }
  }
#pragma unroll
  for (int t = 0; t < 8; ++t) {
    if (t < a.T) {
      float v = acc[t];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane == 0) st1(Y + static_cast<long long>(t) * a.ldy + n, finish<TY>(a, a.row_scale ? v * a.row_scale[t] : v, n));
    }
  }
}

// At most 8 * NB rows of X against a bf16 matrix: mma.sync m16n8k16 with 16 weight rows as the first operand and 8 tokens as
// the second.  A lane loads 16 contiguous bytes (8 k) of its two weight rows and of its token's row; the k index inside a
// 32-wide step is permuted the same way on both sides (lane piece t4 holds k 8 t4 .. 8 t4 + 7, its first half feeds the first
// mma, its second half the second), so no fragment goes through shared memory.  The 8 warps of a CTA are KS slices of K times
// 8 / KS groups of 16 weight rows; the slices' sums meet in shared memory and are added in a fixed order.  An fp32 X is split
// into two bf16 terms, x = hi + lo up to 2^-16 of x.  The order of the sums depends on K alone.
__device__ __forceinline__ uint4 ldx8(const bf16* p, uint4*) { return *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ uint4 ldx8(const float* p, uint4* lo) {
  float v[8];
  ld8(p, v);
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    const __nv_bfloat162 r = __floats2bfloat162_rn(v[2 * i] - __low2float(b), v[2 * i + 1] - __high2float(b));
    h[i] = *reinterpret_cast<const uint32_t*>(&b);
    l[i] = *reinterpret_cast<const uint32_t*>(&r);
  }
  *lo = make_uint4(l[0], l[1], l[2], l[3]);
  return make_uint4(h[0], h[1], h[2], h[3]);
}

// THIN: the same with the operands' parts exchanged, for many rows of X against few rows of W (router logits, scalar gates):
// X streams as the 16-row operand, W's rows 16 y .. 16 y + 15 of grid row y are the "tokens".  One output element is summed in
// the same order as above.
template <typename TX, typename TY, int NB, int U, bool THIN>
__global__ void __launch_bounds__(256) linear_rows_mma_kernel(LinearArgs a, int KS) {
  constexpr bool SPLIT = sizeof(TX) == 4;
  __shared__ float part[8][16][8 * NB + 1];   // [warp][weight row][token]
  const int lane = threadIdx.x & 31, wrp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int ks = wrp % KS, RG = 8 / KS;
  const int n0 = (blockIdx.x * RG + wrp / KS) * 16;
  const long long b = blockIdx.z;
  const int col0 = THIN ? blockIdx.y * 8 * NB : 0;
  // the 16-row operand and its rows, the 8-row operand and its rows
  const bf16* W = THIN ? static_cast<const bf16*>(a.X) : static_cast<const bf16*>(a.W) + b * a.wbs;
  const TX* X = THIN ? static_cast<const TX*>(a.W) + static_cast<long long>(col0) * a.ldw : static_cast<const TX*>(a.X) + b * a.xbs;
  const int ldw = THIN ? a.ldx : a.ldw, ldx = THIN ? a.ldw : a.ldx, rows = THIN ? a.T : a.N, toks = THIN ? min(8 * NB, a.N - col0) : a.T;
  TY* Y = static_cast<TY*>(a.Y) + b * a.ybs;
  const bool r0 = n0 + g < rows, r1 = n0 + g + 8 < rows;
  const bf16* w0 = W + static_cast<long long>(n0 + g) * ldw;
  const bf16* w1 = w0 + 8ll * ldw;
  const TX* xr[NB];
  bool xin[NB];
#pragma unroll
  for (int i = 0; i < NB; ++i) { xin[i] = g + 8 * i < toks; xr[i] = X + static_cast<long long>(g + 8 * i) * ldx; }
  float acc[NB][4];
#pragma unroll
  for (int i = 0; i < NB; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const int steps = (a.K + 31) >> 5, per = (steps + KS - 1) / KS, s1 = min(steps, (ks + 1) * per);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int s = ks * per; s < s1; s += U) {
    uint4 wa[U], wb[U], xv[U][NB], xl[U][SPLIT ? NB : 1];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (s + u) * 32 + t4 * 8;
      const bool in = s + u < s1 && k < a.K;      // K is a multiple of 8: a piece is inside or outside as a whole
      wa[u] = in && r0 ? __ldg(reinterpret_cast<const uint4*>(w0 + k)) : zero;
      wb[u] = in && r1 ? __ldg(reinterpret_cast<const uint4*>(w1 + k)) : zero;
#pragma unroll
      for (int i = 0; i < NB; ++i) {
        xv[u][i] = zero;
        if (SPLIT) xl[u][i] = zero;
        if (in && xin[i]) xv[u][i] = ldx8(xr[i] + k, &xl[u][SPLIT ? i : 0]);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t a0[4] = {wa[u].x, wb[u].x, wa[u].y, wb[u].y}, a1[4] = {wa[u].z, wb[u].z, wa[u].w, wb[u].w};
#pragma unroll
      for (int i = 0; i < NB; ++i) {
        mma_16816(acc[i], a0, xv[u][i].x, xv[u][i].y);
        mma_16816(acc[i], a1, xv[u][i].z, xv[u][i].w);
        if (SPLIT) {
          mma_16816(acc[i], a0, xl[u][i].x, xl[u][i].y);
          mma_16816(acc[i], a1, xl[u][i].z, xl[u][i].w);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NB; ++i) {
    part[wrp][g][8 * i + 2 * t4] = acc[i][0];
    part[wrp][g][8 * i + 2 * t4 + 1] = acc[i][1];
    part[wrp][g + 8][8 * i + 2 * t4] = acc[i][2];
    part[wrp][g + 8][8 * i + 2 * t4 + 1] = acc[i][3];
  }
  __syncthreads();
  for (int e = threadIdx.x; e < RG * 16 * 8 * NB; e += 256) {
    const int r = e % (RG * 16), t = e / (RG * 16), rg = r >> 4;     // neighbouring threads: neighbouring output columns
    const int n = blockIdx.x * RG * 16 + r;
    if (t >= toks || n >= rows) continue;
    float v = 0.f;
    for (int k = 0; k < KS; ++k) v += part[rg * KS + k][r & 15][t];
    const int yr = THIN ? n : t, yc = THIN ? col0 + t : n;
    st1(Y + static_cast<long long>(yr) * a.ldy + yc, finish<TY>(a, a.row_scale ? v * a.row_scale[yr] : v, yc));
  }
}

// A few rows that each name their own source row, destination row and weight matrix (the expert choices of a decode step):
// one warp per (row, output column) streams that matrix's row once, so the step reads every chosen expert's weights at
// streaming rate instead of walking 64-row tiles that are almost empty.
template <typename TX, typename TW, typename TY, int VEC>
__global__ void __launch_bounds__(256) linear_picked_rows_kernel(LinearArgs a, PickedRows p) {
  const int lane = threadIdx.x & 31, wrp = threadIdx.x >> 5;
  const int n = blockIdx.x * 8 + wrp, r = blockIdx.y;
  if (n >= a.N) return;
  if (p.group_limit > 0 && (p.groups[r] < 0 || p.groups[r] >= p.group_limit)) return;   // a choice without a weight matrix
  const long long src = p.src_rows ? p.src_rows[r] : r / p.src_div;
  const long long dst = p.dst_rows[r];
  const TX* x = static_cast<const TX*>(a.X) + src * a.ldx;
  const TW* w = static_cast<const TW*>(a.W) + static_cast<long long>(p.groups[r]) * a.wbs + static_cast<long long>(n) * a.ldw;
  float acc = 0.f;
  for (int k = lane * VEC; k < a.K; k += 32 * VEC) {
    float wv[VEC], xv[VEC];
    if constexpr (VEC == 8) { ld8(w + k, wv); ld8(x + k, xv); } else { wv[0] = ld1(w + k); xv[0] = ld1(x + k); }
#pragma unroll
    for (int v = 0; v < VEC; ++v) acc = fmaf(xv[v], wv[v], acc);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
  if (lane == 0) st1(static_cast<TY*>(a.Y) + dst * a.ldy + n, finish<TY>(a, a.row_scale ? acc * a.row_scale[r] : acc, n));
}

template <typename TX, typename TW, typename TY>
int launch_picked(const LinearArgs& a, const PickedRows& p, cudaStream_t st) {
  const bool vec = a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.wbs % 8 == 0 && reinterpret_cast<uintptr_t>(a.X) % 16 == 0 &&
                   reinterpret_cast<uintptr_t>(a.W) % 16 == 0;
  dim3 grid((a.N + 7) / 8, p.rows);
  if (vec) linear_picked_rows_kernel<TX, TW, TY, 8><<<grid, 256, 0, st>>>(a, p);
  else linear_picked_rows_kernel<TX, TW, TY, 1><<<grid, 256, 0, st>>>(a, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

template <typename TX, typename TW, typename TY>
int launch_linear(const LinearArgs& a, cudaStream_t st) {
  const bool few = a.T <= 8 && !a.x_rows && !a.tile_group;
  if constexpr (sizeof(TW) == 2) {
    // B200_LIN_MMA_ROWS: A/B knob, the most rows that take the fragment kernel (0: none)
    static const int mma_rows = [] { const char* e = getenv("B200_LIN_MMA_ROWS"); return e ? std::min(16, std::max(0, atoi(e))) : 16; }();
    const bool vec = a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.xbs % 8 == 0 && a.wbs % 8 == 0 &&
                     reinterpret_cast<uintptr_t>(a.X) % 16 == 0 && reinterpret_cast<uintptr_t>(a.W) % 16 == 0;
    if (vec && a.T <= mma_rows && !a.x_rows && !a.tile_group) {
      const int steps = (a.K + 31) / 32;
      const int KS = steps >= 32 ? 8 : (steps >= 16 ? 4 : (steps >= 8 ? 2 : 1));
      dim3 grid((a.N + 128 / KS - 1) / (128 / KS), 1, a.batch);
      constexpr int U = sizeof(TX) == 4 ? 4 : 8;
      if (a.T <= 8) linear_rows_mma_kernel<TX, TY, 1, U, false><<<grid, 256, 0, st>>>(a, KS);
      else linear_rows_mma_kernel<TX, TY, 2, U / 2, false><<<grid, 256, 0, st>>>(a, KS);
      return cudaGetLastError() == cudaSuccess ? 0 : -2;
    }
    if constexpr (sizeof(TX) == 2) {
      // B200_LIN_THIN: A/B knob, the most columns that take the exchanged form (0: none)
      static const int thin = [] { const char* e = getenv("B200_LIN_THIN"); return e ? atoi(e) : 64; }();
      if (vec && a.N <= thin && a.batch == 1 && !a.x_rows && !a.tile_group) {
        const int steps = (a.K + 31) / 32;
        const int KS = steps >= 32 ? 8 : (steps >= 16 ? 4 : (steps >= 8 ? 2 : 1));
        dim3 grid((a.T + 128 / KS - 1) / (128 / KS), (a.N + 15) / 16);
        linear_rows_mma_kernel<TX, TY, 2, 4, true><<<grid, 256, 0, st>>>(a, KS);
        return cudaGetLastError() == cudaSuccess ? 0 : -2;
      }
    }
  }
  if (few) {
    const size_t ex = sizeof(TX), ew = sizeof(TW);
    const bool vec = a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.xbs % 8 == 0 && a.wbs % 8 == 0 &&
                     reinterpret_cast<uintptr_t>(a.X) % (8 * ex > 16 ? 16 : 8 * ex) == 0 && reinterpret_cast<uintptr_t>(a.W) % (8 * ew > 16 ? 16 : 8 * ew) == 0;
    dim3 grid((a.N + 7) / 8, 1, a.batch);
    if (vec) linear_rows_kernel<TX, TW, TY, 8><<<grid, 256, 0, st>>>(a);
    else linear_rows_kernel<TX, TW, TY, 1><<<grid, 256, 0, st>>>(a);
  } else {
    dim3 grid((a.N + BN - 1) / BN, (a.T + BM - 1) / BM, a.batch);
    if constexpr (sizeof(TW) == 2) {
      const bool vec = a.K % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.xbs % 8 == 0 && a.wbs % 8 == 0 &&
                       reinterpret_cast<uintptr_t>(a.X) % 16 == 0 && reinterpret_cast<uintptr_t>(a.W) % 16 == 0;
      if (vec) linear_tile_mma_kernel<TX, TY, true><<<grid, 256, 0, st>>>(a);
      else linear_tile_mma_kernel<TX, TY, false><<<grid, 256, 0, st>>>(a);
    } else {
      linear_tile_kernel<TX, TW, TY><<<grid, 256, 0, st>>>(a);
    }
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

int linear(const LinearArgs& a, cudaStream_t st) {
  if (a.T <= 0 || a.N <= 0) return 0;
  if (!a.X || !a.W || !a.Y || a.K <= 0 || a.batch < 1) return -1;
  if (a.tile_group && a.T % BM) return -1;
  const int key = (a.tx == DT_F32 ? 4 : 0) | (a.tw == DT_F32 ? 2 : 0) | (a.ty == DT_F32 ? 1 : 0);
  switch (key) {
    case 0: return launch_linear<bf16, bf16, bf16>(a, st);
    case 1: return launch_linear<bf16, bf16, float>(a, st);
    case 2: return launch_linear<bf16, float, bf16>(a, st);
    case 3: return launch_linear<bf16, float, float>(a, st);
    case 4: return launch_linear<float, bf16, bf16>(a, st);
    case 5: return launch_linear<float, bf16, float>(a, st);
    case 6: return launch_linear<float, float, bf16>(a, st);
    default: return launch_linear<float, float, float>(a, st);
  }
}


int linear_picked_rows(const LinearArgs& a, const PickedRows& p, cudaStream_t st) {
  if (p.rows <= 0 || a.N <= 0) return 0;
  if (!a.X || !a.W || !a.Y || a.K <= 0 || !p.dst_rows || !p.groups || (!p.src_rows && p.src_div < 1) || a.tw != a.tx) return -1;
  if (a.tx == DT_BF16) return a.ty == DT_BF16 ? launch_picked<bf16, bf16, bf16>(a, p, st) : launch_picked<bf16, bf16, float>(a, p, st);
  return a.ty == DT_BF16 ? launch_picked<float, float, bf16>(a, p, st) : launch_picked<float, float, float>(a, p, st);
}

}  // namespace b200
