// The gated delta rule (mixers.h DeltaArgs): a recurrent mixer whose per-head state S [dim, vdim] is a memory from unit keys
// to values.  Every token decays it by one scalar, reads what it holds under the token's key, and writes only beta times
// the difference to the token's value:  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
//
// The sequential scan: the columns of S are independent.  A column's key rows are shared by P neighbouring lanes of one warp
// (P a power of two, at most 32 rows each, in registers for the whole step), so the two sums a token needs over the rows,
// S^T k and S^T q, are P-lane shuffle reductions and the token loop has no barrier.  Both sums are taken over the state in
// front of the write, in one pass: with s = g S^T k and u = beta (v - s), the read-out after the write is
// o = g S^T q + (k . q) u, and k . q is formed once per token while it is staged.  A round stages G tokens in shared
// memory: a warp per token normalises its query and key (sums of squares in fp32), forms k . q, the step size beta and
// the decay g with the accurate library functions.  Everything is fp32, and the same operations run in the same order
// however a sequence was cut into steps.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdlib.h>

#include <algorithm>

#include "mixers.h"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;
__device__ __forceinline__ float ldf(const float* p) { return __ldg(p); }
__device__ __forceinline__ float ldf(const bf16* p) { return __bfloat162float(__ldg(p)); }
__device__ __forceinline__ float softplusf_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

constexpr int kPieces = 8;      // float4 pieces of a state column held by one thread (32 rows)
constexpr int kGroup = 16;      // tokens staged per round (fewer when dim is large)
constexpr int kThreads = 128;

// grid: (ceil(vdim / cols), heads, nseq), cols = kThreads / P.  A column's rows come in float4 pieces dealt to its P lanes in
// turn: lane p's m-th piece holds rows 4 (m P + p) .. + 3, m < M; Dp = 4 P M >= dim is the padded row length.
template <typename T>
__global__ void __launch_bounds__(kThreads) delta_scan_kernel(DeltaArgs a, int P, int M, int G) {
  extern __shared__ __align__(16) float sm[];
  const int seq = blockIdx.z, head = blockIdx.y;
  const int tok0 = a.seqs[seq * 8 + 0], n = a.seqs[seq * 8 + 1], pos0 = a.seqs[seq * 8 + 2], slot = a.seqs[seq * 8 + 3];
  const int D = a.dim, Dv = a.vdim, Dp = 4 * P * M, cols = kThreads / P;
  const int tid = threadIdx.x, lane = tid & 31, wrp = tid >> 5;
  const int p = lane & (P - 1), c = tid / P, j = blockIdx.x * cols + c;
  float* qs = sm;                     // [G][Dp] unit queries times q_scale
  float* ks = qs + G * Dp;            // [G][Dp] unit keys
  float* vs = ks + G * Dp;            // [G][cols]
  float* os = vs + G * cols;          // [G][cols]
  float* sc = os + G * cols;          // [3][G] decay, step size, k . q
  const T* base = static_cast<const T*>(a.qkv);
  const int g = head / (a.heads / a.kv_heads);
  float* Sg = a.states + (static_cast<long long>(slot) * a.heads + head) * D * Dv + j;
  const bool live = j < Dv;
  float S[kPieces][4];
  {
    const float* r = Sg + static_cast<long long>(4 * p) * Dv;      // one pointer walks the lane's rows
    const long long skip = static_cast<long long>(4 * P - 4) * Dv;
    const bool held = live && pos0 > 0;
#pragma unroll
    for (int m = 0; m < kPieces; ++m, r += skip)
#pragma unroll
      for (int e = 0; e < 4; ++e, r += Dv) S[m][e] = (held && m < M && 4 * (m * P + p) + e < D) ? *r : 0.f;
  }
  const float rate = a.rate[head], dt_bias = a.dt_bias[head];
  for (int g0 = 0; g0 < n; g0 += G) {
    const int gn = min(G, n - g0);
    __syncthreads();
    for (int tt = wrp; tt < gn; tt += kThreads / 32) {
      const long long row = static_cast<long long>(tok0) + g0 + tt;
      const T* q = base + row * a.ld + a.q_off + static_cast<long long>(g) * D;
      const T* k = base + row * a.ld + a.k_off + static_cast<long long>(g) * D;
      float qq = 0.f, kk = 0.f, qk = 0.f;
      for (int i = lane; i < D; i += 32) {
        const float x = ldf(q + i), y = ldf(k + i);
        qq = fmaf(x, x, qq); kk = fmaf(y, y, kk); qk = fmaf(x, y, qk);
      }
      for (int o = 16; o > 0; o >>= 1) {
        qq += __shfl_xor_sync(0xffffffffu, qq, o);
        kk += __shfl_xor_sync(0xffffffffu, kk, o);
        qk += __shfl_xor_sync(0xffffffffu, qk, o);
      }
      const float iq = a.q_scale / sqrtf(qq + a.unit_eps), ik = 1.0f / sqrtf(kk + a.unit_eps);
      for (int i = lane; i < Dp; i += 32) {
        qs[tt * Dp + i] = i < D ? ldf(q + i) * iq : 0.f;
        ks[tt * Dp + i] = i < D ? ldf(k + i) * ik : 0.f;
      }
      if (lane == 0) {
        const float b = ldf(static_cast<const T*>(a.beta_pre) + row * a.ld_gate + head);
        const float d = softplusf_(ldf(static_cast<const T*>(a.dt_pre) + row * a.ld_gate + head) + dt_bias);
        sc[tt] = expf(rate * d);
        sc[G + tt] = 1.0f / (1.0f + expf(-b));
        sc[2 * G + tt] = qk * iq * ik;
      }
    }
    for (int e = tid; e < gn * cols; e += kThreads) {
      const int tt = e / cols, cc = e - tt * cols, jc = blockIdx.x * cols + cc;
      vs[e] = jc < Dv ? ldf(base + (static_cast<long long>(tok0) + g0 + tt) * a.ld + a.v_off + static_cast<long long>(head) * Dv + jc) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < gn; ++tt) {
      const float4* q4 = reinterpret_cast<const float4*>(qs + tt * Dp);
      const float4* k4 = reinterpret_cast<const float4*>(ks + tt * Dp);
      const float decay = sc[tt];
      float rk[4] = {0.f, 0.f, 0.f, 0.f}, rq[4] = {0.f, 0.f, 0.f, 0.f};
      float4 kv[kPieces];
#pragma unroll
      for (int m = 0; m < kPieces; ++m) {
        if (m < M) {
          const float4 qa = q4[m * P + p];
          kv[m] = k4[m * P + p];
          rk[0] = fmaf(S[m][0], kv[m].x, rk[0]); rq[0] = fmaf(S[m][0], qa.x, rq[0]);
          rk[1] = fmaf(S[m][1], kv[m].y, rk[1]); rq[1] = fmaf(S[m][1], qa.y, rq[1]);
          rk[2] = fmaf(S[m][2], kv[m].z, rk[2]); rq[2] = fmaf(S[m][2], qa.z, rq[2]);
          rk[3] = fmaf(S[m][3], kv[m].w, rk[3]); rq[3] = fmaf(S[m][3], qa.w, rq[3]);
        }
      }
      float sk = (rk[0] + rk[1]) + (rk[2] + rk[3]), sq = (rq[0] + rq[1]) + (rq[2] + rq[3]);
      for (int o = P >> 1; o > 0; o >>= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
      }
      const float u = sc[G + tt] * fmaf(-decay, sk, vs[tt * cols + c]);
      if (p == 0) os[tt * cols + c] = fmaf(sc[2 * G + tt], u, decay * sq);
#pragma unroll
      for (int m = 0; m < kPieces; ++m) {
        if (m < M) {
          S[m][0] = fmaf(kv[m].x, u, decay * S[m][0]);
          S[m][1] = fmaf(kv[m].y, u, decay * S[m][1]);
          S[m][2] = fmaf(kv[m].z, u, decay * S[m][2]);
          S[m][3] = fmaf(kv[m].w, u, decay * S[m][3]);
        }
      }
    }
    __syncthreads();
    for (int e = tid; e < gn * cols; e += kThreads) {
      const int tt = e / cols, cc = e - tt * cols, jc = blockIdx.x * cols + cc;
      if (jc < Dv) a.o[(static_cast<long long>(tok0) + g0 + tt) * (static_cast<long long>(a.heads) * Dv) + static_cast<long long>(head) * Dv + jc] = os[e];
    }
  }
  if (live) {
    float* r = Sg + static_cast<long long>(4 * p) * Dv;
    const long long skip = static_cast<long long>(4 * P - 4) * Dv;
#pragma unroll
    for (int m = 0; m < kPieces; ++m, r += skip)
#pragma unroll
      for (int e = 0; e < 4; ++e, r += Dv)
        if (m < M && 4 * (m * P + p) + e < D) *r = S[m][e];
  }
}

}  // namespace

int delta_scan(const DeltaArgs& a, cudaStream_t st) {
  if (a.nseq <= 0 || a.T <= 0) return 0;
  if (!a.qkv || !a.beta_pre || !a.dt_pre || !a.dt_bias || !a.rate || !a.states || !a.seqs || !a.o || a.heads < 1 || a.kv_heads < 1 ||
      a.heads % a.kv_heads || a.dim < 1 || a.vdim < 1) return -1;
  if (delta_chunk_fits(a)) {
    // steps that bring portions (B200_DELTA_CHUNK: A/B knob, the mean portion from which the chunked form runs; 0 = never)
    const char* e = getenv("B200_DELTA_CHUNK");
    const int from = e ? atoi(e) : 8;
    if (from > 0 && a.T >= static_cast<long long>(from) * a.nseq) return delta_chunk(a, st);
  }
  int P = 1;
  while (P * 4 * kPieces < a.dim) P <<= 1;
  if (P > 32) return -1;   // dim <= 1024
  const int M = (a.dim + 4 * P - 1) / (4 * P), cols = kThreads / P;
  auto smem_for = [&](int G) { return static_cast<size_t>(G) * (2 * 4 * P * M + 2 * cols + 3) * sizeof(float); };
  int G = kGroup;
  while (G > 1 && smem_for(G) > 44 * 1024) G >>= 1;
  dim3 grid((a.vdim + cols - 1) / cols, a.heads, a.nseq);
  if (a.t == DT_BF16) delta_scan_kernel<bf16><<<grid, kThreads, smem_for(G), st>>>(a, P, M, G);
  else delta_scan_kernel<float><<<grid, kThreads, smem_for(G), st>>>(a, P, M, G);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace b200
