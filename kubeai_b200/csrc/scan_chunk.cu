// The chunked form of the scalar-decay scan (mixers.h GlaArgs, dt_pre) for steps of prompt portions, on the tensor cores.
//
// With a_t = dt_rate d_t (the log decay of token t), c_t = a_1 + ... + a_t inside a chunk of 64 tokens and S the state in
// front of it, the recurrence S <- exp(a_t) S + d_t B_t x_t^T, y_t = S^T C_t unrolls to
//
//   y_t = exp(c_t) S^T C_t + sum_{j <= t} (B_j . C_t) exp(c_t - c_j) d_j x_j,
//   S'  = exp(c_last) S + sum_j exp(c_last - c_j) d_j B_j x_j^T,
//
// four matrix products per chunk.  Every exponent is at most 0 (no factor is ever the inverse of a decay), all sums and the
// state are fp32, and the products keep fp32 precision: B, C and x are bf16 as the convolution left them, so only the other
// operand (state, weighted scores, weighted x) needs more than one bf16 term, and it is split into three, 24 bits
// (mma_frag.cuh).  The result differs from the token-by-token scan by fp32 rounding alone.
//
// One CTA owns 64 value columns of a (head, sequence) and walks its chunks: 4 warps, each with 16 value columns.  The state
// lives transposed (value columns x state rows) in the warps' accumulators, which are the left operand of the next chunk's
// y without leaving the registers; the scores B C^T are computed 16 rows per warp and shared through shared memory.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdlib.h>

#include <algorithm>
#include <atomic>

#include "launch.h"
#include "mixers.h"
#include "mma_frag.cuh"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;
constexpr int kQ = 64;          // tokens per chunk
constexpr int kCols = 64;       // value columns per CTA
constexpr int kThreads = 128;
constexpr int kLdX = kCols + 8, kLdM = kQ + 8;

__device__ __forceinline__ float softplusf_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

size_t chunk_smem(int N) {
  return static_cast<size_t>(2) * kQ * (N + 8) * 2 + static_cast<size_t>(kQ) * kLdX * 2 + 3ull * kQ * kLdM * 2 + 4 * kQ * sizeof(float);
}

// NK: state rows in units of 16, at most (N = a.dim is any multiple of 16 up to 16 NK)
template <int NK>
__global__ void __launch_bounds__(kThreads) scalar_decay_chunk_kernel(GlaArgs a) {
  using namespace frag;
  extern __shared__ __align__(16) unsigned char smraw[];
  const int N = a.dim, P = a.vdim, nk = N / 16, LDN = N + 8;
  bf16* Bs = reinterpret_cast<bf16*>(smraw);     // [kQ][LDN] keys
  bf16* Cs = Bs + kQ * LDN;                      // [kQ][LDN] queries
  bf16* Xs = Cs + kQ * LDN;                      // [kQ][kLdX] values of the CTA's columns
  bf16* Ms = Xs + kQ * kLdX;                     // [3][kQ (t)][kLdM (j)] weighted scores, three bf16 terms
  float* cum = reinterpret_cast<float*>(Ms + 3 * kQ * kLdM);   // [kQ] c_t
  float* ecum = cum + kQ;                        // [kQ] exp(c_t)
  float* dts = ecum + kQ;                        // [kQ] d_t (0 past the portion)
  float* wts = dts + kQ;                         // [kQ] exp(c_last - c_t) d_t
  const int seq = blockIdx.z, head = blockIdx.y, p0 = blockIdx.x * kCols;
  const int tok0 = a.seqs[seq * 8 + 0], n = a.seqs[seq * 8 + 1], pos0 = a.seqs[seq * 8 + 2], slot = a.seqs[seq * 8 + 3];
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const bf16* base = static_cast<const bf16*>(a.qkv);
  const int qk0 = (head / a.group) * N;
  const bool live = p0 + 16 * w < P;             // warps past the last value column only help with the scores
  float* Sg = a.states + (static_cast<long long>(slot) * a.heads + head) * N * P;
  const int pr[2] = {p0 + 16 * w + g, p0 + 16 * w + g + 8};
  float S[NK][2][4];                             // [16 state rows][half][c]: value column pr[c / 2], state row 16 k + 8 half + 2 t4 + c % 2
#pragma unroll
  for (int k = 0; k < NK; ++k)
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int nn = 16 * k + 8 * h + 2 * t4 + (c & 1), p = pr[c >> 1];
        S[k][h][c] = (k < nk && p < P && pos0 > 0) ? Sg[static_cast<long long>(nn) * P + p] : 0.f;
      }
  const float rate = a.dt_rate[head], dbias = a.dt_bias[head];
  const int npiece = N / 8, xpiece = kCols / 8;

  for (int c0 = 0; c0 < n; c0 += kQ) {
    const int q = min(kQ, n - c0);
    __syncthreads();   // the last chunk's tiles are no longer read
    const bf16* rows = base + static_cast<long long>(tok0 + c0) * a.ld;
    for (int e = tid; e < kQ * npiece; e += kThreads) {
      const int t = e / npiece, c = (e - t * npiece) * 8;
      bf16 *db = Bs + t * LDN + c, *dc = Cs + t * LDN + c;
      if (t < q) {
        const bf16* r = rows + static_cast<long long>(t) * a.ld + qk0 + c;
        cp_async16(smem_addr(db), r + a.k_off);
        cp_async16(smem_addr(dc), r + a.q_off);
      } else {
        *reinterpret_cast<uint4*>(db) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(dc) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int e = tid; e < kQ * xpiece; e += kThreads) {
      const int t = e / xpiece, c = (e - t * xpiece) * 8;
      bf16* d = Xs + t * kLdX + c;
      if (t < q && p0 + c < P) cp_async16(smem_addr(d), rows + static_cast<long long>(t) * a.ld + a.v_off + head * P + p0 + c);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
    if (w == 0) {
      // step sizes and running log decays: lane l owns tokens 2l and 2l + 1
      float d[2], s[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        d[i] = t < q ? softplusf_(__bfloat162float(static_cast<const bf16*>(a.dt_pre)[static_cast<long long>(tok0 + c0 + t) * a.ld_dt + head]) + dbias) : 0.f;
        s[i] = rate * d[i];
      }
      float run = s[0] + s[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += v;
      }
      const float last = __shfl_sync(0xffffffffu, run, 31);
      const float before = __shfl_up_sync(0xffffffffu, run, 1);
      const float cc[2] = {(lane ? before : 0.f) + s[0], run};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        cum[t] = cc[i];
        ecum[t] = expf(cc[i]);
        dts[t] = d[i];
        wts[t] = expf(last - cc[i]) * d[i];
      }
    }
    cp_async_wait_all();
    __syncthreads();

    // ---- weighted scores: this warp's 16 keys j against the tokens t >= j's block
    {
      float G[4][2][4];
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) G[tb][h][c] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        if (k < nk) {
          uint32_t af[4];
          ldsm_x4(af, a_addr(Bs, LDN, 16 * w, 16 * k, lane));
#pragma unroll
          for (int tb = 0; tb < 4; ++tb) {
            if (tb >= w) {
              uint32_t bf_[4];
              ldsm_x4(bf_, b_addr(Cs, LDN, 16 * tb, 16 * k, lane));
              mma(G[tb][0], af, bf_[0], bf_[1]);
              mma(G[tb][1], af, bf_[2], bf_[3]);
            }
          }
        }
      }
      const float cj[2] = {cum[16 * w + g], cum[16 * w + g + 8]}, dj[2] = {dts[16 * w + g], dts[16 * w + g + 8]};
#pragma unroll
      for (int tb = 0; tb < 4; ++tb) {
        if (tb >= w) {
#pragma unroll
          for (int h = 0; h < 2; ++h)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              const int j = 16 * w + g + 8 * (c >> 1), t = 16 * tb + 8 * h + 2 * t4 + (c & 1);
              float v = j <= t ? G[tb][h][c] * (expf(cum[t] - cj[c >> 1]) * dj[c >> 1]) : 0.f;
#pragma unroll
              for (int s = 0; s < 3; ++s) {
                const bf16 b = __float2bfloat16_rn(v);
                Ms[(s * kQ + t) * kLdM + j] = b;
                v -= __bfloat162float(b);
              }
            }
        }
      }
    }
    __syncthreads();

    if (live) {
      // ---- y^T [16 value columns x 64 tokens]: the state's part, scaled per token, then the chunk's own
      float Y[4][2][4];
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) Y[tb][h][c] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        if (k < nk) {
          uint32_t s0[4], s1[4], s2[4];
          split3(S[k][0][0], S[k][0][1], &s0[0], &s1[0], &s2[0]);
          split3(S[k][0][2], S[k][0][3], &s0[1], &s1[1], &s2[1]);
          split3(S[k][1][0], S[k][1][1], &s0[2], &s1[2], &s2[2]);
          split3(S[k][1][2], S[k][1][3], &s0[3], &s1[3], &s2[3]);
#pragma unroll
          for (int tb = 0; tb < 4; ++tb) {
            uint32_t b[4];
            ldsm_x4(b, b_addr(Cs, LDN, 16 * tb, 16 * k, lane));
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              mma(Y[tb][h], s2, b[2 * h], b[2 * h + 1]);
              mma(Y[tb][h], s1, b[2 * h], b[2 * h + 1]);
              mma(Y[tb][h], s0, b[2 * h], b[2 * h + 1]);
            }
          }
        }
      }
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const float e0 = ecum[16 * tb + 8 * h + 2 * t4], e1 = ecum[16 * tb + 8 * h + 2 * t4 + 1];
          Y[tb][h][0] *= e0; Y[tb][h][1] *= e1; Y[tb][h][2] *= e0; Y[tb][h][3] *= e1;
        }
      const float decay = ecum[kQ - 1];
#pragma unroll
      for (int k = 0; k < NK; ++k)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[k][h][c] *= decay;
#pragma unroll
      for (int jb = 0; jb < 4; ++jb) {
        if (16 * jb >= q) break;       // no tokens there
        uint32_t xf[4];
        ldsm_x4_trans(xf, at_addr(Xs, kLdX, 16 * jb, 16 * w, lane));
#pragma unroll
        for (int tb = 0; tb < 4; ++tb) {
          if (tb >= jb) {
#pragma unroll
            for (int s = 2; s >= 0; --s) {
              uint32_t b[4];
              ldsm_x4(b, b_addr(Ms + s * kQ * kLdM, kLdM, 16 * tb, 16 * jb, lane));
              mma(Y[tb][0], xf, b[0], b[1]);
              mma(Y[tb][1], xf, b[2], b[3]);
            }
          }
        }
        // the state takes exp(c_last - c_j) d_j x_j B_j^T
        const float2 wl = *reinterpret_cast<const float2*>(wts + 16 * jb + 2 * t4), wh = *reinterpret_cast<const float2*>(wts + 16 * jb + 8 + 2 * t4);
        uint32_t x0[4], x1[4], x2[4];
        split3(low(xf[0]) * wl.x, high(xf[0]) * wl.y, &x0[0], &x1[0], &x2[0]);
        split3(low(xf[1]) * wl.x, high(xf[1]) * wl.y, &x0[1], &x1[1], &x2[1]);
        split3(low(xf[2]) * wh.x, high(xf[2]) * wh.y, &x0[2], &x1[2], &x2[2]);
        split3(low(xf[3]) * wh.x, high(xf[3]) * wh.y, &x0[3], &x1[3], &x2[3]);
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k < nk) {
            uint32_t b[4];
            ldsm_x4_trans(b, bt_addr(Bs, LDN, 16 * jb, 16 * k, lane));
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              mma(S[k][h], x2, b[2 * h], b[2 * h + 1]);
              mma(S[k][h], x1, b[2 * h], b[2 * h + 1]);
              mma(S[k][h], x0, b[2 * h], b[2 * h + 1]);
            }
          }
        }
      }
      float* out = a.o + static_cast<long long>(tok0 + c0) * (a.heads * P) + head * P;
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int t = 16 * tb + 8 * h + 2 * t4 + (c & 1), p = pr[c >> 1];
            if (t < q && p < P) out[static_cast<long long>(t) * (a.heads * P) + p] = Y[tb][h][c];
          }
    }
  }
#pragma unroll
  for (int k = 0; k < NK; ++k)
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int nn = 16 * k + 8 * h + 2 * t4 + (c & 1), p = pr[c >> 1];
        if (k < nk && p < P) Sg[static_cast<long long>(nn) * P + p] = S[k][h][c];
      }
}

template <int NK>
int launch(const GlaArgs& a, cudaStream_t st) {
  static std::atomic<unsigned long long> attr{0};
  const size_t smem = chunk_smem(a.dim);
  if (!ensure_dynamic_smem(scalar_decay_chunk_kernel<NK>, static_cast<int>(chunk_smem(16 * NK)), &attr)) return -2;
  scalar_decay_chunk_kernel<NK><<<dim3((a.vdim + kCols - 1) / kCols, a.heads, a.nseq), kThreads, smem, st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

bool scan_chunk_fits(const GlaArgs& a) {
  auto al = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  return a.dt_pre && a.t == DT_BF16 && a.act == GLA_ACT_NONE && !a.rope && a.q_scale == 1.f && a.k_scale == 1.f && a.dim % 16 == 0 && a.dim <= 128 &&
         a.vdim % 8 == 0 && a.ld % 8 == 0 && a.q_off % 8 == 0 && a.k_off % 8 == 0 && a.v_off % 8 == 0 && al(a.qkv);
}

int scan_chunk(const GlaArgs& a, cudaStream_t st) {
  if (!scan_chunk_fits(a)) return -1;
  if (a.dim <= 32) return launch<2>(a, st);
  return a.dim <= 64 ? launch<4>(a, st) : launch<8>(a, st);
}

}  // namespace b200
