// The chunked form of the gated delta rule (mixers.h DeltaArgs) for steps of prompt portions, on the tensor cores.
//
// Inside a chunk of 64 tokens let c_t be the running log decay (c_t = sum of log g up to t), S the state in front of the
// chunk, k_t and q_t the unit vectors.  Unrolled, the writes u_t of the chunk solve a unit lower triangular system, and
// everything else is a matrix product:
//
//   (I + A) U = R,   A[t, j] = beta_t exp(c_t - c_j) (k_t . k_j)  for j < t,   R_t = beta_t (v_t - exp(c_t) S^T k_t)
//   o_t = exp(c_t) S^T q_t + sum_{j <= t} exp(c_t - c_j) (q_t . k_j) u_j
//   S'  = exp(c_last) S + sum_j exp(c_last - c_j) k_j u_j^T
//
// Every exponent is at most 0.  The running log decays are summed in double and kept as two floats, so that the difference of
// two of them keeps its low bits behind strong decays.  Keys and queries are bf16 as the convolution left them; their norms
// are scalars per token and enter the fp32 side.  The system is solved in blocks of 16 tokens: the four diagonal blocks are
// inverted by substitution (products of contractions, so no entry of an inverse exceeds 1), the rest are products.  Products
// keep fp32 precision: an fp32 operand is split into three bf16 terms (mma_frag.cuh), against a bf16 operand all three count,
// against another fp32 operand the six term pairs down to 2^-24.  The result differs from the token-by-token scan by fp32
// rounding alone.
//
// One CTA owns 64 value columns of a (head, sequence) and walks its chunks: 4 warps, each with 16 value columns.  The state
// lives transposed (value columns x key rows) in the warps' accumulators; R, U and o are value columns x tokens, so U leaves
// the solve as the left operand of the next products without leaving the registers.  A and the weighted scores are formed
// 16 tokens per warp and shared in fp32 through shared memory, where the readers split them.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

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
constexpr int kLdV = kCols + 8;
constexpr int kLdM = kQ + 8;    // floats: the fragment reads (row g, columns 2 t) of a half warp fall into different banks

__device__ __forceinline__ float softplusf_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

constexpr size_t chunk_smem(int D) {
  return static_cast<size_t>(2) * kQ * (D + 8) * 2 + static_cast<size_t>(kQ) * kLdV * 2 + 2ull * kQ * kLdM * 4 + 8 * kQ * 4;
}

// the right operand of a product over 16 columns of a row-major fp32 matrix: rows r0 .. r0 + 15 are its 16 columns.  b[s][r]:
// term s of register r (registers 0, 1: the first eight columns, 2, 3: the rest), every entry multiplied by sign.
__device__ __forceinline__ void load_split(const float* m, int r0, int c0, int lane, float sign, uint32_t (*b)[4]) {
  const int g = lane >> 2, t4 = lane & 3;
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const float2 v = *reinterpret_cast<const float2*>(m + (r0 + 8 * (r >> 1) + g) * kLdM + c0 + 8 * (r & 1) + 2 * t4);
    frag::split3(sign * v.x, sign * v.y, &b[0][r], &b[1][r], &b[2][r]);
  }
}
// the accumulators of 16 tokens (two 8-token tiles) as the left operand of a product over those tokens, in three terms
__device__ __forceinline__ void acc_split(const float (*c)[4], uint32_t (*a)[4]) {
#pragma unroll
  for (int r = 0; r < 4; ++r) frag::split3(c[r >> 1][2 * (r & 1)], c[r >> 1][2 * (r & 1) + 1], &a[0][r], &a[1][r], &a[2][r]);
}
// the term pairs of an fp32 x fp32 product, the smallest first
constexpr int kPairs = 6;
__device__ __forceinline__ constexpr int pair_a(int i) { return i == 0 ? 2 : (i == 1 ? 0 : (i == 2 ? 1 : (i == 3 ? 1 : 0))); }
__device__ __forceinline__ constexpr int pair_b(int i) { return i == 0 ? 0 : (i == 1 ? 2 : (i == 2 ? 1 : (i == 3 ? 0 : (i == 4 ? 1 : 0)))); }

// NK: key rows in units of 16, at most (D = a.dim is any multiple of 16 up to 16 NK)
template <int NK>
__global__ void __launch_bounds__(kThreads, 2) delta_chunk_kernel(DeltaArgs a) {
  using namespace frag;
  extern __shared__ __align__(16) unsigned char smraw[];
  const int D = a.dim, P = a.vdim, nk = D / 16, LDN = D + 8;
  bf16* Ks = reinterpret_cast<bf16*>(smraw);     // [kQ][LDN] keys
  bf16* Qs = Ks + kQ * LDN;                      // [kQ][LDN] queries
  bf16* Vs = Qs + kQ * LDN;                      // [kQ][kLdV] values of the CTA's columns
  float* As = reinterpret_cast<float*>(Vs + kQ * kLdV);   // [kQ (t)][kLdM (j)] A below the diagonal blocks, their inverses on them
  float* Ms = As + kQ * kLdM;                    // [kQ (t)][kLdM (j)] weighted scores of the queries, zero above the diagonal
  float* chi = Ms + kQ * kLdM;                   // [kQ] c_t, high and low part
  float* clo = chi + kQ;
  float* ecum = clo + kQ;                        // [kQ] exp(c_t)
  float* beta = ecum + kQ;                       // [kQ] step sizes (0 past the portion)
  float* ik = beta + kQ;                         // [kQ] 1 / |k_t|
  float* iq = ik + kQ;                           // [kQ] q_scale / |q_t|
  float* wl = iq + kQ;                           // [kQ] exp(c_last - c_t)
  const int seq = blockIdx.z, head = blockIdx.y, p0 = blockIdx.x * kCols;
  const int tok0 = a.seqs[seq * 8 + 0], n = a.seqs[seq * 8 + 1], pos0 = a.seqs[seq * 8 + 2], slot = a.seqs[seq * 8 + 3];
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const bf16* base = static_cast<const bf16*>(a.qkv);
  const bf16 *beta_pre = static_cast<const bf16*>(a.beta_pre), *dt_pre = static_cast<const bf16*>(a.dt_pre);
  const int qk0 = head / (a.heads / a.kv_heads) * D;
  const bool live = p0 + 16 * w < P;             // warps past the last value column only help with the scores
  float* Sg = a.states + (static_cast<long long>(slot) * a.heads + head) * D * P;
  const int pr[2] = {p0 + 16 * w + g, p0 + 16 * w + g + 8};
  float S[NK][2][4];                             // [16 key rows][half][c]: value column pr[c / 2], key row 16 k + 8 half + 2 t4 + c % 2
#pragma unroll
  for (int k = 0; k < NK; ++k)
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int nn = 16 * k + 8 * h + 2 * t4 + (c & 1), p = pr[c >> 1];
        S[k][h][c] = (k < nk && p < P && pos0 > 0) ? Sg[nn * P + p] : 0.f;
      }
  const float rate = a.rate[head], dbias = a.dt_bias[head];
  const int npiece = D / 8, vpiece = kCols / 8;

  for (int c0 = 0; c0 < n; c0 += kQ) {
    const int q = min(kQ, n - c0);
    __syncthreads();   // the last chunk's tiles are no longer read
    const bf16* rows = base + static_cast<long long>(tok0 + c0) * a.ld;
    for (int e = tid; e < kQ * npiece; e += kThreads) {
      const int t = e / npiece, c = (e - t * npiece) * 8;
      bf16 *dk = Ks + t * LDN + c, *dq = Qs + t * LDN + c;
      if (t < q) {
        const bf16* r = rows + static_cast<long long>(t) * a.ld + qk0 + c;
        cp_async16(smem_addr(dk), r + a.k_off);
        cp_async16(smem_addr(dq), r + a.q_off);
      } else {
        *reinterpret_cast<uint4*>(dk) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(dq) = make_uint4(0, 0, 0, 0);
      }
    }
    for (int e = tid; e < kQ * vpiece; e += kThreads) {
      const int t = e / vpiece, c = (e - t * vpiece) * 8;
      bf16* d = Vs + t * kLdV + c;
      if (t < q && p0 + c < P) cp_async16(smem_addr(d), rows + static_cast<long long>(t) * a.ld + a.v_off + head * P + p0 + c);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
    if (w == 0) {
      // step sizes and running log decays: lane l owns tokens 2l and 2l + 1
      float b[2], s[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        b[i] = 0.f; s[i] = 0.f;
        if (t < q) {
          const long long at = static_cast<long long>(tok0 + c0 + t) * a.ld_gate + head;
          b[i] = 1.0f / (1.0f + expf(-__bfloat162float(beta_pre[at])));
          s[i] = rate * softplusf_(__bfloat162float(dt_pre[at]) + dbias);
        }
      }
      double run = static_cast<double>(s[0]) + s[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double v = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += v;
      }
      const double last = __shfl_sync(0xffffffffu, run, 31);
      const double cc[2] = {run - s[1], run};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        chi[t] = static_cast<float>(cc[i]);
        clo[t] = static_cast<float>(cc[i] - chi[t]);
        ecum[t] = expf(chi[t]) * (1.0f + clo[t]);
        wl[t] = expf(static_cast<float>(last - cc[i]));
        beta[t] = b[i];
      }
    }
    cp_async_wait_all();
    __syncthreads();
    {
      // norms: two lanes per token, alternating 16-byte pieces of its key and its query
      const int t = 16 * w + (lane >> 1);
      float kk = 0.f, qq = 0.f;
      for (int c = lane & 1; c < npiece; c += 2) {
        const uint4 kv = *reinterpret_cast<const uint4*>(Ks + t * LDN + 8 * c), qv = *reinterpret_cast<const uint4*>(Qs + t * LDN + 8 * c);
        const uint32_t ku[4] = {kv.x, kv.y, kv.z, kv.w}, qu[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          kk = fmaf(low(ku[i]), low(ku[i]), kk); kk = fmaf(high(ku[i]), high(ku[i]), kk);
          qq = fmaf(low(qu[i]), low(qu[i]), qq); qq = fmaf(high(qu[i]), high(qu[i]), qq);
        }
      }
      kk += __shfl_xor_sync(0xffffffffu, kk, 1);
      qq += __shfl_xor_sync(0xffffffffu, qq, 1);
      if ((lane & 1) == 0) {
        ik[t] = 1.0f / sqrtf(kk + a.unit_eps);
        iq[t] = a.q_scale / sqrtf(qq + a.unit_eps);
      }
    }
    __syncthreads();

    // ---- A and the weighted query scores of this warp's 16 tokens against the keys of its own and earlier blocks
#pragma unroll
    for (int jb = 0; jb < 4; ++jb) {
      if (jb <= w) {
        float GK[2][4], GQ[2][4];
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) GK[h][c] = GQ[h][c] = 0.f;
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k < nk) {
            uint32_t ka[4], qa[4], kb[4];
            ldsm_x4(ka, a_addr(Ks, LDN, 16 * w, 16 * k, lane));
            ldsm_x4(qa, a_addr(Qs, LDN, 16 * w, 16 * k, lane));
            ldsm_x4(kb, b_addr(Ks, LDN, 16 * jb, 16 * k, lane));
            mma(GK[0], ka, kb[0], kb[1]);
            mma(GK[1], ka, kb[2], kb[3]);
            mma(GQ[0], qa, kb[0], kb[1]);
            mma(GQ[1], qa, kb[2], kb[3]);
          }
        }
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int t = 16 * w + g + 8 * hf;
          const float th = chi[t], tl = clo[t], wk = beta[t] * ik[t], wq = iq[t];
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float av[2], mv[2];
#pragma unroll
            for (int c = 0; c < 2; ++c) {
              const int j = 16 * jb + 8 * h + 2 * t4 + c;
              const float f = j <= t ? expf((th - chi[j]) + (tl - clo[j])) * ik[j] : 0.f;
              av[c] = j < t ? GK[h][2 * hf + c] * (f * wk) : 0.f;
              mv[c] = GQ[h][2 * hf + c] * (f * wq);
            }
            const int at = t * kLdM + 16 * jb + 8 * h + 2 * t4;
            *reinterpret_cast<float2*>(As + at) = make_float2(av[0], av[1]);
            *reinterpret_cast<float2*>(Ms + at) = make_float2(mv[0], mv[1]);
          }
        }
      }
    }
    __syncwarp();
    {
      // the inverse of I + A on the warp's diagonal block, in place: lane c (and c + 16 alike) owns its column c
      float* blk = As + 16 * w * kLdM + 16 * w;
      const int c = lane & 15;
      float x[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) {
        float s0 = r == c ? 1.f : 0.f, s1 = 0.f;
        float row[16];
#pragma unroll
        for (int j = 0; j < (r + 3) / 4; ++j) *reinterpret_cast<float4*>(row + 4 * j) = *reinterpret_cast<const float4*>(blk + r * kLdM + 4 * j);
#pragma unroll
        for (int j = 0; j < r; ++j) {
          if (j & 1) s1 = fmaf(-row[j], x[j], s1);
          else s0 = fmaf(-row[j], x[j], s0);
        }
        x[r] = s0 + s1;
      }
      __syncwarp();
      if (lane < 16) {
#pragma unroll
        for (int r = 0; r < 16; ++r) blk[r * kLdM + c] = x[r];
      }
    }
    __syncthreads();

    if (live) {
      // ---- S^T k and S^T q of every token of the chunk, [16 value columns x 64 tokens]
      float R[4][2][4], Y[4][2][4];
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) R[tb][h][c] = Y[tb][h][c] = 0.f;
      if (pos0 + c0 > 0) {      // a sequence's first chunk starts from a zero state
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k < nk) {
            uint32_t s[3][4];
            acc_split(S[k], s);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              uint32_t kb[2][4], qb[2][4];
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                ldsm_x4(kb[i], b_addr(Ks, LDN, 32 * half + 16 * i, 16 * k, lane));
                ldsm_x4(qb[i], b_addr(Qs, LDN, 32 * half + 16 * i, 16 * k, lane));
              }
#pragma unroll
              for (int term = 2; term >= 0; --term)
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                  for (int h = 0; h < 2; ++h) {
                    mma(R[2 * half + i][h], s[term], kb[i][2 * h], kb[i][2 * h + 1]);
                    mma(Y[2 * half + i][h], s[term], qb[i][2 * h], qb[i][2 * h + 1]);
                  }
            }
          }
        }
      }
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int t = 16 * tb + 8 * h + 2 * t4 + (c & 1);
            const float v = __bfloat162float(Vs[t * kLdV + pr[c >> 1] - p0]), e = ecum[t];
            R[tb][h][c] = beta[t] * fmaf(-(e * ik[t]), R[tb][h][c], v);
            Y[tb][h][c] *= e * iq[t];
          }
      const float decay = ecum[kQ - 1];
#pragma unroll
      for (int k = 0; k < NK; ++k)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[k][h][c] *= decay;
      // ---- block by block: the writes U of 16 tokens, then what they change in later right-hand sides, outputs and the state
#pragma unroll
      for (int jb = 0; jb < 4; ++jb) {
        if (16 * jb >= q) break;       // no tokens there
        float U[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        uint32_t us[3][4];
        {
          uint32_t xs[3][4], b[3][4];
          acc_split(R[jb], xs);
          load_split(As, 16 * jb, 16 * jb, lane, 1.f, b);
#pragma unroll
          for (int i = 0; i < kPairs; ++i) {
            mma(U[0], xs[pair_a(i)], b[pair_b(i)][0], b[pair_b(i)][1]);
            mma(U[1], xs[pair_a(i)], b[pair_b(i)][2], b[pair_b(i)][3]);
          }
          acc_split(U, us);
        }
        {
          uint32_t m[3][4];
          load_split(Ms, 16 * jb, 16 * jb, lane, 1.f, m);
#pragma unroll
          for (int i = 0; i < kPairs; ++i) {
            mma(Y[jb][0], us[pair_a(i)], m[pair_b(i)][0], m[pair_b(i)][1]);
            mma(Y[jb][1], us[pair_a(i)], m[pair_b(i)][2], m[pair_b(i)][3]);
          }
        }
#pragma unroll
        for (int tb = jb + 1; tb < 4; ++tb) {
          uint32_t b[3][4], m[3][4];
          load_split(As, 16 * tb, 16 * jb, lane, -1.f, b);
          load_split(Ms, 16 * tb, 16 * jb, lane, 1.f, m);
#pragma unroll
          for (int i = 0; i < kPairs; ++i) {
            mma(R[tb][0], us[pair_a(i)], b[pair_b(i)][0], b[pair_b(i)][1]);
            mma(R[tb][1], us[pair_a(i)], b[pair_b(i)][2], b[pair_b(i)][3]);
            mma(Y[tb][0], us[pair_a(i)], m[pair_b(i)][0], m[pair_b(i)][1]);
            mma(Y[tb][1], us[pair_a(i)], m[pair_b(i)][2], m[pair_b(i)][3]);
          }
        }
        // the state takes exp(c_last - c_j) k_j u_j^T
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const int t = 16 * jb + 8 * h + 2 * t4 + (c & 1);
            U[h][c] *= wl[t] * ik[t];
          }
        acc_split(U, us);
#pragma unroll
        for (int k = 0; k < NK; k += 2) {
          if (k < nk) {
            uint32_t b[2][4];
            ldsm_x4_trans(b[0], bt_addr(Ks, LDN, 16 * jb, 16 * k, lane));
            if (k + 1 < nk) ldsm_x4_trans(b[1], bt_addr(Ks, LDN, 16 * jb, 16 * (k + 1), lane));
#pragma unroll
            for (int term = 2; term >= 0; --term)
#pragma unroll
              for (int i = 0; i < 2; ++i)
                if (k + i < nk) {
                  mma(S[k + i][0], us[term], b[i][0], b[i][1]);
                  mma(S[k + i][1], us[term], b[i][2], b[i][3]);
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
        if (k < nk && p < P) Sg[nn * P + p] = S[k][h][c];
      }
}

template <int NK>
int launch(const DeltaArgs& a, cudaStream_t st) {
  static std::atomic<unsigned long long> attr{0};
  if (!ensure_dynamic_smem(delta_chunk_kernel<NK>, static_cast<int>(chunk_smem(16 * NK)), &attr)) return -2;
  delta_chunk_kernel<NK><<<dim3((a.vdim + kCols - 1) / kCols, a.heads, a.nseq), kThreads, chunk_smem(a.dim), st>>>(a);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace

bool delta_chunk_fits(const DeltaArgs& a) {
  return a.t == DT_BF16 && a.dim % 16 == 0 && a.dim <= 128 && a.vdim % 8 == 0 && a.ld % 8 == 0 && a.q_off % 8 == 0 && a.k_off % 8 == 0 &&
         a.v_off % 8 == 0 && reinterpret_cast<uintptr_t>(a.qkv) % 16 == 0;
}

int delta_chunk(const DeltaArgs& a, cudaStream_t st) {
  if (!delta_chunk_fits(a)) return -1;
  if (a.dim <= 32) return launch<2>(a, st);
  return a.dim <= 64 ? launch<4>(a, st) : launch<8>(a, st);
}

}  // namespace b200
