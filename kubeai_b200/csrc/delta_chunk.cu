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
// Every exponent is at most 0.  The running log decays are summed in double, and factors between two tokens come from
// differences taken before they are rounded, so that weak decays behind strong ones keep their low bits: inside a block of 16
// tokens from the difference itself (c_t as two floats), across blocks as a product of three factors that meet at the block
// borders.  Keys and queries are bf16 as the convolution left them; their norms are scalars per token (taken from the diagonals of
// K K^T and Q Q^T) and enter the fp32 side.  The system is solved in blocks of 16 tokens: the four diagonal blocks are inverted by
// substitution (products of contractions, so no entry of an inverse exceeds 1), the rest are products.  Products keep fp32
// precision: an fp32 operand is split into three bf16 terms (mma_frag.cuh), against a bf16 operand all three count, against
// another fp32 operand the six term pairs down to 2^-24.  The result differs from the token-by-token scan by fp32 rounding alone.
//
// One CTA owns 64 value columns of a (head, sequence) and walks its chunks: 4 warps, each with 16 value columns.  The state
// lives transposed (value columns x key rows) in the warps' accumulators; R, U and o are value columns x tokens, so U leaves
// the solve as the left operand of the next products without leaving the registers.  A and the weighted scores are formed
// 16 tokens per warp and shared through shared memory, already split, as 16 x 16 blocks whose 16-byte halves are swapped in
// every other group of four rows (ldmatrix then meets no bank conflict).  The next chunk's keys, queries, values and gates
// are fetched while the current one is worked on.
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
constexpr int kBlock = 16 * 16;              // entries of a block
constexpr int kBlocks = 10;                  // blocks on and below the diagonal: (tb, jb) at tb (tb + 1) / 2 + jb
constexpr int kLdD = 20;                     // floats: row of a diagonal block while it is inverted

__device__ __forceinline__ float softplusf_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// per token: c_t in two parts, exp(c_t), exp(c_last - c_t), beta, exp(c_t - border before its block), exp(border behind its
// block - c_t); per pair of blocks: exp(border before tb - border behind jb)
struct Gates {
  float chi[kQ], clo[kQ], ecum[kQ], wl[kQ], beta[kQ], ea[kQ], ec[kQ], eb[16];
};

constexpr size_t chunk_smem(int D) {
  return static_cast<size_t>(3) * kQ * (D + 8) * 2 + static_cast<size_t>(kQ) * kLdV * 2 + 2ull * kBlocks * 3 * kBlock * 2 + 4 * 16 * kLdD * 4 + 2 * sizeof(Gates) + 2 * kQ * 4;
}

__device__ __forceinline__ int block_at(int tb, int jb) { return (tb * (tb + 1) / 2 + jb) * 3 * kBlock; }
// where entry (row r, column c) of a block lies
__device__ __forceinline__ int block_pos(int r, int c) { return r * 16 + ((c ^ ((r & 4) << 1)) & 15); }
// the accumulators of 16 tokens (two 8-token tiles) as the left operand of a product over those tokens, in three terms
__device__ __forceinline__ void acc_split(const float (*c)[4], uint32_t (*a)[4]) {
#pragma unroll
  for (int r = 0; r < 4; ++r) frag::split3(c[r >> 1][2 * (r & 1)], c[r >> 1][2 * (r & 1) + 1], &a[0][r], &a[1][r], &a[2][r]);
}
// the term pairs of an fp32 x fp32 product, the smallest first
constexpr int kPairs = 6;
__device__ __forceinline__ constexpr int pair_a(int i) { return i == 0 ? 2 : (i == 1 ? 0 : (i == 2 ? 1 : (i == 3 ? 1 : 0))); }
__device__ __forceinline__ constexpr int pair_b(int i) { return i == 0 ? 0 : (i == 1 ? 2 : (i == 2 ? 1 : (i == 3 ? 0 : (i == 4 ? 1 : 0)))); }

// NK: key rows in units of 16, at most (D = a.dim is any multiple of 16 up to 16 NK); FULL: exactly 16 NK rows, which leaves the
// loops over them without branches
template <int NK, bool FULL>
__global__ void __launch_bounds__(kThreads, 2) delta_chunk_kernel(DeltaArgs a, int sms) {
  using namespace frag;
  extern __shared__ __align__(16) unsigned char smraw[];
  const int D = FULL ? 16 * NK : a.dim, P = a.vdim, nk = FULL ? NK : D / 16, LDN = D + 8;
  bf16* Kbuf = reinterpret_cast<bf16*>(smraw);   // [2][kQ][LDN] keys, this chunk's and the next one's
  bf16* Qs = Kbuf + 2 * kQ * LDN;                // [kQ][LDN] queries
  bf16* Vs = Qs + kQ * LDN;                      // [kQ][kLdV] values of the CTA's columns
  bf16* As = Vs + kQ * kLdV;                     // [kBlocks][3][kBlock]: -A below the diagonal, the inverses of I + A on it
  bf16* Ms = As + kBlocks * 3 * kBlock;          // the weighted scores of the queries
  float* diag = reinterpret_cast<float*>(Ms + kBlocks * 3 * kBlock);   // [4][16][kLdD]
  Gates* gates = reinterpret_cast<Gates*>(diag + 4 * 16 * kLdD);       // [2]
  float* ik = reinterpret_cast<float*>(gates + 2);   // [kQ] 1 / |k_t|
  float* iq = ik + kQ;                               // [kQ] q_scale / |q_t|
  const int seq = blockIdx.z, head = blockIdx.y, p0 = blockIdx.x * kCols;
  const int tok0 = a.seqs[seq * 8 + 0], n = a.seqs[seq * 8 + 1], pos0 = a.seqs[seq * 8 + 2], slot = a.seqs[seq * 8 + 3];
  // later row blocks have more scores: every other wave of CTAs deals them to the warps in the opposite order, so that the two
  // CTAs of an SM load its four schedulers evenly
  const bool flip = ((blockIdx.z * gridDim.y + blockIdx.y) * gridDim.x + blockIdx.x) / sms & 1;
  const int tid = threadIdx.x, lane = tid & 31, w = flip ? 3 - (tid >> 5) : tid >> 5, g = lane >> 2, t4 = lane & 3;
  const bf16* base = static_cast<const bf16*>(a.qkv);
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
  // the piece of a 16-byte row piece grid this thread copies first, and its step to the next one
  const int npiece = D / 8, t_first = tid / npiece, c_first = tid - t_first * npiece, t_step = kThreads / npiece, c_step = kThreads - t_step * npiece;
  // a chunk's rows of one column block, by all threads; rows past the portion become zeros
  auto fetch_rows = [&](bf16* dst, int off, int c0) {
    const bf16* src = base + static_cast<long long>(tok0 + c0) * a.ld + off + qk0;
    int t = t_first, c = c_first;
    while (t < kQ) {
      bf16* d = dst + t * LDN + c * 8;
      if (c0 + t < n) cp_async16(smem_addr(d), src + t * a.ld + c * 8);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
      t += t_step; c += c_step;
      if (c >= npiece) { c -= npiece; ++t; }
    }
  };
  // the warp's own 16 value columns
  auto fetch_values = [&](int c0) {
    const int c = 16 * w + 8 * (lane & 1);
    const bf16* src = base + static_cast<long long>(tok0 + c0) * a.ld + a.v_off + head * P + p0 + c;
    for (int t = lane >> 1; t < kQ; t += 16) {
      bf16* d = Vs + t * kLdV + c;
      if (c0 + t < n && p0 + c < P) cp_async16(smem_addr(d), src + t * a.ld);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
  };
  // step sizes and decay factors of a chunk, by one warp: lane l owns tokens 2l and 2l + 1
  auto make_gates = [&](Gates& G, int c0) {
    const float rate = a.rate[head], dbias = a.dt_bias[head];
    float b[2], s[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      b[i] = 0.f; s[i] = 0.f;
      if (c0 + t < n) {
        const long long at = static_cast<long long>(tok0 + c0 + t) * a.ld_gate + head;
        b[i] = 1.0f / (1.0f + expf(-__bfloat162float(static_cast<const bf16*>(a.beta_pre)[at])));
        s[i] = rate * softplusf_(__bfloat162float(static_cast<const bf16*>(a.dt_pre)[at]) + dbias);
      }
    }
    double run = static_cast<double>(s[0]) + s[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const double last = __shfl_sync(0xffffffffu, run, 31), behind = __shfl_sync(0xffffffffu, run, lane | 7);
    const double prev = __shfl_sync(0xffffffffu, run, ((lane & 24) - 1) & 31), before = lane < 8 ? 0.0 : prev;
    const double cc[2] = {run - s[1], run};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      const float hi = static_cast<float>(cc[i]);
      G.chi[t] = hi;
      G.clo[t] = static_cast<float>(cc[i] - hi);
      G.ecum[t] = expf(hi) * (1.0f + G.clo[t]);
      G.wl[t] = expf(static_cast<float>(last - cc[i]));
      G.ea[t] = expf(static_cast<float>(cc[i] - before));
      G.ec[t] = expf(static_cast<float>(behind - cc[i]));
      G.beta[t] = b[i];
    }
    // lane 4 tb + jb (jb < tb): border before tb is the running sum of lane 8 tb - 1, border behind jb that of lane 8 jb + 7
    const int tb = lane >> 2 & 3, jb = lane & 3;
    const double at = __shfl_sync(0xffffffffu, run, (8 * tb - 1) & 31), from = __shfl_sync(0xffffffffu, run, 8 * jb + 7);
    if (lane < 16) G.eb[lane] = jb < tb ? expf(static_cast<float>(at - from)) : 0.f;
  };

  fetch_rows(Kbuf, a.k_off, 0);
  fetch_rows(Qs, a.q_off, 0);
  fetch_values(0);
  if (w == 0) make_gates(gates[0], 0);
  // the lane's ldmatrix row in a block that is the right operand: its rows are the operand's columns
  const int b_lane = block_pos((lane & 7) + 8 * (lane >> 4), 8 * ((lane >> 3) & 1));
  int buf = 0;
  for (int c0 = 0; c0 < n; c0 += kQ, buf ^= 1) {
    const int q = min(kQ, n - c0);
    const bf16* Ks = Kbuf + buf * kQ * LDN;
    const Gates& G = gates[buf];
    const bool more = c0 + kQ < n;
    cp_async_wait_all();
    __syncthreads();   // this chunk's tiles and gates are in place; nobody works on the last chunk any more
    if (more) fetch_rows(Kbuf + (buf ^ 1) * kQ * LDN, a.k_off, c0 + kQ);

    // ---- A and the weighted query scores of this warp's 16 tokens against the keys of its own and earlier blocks
    {
      float GK[4][2][4], GQ[4][2][4], QQ[2][4];
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          QQ[h][c] = 0.f;
#pragma unroll
          for (int jb = 0; jb < 4; ++jb) GK[jb][h][c] = GQ[jb][h][c] = 0.f;
        }
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        if (k < nk) {
          uint32_t ka[4], qa[4], qb[4], kb[4][4];
          ldsm_x4(ka, a_addr(Ks, LDN, 16 * w, 16 * k, lane));
          ldsm_x4(qa, a_addr(Qs, LDN, 16 * w, 16 * k, lane));
          ldsm_x4(qb, b_addr(Qs, LDN, 16 * w, 16 * k, lane));
#pragma unroll
          for (int jb = 0; jb < 4; ++jb)
            if (jb <= w) ldsm_x4(kb[jb], b_addr(Ks, LDN, 16 * jb, 16 * k, lane));
          mma(QQ[0], qa, qb[0], qb[1]);
          mma(QQ[1], qa, qb[2], qb[3]);
#pragma unroll
          for (int jb = 0; jb < 4; ++jb)
            if (jb <= w) {
              mma(GK[jb][0], ka, kb[jb][0], kb[jb][1]);
              mma(GK[jb][1], ka, kb[jb][2], kb[jb][3]);
              mma(GQ[jb][0], qa, kb[jb][0], kb[jb][1]);
              mma(GQ[jb][1], qa, kb[jb][2], kb[jb][3]);
            }
        }
      }
      // norms from the diagonals: row g + 8 hf meets its own column in half hf, lane t4 = g / 2, entry g % 2
      if (t4 == g >> 1) {
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          float kk = 0.f;
#pragma unroll
          for (int jb = 0; jb < 4; ++jb)
            if (jb == w) kk = (g & 1) ? GK[jb][hf][2 * hf + 1] : GK[jb][hf][2 * hf];
          const float qq = (g & 1) ? QQ[hf][2 * hf + 1] : QQ[hf][2 * hf];
          ik[16 * w + g + 8 * hf] = 1.0f / sqrtf(kk + a.unit_eps);
          iq[16 * w + g + 8 * hf] = a.q_scale / sqrtf(qq + a.unit_eps);
        }
      }
      __syncwarp();
      // the factors of this lane's rows and columns, read before anything is stored
      float wk[2], wq[2], row[2], th[2], tl[2], eb[4];
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int t = 16 * w + g + 8 * hf;
        wk[hf] = -G.beta[t] * ik[t]; wq[hf] = iq[t]; row[hf] = G.ea[t]; th[hf] = G.chi[t]; tl[hf] = G.clo[t];
      }
      float2 ec[4][2], dhi[2], dlo[2], dk[2];
#pragma unroll
      for (int jb = 0; jb < 4; ++jb) {
        eb[jb] = G.eb[4 * w + jb];
#pragma unroll
        for (int h = 0; h < 2; ++h) ec[jb][h] = *reinterpret_cast<const float2*>(G.ec + 16 * jb + 8 * h + 2 * t4);
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int j = 16 * w + 8 * h + 2 * t4;
        dhi[h] = *reinterpret_cast<const float2*>(G.chi + j); dlo[h] = *reinterpret_cast<const float2*>(G.clo + j); dk[h] = *reinterpret_cast<const float2*>(ik + j);
      }
#pragma unroll
      for (int jb = 0; jb < 4; ++jb) {
        if (jb <= w) {
          bf16 *pa = As + block_at(w, jb), *pm = Ms + block_at(w, jb);
#pragma unroll
          for (int hf = 0; hf < 2; ++hf) {
            const int r = g + 8 * hf;
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const int c = 8 * h + 2 * t4, at = block_pos(r, c);
              float f0, f1;
              if (jb < w) {
                const float rb = row[hf] * eb[jb];
                f0 = rb * ec[jb][h].x; f1 = rb * ec[jb][h].y;
              } else {
                const float d0 = expf(fminf((th[hf] - dhi[h].x) + (tl[hf] - dlo[h].x), 0.f)), d1 = expf(fminf((th[hf] - dhi[h].y) + (tl[hf] - dlo[h].y), 0.f));
                f0 = c <= r ? d0 : 0.f; f1 = c + 1 <= r ? d1 : 0.f;
              }
              uint32_t x[3];
              split3(GQ[jb][h][2 * hf] * (f0 * wq[hf]), GQ[jb][h][2 * hf + 1] * (f1 * wq[hf]), &x[0], &x[1], &x[2]);
#pragma unroll
              for (int s = 0; s < 3; ++s) *reinterpret_cast<uint32_t*>(pm + s * kBlock + at) = x[s];
              const float a0 = GK[jb][h][2 * hf] * (f0 * wk[hf]), a1 = GK[jb][h][2 * hf + 1] * (f1 * wk[hf]);     // -A
              if (jb < w) {
                split3(a0, a1, &x[0], &x[1], &x[2]);
#pragma unroll
                for (int s = 0; s < 3; ++s) *reinterpret_cast<uint32_t*>(pa + s * kBlock + at) = x[s];
              } else {
                // inside the block the keys' norms enter here; elsewhere they are factors of the writes
                *reinterpret_cast<float2*>(diag + (w * 16 + r) * kLdD + c) = make_float2(c < r ? a0 * dk[h].x : 0.f, c + 1 < r ? a1 * dk[h].y : 0.f);
              }
            }
          }
        }
      }
      __syncwarp();
      // the inverse of I + A on the warp's diagonal block: lane c (and c + 16 alike) owns its column c
      const float* blk = diag + w * 16 * kLdD;
      const int c = lane & 15;
      float x[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) {
        float s0 = r == c ? 1.f : 0.f, s1 = 0.f;
        float row[16];
#pragma unroll
        for (int j = 0; j < (r + 3) / 4; ++j) *reinterpret_cast<float4*>(row + 4 * j) = *reinterpret_cast<const float4*>(blk + r * kLdD + 4 * j);
#pragma unroll
        for (int j = 0; j < r; ++j) {
          if (j & 1) s1 = fmaf(row[j], x[j], s1);      // the block holds -A
          else s0 = fmaf(row[j], x[j], s0);
        }
        x[r] = s0 + s1;
      }
      bf16* pa = As + block_at(w, w);
      const bool low_half = lane < 16;
#pragma unroll
      for (int i = 0; i < 8; ++i) {       // one half of the lanes writes rows 0 .. 7, the other rows 8 .. 15
        float v = low_half ? x[i] : x[i + 8];
        bf16* d = pa + block_pos(i, c) + (low_half ? 0 : 8 * 16);
#pragma unroll
        for (int s = 0; s < 3; ++s) {
          const bf16 o = __float2bfloat16_rn(v);
          d[s * kBlock] = o;
          v -= __bfloat162float(o);
        }
      }
      if (w == 0 && more) make_gates(gates[buf ^ 1], c0 + kQ);
    }
    __syncthreads();

    float R[4][2][4], Y[4][2][4];
    if (live) {
      // ---- S^T k and S^T q of every token of the chunk, [16 value columns x 64 tokens]
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
        for (int h = 0; h < 2; ++h) {
          const int t = 16 * tb + 8 * h + 2 * t4;
          const bf16* v = Vs + t * kLdV + 16 * w + g;
          const float2 e = *reinterpret_cast<const float2*>(G.ecum + t), b = *reinterpret_cast<const float2*>(G.beta + t);
          const float2 fk = *reinterpret_cast<const float2*>(ik + t), fq = *reinterpret_cast<const float2*>(iq + t);
          R[tb][h][0] = b.x * fmaf(-(e.x * fk.x), R[tb][h][0], __bfloat162float(v[0]));
          R[tb][h][1] = b.y * fmaf(-(e.y * fk.y), R[tb][h][1], __bfloat162float(v[kLdV]));
          R[tb][h][2] = b.x * fmaf(-(e.x * fk.x), R[tb][h][2], __bfloat162float(v[8]));
          R[tb][h][3] = b.y * fmaf(-(e.y * fk.y), R[tb][h][3], __bfloat162float(v[kLdV + 8]));
          const float y0 = e.x * fq.x, y1 = e.y * fq.y;
          Y[tb][h][0] *= y0; Y[tb][h][1] *= y1; Y[tb][h][2] *= y0; Y[tb][h][3] *= y1;
        }
      const float decay = G.ecum[kQ - 1];
#pragma unroll
      for (int k = 0; k < NK; ++k)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) S[k][h][c] *= decay;
    }
    __syncthreads();   // the queries and the values are no longer read
    if (more) {
      fetch_rows(Qs, a.q_off, c0 + kQ);
      fetch_values(c0 + kQ);
    }
    if (live) {
      // ---- block by block: the writes U of 16 tokens, then what they change in later right-hand sides, outputs and the state
#pragma unroll
      for (int jb = 0; jb < 4; ++jb) {
        float U[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
        uint32_t us[3][4];
        {
          uint32_t b[3][4];
#pragma unroll
          for (int s = 0; s < 3; ++s) ldsm_x4(b[s], smem_addr(As + block_at(jb, jb) + s * kBlock + b_lane));
          acc_split(R[jb], us);
#pragma unroll
          for (int i = 0; i < kPairs; ++i) {
            mma(U[0], us[pair_a(i)], b[pair_b(i)][0], b[pair_b(i)][1]);
            mma(U[1], us[pair_a(i)], b[pair_b(i)][2], b[pair_b(i)][3]);
          }
        }
        // from here on the writes carry their keys' norms
        float wl[2][2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = 16 * jb + 8 * h + 2 * t4;
          const float2 fk = *reinterpret_cast<const float2*>(ik + t), l = *reinterpret_cast<const float2*>(G.wl + t);
          U[h][0] *= fk.x; U[h][1] *= fk.y; U[h][2] *= fk.x; U[h][3] *= fk.y;
          wl[h][0] = l.x; wl[h][1] = l.y;
        }
        acc_split(U, us);
#pragma unroll
        for (int tb = jb; tb < 4; ++tb) {
          uint32_t b[3][4], m[3][4];
#pragma unroll
          for (int s = 0; s < 3; ++s) {
            if (tb > jb) ldsm_x4(b[s], smem_addr(As + block_at(tb, jb) + s * kBlock + b_lane));
            ldsm_x4(m[s], smem_addr(Ms + block_at(tb, jb) + s * kBlock + b_lane));
          }
#pragma unroll
          for (int i = 0; i < kPairs; ++i) {
            if (tb > jb) {
              mma(R[tb][0], us[pair_a(i)], b[pair_b(i)][0], b[pair_b(i)][1]);
              mma(R[tb][1], us[pair_a(i)], b[pair_b(i)][2], b[pair_b(i)][3]);
            }
            mma(Y[tb][0], us[pair_a(i)], m[pair_b(i)][0], m[pair_b(i)][1]);
            mma(Y[tb][1], us[pair_a(i)], m[pair_b(i)][2], m[pair_b(i)][3]);
          }
        }
        // the state takes exp(c_last - c_j) k_j u_j^T
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int c = 0; c < 4; ++c) U[h][c] *= wl[h][c & 1];
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
      const long long ldo = static_cast<long long>(a.heads) * P;
      float* out = a.o + static_cast<long long>(tok0 + c0 + 2 * t4) * ldo + head * P + pr[0];
      const bool in1 = pr[1] < P;
#pragma unroll
      for (int tb = 0; tb < 4; ++tb)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = 16 * tb + 8 * h + e;
            if (t + 2 * t4 < q && pr[0] < P) {
              float* d = out + t * ldo;
              d[0] = Y[tb][h][e];
              if (in1) d[8] = Y[tb][h][2 + e];
            }
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

template <int NK, bool FULL>
int launch(const DeltaArgs& a, cudaStream_t st) {
  static std::atomic<unsigned long long> attr{0};
  if (!ensure_dynamic_smem(delta_chunk_kernel<NK, FULL>, static_cast<int>(chunk_smem(16 * NK)), &attr)) return -2;
  int dev = 0, sms = 148;
  if (cudaGetDevice(&dev) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  delta_chunk_kernel<NK, FULL><<<dim3((a.vdim + kCols - 1) / kCols, a.heads, a.nseq), kThreads, chunk_smem(a.dim), st>>>(a, sms);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}
template <int NK>
int launch(const DeltaArgs& a, cudaStream_t st) { return a.dim == 16 * NK ? launch<NK, true>(a, st) : launch<NK, false>(a, st); }

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
