// Grouped projection GEMM for mixtures of experts (tcgen05 cta_group::2): the rows of every expert, sorted by expert, times
// that expert's matrix, in ONE launch whose tile list is read from device memory.
//     out[r, n] = sum_k X[r, k] * W[e(r) * N + n, k]        (bf16 x bf16 -> fp32 -> bf16)
// X holds the rows of expert e at [first_e, first_e + rows_e) (the table moe_align leaves, so no count ever travels to the
// host); W is the experts' matrices stacked row-wise.  With `glu` the rows of W alternate in blocks of 64 gate rows and their 64
// up rows, and the epilogue writes silu(gate) * up, half as many columns.
//
// A CTA pair works on a tile of 256 weight rows x up to 256 rows of one expert; an expert's rows are cut into equal tiles.
// Work items run expert by expert, weight tile by weight tile with its row tiles side by side, so that neighbouring pairs use
// one weight slab at the same time, and are dealt to the pairs in turn.  Per CTA: one producer thread (TMA: its own 128
// weight rows and its half of the row tile), one issuing thread in the leader, four epilogue warps that drain one of two
// accumulators while the other is being filled.  Every wait has an iteration limit: a pair that gives up stops its work, sets
// an error flag for the host, and still meets its peer before the tensor memory is freed.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <atomic>

#include "gemm.h"
#include "launch.h"
#include "ptx.cuh"
#include "umma2.cuh"

namespace b200 {
namespace {

typedef __nv_bfloat16 bf16;
constexpr int kSlab = 128;      // weight rows per CTA
constexpr int kRows = 256;      // rows of X per tile, at most
constexpr int kBlockK = 64, kUmmaK = 16;
constexpr int kThreads = 192;
constexpr int kABytes = kSlab * kBlockK * 2, kBBytes = kRows / 2 * kBlockK * 2, kStageBytes = kABytes + kBBytes;
constexpr int kStages = 6;
constexpr int kOutRows = 64;    // rows of X per epilogue round
constexpr int kOutBytes = kOutRows * kSlab * 2;
constexpr int kSmem = 1024 + kStages * kStageBytes + 256 + 2 * kOutBytes;
constexpr int kWaitLimit = 1 << 22;

struct Tile {
  int wrow;      // first row of the stacked weight matrix
  int n0;        // the same within the expert's matrix
  int row0;      // first row of X
  int rows;      // rows of X (at most kRows)
};

// Walks this pair's items: `next` advances by one item of the pair, expert by expert.
struct Walk {
  const int* expert_rows;
  int experts, mt, N, rows;   // without a table: one matrix, `rows` rows from 0
  int e = 0;
  long long base = 0;    // items of the experts before e
  __device__ bool at(long long item, Tile* t) {
    while (e < experts) {
      const int cnt = expert_rows ? expert_rows[2 * e + 1] : rows;
      const int ntt = (cnt + kRows - 1) / kRows;
      const long long n = static_cast<long long>(ntt) * mt;
      if (item < base + n) {
        const int r = static_cast<int>(item - base), m = r / ntt, tt = r - m * ntt;
        const int per = ((cnt + ntt - 1) / ntt + 15) & ~15;     // equal tiles, whole 16-row steps (at most kRows)
        t->n0 = m * 2 * kSlab;
        t->wrow = e * N + t->n0;
        t->row0 = (expert_rows ? expert_rows[2 * e] : 0) + tt * per;
        t->rows = min(per, cnt - tt * per);
        if (t->rows > 0) return true;
        t->rows = 0;       // rounding up to 16 may leave the last tile of an expert empty
        return true;
      }
      base += n;
      ++e;
    }
    return false;
  }
};

__device__ __forceinline__ bool wait_limited(uint32_t bar, uint32_t parity) {
  for (int i = 0; i < kWaitLimit; ++i)
    if (mbar_try_wait(bar, parity)) return true;
  return false;
}
// whether all 128 epilogue threads say yes (they also meet here)
__device__ __forceinline__ bool all_epilogue(bool v) {
  uint32_t r;
  asm volatile(
      "{\n"
      ".reg .pred p, q;\n"
      "setp.ne.u32 p, %1, 0;\n"
      "barrier.cta.red.and.pred q, 2, 128, p;\n"
      "selp.u32 %0, 1, 0, q;\n"
      "}\n"
      : "=r"(r)
      : "r"(v ? 1u : 0u)
      : "memory");
  return r != 0;
}

__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(kThreads, 1)
gemm_grouped_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const int* expert_rows, int experts, int rows,
                    bf16* out, int ldo, int N, int K, int glu, int* error) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t bar_base = smem_base + kStages * kStageBytes;
  auto full_bar = [&](int s) { return bar_base + 8u * s; };                     // the leader's copy is the live one
  auto empty_bar = [&](int s) { return bar_base + 8u * (kStages + s); };        // both CTAs
  auto tfull_bar = [&](int a) { return bar_base + 8u * (2 * kStages + a); };    // both CTAs
  auto tempty_bar = [&](int a) { return bar_base + 8u * (2 * kStages + 2 + a); };   // the leader's copy, 8 arrivals
  const uint32_t tmem_slot = bar_base + 8u * (2 * kStages + 4);
  uint8_t* stage_out = smem_raw + (bar_base + 256 - smem_u32(smem_raw));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t rank = cluster_ctarank();
  const bool leader = rank == 0;
  const int units = gridDim.x >> 1, unit = blockIdx.x >> 1, KB = (K + kBlockK - 1) / kBlockK;
  Walk walk;
  walk.expert_rows = expert_rows; walk.experts = experts; walk.mt = (N + 2 * kSlab - 1) / (2 * kSlab); walk.N = N; walk.rows = rows;

  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_x);
  }
  if (warp == 1) {
    if (lane == 0) {
      for (int s = 0; s < kStages; ++s) { mbar_init(full_bar(s), 1); mbar_init(empty_bar(s), 1); }
      for (int a = 0; a < 2; ++a) { mbar_init(tfull_bar(a), 1); mbar_init(tempty_bar(a), 8); }   // 4 epilogue warps of each CTA
      fence_mbar_init();
    }
    __syncwarp();
    tmem_alloc2(tmem_slot, 512);
    tmem_relinquish2();
  }
  tc_fence_before();
  cluster_sync_all();   // barrier inits and the TMEM allocation are visible to the peer
  tc_fence_after();
  const uint32_t tmem_base = *reinterpret_cast<volatile uint32_t*>(smem_raw + (tmem_slot - smem_u32(smem_raw)));
  bool ok = true;

  if (warp == 0) {
    if (lane == 0) {
      int stage = 0;
      uint32_t phase = 0;
      Tile t;
      for (long long item = unit; ok && walk.at(item, &t); item += units) {
        if (!t.rows) continue;
        const int nc = (t.rows + 15) & ~15;
        for (int kb = 0; kb < KB; ++kb) {
          if (!wait_limited(empty_bar(stage), phase ^ 1u)) { ok = false; break; }
          const uint32_t sa = smem_base + stage * kStageBytes;
          if (leader) mbar_arrive_expect_tx(full_bar(stage), 2u * kStageBytes);
          tma_load_2d_pair(sa, &tm_w, full_bar(stage), kb * kBlockK, t.wrow + static_cast<int>(rank) * kSlab, kEvictNormal);
          // this CTA stages the rank-th half of the row tile (the box is always kRows / 2 rows; rows past nc / 2 are not used)
          tma_load_2d_pair(sa + kABytes, &tm_x, full_bar(stage), kb * kBlockK, t.row0 + static_cast<int>(rank) * (nc >> 1), kEvictLast);
          if (++stage == kStages) { stage = 0; phase ^= 1u; }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && leader) {
      int stage = 0, acc = 0;
      uint32_t phase = 0, acc_phase = 0;
      Tile t;
      for (long long item = unit; ok && walk.at(item, &t); item += units) {
        if (!t.rows) continue;
        const uint32_t idesc = umma_idesc_bf16(2 * kSlab, (t.rows + 15) & ~15);
        if (!wait_limited(tempty_bar(acc), acc_phase ^ 1u)) { ok = false; break; }
        tc_fence_after();
        for (int kb = 0; kb < KB; ++kb) {
          if (!wait_limited(full_bar(stage), phase)) { ok = false; break; }
          tc_fence_after();
          const uint32_t sa = smem_base + stage * kStageBytes;
          const uint64_t a_desc = umma_desc_kmajor_sw128(sa), b_desc = umma_desc_kmajor_sw128(sa + kABytes);
#pragma unroll
          for (int k = 0; k < kBlockK / kUmmaK; ++k)
            umma2_bf16(tmem_base + acc * kRows, a_desc + 2u * k, b_desc + 2u * k, idesc, (kb > 0 || k > 0) ? 1u : 0u);
          umma2_commit_pair(empty_bar(stage), 3);
          if (kb == KB - 1) umma2_commit_pair(tfull_bar(acc), 3);
          if (++stage == kStages) { stage = 0; phase ^= 1u; }
        }
        if (++acc == 2) { acc = 0; acc_phase ^= 1u; }
      }
    }
  } else {
    const int q = warp & 3, row = q * 32 + lane, et = threadIdx.x - 64;
    int acc = 0, sbuf = 0;
    uint32_t acc_phase = 0;
    Tile t;
    for (long long item = unit; ok && walk.at(item, &t); item += units) {
      if (!t.rows) continue;
      ok = all_epilogue(wait_limited(tfull_bar(acc), acc_phase));
      if (!ok) break;
      tc_fence_after();
      const int n0 = t.n0 + static_cast<int>(rank) * kSlab;    // first column of this CTA's slab in the expert's output
      const uint32_t taddr = tmem_base + (static_cast<uint32_t>(q * 32) << 16) + acc * kRows;
      for (int c0 = 0; c0 < t.rows; c0 += kOutRows) {
        const bool two = c0 + 32 < t.rows;
        uint32_t v0[32], v1[32];
        tmem_ld_32x32(taddr + c0, v0);
        if (two) tmem_ld_32x32(taddr + c0 + 32, v1);
        tmem_ld_wait();
        bf16* sb = reinterpret_cast<bf16*>(stage_out + sbuf * kOutBytes);
#pragma unroll
        for (int j = 0; j < 32; ++j) sb[j * kSlab + row] = __float2bfloat16_rn(__uint_as_float(v0[j]));
        if (two) {
#pragma unroll
          for (int j = 0; j < 32; ++j) sb[(32 + j) * kSlab + row] = __float2bfloat16_rn(__uint_as_float(v1[j]));
        }
        // one barrier per round: a thread past it has finished its pass over the buffer staged two rounds ago
        asm volatile("bar.sync 1, 128;" ::: "memory");
        const int left = t.rows - c0;
        bf16* dst = out + static_cast<size_t>(t.row0 + c0) * ldo;
        if (glu) {
          // rows 0..63 of the slab are gate rows, 64..127 the matching up rows: output columns n0 / 2 ..
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int it = et + i * 128, j = it >> 3, c = (it & 7) * 8;
            if (j < left && n0 + kSlab <= N) {
              const uint4 g = *reinterpret_cast<const uint4*>(sb + j * kSlab + c), u = *reinterpret_cast<const uint4*>(sb + j * kSlab + 64 + c);
              const uint32_t gu[4] = {g.x, g.y, g.z, g.w}, uu[4] = {u.x, u.y, u.z, u.w};
              uint32_t o[4];
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                const float g0 = __uint_as_float(gu[k] << 16), g1 = __uint_as_float(gu[k] & 0xffff0000u);
                o[k] = pack_bf16x2(__fdividef(g0, 1.0f + __expf(-g0)) * __uint_as_float(uu[k] << 16),
                                   __fdividef(g1, 1.0f + __expf(-g1)) * __uint_as_float(uu[k] & 0xffff0000u));
              }
              *reinterpret_cast<uint4*>(dst + static_cast<size_t>(j) * ldo + n0 / 2 + c) = make_uint4(o[0], o[1], o[2], o[3]);
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const int it = et + i * 128, j = it >> 4, c = (it & 15) * 8;
            if (j < left && n0 + c < N)
              *reinterpret_cast<uint4*>(dst + static_cast<size_t>(j) * ldo + n0 + c) = *reinterpret_cast<const uint4*>(sb + j * kSlab + c);
          }
        }
        sbuf ^= 1;
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) {
        if (leader) mbar_arrive(tempty_bar(acc));
        else mbar_arrive_cluster_relaxed(tempty_bar(acc), 0);
      }
      if (++acc == 2) { acc = 0; acc_phase ^= 1u; }
    }
  }
  if (!ok && error) *reinterpret_cast<volatile int*>(error) = 1;
  tc_fence_before();
  __syncwarp();
  cluster_sync_all();   // nobody of the pair works any more
  tc_fence_after();
  if (warp == 1) tmem_dealloc2(tmem_base, 512);
}

}  // namespace

int gemm_grouped_plan(GroupedPlan* p, const void* W, int experts, int N, int K) {
  if (experts < 1 || N < 8 || K < 8 || N % 8 || K % 8 || reinterpret_cast<uintptr_t>(W) % 16) return -1;
  p->experts = experts; p->N = N; p->K = K;
  return tmap_encode_bf16_2d(&p->tm_w, W, static_cast<uint64_t>(experts) * N, K, K, kSlab, kBlockK, 1);
}

int gemm_grouped_x_map(CUtensorMap* tm, const void* X, int rows, int K) { return tmap_encode_bf16_2d(tm, X, rows, K, K, kRows / 2, kBlockK, 1); }

int gemm_grouped_run(const GroupedPlan& p, const CUtensorMap& tm_x, const int* expert_rows, void* out, int ldo, bool glu, int sms, int* error,
                     cudaStream_t st, int rows) {
  if ((!expert_rows && (p.experts != 1 || rows < 1)) || !out || ldo % 8 || reinterpret_cast<uintptr_t>(out) % 16 || sms < 2 || (glu && p.N % kSlab)) return -1;
  static std::atomic<unsigned long long> attr{0};
  if (!ensure_dynamic_smem(gemm_grouped_kernel, kSmem, &attr)) return -2;
  gemm_grouped_kernel<<<sms / 2 * 2, kThreads, kSmem, st>>>(p.tm_w, tm_x, expert_rows, p.experts, rows, static_cast<bf16*>(out), ldo, p.N, p.K, glu ? 1 : 0, error);
  return cudaGetLastError() == cudaSuccess ? 0 : -2;
}

}  // namespace b200
