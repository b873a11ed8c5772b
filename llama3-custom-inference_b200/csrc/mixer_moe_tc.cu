// Experts' products on the 5th-generation tensor cores: sorted token rows x [rows, K] times their expert's matrix [N, K],
// bf16 operands, fp32 accumulation (include/l3ci_mixers.h, l3ci_moe_gemm).
//
// Persistent CTAs walk the tiles (128 rows of one expert) x (BN columns).  Warp 0 asks for the operand tiles (bulk tensor
// copies, 64 columns of K per stage, 128-byte swizzle), warp 1 issues tcgen05.mma into one of two accumulators in tensor memory,
// warps 4-7 take the finished accumulator of the tile before: a thread owns a row.  A gated product has its gate columns in the
// first and its up columns in the second half of the accumulator, so that the activation needs no pass of its own.  A tile's
// rows behind the expert's last one are other experts' rows or nothing (read as zeros); they are not stored.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "bf16x8.cuh"
#include "mixer_moe.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "tcgen05.cuh"
#include "tensor_map.h"

namespace l3ci {
namespace {

constexpr int kRows = 128;
constexpr int kDeep = 64;                         // columns of K per stage: 128 bytes
constexpr int kThreads = 256;
constexpr int kXBytes = kRows * 128;

struct MoeTcParams {
  l3ci_moe_gemm_args a;
  int col_tiles;
};

template <int BN>
struct MoeShape {
  static constexpr int kWBytes = BN * 128;
  static constexpr int kStageBytes = kXBytes + kWBytes;
  static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 6 : 8;
  static constexpr uint32_t kTmem = 2 * BN;       // two accumulators
  static constexpr size_t kSmem = 1024 + (size_t)kStages * kStageBytes + (2 * kStages + 4) * 8 + 16;
};

template <int BN, bool GATED>
__global__ void __launch_bounds__(kThreads, 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap xmap, const __grid_constant__ CUtensorMap wmap, const __grid_constant__ MoeTcParams p) {
  using Sh = MoeShape<BN>;
  constexpr int kStages = Sh::kStages;
  constexpr int kCols = GATED ? BN / 2 : BN;      // output columns of a tile
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t ring = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kStages * Sh::kStageBytes);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * kStages + 4);
  const uint32_t full0 = smem_u32(bars), empty0 = full0 + kStages * 8, done0 = empty0 + kStages * 8, read0 = done0 + 16;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const l3ci_moe_gemm_args& a = p.a;

  if (threadIdx.x == 0) {
    for (int i = 0; i < kStages; ++i) {
      mbar_init(full0 + i * 8, 1);
      mbar_init(empty0 + i * 8, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(done0 + i * 8, 1);
      mbar_init(read0 + i * 8, 4);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&xmap)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&wmap)) : "memory");
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), Sh::kTmem);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_wait();
  pdl_launch_dependents();
  const uint32_t tmem = *tmem_slot;
  const int steps = (a.K + kDeep - 1) / kDeep;
  // consecutive tiles share their rows' expert: the columns run fastest
  struct Tile { int expert, rows, col; long long row0; bool valid; };
  auto tile_of = [&](int round) {
    Tile t;
    const long long id = (long long)round * gridDim.x + blockIdx.x;
    t.valid = expert_tile(a.counts, a.n_experts, kRows, id / p.col_tiles, t.expert, t.row0, t.rows) && t.row0 < a.rows;
    t.col = (int)(id % p.col_tiles) * kCols;
    return t;
  };
  bool ok = true;

  if (warp == 0) {
    // ---- producer ----
    const uint64_t policy_w = l2_evict_first_policy();
    uint64_t policy_x;
    asm volatile("createpolicy.fractional.L2::evict_last.b64 %0, 1.0;" : "=l"(policy_x));
    int fill = 0;
    for (int round = 0; ok; ++round) {
      const Tile t = tile_of(round);
      if (!t.valid) break;
      for (int k = 0; k < steps; ++k, ++fill) {
        const int s = fill % kStages;
        if (fill >= kStages && !mbar_wait_bounded(empty0 + s * 8, ((fill / kStages) - 1) & 1)) { ok = false; break; }
        if (lane == 0) {
          const uint32_t dst = ring + s * Sh::kStageBytes, bar = full0 + s * 8;
          mbar_expect_tx(bar, Sh::kStageBytes);
          tma_load_4d(dst, &xmap, bar, k * kDeep, (int)t.row0, 0, 0, policy_x);
          if (GATED) {
            tma_load_4d(dst + kXBytes, &wmap, bar, k * kDeep, t.col, 0, t.expert, policy_w);
            tma_load_4d(dst + kXBytes + Sh::kWBytes / 2, &wmap, bar, k * kDeep, t.col, 1, t.expert, policy_w);
          } else {
            tma_load_4d(dst + kXBytes, &wmap, bar, k * kDeep, t.col, 0, t.expert, policy_w);
          }
        }
        __syncwarp();
      }
    }
  } else if (warp == 1) {
    // ---- MMA issue: all lanes run the code, one elected lane predicates the instructions ----
    constexpr uint32_t idesc = instr_desc(kRows, BN, false);
    const uint32_t elected = lane == 0 ? 1u : 0u;
    int fill = 0;
    for (int round = 0; ok; ++round) {
      const Tile t = tile_of(round);
      if (!t.valid) break;
      const int acc = round & 1;
      if (round >= 2 && !mbar_wait_bounded(read0 + acc * 8, ((round >> 1) - 1) & 1)) { ok = false; break; }
      tc_fence_after();
      for (int k = 0; k < steps; ++k, ++fill) {
        const int s = fill % kStages;
        if (!mbar_wait_bounded(full0 + s * 8, (fill / kStages) & 1)) { ok = false; break; }
        tc_fence_after();
        const uint64_t xd = smem_desc(ring + s * Sh::kStageBytes, 16, 1024);
        const uint64_t wd = smem_desc(ring + s * Sh::kStageBytes + kXBytes, 16, 1024);
#pragma unroll
        for (int i = 0; i < kDeep / 16; ++i) mma_ss(tmem + acc * BN, xd + i * 2, wd + i * 2, idesc, (k > 0 || i > 0) ? 1u : 0u, elected);
        tc_commit(empty0 + s * 8, elected);
      }
      if (ok) tc_commit(done0 + acc * 8, elected);
    }
    // an accumulator that nobody waits for any more must not be freed under a running product: the output warps wait for the
    // last product of every tile, and this warp joins them at the CTA's last barrier
  } else if (warp >= 4) {
    // ---- output: thread owns row r ----
    const int q4 = warp & 3, r = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    for (int round = 0; ok; ++round) {
      const Tile t = tile_of(round);
      if (!t.valid) break;
      const int acc = round & 1;
      if (!mbar_wait_bounded(done0 + acc * 8, (round >> 1) & 1)) { ok = false; break; }
      tc_fence_after();
      const uint32_t at = tmem + acc * BN + lane_addr;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + (t.row0 + r) * a.N + t.col;
      const bool mine = r < t.rows;
#pragma unroll
      for (int c = 0; c < kCols; c += 32) {
        if (t.col + c >= a.N) break;
        uint32_t y[32], z[32];
        tmem_ld32(at + c, y);
        if (GATED) tmem_ld32(at + kCols + c, z);
        tc_wait_ld();
        if (mine) {
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            if (t.col + c + v * 8 >= a.N) break;
            float f[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              f[i] = __uint_as_float(y[v * 8 + i]);
              if (GATED) f[i] = gated_activation_fast(f[i], __uint_as_float(z[v * 8 + i]), a.limit, a.alpha);
            }
            *reinterpret_cast<uint4*>(dst + c + v * 8) = pack8(f);
          }
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(read0 + acc * 8);
    }
  }
  if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, Sh::kTmem);
}

// [rows of a matrix] x [matrices] x [experts] map: 64 columns of K by `box` rows
int make_weights_map(CUtensorMap* map, const l3ci_moe_gemm_args* a, int box) {
  const int mats = a->gated ? 2 : 1;
  const long long one = (long long)a->N * a->K;
  return make_rows_map(map, a->w, a->K, a->N, mats, a->n_experts, a->K, one, one * mats, box);
}

template <int BN, bool GATED>
int launch(const l3ci_moe_gemm_args* a, cudaStream_t stream) {
  using Sh = MoeShape<BN>;
  constexpr int kCols = GATED ? BN / 2 : BN;
  MoeTcParams p = {};
  p.a = *a;
  p.col_tiles = (a->N + kCols - 1) / kCols;
  CUtensorMap xmap, wmap;
  if (int st = make_rows_map(&xmap, a->x, a->K, (int)a->rows, 1, 1, a->K, 0, 0, kRows)) return st;
  if (int st = make_weights_map(&wmap, a, kCols)) return st;
  static bool configured[64] = {false};
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(moe_tc_kernel<BN, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::kSmem));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const long long tiles = (a->rows / kRows + (a->rows < a->n_experts ? a->rows : a->n_experts)) * p.col_tiles;
  const int sms = sm_count() > 0 ? sm_count() : 148;
  const unsigned ctas = (unsigned)(tiles < sms ? tiles : sms);
  L3CI_LAUNCH("moe_tc_kernel", moe_tc_kernel<BN, GATED>, dim3(ctas), dim3(kThreads), Sh::kSmem, stream, xmap, wmap, p);
  return L3CI_OK;
}

template <bool GATED>
int launch_any(const l3ci_moe_gemm_args* a, cudaStream_t stream) {
  // the widest tile that still gives every SM one
  const int sms = sm_count() > 0 ? sm_count() : 148;
  const long long row_tiles = a->rows / kRows + (a->rows < a->n_experts ? a->rows : a->n_experts);
  const int mats = GATED ? 2 : 1;
  auto tiles = [&](int bn) { return row_tiles * ((a->N + bn / mats - 1) / (bn / mats)); };
  if (tiles(256) >= 2LL * sms) return launch<256, GATED>(a, stream);
  if (tiles(128) >= sms) return launch<128, GATED>(a, stream);
  return launch<64, GATED>(a, stream);
}

}  // namespace

bool moe_tc_applies(const l3ci_moe_gemm_args* a) {
  return a->dtype == L3CI_BF16 && a->K % 8 == 0 && a->N % 8 == 0 && aligned16(a->x) && aligned16(a->w) && aligned16(a->out);
}

int moe_tc_launch(const l3ci_moe_gemm_args* a) {
  cudaStream_t s = reinterpret_cast<cudaStream_t>(a->stream);
  return a->gated ? launch_any<true>(a, s) : launch_any<false>(a, s);
}

}  // namespace l3ci
