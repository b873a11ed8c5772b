// Shared by the mixture-of-experts kernels.
#pragma once

#include "../../include/l3ci_mixers.h"
#include "host_common.h"

namespace l3ci {

constexpr int kMaxExperts = 1024;

// tcgen05, 128 sorted rows per tile (mixer_moe_tc.cu).
bool moe_tc_applies(const l3ci_moe_gemm_args* a);
int moe_tc_launch(const l3ci_moe_gemm_args* a);

#if defined(__CUDACC__)
// Row tiles of the experts' runs of sorted rows: the expert of tile `tile` (tiles of `tile_rows` rows, expert by expert), its
// first row and how many rows of the expert it has.  Called by a whole warp; false: there is no such tile.
__device__ __forceinline__ bool expert_tile(const int* counts, int n_experts, int tile_rows, long long tile, int& expert, long long& row0, int& rows) {
  const int lane = threadIdx.x & 31;
  long long tiles_before = 0, rows_before = 0;
  for (int e0 = 0; e0 < n_experts; e0 += 32) {
    const int c = e0 + lane < n_experts ? counts[e0 + lane] : 0;
    int tiles = (c + tile_rows - 1) / tile_rows, t = tiles, r = c;   // inclusive sums over the 32 experts
#pragma unroll
    for (int m = 1; m < 32; m *= 2) {
      const int u = __shfl_up_sync(0xffffffffu, t, m), v = __shfl_up_sync(0xffffffffu, r, m);
      if (lane >= m) { t += u; r += v; }
    }
    const unsigned hit = __ballot_sync(0xffffffffu, tile < tiles_before + t);
    if (hit) {
      const int who = __ffs(hit) - 1;
      const int first = (int)(tile - (tiles_before + __shfl_sync(0xffffffffu, t - tiles, who)));
      const int cnt = __shfl_sync(0xffffffffu, c, who);
      expert = e0 + who;
      row0 = rows_before + __shfl_sync(0xffffffffu, r - c, who) + (long long)first * tile_rows;
      rows = min(tile_rows, cnt - first * tile_rows);
      return true;
    }
    tiles_before += __shfl_sync(0xffffffffu, t, 31);
    rows_before += __shfl_sync(0xffffffffu, r, 31);
  }
  return false;
}
#endif

}  // namespace l3ci
