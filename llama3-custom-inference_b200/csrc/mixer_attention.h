// Shared by the mixer attention kernels: the launchers behind l3ci_mixer_attention and the per-query score constants.
#pragma once

#include "../../include/l3ci_mixers.h"
#include "host_common.h"

namespace l3ci {

// Key tiles of 64, 8 warps, keys split over CTAs (mixer_attention_mma.cu).
bool mixer_mma_applies(const l3ci_mixer_attn_args* a);
size_t mixer_mma_scratch_bytes(const l3ci_mixer_attn_args* a);
int mixer_mma_launch(const l3ci_mixer_attn_args* a);

// tcgen05, 128 query rows per CTA (mixer_attention_tc.cu).
bool mixer_tc_applies(const l3ci_mixer_attn_args* a);
size_t mixer_tc_scratch_bytes(const l3ci_mixer_attn_args* a);
int mixer_tc_launch(const l3ci_mixer_attn_args* a);

#if defined(__CUDACC__)
// 1 + coef * ln(floor((p + 1) / every) + 1); `every` 0 means no temperature.
__device__ __forceinline__ float query_temperature(int p, float coef, float every) {
  return every > 0.f ? fmaf(coef, logf(floorf(__fdiv_rn((float)(p + 1), every)) + 1.f), 1.f) : 1.f;
}
// First key of position p's window (0: no window).
__device__ __forceinline__ int window_start(int p, int window) { return window > 0 ? max(0, p - window + 1) : 0; }
// 2^(-range (h + 1) / H): what a head takes off a score per position of distance; range 0: nothing.
__device__ __forceinline__ float head_slope(float range, int h, int H) {
  return range > 0.f ? exp2f(-range * (float)(h + 1) / (float)H) : 0.f;
}
#endif

}  // namespace l3ci
