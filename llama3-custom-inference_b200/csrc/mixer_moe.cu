// Mixture of experts: routing, sorting of the token rows by expert, and the plain form of the experts' products
// (mixer_moe_tc.cu has the tensor-core form).
//
// route: a warp picks a token's experts from its fp32 logits.  The place of a (token, expert) pair among its expert's pairs is
// counted in shared memory per CTA and placed with one atomic per CTA and expert.  The order of an expert's rows is whatever that gives: a row's result does not depend on its place.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "mixer_moe.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kRouteWarps = 8, kRouteWarpsMax = 32;

// Order of the floats as unsigned numbers; NaN is below every number.
__device__ __forceinline__ unsigned ordered(float z) {
  const unsigned u = __float_as_uint(z);
  return z != z ? 0u : u & 0x80000000u ? ~u : u | 0x80000000u;
}

__global__ void __launch_bounds__(32 * kRouteWarpsMax)
moe_route_kernel(const float* __restrict__ logits, const float* __restrict__ bias, int* __restrict__ experts, int* __restrict__ ranks,
                 float* __restrict__ weights, int* __restrict__ counts, long long rows, int tokens, int E, int top) {
  extern __shared__ float sh[];
  const int warps = blockDim.x / kWarp;
  float* row = sh;                                                // [warps][E]
  int* count = reinterpret_cast<int*>(row + warps * E);           // [E], then the expert's first rank of this CTA
  int* chosen = count + E;                                        // [tokens][top]
  int* place = chosen + tokens * top;                             // [tokens][top]
  float* weight = reinterpret_cast<float*>(place + tokens * top);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int e = tid; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const long long row0 = (long long)blockIdx.x * tokens;
  const int n = (int)min((long long)tokens, rows - row0);
  float* z = row + warp * E;
  for (int t = warp; t < n; t += warps) {
    for (int e = lane; e < E; e += 32) z[e] = logits[(row0 + t) * E + e] + bias[e];
    __syncwarp();
    float first = 0.f, sum = 0.f;
    for (int j = 0; j < top; ++j) {
      // the lane's largest logit that is not taken (taken ones are NaN), then the warp's; ties: the smaller index
      unsigned best = 0u;
      int at = E;
      for (int e = lane; e < E; e += 32) {
        const unsigned o = ordered(z[e]);
        if (o > best) { best = o; at = e; }
      }
      const unsigned most = __reduce_max_sync(kFullMask, best);
      at = __reduce_min_sync(kFullMask, best == most ? at : E);
      if (at >= E) at = j;                                        // nothing but NaN left: any place within bounds
      const float v = z[at];
      if (j == 0) first = v;
      const float p = expf(v - first);
      sum += p;
      __syncwarp();
      if (lane == 0) {
        z[at] = __int_as_float(0x7fffffff);
        chosen[t * top + j] = at;
        place[t * top + j] = atomicAdd(count + at, 1);
        weight[t * top + j] = p;
      }
      __syncwarp();
    }
    for (int j = lane; j < top; j += 32) weights[(row0 + t) * top + j] = weight[t * top + j] / sum;
  }
  __syncthreads();
  if (gridDim.x == 1) {                                           // these are all the tokens there are
    for (int e = tid; e < E; e += blockDim.x) {
      counts[e] = count[e];
      count[e] = 0;
    }
  } else {
    for (int e = tid; e < E; e += blockDim.x)
      if (count[e] > 0) count[e] = atomicAdd(counts + e, count[e]);
  }
  __syncthreads();
  for (int i = tid; i < n * top; i += blockDim.x) {
    experts[row0 * top + i] = chosen[i];
    ranks[row0 * top + i] = count[chosen[i]] + place[i];
  }
}

// A CTA per token: its row to the places of its pairs.
template <typename S, int VEC>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const S* __restrict__ h, const int* __restrict__ experts, const int* __restrict__ ranks, const int* __restrict__ counts,
                  S* __restrict__ out, int* __restrict__ part_rows, long long rows, int width, int E, int top) {
  extern __shared__ int at_s[];
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x / kWarp;
  for (int j = warp; j < top; j += warps) {
    const int e = experts[row * top + j];
    int before = 0;
    for (int i = lane; i < e; i += 32) before += counts[i];
    before = __reduce_add_sync(kFullMask, before);
    if (lane == 0) {
      const int at = before + ranks[row * top + j];
      part_rows[row * top + j] = at;
      at_s[j] = at;
    }
  }
  __syncthreads();
  using R = typename Raw<VEC * sizeof(S)>::type;
  for (int c = tid * VEC; c < width; c += blockDim.x * VEC) {
    const R x = *reinterpret_cast<const R*>(h + row * width + c);
    for (int j = 0; j < top; ++j) {
      const long long at = at_s[j];
      if (at >= 0 && at < rows * top) *reinterpret_cast<R*>(out + at * width + c) = x;
    }
  }
}

// ---- plain products: 64 x 64 tiles, 16 deep, fp32 -----------------------------------------------------------------
constexpr int kTile = 64, kDeep = 16;

template <typename S, bool GATED>
__global__ void __launch_bounds__(256) moe_plain_kernel(const l3ci_moe_gemm_args a) {
  constexpr int kMats = GATED ? 2 : 1;
  __shared__ float xs[kDeep][kTile + 4];
  __shared__ float ws[kMats][kDeep][kTile + 4];
  pdl_wait();
  pdl_launch_dependents();
  int expert, rows;
  long long row0;
  if (!expert_tile(a.counts, a.n_experts, kTile, blockIdx.x, expert, row0, rows)) return;
  const int n0 = blockIdx.y * kTile, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const S* x = static_cast<const S*>(a.x);
  const S* w = static_cast<const S*>(a.w) + (long long)expert * kMats * a.N * a.K;
  float acc[kMats][4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += kDeep) {
    __syncthreads();
    for (int i = tid; i < kTile * kDeep; i += 256) {
      const int r = i / kDeep, k = i % kDeep;
      xs[k][r] = r < rows && k0 + k < a.K && row0 + r < a.rows ? to_f32(x[(row0 + r) * a.K + k0 + k]) : 0.f;
#pragma unroll
      for (int m = 0; m < kMats; ++m)
        ws[m][k][r] = n0 + r < a.N && k0 + k < a.K ? to_f32(w[((long long)m * a.N + n0 + r) * a.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kDeep; ++k) {
      float xv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) xv[i] = xs[k][ty * 4 + i];
#pragma unroll
      for (int m = 0; m < kMats; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float wv = ws[m][k][tx + 16 * j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[m][i][j] = fmaf(xv[i], wv, acc[m][i][j]);
        }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = ty * 4 + i, c = n0 + tx + 16 * j;
      if (r >= rows || c >= a.N || row0 + r >= a.rows) continue;
      const float y = GATED ? gated_activation(acc[0][i][j], acc[kMats - 1][i][j], a.limit, a.alpha) : acc[0][i][j];
      static_cast<S*>(a.out)[(row0 + r) * a.N + c] = from_f32<S>(y);
    }
}

int validate(const l3ci_moe_gemm_args* a) {
  if (!a) return fail(L3CI_ERR_INVALID, "moe_gemm: null args");
  if (a->rows < 0 || a->rows > 0x7fffffffLL || a->K <= 0 || a->N <= 0 || a->n_experts <= 0 || a->n_experts > kMaxExperts ||
      (a->dtype != L3CI_BF16 && a->dtype != L3CI_F32) || a->variant < 0 || a->variant > 2 || !(a->limit >= 0.f))
    return fail(L3CI_ERR_INVALID, "moe_gemm: rows=%lld K=%d N=%d experts=%d dtype=%d", (long long)a->rows, a->K, a->N, a->n_experts, a->dtype);
  if (a->rows > 0 && (!a->x || !a->w || !a->out || !a->counts)) return fail(L3CI_ERR_INVALID, "moe_gemm: null pointer");
  return L3CI_OK;
}

int choose(const l3ci_moe_gemm_args* a) {
  if (a->variant == 1) return 1;
  const bool tc = moe_tc_applies(a);
  if (a->variant == 2) return tc ? 2 : -1;
  return tc ? 2 : 1;
}

}  // namespace
}  // namespace l3ci

extern "C" {

int l3ci_moe_route(const float* logits, const float* bias, int32_t* experts, int32_t* ranks, float* weights, int32_t* counts, int64_t rows,
                   int32_t E, int32_t top, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (rows < 0 || rows > 0x7fffffffLL / 8 || E <= 0 || E > kMaxExperts || top <= 0 || top > E || rows * top > 0x7fffffffLL)
    return fail(L3CI_ERR_INVALID, "moe_route: rows=%lld experts=%d top=%d", (long long)rows, E, top);
  if (!counts) return fail(L3CI_ERR_INVALID, "moe_route: null pointer");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  if (rows == 0) {
    L3CI_CUDA_TRY(cudaMemsetAsync(counts, 0, sizeof(int32_t) * E, s));
    return L3CI_OK;
  }
  if (!logits || !bias || !experts || !ranks || !weights) return fail(L3CI_ERR_INVALID, "moe_route: null pointer");
  // few tokens: one CTA, which needs no counting across CTAs
  const int sms = sm_count() > 0 ? sm_count() : 148;
  auto bytes = [&](int warps, int n) { return sizeof(float) * ((size_t)warps * E + E + 3 * (size_t)n * top); };
  int warps = (int)(rows < kRouteWarpsMax ? rows : kRouteWarpsMax), tokens = (int)(rows < 4 * kRouteWarpsMax ? rows : 4 * kRouteWarpsMax);
  if (rows > tokens || bytes(warps, tokens) > (48 << 10)) {
    warps = kRouteWarps;
    tokens = rows >= 16LL * sms ? 4 * kRouteWarps : kRouteWarps;
    while (tokens > 1 && bytes(warps, tokens) > (48 << 10)) tokens /= 2;
    if (bytes(warps, tokens) > (48 << 10)) return fail(L3CI_ERR_UNSUPPORTED, "moe_route: experts=%d top=%d", E, top);
  }
  if (rows > tokens) L3CI_CUDA_TRY(cudaMemsetAsync(counts, 0, sizeof(int32_t) * E, s));
  L3CI_LAUNCH("moe_route_kernel", moe_route_kernel, dim3((unsigned)((rows + tokens - 1) / tokens)), dim3(32 * warps), bytes(warps, tokens), s, logits,
              bias, experts, ranks, weights, counts, (long long)rows, tokens, E, top);
  return L3CI_OK;
}

int l3ci_moe_gather(const void* h, const int32_t* experts, const int32_t* ranks, const int32_t* counts, void* out, int32_t* part_rows,
                    int64_t rows, int64_t width, int32_t E, int32_t top, int32_t dtype, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (rows < 0 || rows > 0x7fffffffLL || width <= 0 || width > 0x3fffffffLL || E <= 0 || E > kMaxExperts || top <= 0 || top > E ||
      rows * top > 0x7fffffffLL || (dtype != L3CI_BF16 && dtype != L3CI_F32))
    return fail(L3CI_ERR_INVALID, "moe_gather: rows=%lld width=%lld experts=%d top=%d", (long long)rows, (long long)width, E, top);
  if (rows == 0) return L3CI_OK;
  if (!h || !experts || !ranks || !counts || !out || !part_rows) return fail(L3CI_ERR_INVALID, "moe_gather: null pointer");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    constexpr int kVec = 16 / sizeof(S);
    const bool v = width % kVec == 0 && aligned16(h) && aligned16(out);
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("moe_gather_kernel", kernel, dim3((unsigned)rows), dim3(128), sizeof(int) * top, s, static_cast<const S*>(h), experts, ranks, counts,
                  static_cast<S*>(out), part_rows, (long long)rows, (int)width, E, top);
      return L3CI_OK;
    };
    return v ? go(moe_gather_kernel<S, kVec>) : go(moe_gather_kernel<S, 1>);
  };
  return dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

int l3ci_moe_gemm_variant(const l3ci_moe_gemm_args* a) {
  using namespace l3ci;
  clear_error();
  return validate(a) == L3CI_OK ? choose(a) : -1;
}

int l3ci_moe_gemm(const l3ci_moe_gemm_args* a) {
  using namespace l3ci;
  clear_error();
  if (int st = validate(a)) return st;
  if (a->rows == 0) return L3CI_OK;
  const int v = choose(a);
  if (v < 0) return fail(L3CI_ERR_UNSUPPORTED, "moe_gemm: variant %d does not take these sizes", a->variant);
  if (v == 2) return moe_tc_launch(a);
  // at most one tile of every expert is not full
  const long long tiles = a->rows / kTile + (a->rows < a->n_experts ? a->rows : a->n_experts);
  if (tiles > 0x7fffffffLL || (a->N + kTile - 1) / kTile > 65535) return fail(L3CI_ERR_UNSUPPORTED, "moe_gemm: N=%d", a->N);
  const dim3 grid((unsigned)tiles, (unsigned)((a->N + kTile - 1) / kTile));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(a->stream);
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("moe_plain_kernel", kernel, grid, dim3(256), 0, s, *a);
    return L3CI_OK;
  };
  if (a->dtype == L3CI_BF16) return a->gated ? go(moe_plain_kernel<__nv_bfloat16, true>) : go(moe_plain_kernel<__nv_bfloat16, false>);
  return a->gated ? go(moe_plain_kernel<float, true>) : go(moe_plain_kernel<float, false>);
}

}  // extern "C"
