// The step between two sublayers of a decoder with a 32-bit residual stream and a norm on both sides of a sublayer, in one
// pass over a row:
//
//   y  = sum over the parts of (part weight *) y_part          (the combination of a token's experts)
//   x  = x + layer_norm(y)  |  y + step  |  table[token] * scale + sinusoid(position)
//   out = layer_norm(x)     |  x
//
// A CTA takes a row and keeps it in registers from the first load to the last store.  A layer norm's statistics are formed
// per warp in two passes (mean, then squared deviations from it) and merged over the warps by their counts, so that each
// norm costs one barrier and nothing is lost to cancellation.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "../../include/l3ci_mixers.h"
#include "host_common.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kMaxWarps = 16;
constexpr int kManyVpt = 8;    // vectors of a thread when there are many rows

// Mean and 1 / sqrt(variance + eps) of a row of `width` values; the thread's values are the first `valid` of v.
template <int N>
__device__ __forceinline__ void row_stats(const float (&v)[N], int valid, int width, float eps, float (*sm)[3], float& mean, float& inv) {
  const int warps = blockDim.x / kWarp, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i)
    if (i < valid) s += v[i];
  const float cnt = warps > 1 ? (float)__reduce_add_sync(kFullMask, valid) : (float)width;
  mean = cnt > 0.f ? group_sum<kWarp>(s) / cnt : 0.f;
  float m2 = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i)
    if (i < valid) m2 = fmaf(v[i] - mean, v[i] - mean, m2);
  m2 = group_sum<kWarp>(m2);
  if (warps > 1) {
    if (lane == 0) {
      sm[warp][0] = mean;
      sm[warp][1] = m2;
      sm[warp][2] = cnt;
    }
    __syncthreads();
    const float wm = lane < warps ? sm[lane][0] : 0.f, wm2 = lane < warps ? sm[lane][1] : 0.f, wc = lane < warps ? sm[lane][2] : 0.f;
    mean = group_sum<kWarp>(wm * wc) / (float)width;
    m2 = group_sum<kWarp>(fmaf(wc * (wm - mean), wm - mean, wm2));
  }
  inv = 1.f / sqrtf(m2 / (float)width + eps);
}

// sin or cos of p * freq, the product and its reduction to one turn in double
__device__ __forceinline__ float sinusoid(int p, double freq, bool cosine) {
  const double turns = (double)p * freq * 0.15915494309189533577;
  const float angle = (float)((turns - rint(turns)) * 6.283185307179586477);
  return cosine ? cosf(angle) : sinf(angle);
}

template <typename S, int VEC, int VPT>
__global__ void __launch_bounds__(VPT >= 16 ? 256 : 512) residual_norm_kernel(const l3ci_residual_norm_args a) {
  __shared__ float sm[2][kMaxWarps][3];
  const int tid = threadIdx.x, width = (int)a.width;
  int col[VPT], chunks = 0;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    col[i] = (i * (int)blockDim.x + tid) * VEC;
    if (col[i] < width) chunks = i + 1;
  }
  const int valid = chunks * VEC;
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  float* xr = a.x + row * width;
  float x[VPT * VEC], y[VPT * VEC];
#pragma unroll
  for (int i = 0; i < VPT * VEC; ++i) x[i] = y[i] = 0.f;
  if (a.tokens) {
    const long long tok = a.tokens[row];
    const S* src = tok >= 0 && tok < a.vocab ? static_cast<const S*>(a.table) + tok * width : nullptr;
    const int pos = a.positions[row / a.T] + (int)(row % a.T);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      if (i >= chunks) break;
      float f[VEC] = {};
      if (src) load_vec<S, VEC>(src + col[i], f);
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        float v = f[k] * a.embed_scale;
        if (a.freqs) v += sinusoid(pos, a.freqs[(col[i] + k) / 2], (col[i] + k) % 2);
        x[i * VEC + k] = f[k] = v;
      }
      if (a.x0) store_vec<S, VEC>(static_cast<S*>(a.x0) + row * a.x0_stride + col[i], f);
      store_vec<float, VEC>(xr + col[i], f);
    }
  } else {
    if (!a.reset) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if (i >= chunks) break;
        float f[VEC];
        load_vec<float, VEC>(xr + col[i], f);
#pragma unroll
        for (int k = 0; k < VEC; ++k) x[i * VEC + k] = f[k];
      }
    }
    if (a.y) {
      for (int p = 0; p < a.parts; ++p) {
        const float w = a.part_weights ? a.part_weights[row * a.parts + p] : 1.f;
        const long long at = (a.part_rows ? a.part_rows[row * a.parts + p] : row * a.parts + p) * (long long)width;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          if (i >= chunks) break;
          float f[VEC];
          if (a.y_dtype == L3CI_F32) load_vec<float, VEC>(static_cast<const float*>(a.y) + at + col[i], f);
          else load_vec<__nv_bfloat16, VEC>(static_cast<const __nv_bfloat16*>(a.y) + at + col[i], f);
#pragma unroll
          for (int k = 0; k < VEC; ++k) y[i * VEC + k] = fmaf(w, f[k], y[i * VEC + k]);
        }
      }
      if (a.post_w) {
        float mean, inv;
        row_stats(y, valid, width, a.eps, sm[0], mean, inv);
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          if (i >= chunks) break;
          float w[VEC], b[VEC];
          load_vec<float, VEC>(a.post_w + col[i], w);
          load_vec<float, VEC>(a.post_b + col[i], b);
#pragma unroll
          for (int k = 0; k < VEC; ++k) y[i * VEC + k] = fmaf((y[i * VEC + k] - mean) * inv, w[k], b[k]);
        }
      }
#pragma unroll
      for (int i = 0; i < VPT * VEC; ++i) x[i] += y[i];
    }
    if (a.step) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if (i >= chunks) break;
        float f[VEC];
        load_vec<float, VEC>(a.step + col[i], f);
#pragma unroll
        for (int k = 0; k < VEC; ++k) x[i * VEC + k] += f[k];
      }
    }
    if (a.y || a.step) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        if (i >= chunks) break;
        float f[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) f[k] = x[i * VEC + k];
        store_vec<float, VEC>(xr + col[i], f);
      }
    }
  }
  if (!a.out) return;
  S* out = static_cast<S*>(a.out) + row * a.out_stride;
  float mean = 0.f, inv = 1.f;
  if (a.pre_w) row_stats(x, valid, width, a.eps, sm[1], mean, inv);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if (i >= chunks) break;
    float f[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) f[k] = x[i * VEC + k];
    if (a.pre_w) {
      float w[VEC], b[VEC];
      load_vec<float, VEC>(a.pre_w + col[i], w);
      load_vec<float, VEC>(a.pre_b + col[i], b);
#pragma unroll
      for (int k = 0; k < VEC; ++k) f[k] = fmaf((f[k] - mean) * inv, w[k], b[k]);
    }
    store_vec<S, VEC>(out + col[i], f);
  }
}

template <typename S>
int residual_norm_typed(const l3ci_residual_norm_args* a) {
  auto ok = [](const void* p, int bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; };
  const int s4 = 4 * (int)sizeof(S);
  const bool v4 = a->width % 4 == 0 && ok(a->x, 16) && ok(a->y, a->y_dtype == L3CI_F32 ? 16 : 8) && ok(a->post_w, 16) && ok(a->post_b, 16) &&
                  ok(a->step, 16) && ok(a->pre_w, 16) && ok(a->pre_b, 16) && ok(a->out, s4) && a->out_stride % 4 == 0 && ok(a->table, s4) &&
                  ok(a->x0, s4) && a->x0_stride % 4 == 0;
  const long long units = v4 ? a->width / 4 : a->width;
  // few rows: as many threads as there are vectors; many rows: few threads with many vectors each, so that little of the work
  // is reductions and many rows are on an SM
  const bool many = a->rows > 4LL * (sm_count() > 0 ? sm_count() : 148);
  int threads = 32, vpt = 1;
  while ((many && v4 ? kManyVpt : 1) * threads < units && threads < 512) threads *= 2;
  while ((long long)vpt * threads < units) vpt *= 2;
  if (threads > (vpt >= 16 ? 256 : 512)) return fail(L3CI_ERR_UNSUPPORTED, "residual_norm: width %lld", (long long)a->width);
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("residual_norm_kernel", kernel, dim3((unsigned)a->rows), dim3(threads), 0, reinterpret_cast<cudaStream_t>(a->stream), *a);
    return L3CI_OK;
  };
  if (v4) {
    switch (vpt) {
      case 1: return go(residual_norm_kernel<S, 4, 1>);
      case 2: return go(residual_norm_kernel<S, 4, 2>);
      case 4: return go(residual_norm_kernel<S, 4, 4>);
      case 8: return go(residual_norm_kernel<S, 4, 8>);
      case 16: return go(residual_norm_kernel<S, 4, 16>);
    }
  } else {
    switch (vpt) {
      case 1: return go(residual_norm_kernel<S, 1, 1>);
      case 2: return go(residual_norm_kernel<S, 1, 2>);
      case 4: return go(residual_norm_kernel<S, 1, 4>);
      case 8: return go(residual_norm_kernel<S, 1, 8>);
    }
  }
  return fail(L3CI_ERR_UNSUPPORTED, "residual_norm: width %lld", (long long)a->width);
}

}  // namespace
}  // namespace l3ci

extern "C" int l3ci_residual_norm(const l3ci_residual_norm_args* a) {
  using namespace l3ci;
  clear_error();
  if (!a) return fail(L3CI_ERR_INVALID, "residual_norm: null args");
  if (a->rows < 0 || a->rows > 0x7fffffffLL || a->width <= 0 || a->width > 0x7fffffffLL || (a->dtype != L3CI_BF16 && a->dtype != L3CI_F32) ||
      (a->y && (a->parts <= 0 || (a->y_dtype != L3CI_BF16 && a->y_dtype != L3CI_F32))) || (a->out && a->out_stride < a->width) ||
      (a->x0 && a->x0_stride < a->width))
    return fail(L3CI_ERR_INVALID, "residual_norm: rows=%lld width=%lld parts=%d dtype=%d", (long long)a->rows, (long long)a->width, a->parts, a->dtype);
  if (a->rows == 0) return L3CI_OK;
  if (!a->x || (!a->post_w) != (!a->post_b) || (!a->pre_w) != (!a->pre_b) || (a->reset && !a->y) ||
      (a->tokens && (!a->table || !a->positions || a->T <= 0 || a->vocab <= 0 || a->y)))
    return fail(L3CI_ERR_INVALID, "residual_norm: null pointer, or both y and tokens");
  return a->dtype == L3CI_BF16 ? residual_norm_typed<__nv_bfloat16>(a) : residual_norm_typed<float>(a);
}
