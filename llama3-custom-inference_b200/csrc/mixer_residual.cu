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
constexpr int kManyVpt = 2;    // vectors of a thread when there are many rows
constexpr int kPartsAhead = 4;

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

// Y: type of y.
template <typename S, typename Y, int VEC, int VPT>
__global__ void __launch_bounds__(512) residual_norm_kernel(const l3ci_residual_norm_args a) {
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
      const Y* ys = static_cast<const Y*>(a.y);
      if (a.parts == 1 && !a.part_rows) {
        const float w = a.part_weights ? a.part_weights[row] : 1.f;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
          if (i >= chunks) break;
          float f[VEC];
          load_vec<Y, VEC>(ys + row * width + col[i], f);
#pragma unroll
          for (int k = 0; k < VEC; ++k) y[i * VEC + k] = w * f[k];
        }
      } else {
        for (int p0 = 0; p0 < a.parts; p0 += kPartsAhead) {      // several parts' rows in flight
          long long at[kPartsAhead];
          float w[kPartsAhead];
#pragma unroll
          for (int p = 0; p < kPartsAhead; ++p) {
            const long long id = row * a.parts + min(p0 + p, a.parts - 1);
            at[p] = (a.part_rows ? a.part_rows[id] : id) * (long long)width;
            w[p] = p0 + p >= a.parts ? 0.f : a.part_weights ? a.part_weights[id] : 1.f;
          }
#pragma unroll
          for (int i = 0; i < VPT; ++i) {
            if (i >= chunks) break;
            using R = typename Raw<VEC * sizeof(Y)>::type;
            R raw[kPartsAhead];
#pragma unroll
            for (int p = 0; p < kPartsAhead; ++p) raw[p] = *reinterpret_cast<const R*>(ys + at[p] + col[i]);
#pragma unroll
            for (int p = 0; p < kPartsAhead; ++p) {
              if (p0 + p >= a.parts) break;
              float f[VEC];
              load_vec<Y, VEC>(reinterpret_cast<const Y*>(&raw[p]), f);
#pragma unroll
              for (int k = 0; k < VEC; ++k) y[i * VEC + k] = fmaf(w[p], f[k], y[i * VEC + k]);
            }
          }
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

template <typename S, typename Y>
int residual_norm_typed(const l3ci_residual_norm_args* a) {
  constexpr int kVec = 8;
  auto ok = [](const void* p) { return aligned16(p); };
  const bool vec = a->width % kVec == 0 && ok(a->x) && ok(a->y) && ok(a->post_w) && ok(a->post_b) && ok(a->step) && ok(a->pre_w) && ok(a->pre_b) &&
                   ok(a->out) && a->out_stride % kVec == 0 && ok(a->table) && ok(a->x0) && a->x0_stride % kVec == 0;
  const long long units = vec ? a->width / kVec : a->width;
  // few rows: as many threads as there are vectors; many rows: few threads with many vectors each, so that little of the work
  // is reductions and many rows are on an SM
  const bool many = a->rows > 4LL * (sm_count() > 0 ? sm_count() : 148);
  int threads = 32, vpt = 1;
  while ((many && vec ? kManyVpt : 1) * threads < units && threads < 512) threads *= 2;
  while ((long long)vpt * threads < units) vpt *= 2;
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("residual_norm_kernel", kernel, dim3((unsigned)a->rows), dim3(threads), 0, reinterpret_cast<cudaStream_t>(a->stream), *a);
    return L3CI_OK;
  };
  if (vec) {
    switch (vpt) {
      case 1: return go(residual_norm_kernel<S, Y, kVec, 1>);
      case 2: return go(residual_norm_kernel<S, Y, kVec, 2>);
      case 4: return go(residual_norm_kernel<S, Y, kVec, 4>);
    }
  } else {
    switch (vpt) {
      case 1: return go(residual_norm_kernel<S, Y, 1, 1>);
      case 2: return go(residual_norm_kernel<S, Y, 1, 2>);
      case 4: return go(residual_norm_kernel<S, Y, 1, 4>);
      case 8: return go(residual_norm_kernel<S, Y, 1, 8>);
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
  const bool y32 = a->y && a->y_dtype == L3CI_F32;
  if (a->dtype == L3CI_F32) return y32 || !a->y ? residual_norm_typed<float, float>(a) : residual_norm_typed<float, __nv_bfloat16>(a);
  return y32 ? residual_norm_typed<__nv_bfloat16, float>(a) : residual_norm_typed<__nv_bfloat16, __nv_bfloat16>(a);
}
