// Causal attention over cached keys and values for the mixers (include/l3ci_mixers.h): the choice between the
// kernels, and the plain one that takes any size and both storage types.
//
// mixer_rows_kernel: a CTA per query (token, head, sequence), both maps of a differential head in one pass over the
// values.  Keys in blocks of 128: a thread takes a key's dot product in fp32, the block's maximum moves the running
// one, then every thread folds the block into its own value columns.  It is the path of 32-bit models and of sizes
// the tensor-core kernels cannot address (rows that do not start on 16 bytes).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "mixer_attention.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kRowThreads = 128;
constexpr int kRowCols = 8;  // value columns per thread

__device__ __forceinline__ float cta_max(float v, float* smem) {
  v = group_max<kWarp>(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __syncthreads();
  if (lane == 0) smem[warp] = v;
  __syncthreads();
  return fmaxf(fmaxf(smem[0], smem[1]), fmaxf(smem[2], smem[3]));
}

template <typename S, int MAPS>
__global__ void __launch_bounds__(kRowThreads) mixer_rows_kernel(const l3ci_mixer_attn_args a) {
  extern __shared__ float sh[];
  __shared__ float red[32];
  __shared__ float pk[MAPS][kRowThreads];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (a.H / a.G), tid = threadIdx.x;
  const int pos = a.positions[b] + t;
  // the keys in sight: the first `kept` ones, then those from `lo` on
  const int lo = window_start(pos, a.window), kept = min(a.keep_first, lo);
  const int keys = kept + max(0, min(pos + 1, a.n_keys) - lo);
  const float slope = head_slope(a.bias_range, h, a.H);
  float* qs = sh;  // [MAPS][Da + Db]
  const int dk = a.Da + a.Db;
  const S* qa = static_cast<const S*>(a.qa) + b * a.qa_sb + t * a.qa_st + h * a.qa_sh;
  const S* qb = static_cast<const S*>(a.qb) + b * a.qb_sb + t * a.qb_st + h * a.qb_sh;
  for (int i = tid; i < MAPS * dk; i += kRowThreads) {
    const int m = i / dk, d = i % dk;
    qs[i] = to_f32(d < a.Da ? qa[m * a.Da + d] : qb[d - a.Da]);
  }
  __syncthreads();
  const float scale = a.scale * query_temperature(pos, a.temp_coef, a.temp_every);
  const S* ka = static_cast<const S*>(a.ka) + b * a.ka_sb + g * a.ka_sh;
  const S* kb = static_cast<const S*>(a.kb) + b * a.kb_sb + g * a.kb_sh;
  const S* v = static_cast<const S*>(a.v) + b * a.v_sb + g * a.v_sh;
  float acc[MAPS][kRowCols], m_run[MAPS], l_run[MAPS];
#pragma unroll
  for (int m = 0; m < MAPS; ++m) {
    m_run[m] = a.sink ? 0.f : -INFINITY;
    l_run[m] = a.sink ? 1.f : 0.f;
#pragma unroll
    for (int c = 0; c < kRowCols; ++c) acc[m][c] = 0.f;
  }
  for (int j0 = 0; j0 < keys; j0 += kRowThreads) {
    const bool seen = j0 + tid < keys;
    const int j = j0 + tid < kept ? j0 + tid : lo + j0 + tid - kept;
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
      float s = -INFINITY;
      if (seen) {
        const S* kr = ka + j * a.ka_st + m * a.Da;
        s = 0.f;
        for (int d = 0; d < a.Da; ++d) s = fmaf(qs[m * dk + d], to_f32(kr[d]), s);
        const S* kr2 = kb + j * a.kb_st;
        for (int d = 0; d < a.Db; ++d) s = fmaf(qs[m * dk + a.Da + d], to_f32(kr2[d]), s);
        s *= scale;
        if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
        s -= slope * (float)(pos - j);
      }
      const float mx = fmaxf(m_run[m], cta_max(s, red));
      const float p = seen ? expf(s - mx) : 0.f;
      const float alpha = m_run[m] == -INFINITY ? 0.f : expf(m_run[m] - mx);
      m_run[m] = mx;
      l_run[m] = fmaf(l_run[m], alpha, cta_sum(p, red, kRowThreads / kWarp));
      pk[m][tid] = p;
#pragma unroll
      for (int c = 0; c < kRowCols; ++c) acc[m][c] *= alpha;
    }
    __syncthreads();
    const int n = min(kRowThreads, keys - j0);
#pragma unroll
    for (int c = 0; c < kRowCols; ++c) {
      const int col = tid + c * kRowThreads;
      if (col >= a.Dv) continue;
      for (int i = 0; i < n; ++i) {
        const int at = j0 + i < kept ? j0 + i : lo + j0 + i - kept;
        const float x = to_f32(v[at * a.v_st + col]);
#pragma unroll
        for (int m = 0; m < MAPS; ++m) acc[m][c] = fmaf(pk[m][i], x, acc[m][c]);
      }
    }
    __syncthreads();
  }
  S* o = static_cast<S*>(a.out) + b * a.o_sb + t * a.o_st + h * a.o_sh;
  float post = 1.f, ss = 0.f;
#pragma unroll
  for (int c = 0; c < kRowCols; ++c) {
    acc[0][c] = l_run[0] > 0.f ? acc[0][c] / l_run[0] : 0.f;
    if (MAPS == 2) acc[0][c] -= l_run[MAPS - 1] > 0.f ? a.lambda * (acc[MAPS - 1][c] / l_run[MAPS - 1]) : 0.f;
    ss = fmaf(acc[0][c], acc[0][c], ss);
  }
  if (MAPS == 2) {
    ss = cta_sum(ss, red, kRowThreads / kWarp);
    post = a.post * __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)a.Dv), a.eps));
    if (a.gate) {
      const float z = to_f32(static_cast<const S*>(a.gate)[b * a.g_sb + t * a.g_st + h]);
      post *= 1.f / (1.f + expf(-z));
    }
  }
#pragma unroll
  for (int c = 0; c < kRowCols; ++c) {
    const int col = tid + c * kRowThreads;
    if (col < a.Dv) o[col] = from_f32<S>(acc[0][c] * post);
  }
}

template <typename S, int MAPS>
int launch_rows(const l3ci_mixer_attn_args* a) {
  const size_t smem = (size_t)MAPS * (a->Da + a->Db) * sizeof(float);
  L3CI_LAUNCH("mixer_rows_kernel", mixer_rows_kernel<S, MAPS>, dim3((unsigned)a->T, (unsigned)a->H, (unsigned)a->B), dim3(kRowThreads),
              smem, reinterpret_cast<cudaStream_t>(a->stream), *a);
  return L3CI_OK;
}

int validate(const l3ci_mixer_attn_args* a) {
  if (!a) return fail(L3CI_ERR_INVALID, "mixer_attention: null args");
  if (a->B < 0 || a->T < 0 || a->H <= 0 || a->G <= 0 || a->H % a->G || (a->maps != 1 && a->maps != 2) || a->Da <= 0 || a->Db < 0 ||
      a->Dv <= 0 || a->n_keys < 0 || (a->dtype != L3CI_BF16 && a->dtype != L3CI_F32) || a->variant < 0 || a->variant > 3)
    return fail(L3CI_ERR_INVALID, "mixer_attention: bad size B=%d T=%d H=%d G=%d maps=%d Da=%d Db=%d Dv=%d", a->B, a->T, a->H, a->G,
                a->maps, a->Da, a->Db, a->Dv);
  if (a->window < 0 || a->keep_first < 0 || !(a->bias_range >= 0.f)) return fail(L3CI_ERR_INVALID, "mixer_attention: window=%d keep_first=%d", a->window, a->keep_first);
  if (a->maps == 2 && (a->window || a->sink || a->bias_range > 0.f))
    return fail(L3CI_ERR_UNSUPPORTED, "mixer_attention: two maps take no window, sink or distance bias");
  if (a->maps == 2 && a->Db) return fail(L3CI_ERR_UNSUPPORTED, "mixer_attention: two maps have one key part");
  if (a->B == 0 || a->T == 0) return L3CI_OK;
  if (!a->qa || !a->ka || !a->v || !a->out || !a->positions || (a->Db && (!a->qb || !a->kb)))
    return fail(L3CI_ERR_INVALID, "mixer_attention: null pointer");
  return L3CI_OK;
}

int choose(const l3ci_mixer_attn_args* a) {
  const bool mma = mixer_mma_applies(a), tc = mixer_tc_applies(a);
  if (a->variant == 1) return 1;
  if (a->variant == 2) return mma ? 2 : -1;
  if (a->variant == 3) return tc ? 3 : -1;
  if (tc && (a->T >= 128 || !mma)) return 3;
  return mma ? 2 : 1;
}

}  // namespace
}  // namespace l3ci

extern "C" {

int l3ci_mixer_attention_variant(const l3ci_mixer_attn_args* a) {
  using namespace l3ci;
  clear_error();
  return validate(a) == L3CI_OK ? choose(a) : -1;
}

size_t l3ci_mixer_attention_scratch_bytes(const l3ci_mixer_attn_args* a) {
  using namespace l3ci;
  clear_error();
  if (validate(a) != L3CI_OK || a->B == 0 || a->T == 0) return 0;
  const int v = choose(a);
  return v == 2 ? mixer_mma_scratch_bytes(a) : v == 3 ? mixer_tc_scratch_bytes(a) : 0;
}

int l3ci_mixer_attention(const l3ci_mixer_attn_args* a) {
  using namespace l3ci;
  clear_error();
  if (int st = validate(a)) return st;
  if (a->B == 0 || a->T == 0) return L3CI_OK;
  const int v = choose(a);
  if (v == 2) return mixer_mma_launch(a);
  if (v == 3) return mixer_tc_launch(a);
  if (v < 0) return fail(L3CI_ERR_UNSUPPORTED, "mixer_attention: variant %d does not take these sizes or layouts", a->variant);
  if (a->Dv > kRowThreads * kRowCols || a->maps * (a->Da + a->Db) > 12000 || a->H > 65535 || a->B > 65535)
    return fail(L3CI_ERR_UNSUPPORTED, "mixer_attention: sizes beyond the plain kernel (Da=%d Db=%d Dv=%d)", a->Da, a->Db, a->Dv);
  if (a->dtype == L3CI_BF16) return a->maps == 2 ? launch_rows<__nv_bfloat16, 2>(a) : launch_rows<__nv_bfloat16, 1>(a);
  return a->maps == 2 ? launch_rows<float, 2>(a) : launch_rows<float, 1>(a);
}

}  // extern "C"
