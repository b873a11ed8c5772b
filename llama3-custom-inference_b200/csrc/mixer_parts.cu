// The memory-bound steps around the mixers of a decoder with a 32-bit residual stream: residual add + dynamic-tanh
// norm (with the embedding lookup as its first form), activations, the passes that turn a fused projection row into
// queries and cache rows, and the mixes of a token with the one before it.  Storage is bf16 or fp32 (template), arithmetic fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "host_common.h"
#include "../../include/l3ci_mixers.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

// ---- x += y (or x = table[token]);  out = tanh(alpha x) * w + b ------------------------------------------------
// A CTA per row; VEC elements per access (4: 16 bytes of the fp32 stream, 8 or 16 of the storage type).
template <typename S, int VEC>
__global__ void __launch_bounds__(512)
add_dyn_tanh_kernel(const S* __restrict__ y, const long long* __restrict__ tokens, const S* __restrict__ table, long long vocab,
                    float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, float alpha,
                    S* __restrict__ out, int width) {
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  float* xr = x + row * width;
  const S* add = y ? y + row * width : nullptr;
  if (tokens) {
    const long long tok = tokens[row];
    add = tok >= 0 && tok < vocab ? table + tok * width : nullptr;
  }
  for (int c = threadIdx.x * VEC; c < width; c += blockDim.x * VEC) {
    float v[VEC], a[VEC];
    if (tokens) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    } else {
      load_vec<float, VEC>(xr + c, v);
    }
    if (add) {
      load_vec<S, VEC>(add + c, a);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += a[i];
    }
    if (add || tokens) store_vec<float, VEC>(xr + c, v);
    float wv[VEC], bv[VEC];
    load_vec<float, VEC>(w + c, wv);
    load_vec<float, VEC>(b + c, bv);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = fmaf(tanhf(alpha * v[i]), wv[i], bv[i]);
    store_vec<S, VEC>(out + row * width + c, v);
  }
}

enum { kGelu = 0, kTanh = 1 };

template <typename S, int VEC, int KIND>
__global__ void __launch_bounds__(256) activation_kernel(const S* __restrict__ z, S* __restrict__ out, long long n) {
  pdl_wait();
  pdl_launch_dependents();
  const long long i0 = ((long long)blockIdx.x * 256 + threadIdx.x) * VEC;
  if (i0 >= n) return;
  float v[VEC];
  load_vec<S, VEC>(z + i0, v);
#pragma unroll
  for (int i = 0; i < VEC; ++i) v[i] = KIND == kTanh ? tanhf(v[i]) : 0.5f * v[i] * (1.f + erff(v[i] * 0.70710678118654752f));
  store_vec<S, VEC>(out + i0, v);
}

// ---- gated feed-forward activation of rows [gate | up] -----------------------------------------------------------
template <typename S, int VEC>
__global__ void __launch_bounds__(256)
gated_act_kernel(const S* __restrict__ gu, S* __restrict__ out, long long units, int per_row, float limit, float alpha) {
  pdl_wait();
  pdl_launch_dependents();
  const long long id = (long long)blockIdx.x * 256 + threadIdx.x;
  if (id >= units) return;
  const long long row = units <= 0xffffffffLL ? (unsigned)id / (unsigned)per_row : id / per_row;
  const int c = (int)(id - row * per_row) * VEC, ff = per_row * VEC;
  float g[VEC], u[VEC];
  load_vec<S, VEC>(gu + row * 2 * ff + c, g);
  load_vec<S, VEC>(gu + row * 2 * ff + ff + c, u);
#pragma unroll
  for (int i = 0; i < VEC; ++i) g[i] = gated_activation(g[i], u[i], limit, alpha);
  store_vec<S, VEC>(out + row * ff + c, g);
}

// ---- whole-row RMS norm of q and k, k and v into the caches ------------------------------------------------------
struct QkNormRow {
  long long stride, k_sb, k_st, v_sb, v_st, cache_len;
  int q_width, k_width, v_width, T;
  float eps;
};

template <typename S, int VEC>
__global__ void __launch_bounds__(256)
qk_norm_cache_kernel(S* __restrict__ qkv, const float* __restrict__ qw, const float* __restrict__ kw, S* __restrict__ ck,
                     S* __restrict__ cv, const int* __restrict__ positions, const QkNormRow p) {
  __shared__ float red[2][8];
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  const int b = (int)(row / p.T), t = (int)(row % p.T), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x / kWarp;
  const long long pos = (long long)positions[b] + t;
  S* r = qkv + row * p.stride;
  const int qk = p.q_width + p.k_width, step = blockDim.x * VEC;
  float ss[2] = {0.f, 0.f};
  for (int c = tid * VEC; c < qk; c += step) {
    float f[VEC];
    load_vec<S, VEC>(r + c, f);
    const int part = c < p.q_width ? 0 : 1;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      if (part == 0) ss[0] = fmaf(f[i], f[i], ss[0]);
      else ss[1] = fmaf(f[i], f[i], ss[1]);
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) ss[i] = group_sum<kWarp>(ss[i]);
  if (lane == 0) {
    red[0][warp] = ss[0];
    red[1][warp] = ss[1];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) ss[i] = group_sum<8>(lane % 8 < warps ? red[i][lane % 8] : 0.f);
  const float iq = 1.f / sqrtf(ss[0] / (float)p.q_width + p.eps), ik = 1.f / sqrtf(ss[1] / (float)p.k_width + p.eps);
  const bool cached = pos >= 0 && pos < p.cache_len;
  S* kr = ck + b * p.k_sb + pos * p.k_st;
  S* vr = cv + b * p.v_sb + pos * p.v_st;
  for (int c = tid * VEC; c < qk + p.v_width; c += step) {
    float f[VEC], w[VEC];
    load_vec<S, VEC>(r + c, f);
    if (c < qk) {
      const bool is_q = c < p.q_width;
      load_vec<float, VEC>(is_q ? qw + c : kw + (c - p.q_width), w);
#pragma unroll
      for (int i = 0; i < VEC; ++i) f[i] = f[i] * (is_q ? iq : ik) * w[i];
      if (is_q) store_vec<S, VEC>(r + c, f);
      else if (cached) store_vec<S, VEC>(kr + (c - p.q_width), f);
    } else if (cached) {
      store_vec<S, VEC>(vr + (c - qk), f);
    }
  }
}

// ---- token shift: n mixes of a row with the one before it ----------------------------------------------------------
template <typename S, int VEC>
__global__ void __launch_bounds__(256)
token_shift_kernel(const S* __restrict__ h, const float* __restrict__ mu, S* __restrict__ last, long long last_sb,
                   const int* __restrict__ positions, S* __restrict__ out, int n_mix, int T, long long rows, int width) {
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  const int b = (int)(row / T), t = (int)(row % T);
  const bool fresh = positions[b] == 0;
  S* carried = last + b * last_sb;
  for (int c = threadIdx.x * VEC; c < width; c += blockDim.x * VEC) {
    float x[VEC], d[VEC] = {};
    load_vec<S, VEC>(h + row * width + c, x);
    if (t > 0) {
      load_vec<S, VEC>(h + (row - 1) * width + c, d);
    } else {
      if (!fresh) load_vec<S, VEC>(carried + c, d);
      float end[VEC];                                       // the thread that has read the old value writes the new one
      load_vec<S, VEC>(h + (row + T - 1) * width + c, end);
      store_vec<S, VEC>(carried + c, end);
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) d[i] -= x[i];
    for (int s = 0; s < n_mix; ++s) {
      float m[VEC];
      load_vec<float, VEC>(mu + (long long)s * width + c, m);
#pragma unroll
      for (int i = 0; i < VEC; ++i) m[i] = fmaf(d[i], m[i], x[i]);
      store_vec<S, VEC>(out + ((long long)s * rows + row) * width + c, m);
    }
  }
}

// ---- latent attention: query rotation in place, latent norm, key rotation, cache row ---------------------------
struct LatentRow {
  long long qd_stride, table_rows, cache_sb, cache_st, cache_len;
  int T, H, dim, rot, rank;
  float eps;
};

template <typename S>
__global__ void __launch_bounds__(256)
latent_cache_kernel(S* __restrict__ qd, const float* __restrict__ table, const float* __restrict__ nw, S* __restrict__ cache,
                    const int* __restrict__ positions, const LatentRow p) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  const int b = (int)(row / p.T), t = (int)(row % p.T);
  const long long pos = (long long)positions[b] + t;
  if (pos < 0 || pos >= p.table_rows || pos >= p.cache_len) return;
  S* r = qd + row * p.qd_stride;
  const int half = p.rot / 2, head = p.dim + p.rot;
  const float* cs = table + pos * p.rot;
  const S* down = r + (long long)p.H * head;
  S* dst = cache + b * p.cache_sb + pos * p.cache_st;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.rank; c += blockDim.x) {
    const float v = to_f32(down[c]);
    ss = fmaf(v, v, ss);
  }
  ss = cta_sum(ss, red, blockDim.x / kWarp);
  const float inv = __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)p.rank), p.eps));
  for (int c = threadIdx.x; c < p.rank; c += blockDim.x) dst[c] = from_f32<S>(to_f32(down[c]) * inv * nw[c]);
  // the shared key part, then the query heads: (H + 1) * rot/2 pairs
  for (int i = threadIdx.x; i < (p.H + 1) * half; i += blockDim.x) {
    const int n = i / half, j = i % half;
    const float c = cs[2 * j], s = cs[2 * j + 1];
    const S* src = n < p.H ? r + (long long)n * head + p.dim : down + p.rank;
    const float u = to_f32(src[j]), v = to_f32(src[j + half]);
    S* to = n < p.H ? r + (long long)n * head + p.dim : dst + p.rank;
    to[j] = from_f32<S>(u * c - v * s);
    to[j + half] = from_f32<S>(v * c + u * s);
  }
}

// The same in 16-byte vectors (bf16; rank a multiple of 8, rot_dim of 16, rows on 16 bytes): all loads of a row are in
// flight before the reduction of its latent.
constexpr int kLatentThreads = 128;
constexpr int kLatentVecs = 8;   // latent vectors per thread at most: rank <= 8192

template <int VPT>
__global__ void __launch_bounds__(kLatentThreads)
latent_cache_vec_kernel(__nv_bfloat16* __restrict__ qd, const float* __restrict__ table, const float* __restrict__ nw,
                        __nv_bfloat16* __restrict__ cache, const int* __restrict__ positions, const LatentRow p) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const long long row = blockIdx.x;
  const int b = (int)(row / p.T), t = (int)(row % p.T), tid = threadIdx.x;
  // the row's own loads do not wait for the position
  const long long pos = (long long)positions[b] + t;
  __nv_bfloat16* r = qd + row * p.qd_stride;
  const int head = p.dim + p.rot, half = p.rot / 2, per_head = half / 8, tasks = (p.H + 1) * per_head;   // pairs of vectors
  const __nv_bfloat16* down = r + (long long)p.H * head;
  uint4 c[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = tid + i * kLatentThreads;
    c[i] = v * 8 < p.rank ? *reinterpret_cast<const uint4*>(down + v * 8) : make_uint4(0, 0, 0, 0);
  }
  auto load_pair = [&](int i, uint4& u, uint4& v) {
    const int n = i / per_head, j = (i - n * per_head) * 8;
    const __nv_bfloat16* src = n < p.H ? r + (long long)n * head + p.dim : down + p.rank;
    u = *reinterpret_cast<const uint4*>(src + j);
    v = *reinterpret_cast<const uint4*>(src + j + half);
  };
  uint4 uv = make_uint4(0, 0, 0, 0), vv = uv;
  if (tid < tasks) load_pair(tid, uv, vv);
  if (pos < 0 || pos >= p.table_rows || pos >= p.cache_len) return;
  __nv_bfloat16* dst = cache + b * p.cache_sb + pos * p.cache_st;
  const float* cs = table + pos * p.rot;
  for (int i = tid; i < tasks; i += kLatentThreads) {
    const int n = i / per_head, j = (i - n * per_head) * 8;
    __nv_bfloat16* to = n < p.H ? r + (long long)n * head + p.dim : dst + p.rank;
    if (i != tid) load_pair(i, uv, vv);
    float u[8], v[8], x[8], y[8];
    unpack8(uv, u);
    unpack8(vv, v);
#pragma unroll
    for (int k = 0; k < 8; k += 2) {
      const float4 f = __ldg(reinterpret_cast<const float4*>(cs + 2 * (j + k)));   // cos, sin of pairs j + k, j + k + 1
      x[k] = u[k] * f.x - v[k] * f.y;
      y[k] = v[k] * f.x + u[k] * f.y;
      x[k + 1] = u[k + 1] * f.z - v[k + 1] * f.w;
      y[k + 1] = v[k + 1] * f.z + u[k + 1] * f.w;
    }
    *reinterpret_cast<uint4*>(to + j) = pack8(x);
    *reinterpret_cast<uint4*>(to + j + half) = pack8(y);
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    float f[8];
    unpack8(c[i], f);
#pragma unroll
    for (int k = 0; k < 8; ++k) ss = fmaf(f[k], f[k], ss);
  }
  ss = cta_sum(ss, red, kLatentThreads / kWarp);
  const float inv = __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)p.rank), p.eps));
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = tid + i * kLatentThreads;
    if (v * 8 < p.rank) {
      float f[8];
      unpack8(c[i], f);
      const float4 w0 = __ldg(reinterpret_cast<const float4*>(nw + v * 8)), w1 = __ldg(reinterpret_cast<const float4*>(nw + v * 8 + 4));
      const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
      for (int k = 0; k < 8; ++k) f[k] = f[k] * inv * w[k];
      *reinterpret_cast<uint4*>(dst + v * 8) = pack8(f);
    }
  }
}

// Many tokens: a warp per token, no barrier, the token's latent and its first 32 * kPairsAhead vector pairs in flight at once.
constexpr int kPairsAhead = 3;

template <int VPL>
__global__ void __launch_bounds__(256)
latent_cache_rows_kernel(__nv_bfloat16* __restrict__ qd, const float* __restrict__ table, const float* __restrict__ nw,
                         __nv_bfloat16* __restrict__ cache, const int* __restrict__ positions, const LatentRow p, long long rows) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int b = (int)(row / p.T), t = (int)(row - (long long)b * p.T);
  const long long pos = (long long)positions[b] + t;
  __nv_bfloat16* r = qd + row * p.qd_stride;
  const int head = p.dim + p.rot, half = p.rot / 2, per_head = half / 8, tasks = (p.H + 1) * per_head;
  const __nv_bfloat16* down = r + (long long)p.H * head;
  uint4 c[VPL], u[kPairsAhead], v[kPairsAhead];
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int x = lane + 32 * i;
    c[i] = x * 8 < p.rank ? ld_stream16(down + x * 8) : make_uint4(0, 0, 0, 0);
  }
  auto source = [&](int i) {
    const int n = i / per_head, j = (i - n * per_head) * 8;
    return (n < p.H ? r + (long long)n * head + p.dim : const_cast<__nv_bfloat16*>(down) + p.rank) + j;
  };
  auto load = [&](int i0) {
#pragma unroll
    for (int k = 0; k < kPairsAhead; ++k) {
      const int i = i0 + lane + 32 * k;
      if (i < tasks) {
        const __nv_bfloat16* src = source(i);
        u[k] = *reinterpret_cast<const uint4*>(src);
        v[k] = *reinterpret_cast<const uint4*>(src + half);
      }
    }
  };
  load(0);
  if (pos < 0 || pos >= p.table_rows || pos >= p.cache_len) return;
  __nv_bfloat16* dst = cache + b * p.cache_sb + pos * p.cache_st;
  const float* cs = table + pos * p.rot;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    float f[8];
    unpack8(c[i], f);
#pragma unroll
    for (int k = 0; k < 8; ++k) ss = fmaf(f[k], f[k], ss);
  }
  ss = group_sum<32>(ss);
  const float inv = __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)p.rank), p.eps));
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int x = lane + 32 * i;
    if (x * 8 < p.rank) {
      float f[8];
      unpack8(c[i], f);
      const float4 w0 = __ldg(reinterpret_cast<const float4*>(nw + x * 8)), w1 = __ldg(reinterpret_cast<const float4*>(nw + x * 8 + 4));
      const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
      for (int k = 0; k < 8; ++k) f[k] = f[k] * inv * w[k];
      *reinterpret_cast<uint4*>(dst + x * 8) = pack8(f);
    }
  }
  for (int i0 = 0;; ) {
#pragma unroll
    for (int k = 0; k < kPairsAhead; ++k) {
      const int i = i0 + lane + 32 * k;
      if (i >= tasks) continue;
      const int n = i / per_head, j = (i - n * per_head) * 8;
      __nv_bfloat16* to = n < p.H ? source(i) : dst + p.rank + j;
      float a[8], d[8], x[8], y[8];
      unpack8(u[k], a);
      unpack8(v[k], d);
#pragma unroll
      for (int q = 0; q < 8; q += 2) {
        const float4 f = __ldg(reinterpret_cast<const float4*>(cs + 2 * (j + q)));
        x[q] = a[q] * f.x - d[q] * f.y;
        y[q] = d[q] * f.x + a[q] * f.y;
        x[q + 1] = a[q + 1] * f.z - d[q + 1] * f.w;
        y[q + 1] = d[q + 1] * f.z + a[q + 1] * f.w;
      }
      *reinterpret_cast<uint4*>(to) = pack8(x);
      *reinterpret_cast<uint4*>(to + half) = pack8(y);
    }
    i0 += 32 * kPairsAhead;
    if (i0 >= tasks) break;
    load(i0);
  }
}

// ---- k and v columns of a projection row into the caches ------------------------------------------------------
// A thread copies COPIES accesses of VEC elements, all loaded before the first is stored.
template <typename S, int VEC, int COPIES>
__global__ void __launch_bounds__(128)
kv_cache_write_kernel(const S* __restrict__ src, long long stride, long long k_col, int k_width, long long v_col, int v_width,
                      S* __restrict__ ck, long long k_sb, long long k_st, S* __restrict__ cv, long long v_sb, long long v_st,
                      long long cache_len, const int* __restrict__ positions, int T, int rows) {
  pdl_wait();
  pdl_launch_dependents();
  using R = typename Raw<VEC * sizeof(S)>::type;
  const unsigned per_row = (k_width + v_width) / VEC;
  R data[COPIES];
  S* to[COPIES];
#pragma unroll
  for (int u = 0; u < COPIES; ++u) {
    to[u] = nullptr;
    const long long id = ((long long)blockIdx.x * COPIES + u) * 128 + threadIdx.x;
    if (id >= (long long)rows * per_row) continue;
    const long long row = per_row * (long long)rows <= 0xffffffffLL ? (unsigned)id / per_row : id / per_row;
    const int i = (int)(id - row * per_row) * VEC, b = (int)(row / T), t = (int)(row % T);
    const long long pos = (long long)positions[b] + t;
    if (pos < 0 || pos >= cache_len) continue;
    const bool is_k = i < k_width;
    data[u] = *reinterpret_cast<const R*>(src + row * stride + (is_k ? k_col + i : v_col + (i - k_width)));
    to[u] = is_k ? ck + b * k_sb + pos * k_st + i : cv + b * v_sb + pos * v_st + (i - k_width);
  }
#pragma unroll
  for (int u = 0; u < COPIES; ++u)
    if (to[u]) *reinterpret_cast<R*>(to[u]) = data[u];
}

bool bad_dtype(int dtype) { return dtype != L3CI_BF16 && dtype != L3CI_F32; }
template <typename S>
bool vec_ok(const void* p, int vec) { return (reinterpret_cast<uintptr_t>(p) % (vec * sizeof(S))) == 0; }

template <typename S>
int add_dyn_tanh_typed(const void* y, const int64_t* tokens, const void* table, int64_t vocab, float* x, const float* w,
                       const float* b, float alpha, void* out, int64_t rows, int64_t width, cudaStream_t stream) {
  const bool v4 = width % 4 == 0 && vec_ok<S>(y, 4) && vec_ok<S>(table, 4) && vec_ok<S>(out, 4) && vec_ok<float>(x, 4) &&
                  vec_ok<float>(w, 4) && vec_ok<float>(b, 4);
  const int units = (int)(v4 ? width / 4 : width);
  int threads = 32;
  while (threads < 512 && threads < units) threads *= 2;
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("add_dyn_tanh_kernel", kernel, dim3((unsigned)rows), dim3(threads), 0, stream, static_cast<const S*>(y),
                reinterpret_cast<const long long*>(tokens), static_cast<const S*>(table), (long long)vocab, x, w, b, alpha,
                static_cast<S*>(out), (int)width);
    return L3CI_OK;
  };
  return v4 ? go(add_dyn_tanh_kernel<S, 4>) : go(add_dyn_tanh_kernel<S, 1>);
}

template <typename S, int KIND>
int activation_typed(const void* z, void* out, int64_t n, cudaStream_t stream) {
  constexpr int kVec = 16 / sizeof(S);
  const bool v = n % kVec == 0 && vec_ok<S>(z, kVec) && vec_ok<S>(out, kVec);
  const long long units = v ? n / kVec : n, ctas = (units + 255) / 256;
  if (ctas > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "activation: tensor too large");
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("activation_kernel", kernel, dim3((unsigned)ctas), dim3(256), 0, stream, static_cast<const S*>(z), static_cast<S*>(out), (long long)n);
    return L3CI_OK;
  };
  return v ? go(activation_kernel<S, kVec, KIND>) : go(activation_kernel<S, 1, KIND>);
}

template <int KIND>
int activation(const char* name, const void* z, void* out, int64_t n, int32_t dtype, cudaStream_t stream) {
  clear_error();
  if (n < 0 || bad_dtype(dtype)) return fail(L3CI_ERR_INVALID, "%s: n=%lld dtype=%d", name, (long long)n, dtype);
  if (n == 0) return L3CI_OK;
  if (!z || !out) return fail(L3CI_ERR_INVALID, "%s: null pointer", name);
  return dtype == L3CI_BF16 ? activation_typed<__nv_bfloat16, KIND>(z, out, n, stream) : activation_typed<float, KIND>(z, out, n, stream);
}

}  // namespace
}  // namespace l3ci

extern "C" {

const char* l3ci_mixers_last_error(void) { return l3ci_last_error(); }
int l3ci_mixers_set_programmatic_launch(int on) { return l3ci_set_programmatic_launch(on); }

int l3ci_add_dyn_tanh(const void* y, const int64_t* tokens, const void* table, int64_t vocab, float* x, const float* weight,
                      const float* bias, float alpha, void* out, int64_t rows, int64_t width, int32_t dtype,
                      l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (rows < 0 || width <= 0 || width > 0x7fffffffLL || rows > 0x7fffffffLL || bad_dtype(dtype))
    return fail(L3CI_ERR_INVALID, "add_dyn_tanh: rows=%lld width=%lld dtype=%d", (long long)rows, (long long)width, dtype);
  if (rows == 0) return L3CI_OK;
  if (!x || !weight || !bias || !out || (tokens && (!table || vocab <= 0 || y)))
    return fail(L3CI_ERR_INVALID, "add_dyn_tanh: null pointer, or both y and tokens");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  return dtype == L3CI_BF16 ? add_dyn_tanh_typed<__nv_bfloat16>(y, tokens, table, vocab, x, weight, bias, alpha, out, rows, width, s)
                            : add_dyn_tanh_typed<float>(y, tokens, table, vocab, x, weight, bias, alpha, out, rows, width, s);
}

int l3ci_gelu(const void* z, void* out, int64_t n, int32_t dtype, l3ci_stream_t stream) {
  return l3ci::activation<l3ci::kGelu>("gelu", z, out, n, dtype, reinterpret_cast<cudaStream_t>(stream));
}

int l3ci_tanh(const void* z, void* out, int64_t n, int32_t dtype, l3ci_stream_t stream) {
  return l3ci::activation<l3ci::kTanh>("tanh", z, out, n, dtype, reinterpret_cast<cudaStream_t>(stream));
}

int l3ci_gated_act(const void* gu, void* out, int64_t rows, int64_t ff, float limit, float alpha, int32_t dtype, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (rows < 0 || ff <= 0 || ff > 0x3fffffffLL || bad_dtype(dtype) || !(limit >= 0.f))
    return fail(L3CI_ERR_INVALID, "gated_act: rows=%lld ff=%lld dtype=%d", (long long)rows, (long long)ff, dtype);
  if (rows == 0) return L3CI_OK;
  if (!gu || !out) return fail(L3CI_ERR_INVALID, "gated_act: null pointer");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    constexpr int kVec = 16 / sizeof(S);
    const bool v = ff % kVec == 0 && aligned16(gu) && aligned16(out);
    const long long units = rows * (v ? ff / kVec : ff), ctas = (units + 255) / 256;
    if (ctas > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "gated_act: too much");
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("gated_act_kernel", kernel, dim3((unsigned)ctas), dim3(256), 0, s, static_cast<const S*>(gu), static_cast<S*>(out), units,
                  (int)(units / rows), limit, alpha);
      return L3CI_OK;
    };
    return v ? go(gated_act_kernel<S, kVec>) : go(gated_act_kernel<S, 1>);
  };
  return dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

int l3ci_qk_norm_cache(void* qkv, int64_t stride, int64_t q_width, int64_t k_width, int64_t v_width, const float* q_norm,
                       const float* k_norm, float eps, void* cache_k, int64_t k_sb, int64_t k_st, void* cache_v, int64_t v_sb,
                       int64_t v_st, int64_t cache_len, const int32_t* positions, int32_t B, int32_t T, int32_t dtype,
                       l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (B < 0 || T < 0 || q_width <= 0 || k_width <= 0 || v_width <= 0 || q_width + k_width + v_width > 0x3fffffffLL ||
      stride < q_width + k_width + v_width || bad_dtype(dtype))
    return fail(L3CI_ERR_INVALID, "qk_norm_cache: B=%d T=%d widths %lld %lld %lld", B, T, (long long)q_width, (long long)k_width, (long long)v_width);
  if (B == 0 || T == 0) return L3CI_OK;
  if (!qkv || !q_norm || !k_norm || !cache_k || !cache_v || !positions) return fail(L3CI_ERR_INVALID, "qk_norm_cache: null pointer");
  const long long rows = (long long)B * T;
  if (rows > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "qk_norm_cache: too many rows");
  const QkNormRow p{stride, k_sb, k_st, v_sb, v_st, cache_len, (int)q_width, (int)k_width, (int)v_width, T, eps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    constexpr int kVec = 16 / sizeof(S);
    const int64_t all = stride | q_width | k_width | v_width | k_sb | k_st | v_sb | v_st;
    const bool v = all % kVec == 0 && aligned16(qkv) && aligned16(cache_k) && aligned16(cache_v) && aligned16(q_norm) && aligned16(k_norm);
    const long long units = (q_width + k_width + v_width) / (v ? kVec : 1);
    int threads = 32;
    while (threads < 256 && threads < units) threads *= 2;
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("qk_norm_cache_kernel", kernel, dim3((unsigned)rows), dim3(threads), 0, s, static_cast<S*>(qkv), q_norm, k_norm,
                  static_cast<S*>(cache_k), static_cast<S*>(cache_v), positions, p);
      return L3CI_OK;
    };
    if constexpr (sizeof(S) == 4) {
      return v ? go(qk_norm_cache_kernel<S, 4>) : go(qk_norm_cache_kernel<S, 1>);
    } else {
      // (weights are read in as many elements as the row: 32 bytes, two accesses)
      return v ? go(qk_norm_cache_kernel<S, 8>) : go(qk_norm_cache_kernel<S, 1>);
    }
  };
  return dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

int l3ci_token_shift(const void* h, const float* mu, void* last, int64_t last_sb, const int32_t* positions, void* out, int32_t n_mix,
                     int32_t B, int32_t T, int64_t width, int32_t dtype, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (B < 0 || T < 0 || n_mix <= 0 || width <= 0 || width > 0x3fffffffLL || bad_dtype(dtype) || (B > 1 && last_sb < width))
    return fail(L3CI_ERR_INVALID, "token_shift: B=%d T=%d n_mix=%d width=%lld", B, T, n_mix, (long long)width);
  if (B == 0 || T == 0) return L3CI_OK;
  if (!h || !mu || !last || !positions || !out) return fail(L3CI_ERR_INVALID, "token_shift: null pointer");
  const long long rows = (long long)B * T;
  if (rows > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "token_shift: too many rows");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    constexpr int kVec = 16 / sizeof(S);
    const bool v = (width | last_sb) % kVec == 0 && aligned16(h) && aligned16(mu) && aligned16(last) && aligned16(out);
    const long long units = width / (v ? kVec : 1);
    int threads = 32;
    while (threads < 256 && threads < units) threads *= 2;
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("token_shift_kernel", kernel, dim3((unsigned)rows), dim3(threads), 0, s, static_cast<const S*>(h), mu, static_cast<S*>(last),
                  (long long)last_sb, positions, static_cast<S*>(out), n_mix, T, rows, (int)width);
      return L3CI_OK;
    };
    return v ? go(token_shift_kernel<S, kVec>) : go(token_shift_kernel<S, 1>);
  };
  return dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

int l3ci_latent_cache(void* qd, int64_t qd_stride, const float* table, int64_t table_rows, const float* norm_weight, float eps,
                      void* cache, int64_t cache_sb, int64_t cache_st, int64_t cache_len, const int32_t* positions, int32_t B,
                      int32_t T, int32_t H, int32_t dim, int32_t rot_dim, int32_t rank, int32_t dtype, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (B < 0 || T < 0 || H <= 0 || dim < 0 || rot_dim < 0 || rot_dim % 2 || rank <= 0 || bad_dtype(dtype) ||
      qd_stride < (int64_t)H * (dim + rot_dim) + rank + rot_dim || cache_st < rank + rot_dim)
    return fail(L3CI_ERR_INVALID, "latent_cache: B=%d T=%d H=%d dim=%d rot_dim=%d rank=%d", B, T, H, dim, rot_dim, rank);
  if (B == 0 || T == 0) return L3CI_OK;
  if (!qd || (!table && rot_dim) || !norm_weight || !cache || !positions) return fail(L3CI_ERR_INVALID, "latent_cache: null pointer");
  const long long rows = (long long)B * T;
  if (rows > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "latent_cache: too many rows");
  LatentRow p{qd_stride, table_rows, cache_sb, cache_st, cache_len, T, H, dim, rot_dim, rank, eps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  const bool vec = dtype == L3CI_BF16 && rank % 8 == 0 && rot_dim % 16 == 0 && dim % 8 == 0 && qd_stride % 8 == 0 && cache_sb % 8 == 0 &&
                   cache_st % 8 == 0 && rank <= 8 * kLatentVecs * kLatentThreads && aligned16(qd) && aligned16(cache) &&
                   aligned16(table) && aligned16(norm_weight);
  if (vec && rank <= 1024 && rows >= 16LL * sm_count()) {
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("latent_cache_rows_kernel", kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, s, static_cast<__nv_bfloat16*>(qd),
                  table, norm_weight, static_cast<__nv_bfloat16*>(cache), positions, p, rows);
      return L3CI_OK;
    };
    return rank <= 512 ? go(latent_cache_rows_kernel<2>) : go(latent_cache_rows_kernel<4>);
  }
  if (vec) {
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("latent_cache_vec_kernel", kernel, dim3((unsigned)rows), dim3(kLatentThreads), 0, s, static_cast<__nv_bfloat16*>(qd),
                  table, norm_weight, static_cast<__nv_bfloat16*>(cache), positions, p);
      return L3CI_OK;
    };
    return rank <= 8 * kLatentThreads ? go(latent_cache_vec_kernel<1>) : go(latent_cache_vec_kernel<kLatentVecs>);
  }
  if (dtype == L3CI_BF16)
    L3CI_LAUNCH("latent_cache_kernel", latent_cache_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(256), 0, s,
                static_cast<__nv_bfloat16*>(qd), table, norm_weight, static_cast<__nv_bfloat16*>(cache), positions, p);
  else
    L3CI_LAUNCH("latent_cache_kernel", latent_cache_kernel<float>, dim3((unsigned)rows), dim3(256), 0, s, static_cast<float*>(qd),
                table, norm_weight, static_cast<float*>(cache), positions, p);
  return L3CI_OK;
}

int l3ci_kv_cache_write(const void* src, int64_t src_stride, int64_t k_col, int64_t k_width, int64_t v_col, int64_t v_width,
                        void* cache_k, int64_t k_sb, int64_t k_st, void* cache_v, int64_t v_sb, int64_t v_st, int64_t cache_len,
                        const int32_t* positions, int32_t B, int32_t T, int32_t dtype, l3ci_stream_t stream_) {
  using namespace l3ci;
  clear_error();
  if (B < 0 || T < 0 || k_width <= 0 || v_width <= 0 || k_width + v_width > 0x7fffffffLL || k_col < 0 || v_col < 0 ||
      k_col + k_width > src_stride || v_col + v_width > src_stride || bad_dtype(dtype))
    return fail(L3CI_ERR_INVALID, "kv_cache_write: B=%d T=%d widths %lld %lld", B, T, (long long)k_width, (long long)v_width);
  if (B == 0 || T == 0) return L3CI_OK;
  if (!src || !cache_k || !cache_v || !positions) return fail(L3CI_ERR_INVALID, "kv_cache_write: null pointer");
  const long long rows = (long long)B * T;
  if (rows > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "kv_cache_write: too many rows");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream_);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    constexpr int kVec = 16 / sizeof(S);
    const int64_t all = src_stride | k_col | k_width | v_col | v_width | k_sb | k_st | v_sb | v_st;
    const bool v = all % kVec == 0 && aligned16(src) && aligned16(cache_k) && aligned16(cache_v);
    auto go = [&](auto kernel, int width, int copies) -> int {
      const long long units = rows * ((k_width + v_width) / width), per_cta = 128LL * copies;
      if ((units + per_cta - 1) / per_cta > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "kv_cache_write: too much");
      L3CI_LAUNCH("kv_cache_write_kernel", kernel, dim3((unsigned)((units + per_cta - 1) / per_cta)), dim3(128), 0, s, static_cast<const S*>(src), (long long)src_stride,
                  (long long)k_col, (int)k_width, (long long)v_col, (int)v_width, static_cast<S*>(cache_k), (long long)k_sb,
                  (long long)k_st, static_cast<S*>(cache_v), (long long)v_sb, (long long)v_st, (long long)cache_len, positions, T, (int)rows);
      return L3CI_OK;
    };
    if (!v) return go(kv_cache_write_kernel<S, 1, 1>, 1, 1);
    return rows < 1024 ? go(kv_cache_write_kernel<S, kVec, 1>, kVec, 1) : go(kv_cache_write_kernel<S, kVec, 4>, kVec, 4);
  };
  return dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

}  // extern "C"
