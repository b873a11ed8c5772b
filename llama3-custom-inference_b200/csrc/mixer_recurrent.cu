// Linear recurrences over a matrix state per (sequence, head), fp32: the gated delta rule with a decay per key channel, and
// time mixing with a bonus for the current token (include/l3ci_mixers.h).
//
// recurrent_scan_kernel.  The columns of the state do not depend on one another, so a CTA takes a run of columns of one head
// through all tokens of the call.  The state lives in registers: 8 lanes share C columns, a lane holds NR of their rows (rows
// 4 l .. 4 l + 3 of every 32, so that the 8 lanes' 16-byte reads of a token's q, k, g cover 128 bytes of shared memory).  Both
// products of the delta rule are taken over the decayed state in one pass,
//     S^T k  and  S^T q,   u = beta (v - S^T k),   o = S^T q + (k . q) u,
// so that a token costs one reduction over the 8 lanes; k . q (and the bonus product of time mixing) is the same for all
// columns and comes with the token.  Rows go two at a time through packed fp32 instructions.
// Four producer warps stage the next tokens (convert, form decays, take the scalar products) in a ring of two chunks while
// the others compute; a chunk's loads are all in flight before the chunk ahead of it is handed over.  The head's output norm
// and gate follow in a pass over the output rows (head_norm_gate_kernel).
//
// recurrent_step_kernel: one token.  A CTA per head streams the state through registers, four columns and every n-th row a
// thread (whole rows per warp access), meets in shared memory for the two products, and applies norm and gate itself.
//
// delta_inputs_kernel: convolution, activation, unit norms, step sizes and decays of all tokens at once; a warp per run of
// tokens and head of one of q, k, v or the decay.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "../../include/l3ci_mixers.h"
#include "host_common.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "tcgen05.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kDelta = 0, kTimeMix = 1;
constexpr int kChunk = 16;         // tokens per stage
constexpr int kRing = 2;           // stages
constexpr int kProducers = 4;      // warps
constexpr int kPerProducer = kChunk / kProducers;
constexpr int kMaxConsumers = 8;   // warps
constexpr int kScanThreads = 32 * (kMaxConsumers + kProducers);

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gate_value(float z, int act) { return act == 0 ? sigmoid(z) : z * sigmoid(z); }

struct ScanParams {
  l3ci_recurrent_scan_args a;
  int splits, cols;              // column runs per head, columns per run
  int consumers;                 // warps
  int vec;                       // q, k, g (and their fp32 companions) allow accesses of four elements
};

// Four channels from d on, zeros behind the last one (loaded from a place that exists, so that no load hangs on a branch).
template <typename S>
__device__ __forceinline__ float4 fetch4(const S* p, int d, int D, int vec) {
  float f[4];
  if (vec) {
    load_vec<S, 4>(p + (d < D ? d : 0), f);
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = d < D ? f[e] : 0.f;
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = to_f32(p[d + e < D ? d + e : 0]);
#pragma unroll
    for (int e = 0; e < 4; ++e) f[e] = d + e < D ? f[e] : 0.f;
  }
  return make_float4(f[0], f[1], f[2], f[3]);
}

// The convolution's carried inputs: row r of the tail becomes the input of token T - (taps - 1) + r.  Channel c of a sequence,
// by one thread.
template <typename S>
__device__ __forceinline__ void move_tail(const l3ci_recurrent_scan_args& a, S* tail, const S* in, long long channels, long long c, bool fresh) {
  const int rows = a.taps - 1;
  for (int r = 0; r < rows; ++r) {
    const int t = a.T - rows + r;
    tail[r * channels + c] = t >= 0 ? in[t * a.conv_st + c] : fresh ? from_f32<S>(0.f) : tail[(r + a.T) * channels + c];
  }
}

// Those of head h's values and, by the first head that reads them, of its queries and keys; `i` of `n` threads.
template <typename S>
__device__ __forceinline__ void move_tails(const l3ci_recurrent_scan_args& a, int b, int h, int i, int n, bool fresh) {
  const int GD = a.G * a.D, R = a.H / a.G;
  const long long channels = 2LL * GD + (long long)a.H * a.V;
  S* tail = static_cast<S*>(a.tail) + b * a.tail_sb;
  const S* in = static_cast<const S*>(a.conv_in) + (long long)b * a.T * a.conv_st;
  for (int c = i; c < a.V; c += n) move_tail<S>(a, tail, in, channels, 2LL * GD + (long long)h * a.V + c, fresh);
  if (h % R == 0)
    for (int c = i; c < 2 * a.D; c += n) move_tail<S>(a, tail, in, channels, c < a.D ? (h / R) * a.D + c : GD + (h / R) * a.D + c - a.D, fresh);
}

// S: storage type of v, gate, out; Q: type of q, k, g.
template <typename S, typename Q, int KIND, int NR, int C>
__global__ void __launch_bounds__(kScanThreads) recurrent_scan_kernel(const __grid_constant__ ScanParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ __align__(16) float smem[];
  const l3ci_recurrent_scan_args& a = p.a;
  const int cols = p.cols;
  const int stage_floats = kChunk * (3 * DP + cols + 2);
  float* stages = smem;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + kRing * stage_floats);
  const uint32_t full0 = smem_u32(bars), empty0 = full0 + kRing * 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x % p.splits, h = (blockIdx.x / p.splits) % a.H, b = blockIdx.x / (p.splits * a.H);
  const int D = a.D, V = a.V, T = a.T, R = a.H / a.G, col0 = split * cols;
  if (tid == 0) {
    for (int i = 0; i < kRing; ++i) {
      mbar_init(full0 + i * 8, kProducers);
      mbar_init(empty0 + i * 8, p.consumers);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const bool fresh = a.positions[b] == 0;
  const int chunks = (T + kChunk - 1) / kChunk;
  bool ok = true;

  if (warp >= p.consumers) {
    // ---- producers ----
    const int pw = warp - p.consumers;
    const long long row0 = (long long)b * T;
    const Q* qp = static_cast<const Q*>(a.q) + (h / R) * a.qk_sh;
    const Q* kp = static_cast<const Q*>(a.k) + (h / R) * a.qk_sh;
    const Q* gp = static_cast<const Q*>(a.g) + h * a.g_sh;
    const S* vp = static_cast<const S*>(a.v) + h * a.v_sh + col0;
    const int n_cols = min(cols, V - col0);
    constexpr int kWide = (DP + 127) / 128;      // accesses of four channels per lane and row
    constexpr int kCols = 4;                     // value columns per lane (a CTA has at most 128)
    float4 q[kPerProducer][kWide], k[kPerProducer][kWide], g[kPerProducer][kWide];
    float v[kPerProducer][kCols], beta[kPerProducer];
    // all loads of this warp's tokens of chunk i (tokens behind the last one: the last one's, never used)
    auto fetch = [&](int i) {
#pragma unroll
      for (int x = 0; x < kPerProducer; ++x) {
        const long long row = row0 + min(i * kChunk + pw * kPerProducer + x, T - 1);
#pragma unroll
        for (int j = 0; j < kWide; ++j) {
          const int d = j * 128 + lane * 4;
          q[x][j] = fetch4<Q>(qp + row * a.qk_st, d, D, p.vec);
          k[x][j] = fetch4<Q>(kp + row * a.qk_st, d, D, p.vec);
          g[x][j] = fetch4<Q>(gp + row * a.g_st, d, D, p.vec);
        }
#pragma unroll
        for (int c = 0; c < kCols; ++c) v[x][c] = to_f32(vp[row * a.v_st + min(c * 32 + lane, n_cols - 1)]);
        beta[x] = KIND == kDelta ? a.beta[row * a.H + h] : 0.f;
      }
    };
    float4 bonus[kWide], gb[kWide];
    if (KIND == kTimeMix) {
#pragma unroll
      for (int j = 0; j < kWide; ++j) {
        bonus[j] = fetch4<float>(a.bonus + h * D, j * 128 + lane * 4, D, p.vec);
        gb[j] = fetch4<float>(a.g_bias + h * D, j * 128 + lane * 4, D, p.vec);
      }
    }
    fetch(0);
    for (int i = 0; i < chunks; ++i) {
      const int s = i % kRing;
      if (i >= kRing && !mbar_wait_bounded(empty0 + s * 8, ((i / kRing) - 1) & 1)) { ok = false; break; }
      float* st = stages + s * stage_floats;
      float* vs = st + kChunk * 3 * DP;
      float* sc = vs + kChunk * cols;
      float scalar[kPerProducer];
#pragma unroll
      for (int x = 0; x < kPerProducer; ++x) {
        const int at = pw * kPerProducer + x;
        scalar[x] = 0.f;
#pragma unroll
        for (int j = 0; j < kWide; ++j) {
          const int d = j * 128 + lane * 4;
          const float4 qq = q[x][j], kk = k[x][j];
          float4 gg = g[x][j];
          if (KIND == kTimeMix) {
            gg.x = expf(-expf(gg.x + gb[j].x));
            gg.y = expf(-expf(gg.y + gb[j].y));
            gg.z = expf(-expf(gg.z + gb[j].z));
            gg.w = expf(-expf(gg.w + gb[j].w));
            scalar[x] += qq.x * kk.x * bonus[j].x + qq.y * kk.y * bonus[j].y + qq.z * kk.z * bonus[j].z + qq.w * kk.w * bonus[j].w;
          } else {
            scalar[x] += qq.x * kk.x + qq.y * kk.y + qq.z * kk.z + qq.w * kk.w;
          }
          if (d < DP) {
            float* row = st + at * 3 * DP + d;
            *reinterpret_cast<float4*>(row) = qq;
            *reinterpret_cast<float4*>(row + DP) = kk;
            *reinterpret_cast<float4*>(row + 2 * DP) = gg;
          }
        }
#pragma unroll
        for (int c = 0; c < kCols; ++c)
          if (c * 32 + lane < cols) vs[at * cols + c * 32 + lane] = c * 32 + lane < n_cols ? v[x][c] : 0.f;
      }
#pragma unroll
      for (int x = 0; x < kPerProducer; ++x) scalar[x] = group_sum<kWarp>(scalar[x]);
      if (lane == 0) {
#pragma unroll
        for (int x = 0; x < kPerProducer; ++x) {
          sc[(pw * kPerProducer + x) * 2] = scalar[x];
          sc[(pw * kPerProducer + x) * 2 + 1] = beta[x];
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(full0 + s * 8);
      if (i + 1 < chunks) fetch(i + 1);
    }
    if (a.tail && split == 0) move_tails<S>(a, b, h, pw * 32 + lane, 32 * kProducers, fresh);
    if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
    return;
  }

  // ---- consumers: lane l of a group of 8 holds rows 32 i + 4 l + e of the group's C columns ----
  const int l = lane & 7, c_loc = (warp * 4 + (lane >> 3)) * C, c0 = col0 + c_loc;
  const bool live = c_loc < cols && c0 < V;    // (V and cols are multiples of C)
  float* state = a.state + b * a.state_sb + (long long)h * D * V + c0;
  unsigned long long S2[C][NR / 2];            // rows in pairs
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    float f[4][C];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
#pragma unroll
      for (int c = 0; c < C; ++c) f[e][c] = 0.f;
      const int row = 32 * i + 4 * l + e;
      if (live && !fresh && row < D) load_vec<float, C>(state + (long long)row * V, f[e]);
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
      S2[c][2 * i] = f2_packf(f[0][c], f[1][c]);
      S2[c][2 * i + 1] = f2_packf(f[2][c], f[3][c]);
    }
  }
  S* out = static_cast<S*>(a.out) + (long long)b * T * a.out_st + h * a.out_sh + c0;
  float o[C];
  for (int i = 0; i < chunks; ++i) {
    const int s = i % kRing, n = min(kChunk, T - i * kChunk);
    if (!mbar_wait_bounded(full0 + s * 8, (i / kRing) & 1)) { ok = false; break; }
    const float* st = stages + s * stage_floats + 4 * l;
    const float* vs = stages + s * stage_floats + kChunk * 3 * DP + (live ? c_loc : 0);
    const float* sc = stages + s * stage_floats + kChunk * (3 * DP + cols);
#pragma unroll 2
    for (int x = 0; x < n; ++x, st += 3 * DP, vs += cols, sc += 2) {
      unsigned long long q2[NR / 2], k2[NR / 2], g2[NR / 2];
#pragma unroll
      for (int j = 0; j < NR / 4; ++j) {
        const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(st + 32 * j);
        const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(st + DP + 32 * j);
        const ulonglong2 gg = *reinterpret_cast<const ulonglong2*>(st + 2 * DP + 32 * j);
        q2[2 * j] = qq.x; q2[2 * j + 1] = qq.y;
        k2[2 * j] = kk.x; k2[2 * j + 1] = kk.y;
        g2[2 * j] = gg.x; g2[2 * j + 1] = gg.y;
      }
      const float scalar = sc[0], beta = sc[1];
      float v[C], dk[C], dq[C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        v[c] = vs[c];
        // two chains each
        unsigned long long aq[2] = {0ull, 0ull}, ak[2] = {0ull, 0ull};
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) {
          if (KIND == kDelta) {
            S2[c][j] = f2_mul(S2[c][j], g2[j]);
            ak[j & 1] = f2_fma(S2[c][j], k2[j], ak[j & 1]);
          }
          aq[j & 1] = f2_fma(S2[c][j], q2[j], aq[j & 1]);
        }
        float x0, x1;
        f2_unpack(f2_add(aq[0], aq[1]), x0, x1);
        dq[c] = x0 + x1;
        if (KIND == kDelta) {
          f2_unpack(f2_add(ak[0], ak[1]), x0, x1);
          dk[c] = x0 + x1;
        }
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        if (KIND == kDelta) dk[c] = group_sum<8>(dk[c]);
        dq[c] = group_sum<8>(dq[c]);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float u = KIND == kDelta ? beta * (v[c] - dk[c]) : v[c];
        o[c] = fmaf(scalar, u, dq[c]);
        const unsigned long long u2 = f2_packf(u, u);
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) S2[c][j] = f2_fma(k2[j], u2, KIND == kDelta ? S2[c][j] : f2_mul(S2[c][j], g2[j]));
      }
      if (l == 0 && live) {
#pragma unroll
        for (int c = 0; c < C; ++c) out[c] = from_f32<S>(o[c]);
      }
      out += a.out_st;
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty0 + s * 8);
  }
  if (!ok) {
    if (lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
  } else {
#pragma unroll
    for (int i = 0; i < NR / 4; ++i) {
      float f[4][C];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        f2_unpack(S2[c][2 * i], f[0][c], f[1][c]);
        f2_unpack(S2[c][2 * i + 1], f[2][c], f[3][c]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = 32 * i + 4 * l + e;
        if (live && row < D) store_vec<float, C>(state + (long long)row * V, f[e]);
      }
    }
  }
}

// ---- one token ----------------------------------------------------------------------------------------------------
constexpr int kStepThreads = 256;

template <typename S, typename Q, int KIND, int RP>
__global__ void __launch_bounds__(kStepThreads, RP <= 4 ? 5 : RP <= 8 ? 3 : 2) recurrent_step_kernel(const __grid_constant__ l3ci_recurrent_scan_args a) {
  extern __shared__ __align__(16) float smem[];
  __shared__ float red[32];
  const int D = a.D, V = a.V, tid = threadIdx.x;
  float *qs = smem, *ks = qs + D, *gs = ks + D;
  float4* part = reinterpret_cast<float4*>(smem + (3 * D + 3) / 4 * 4);    // [2][groups][V / 4]
  const int quads = V / 4, groups = kStepThreads / quads, quad = tid % quads, grp = tid / quads;
  const int h = blockIdx.x % a.H, b = blockIdx.x / a.H, R = a.H / a.G;
  const bool active = grp < groups;
  pdl_wait();
  pdl_launch_dependents();
  const bool fresh = a.positions[b] == 0;
  float4* state = reinterpret_cast<float4*>(a.state + b * a.state_sb + (long long)h * D * V) + quad;
  float4 s[RP];
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = grp + i * groups;
    s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && !fresh && r < D) s[i] = __ldcs(state + (long long)r * quads);
  }
  const S* vp = static_cast<const S*>(a.v) + b * a.v_st + h * a.v_sh + 4 * quad;
  const S* zp = static_cast<const S*>(a.gate) + b * a.gate_st + h * a.gate_sh + 4 * quad;
  float v[4], z[4], w[4];
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    v[c] = to_f32(vp[c]);
    z[c] = to_f32(zp[c]);
    w[c] = a.norm[h * a.norm_sh + 4 * quad + c];
  }
  const float beta = KIND == kDelta ? a.beta[(long long)b * a.H + h] : 0.f;
  float scalar = 0.f;
  for (int d = tid; d < D; d += kStepThreads) {
    const float q = to_f32(static_cast<const Q*>(a.q)[b * a.qk_st + (h / R) * a.qk_sh + d]);
    const float k = to_f32(static_cast<const Q*>(a.k)[b * a.qk_st + (h / R) * a.qk_sh + d]);
    float g = to_f32(static_cast<const Q*>(a.g)[b * a.g_st + h * a.g_sh + d]);
    if (KIND == kTimeMix) {
      g = expf(-expf(g + a.g_bias[h * D + d]));
      scalar = fmaf(q * k, a.bonus[h * D + d], scalar);
    } else {
      scalar = fmaf(q, k, scalar);
    }
    qs[d] = q;
    ks[d] = k;
    gs[d] = g;
  }
  scalar = cta_sum(scalar, red, kStepThreads / kWarp);                     // (its barriers publish the vectors as well)
  float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = grp + i * groups;
    if (!active || r >= D) continue;
    const float q = qs[r], g = gs[r];
    if (KIND == kDelta) {
      const float k = ks[r];
      s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
      ak.x = fmaf(s[i].x, k, ak.x); ak.y = fmaf(s[i].y, k, ak.y); ak.z = fmaf(s[i].z, k, ak.z); ak.w = fmaf(s[i].w, k, ak.w);
    }
    aq.x = fmaf(s[i].x, q, aq.x); aq.y = fmaf(s[i].y, q, aq.y); aq.z = fmaf(s[i].z, q, aq.z); aq.w = fmaf(s[i].w, q, aq.w);
    if (KIND == kTimeMix) { s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g; }
  }
  if (active) {
    if (KIND == kDelta) part[grp * quads + quad] = ak;
    part[(groups + grp) * quads + quad] = aq;
  }
  __syncthreads();
  float u[4] = {v[0], v[1], v[2], v[3]}, o[4] = {0.f, 0.f, 0.f, 0.f};
  if (KIND == kDelta) {
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < groups; ++i) {
      const float4 x = part[i * quads + quad];
      sum.x += x.x; sum.y += x.y; sum.z += x.z; sum.w += x.w;
    }
    u[0] = beta * (v[0] - sum.x); u[1] = beta * (v[1] - sum.y); u[2] = beta * (v[2] - sum.z); u[3] = beta * (v[3] - sum.w);
  }
#pragma unroll
  for (int i = 0; i < RP; ++i) {
    const int r = grp + i * groups;
    if (!active || r >= D) continue;
    const float k = ks[r];
    s[i].x = fmaf(k, u[0], s[i].x); s[i].y = fmaf(k, u[1], s[i].y); s[i].z = fmaf(k, u[2], s[i].z); s[i].w = fmaf(k, u[3], s[i].w);
    __stcs(state + (long long)r * quads, s[i]);
  }
  float ss = 0.f;
  if (grp == 0) {
    for (int i = 0; i < groups; ++i) {
      const float4 x = part[(groups + i) * quads + quad];
      o[0] += x.x; o[1] += x.y; o[2] += x.z; o[3] += x.w;
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      o[c] = fmaf(scalar, u[c], o[c]);
      ss = fmaf(o[c], o[c], ss);
    }
  }
  ss = cta_sum(ss, red, kStepThreads / kWarp);
  if (grp == 0) {
    const float inv = 1.f / sqrtf(ss / (float)V + a.eps);
    S* dst = static_cast<S*>(a.out) + b * a.out_st + h * a.out_sh + 4 * quad;
#pragma unroll
    for (int c = 0; c < 4; ++c) dst[c] = from_f32<S>(o[c] * inv * w[c] * gate_value(z[c], a.act));
  }
  if (a.tail) move_tails<S>(a, b, h, tid, kStepThreads, fresh);
}

// out[row, h, :] <- out / rms(out) * norm * act(gate), in place: a warp per (row, head)
template <typename S, int VEC>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(S* __restrict__ out, long long out_st, long long out_sh, const S* __restrict__ gate, long long gate_st,
                      long long gate_sh, const float* __restrict__ norm, long long norm_sh, int H, int V, long long units, int act, float eps) {
  pdl_wait();
  pdl_launch_dependents();
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (id >= units) return;
  const long long row = id / H;
  const int h = (int)(id - row * H);
  S* o = out + row * out_st + h * out_sh;
  const S* g = gate + row * gate_st + h * gate_sh;
  const float* w = norm + h * norm_sh;
  constexpr int kKeep = 4;                     // vectors of a lane that stay in registers
  float x[kKeep][VEC];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * 32 + lane) * VEC;
    if (c < V) {
      load_vec<S, VEC>(o + c, x[i]);
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(x[i][k], x[i][k], ss);
    }
  }
  for (int c = (kKeep * 32 + lane) * VEC; c < V; c += 32 * VEC) {
    float y[VEC];
    load_vec<S, VEC>(o + c, y);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(y[k], y[k], ss);
  }
  const float inv = 1.f / sqrtf(group_sum<kWarp>(ss) / (float)V + eps);
  auto finish = [&](int c, float (&y)[VEC]) {
    float z[VEC], n[VEC];
    load_vec<S, VEC>(g + c, z);
    load_vec<float, VEC>(w + c, n);
#pragma unroll
    for (int k = 0; k < VEC; ++k) y[k] = y[k] * inv * n[k] * gate_value(z[k], act);
    store_vec<S, VEC>(o + c, y);
  };
#pragma unroll
  for (int i = 0; i < kKeep; ++i) {
    const int c = (i * 32 + lane) * VEC;
    if (c < V) finish(c, x[i]);
  }
  for (int c = (kKeep * 32 + lane) * VEC; c < V; c += 32 * VEC) {
    float y[VEC];
    load_vec<S, VEC>(o + c, y);
    finish(c, y);
  }
}

// ---- inputs of the delta rule -----------------------------------------------------------------------------------
constexpr int kRun = 8;            // consecutive tokens of a warp
constexpr int kMaxTaps = 4;        // taps whose inputs stay in registers along the run

// TAPS > 0: the run's inputs are all asked for at once and every one is loaded once; 0: any number of taps.
template <typename S, int VEC, int TAPS>
__global__ void __launch_bounds__(256) delta_inputs_kernel(const l3ci_delta_inputs_args a, int runs, long long tasks) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= tasks) return;
  const int kinds = 2 * a.G + 2 * a.H;         // q heads, k heads, v heads, decay heads
  // neighbouring warps take neighbouring heads of the same tokens
  const int what = (int)(id % kinds);
  const long long run = id / kinds;
  const int b = (int)(run / runs), t0 = (int)(run % runs) * kRun, n = min(kRun, a.T - t0);
  const long long row0 = (long long)b * a.T;
  const int GD = a.G * a.D;
  const long long C_all = 2LL * GD + (long long)a.H * a.V;
  if (what >= 2 * a.G + a.H) {
    const int h = what - 2 * a.G - a.H;
    const float rate = expf(a.a_log[h]);
    const S* src = static_cast<const S*>(a.a) + (row0 + t0) * a.a_st + (long long)h * a.D;
    if (lane < n) {
      const float z = to_f32(static_cast<const S*>(a.b)[(row0 + t0 + lane) * a.b_st + h]);
      a.beta_out[(row0 + t0 + lane) * a.H + h] = sigmoid(z);
    }
    for (int c = lane * VEC; c < a.D; c += 32 * VEC) {
      float z[kRun][VEC], bias[VEC];
      load_vec<float, VEC>(a.dt_bias + (long long)h * a.D + c, bias);
#pragma unroll
      for (int x = 0; x < kRun; ++x) load_vec<S, VEC>(src + min(x, n - 1) * a.a_st + c, z[x]);
#pragma unroll
      for (int x = 0; x < kRun; ++x) {
        if (x >= n) break;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          const float y = z[x][k] + bias[k];
          z[x][k] = expf(-rate * (fmaxf(y, 0.f) + log1pf(expf(-fabsf(y)))));
        }
        store_vec<float, VEC>(a.decay_out + ((row0 + t0 + x) * a.H + h) * a.D + c, z[x]);
      }
    }
    return;
  }
  const bool is_v = what >= 2 * a.G;
  const int size = is_v ? a.V : a.D;
  const long long ch0 = is_v ? 2LL * GD + (long long)(what - 2 * a.G) * a.V : (long long)what * a.D;
  const bool fresh = a.positions[b] == 0;
  const S* in = static_cast<const S*>(a.p) + row0 * a.p_st + ch0;
  const S* tail = static_cast<const S*>(a.tail) + b * a.tail_sb + ch0;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  constexpr int kKeep = VEC >= 4 ? 2 : 8;      // 256 channels
  auto activation = [](float z) {
    if constexpr (sizeof(S) == 4) return z * sigmoid(z);
    else return __fdividef(z, 1.f + __expf(-z));   // (bf16 models: rounded to bf16, or made a unit vector, right after)
  };
  // input of the sequence's token t (of this call; before it: the carried ones) at channel c
  auto input = [&](int t, int c, float (&f)[VEC]) {
    if (t >= 0) {
      load_vec<S, VEC>(in + (long long)t * a.p_st + c, f);
    } else {
#pragma unroll
      for (int k = 0; k < VEC; ++k) f[k] = 0.f;
      if (!fresh) load_vec<S, VEC>(tail + (taps - 1 + t) * C_all + c, f);
    }
  };
  auto store = [&](int x, int c, const float (&y)[VEC], float f) {
    float r[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) r[k] = y[k] * f;
    const long long row = row0 + t0 + x;
    if (is_v) store_vec<S, VEC>(static_cast<S*>(a.v_out) + row * a.H * a.V + (long long)(what - 2 * a.G) * a.V + c, r);
    else store_vec<float, VEC>(a.qk_out + row * 2 * GD + ch0 + c, r);
  };
  auto unit = [&](float ss) { return is_v ? 1.f : 1.f / sqrtf(ss + a.unit_eps) / (what < a.G ? sqrtf((float)a.D) : 1.f); };
  if (TAPS > 0 && (is_v || size <= 32 * VEC)) {
    constexpr int kTaps = TAPS > 0 ? TAPS : 1;
    for (int c = lane * VEC; c < (is_v ? size : 32 * VEC); c += 32 * VEC) {    // (every lane takes part in a unit vector's sums)
      const bool mine = c < size;
      const int at = mine ? c : 0;
      float f[kRun + kTaps - 1][VEC], w[kTaps][VEC];
#pragma unroll
      for (int i = 0; i < kRun + kTaps - 1; ++i) input(min(t0 - (kTaps - 1) + i, a.T - 1), at, f[i]);
#pragma unroll
      for (int i = 0; i < kTaps; ++i) load_vec<float, VEC>(a.conv + i * C_all + ch0 + at, w[i]);
#pragma unroll
      for (int x = 0; x < kRun; ++x) {
        if (x >= n) break;
        float y[VEC], ss = 0.f;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          y[k] = 0.f;
#pragma unroll
          for (int i = 0; i < kTaps; ++i) y[k] = fmaf(f[x + i][k], w[i][k], y[k]);
          y[k] = activation(y[k]);
          ss = mine ? fmaf(y[k], y[k], ss) : ss;
        }
        if (!is_v) ss = group_sum<kWarp>(ss);
        if (mine) store(x, c, y, unit(ss));
      }
    }
    return;
  }
  for (int x = 0; x < n; ++x) {
    auto convolve = [&](int c, float (&y)[VEC]) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) y[k] = 0.f;
      for (int i = 0; i < taps; ++i) {
        float f[VEC], w[VEC];
        input(t0 + x - (taps - 1) + i, c, f);
        load_vec<float, VEC>(a.conv + i * C_all + ch0 + c, w);
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[k] = fmaf(f[k], w[k], y[k]);
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) y[k] = activation(y[k]);
    };
    if (is_v) {
      for (int c = lane * VEC; c < size; c += 32 * VEC) {
        float y[VEC];
        convolve(c, y);
        store(x, c, y, 1.f);
      }
      continue;
    }
    float y[kKeep][VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = (i * 32 + lane) * VEC;
      if (c < size) {
        convolve(c, y[i]);
#pragma unroll
        for (int k = 0; k < VEC; ++k) ss = fmaf(y[i][k], y[i][k], ss);
      }
    }
    const float f = unit(group_sum<kWarp>(ss));
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = (i * 32 + lane) * VEC;
      if (c < size) store(x, c, y[i], f);
    }
  }
}

constexpr int kMaxD = 256;         // key channels of a head

template <typename S, typename Q, int KIND, int NR, int C>
int launch_scan(const ScanParams& p, cudaStream_t stream) {
  const size_t smem = (size_t)kRing * kChunk * (3 * NR * 8 + p.cols + 2) * 4 + 2 * kRing * 8;
  static bool configured[64] = {false};
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (smem > (48 << 10) && (dev < 0 || dev >= 64 || !configured[dev])) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(recurrent_scan_kernel<S, Q, KIND, NR, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem_optin()));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  L3CI_LAUNCH("recurrent_scan_kernel", recurrent_scan_kernel<S, Q, KIND, NR, C>, dim3((unsigned)((long long)p.a.B * p.a.H * p.splits)),
              dim3(32 * (p.consumers + kProducers)), smem, stream, p);
  return L3CI_OK;
}

// One token per sequence, if its sizes suit: rows of whole 16-byte vectors, at most 16 of them per thread.
template <typename S, typename Q, int KIND>
bool step_applies(const l3ci_recurrent_scan_args* a) {
  if (a->T != 1 || a->V % 4 || a->V > 4 * kStepThreads || a->state_sb % 4 || !aligned16(a->state)) return false;
  const int groups = kStepThreads / (a->V / 4);
  return (a->D + groups - 1) / groups <= 16;
}
template <typename S, typename Q, int KIND>
int step_launch(const l3ci_recurrent_scan_args* a, cudaStream_t stream) {
  const int quads = a->V / 4, groups = kStepThreads / quads, rows = (a->D + groups - 1) / groups;
  const size_t smem = sizeof(float) * ((3 * a->D + 3) / 4 * 4 + 2 * (size_t)groups * a->V);
  const long long ctas = (long long)a->B * a->H;
  if (ctas > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "recurrent_scan: too many sequences");
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("recurrent_step_kernel", kernel, dim3((unsigned)ctas), dim3(kStepThreads), smem, stream, *a);
    return L3CI_OK;
  };
  return rows <= 4 ? go(recurrent_step_kernel<S, Q, KIND, 4>) : rows <= 8 ? go(recurrent_step_kernel<S, Q, KIND, 8>)
                                                                         : go(recurrent_step_kernel<S, Q, KIND, 16>);
}

template <typename S, typename Q, int KIND>
int scan_typed(const l3ci_recurrent_scan_args* a, cudaStream_t stream) {
  if (step_applies<S, Q, KIND>(a)) return step_launch<S, Q, KIND>(a, stream);
  ScanParams p = {};
  p.a = *a;
  const long long heads = (long long)a->B * a->H;
  const int sms = sm_count() > 0 ? sm_count() : 148;
  // columns per thread: as many as leave enough CTAs for the device
  const int widest = a->V % 4 == 0 && a->state_sb % 4 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 15) == 0   ? 4
                     : a->V % 2 == 0 && a->state_sb % 2 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 7) == 0 ? 2
                                                                                                                 : 1;
  int C = 1;
  const struct { int C, W; } shapes[] = {{4, 8}, {2, 8}, {2, 4}, {1, 4}, {1, 2}};
  for (const auto& s : shapes) {
    if (s.C > widest && s.C > 1) continue;
    C = s.C;
    p.consumers = s.W;
    p.splits = (a->V + 4 * C * s.W - 1) / (4 * C * s.W);
    if (heads * p.splits * 5 >= 4LL * sms) break;
  }
  const int need = (a->V + 4 * C - 1) / (4 * C);
  if (p.consumers > need) p.consumers = need;
  p.cols = 4 * C * p.consumers;
  if (p.splits * (long long)p.cols < a->V) p.splits = (a->V + p.cols - 1) / p.cols;
  if (heads * p.splits > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "recurrent_scan: too many sequences");
  auto on = [](const void* x, int bytes) { return (reinterpret_cast<uintptr_t>(x) & (bytes - 1)) == 0; };
  const int q4 = 4 * (int)sizeof(Q);
  p.vec = a->D % 4 == 0 && (a->qk_st | a->qk_sh | a->g_st | a->g_sh) % 4 == 0 && on(a->q, q4) && on(a->k, q4) && on(a->g, q4) &&
          on(a->bonus, 16) && on(a->g_bias, 16);
  auto rows = [&](auto c) -> int {
    constexpr int CC = decltype(c)::value;
    if (a->D <= 32) return launch_scan<S, Q, KIND, 4, CC>(p, stream);
    if (a->D <= 64) return launch_scan<S, Q, KIND, 8, CC>(p, stream);
    if (a->D <= 128) return launch_scan<S, Q, KIND, 16, CC>(p, stream);
    return launch_scan<S, Q, KIND, 32, CC>(p, stream);
  };
  int st;
  if (C == 4) st = rows(std::integral_constant<int, 4>{});
  else if (C == 2) st = rows(std::integral_constant<int, 2>{});
  else st = rows(std::integral_constant<int, 1>{});
  if (st) return st;
  // norm and gate of the rows the scan has written
  const long long units = heads * a->T;
  if ((units + 7) / 8 > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "recurrent_scan: too many rows");
  const bool v4 = (a->V | a->out_st | a->out_sh | a->gate_st | a->gate_sh | a->norm_sh) % 4 == 0 && on(a->out, 4 * sizeof(S)) &&
                  on(a->gate, 4 * sizeof(S)) && on(a->norm, 16);
  auto go = [&](auto kernel) -> int {
    L3CI_LAUNCH("head_norm_gate_kernel", kernel, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, stream, static_cast<S*>(a->out),
                (long long)a->out_st, (long long)a->out_sh, static_cast<const S*>(a->gate), (long long)a->gate_st, (long long)a->gate_sh,
                a->norm, (long long)a->norm_sh, a->H, a->V, units, a->act, a->eps);
    return L3CI_OK;
  };
  return v4 ? go(head_norm_gate_kernel<S, 4>) : go(head_norm_gate_kernel<S, 1>);
}

}  // namespace
}  // namespace l3ci

extern "C" {

int l3ci_delta_inputs(const l3ci_delta_inputs_args* a) {
  using namespace l3ci;
  clear_error();
  if (!a) return fail(L3CI_ERR_INVALID, "delta_inputs: null args");
  if (a->B < 0 || a->T < 0 || a->H <= 0 || a->G <= 0 || a->H % a->G || a->D <= 0 || a->V <= 0 || a->taps <= 0 ||
      (a->dtype != L3CI_BF16 && a->dtype != L3CI_F32) || a->p_st < 2LL * a->G * a->D + (int64_t)a->H * a->V || a->a_st < (int64_t)a->H * a->D)
    return fail(L3CI_ERR_INVALID, "delta_inputs: bad size B=%d T=%d H=%d G=%d D=%d V=%d taps=%d", a->B, a->T, a->H, a->G, a->D, a->V, a->taps);
  if (a->D > kMaxD) return fail(L3CI_ERR_UNSUPPORTED, "delta_inputs: %d key channels per head, at most %d", a->D, kMaxD);
  if (a->B == 0 || a->T == 0) return L3CI_OK;
  if (!a->p || !a->a || !a->b || !a->conv || !a->a_log || !a->dt_bias || (!a->tail && a->taps > 1) || !a->positions || !a->qk_out || !a->beta_out ||
      !a->decay_out || !a->v_out)
    return fail(L3CI_ERR_INVALID, "delta_inputs: null pointer");
  const int runs = (a->T + kRun - 1) / kRun;
  const long long tasks = (long long)a->B * runs * (2 * a->G + 2 * a->H);
  if ((tasks + 7) / 8 > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "delta_inputs: too many rows");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(a->stream);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    auto on = [](const void* x, int bytes) { return (reinterpret_cast<uintptr_t>(x) & (bytes - 1)) == 0; };
    const int s4 = 4 * (int)sizeof(S);
    const bool v4 = (a->D | a->V | a->p_st | a->a_st | a->tail_sb) % 4 == 0 && on(a->p, s4) && on(a->a, s4) && on(a->tail, s4) && on(a->v_out, s4) &&
                    on(a->conv, 16) && on(a->dt_bias, 16) && on(a->qk_out, 16) && on(a->decay_out, 16);
    auto go = [&](auto kernel) -> int {
      L3CI_LAUNCH("delta_inputs_kernel", kernel, dim3((unsigned)((tasks + 7) / 8)), dim3(256), 0, s, *a, runs, tasks);
      return L3CI_OK;
    };
    if (!v4) return go(delta_inputs_kernel<S, 1, 0>);
    switch (a->taps) {
      case 1: return go(delta_inputs_kernel<S, 4, 1>);
      case 2: return go(delta_inputs_kernel<S, 4, 2>);
      case 3: return go(delta_inputs_kernel<S, 4, 3>);
      case kMaxTaps: return go(delta_inputs_kernel<S, 4, kMaxTaps>);
    }
    return go(delta_inputs_kernel<S, 4, 0>);
  };
  return a->dtype == L3CI_BF16 ? typed(__nv_bfloat16{}) : typed(float{});
}

int l3ci_recurrent_scan(const l3ci_recurrent_scan_args* a) {
  using namespace l3ci;
  clear_error();
  if (!a) return fail(L3CI_ERR_INVALID, "recurrent_scan: null args");
  if (a->B < 0 || a->T < 0 || a->H <= 0 || a->G <= 0 || a->H % a->G || a->D <= 0 || a->V <= 0 || (a->kind != 0 && a->kind != 1) ||
      (a->dtype != L3CI_BF16 && a->dtype != L3CI_F32) || (a->kind == 1 && a->G != a->H) || (a->tail && a->taps < 1))
    return fail(L3CI_ERR_INVALID, "recurrent_scan: bad size B=%d T=%d H=%d G=%d D=%d V=%d kind=%d", a->B, a->T, a->H, a->G, a->D, a->V, a->kind);
  if (a->D > kMaxD) return fail(L3CI_ERR_UNSUPPORTED, "recurrent_scan: %d key channels per head, at most %d", a->D, kMaxD);
  if (a->B == 0 || a->T == 0) return L3CI_OK;
  if (!a->q || !a->k || !a->v || !a->g || !a->state || !a->out || !a->positions || !a->norm || !a->gate || (a->kind == 0 && !a->beta) ||
      (a->kind == 1 && (!a->bonus || !a->g_bias)) || (a->tail && !a->conv_in))
    return fail(L3CI_ERR_INVALID, "recurrent_scan: null pointer");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(a->stream);
  if (a->kind == 0)
    return a->dtype == L3CI_BF16 ? scan_typed<__nv_bfloat16, float, kDelta>(a, s) : scan_typed<float, float, kDelta>(a, s);
  return a->dtype == L3CI_BF16 ? scan_typed<__nv_bfloat16, __nv_bfloat16, kTimeMix>(a, s) : scan_typed<float, float, kTimeMix>(a, s);
}

}  // extern "C"
