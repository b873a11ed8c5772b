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
// the others compute.  One token, all columns in the CTA: the head's output norm and gate are applied in place of the plain
// store; otherwise head_norm_gate_kernel does it in a pass over the output rows.
//
// delta_inputs_kernel: convolution, activation, unit norms, step sizes and decays of all tokens at once; a warp per (token,
// head) of one of q, k, v or the decay.
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

template <typename S>
__device__ __forceinline__ float4 fetch4(const S* p, int d, int D, int vec) {
  float f[4] = {0.f, 0.f, 0.f, 0.f};
  if (vec) {
    if (d < D) load_vec<S, 4>(p + d, f);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (d + e < D) f[e] = to_f32(p[d + e]);
  }
  return make_float4(f[0], f[1], f[2], f[3]);
}

// S: storage type of v, gate, out; Q: type of q, k, g.
template <typename S, typename Q, int KIND, int NR, int C, bool FUSE>
__global__ void __launch_bounds__(kScanThreads) recurrent_scan_kernel(const __grid_constant__ ScanParams p) {
  constexpr int DP = NR * 8;
  extern __shared__ __align__(16) float smem[];
  const l3ci_recurrent_scan_args& a = p.a;
  const int cols = p.cols;
  const int stage_floats = kChunk * (3 * DP + cols + 2);
  float* stages = smem;
  float* red = smem + kRing * stage_floats;                               // [kMaxConsumers]
  uint64_t* bars = reinterpret_cast<uint64_t*>(red + kMaxConsumers);
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
    for (int i = 0; i < chunks; ++i) {
      const int s = i % kRing;
      if (i >= kRing && !mbar_wait_bounded(empty0 + s * 8, ((i / kRing) - 1) & 1)) { ok = false; break; }
      float* st = stages + s * stage_floats;
      const int t0 = i * kChunk + pw * kPerProducer, n = min(kPerProducer, T - t0);
      float scalar[kPerProducer];
#pragma unroll
      for (int x = 0; x < kPerProducer; ++x) scalar[x] = 0.f;
#pragma unroll
      for (int d0 = 0; d0 < DP; d0 += 128) {
        const int d = d0 + lane * 4;
        if (d >= DP) break;
        float4 q[kPerProducer], k[kPerProducer], g[kPerProducer];
#pragma unroll
        for (int x = 0; x < kPerProducer; ++x) {
          if (x >= n) continue;
          const long long row = row0 + t0 + x;
          q[x] = fetch4<Q>(qp + row * a.qk_st, d, D, p.vec);
          k[x] = fetch4<Q>(kp + row * a.qk_st, d, D, p.vec);
          g[x] = fetch4<Q>(gp + row * a.g_st, d, D, p.vec);
        }
        float4 bonus = make_float4(1.f, 1.f, 1.f, 1.f), gb = make_float4(0.f, 0.f, 0.f, 0.f);
        if (KIND == kTimeMix) {
          bonus = fetch4<float>(a.bonus + h * D, d, D, p.vec);
          gb = fetch4<float>(a.g_bias + h * D, d, D, p.vec);
        }
#pragma unroll
        for (int x = 0; x < kPerProducer; ++x) {
          if (x >= n) continue;
          if (KIND == kTimeMix) {
            g[x].x = expf(-expf(g[x].x + gb.x));
            g[x].y = expf(-expf(g[x].y + gb.y));
            g[x].z = expf(-expf(g[x].z + gb.z));
            g[x].w = expf(-expf(g[x].w + gb.w));
          }
          scalar[x] += q[x].x * k[x].x * bonus.x + q[x].y * k[x].y * bonus.y + q[x].z * k[x].z * bonus.z + q[x].w * k[x].w * bonus.w;
          float* row = st + (pw * kPerProducer + x) * 3 * DP + d;
          *reinterpret_cast<float4*>(row) = q[x];
          *reinterpret_cast<float4*>(row + DP) = k[x];
          *reinterpret_cast<float4*>(row + 2 * DP) = g[x];
        }
      }
      float* vs = st + kChunk * 3 * DP;
      float* sc = vs + kChunk * cols;
#pragma unroll
      for (int x = 0; x < kPerProducer; ++x) {
        if (x >= n) continue;
        const int at = pw * kPerProducer + x;
        const long long row = row0 + t0 + x;
        for (int c = lane; c < cols; c += 32) vs[at * cols + c] = c < n_cols ? to_f32(vp[row * a.v_st + c]) : 0.f;
        const float sum = group_sum<kWarp>(scalar[x]);
        if (lane == 0) {
          sc[at * 2] = sum;
          sc[at * 2 + 1] = KIND == kDelta ? a.beta[row * a.H + h] : 0.f;
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(full0 + s * 8);
    }
    // the convolution's last inputs: row r of the tail becomes the input of token T - (taps - 1) + r
    if (a.tail && split == 0) {
      const int rows = a.taps - 1, GD = a.G * D;
      const long long C_all = 2LL * GD + (long long)a.H * V;
      S* tail = static_cast<S*>(a.tail) + b * a.tail_sb;
      const S* in = static_cast<const S*>(a.conv_in) + row0 * a.conv_st;
      auto move = [&](long long c) {
        for (int r = 0; r < rows; ++r) {
          const int t = T - rows + r;
          tail[r * C_all + c] = t >= 0 ? in[t * a.conv_st + c] : fresh ? from_f32<S>(0.f) : tail[(r + T) * C_all + c];
        }
      };
      for (int c = pw * 32 + lane; c < V; c += 32 * kProducers) move(2LL * GD + (long long)h * V + c);
      if (h % R == 0)
        for (int c = pw * 32 + lane; c < 2 * D; c += 32 * kProducers) move(c < D ? (h / R) * D + c : GD + (h / R) * D + c - D);
    }
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
      if (!FUSE && l == 0 && live) {
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
  if (FUSE) {
    // one token: the head's output is in this CTA (columns that do not exist are zeros)
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < C; ++c) ss = live ? fmaf(o[c], o[c], ss) : ss;
    ss = group_sum<kWarp>(l == 0 ? ss : 0.f);
    if (lane == 0) red[warp] = ss;
    asm volatile("bar.sync 1, %0;" ::"r"(32 * p.consumers) : "memory");
    ss = group_sum<kMaxConsumers>(lane % kMaxConsumers < p.consumers ? red[lane % kMaxConsumers] : 0.f);
    const float inv = 1.f / sqrtf(ss / (float)V + a.eps);
    if (l == 0 && live && ok) {
      const S* gate = static_cast<const S*>(a.gate) + b * a.gate_st + h * a.gate_sh + c0;
      S* dst = static_cast<S*>(a.out) + b * a.out_st + h * a.out_sh + c0;
#pragma unroll
      for (int c = 0; c < C; ++c)
        dst[c] = from_f32<S>(o[c] * inv * a.norm[h * a.norm_sh + c0 + c] * gate_value(to_f32(gate[c]), a.act));
    }
  }
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
constexpr int kRun = 4;            // consecutive tokens of a warp

template <typename S, int VEC>
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
    for (int x = 0; x < n; ++x) {
      const long long row = row0 + t0 + x;
      const S* src = static_cast<const S*>(a.a) + row * a.a_st + (long long)h * a.D;
      for (int c = lane * VEC; c < a.D; c += 32 * VEC) {
        float z[VEC], bias[VEC];
        load_vec<S, VEC>(src + c, z);
        load_vec<float, VEC>(a.dt_bias + (long long)h * a.D + c, bias);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          const float y = z[k] + bias[k];
          const float sp = fmaxf(y, 0.f) + log1pf(expf(-fabsf(y)));
          z[k] = expf(-rate * sp);
        }
        store_vec<float, VEC>(a.decay_out + (row * a.H + h) * a.D + c, z);
      }
      if (lane == 0) a.beta_out[row * a.H + h] = sigmoid(to_f32(static_cast<const S*>(a.b)[row * a.b_st + h]));
    }
    return;
  }
  const bool is_v = what >= 2 * a.G;
  const int size = is_v ? a.V : a.D;
  const long long ch0 = is_v ? 2LL * GD + (long long)(what - 2 * a.G) * a.V : (long long)what * a.D;
  const bool fresh = a.positions[b] == 0;
  const S* in = static_cast<const S*>(a.p) + row0 * a.p_st + ch0;
  const S* tail = static_cast<const S*>(a.tail) + b * a.tail_sb + ch0;
  for (int x = 0; x < n; ++x) {
    const int t = t0 + x;
    const long long row = row0 + t;
    auto convolve = [&](int c, float (&y)[VEC]) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) y[k] = 0.f;
      for (int i = 0; i < a.taps; ++i) {
        const int at = t - (a.taps - 1) + i;
        if (at < 0 && fresh) continue;
        float f[VEC], w[VEC];
        load_vec<S, VEC>(at >= 0 ? in + (long long)at * a.p_st + c : tail + (a.taps - 1 + at) * C_all + c, f);
        load_vec<float, VEC>(a.conv + i * C_all + ch0 + c, w);
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[k] = fmaf(f[k], w[k], y[k]);
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) y[k] *= sigmoid(y[k]);
    };
    if (is_v) {
      for (int c = lane * VEC; c < size; c += 32 * VEC) {
        float y[VEC];
        convolve(c, y);
        store_vec<S, VEC>(static_cast<S*>(a.v_out) + row * a.H * a.V + (long long)(what - 2 * a.G) * a.V + c, y);
      }
      continue;
    }
    constexpr int kKeep = VEC >= 4 ? 2 : 8;    // 256 channels
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
    float f = 1.f / sqrtf(group_sum<kWarp>(ss) + a.unit_eps);
    if (what < a.G) f /= sqrtf((float)a.D);
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int c = (i * 32 + lane) * VEC;
      if (c < size) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) y[i][k] *= f;
        store_vec<float, VEC>(a.qk_out + row * 2 * GD + ch0 + c, y[i]);
      }
    }
  }
}

constexpr int kMaxD = 256;         // key channels of a head

template <typename S, typename Q, int KIND, int NR, int C>
int launch_scan(const ScanParams& p, cudaStream_t stream) {
  const size_t smem = (size_t)kRing * kChunk * (3 * NR * 8 + p.cols + 2) * 4 + kMaxConsumers * 4 + 2 * kRing * 8;
  const dim3 grid((unsigned)((long long)p.a.B * p.a.H * p.splits)), block(32 * (p.consumers + kProducers));
  static bool configured[2][64] = {};
  auto go = [&](auto kernel, int which) -> int {
    int dev = 0;
    L3CI_CUDA_TRY(cudaGetDevice(&dev));
    if (smem > (48 << 10) && (dev < 0 || dev >= 64 || !configured[which][dev])) {
      L3CI_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem_optin()));
      if (dev >= 0 && dev < 64) configured[which][dev] = true;
    }
    L3CI_LAUNCH("recurrent_scan_kernel", kernel, grid, block, smem, stream, p);
    return L3CI_OK;
  };
  if (p.a.T == 1 && p.splits == 1) return go(recurrent_scan_kernel<S, Q, KIND, NR, C, true>, 1);
  return go(recurrent_scan_kernel<S, Q, KIND, NR, C, false>, 0);
}

template <typename S, typename Q, int KIND>
int scan_typed(const l3ci_recurrent_scan_args* a, cudaStream_t stream) {
  ScanParams p = {};
  p.a = *a;
  const long long heads = (long long)a->B * a->H;
  const int sms = sm_count() > 0 ? sm_count() : 148;
  // columns per thread: as many as one CTA per head allows for a single token (wide accesses of the state), else what leaves
  // enough CTAs for the device
  const int widest = a->V % 4 == 0 && a->state_sb % 4 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 15) == 0   ? 4
                     : a->V % 2 == 0 && a->state_sb % 2 == 0 && (reinterpret_cast<uintptr_t>(a->state) & 7) == 0 ? 2
                                                                                                                 : 1;
  int C = widest;
  if (a->T == 1) {
    const int per = 4 * C * kMaxConsumers;
    p.splits = (a->V + per - 1) / per;
    p.consumers = ((a->V + p.splits - 1) / p.splits + 4 * C - 1) / (4 * C);
  } else {
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
  }
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
  if (st || (a->T == 1 && p.splits == 1)) return st;
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
    return v4 ? go(delta_inputs_kernel<S, 4>) : go(delta_inputs_kernel<S, 1>);
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
