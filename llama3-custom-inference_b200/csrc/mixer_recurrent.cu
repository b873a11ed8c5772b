// Linear recurrences over a matrix state per (sequence, head), fp32: the gated delta rule with a decay per key channel, and
// time mixing with a bonus for the current token (include/l3ci_mixers.h).
//
// recurrent_scan_kernel: several tokens.  The columns of the state do not depend on one another, so a warp takes C columns of one
// head through all tokens of the call, the state in its registers: a lane holds NR rows of the C columns, rows two at a time
// through packed fp32 instructions.  What the tokens bring (q, k, g, v) is the same for all columns of a head; it comes
// through a ring of stages of 16 tokens in shared memory, filled by bulk tensor copies.
//   The delta rule's chain runs through S^T k, a sum over all rows.  With S'_t = g_t S_{t-1} (decayed, not yet written to),
//       S'_t^T k_t = (g_t k_t)^T S'_{t-1} + ((g_t k_t) . k_{t-1}) u_{t-1},
//   so the sum over the state that token t needs is taken of S'_{t-1}, before u_{t-1} is known, and only two
//   multiply-adds follow u_{t-1} on the way to u_t.  The scalar (g_t k_t) . k_{t-1} is the same for all columns: a helper
//   warp forms it.  Outputs are not on the chain: the lanes' shares of 32 of them (32 / C tokens of C
//   columns) meet in a patch of shared memory of the warp, after which a lane holds one output.
//   Time mixing has no chain through the sums; its helper warps form the decays.
// The head's output norm and gate follow in a pass over the output rows (head_norm_gate_kernel).
//
// recurrent_step_kernel: one token.  A CTA per head streams the state through registers, four columns and every n-th row a
// thread (whole rows per warp access), meets in shared memory for the two products, and applies norm and gate itself.
//
// delta_inputs_kernel: convolution, activation, unit norms, step sizes and decays of all tokens at once; a warp per run of
// tokens and head of one of q, k, v or the decay.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "../../include/l3ci_mixers.h"
#include "host_common.h"
#include "mixer_types.cuh"
#include "ptx_sm100.cuh"
#include "tcgen05.cuh"
#include "tensor_map.h"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kDelta = 0, kTimeMix = 1;
constexpr int kChunk = 16;         // tokens per stage
constexpr int kMaxRing = 4;        // stages
constexpr int kMaxConsumers[2] = {8, 16};   // warps, by kind
constexpr int kHelpers[2] = {1, 2};   // warps, by kind
// A warp's patch of output shares: 32 / C tokens of 32 lanes of C floats, tokens a little apart (no bank conflicts).
template <int C>
constexpr int kPatchToken = 32 * C + (C == 2 ? 4 : C == 4 ? 16 : 32);   // floats
constexpr int kPatchBytes = 8 * kPatchToken<4> * 4;
static_assert(kPatchBytes >= 4 * kPatchToken<8> * 4 && kPatchBytes >= 16 * kPatchToken<2> * 4, "a patch holds every form");

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gate_value(float z, int act) { return act == 0 ? sigmoid(z) : z * sigmoid(z); }

struct ScanParams {
  l3ci_recurrent_scan_args a;
  int splits, cols;              // column runs per head, columns per run
  int consumers;                 // warps
  int ring;                      // stages
  int bulk;                      // the tokens' rows can be fetched by bulk tensor copies
  int wide;                      // state rows allow accesses of four columns
};

// Bytes of a stage, part by part: q, k, g as they come, the decays (time mixing), v, two scalars per token.
template <typename S, typename Q, int KIND, int DP>
struct ScanStage {
  static constexpr int kQ = kChunk * DP * (int)sizeof(Q);
  static constexpr int kK = kQ, kG = kQ;
  static constexpr int kDecay = KIND == kTimeMix ? kChunk * DP * 4 : 0;
  static constexpr int kV0 = kQ + kK + kG + kDecay;
  static constexpr int kScalars = kChunk * 2 * 4;
  __host__ __device__ static constexpr int bytes(int cols) { return kV0 + kChunk * cols * (int)sizeof(S) + kScalars; }
  __host__ __device__ static constexpr int loaded(int cols) { return kQ + kK + kG + kChunk * cols * (int)sizeof(S); }
};

// NR rows of a lane as pairs: rows i * 32 * W + lane * W + e, W = min(NR, 4) neighbours.
template <typename Q, int NR>
__device__ __forceinline__ void load_rows(const Q* p, int lane, unsigned long long (&r)[NR / 2]) {
  constexpr int W = NR < 4 ? NR : 4;
#pragma unroll
  for (int i = 0; i < NR / W; ++i) {
    const Q* at = p + i * 32 * W + lane * W;
    if constexpr (sizeof(Q) == 4) {
      if constexpr (W == 4) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(at);
        r[2 * i] = x.x;
        r[2 * i + 1] = x.y;
      } else {
        r[i] = *reinterpret_cast<const unsigned long long*>(at);
      }
    } else {
#pragma unroll
      for (int e = 0; e < W / 2; ++e) {
        const uint32_t x = reinterpret_cast<const uint32_t*>(at)[e];
        r[i * (W / 2) + e] = f2_packf(bf16lo_to_f32(x), bf16hi_to_f32(x));
      }
    }
  }
}
// N neighbouring fp32 columns (2, or a multiple of 4).
template <int N>
__device__ __forceinline__ void load_cols(const float* p, float* f) {
  if constexpr (N == 2) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    f[0] = x.x; f[1] = x.y;
  } else {
#pragma unroll
    for (int c = 0; c < N; c += 4) {
      const float4 x = *reinterpret_cast<const float4*>(p + c);
      f[c] = x.x; f[c + 1] = x.y; f[c + 2] = x.z; f[c + 3] = x.w;
    }
  }
}
template <int N>
__device__ __forceinline__ void store_cols(float* p, const float* f) {
  if constexpr (N == 2) {
    *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
  } else {
#pragma unroll
    for (int c = 0; c < N; c += 4) *reinterpret_cast<float4*>(p + c) = make_float4(f[c], f[c + 1], f[c + 2], f[c + 3]);
  }
}
template <int N>
__device__ __forceinline__ float pairs_dot(const unsigned long long (&a)[N], const unsigned long long (&b)[N]) {
  unsigned long long s[2] = {0ull, 0ull};
#pragma unroll
  for (int j = 0; j < N; ++j) s[j & 1] = f2_fma(a[j], b[j], s[j & 1]);
  float x, y;
  f2_unpack(N > 1 ? f2_add(s[0], s[1]) : s[0], x, y);
  return x + y;
}

// Sums over the lanes of N values each (a power of two up to 32), halved lane by lane: the lanes of value i are i * 32 / N
// onwards, and all of them end with its sum.
template <int N>
__device__ __forceinline__ float scatter_sum(float (&v)[N], int lane) {
  int m = 16;
#pragma unroll
  for (int n = N / 2; n >= 1; n /= 2, m /= 2) {
    const bool upper = lane & m;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      if (i >= n) break;
      const float send = upper ? v[i] : v[i + n], mine = upper ? v[i + n] : v[i];
      v[i] = mine + __shfl_xor_sync(kFullMask, send, m);
    }
  }
  float r = v[0];
#pragma unroll
  for (int k = 16; k >= 1; k /= 2)
    if (k < 32 / N) r += __shfl_xor_sync(kFullMask, r, k);
  return r;
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
__global__ void __launch_bounds__(32 * (kMaxConsumers[KIND] + 1 + kHelpers[KIND]), 1)
recurrent_scan_kernel(const __grid_constant__ CUtensorMap qmap, const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap gmap,
                      const __grid_constant__ CUtensorMap vmap, const __grid_constant__ ScanParams p) {
  constexpr int DP = 32 * NR;
  using St = ScanStage<S, Q, KIND, DP>;
  constexpr int kHelp = kHelpers[KIND];
  extern __shared__ __align__(128) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 127) & ~uintptr_t(127));
  const l3ci_recurrent_scan_args& a = p.a;
  const int cols = p.cols, stage_bytes = St::bytes(cols), ring = p.ring;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + ring * stage_bytes);
  const uint32_t full0 = smem_u32(bars), ready0 = full0 + kMaxRing * 8, empty0 = ready0 + kMaxRing * 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x % p.splits, h = (blockIdx.x / p.splits) % a.H, b = blockIdx.x / (p.splits * a.H);
  const int D = a.D, V = a.V, T = a.T, R = a.H / a.G, col0 = split * cols;
  if (tid == 0) {
    for (int i = 0; i < ring; ++i) {
      mbar_init(full0 + i * 8, 1);
      mbar_init(ready0 + i * 8, kHelp);
      mbar_init(empty0 + i * 8, p.consumers);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const bool fresh = a.positions[b] == 0;
  const int chunks = (T + kChunk - 1) / kChunk;
  const long long row0 = (long long)b * T;
  bool ok = true;

  if (warp == p.consumers) {
    // ---- producer ----
    const uint64_t policy = l2_evict_first_policy();
    for (int i = 0, s = 0, phase = 1; i < chunks; ++i, s = s + 1 == ring ? 0 : s + 1, phase ^= s == 0) {
      if (i >= ring && !mbar_wait_bounded(empty0 + s * 8, phase)) { ok = false; break; }
      uint8_t* st = smem + s * stage_bytes;
      if (p.bulk) {
        if (lane == 0) {
          const uint32_t bar = full0 + s * 8, dst = smem_u32(st);
          mbar_expect_tx(bar, St::loaded(cols));
          tma_load_4d(dst, &qmap, bar, 0, i * kChunk, h / R, b, policy);
          tma_load_4d(dst + St::kQ, &kmap, bar, 0, i * kChunk, h / R, b, policy);
          tma_load_4d(dst + St::kQ + St::kK, &gmap, bar, 0, i * kChunk, h, b, policy);
          tma_load_4d(dst + St::kV0, &vmap, bar, col0, i * kChunk, h, b, policy);
        }
      } else {
        const int n = min(kChunk, T - i * kChunk);
        Q *qs = reinterpret_cast<Q*>(st), *ks = qs + kChunk * DP, *gs = ks + kChunk * DP;
        S* vs = reinterpret_cast<S*>(st + St::kV0);
        for (int x = 0; x < n; ++x) {
          const long long row = row0 + i * kChunk + x;
          for (int d = lane; d < DP; d += 32) {
            const bool in = d < D;
            qs[x * DP + d] = in ? static_cast<const Q*>(a.q)[row * a.qk_st + (h / R) * a.qk_sh + d] : from_f32<Q>(0.f);
            ks[x * DP + d] = in ? static_cast<const Q*>(a.k)[row * a.qk_st + (h / R) * a.qk_sh + d] : from_f32<Q>(0.f);
            gs[x * DP + d] = in ? static_cast<const Q*>(a.g)[row * a.g_st + h * a.g_sh + d] : from_f32<Q>(0.f);
          }
          for (int c = lane; c < cols; c += 32)
            vs[x * cols + c] = col0 + c < V ? static_cast<const S*>(a.v)[row * a.v_st + h * a.v_sh + col0 + c] : from_f32<S>(0.f);
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(full0 + s * 8);
      }
      __syncwarp();
    }
    if (a.tail && split == 0) move_tails<S>(a, b, h, lane, 32, fresh);
    if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
    return;
  }

  if (warp > p.consumers) {
    // ---- helpers ----
    const int hw = warp - p.consumers - 1;
    unsigned long long k_before[NR / 2], gb[NR / 2];
#pragma unroll
    for (int j = 0; j < NR / 2; ++j) k_before[j] = gb[j] = 0ull;
    if (KIND == kTimeMix) {
      constexpr int W = NR < 4 ? NR : 4;
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) {
        const int d = (2 * j / W) * 32 * W + lane * W + 2 * j % W;
        gb[j] = f2_packf(d < D ? a.g_bias[h * D + d] : 0.f, d + 1 < D ? a.g_bias[h * D + d + 1] : 0.f);
      }
    }
    auto step_size = [&](int i) {      // of token `lane` of chunk i
      return KIND == kDelta && lane < kChunk ? a.beta[(row0 + min(i * kChunk + lane, T - 1)) * a.H + h] : 0.f;
    };
    float beta = step_size(0);
    for (int i = 0, s = 0, phase = 0; i < chunks; ++i, s = s + 1 == ring ? 0 : s + 1, phase ^= s == 0) {
      if (!mbar_wait_bounded(full0 + s * 8, phase)) { ok = false; break; }
      uint8_t* st = smem + s * stage_bytes;
      if (KIND == kDelta) {
        const Q *ks = reinterpret_cast<const Q*>(st + St::kQ), *gs = reinterpret_cast<const Q*>(st + St::kQ + St::kK);
        float part[kChunk];
#pragma unroll
        for (int x = 0; x < kChunk; ++x) {
          unsigned long long k[NR / 2], g[NR / 2];
          load_rows<Q, NR>(ks + x * DP, lane, k);
          load_rows<Q, NR>(gs + x * DP, lane, g);
#pragma unroll
          for (int j = 0; j < NR / 2; ++j) {
            g[j] = f2_mul(g[j], k[j]);
          }
          part[x] = pairs_dot(g, k_before);
#pragma unroll
          for (int j = 0; j < NR / 2; ++j) k_before[j] = k[j];
        }
        const float sum = scatter_sum<kChunk>(part, lane);       // lanes 2 x, 2 x + 1: token x
        float* sc = reinterpret_cast<float*>(st + stage_bytes - St::kScalars);
        if (lane % 2 == 0) sc[lane + 1] = sum;
        if (lane < kChunk) sc[2 * lane] = beta;
        beta = step_size(min(i + 1, chunks - 1));
      } else {
        const Q* gs = reinterpret_cast<const Q*>(st + St::kQ + St::kK);
        float* ds = reinterpret_cast<float*>(st + St::kQ + St::kK + St::kG);
        constexpr int W = NR < 4 ? NR : 4;
#pragma unroll
        for (int x0 = 0; x0 < kChunk / kHelp; ++x0) {
          const int x = x0 * kHelp + hw;
          unsigned long long g[NR / 2];
          load_rows<Q, NR>(gs + x * DP, lane, g);
#pragma unroll
          for (int j = 0; j < NR / 2; ++j) {
            float u, v;
            f2_unpack(f2_add(g[j], gb[j]), u, v);
            *reinterpret_cast<unsigned long long*>(ds + x * DP + (2 * j / W) * 32 * W + lane * W + 2 * j % W) = f2_packf(expf(-expf(u)), expf(-expf(v)));
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(ready0 + s * 8);
    }
    if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
    return;
  }

  // ---- consumers ----
  constexpr int W = NR < 4 ? NR : 4;
  constexpr int kBlock = 32 / C;                 // tokens whose outputs are summed together
  constexpr int kShift = KIND == kDelta ? 1 : 0; // the delta rule writes a token's output while it takes the next one
  const int c_loc = warp * C, c0 = col0 + c_loc;
  float* state = a.state + b * a.state_sb + (long long)h * D * V + c0;
  const bool wide = p.wide && c0 + C <= V;
  unsigned long long A[C][NR / 2];
  auto row_of = [&](int j) { return (2 * j / W) * 32 * W + lane * W + 2 * j % W; };   // first row of pair j
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    float f[2][C];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = row_of(j) + e;
#pragma unroll
      for (int c = 0; c < C; ++c) f[e][c] = 0.f;
      if (fresh || row >= D) continue;
      const float* at = state + (long long)row * V;
      if (wide) {
        load_cols<C>(at, f[e]);
      } else {
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (c0 + c < V) f[e][c] = at[c];
      }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) A[c][j] = f2_packf(f[0][c], f[1][c]);
  }
  // carried from the token before (delta rule): k, q, its value, step size, scalar and sum over the state of this lane's
  // column, and the u of the token before that
  unsigned long long kp[NR / 2], qp[NR / 2];
  float v_p = 0.f, beta_p = 0.f, cross_p = 0.f, seen_p = 0.f, u_p = 0.f;
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) kp[j] = qp[j] = 0ull;
  unsigned long long bonus[NR / 2];
  if (KIND == kTimeMix) {
#pragma unroll
    for (int j = 0; j < NR / 2; ++j) {
      const int d = row_of(j);
      bonus[j] = f2_packf(d < D ? a.bonus[h * D + d] : 0.f, d + 1 < D ? a.bonus[h * D + d + 1] : 0.f);
    }
  }
  S* out = static_cast<S*>(a.out) + row0 * a.out_st + h * a.out_sh + c0;
  // the warp's patch: this lane's shares of the outputs, C floats per token
  float* patch = reinterpret_cast<float*>(smem + ring * stage_bytes + 3 * kMaxRing * 8 + warp * kPatchBytes);
  // (stored behind the block's last token: between the tokens the stores would hold up the loads of the next one)
  auto share = [&](int x, const float* part) {
    constexpr int kV = C < 4 ? C : 4;
#pragma unroll
    for (int c = 0; c < C; c += kV) store_cols<kV>(patch + x * kPatchToken<C> + c * 32 + lane * kV, part + c);
  };
  // the outputs of the block's n tokens from t0 on: C lanes per token sum the shares of 32 / C lanes each, all columns, and
  // then halve the columns among themselves
  auto write = [&](int t0, int n) {
    __syncwarp();
    constexpr int kV = C < 4 ? C : 4;
    const int x = lane / C, part = lane % C;
    float sums[C];
#pragma unroll
    for (int c = 0; c < C; ++c) sums[c] = 0.f;
#pragma unroll
    for (int i = 0; i < 32 / C; ++i)
#pragma unroll
      for (int c = 0; c < C; c += kV) {
        float y[kV];
        load_cols<kV>(patch + x * kPatchToken<C> + c * 32 + (i * C + part) * kV, y);
#pragma unroll
        for (int k = 0; k < kV; ++k) sums[c + k] += y[k];
      }
#pragma unroll
    for (int m = C / 2; m >= 1; m /= 2) {
      const bool upper = part & m;
#pragma unroll
      for (int c = 0; c < m; ++c) {
        const float send = upper ? sums[c] : sums[c + m], mine = upper ? sums[c + m] : sums[c];
        sums[c] = mine + __shfl_xor_sync(kFullMask, send, m);
      }
    }
    const int t = t0 + x - kShift;
    if (x < n && t >= 0 && c0 + part < V) out[t * a.out_st + part] = from_f32<S>(sums[0]);
    __syncwarp();
  };
  // u of the token before, now that its sum over the state is there: this lane's column, then every column, twice
  auto finish = [&](unsigned long long (&ub)[C]) {
    u_p = beta_p * (v_p - fmaf(cross_p, u_p, seen_p));
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const float u = __shfl_sync(kFullMask, u_p, c * (32 / C));
      ub[c] = f2_packf(u, u);
    }
  };
  // token x of the stage; part: this lane's shares of the outputs
  auto token = [&](const uint8_t* st, int x, float* part) {
    unsigned long long q[NR / 2], k[NR / 2], g[NR / 2];
    load_rows<Q, NR>(reinterpret_cast<const Q*>(st) + x * DP, lane, q);
    load_rows<Q, NR>(reinterpret_cast<const Q*>(st + St::kQ) + x * DP, lane, k);
    load_rows<float, NR>(reinterpret_cast<const float*>(st + St::kQ + St::kK + (KIND == kTimeMix ? St::kG : 0)) + x * DP, lane, g);
    const S* vs = reinterpret_cast<const S*>(st + St::kV0) + x * cols + c_loc;
    if constexpr (KIND == kDelta) {
      const float* sc = reinterpret_cast<const float*>(st + stage_bytes - St::kScalars) + 2 * x;
      unsigned long long ub[C], gk[NR / 2];
      finish(ub);
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) gk[j] = f2_mul(g[j], k[j]);
      float sums[C];
#pragma unroll
      for (int c = 0; c < C; ++c) sums[c] = pairs_dot(gk, A[c]);
      seen_p = scatter_sum<C>(sums, lane);
#pragma unroll
      for (int c = 0; c < C; ++c) {
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) A[c][j] = f2_fma(kp[j], ub[c], A[c][j]);       // S_{t-1}
        part[c] = pairs_dot(qp, A[c]);
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) A[c][j] = f2_mul(A[c][j], g[j]);               // S'_t
      }
      v_p = to_f32(vs[lane / (32 / C)]);
      beta_p = sc[0];
      cross_p = sc[1];
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) {
        kp[j] = k[j];
        qp[j] = q[j];
      }
    } else {
      unsigned long long qb[NR / 2];
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) qb[j] = f2_mul(f2_mul(q[j], bonus[j]), k[j]);
      float v[C];
      load_vec<S, C>(vs, v);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const unsigned long long v2 = f2_packf(v[c], v[c]);
        unsigned long long sum = 0ull;
#pragma unroll
        for (int j = 0; j < NR / 2; ++j) {
          sum = f2_fma(q[j], A[c][j], f2_fma(qb[j], v2, sum));
          A[c][j] = f2_fma(k[j], v2, f2_mul(A[c][j], g[j]));
        }
        float y, z;
        f2_unpack(sum, y, z);
        part[c] = y + z;
      }
    }
  };
  for (int i = 0, s = 0, phase = 0; i < chunks; ++i, s = s + 1 == ring ? 0 : s + 1, phase ^= s == 0) {
    const int n = min(kChunk, T - i * kChunk);
    if (!mbar_wait_bounded(ready0 + s * 8, phase) || !mbar_wait_bounded(full0 + s * 8, phase)) { ok = false; break; }
    const uint8_t* st = smem + s * stage_bytes;
    for (int x0 = 0; x0 < n; x0 += kBlock) {
      if (n - x0 >= kBlock) {
        float part[kBlock * C];
#pragma unroll
        for (int x = 0; x < kBlock; ++x) token(st, x0 + x, part + x * C);
#pragma unroll
        for (int x = 0; x < kBlock; ++x) share(x, part + x * C);
        write(i * kChunk + x0, kBlock);
      } else {
        for (int x = 0; x < n - x0; ++x) {
          float part[C];
          token(st, x0 + x, part);
          share(x, part);
        }
        write(i * kChunk + x0, n - x0);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(empty0 + s * 8);
  }
  if (!ok) {
    if (lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
    return;
  }
  if (KIND == kDelta) {
    // the last token's write and output
    unsigned long long ub[C];
    finish(ub);
    float part[C];
#pragma unroll
    for (int c = 0; c < C; ++c) {
#pragma unroll
      for (int j = 0; j < NR / 2; ++j) A[c][j] = f2_fma(kp[j], ub[c], A[c][j]);
      part[c] = pairs_dot(qp, A[c]);
    }
    share(0, part);
    write(T, 1);
  }
#pragma unroll
  for (int j = 0; j < NR / 2; ++j) {
    float f[2][C];
#pragma unroll
    for (int c = 0; c < C; ++c) f2_unpack(A[c][j], f[0][c], f[1][c]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = row_of(j) + e;
      if (row >= D) continue;
      float* at = state + (long long)row * V;
      if (wide) {
        store_cols<C>(at, f[e]);
      } else {
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (c0 + c < V) at[c] = f[e][c];
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

// out[row, h, :] <- out / rms(out) * norm * act(gate), in place: LANES lanes per (row, head), a vector per lane
template <typename S, int VEC, int LANES>
__global__ void __launch_bounds__(256)
head_norm_gate_vec_kernel(S* __restrict__ out, long long out_st, long long out_sh, const S* __restrict__ gate, long long gate_st,
                          long long gate_sh, const float* __restrict__ norm, long long norm_sh, int H, int V, long long units, int act, float eps) {
  pdl_wait();
  pdl_launch_dependents();
  const long long id = (long long)blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
  const int c = (threadIdx.x % LANES) * VEC;
  const bool mine = id < units && c < V;
  const long long row = units <= 0xffffffffLL ? (unsigned)id / (unsigned)H : id / H;
  const int h = (int)(id - row * H);
  float x[VEC], z[VEC], w[VEC];
#pragma unroll
  for (int k = 0; k < VEC; ++k) x[k] = 0.f;
  if (mine) {
    load_vec<S, VEC>(out + row * out_st + h * out_sh + c, x);
    load_vec<S, VEC>(gate + row * gate_st + h * gate_sh + c, z);
    load_vec<float, VEC>(norm + h * norm_sh + c, w);
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VEC; ++k) ss = fmaf(x[k], x[k], ss);
  const float inv = 1.f / sqrtf(group_sum<LANES>(ss) / (float)V + eps);
  if (!mine) return;
#pragma unroll
  for (int k = 0; k < VEC; ++k) {
    const float s = sizeof(S) == 4 ? sigmoid(z[k]) : __fdividef(1.f, 1.f + __expf(-z[k]));
    x[k] = x[k] * inv * w[k] * (act == 0 ? s : z[k] * s);
  }
  store_vec<S, VEC>(out + row * out_st + h * out_sh + c, x);
}

// The same for any size: a warp per (row, head)
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
constexpr int kRun = 8;            // consecutive tokens of a warp (one token per sequence: 1)
constexpr int kMaxTaps = 4;        // taps whose inputs stay in registers along the run

// exp(-rate * softplus(y)).  For bf16 models (y itself carries a bf16 rounding) with the short forms of exp and log; log1p(e) by
// its series where 1 + e would round e away.
template <typename S>
__device__ __forceinline__ float decay_of(float y, float rate) {
  if constexpr (sizeof(S) == 4) {
    return expf(-rate * (fmaxf(y, 0.f) + log1pf(expf(-fabsf(y)))));
  } else {
    const float e = __expf(-fabsf(y));
    const float l = e > 0.01f ? __logf(1.f + e) : e * fmaf(e, fmaf(e, 0.33333333f, -0.5f), 1.f);
    return __expf(-rate * (fmaxf(y, 0.f) + l));
  }
}

// TAPS > 0: the run's inputs are all asked for at once and every one is loaded once; 0: any number of taps.
template <typename S, int VEC, int TAPS, int RUN>
__global__ void __launch_bounds__(256, 3) delta_inputs_kernel(const l3ci_delta_inputs_args a, int runs, long long tasks) {
  pdl_wait();
  pdl_launch_dependents();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (id >= tasks) return;
  const int kinds = 2 * a.G + 2 * a.H;         // q heads, k heads, v heads, decay heads
  // neighbouring warps take neighbouring heads of the same tokens
  const int what = (int)(id % kinds);
  const long long run = id / kinds;
  const int b = (int)(run / runs), t0 = (int)(run % runs) * RUN, n = min(RUN, a.T - t0);
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
      using R = typename Raw<VEC * sizeof(S)>::type;
      R raw[RUN];
      float bias[VEC];
#pragma unroll
      for (int x = 0; x < RUN; ++x) raw[x] = *reinterpret_cast<const R*>(src + min(x, n - 1) * a.a_st + c);
      load_vec<float, VEC>(a.dt_bias + (long long)h * a.D + c, bias);
#pragma unroll
      for (int x = 0; x < RUN; ++x) {
        if (x >= n) break;
        float z[VEC];
        load_vec<S, VEC>(reinterpret_cast<const S*>(&raw[x]), z);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
          z[k] = decay_of<S>(z[k] + bias[k], rate);
        }
        store_vec<float, VEC>(a.decay_out + ((row0 + t0 + x) * a.H + h) * a.D + c, z);
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
  const float length = what < a.G ? rsqrtf((float)a.D) : 1.f;
  auto unit = [&](float ss) { return is_v ? 1.f : rsqrtf(ss + a.unit_eps) * length; };
  if (TAPS > 0 && (is_v || size <= 32 * VEC)) {
    constexpr int kTaps = TAPS > 0 ? TAPS : 1;
    for (int c = lane * VEC; c < (is_v ? size : 32 * VEC); c += 32 * VEC) {    // (every lane takes part in a unit vector's sums)
      const bool mine = c < size;
      const int at = mine ? c : 0;
      using R = typename Raw<VEC * sizeof(S)>::type;
      R raw[RUN + kTaps - 1];
      float f[RUN + kTaps - 1][VEC], w[kTaps][VEC];
      // (addresses chosen, not branches taken: every load is in flight before the first is used)
#pragma unroll
      for (int i = 0; i < RUN + kTaps - 1; ++i) {
        const int t = min(t0 - (kTaps - 1) + i, a.T - 1);
        const S* from = t >= 0 || fresh ? in + (long long)max(t, 0) * a.p_st : tail + (kTaps - 1 + t) * C_all;
        raw[i] = *reinterpret_cast<const R*>(from + at);
      }
#pragma unroll
      for (int i = 0; i < kTaps; ++i) load_vec<float, VEC>(a.conv + i * C_all + ch0 + at, w[i]);
#pragma unroll
      for (int i = 0; i < RUN + kTaps - 1; ++i) {
        load_vec<S, VEC>(reinterpret_cast<const S*>(&raw[i]), f[i]);
        if (i < kTaps - 1 && fresh && t0 - (kTaps - 1) + i < 0) {
#pragma unroll
          for (int k = 0; k < VEC; ++k) f[i][k] = 0.f;
        }
      }
#pragma unroll
      for (int x = 0; x < RUN; ++x) {
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
int launch_scan(ScanParams p, cudaStream_t stream) {
  constexpr int DP = 32 * NR;
  using St = ScanStage<S, Q, KIND, DP>;
  const l3ci_recurrent_scan_args& a = p.a;
  const size_t fixed = 128 + 3 * kMaxRing * 8 + (size_t)p.consumers * kPatchBytes;
  p.ring = (int)((max_smem_optin() - fixed) / St::bytes(p.cols));
  if (p.ring > kMaxRing) p.ring = kMaxRing;
  if (p.ring < 1) return fail(L3CI_ERR_UNSUPPORTED, "recurrent_scan: D=%d V=%d", a.D, a.V);
  const size_t smem = fixed + (size_t)p.ring * St::bytes(p.cols);
  static bool configured[64] = {false};
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(recurrent_scan_kernel<S, Q, KIND, NR, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem_optin()));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  CUtensorMap q = {}, k = {}, g = {}, v = {};
  if (p.bulk) {
    if (int st = make_box_map(&q, a.q, sizeof(Q), a.D, a.T, a.G, a.B, a.qk_st, a.qk_sh, a.T * a.qk_st, DP, kChunk)) return st;
    if (int st = make_box_map(&k, a.k, sizeof(Q), a.D, a.T, a.G, a.B, a.qk_st, a.qk_sh, a.T * a.qk_st, DP, kChunk)) return st;
    if (int st = make_box_map(&g, a.g, sizeof(Q), a.D, a.T, a.H, a.B, a.g_st, a.g_sh, a.T * a.g_st, DP, kChunk)) return st;
    if (int st = make_box_map(&v, a.v, sizeof(S), a.V, a.T, a.H, a.B, a.v_st, a.v_sh, a.T * a.v_st, p.cols, kChunk)) return st;
  }
  L3CI_LAUNCH("recurrent_scan_kernel", recurrent_scan_kernel<S, Q, KIND, NR, C>, dim3((unsigned)((long long)a.B * a.H * p.splits)),
              dim3(32 * (p.consumers + 1 + kHelpers[KIND])), smem, stream, q, k, g, v, p);
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
  p.wide = a->V % 4 == 0 && a->state_sb % 4 == 0 && aligned16(a->state);
  // rows the copy engine can address: whole 16-byte vectors
  auto rows16 = [](const void* x, size_t size, int64_t st, int64_t sh) { return aligned16(x) && st > 0 && sh > 0 && (st * size) % 16 == 0 && (sh * size) % 16 == 0; };
  p.bulk = rows16(a->q, sizeof(Q), a->qk_st, a->qk_sh) && rows16(a->k, sizeof(Q), a->qk_st, a->qk_sh) && rows16(a->g, sizeof(Q), a->g_st, a->g_sh) &&
           rows16(a->v, sizeof(S), a->v_st, a->v_sh);
  // columns per warp and warps per CTA: as many as leave enough CTAs for the device
  // (the delta rule wants the registers, time mixing the warps)
  const struct { int C, W; } by_kind[2][4] = {{{8, 8}, {8, 4}, {2, 8}, {2, 4}}, {{4, 16}, {4, 8}, {2, 8}, {2, 4}}};
  int C = 4;
  for (const auto& s : by_kind[KIND]) {
    C = s.C;
    p.consumers = s.W;
    p.cols = C * s.W;
    p.splits = (a->V + p.cols - 1) / p.cols;
    if (p.cols < 2 * a->V && heads * p.splits * 5 >= 4LL * sms) break;
  }
  if (heads * p.splits > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "recurrent_scan: too many sequences");
  auto on = [](const void* x, int bytes) { return (reinterpret_cast<uintptr_t>(x) & (bytes - 1)) == 0; };
  int st;
  auto by_rows = [&](auto c) -> int {
    constexpr int CC = decltype(c)::value;
    return a->D <= 64 ? launch_scan<S, Q, KIND, 2, CC>(p, stream) : a->D <= 128 ? launch_scan<S, Q, KIND, 4, CC>(p, stream)
                                                                              : launch_scan<S, Q, KIND, 8, CC>(p, stream);
  };
  st = C == 2 ? by_rows(std::integral_constant<int, 2>{}) : by_rows(std::integral_constant<int, KIND == kDelta ? 8 : 4>{});
  if (st) return st;
  // norm and gate of the rows the scan has written
  const long long units = heads * a->T;
  if ((units + 7) / 8 > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "recurrent_scan: too many rows");
  auto go = [&](auto kernel, int per_cta) -> int {
    L3CI_LAUNCH("head_norm_gate_kernel", kernel, dim3((unsigned)((units + per_cta - 1) / per_cta)), dim3(256), 0, stream, static_cast<S*>(a->out),
                (long long)a->out_st, (long long)a->out_sh, static_cast<const S*>(a->gate), (long long)a->gate_st, (long long)a->gate_sh,
                a->norm, (long long)a->norm_sh, a->H, a->V, units, a->act, a->eps);
    return L3CI_OK;
  };
  constexpr int kVec = 16 / sizeof(S);
  const bool vec = (a->V | a->out_st | a->out_sh | a->gate_st | a->gate_sh | a->norm_sh) % kVec == 0 && aligned16(a->out) && aligned16(a->gate) &&
                   aligned16(a->norm);
  if (vec && a->V <= 8 * kVec) return go(head_norm_gate_vec_kernel<S, kVec, 8>, 32);
  if (vec && a->V <= 16 * kVec) return go(head_norm_gate_vec_kernel<S, kVec, 16>, 16);
  if (vec && a->V <= 32 * kVec) return go(head_norm_gate_vec_kernel<S, kVec, 32>, 8);
  return go(head_norm_gate_kernel<S, 1>, 8);
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
  const int run = a->T == 1 ? 1 : kRun, runs = (a->T + run - 1) / run;
  const long long tasks = (long long)a->B * runs * (2 * a->G + 2 * a->H);
  if ((tasks + 7) / 8 > 0x7fffffffLL) return fail(L3CI_ERR_INVALID, "delta_inputs: too many rows");
  cudaStream_t s = reinterpret_cast<cudaStream_t>(a->stream);
  auto typed = [&](auto zero) -> int {
    using S = decltype(zero);
    auto on = [](const void* x, int bytes) { return (reinterpret_cast<uintptr_t>(x) & (bytes - 1)) == 0; };
    const int s4 = 4 * (int)sizeof(S);
    const bool v4 = (a->D | a->V | a->p_st | a->a_st | a->tail_sb) % 4 == 0 && on(a->p, s4) && on(a->a, s4) && on(a->tail, s4) && on(a->v_out, s4) &&
                    on(a->conv, 16) && on(a->dt_bias, 16) && on(a->qk_out, 16) && on(a->decay_out, 16);
    auto go = [&](auto one, auto many) -> int {
      L3CI_LAUNCH("delta_inputs_kernel", run == 1 ? one : many, dim3((unsigned)((tasks + 7) / 8)), dim3(256), 0, s, *a, runs, tasks);
      return L3CI_OK;
    };
    if (!v4) return go(delta_inputs_kernel<S, 1, 0, 1>, delta_inputs_kernel<S, 1, 0, kRun>);
    switch (a->taps) {
      case 1: return go(delta_inputs_kernel<S, 4, 1, 1>, delta_inputs_kernel<S, 4, 1, kRun>);
      case 2: return go(delta_inputs_kernel<S, 4, 2, 1>, delta_inputs_kernel<S, 4, 2, kRun>);
      case 3: return go(delta_inputs_kernel<S, 4, 3, 1>, delta_inputs_kernel<S, 4, 3, kRun>);
      case kMaxTaps: return go(delta_inputs_kernel<S, 4, kMaxTaps, 1>, delta_inputs_kernel<S, 4, kMaxTaps, kRun>);
    }
    return go(delta_inputs_kernel<S, 4, 0, 1>, delta_inputs_kernel<S, 4, 0, kRun>);
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
