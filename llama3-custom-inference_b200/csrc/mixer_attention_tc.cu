// Prefill attention of the mixers on the 5th-generation tensor cores: 128 query rows per tile, tcgen05.mma with operands
// in shared memory (bulk tensor copies, 128-byte swizzle) or tensor memory, accumulators in tensor memory.  The
// machinery (roles, barriers, lazy reference maximum, P over S, register re-deal) is that of prefill_attention_tc.cu.
//
// mixer_tc_kernel<KA, KB, VC, BIAS>: one map; a query / key vector is two parts (KA and KB boxes of 64 columns, zero-filled
//   where a part ends), which come from their own tensors: expanded latent attention reads its unrotated keys from the
//   expansion and the rotated part, shared by the heads, from the cache.  One head per CTA, the two softmax groups take
//   the even and the odd key tiles and merge at the end.  A window (with kept first keys) skips the tiles no row sees; BIAS
//   takes a head's distance bias off the scores; a sink is a first score of 0 without a value.
// mixer_tc_maps_kernel<VC, CAP>: differential attention.  Softmax group e owns map e of a head (its own Q, K, S_e, O_e;
//   the value tile is loaded once), a persistent grid walks the (head, query block) items longest first, and the output
//   warpgroup, whose thread holds a row of both maps' outputs, forms the difference, its root mean square over the row
//   and the gate before it writes.  The query temperature is a factor of a thread's row; the soft cap is an odd
//   polynomial of the raw score while a row's scores stay within its range, the exact form otherwise.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "bf16x8.cuh"
#include "mixer_attention.h"
#include "ptx_sm100.cuh"
#include "tcgen05.cuh"
#include "tensor_map.h"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kRows = 128;                       // query rows per tile (M of the MMA)
constexpr int kKeys = 128;                       // keys per tile (N of S, K of P V)
constexpr int kStages = 2;
constexpr int kBox = 128 * 128;                  // 128 rows of 64 columns
constexpr int kSoftmaxWarps = 8;                 // two groups of four
constexpr int kOneThreads = 32 * (4 + kSoftmaxWarps);
constexpr int kOneRegsLow = 56, kOneRegsHigh = 224;
static_assert(4 * kOneRegsLow + kSoftmaxWarps * kOneRegsHigh <= 12 * 168, "the re-deal stays within the CTA's registers");
constexpr int kMapsThreads = kOneThreads + 128;  // + the output warpgroup
constexpr int kMapsRegsLow = 56, kMapsRegsHigh = 192, kMapsRegsOut = 72;
static_assert(4 * kMapsRegsLow + kSoftmaxWarps * kMapsRegsHigh + 4 * kMapsRegsOut <= 16 * 128, "register re-deal");
constexpr uint32_t kTmem = 512;                  // S_0, S_1 (128 columns each), O_0, O_1
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kLazy = 8.f;                     // log2 of how far the running maximum may outgrow the reference maximum
constexpr int kOutPitch = 64 + 16;               // staging row of mixer_tc_maps_kernel: 32 output columns + padding

struct TcMixParams {
  l3ci_mixer_attn_args a;
  int R, m_blocks, n_keys;
  int shared_b;                                  // the second key part has one head
};

__device__ __forceinline__ void prefetch_map(const CUtensorMap* m) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(m)) : "memory");
}

// O (columns of this thread's row) *= alpha, in tensor memory
template <int COLS>
__device__ __forceinline__ void rescale_row(uint32_t to, float alpha) {
#pragma unroll
  for (int c = 0; c < COLS / 32; ++c) {
    uint32_t y[32];
    tmem_ld32(to + c * 32, y);
    tc_wait_ld();
    uint32_t lo[16], hi[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      lo[i] = __float_as_uint(__uint_as_float(y[i]) * alpha);
      hi[i] = __float_as_uint(__uint_as_float(y[16 + i]) * alpha);
    }
    tmem_st16(to + c * 32, lo);
    tmem_st16(to + c * 32 + 16, hi);
  }
}

// tanh(y), |error| about 1e-7
__device__ __forceinline__ float tanh_exact(float y) { return 1.f - __fdividef(2.f, 1.f + fast_exp2(2.f * kLog2e * y)); }
// tanh(y) / y as a polynomial of y^2 for |y| <= kPolyRange: least squares with reweighting towards the minimax fit,
// relative error below 3e-7
constexpr float kPolyRange = 0.7f;
__device__ constexpr float kPoly[5] = {0.999999718f, -0.333303491f, 0.132824955f, -0.0508812513f, 0.0138195432f};

// ---------------------------------------------------------------------------------------------------------------
template <int KA, int KB, int VC, bool BIAS>
__global__ void __launch_bounds__(kOneThreads, 1)
mixer_tc_kernel(const __grid_constant__ CUtensorMap qamap, const __grid_constant__ CUtensorMap qbmap,
                const __grid_constant__ CUtensorMap kamap, const __grid_constant__ CUtensorMap kbmap,
                const __grid_constant__ CUtensorMap vmap, const __grid_constant__ TcMixParams p) {
  constexpr int kQBytes = (KA + KB) * kBox, kVBytes = VC * kBox, D = VC * 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t q_smem = smem_u32(smem);
  const uint32_t k_smem = q_smem + kQBytes;                    // [kStages]
  const uint32_t v_smem = k_smem + kStages * kQBytes;          // [kStages]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (1 + kStages) * kQBytes + kStages * kVBytes);
  enum { Q_FULL = 0, K_FULL = 1, K_EMPTY = 3, V_FULL = 5, V_EMPTY = 7, S_FULL = 9, P_FULL = 11, O_FULL = 13, N_BARS = 15 };
  float* xchg = reinterpret_cast<float*>(bars + N_BARS);       // [2 groups][128 rows][m_ref, l]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(xchg + 4 * kRows);
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const l3ci_mixer_attn_args& a = p.a;

  if (threadIdx.x == 0) {
    for (int i = 0; i < N_BARS; ++i) mbar_init(bar(i), (i == P_FULL || i == P_FULL + 1) ? kSoftmaxWarps / 2 : 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    prefetch_map(&qamap);
    prefetch_map(&kamap);
    prefetch_map(&vmap);
    if (KB) {
      prefetch_map(&qbmap);
      prefetch_map(&kbmap);
    }
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), kTmem);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t t_s[2] = {tmem, tmem + 128u};
  const uint32_t t_o[2] = {tmem + 256u, tmem + 256u + (uint32_t)D};

  // longest query blocks first over the whole launch
  const int heads_all = a.H * a.B;
  const int mb = p.m_blocks - 1 - (int)(blockIdx.x / heads_all);
  const int hq = (int)(blockIdx.x % heads_all) % a.H;
  const int b = (int)(blockIdx.x % heads_all) / a.H;
  const int hkv = hq / p.R;
  const int m0 = mb * kRows;
  const int keys = min(p.n_keys, a.start_pos + min(m0 + kRows, a.T));
  // key tiles in sight of any row: those of the kept first keys, then from the first row's window on
  const int w_tile = window_start(a.start_pos + m0, a.window) / kKeys;
  const int kept_tiles = min(w_tile, (a.keep_first + kKeys - 1) / kKeys), skipped = w_tile - kept_tiles;
  const int n_tiles = (keys + kKeys - 1) / kKeys - skipped;
  auto first_key = [&](int j) { return (j + (j >= kept_tiles ? skipped : 0)) * kKeys; };   // of tile j
  bool ok = true;

  if (warp == 0) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kOneRegsLow));
    // ---- producer ----
    const uint64_t policy = l2_evict_first_policy();
    auto load_k = [&](uint32_t dst, uint32_t bar_, int j) {
#pragma unroll
      for (int c = 0; c < KA; ++c) tma_load_4d(dst + c * kBox, &kamap, bar_, c * 64, first_key(j), hkv, b, policy);
#pragma unroll
      for (int c = 0; c < KB; ++c) tma_load_4d(dst + (KA + c) * kBox, &kbmap, bar_, c * 64, first_key(j), p.shared_b ? 0 : hkv, b, policy);
    };
    if (lane == 0) {
      mbar_expect_tx(bar(Q_FULL), kQBytes);
#pragma unroll
      for (int c = 0; c < KA; ++c) tma_load_4d(q_smem + c * kBox, &qamap, bar(Q_FULL), c * 64, m0, hq, b, policy);
#pragma unroll
      for (int c = 0; c < KB; ++c) tma_load_4d(q_smem + (KA + c) * kBox, &qbmap, bar(Q_FULL), c * 64, m0, hq, b, policy);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int s = j % kStages;
      const uint32_t par = ((j / kStages) - 1) & 1;
      if (j >= kStages && !mbar_wait_bounded(bar(K_EMPTY + s), par)) { ok = false; break; }
      if (lane == 0) {
        mbar_expect_tx(bar(K_FULL + s), kQBytes);
        load_k(k_smem + s * kQBytes, bar(K_FULL + s), j);
      }
      if (j >= kStages && !mbar_wait_bounded(bar(V_EMPTY + s), par)) { ok = false; break; }
      if (lane == 0) {
        mbar_expect_tx(bar(V_FULL + s), kVBytes);
#pragma unroll
        for (int c = 0; c < VC; ++c) tma_load_4d(v_smem + s * kVBytes + c * kBox, &vmap, bar(V_FULL + s), c * 64, first_key(j), hkv, b, policy);
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kOneRegsLow));
    // ---- MMA issue: all lanes run the code, one elected lane predicates the instructions ----
    constexpr uint32_t idesc_qk = instr_desc(kRows, kKeys, false);
    constexpr uint32_t idesc_pv = instr_desc(kRows, D, true);
    const uint32_t elected = lane == 0 ? 1u : 0u;
    const uint64_t q_desc = smem_desc(q_smem, 16, 1024);
    const uint64_t k_desc = smem_desc(k_smem, 16, 1024);
    const uint64_t v_desc = smem_desc(v_smem, kBox, 1024);
    auto issue_s = [&](int j) {
      const int s = j % kStages;
      const uint64_t kd = k_desc + (uint64_t)((s * kQBytes) >> 4);
#pragma unroll
      for (int ks = 0; ks < (KA + KB) * 4; ++ks) {
        const uint64_t step = (uint64_t)(((ks >> 2) * kBox + (ks & 3) * 32) / 16);
        mma_ss(t_s[j & 1], q_desc + step, kd + step, idesc_qk, ks > 0, elected);
      }
      tc_commit(bar(S_FULL + (j & 1)), elected);
      tc_commit(bar(K_EMPTY + s), elected);
    };
    if (!mbar_wait_bounded(bar(Q_FULL), 0)) ok = false;
    if (ok && !mbar_wait_bounded(bar(K_FULL), 0)) ok = false;
    if (ok) {
      tc_fence_after();
      issue_s(0);
    }
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int s = j % kStages;
      if (j + 1 < n_tiles) {
        if (!mbar_wait_bounded(bar(K_FULL + (j + 1) % kStages), ((j + 1) / kStages) & 1)) { ok = false; break; }
        tc_fence_after();
        issue_s(j + 1);
      }
      if (!mbar_wait_bounded(bar(P_FULL + (j & 1)), (j >> 1) & 1)) { ok = false; break; }
      if (!mbar_wait_bounded(bar(V_FULL + s), (j / kStages) & 1)) { ok = false; break; }
      tc_fence_after();
      const uint64_t vd = v_desc + (uint64_t)((s * kVBytes) >> 4);
#pragma unroll
      for (int kk = 0; kk < kKeys / 16; ++kk)
        mma_ts(t_o[j & 1], t_s[j & 1] + kk * 8, vd + (uint64_t)(kk * 128), idesc_pv, (j > 1 || kk > 0) ? 1u : 0u, elected);
      tc_commit(bar(O_FULL + (j & 1)), elected);
      tc_commit(bar(V_EMPTY + s), elected);
    }
  } else if (warp >= 4) {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kOneRegsHigh));
    // ---- softmax and output: group e = tiles j % 2 == e; thread owns query row r of its group's tiles ----
    const int q4 = warp & 3;
    const int e = (warp - 4) >> 2;
    const int r = q4 * 32 + lane;
    const int limit = a.start_pos + m0 + r;        // last key this row sees
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const uint32_t ts = t_s[e] + lane_addr, to = t_o[e] + lane_addr;
    const float scale_log2e = a.scale * kLog2e;
    const float slope = BIAS ? head_slope(a.bias_range, hq, a.H) * kLog2e : 0.f;
    const int row_lo = window_start(limit, a.window);
    // the sink is a score of 0 that the first group has seen before its first tile
    float m_ref = a.sink && e == 0 ? 0.f : -INFINITY, l_run = a.sink && e == 0 ? 1.f : 0.f;
    int done = 0;
    for (int j = e; j < n_tiles && ok; j += 2, ++done) {
      if (!mbar_wait_bounded(bar(S_FULL + e), done & 1)) { ok = false; break; }
      tc_fence_after();
      const int j0 = first_key(j);
      // a tile that every row sees whole needs no mask
      const bool edge = j0 + kKeys - 1 > a.start_pos + m0 || j0 + kKeys > p.n_keys ||
                        (j0 < window_start(a.start_pos + m0 + kRows - 1, a.window) && j0 + kKeys > a.keep_first);
      uint32_t x[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(ts + c * 32, x[c]);
      tc_wait_ld();
      if (edge) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int key = j0 + c * 32 + i;
            if (key > limit || key >= p.n_keys || (key < row_lo && key >= a.keep_first)) x[c][i] = 0xff800000u;  // -inf
          }
      }
      if (BIAS) {
        // scores in the log2 domain with the distance taken off: slope * (i - (limit - j0)) for key j0 + i
        const float base = slope * (float)(j0 - limit);
        const unsigned long long sc2 = f2_packf(scale_log2e, scale_log2e), slope2 = f2_packf(slope, slope), base2 = f2_packf(base, base);
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float t0, t1;
            f2_unpack(f2_fma(f2_pack(x[c][i], x[c][i + 1]), sc2, f2_fma(f2_packf((float)(c * 32 + i), (float)(c * 32 + i + 1)), slope2, base2)), t0, t1);
            x[c][i] = __float_as_uint(t0);
            x[c][i + 1] = __float_as_uint(t1);
          }
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; i += 2)
          mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], __uint_as_float(x[c][i]), __uint_as_float(x[c][i + 1]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * (BIAS ? 1.f : scale_log2e);
      if (__any_sync(kFullMask, mx > m_ref + kLazy)) {
        const float m_new = fmaxf(m_ref, mx);
        const float alpha = m_new == -INFINITY ? 1.f : fast_exp2(m_ref - m_new);
        if (done > 0) {
          if (!mbar_wait_bounded(bar(O_FULL + e), (done - 1) & 1)) { ok = false; break; }
          tc_fence_after();
          rescale_row<D>(to, alpha);
        }
        l_run *= alpha;
        m_ref = m_new;
      }
      const float mu = m_ref == -INFINITY ? 0.f : m_ref;
      const unsigned long long scale2 = f2_packf(BIAS ? 1.f : scale_log2e, BIAS ? 1.f : scale_log2e), nmu2 = f2_packf(-mu, -mu);
      unsigned long long ps2[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
        unsigned long long t2[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) t2[i] = f2_fma(f2_pack(x[c][2 * i], x[c][2 * i + 1]), scale2, nmu2);
        float pe[32];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          float t0, t1;
          f2_unpack(t2[i], t0, t1);
          pe[2 * i] = fast_exp2(t0);
          pe[2 * i + 1] = fast_exp2(t1);
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          ps2[i & 3] = f2_add(ps2[i & 3], f2_packf(pe[2 * i], pe[2 * i + 1]));
          pk[i] = pack_bf16x2(pe[2 * i], pe[2 * i + 1]);
        }
        tmem_st16(ts + c * 16, pk);
      }
      float a0, a1, b0, b1;
      f2_unpack(f2_add(ps2[0], ps2[1]), a0, a1);
      f2_unpack(f2_add(ps2[2], ps2[3]), b0, b1);
      l_run += (a0 + a1) + (b0 + b1);
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(P_FULL + e));
    }
    if (ok && done > 0 && !mbar_wait_bounded(bar(O_FULL + e), (done - 1) & 1)) ok = false;
    tc_fence_after();
    // merge the two groups' partial results of a row; each of its two threads writes one half of the output columns
    xchg[(e * kRows + r) * 2] = m_ref;
    xchg[(e * kRows + r) * 2 + 1] = l_run;
    asm volatile("bar.sync 1, %0;" ::"r"(32 * kSoftmaxWarps) : "memory");
    const float m_other = xchg[((e ^ 1) * kRows + r) * 2], l_other = xchg[((e ^ 1) * kRows + r) * 2 + 1];
    const float m_all = fmaxf(m_ref, m_other);
    const float a_me = m_ref == -INFINITY ? 0.f : fast_exp2(m_ref - m_all);
    const float a_ot = m_other == -INFINITY ? 0.f : fast_exp2(m_other - m_all);
    const float l_all = l_run * a_me + l_other * a_ot;
    const float inv = l_all > 0.f ? 1.f / l_all : 0.f;
    constexpr int kHalf = D / 2;
    const bool any_me = __any_sync(kFullMask, a_me != 0.f), any_ot = __any_sync(kFullMask, a_ot != 0.f);
    // through the K and V stages, which are free: both groups have seen their last product complete
    constexpr int kPitch = D * 2 + 16;
    static_assert(kRows * kPitch <= kStages * (kQBytes + kVBytes), "output staging fits the stages");
    uint8_t* stage = smem + kQBytes;
#pragma unroll
    for (int c = 0; c < kHalf / 32; ++c) {
      uint32_t y0[32], y1[32];
      // (a group without tiles never wrote its accumulator: its columns are not read, let alone used)
      if (any_me) tmem_ld32(t_o[e] + lane_addr + e * kHalf + c * 32, y0);
      if (any_ot) tmem_ld32(t_o[e ^ 1] + lane_addr + e * kHalf + c * 32, y1);
      tc_wait_ld();
      uint32_t w[16];
#pragma unroll
      for (int i = 0; i < 32; i += 2) {
        float v0 = 0.f, v1 = 0.f;
        if (a_me != 0.f) {
          v0 = __uint_as_float(y0[i]) * a_me;
          v1 = __uint_as_float(y0[i + 1]) * a_me;
        }
        if (a_ot != 0.f) {
          v0 = fmaf(__uint_as_float(y1[i]), a_ot, v0);
          v1 = fmaf(__uint_as_float(y1[i + 1]), a_ot, v1);
        }
        w[i >> 1] = pack_bf16x2(v0 * inv, v1 * inv);
      }
      uint4* dst = reinterpret_cast<uint4*>(stage + r * kPitch + (e * kHalf + c * 32) * 2);
#pragma unroll
      for (int q = 0; q < 4; ++q) dst[q] = make_uint4(w[4 * q], w[4 * q + 1], w[4 * q + 2], w[4 * q + 3]);
    }
    asm volatile("bar.sync 1, %0;" ::"r"(32 * kSoftmaxWarps) : "memory");
    constexpr int kChunks = D * 2 / 16;
    const int sidx = (int)threadIdx.x - 128;
    __nv_bfloat16* obase = static_cast<__nv_bfloat16*>(a.out) + b * a.o_sb + hq * a.o_sh;
    for (int id = sidx; id < kRows * kChunks; id += 32 * kSoftmaxWarps) {
      const int row = id / kChunks, ch = id % kChunks;
      if (m0 + row < a.T && ch * 8 < a.Dv)
        *reinterpret_cast<uint4*>(obase + (m0 + row) * a.o_st + ch * 8) = *reinterpret_cast<const uint4*>(stage + row * kPitch + ch * 16);
    }
  } else {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kOneRegsLow));   // the two idle warps of the first warpgroup
  }
  if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, kTmem);
}

// ---------------------------------------------------------------------------------------------------------------
template <int VC, bool CAP>
__global__ void __launch_bounds__(kMapsThreads, 1)
mixer_tc_maps_kernel(const __grid_constant__ CUtensorMap q0map, const __grid_constant__ CUtensorMap q1map,
                     const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap,
                     const __grid_constant__ TcMixParams p) {
  constexpr int kVBytes = VC * kBox, D = VC * 64;
  constexpr int kKBytes = 2 * kBox;                            // both maps' boxes
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t q_smem = smem_u32(smem);                      // [2 maps]
  const uint32_t k_smem = q_smem + 2 * kBox;                   // [kStages][2 maps]
  const uint32_t v_smem = k_smem + kStages * kKBytes;          // [kStages]
  uint8_t* stage = smem + 2 * kBox + kStages * (kKBytes + kVBytes);   // [128 rows][kOutPitch]
  uint64_t* bars = reinterpret_cast<uint64_t*>(stage + kRows * kOutPitch);
  // Q_EMPTY: the item's last scores have been computed; L_FULL: a map's row sums are in shared memory; O_READ: the output
  // warpgroup has the map's O (the accumulator may take the next item's products)
  enum { Q_FULL = 0, K_FULL = 1, K_EMPTY = 3, V_FULL = 5, V_EMPTY = 7, S_FULL = 9, P_FULL = 11, O_FULL = 13, Q_EMPTY = 15,
         L_FULL = 16, O_READ = 18, N_BARS = 20 };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + N_BARS);
  float* lrow = reinterpret_cast<float*>(bars + N_BARS + 2);   // [2 maps][128 rows]
  const uint32_t bar0 = smem_u32(bars);
  auto bar = [&](int i) { return bar0 + 8u * i; };
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const l3ci_mixer_attn_args& a = p.a;

  if (threadIdx.x == 0) {
    for (int i = 0; i < N_BARS; ++i) mbar_init(bar(i), (i == P_FULL || i == P_FULL + 1 || i >= L_FULL) ? kSoftmaxWarps / 2 : 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    prefetch_map(&q0map);
    prefetch_map(&q1map);
    prefetch_map(&kmap);
    prefetch_map(&vmap);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), kTmem);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t t_s[2] = {tmem, tmem + 128u};
  const uint32_t t_o[2] = {tmem + 256u, tmem + 256u + (uint32_t)D};

  // items (head, query block): longest query blocks first, dealt in snake order over the CTAs
  const int heads_all = a.H * a.B;
  const long long n_items = (long long)heads_all * p.m_blocks;
  struct Item { int hq, b, hkv, m0, n_tiles; bool valid; };
  auto item_of = [&](int round) {
    Item it;
    const long long idx = (long long)round * gridDim.x + ((round & 1) ? gridDim.x - 1 - blockIdx.x : blockIdx.x);
    it.valid = idx < n_items;
    const int mb = p.m_blocks - 1 - (int)(idx / heads_all);
    it.hq = (int)(idx % heads_all) % a.H;
    it.b = (int)(idx % heads_all) / a.H;
    it.hkv = it.hq / p.R;
    it.m0 = mb * kRows;
    const int keys = min(p.n_keys, a.start_pos + min(it.m0 + kRows, a.T));
    it.n_tiles = (keys + kKeys - 1) / kKeys;
    return it;
  };
  bool ok = true;

  if (warp == 0) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kMapsRegsLow));
    // ---- producer ----
    const uint64_t policy = l2_evict_first_policy();
    int fill = 0;
    for (int round = 0; ok; ++round) {
      const Item it = item_of(round);
      if (!it.valid) break;
      if (round > 0 && !mbar_wait_bounded(bar(Q_EMPTY), (round - 1) & 1)) { ok = false; break; }
      if (lane == 0) {
        mbar_expect_tx(bar(Q_FULL), 2 * kBox);
        tma_load_4d(q_smem, &q0map, bar(Q_FULL), 0, it.m0, it.hq, it.b, policy);
        tma_load_4d(q_smem + kBox, &q1map, bar(Q_FULL), 0, it.m0, it.hq, it.b, policy);
      }
      for (int j = 0; j < it.n_tiles && ok; ++j, ++fill) {
        const int s = fill % kStages;
        const uint32_t par = ((fill / kStages) - 1) & 1;
        if (fill >= kStages && !mbar_wait_bounded(bar(K_EMPTY + s), par)) { ok = false; break; }
        if (lane == 0) {
          mbar_expect_tx(bar(K_FULL + s), kKBytes);
#pragma unroll
          for (int e = 0; e < 2; ++e)
            tma_load_4d(k_smem + s * kKBytes + e * kBox, &kmap, bar(K_FULL + s), e * a.Da, j * kKeys, it.hkv, it.b, policy);
        }
        if (fill >= kStages && !mbar_wait_bounded(bar(V_EMPTY + s), par)) { ok = false; break; }
        if (lane == 0) {
          mbar_expect_tx(bar(V_FULL + s), kVBytes);
#pragma unroll
          for (int c = 0; c < VC; ++c)
            tma_load_4d(v_smem + s * kVBytes + c * kBox, &vmap, bar(V_FULL + s), c * 64, j * kKeys, it.hkv, it.b, policy);
        }
        __syncwarp();
      }
    }
  } else if (warp == 1) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kMapsRegsLow));
    // ---- MMA issue ----
    constexpr uint32_t idesc_qk = instr_desc(kRows, kKeys, false);
    constexpr uint32_t idesc_pv = instr_desc(kRows, D, true);
    const uint32_t elected = lane == 0 ? 1u : 0u;
    const uint64_t q_desc = smem_desc(q_smem, 16, 1024);
    const uint64_t k_desc = smem_desc(k_smem, 16, 1024);
    const uint64_t v_desc = smem_desc(v_smem, kBox, 1024);
    // S_{e,g} = Q_e K_e^T (g: tile number over all items) into map e's score accumulator, which held P_{e,g-1}
    auto issue_s = [&](int e, int g, bool last) {
      const int s = g % kStages;
      const uint64_t qd = q_desc + (uint64_t)((e * kBox) >> 4);
      const uint64_t kd = k_desc + (uint64_t)((s * kKBytes + e * kBox) >> 4);
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) mma_ss(t_s[e], qd + ks * 2, kd + ks * 2, idesc_qk, ks > 0, elected);
      tc_commit(bar(S_FULL + e), elected);
      if (e == 1) {
        tc_commit(bar(K_EMPTY + s), elected);
        if (last) tc_commit(bar(Q_EMPTY), elected);
      }
    };
    int g0 = 0;
    for (int round = 0; ok; ++round) {
      const Item it = item_of(round);
      if (!it.valid) break;
      const int n_tiles = it.n_tiles;
      if (!mbar_wait_bounded(bar(Q_FULL), round & 1)) { ok = false; break; }
      if (!mbar_wait_bounded(bar(K_FULL + g0 % kStages), (g0 / kStages) & 1)) { ok = false; break; }
      tc_fence_after();
      issue_s(0, g0, n_tiles == 1);
      issue_s(1, g0, n_tiles == 1);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int g = g0 + j, s = g % kStages;
        if (!mbar_wait_bounded(bar(V_FULL + s), (g / kStages) & 1)) { ok = false; break; }
        for (int e = 0; e < 2; ++e) {
          if (!mbar_wait_bounded(bar(P_FULL + e), g & 1)) { ok = false; break; }
          if (j == 0 && round > 0 && !mbar_wait_bounded(bar(O_READ + e), (round - 1) & 1)) { ok = false; break; }
          tc_fence_after();
          const uint64_t vd = v_desc + (uint64_t)((s * kVBytes) >> 4);
#pragma unroll
          for (int kk = 0; kk < kKeys / 16; ++kk)
            mma_ts(t_o[e], t_s[e] + kk * 8, vd + (uint64_t)(kk * 128), idesc_pv, (j > 0 || kk > 0) ? 1u : 0u, elected);
          tc_commit(bar(O_FULL + e), elected);
          if (e == 1) tc_commit(bar(V_EMPTY + s), elected);
          if (j + 1 < n_tiles) {
            if (e == 0) {
              if (!mbar_wait_bounded(bar(K_FULL + (g + 1) % kStages), ((g + 1) / kStages) & 1)) { ok = false; break; }
              tc_fence_after();
            }
            issue_s(e, g + 1, j + 2 == n_tiles);
          }
        }
      }
      g0 += n_tiles;
    }
  } else if (warp >= 4 && warp < 4 + kSoftmaxWarps) {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(kMapsRegsHigh));
    // ---- softmax: group e = map e, all key tiles; thread owns query row r ----
    const int q4 = warp & 3;
    const int e = (warp - 4) >> 2;
    const int r = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const uint32_t ts = t_s[e] + lane_addr, to = t_o[e] + lane_addr;
    int g0 = 0;
    for (int round = 0; ok; ++round) {
      const Item it = item_of(round);
      if (!it.valid) break;
      const int m0 = it.m0, n_tiles = it.n_tiles;
      const int limit = a.start_pos + m0 + r;      // last key this row sees
      // score = x * sc;  capped: out * tanh(x * sc / cap)
      const float sc = a.scale * query_temperature(limit, a.temp_coef, a.temp_every);
      const float cs = CAP ? sc / a.softcap : sc * kLog2e, out = CAP ? a.softcap * kLog2e : 1.f;
      auto transform = [&](float x) { return CAP ? out * tanh_exact(x * cs) : x * cs; };
      float m_ref = -INFINITY, l_run = 0.f;
      int done = 0;
      for (int j = 0; j < n_tiles && ok; ++j, ++done) {
        if (!mbar_wait_bounded(bar(S_FULL + e), (g0 + j) & 1)) { ok = false; break; }
        tc_fence_after();
        const int j0 = j * kKeys;
        const bool edge = j0 + kKeys - 1 > a.start_pos + m0 || j0 + kKeys > p.n_keys;
        const int visible = edge ? min(limit + 1, p.n_keys) - j0 : kKeys;   // keys of the tile this row sees (may be <= 0)
        uint32_t x[4][32];
#pragma unroll
        for (int c = 0; c < 4; ++c) tmem_ld32(ts + c * 32, x[c]);
        tc_wait_ld();
        // the extremes of the visible raw scores (a negative factor makes the smallest the largest); keys behind the
        // row's last one take its first score in their place, so that nothing else has to know about them
        if (edge && visible < kKeys) {
#pragma unroll
          for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (c * 32 + i >= visible) x[c][i] = visible > 0 ? x[0][0] : 0u;
        }
        float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY}, mn4[4] = {INFINITY, INFINITY, INFINITY, INFINITY};
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float u = __uint_as_float(x[c][i]), v = __uint_as_float(x[c][i + 1]);
            mx4[(i >> 1) & 3] = fmax3(mx4[(i >> 1) & 3], u, v);
            mn4[(i >> 1) & 3] = fmin3(mn4[(i >> 1) & 3], u, v);
          }
        const float hi = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])), lo = fminf(fminf(mn4[0], mn4[1]), fminf(mn4[2], mn4[3]));
        const float mx = visible > 0 ? fmaxf(transform(hi), transform(lo)) : -INFINITY;
        if (__any_sync(kFullMask, mx > m_ref + kLazy)) {
          const float m_new = fmaxf(m_ref, mx);
          const float alpha = m_new == -INFINITY ? 1.f : fast_exp2(m_ref - m_new);
          if (done > 0) {
            if (!mbar_wait_bounded(bar(O_FULL + e), (g0 + done - 1) & 1)) { ok = false; break; }
            tc_fence_after();
            rescale_row<D>(to, alpha);
            l_run *= alpha;
          }
          m_ref = m_new;
        }
        const float mu = m_ref == -INFINITY ? 0.f : m_ref;
        const unsigned long long nmu2 = f2_packf(-mu, -mu);
        unsigned long long ps2[4] = {0ull, 0ull, 0ull, 0ull};
        auto probabilities = [&](auto exponent) {      // exponent(pair of raw scores) -> log2 of the pair's weights
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t pk[16];
            unsigned long long t2[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) t2[i] = exponent(f2_pack(x[c][2 * i], x[c][2 * i + 1]));
            float pe[32];
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              float t0, t1;
              f2_unpack(t2[i], t0, t1);
              pe[2 * i] = fast_exp2(t0);
              pe[2 * i + 1] = fast_exp2(t1);
            }
            if (edge) {
#pragma unroll
              for (int i = 0; i < 32; ++i)
                if (c * 32 + i >= visible) pe[i] = 0.f;
            }
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              ps2[i & 3] = f2_add(ps2[i & 3], f2_packf(pe[2 * i], pe[2 * i + 1]));
              pk[i] = pack_bf16x2(pe[2 * i], pe[2 * i + 1]);
            }
            tmem_st16(ts + c * 16, pk);
          }
        };
        if constexpr (!CAP) {
          const unsigned long long cs2 = f2_packf(cs, cs);
          probabilities([&](unsigned long long v) { return f2_fma(v, cs2, nmu2); });
        } else if (__all_sync(kFullMask, fmaxf(fabsf(hi), fabsf(lo)) * fabsf(cs) <= kPolyRange)) {
          // out * tanh(x cs) = x (q0 + x^2 (q1 + ...)) with the powers of cs in the coefficients
          unsigned long long q[5];
          float f = out * cs;
#pragma unroll
          for (int i = 0; i < 5; ++i) {
            q[i] = f2_packf(kPoly[i] * f, kPoly[i] * f);
            f *= cs * cs;
          }
          probabilities([&](unsigned long long v) {
            const unsigned long long w = f2_mul(v, v);
            return f2_fma(v, f2_fma(w, f2_fma(w, f2_fma(w, f2_fma(w, q[4], q[3]), q[2]), q[1]), q[0]), nmu2);
          });
        } else {
          probabilities([&](unsigned long long v) {
            float v0, v1;
            f2_unpack(v, v0, v1);
            return f2_packf(out * tanh_exact(v0 * cs) - mu, out * tanh_exact(v1 * cs) - mu);
          });
        }
        float a0, a1, b0, b1;
        f2_unpack(f2_add(ps2[0], ps2[1]), a0, a1);
        f2_unpack(f2_add(ps2[2], ps2[3]), b0, b1);
        l_run += (a0 + a1) + (b0 + b1);
        tc_wait_st();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(bar(P_FULL + e));
      }
      if (!ok) break;
      if (round > 0 && !mbar_wait_bounded(bar(O_READ + e), (round - 1) & 1)) { ok = false; break; }
      lrow[e * kRows + r] = l_run;
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(L_FULL + e));
      g0 += n_tiles;
    }
  } else if (warp >= 4 + kSoftmaxWarps) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kMapsRegsOut));
    // ---- output: thread owns row r of both maps' O ----
    const int q4 = warp & 3;
    const int r = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const uint32_t to0 = t_o[0] + lane_addr, to1 = t_o[1] + lane_addr;
    int g0 = 0;
    for (int round = 0;; ++round) {
      const Item it = item_of(round);
      if (!it.valid) break;
      const int t = it.m0 + r;
      float factor = a.post;
      if (a.gate && t < a.T) {
        const float z = __bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[it.b * a.g_sb + t * a.g_st + it.hq]);
        factor *= 1.f / (1.f + expf(-z));
      }
      // a wait that runs out ends in the status word; the warp goes on through the warpgroup's barriers and writes nothing
      float inv[2];
      for (int e = 0; e < 2; ++e) {
        if (ok && !mbar_wait_bounded(bar(L_FULL + e), round & 1)) ok = false;
        const float l = lrow[e * kRows + r];
        inv[e] = l > 0.f ? 1.f / l : 0.f;
        if (ok && !mbar_wait_bounded(bar(O_FULL + e), (g0 + it.n_tiles - 1) & 1)) ok = false;   // the map's last product
      }
      tc_fence_after();
      const float w0 = inv[0], w1 = -a.lambda * inv[1];
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < D / 16; ++c) {
        uint32_t y0[16], y1[16];
        tmem_ld16(to0 + c * 16, y0);
        tmem_ld16(to1 + c * 16, y1);
        tc_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          // (columns behind Dv are products of the zeros that fill the value boxes)
          const float o = fmaf(__uint_as_float(y0[i]), w0, __uint_as_float(y1[i]) * w1);
          ss = fmaf(o, o, ss);
        }
      }
      factor *= __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)a.Dv), a.eps));
      const float f0 = w0 * factor, f1 = w1 * factor;
      __nv_bfloat16* obase = static_cast<__nv_bfloat16*>(a.out) + it.b * a.o_sb + it.hq * a.o_sh;
#pragma unroll
      for (int c = 0; c < D / 32; ++c) {
        // 32 columns at a time through the staging rows, then 16-byte chunks, a row's four chunks on neighbouring threads
        uint4* dst = reinterpret_cast<uint4*>(stage + r * kOutPitch);
#pragma unroll
        for (int hc = 0; hc < 2; ++hc) {
          uint32_t y0[16], y1[16];
          tmem_ld16(to0 + c * 32 + hc * 16, y0);
          tmem_ld16(to1 + c * 32 + hc * 16, y1);
          tc_wait_ld();
          uint32_t w[8];
#pragma unroll
          for (int i = 0; i < 16; i += 2)
            w[i >> 1] = pack_bf16x2(fmaf(__uint_as_float(y0[i]), f0, __uint_as_float(y1[i]) * f1),
                                    fmaf(__uint_as_float(y0[i + 1]), f0, __uint_as_float(y1[i + 1]) * f1));
          dst[2 * hc] = make_uint4(w[0], w[1], w[2], w[3]);
          dst[2 * hc + 1] = make_uint4(w[4], w[5], w[6], w[7]);
        }
        if (c == D / 32 - 1) {   // both accumulators have been read: they may take the next item's products
          tc_fence_before();
          __syncwarp();
          if (lane == 0) {
            mbar_arrive(bar(O_READ));
            mbar_arrive(bar(O_READ + 1));
          }
        }
        asm volatile("bar.sync 2, 128;" ::: "memory");
#pragma unroll
        for (int id = r; id < kRows * 4; id += 128) {
          const int row = id >> 2, ch = id & 3, col = c * 32 + ch * 8;
          if (ok && it.m0 + row < a.T && col < a.Dv)
            *reinterpret_cast<uint4*>(obase + (it.m0 + row) * a.o_st + col) = *reinterpret_cast<const uint4*>(stage + row * kOutPitch + ch * 16);
        }
        asm volatile("bar.sync 2, 128;" ::: "memory");
      }
      g0 += it.n_tiles;
    }
  } else {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(kMapsRegsLow));
  }
  if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, kTmem);
}

// ---------------------------------------------------------------------------------------------------------------
int set_smem(const void* fn, size_t smem, bool (&configured)[64]) {
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  return L3CI_OK;
}

template <int KA, int KB, int VC, bool BIAS = false>
int launch_one(const CUtensorMap (&m)[5], const TcMixParams& p, unsigned ctas, cudaStream_t stream) {
  constexpr size_t smem = 1024 + (size_t)((1 + kStages) * (KA + KB) + kStages * VC) * kBox + 15 * 8 + 4 * kRows * 4 + 16;
  static_assert(smem <= (227 << 10), "shared memory");
  static bool configured[64] = {false};
  if (int st = set_smem(reinterpret_cast<const void*>(mixer_tc_kernel<KA, KB, VC, BIAS>), smem, configured)) return st;
  mixer_tc_kernel<KA, KB, VC, BIAS><<<ctas, kOneThreads, smem, stream>>>(m[0], m[1], m[2], m[3], m[4], p);
  L3CI_CHECK_LAUNCH("mixer_tc_kernel");
  return L3CI_OK;
}

template <int VC, bool CAP>
int launch_maps(const CUtensorMap& q0, const CUtensorMap& q1, const CUtensorMap& k, const CUtensorMap& v, const TcMixParams& p,
                unsigned ctas, cudaStream_t stream) {
  constexpr size_t smem = 1024 + (size_t)(2 + kStages * (2 + VC)) * kBox + kRows * kOutPitch + 20 * 8 + 16 + 2 * kRows * 4;
  static bool configured[64] = {false};
  if (int st = set_smem(reinterpret_cast<const void*>(mixer_tc_maps_kernel<VC, CAP>), smem, configured)) return st;
  mixer_tc_maps_kernel<VC, CAP><<<ctas, kMapsThreads, smem, stream>>>(q0, q1, k, v, p);
  L3CI_CHECK_LAUNCH("mixer_tc_maps_kernel");
  return L3CI_OK;
}

}  // namespace

bool mixer_tc_applies(const l3ci_mixer_attn_args* a) {
  if (a->dtype != L3CI_BF16 || a->start_pos < 0 || a->start_pos + a->T > a->n_keys || a->Dv > 128 || a->Dv % 8 || a->Da % 8 || a->Db % 8)
    return false;
  if (a->maps == 1 && a->bias_range > 0.f && a->Db) return false;
  if (a->maps == 2 ? a->Da > 64 : a->Da > 128 || a->Db > 64 || a->softcap > 0.f || a->temp_every > 0.f || !(a->scale > 0.f)) return false;
  if ((long long)a->B * a->H * ((a->T + kRows - 1) / kRows) > 0x7fffffffLL) return false;
  // rows the copy engine can address: positive strides of whole 16-byte vectors (an axis of extent 1 may have any)
  auto rows = [&](const void* ptr, int64_t sb, int64_t st, int64_t sh, int n, int heads) {
    return aligned16(ptr) && (n <= 1 || (st > 0 && st % 8 == 0)) && (heads <= 1 || (sh > 0 && sh % 8 == 0)) &&
           (a->B <= 1 || (sb > 0 && sb % 8 == 0));
  };
  if (!rows(a->qa, a->qa_sb, a->qa_st, a->qa_sh, a->T, a->H) || !rows(a->ka, a->ka_sb, a->ka_st, a->ka_sh, a->n_keys, a->G) ||
      !rows(a->v, a->v_sb, a->v_st, a->v_sh, a->n_keys, a->G) || !rows(a->out, a->o_sb, a->o_st, a->o_sh, a->T, a->H))
    return false;
  if (a->Db && (!rows(a->qb, a->qb_sb, a->qb_st, a->qb_sh, a->T, a->H) ||
                !rows(a->kb, a->kb_sb, a->kb_st, a->kb_sh, a->n_keys, a->kb_sh == 0 ? 1 : a->G)))
    return false;
  return true;
}

size_t mixer_tc_scratch_bytes(const l3ci_mixer_attn_args*) { return 0; }

int mixer_tc_launch(const l3ci_mixer_attn_args* a) {
  TcMixParams p = {};
  p.a = *a;
  p.R = a->H / a->G;
  p.m_blocks = (a->T + kRows - 1) / kRows;
  p.n_keys = a->start_pos + a->T;   // rows behind the portion are not read: they count as zeros
  p.shared_b = a->kb_sh == 0;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(a->stream);
  const long long items = (long long)a->B * a->H * p.m_blocks;
  const int T = a->T, H = a->H, G = a->G, B = a->B, S = p.n_keys;
  if (a->maps == 2) {
    CUtensorMap q0, q1, k, v;
    const auto qa = static_cast<const __nv_bfloat16*>(a->qa);
    if (int st = make_rows_map(&q0, qa, a->Da, T, H, B, a->qa_st, a->qa_sh, a->qa_sb, kRows)) return st;
    if (int st = make_rows_map(&q1, qa + a->Da, a->Da, T, H, B, a->qa_st, a->qa_sh, a->qa_sb, kRows)) return st;
    if (int st = make_rows_map(&k, a->ka, 2 * a->Da, S, G, B, a->ka_st, a->ka_sh, a->ka_sb, kKeys)) return st;
    if (int st = make_rows_map(&v, a->v, a->Dv, S, G, B, a->v_st, a->v_sh, a->v_sb, kKeys)) return st;
    const int sms = sm_count();
    const unsigned ctas = (unsigned)(sms > 0 && items > sms ? sms : items);
    if (a->Dv <= 64) return a->softcap > 0.f ? launch_maps<1, true>(q0, q1, k, v, p, ctas, stream) : launch_maps<1, false>(q0, q1, k, v, p, ctas, stream);
    return a->softcap > 0.f ? launch_maps<2, true>(q0, q1, k, v, p, ctas, stream) : launch_maps<2, false>(q0, q1, k, v, p, ctas, stream);
  }
  CUtensorMap m[5];
  if (int st = make_rows_map(&m[0], a->qa, a->Da, T, H, B, a->qa_st, a->qa_sh, a->qa_sb, kRows)) return st;
  if (int st = make_rows_map(&m[2], a->ka, a->Da, S, G, B, a->ka_st, a->ka_sh, a->ka_sb, kKeys)) return st;
  if (int st = make_rows_map(&m[4], a->v, a->Dv, S, G, B, a->v_st, a->v_sh, a->v_sb, kKeys)) return st;
  m[1] = m[0];
  m[3] = m[2];
  if (a->Db) {
    if (int st = make_rows_map(&m[1], a->qb, a->Db, T, H, B, a->qb_st, a->qb_sh, a->qb_sb, kRows)) return st;
    if (int st = make_rows_map(&m[3], a->kb, a->Db, S, p.shared_b ? 1 : G, B, a->kb_st, a->kb_sh, a->kb_sb, kKeys)) return st;
  }
  const unsigned ctas = (unsigned)items;
  const int ka = a->Da <= 64 ? 1 : 2, kb = a->Db ? 1 : 0, vc = a->Dv <= 64 ? 1 : 2;
  if (kb) {
    if (ka == 1) return vc == 1 ? launch_one<1, 1, 1>(m, p, ctas, stream) : launch_one<1, 1, 2>(m, p, ctas, stream);
    return vc == 1 ? launch_one<2, 1, 1>(m, p, ctas, stream) : launch_one<2, 1, 2>(m, p, ctas, stream);
  }
  if (a->bias_range > 0.f) {
    if (ka == 1) return vc == 1 ? launch_one<1, 0, 1, true>(m, p, ctas, stream) : launch_one<1, 0, 2, true>(m, p, ctas, stream);
    return vc == 1 ? launch_one<2, 0, 1, true>(m, p, ctas, stream) : launch_one<2, 0, 2, true>(m, p, ctas, stream);
  }
  if (ka == 1) return vc == 1 ? launch_one<1, 0, 1>(m, p, ctas, stream) : launch_one<1, 0, 2>(m, p, ctas, stream);
  return vc == 1 ? launch_one<2, 0, 1>(m, p, ctas, stream) : launch_one<2, 0, 2>(m, p, ctas, stream);
}

}  // namespace l3ci
