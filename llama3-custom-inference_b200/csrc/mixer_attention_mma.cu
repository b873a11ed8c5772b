// Attention of a few query rows over a long cache for the mixers (decode, short portions): bf16, mma.sync tensor
// cores, the key axis split over CTAs.
//
// A unit is 16 rows of one key/value head of one sequence; rows are (token, query head) pairs.  Differential attention
// puts 8 pairs into a unit: rows 0-7 are their first maps, rows 8-15 the second ones, so that a thread of the
// m16n8k16 accumulator (rows g and g + 8) holds both maps of a pair and the difference is taken in registers.
//
// CTA = a producer warp (bulk tensor copies into a ring of stages, 128-byte swizzle) and WARPS warps that share every
// tile of 64 keys:
//   scores   a warp takes 16 keys and one part of the query / key vector, whose A fragments it keeps in registers for
//            the whole launch (WARPS = 4 key groups x parts).  For one map the parts' products are added on
//            the way through shared memory; for two maps part i IS map i.
//   softmax  2 WARPS threads per row: add the parts, scale, cap, mask, online maximum in the log2 domain, p to shared
//            memory as bf16, rescale factors beside it.
//   output   a warp owns 8 * NB value columns: O = O * alpha + P V.
// A warp's work per tile is a chain of dependent instructions; the warps of an SM are what hides it.  Two maps: 8 warps,
// two CTAs per SM, and the scores of tile i + 1 are computed before the softmax of tile i into double buffers, so that
// one barrier per tile separates all three steps.  One map (long latent rows, which leave room for one CTA per SM): 16
// warps, four parts, the steps of a tile in order with two barriers, and a tile is two stages of 32 keys, so that the
// stages which fit are three more than the tile in hand needs.  A latent cache row is key and value at once (value = its first Dv columns): it is
// loaded once.  With more than one split the units' (m, l, O) go to scratch as fp32 and mixer_merge_kernel finishes
// the rows.
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "bf16x8.cuh"
#include "mixer_attention.h"
#include "ptx_sm100.cuh"
#include "tensor_map.h"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kMmRows = 16;
constexpr int kMmMaxStages = 8;
constexpr float kLog2e = 1.4426950408889634f;

constexpr int KEYS = 64;                             // keys per tile

template <int MAPS>
struct MmShape {
  static constexpr bool kAhead = MAPS == 2;                        // scores one tile ahead of the softmax
  static constexpr int kBufs = kAhead ? 2 : 1;                     // score and probability buffers
  static constexpr int kSub = MAPS == 2 ? 1 : 2;                   // stages per tile
  static constexpr int kStageKeys = KEYS / kSub;
  static constexpr int kWarps = MAPS == 2 ? 8 : 16;                // + the producer warp
  static constexpr int kThreads = 32 * (kWarps + 1);
  static constexpr int kParts = kWarps / (KEYS / 16);              // parts of the query / key vector
  static constexpr int kRowThreads = 2 * kWarps;                   // threads of a softmax row
  static constexpr int kPartRows = MAPS == 2 ? 8 : 16;             // score rows of a part
  static constexpr int kSPitch = KEYS + 8;                         // floats per score row
  static constexpr int kPPitch = KEYS * 2 + 16;                    // bytes per probability row
  static constexpr int kSBuf = kParts * kPartRows * kSPitch;       // floats per score buffer
  static constexpr int kFixed = kBufs * kSBuf * 4 + kBufs * kMmRows * kPPitch + 2 * kMmRows * 4 + 2 * kMmRows * 4 + kWarps * 8 * 4 +
                                2 * kMmMaxStages * 8;              // bytes beside the stages
  static_assert(MAPS == 1 || kParts == 2, "a part is a map");
  static constexpr int kQueryBytes = kBufs * kSBuf * 4 + kBufs * kMmRows * kPPitch;   // room of the query rows
};

struct MmParams {
  l3ci_mixer_attn_args a;
  int R, row_blocks, units, splits;
  int stages;                                   // stages of the ring
  int k_boxes, v_boxes;                         // 64-column boxes of a key / value row (v_boxes 0: values are in the key row)
  int q_pitch;                                  // bytes per query row in shared memory
  int part_cols;                                // columns of the query / key vector per part
  float* o_part;                                // [units][splits][16][dv_pad]
  float* ml_part;                               // [units][splits][16][2]
  int dv_pad;
  int merge_cols;                               // columns per CTA of the merge
};

__device__ __forceinline__ void ldsm_x2_trans(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ uint64_t l2_evict_normal_policy() {
  uint64_t pol;
  asm volatile("createpolicy.fractional.L2::evict_normal.b64 %0, 1.0;" : "=l"(pol));
  return pol;
}

// Finishes one (token, head) row of differential attention from the normalised outputs of its maps: the factor that
// the difference o (sum of squares `ss` over Dv columns) is multiplied by.
__device__ __forceinline__ float differential_factor(const l3ci_mixer_attn_args& a, float ss, int b, int t, int h) {
  float f = a.post * __frsqrt_rn(__fadd_rn(__fdiv_rn(ss, (float)a.Dv), a.eps));
  if (a.gate) {
    const float z = __bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[b * a.g_sb + t * a.g_st + h]);
    f *= 1.f / (1.f + expf(-z));
  }
  return f;
}

template <int KS, int NB, int MAPS>
__global__ void __launch_bounds__(MmShape<MAPS>::kThreads, (MAPS == 2 && KS <= 4 && NB <= 2) ? 2 : 1)
mixer_mma_kernel(const __grid_constant__ CUtensorMap kmap, const __grid_constant__ CUtensorMap vmap, const __grid_constant__ MmParams p) {
  using Sh = MmShape<MAPS>;
  constexpr int kStageKeys = Sh::kStageKeys;
  constexpr int kBoxBytes = kStageKeys * 128;
  constexpr int kGroups = KEYS / 16;
  constexpr int kWarps = Sh::kWarps;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const l3ci_mixer_attn_args& a = p.a;
  const int stages = p.stages;
  const uint32_t stage_bytes = (p.k_boxes + p.v_boxes) * kBoxBytes;
  const uint32_t ring = smem_u32(smem);
  float* sx = reinterpret_cast<float*>(smem + stages * stage_bytes);             // [bufs][parts][rows][kSPitch]
  uint8_t* pb = reinterpret_cast<uint8_t*>(sx + Sh::kBufs * Sh::kSBuf);          // [bufs][16][kPPitch]
  float* s_alpha = reinterpret_cast<float*>(pb + Sh::kBufs * kMmRows * Sh::kPPitch);   // [2][16]
  float* s_ml = s_alpha + 2 * kMmRows;                                           // [16][2]
  float* s_ss = s_ml + 2 * kMmRows;                                              // [8 warps][8 rows]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_ss + kWarps * 8);             // full[], empty[]
  const uint32_t full0 = smem_u32(bars), empty0 = full0 + kMmMaxStages * 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;

  if (tid == 0) {
    for (int i = 0; i < stages; ++i) {
      mbar_init(full0 + i * 8, 1);
      mbar_init(empty0 + i * 8, kWarps);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&kmap)) : "memory");
    if (p.v_boxes) asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&vmap)) : "memory");
  }
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();

  constexpr int kPairs = MAPS == 2 ? kMmRows / 2 : kMmRows;   // (token, head) pairs per unit
  const int unit = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  const int rb = unit % p.row_blocks, g = (unit / p.row_blocks) % a.G, b = unit / (p.row_blocks * a.G);
  const int pair0 = rb * kPairs, n_pairs = min(kPairs, a.T * p.R - pair0);
  const int pos0 = a.positions[b];
  const int keys = max(0, min(a.n_keys, pos0 + (pair0 + n_pairs - 1) / p.R + 1));
  // key tiles in sight of any of the unit's rows: those of the kept first keys, then from the first row's window on
  const int w_tile = window_start(pos0 + pair0 / p.R, a.window) / KEYS;
  const int kept_tiles = min(w_tile, (a.keep_first + KEYS - 1) / KEYS), skipped = w_tile - kept_tiles;
  const int tiles = max(0, (keys + KEYS - 1) / KEYS - skipped);
  const int per_split = (tiles + p.splits - 1) / p.splits;
  const int tile0 = split * per_split;
  const int n = max(0, min(tiles, tile0 + per_split) - tile0);
  auto first_key = [&](int i) { return (tile0 + i + (tile0 + i >= kept_tiles ? skipped : 0)) * KEYS; };   // of the CTA's tile i
  bool ok = true;

  if (warp == kWarps) {
    // ---- producer ----
    const uint64_t policy = p.row_blocks == 1 ? l2_evict_first_policy() : l2_evict_normal_policy();
    for (int i = 0, s = 0, phase = 1; i < n * Sh::kSub; ++i) {
      if (i >= stages && !mbar_wait_bounded(empty0 + s * 8, phase)) { ok = false; break; }
      if (lane == 0) {
        const uint32_t bar = full0 + s * 8, dst = ring + s * stage_bytes;
        mbar_expect_tx(bar, stage_bytes);
        const int j0 = first_key(i / Sh::kSub) + i % Sh::kSub * kStageKeys;
        for (int c = 0; c < p.k_boxes; ++c) tma_load_4d(dst + c * kBoxBytes, &kmap, bar, c * 64, j0, g, b, policy);
        for (int c = 0; c < p.v_boxes; ++c) tma_load_4d(dst + (p.k_boxes + c) * kBoxBytes, &vmap, bar, c * 64, j0, g, b, policy);
      }
      __syncwarp();
      if (++s == stages) { s = 0; phase ^= 1; }
    }
    if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);
    return;
  }

  // ---- query fragments of this warp's part ----
  const int kgroup = warp % kGroups, part = warp / kGroups;
  const int dk = MAPS == 2 ? a.Da : a.Da + a.Db;
  const int col_lo = MAPS == 2 ? 0 : part * p.part_cols;                       // within the pair's vector (or map)
  const int col_hi = MAPS == 2 ? dk : min(dk, col_lo + p.part_cols);
  const int n_ks = (max(0, col_hi - col_lo) + 15) / 16;
  const int mat = lane >> 3, r8 = lane & 7;
  auto sync_compute = [] { asm volatile("bar.sync 1, %0;" ::"n"(32 * kWarps) : "memory"); };
  uint32_t qf[KS][4];
  {
    // through shared memory (the score and probability buffers are not in use yet): rows in whole 16-byte vectors
    const int q_cols = MAPS == 2 ? Sh::kParts * a.Da : dk, q_pitch = p.q_pitch, chunks = q_pitch / 16;
    uint8_t* qs = reinterpret_cast<uint8_t*>(sx);
    for (int x = tid; x < kPairs * chunks; x += 32 * kWarps) {
      const int row = x / chunks, col = (x - row * chunks) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (row < n_pairs && col < q_cols) {
        const int idx = pair0 + row, t = idx / p.R, h = g * p.R + idx % p.R;
        const __nv_bfloat16* src = MAPS == 2 || col < a.Da
            ? static_cast<const __nv_bfloat16*>(a.qa) + b * a.qa_sb + t * a.qa_st + h * a.qa_sh + col
            : static_cast<const __nv_bfloat16*>(a.qb) + b * a.qb_sb + t * a.qb_st + h * a.qb_sh + (col - a.Da);
        v = *reinterpret_cast<const uint4*>(src);
      }
      *reinterpret_cast<uint4*>(qs + row * q_pitch + col * 2) = v;
    }
    sync_compute();
    // A fragments: matrices (rows 0-7, cols c), (rows 8-15, c), (rows 0-7, c + 8), (rows 8-15, c + 8)
    const int c0 = MAPS == 2 ? part * a.Da : col_lo;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      qf[ks][0] = qf[ks][1] = qf[ks][2] = qf[ks][3] = 0u;
      if (ks < n_ks) {
        const uint32_t addr = smem_u32(qs) + (c0 + ks * 16 + 8 * (mat >> 1)) * 2;
        if (MAPS == 2) {
          // accumulator rows 8-15 of a part are not used (its 8 pairs sit in rows 0-7): two matrices, and columns of
          // the other map, which a last half step reads, count as 0
          ldsm_x2(smem_u32(qs) + r8 * q_pitch + (c0 + ks * 16 + 8 * (mat & 1)) * 2, qf[ks][0], qf[ks][2]);
          if (ks * 16 + 8 >= dk) qf[ks][2] = 0u;
        } else {
          ldsm_x4(addr + (r8 + 8 * (mat & 1)) * q_pitch, qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3]);
        }
      }
    }
    sync_compute();
  }

  // ---- this thread's softmax row and its kPer neighbouring keys of a tile ----
  constexpr int kPer = KEYS / Sh::kRowThreads;
  const int srow = tid / Sh::kRowThreads, skey = (tid % Sh::kRowThreads) * kPer;
  const bool row_lead = tid % Sh::kRowThreads == 0;
  const int spair = MAPS == 2 ? (srow & 7) : srow;
  const int limit = pos0 + (pair0 + min(spair, n_pairs - 1)) / p.R;            // last key the row sees
  const float scale = a.scale * query_temperature(limit, a.temp_coef, a.temp_every);
  const float cap = a.softcap, cap_scale = cap > 0.f ? scale / cap : scale * kLog2e, cap_out = cap * kLog2e;
  const int row_head = g * p.R + (pair0 + min(spair, n_pairs - 1)) % p.R;
  const float slope = MAPS == 1 ? head_slope(a.bias_range, row_head, a.H) * kLog2e : 0.f;
  const int row_lo = window_start(limit, a.window);
  // the sink is a score of 0 that the first split has seen before its first tile
  const bool sink = MAPS == 1 && a.sink && split == 0;
  float m_run = sink ? 0.f : -INFINITY, l_run = sink && row_lead ? 1.f : 0.f;

  float o[NB][4];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f;
  // K: matrices (keys 0-7, cols c..), (keys 0-7, c + 8), (keys 8-15, c), (keys 8-15, c + 8) of the warp's 16 keys;
  // chunk = 16 bytes of a row, chunk c of row r lies at c ^ (r % 8) of its 128-byte box row
  uint32_t k_off[KS];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    const int c = (MAPS == 2 ? part * a.Da : col_lo) / 8 + (mat & 1) + 2 * ks;
    k_off[ks] = (kgroup * 16 % kStageKeys + r8 + 8 * (mat >> 1)) * 128 + (c >> 3) * kBoxBytes + (((c & 7) ^ r8) << 4);
  }
  // V transposed: matrices (keys 0-7, cols c), (keys 8-15, c), (keys 0-7, c + 8), (keys 8-15, c + 8)
  const uint32_t v_base = p.v_boxes ? p.k_boxes * kBoxBytes : 0;
  const int v_col0 = warp * NB * 8;
  constexpr int kPairsOfBlocks = NB > 1 ? NB / 2 : 1;
  uint32_t v_off[kPairsOfBlocks];
#pragma unroll
  for (int np = 0; np < kPairsOfBlocks; ++np) {
    const int c = warp * NB + 2 * np + (NB > 1 ? (mat >> 1) : 0);
    v_off[np] = v_base + (r8 + 8 * (mat & 1)) * 128 + (c >> 3) * kBoxBytes + (((c & 7) ^ r8) << 4);
  }
  const int v_blocks = max(0, min(kPairsOfBlocks, (a.Dv - v_col0 + 15) / 16));   // with real columns
  // P: matrices (rows 0-7, keys c), (rows 8-15, c), (rows 0-7, c + 8), (rows 8-15, c + 8)
  const uint32_t p_off = smem_u32(pb) + (r8 + 8 * (mat & 1)) * Sh::kPPitch + (mat >> 1) * 16;

  // stage (and phase) of the tile whose scores are next; the warp reads the stage its key group lies in, and keeps up
  // with the arrival of the tile's other stage, which its output columns need
  int s_full = 0, f_phase = 0;
  auto scores = [&](int i) {
    int s_keys = s_full;
#pragma unroll
    for (int u = 0; u < Sh::kSub; ++u) {
      if (ok && !mbar_wait_bounded(full0 + s_full * 8, f_phase)) ok = false;
      if (kgroup * 16 / kStageKeys == u) s_keys = s_full;
      if (++s_full == stages) { s_full = 0; f_phase ^= 1; }
    }
    const uint32_t kt = ring + s_keys * stage_bytes;
    float acc[2][2][4] = {};                                                    // [k-step parity][8 keys]
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      if (ks < n_ks) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(kt + k_off[ks], b0, b1, b2, b3);
        mma_bf16(acc[ks & 1][0], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
        mma_bf16(acc[ks & 1][1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
      }
    }
    float* dst = sx + (Sh::kAhead ? (i & 1) * Sh::kSBuf : 0) + (part * Sh::kPartRows + gid) * Sh::kSPitch + kgroup * 16 + 2 * tig;
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      *reinterpret_cast<float2*>(dst + m * 8) = make_float2(acc[0][m][0] + acc[1][m][0], acc[0][m][1] + acc[1][m][1]);
      if (MAPS == 1)
        *reinterpret_cast<float2*>(dst + 8 * Sh::kSPitch + m * 8) = make_float2(acc[0][m][2] + acc[1][m][2], acc[0][m][3] + acc[1][m][3]);
    }
  };

  if (Sh::kAhead) {
    if (n > 0) scores(0);
    sync_compute();
  }
  for (int i = 0, st = 0; i < n; ++i) {   // st: the tile's first stage
    const int buf = Sh::kAhead ? (i & 1) : 0;
    int st_of[Sh::kSub];
#pragma unroll
    for (int u = 0; u < Sh::kSub; ++u) {
      st_of[u] = st;
      if (++st == stages) st = 0;
    }
    if (!Sh::kAhead) {
      scores(i);
      sync_compute();
    } else if (i + 1 < n) {
      scores(i + 1);
    }
    {
      // ---- softmax of tile i ----
      float v[kPer];
      const float* src = sx + (Sh::kAhead ? (i & 1) * Sh::kSBuf : 0);
      if (MAPS == 2) {
        const float* row = src + ((srow >> 3) * 8 + (srow & 7)) * Sh::kSPitch + skey;
#pragma unroll
        for (int e = 0; e < kPer; ++e) v[e] = row[e];
      } else {
#pragma unroll
        for (int e = 0; e < kPer; ++e) v[e] = 0.f;
#pragma unroll
        for (int q = 0; q < Sh::kParts; ++q) {
          const float* row = src + (q * 16 + srow) * Sh::kSPitch + skey;
#pragma unroll
          for (int e = 0; e < kPer; ++e) v[e] += row[e];
        }
      }
      const int j0 = first_key(i), j = j0 + skey;
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < kPer; ++e) {
        v[e] *= cap_scale;
        if (cap > 0.f) v[e] = cap_out * tanhf(v[e]);
        if (MAPS == 1) v[e] = fmaf(-slope, (float)(limit - j - e), v[e]);
        if (j + e > limit || j + e >= keys || (MAPS == 1 && j + e < row_lo && j + e >= a.keep_first)) v[e] = -INFINITY;
        mx = fmaxf(mx, v[e]);
      }
      mx = fmaxf(m_run, group_max<Sh::kRowThreads>(mx));
      const float mu = mx == -INFINITY ? 0.f : mx;
      const float alpha = fast_exp2(m_run - mu);                                // 0 at the row's first visible key
      m_run = mx;
      float sum = 0.f;
#pragma unroll
      for (int e = 0; e < kPer; ++e) {
        v[e] = fast_exp2(v[e] - mu);
        sum += v[e];
      }
      l_run = fmaf(l_run, alpha, sum);
      uint8_t* dst = pb + (buf * kMmRows + srow) * Sh::kPPitch + skey * 2;
      if constexpr (kPer == 1) {
        *reinterpret_cast<__nv_bfloat16*>(dst) = __float2bfloat16_rn(v[0]);
      } else {
#pragma unroll
        for (int e = 0; e < kPer; e += 2) reinterpret_cast<uint32_t*>(dst)[e / 2] = pack_bf16x2(v[e], v[(e + 1) % kPer]);
      }
      if (row_lead) s_alpha[buf * kMmRows + srow] = alpha;
      if (j0 + KEYS > keys) {
        // rows behind the last visible key hold whatever the cache holds there (their weights are 0, they may be
        // NaN): the value part of those rows becomes 0.  It is the last tile of this ring, nothing is loaded over it.
        const int first = keys - j0, boxes = p.v_boxes ? p.v_boxes : p.k_boxes;
        for (int x = tid; x < (KEYS - first) * boxes * 8; x += 32 * kWarps) {
          const int row = first + x / (8 * boxes);
          uint8_t* vt = smem + (row < kStageKeys ? st_of[0] : st_of[Sh::kSub - 1]) * stage_bytes + v_base;
          *reinterpret_cast<uint4*>(vt + (x / 8 % boxes) * kBoxBytes + (row % kStageKeys) * 128 + (x & 7) * 16) = make_uint4(0, 0, 0, 0);
        }
      }
    }
    sync_compute();
    {
      // ---- output of tile i ----
      const float al = s_alpha[buf * kMmRows + gid], ah = s_alpha[buf * kMmRows + gid + 8];
      if (__any_sync(kFullMask, al != 1.f || ah != 1.f)) {
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) { o[nb][0] *= al; o[nb][1] *= al; o[nb][2] *= ah; o[nb][3] *= ah; }
      }
      const uint32_t pt = p_off + buf * kMmRows * Sh::kPPitch;
#pragma unroll
      for (int kk = 0; kk < KEYS / 16; ++kk) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(pt + kk * 32, a0, a1, a2, a3);
        const uint32_t vt = ring + st_of[kk * 16 / kStageKeys] * stage_bytes + (kk * 16 % kStageKeys) * 128;
#pragma unroll
        for (int np = 0; np < kPairsOfBlocks; ++np) {
          if (np >= v_blocks) continue;
          uint32_t b0, b1, b2, b3;
          if constexpr (NB == 1) {
            ldsm_x2_trans(vt + v_off[0], b0, b1);
            mma_bf16(o[0], a0, a1, a2, a3, b0, b1);
          } else {
            ldsm_x4_trans(vt + v_off[np], b0, b1, b2, b3);
            mma_bf16(o[2 * np], a0, a1, a2, a3, b0, b1);
            mma_bf16(o[(2 * np + 1) % NB], a0, a1, a2, a3, b2, b3);
          }
        }
      }
      __syncwarp();
      if (lane == 0) {
#pragma unroll
        for (int u = 0; u < Sh::kSub; ++u) mbar_arrive(empty0 + st_of[u] * 8);
      }
    }
  }
  if (!ok && lane == 0 && a.status) atomicExch(a.status, (int)L3CI_ERR_DEVICE_WAIT);

  // ---- the rows' sums, then the output or the partial record ----
  const float l_all = group_sum<Sh::kRowThreads>(l_run);
  if (row_lead) {
    s_ml[2 * srow] = m_run;
    s_ml[2 * srow + 1] = l_all;
  }
  sync_compute();
  if (p.splits > 1) {
    const long long rec = (long long)unit * p.splits + split;
    if (tid < 2 * kMmRows) p.ml_part[rec * 2 * kMmRows + tid] = s_ml[tid];
    if (n == 0) return;   // the record's sums are 0: its outputs are not read
    float* dst = p.o_part + rec * kMmRows * p.dv_pad;
    const bool lo = gid < n_pairs, hi = MAPS == 2 ? lo : gid + 8 < n_pairs;   // rows of real pairs
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int col = v_col0 + nb * 8 + 2 * tig;
      if (col >= a.Dv) continue;
      if (lo) *reinterpret_cast<float2*>(dst + gid * p.dv_pad + col) = make_float2(o[nb][0], o[nb][1]);
      if (hi) *reinterpret_cast<float2*>(dst + (gid + 8) * p.dv_pad + col) = make_float2(o[nb][2], o[nb][3]);
    }
    return;
  }
  const float l0 = s_ml[2 * gid + 1], l1 = s_ml[2 * (gid + 8) + 1];
  const float i0 = l0 > 0.f ? 1.f / l0 : 0.f, i1 = l1 > 0.f ? 1.f / l1 : 0.f;
  auto out_row = [&](int pair) {
    const int idx = pair0 + pair, t = idx / p.R, h = g * p.R + idx % p.R;
    return static_cast<__nv_bfloat16*>(a.out) + b * a.o_sb + t * a.o_st + h * a.o_sh;
  };
  if (MAPS == 2) {
    float ss = 0.f;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        o[nb][e] = o[nb][e] * i0 - a.lambda * (o[nb][2 + e] * i1);
        if (v_col0 + nb * 8 + 2 * tig + e < a.Dv) ss = fmaf(o[nb][e], o[nb][e], ss);
      }
    ss = group_sum<4>(ss);
    if (tig == 0) s_ss[warp * 8 + gid] = ss;
    sync_compute();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) ss += s_ss[w * 8 + gid];
    if (gid < n_pairs) {
      const int idx = pair0 + gid;
      const float f = differential_factor(a, ss, b, idx / p.R, g * p.R + idx % p.R);
      __nv_bfloat16* dst = out_row(gid);
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        const int col = v_col0 + nb * 8 + 2 * tig;
        if (col < a.Dv) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(o[nb][0] * f, o[nb][1] * f);
      }
    }
  } else {
#pragma unroll
    for (int hi = 0; hi < 2; ++hi) {
      const int pair = gid + 8 * hi;
      if (pair >= n_pairs) continue;
      const float inv = hi ? i1 : i0;
      __nv_bfloat16* dst = out_row(pair);
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) {
        const int col = v_col0 + nb * 8 + 2 * tig;
        if (col < a.Dv) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(o[nb][2 * hi] * inv, o[nb][2 * hi + 1] * inv);
      }
    }
  }
}

// Folds the splits of one (token, head) pair: a CTA per pair (with one map, where pairs are few, per pair and run of
// columns).  A thread takes four columns and a group of the splits (one
// group when there are few); the splits' weights are formed once in shared memory, the groups' sums meet there.
constexpr int kMaxSplits = 128;
constexpr int kMaxDv = 512;
constexpr int kMergeMax = 512;   // threads

template <int MAPS>
__global__ void __launch_bounds__(kMergeMax) mixer_merge_kernel(const __grid_constant__ MmParams p) {
  __shared__ float red[32];
  __shared__ float wt[MAPS][kMaxSplits];
  __shared__ float4 sum[MAPS][kMergeMax];
  pdl_wait();
  pdl_launch_dependents();
  const l3ci_mixer_attn_args& a = p.a;
  constexpr int kPairs = MAPS == 2 ? kMmRows / 2 : kMmRows;
  const int unit = blockIdx.x / kPairs, pair = blockIdx.x % kPairs;
  const int rb = unit % p.row_blocks, g = (unit / p.row_blocks) % a.G, b = unit / (p.row_blocks * a.G);
  const int idx = rb * kPairs + pair;
  if (idx >= a.T * p.R) return;
  const int t = idx / p.R, h = g * p.R + idx % p.R, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // weight of split s: exp2(m_s - max) / sum of l_s exp2(m_s - max); 0 for a split without a visible key
  if (warp < MAPS) {
    const float2* ml = reinterpret_cast<const float2*>(p.ml_part) + (long long)unit * p.splits * kMmRows + pair + 8 * warp;
    float mx = -INFINITY, all = 0.f;
    for (int s = lane; s < p.splits; s += 32) mx = fmaxf(mx, ml[s * kMmRows].x);
    mx = group_max<kWarp>(mx);
    for (int s = lane; s < p.splits; s += 32) {
      const float2 x = ml[s * kMmRows];
      const float w = x.y > 0.f ? fast_exp2(x.x - mx) : 0.f;
      wt[warp][s] = w;
      all = fmaf(x.y, w, all);
    }
    all = group_sum<kWarp>(all);
    const float inv = all > 0.f ? 1.f / all : 0.f;
    for (int s = lane; s < p.splits; s += 32) wt[warp][s] *= inv;
  }
  __syncthreads();
  const int col0 = blockIdx.y * p.merge_cols, quads = min(p.merge_cols, a.Dv - col0) / 4;
  int lanes = 16;                                                // threads along the columns, a power of two
  while (lanes < quads) lanes *= 2;
  const int groups = blockDim.x / lanes, grp = tid / lanes, c = tid % lanes;
  const long long step = (long long)kMmRows * p.dv_pad;
#pragma unroll
  for (int m = 0; m < MAPS; ++m) {
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < quads) {
      const float* src = p.o_part + ((long long)unit * p.splits * kMmRows + pair + 8 * m) * p.dv_pad + col0 + 4 * c;
#pragma unroll 4
      for (int s = grp; s < p.splits; s += groups) {
        const float w = wt[m][s];
        const float4 y = *reinterpret_cast<const float4*>(src + s * step);
        if (w != 0.f) {   // a record of weight 0 may never have been written
          x.x = fmaf(y.x, w, x.x);
          x.y = fmaf(y.y, w, x.y);
          x.z = fmaf(y.z, w, x.z);
          x.w = fmaf(y.w, w, x.w);
        }
      }
    }
    sum[m][tid] = x;
  }
  if (groups > 1) __syncthreads();
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  if (grp == 0) {
#pragma unroll
    for (int m = 0; m < MAPS; ++m) {
      const float f = m ? -a.lambda : 1.f;
      for (int q = 0; q < groups; ++q) {
        const float4 y = sum[m][q * lanes + c];
        o[0] = fmaf(y.x, f, o[0]);
        o[1] = fmaf(y.y, f, o[1]);
        o[2] = fmaf(y.z, f, o[2]);
        o[3] = fmaf(y.w, f, o[3]);
      }
    }
  }
  float f = 1.f;
  if (MAPS == 2)
    f = differential_factor(a, cta_sum(o[0] * o[0] + o[1] * o[1] + o[2] * o[2] + o[3] * o[3], red, blockDim.x / kWarp), b, t, h);
  if (grp == 0 && c < quads) {
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + b * a.o_sb + t * a.o_st + h * a.o_sh + col0 + 4 * c;
    reinterpret_cast<uint32_t*>(dst)[0] = pack_bf16x2(o[0] * f, o[1] * f);   // rows start on 4 bytes
    reinterpret_cast<uint32_t*>(dst)[1] = pack_bf16x2(o[2] * f, o[3] * f);
  }
}
int merge_threads(const MmParams& p) {
  int lanes = 16;
  while (lanes < p.merge_cols / 4) lanes *= 2;
  int threads = lanes < 64 ? 64 : lanes;
  while (threads < kMergeMax && threads / lanes * 4 < p.splits) threads *= 2;
  return threads;
}

constexpr int kMaxSteps1 = 9, kMaxSteps2 = 16;   // k-steps of a part

int steps_per_part(const l3ci_mixer_attn_args* a) {
  return a->maps == 2 ? (a->Da + 15) / 16 : ((a->Da + a->Db + 15) / 16 + 3) / 4;
}
bool values_in_keys(const l3ci_mixer_attn_args* a) {
  return a->v == a->ka && a->v_st == a->ka_st && a->v_sb == a->ka_sb && (a->G == 1 || a->v_sh == a->ka_sh) && a->Dv <= a->maps * a->Da + a->Db;
}

MmParams mma_params(const l3ci_mixer_attn_args* a) {
  MmParams p = {};
  p.a = *a;
  p.R = a->H / a->G;
  const int pairs = a->maps == 2 ? kMmRows / 2 : kMmRows;
  p.row_blocks = (int)(((long long)a->T * p.R + pairs - 1) / pairs);
  p.units = a->B * a->G * p.row_blocks;
  p.k_boxes = (a->maps * a->Da + a->Db + 63) / 64;
  p.v_boxes = values_in_keys(a) ? 0 : (a->Dv + 63) / 64;
  p.part_cols = steps_per_part(a) * 16;
  const int q_cols = a->maps == 2 ? 2 * a->Da + 8 : 4 * p.part_cols;   // what the fragments read
  p.q_pitch = ((q_cols * 2 + 15) / 16 | 1) * 16;                       // an odd number of 16-byte vectors
  p.dv_pad = a->Dv <= 64 ? 64 : a->Dv <= 128 ? 128 : a->Dv <= 256 ? 256 : 512;
  // stages: as many as fit beside a second CTA on the SM where the registers allow one and three stages fit, else alone
  const int stage = (p.k_boxes + p.v_boxes) * (a->maps == 2 ? MmShape<2>::kStageKeys : MmShape<1>::kStageKeys) * 128;
  const int fixed = 1024 + (a->maps == 2 ? MmShape<2>::kFixed : MmShape<1>::kFixed);
  const bool small = a->maps == 2 && steps_per_part(a) <= 4 && p.dv_pad <= 128;
  const int half = ((228 << 10) / 2 - 1024 - fixed) / stage, whole = ((227 << 10) - fixed) / stage;
  const int per_sm = small && half >= 3 ? 2 : 1;
  p.stages = per_sm == 2 ? half : whole;
  if (p.stages > kMmMaxStages) p.stages = kMmMaxStages;
  // splits: whole waves of CTAs over the device, each a run of tiles plus a fixed cost of a few
  const int sms = sm_count() > 0 ? sm_count() : 148;
  const long long slots = (long long)sms * per_sm;
  const int keys = a->start_pos >= 0 && a->start_pos + a->T < a->n_keys ? a->start_pos + a->T : a->n_keys;
  int tiles = keys > 0 ? (keys + KEYS - 1) / KEYS : 1;
  if (a->window > 0) {   // most tiles a unit sees: its window at the worst place, and the kept keys
    const long long seen = ((long long)a->window + (pairs + p.R - 1) / p.R + KEYS - 1) / KEYS + 1 + (a->keep_first + KEYS - 1) / KEYS;
    if (seen < tiles) tiles = (int)seen;
  }
  double best = 0;
  p.splits = 1;
  for (int s = 1; s <= tiles && s <= kMaxSplits; ++s) {
    if (s > 1 && (long long)p.units * s > 4 * slots) break;
    const long long waves = ((long long)p.units * s + slots - 1) / slots;
    const double cost = waves * ((tiles + s - 1) / s + 4.0) + (s > 1 ? 3.0 + s / 32.0 : 0.0);
    if (s == 1 || cost < best) { best = cost; p.splits = s; }
  }
  p.merge_cols = p.dv_pad;
  while (a->maps == 1 && p.splits > 8 && p.merge_cols > 64 && (long long)a->B * a->T * a->H * (p.dv_pad / p.merge_cols) < sms) p.merge_cols /= 2;
  return p;
}
size_t mma_smem(const MmParams& p) {
  const l3ci_mixer_attn_args* a = &p.a;
  return 1024 + (size_t)p.stages * (p.k_boxes + p.v_boxes) * (a->maps == 2 ? MmShape<2>::kStageKeys : MmShape<1>::kStageKeys) * 128 +
         (p.a.maps == 2 ? MmShape<2>::kFixed : MmShape<1>::kFixed);
}

template <int KS, int NB, int MAPS>
int launch_mma(const CUtensorMap& kmap, const CUtensorMap& vmap, const MmParams& p, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(mixer_mma_kernel<KS, NB, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem_optin()));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  L3CI_LAUNCH("mixer_mma_kernel", mixer_mma_kernel<KS, NB, MAPS>, dim3((unsigned)(p.units * p.splits)), dim3(MmShape<MAPS>::kThreads), mma_smem(p), stream, kmap, vmap, p);
  return L3CI_OK;
}
template <int KS, int MAPS>
int launch_mma_nb(const CUtensorMap& kmap, const CUtensorMap& vmap, const MmParams& p, cudaStream_t stream) {
  constexpr int kUnit = 8 * MmShape<MAPS>::kWarps;   // value columns of the CTA per n-block
  if (p.dv_pad <= kUnit) return launch_mma<KS, 1, MAPS>(kmap, vmap, p, stream);
  if (p.dv_pad <= 2 * kUnit) return launch_mma<KS, 2, MAPS>(kmap, vmap, p, stream);
  if (p.dv_pad <= 4 * kUnit) return launch_mma<KS, 4, MAPS>(kmap, vmap, p, stream);
  if constexpr (MAPS == 2) return launch_mma<KS, 8, MAPS>(kmap, vmap, p, stream);
  return fail(L3CI_ERR_UNSUPPORTED, "mixer_attention: value size %d", p.a.Dv);
}
size_t scratch_of(const MmParams& p) {
  return p.splits > 1 ? (size_t)p.units * p.splits * kMmRows * (p.dv_pad + 2) * sizeof(float) : 0;
}

}  // namespace

bool mixer_mma_applies(const l3ci_mixer_attn_args* a) {
  if (a->dtype != L3CI_BF16 || a->Dv > kMaxDv || a->Dv % 8 || a->Da % 8 || a->Db % 8 ||
      steps_per_part(a) > (a->maps == 2 ? kMaxSteps2 : kMaxSteps1))
    return false;
  if (a->Db && (static_cast<const uint16_t*>(a->kb) != static_cast<const uint16_t*>(a->ka) + a->Da || a->kb_st != a->ka_st ||
                a->kb_sb != a->ka_sb || (a->G > 1 && a->kb_sh != a->ka_sh)))
    return false;   // the two key parts must be one row
  // rows the copy engine can address: positive strides of whole 16-byte vectors (an axis of extent 1 may have any)
  auto rows16 = [&](const void* ptr, int64_t sb, int64_t st, int64_t sh) {
    return aligned16(ptr) && (a->n_keys <= 1 || (st > 0 && st % 8 == 0)) && (a->G <= 1 || (sh > 0 && sh % 8 == 0)) &&
           (a->B <= 1 || (sb > 0 && sb % 8 == 0));
  };
  auto rows4 = [](const void* ptr, int64_t sb, int64_t st, int64_t sh) {
    return reinterpret_cast<uintptr_t>(ptr) % 4 == 0 && (sb | st | sh) % 2 == 0;
  };
  if (!rows16(a->ka, a->ka_sb, a->ka_st, a->ka_sh) || !rows16(a->v, a->v_sb, a->v_st, a->v_sh)) return false;
  auto vectors = [](const void* ptr, int64_t sb, int64_t st, int64_t sh) { return aligned16(ptr) && (sb | st | sh) % 8 == 0; };
  if (!vectors(a->qa, a->qa_sb, a->qa_st, a->qa_sh) || (a->Db && !vectors(a->qb, a->qb_sb, a->qb_st, a->qb_sh)) ||
      !rows4(a->out, a->o_sb, a->o_st, a->o_sh))
    return false;
  const long long rows = (long long)a->T * (a->H / a->G);
  if ((long long)a->B * a->G * ((rows + 7) / 8) * kMaxSplits > 0x7fffffffLL || rows > 0x7fffffffLL) return false;
  const MmParams p = mma_params(a);
  return a->maps == 2 ? p.stages >= 2 && 8 * p.q_pitch <= MmShape<2>::kQueryBytes : p.stages >= 4 && 16 * p.q_pitch <= MmShape<1>::kQueryBytes;
}

size_t mixer_mma_scratch_bytes(const l3ci_mixer_attn_args* a) { return scratch_of(mma_params(a)); }

int mixer_mma_launch(const l3ci_mixer_attn_args* a) {
  MmParams p = mma_params(a);
  const size_t need = scratch_of(p);
  if (need > 0) {
    if (!a->scratch || a->scratch_bytes < need || !aligned16(a->scratch))
      return fail(L3CI_ERR_SCRATCH, "mixer_attention: %zu bytes of scratch needed, %zu given", need, a->scratch_bytes);
    p.o_part = static_cast<float*>(a->scratch);
    p.ml_part = p.o_part + (size_t)p.units * p.splits * kMmRows * p.dv_pad;
  }
  CUtensorMap kmap, vmap;
  const int stage_keys = a->maps == 2 ? MmShape<2>::kStageKeys : MmShape<1>::kStageKeys;
  if (int st = make_rows_map(&kmap, a->ka, a->maps * a->Da + a->Db, a->n_keys, a->G, a->B, a->ka_st, a->ka_sh, a->ka_sb, stage_keys)) return st;
  vmap = kmap;
  if (p.v_boxes)
    if (int st = make_rows_map(&vmap, a->v, a->Dv, a->n_keys, a->G, a->B, a->v_st, a->v_sh, a->v_sb, stage_keys)) return st;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(a->stream);
  const int ks = steps_per_part(a);
  const int st = a->maps == 2 ? (ks <= 4   ? launch_mma_nb<4, 2>(kmap, vmap, p, stream)
                                 : ks <= 8 ? launch_mma_nb<8, 2>(kmap, vmap, p, stream)
                                           : launch_mma_nb<kMaxSteps2, 2>(kmap, vmap, p, stream))
                              : (ks <= 3 ? launch_mma_nb<3, 1>(kmap, vmap, p, stream)
                                         : launch_mma_nb<kMaxSteps1, 1>(kmap, vmap, p, stream));
  if (st) return st;
  if (p.splits > 1) {
    const unsigned ctas = (unsigned)(p.units * (a->maps == 2 ? kMmRows / 2 : kMmRows));
    if (a->maps == 2) L3CI_LAUNCH("mixer_merge_kernel", mixer_merge_kernel<2>, dim3(ctas), dim3(merge_threads(p)), 0, stream, p);
    else L3CI_LAUNCH("mixer_merge_kernel", mixer_merge_kernel<1>, dim3(ctas, (unsigned)((a->Dv + p.merge_cols - 1) / p.merge_cols)), dim3(merge_threads(p)), 0, stream, p);
  }
  return L3CI_OK;
}

}  // namespace l3ci
