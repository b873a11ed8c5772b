// Attention of a few query rows over a long cache for the mixers (decode, short portions): bf16, mma.sync tensor
// cores, the key axis split over CTAs.
//
// A unit is 16 rows of one key/value head of one sequence; rows are (token, query head) pairs.  Differential attention
// puts 8 pairs into a unit: rows 0-7 are their first maps, rows 8-15 the second ones, so that a thread of the
// m16n8k16 accumulator (rows g and g + 8) holds both maps of a pair and the difference is taken in registers.
//
// CTA = 8 warps over tiles of 64 keys, two tiles in flight (cp.async into padded rows: conflict-free ldmatrix):
//   scores   warp w takes 16 keys (w % 4) and one half (w / 4) of the query / key vector, whose A fragments it keeps in
//            registers for the whole launch.  For one map the halves are halves of the vector and their products are
//            added on the way through shared memory; for two maps half i IS map i.
//   softmax  16 threads per row, 4 keys each: add the halves, scale, cap, mask, online maximum in the log2 domain
//            (all inside a half-warp), p to shared memory as bf16, rescale factors beside it.
//   output   warp w owns 8 * NB value columns: O = O * alpha + P V.
// A latent cache row is key and value at once (value = its first Dv columns): it is loaded once.
// With more than one split the units' (m, l, O) go to scratch as fp32 and mixer_merge_kernel finishes the rows.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>

#include "bf16x8.cuh"
#include "mixer_attention.h"
#include "ptx_sm100.cuh"
#include "warp_reduce.cuh"

namespace l3ci {
namespace {

constexpr int kMmThreads = 256;
constexpr int kMmKeys = 64;
constexpr int kMmRows = 16;
constexpr int kMmStages = 2;
constexpr int kSPitch = kMmKeys + 4;            // floats per score row
constexpr int kPPitch = kMmKeys * 2 + 16;       // bytes per probability row
constexpr float kLog2e = 1.4426950408889634f;

struct MmParams {
  l3ci_mixer_attn_args a;
  int R, row_blocks, units, splits;
  int k_chunks, v_chunks;                       // 16-byte chunks of a key / value row (v_chunks 0: values are in the key row)
  unsigned k_magic, v_magic;                    // ceil(2^32 / chunks), 0 for one chunk
  int k_pitch, v_pitch;                         // bytes per row in shared memory
  int half_cols;                                // columns of the query / key vector per warp half
  float* o_part;                                // [units][splits][16][dv_pad]
  float* ml_part;                               // [units][splits][16][2]
  int dv_pad;
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x2_trans(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}

// i / chunks for small i, by the chunks' magic number.
__device__ __forceinline__ int div_chunks(int i, unsigned magic) { return magic ? (int)__umulhi((unsigned)i, magic) : i; }

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
__global__ void __launch_bounds__(kMmThreads) mixer_mma_kernel(const MmParams p) {
  extern __shared__ __align__(16) uint8_t smem[];
  const l3ci_mixer_attn_args& a = p.a;
  const uint32_t stage_bytes = kMmKeys * (p.k_pitch + p.v_pitch);
  const uint32_t k_smem = smem_u32(smem);
  float* sx = reinterpret_cast<float*>(smem + kMmStages * stage_bytes);   // [2 halves][16][kSPitch]
  uint8_t* pb = reinterpret_cast<uint8_t*>(sx + 2 * kMmRows * kSPitch);   // [16][kPPitch]
  float* s_alpha = reinterpret_cast<float*>(pb + kMmRows * kPPitch);      // [16]
  float* s_ml = s_alpha + kMmRows;                                        // [16][2]
  float* s_ss = s_ml + 2 * kMmRows;                                       // [8 warps][8 rows]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;

  // key columns beyond the row (up to a whole k-step) read as zero: the copies never write them
  for (int i = tid; i < kMmStages * kMmKeys; i += kMmThreads) {
    uint8_t* row = smem + (i / kMmKeys) * stage_bytes + (i % kMmKeys) * p.k_pitch;
    for (int c = p.k_chunks * 16; c < p.k_pitch; c += 16) *reinterpret_cast<uint4*>(row + c) = make_uint4(0, 0, 0, 0);
  }

  pdl_wait();
  pdl_launch_dependents();

  constexpr int kPairs = MAPS == 2 ? kMmRows / 2 : kMmRows;   // (token, head) pairs per unit
  const int unit = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  const int rb = unit % p.row_blocks, g = (unit / p.row_blocks) % a.G, b = unit / (p.row_blocks * a.G);
  const int pair0 = rb * kPairs, n_pairs = min(kPairs, a.T * p.R - pair0);
  const int pos0 = a.positions[b];
  const int keys = max(0, min(a.n_keys, pos0 + (pair0 + n_pairs - 1) / p.R + 1));
  const int tiles = (keys + kMmKeys - 1) / kMmKeys;
  const int per_split = (tiles + p.splits - 1) / p.splits;
  const int tile0 = split * per_split, tile1 = min(tiles, tile0 + per_split);

  const __nv_bfloat16* kg = static_cast<const __nv_bfloat16*>(a.ka) + b * a.ka_sb + g * a.ka_sh;
  const __nv_bfloat16* vg = static_cast<const __nv_bfloat16*>(a.v) + b * a.v_sb + g * a.v_sh;
  auto load_tile = [&](int tile, int stage) {
    const int j0 = tile * kMmKeys;
    const uint32_t dst = k_smem + stage * stage_bytes;
    for (int i = tid; i < kMmKeys * p.k_chunks; i += kMmThreads) {
      const int row = div_chunks(i, p.k_magic), c = i - row * p.k_chunks, j = j0 + row;
      cp_async16(dst + row * p.k_pitch + c * 16, kg + (j < keys ? j : 0) * a.ka_st + c * 8, j < keys);
    }
    const uint32_t vdst = dst + kMmKeys * p.k_pitch;
    for (int i = tid; i < kMmKeys * p.v_chunks; i += kMmThreads) {
      const int row = div_chunks(i, p.v_magic), c = i - row * p.v_chunks, j = j0 + row;
      cp_async16(vdst + row * p.v_pitch + c * 16, vg + (j < keys ? j : 0) * a.v_st + c * 8, j < keys);
    }
  };
  if (tile0 < tile1) load_tile(tile0, 0);
  cp_async_commit();
  if (tile0 + 1 < tile1) load_tile(tile0 + 1, 1);
  cp_async_commit();

  // ---- query fragments of this warp's half ----
  const int kg_warp = warp & 3, half = warp >> 2;
  const int dk = MAPS == 2 ? a.Da : a.Da + a.Db;
  const int col_lo = MAPS == 2 ? 0 : half * p.half_cols;                       // within the pair's vector (or map)
  const int col_hi = MAPS == 2 ? dk : min(dk, col_lo + p.half_cols);
  const int n_ks = (max(0, col_hi - col_lo) + 15) / 16;
  const int k_col0 = MAPS == 2 ? half * a.Da : col_lo;                         // first key column of the half
  uint32_t qf[KS][4];
  {
    auto q_word = [&](int row, int col) -> uint32_t {                          // columns col, col + 1 of pair `row`
      if (row >= n_pairs || col >= col_hi) return 0u;
      const int idx = pair0 + row, t = idx / p.R, h = g * p.R + idx % p.R;
      const __nv_bfloat16* qa = static_cast<const __nv_bfloat16*>(a.qa) + b * a.qa_sb + t * a.qa_st + h * a.qa_sh;
      if (MAPS == 2) return ld_global_u32(qa + half * a.Da + col);
      if (col < a.Da) return ld_global_u32(qa + col);
      return ld_global_u32(static_cast<const __nv_bfloat16*>(a.qb) + b * a.qb_sb + t * a.qb_st + h * a.qb_sh + (col - a.Da));
    };
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const int c = col_lo + ks * 16 + 2 * tig;
      // two maps: accumulator rows 8-15 of a half are not used (its 8 pairs sit in rows 0-7)
      qf[ks][0] = q_word(gid, c);
      qf[ks][1] = MAPS == 2 ? 0u : q_word(gid + 8, c);
      qf[ks][2] = q_word(gid, c + 8);
      qf[ks][3] = MAPS == 2 ? 0u : q_word(gid + 8, c + 8);
    }
  }

  // ---- this thread's softmax row: 16 threads per row, keys 4 * (tid % 16) .. + 3 of a tile ----
  const int srow = tid >> 4, skey = (tid & 15) * 4;
  const int spair = MAPS == 2 ? (srow & 7) : srow;
  const int st = (pair0 + min(spair, n_pairs - 1)) / p.R;
  const int limit = pos0 + st;                                                  // last key the row sees
  const float scale = a.scale * query_temperature(limit, a.temp_coef, a.temp_every);
  const float cap = a.softcap, cap_scale = cap > 0.f ? scale / cap : scale * kLog2e, cap_out = cap * kLog2e;
  float m_run = -INFINITY, l_run = 0.f;

  float o[NB][4];
#pragma unroll
  for (int nb = 0; nb < NB; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f;
  const int mat = lane >> 3, r8 = lane & 7;
  // K: matrices (keys 0-7, cols c..), (keys 0-7, c + 8), (keys 8-15, c), (keys 8-15, c + 8) of the warp's 16 keys
  const uint32_t k_off = (kg_warp * 16 + r8 + 8 * (mat >> 1)) * p.k_pitch + (k_col0 + 8 * (mat & 1)) * 2;
  // V transposed: matrices (keys 0-7, cols c), (keys 8-15, c), (keys 0-7, c + 8), (keys 8-15, c + 8)
  const bool v_shared = p.v_chunks == 0;
  const int v_pitch = v_shared ? p.k_pitch : p.v_pitch;
  const int v_col0 = warp * NB * 8;
  const uint32_t v_off = (v_shared ? 0u : (uint32_t)(kMmKeys * p.k_pitch)) + (r8 + 8 * (mat & 1)) * v_pitch +
                         (v_col0 + (NB > 1 ? 8 * (mat >> 1) : 0)) * 2;
  // P: matrices (rows 0-7, keys c), (rows 8-15, c), (rows 0-7, c + 8), (rows 8-15, c + 8)
  const uint32_t p_off = smem_u32(pb) + (r8 + 8 * (mat & 1)) * kPPitch + (mat >> 1) * 16;

  for (int tile = tile0; tile < tile1; ++tile) {
    const int stage = (tile - tile0) & 1;
    cp_async_wait<1>();
    __syncthreads();
    const uint32_t kt = k_smem + stage * stage_bytes;
    {
      float s[2][2][4] = {};                                                    // [k-step parity][8 keys]
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        if (ks < n_ks) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(kt + k_off + ks * 32, b0, b1, b2, b3);
          mma_bf16(s[ks & 1][0], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
          mma_bf16(s[ks & 1][1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
        }
      }
      float* dst = sx + half * kMmRows * kSPitch + gid * kSPitch + kg_warp * 16 + 2 * tig;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(s[0][n][0] + s[1][n][0], s[0][n][1] + s[1][n][1]);
        if (MAPS == 1)
          *reinterpret_cast<float2*>(dst + 8 * kSPitch + n * 8) = make_float2(s[0][n][2] + s[1][n][2], s[0][n][3] + s[1][n][3]);
      }
    }
    __syncthreads();
    {
      float v[4];
      if (MAPS == 2) {
        const float4 x = *reinterpret_cast<const float4*>(sx + ((srow >> 3) * kMmRows + (srow & 7)) * kSPitch + skey);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
      } else {
        const float4 x = *reinterpret_cast<const float4*>(sx + srow * kSPitch + skey);
        const float4 y = *reinterpret_cast<const float4*>(sx + (kMmRows + srow) * kSPitch + skey);
        v[0] = x.x + y.x; v[1] = x.y + y.y; v[2] = x.z + y.z; v[3] = x.w + y.w;
      }
      const int j = tile * kMmKeys + skey;
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[i] *= cap_scale;
        if (cap > 0.f) v[i] = cap_out * tanhf(v[i]);
        if (j + i > limit || j + i >= keys) v[i] = -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
      mx = fmaxf(m_run, group_max<16>(mx));
      const float mu = mx == -INFINITY ? 0.f : mx;
      const float alpha = fast_exp2(m_run - mu);                                // 0 at the row's first visible key
      m_run = mx;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[i] = fast_exp2(v[i] - mu);
        sum += v[i];
      }
      l_run = fmaf(l_run, alpha, sum);
      *reinterpret_cast<uint2*>(pb + srow * kPPitch + skey * 2) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
      if ((tid & 15) == 0) s_alpha[srow] = alpha;
    }
    __syncthreads();
    {
      const float al = s_alpha[gid], ah = s_alpha[gid + 8];
#pragma unroll
      for (int nb = 0; nb < NB; ++nb) { o[nb][0] *= al; o[nb][1] *= al; o[nb][2] *= ah; o[nb][3] *= ah; }
#pragma unroll
      for (int kk = 0; kk < kMmKeys / 16; ++kk) {
        uint32_t a0, a1, a2, a3;
        ldsm_x4(p_off + kk * 32, a0, a1, a2, a3);
        const uint32_t vb = kt + v_off + kk * 16 * v_pitch;
        if (NB == 1) {
          if (v_col0 < a.Dv) {
            uint32_t b0, b1;
            ldsm_x2_trans(vb, b0, b1);
            mma_bf16(o[0], a0, a1, a2, a3, b0, b1);
          }
        } else {
#pragma unroll
          for (int np = 0; np < NB / 2; ++np) {
            if (v_col0 + np * 16 < a.Dv) {
              uint32_t b0, b1, b2, b3;
              ldsm_x4_trans(vb + np * 32, b0, b1, b2, b3);
              mma_bf16(o[2 * np], a0, a1, a2, a3, b0, b1);
              mma_bf16(o[(2 * np + 1) % NB], a0, a1, a2, a3, b2, b3);
            }
          }
        }
      }
    }
    __syncthreads();   // every warp is done with this stage
    if (tile + 2 < tile1) load_tile(tile + 2, stage);
    cp_async_commit();
  }
  cp_async_wait<0>();

  // ---- the rows' sums, then the output or the partial record ----
  const float l_all = group_sum<16>(l_run);
  if ((tid & 15) == 0) {
    s_ml[2 * srow] = m_run;
    s_ml[2 * srow + 1] = l_all;
  }
  __syncthreads();
  if (p.splits > 1) {
    const long long rec = (long long)unit * p.splits + split;
    if (tid < 2 * kMmRows) p.ml_part[rec * 2 * kMmRows + tid] = s_ml[tid];
    float* dst = p.o_part + rec * kMmRows * p.dv_pad;
#pragma unroll
    for (int nb = 0; nb < NB; ++nb) {
      const int col = v_col0 + nb * 8 + 2 * tig;
      *reinterpret_cast<float2*>(dst + gid * p.dv_pad + col) = make_float2(o[nb][0], o[nb][1]);
      *reinterpret_cast<float2*>(dst + (gid + 8) * p.dv_pad + col) = make_float2(o[nb][2], o[nb][3]);
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
      for (int i = 0; i < 2; ++i) {
        o[nb][i] = o[nb][i] * i0 - a.lambda * (o[nb][2 + i] * i1);
        if (v_col0 + nb * 8 + 2 * tig + i < a.Dv) ss = fmaf(o[nb][i], o[nb][i], ss);
      }
    ss = group_sum<4>(ss);
    if (tig == 0) s_ss[warp * 8 + gid] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += s_ss[w * 8 + gid];
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

// Folds the splits of one (token, head) pair: a CTA per pair.
constexpr int kMergeThreads = 128;
constexpr int kMergeCols = 4;   // pairs of columns per thread: Dv <= 1024

template <int MAPS>
__global__ void __launch_bounds__(kMergeThreads) mixer_merge_kernel(const MmParams p) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const l3ci_mixer_attn_args& a = p.a;
  constexpr int kPairs = MAPS == 2 ? kMmRows / 2 : kMmRows;
  const int unit = blockIdx.x / kPairs, pair = blockIdx.x % kPairs;
  const int rb = unit % p.row_blocks, g = (unit / p.row_blocks) % a.G, b = unit / (p.row_blocks * a.G);
  const int idx = rb * kPairs + pair;
  if (idx >= a.T * p.R) return;
  const int t = idx / p.R, h = g * p.R + idx % p.R;
  float acc[MAPS][kMergeCols][2];
#pragma unroll
  for (int m = 0; m < MAPS; ++m) {
    const float* ml = p.ml_part + ((long long)unit * p.splits * kMmRows + pair + 8 * m) * 2;
    float mx = -INFINITY;
    for (int s = 0; s < p.splits; ++s) mx = fmaxf(mx, ml[s * 2 * kMmRows]);
    const float mu = mx == -INFINITY ? 0.f : mx;
    float l = 0.f;
#pragma unroll
    for (int c = 0; c < kMergeCols; ++c) acc[m][c][0] = acc[m][c][1] = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float ls = ml[s * 2 * kMmRows + 1];
      const float w = fast_exp2(ml[s * 2 * kMmRows] - mu);
      if (!(ls > 0.f)) continue;   // a split without a visible key
      l = fmaf(ls, w, l);
      const float* src = p.o_part + (((long long)unit * p.splits + s) * kMmRows + pair + 8 * m) * p.dv_pad;
#pragma unroll
      for (int c = 0; c < kMergeCols; ++c) {
        const int col = 2 * (threadIdx.x + c * kMergeThreads);
        if (col < a.Dv) {
          const float2 x = *reinterpret_cast<const float2*>(src + col);
          acc[m][c][0] = fmaf(x.x, w, acc[m][c][0]);
          acc[m][c][1] = fmaf(x.y, w, acc[m][c][1]);
        }
      }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int c = 0; c < kMergeCols; ++c) { acc[m][c][0] *= inv; acc[m][c][1] *= inv; }
  }
  float f = 1.f;
  if (MAPS == 2) {
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < kMergeCols; ++c)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        acc[0][c][i] -= a.lambda * acc[MAPS - 1][c][i];
        ss = fmaf(acc[0][c][i], acc[0][c][i], ss);
      }
    f = differential_factor(a, cta_sum(ss, red, kMergeThreads / kWarp), b, t, h);
  }
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + b * a.o_sb + t * a.o_st + h * a.o_sh;
#pragma unroll
  for (int c = 0; c < kMergeCols; ++c) {
    const int col = 2 * (threadIdx.x + c * kMergeThreads);
    if (col < a.Dv) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(acc[0][c][0] * f, acc[0][c][1] * f);
  }
}

int steps_per_half(const l3ci_mixer_attn_args* a) {
  return a->maps == 2 ? (a->Da + 15) / 16 : ((a->Da + a->Db + 15) / 16 + 1) / 2;
}
bool values_in_keys(const l3ci_mixer_attn_args* a) {
  return a->v == a->ka && a->v_st == a->ka_st && a->v_sb == a->ka_sb && (a->G == 1 || a->v_sh == a->ka_sh) && a->Dv <= a->maps * a->Da + a->Db;
}
size_t mma_smem(const MmParams& p) {
  return (size_t)kMmStages * kMmKeys * (p.k_pitch + p.v_pitch) + 2 * kMmRows * kSPitch * 4 + kMmRows * kPPitch + 3 * kMmRows * 4 + 64 * 4;
}

MmParams mma_params(const l3ci_mixer_attn_args* a) {
  MmParams p = {};
  p.a = *a;
  p.R = a->H / a->G;
  const int pairs = a->maps == 2 ? kMmRows / 2 : kMmRows;
  p.row_blocks = (int)(((long long)a->T * p.R + pairs - 1) / pairs);
  p.units = a->B * a->G * p.row_blocks;
  const int width = a->maps * a->Da + a->Db;
  const bool shared = values_in_keys(a);
  p.k_chunks = width / 8;
  p.v_chunks = shared ? 0 : a->Dv / 8;
  auto magic = [](int n) { return n > 1 ? (unsigned)((0x100000000ull + n - 1) / n) : 0u; };
  p.k_magic = magic(p.k_chunks);
  p.v_magic = magic(p.v_chunks);
  // rows as long as the last k-step (or column pair) reads, an odd number of 16-byte chunks apart
  auto pitch = [](int bytes) { return (bytes + 15) / 16 * 16 + (((bytes + 15) / 16) % 2 ? 0 : 16); };
  const int ks = steps_per_half(a);
  p.half_cols = ks * 16;
  const int k_read = a->maps == 2 ? (a->Da + ks * 16) : 2 * ks * 16, v_read = (a->Dv + 15) / 16 * 16;
  p.k_pitch = pitch(2 * (shared && v_read > k_read ? v_read : k_read > width ? k_read : width));
  p.v_pitch = shared ? 0 : pitch(2 * v_read);
  p.dv_pad = a->Dv <= 64 ? 64 : a->Dv <= 128 ? 128 : a->Dv <= 256 ? 256 : 512;
  // splits: whole waves of CTAs over the device, each a run of tiles plus a fixed cost of about two
  const int sms = sm_count() > 0 ? sm_count() : 148;
  const int per_sm = (int)((size_t)(220 << 10) / mma_smem(p));
  const long long slots = (long long)sms * (per_sm < 1 ? 1 : per_sm > 2 ? 2 : per_sm);
  const int keys = a->start_pos >= 0 && a->start_pos + a->T < a->n_keys ? a->start_pos + a->T : a->n_keys;
  const int tiles = keys > 0 ? (keys + kMmKeys - 1) / kMmKeys : 1;
  double best = 0;
  p.splits = 1;
  for (int s = 1; s <= tiles && s <= 64; ++s) {
    if (s > 1 && (long long)p.units * s > 4 * slots) break;
    const long long waves = ((long long)p.units * s + slots - 1) / slots;
    const double cost = waves * ((tiles + s - 1) / s + 2.0) + (s > 1 ? 2.0 : 0.0);
    if (s == 1 || cost < best) { best = cost; p.splits = s; }
  }
  return p;
}

template <int KS, int NB, int MAPS>
int launch_mma(const MmParams& p, size_t smem, cudaStream_t stream) {
  static bool configured[64] = {false};
  int dev = 0;
  L3CI_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    L3CI_CUDA_TRY(cudaFuncSetAttribute(mixer_mma_kernel<KS, NB, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, max_smem_optin()));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  L3CI_LAUNCH("mixer_mma_kernel", mixer_mma_kernel<KS, NB, MAPS>, dim3((unsigned)(p.units * p.splits)), dim3(kMmThreads), smem, stream, p);
  return L3CI_OK;
}
template <int KS, int MAPS>
int launch_mma_nb(const MmParams& p, size_t smem, cudaStream_t stream) {
  switch (p.dv_pad) {
    case 64: return launch_mma<KS, 1, MAPS>(p, smem, stream);
    case 128: return launch_mma<KS, 2, MAPS>(p, smem, stream);
    case 256: return launch_mma<KS, 4, MAPS>(p, smem, stream);
    default: return launch_mma<KS, 8, MAPS>(p, smem, stream);
  }
}
template <int MAPS>
int launch_mma_ks(const MmParams& p, size_t smem, cudaStream_t stream) {
  const int ks = steps_per_half(&p.a);
  if (ks <= 4) return launch_mma_nb<4, MAPS>(p, smem, stream);
  if (ks <= 8) return launch_mma_nb<8, MAPS>(p, smem, stream);
  return launch_mma_nb<18, MAPS>(p, smem, stream);
}
size_t scratch_of(const MmParams& p) {
  return p.splits > 1 ? (size_t)p.units * p.splits * kMmRows * (p.dv_pad + 2) * sizeof(float) : 0;
}

}  // namespace

bool mixer_mma_applies(const l3ci_mixer_attn_args* a) {
  if (a->dtype != L3CI_BF16 || a->Dv > 512 || a->Dv % 8 || a->Da % 8 || a->Db % 8 || steps_per_half(a) > 18) return false;
  if (a->Db && (static_cast<const uint16_t*>(a->kb) != static_cast<const uint16_t*>(a->ka) + a->Da || a->kb_st != a->ka_st ||
                a->kb_sb != a->ka_sb || (a->G > 1 && a->kb_sh != a->ka_sh)))
    return false;   // the two key parts must be one row
  auto rows16 = [](const void* ptr, int64_t sb, int64_t st, int64_t sh) { return aligned16(ptr) && (sb | st | sh) % 8 == 0; };
  auto rows4 = [](const void* ptr, int64_t sb, int64_t st, int64_t sh) {
    return reinterpret_cast<uintptr_t>(ptr) % 4 == 0 && (sb | st | sh) % 2 == 0;
  };
  if (!rows16(a->ka, a->ka_sb, a->ka_st, a->G > 1 ? a->ka_sh : 0) || !rows16(a->v, a->v_sb, a->v_st, a->G > 1 ? a->v_sh : 0)) return false;
  if (!rows4(a->qa, a->qa_sb, a->qa_st, a->qa_sh) || (a->Db && !rows4(a->qb, a->qb_sb, a->qb_st, a->qb_sh)) ||
      !rows4(a->out, a->o_sb, a->o_st, a->o_sh))
    return false;
  const long long rows = (long long)a->T * (a->H / a->G);
  if ((long long)a->B * a->G * ((rows + 7) / 8) * 64 > 0x7fffffffLL || rows > 0x7fffffffLL) return false;
  const MmParams p = mma_params(a);
  return mma_smem(p) <= (size_t)(227 << 10);
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
  const size_t smem = mma_smem(p);
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(a->stream);
  if (int st = a->maps == 2 ? launch_mma_ks<2>(p, smem, stream) : launch_mma_ks<1>(p, smem, stream)) return st;
  if (p.splits > 1) {
    const unsigned ctas = (unsigned)(p.units * (a->maps == 2 ? kMmRows / 2 : kMmRows));
    if (a->maps == 2) L3CI_LAUNCH("mixer_merge_kernel", mixer_merge_kernel<2>, dim3(ctas), dim3(kMergeThreads), 0, stream, p);
    else L3CI_LAUNCH("mixer_merge_kernel", mixer_merge_kernel<1>, dim3(ctas), dim3(kMergeThreads), 0, stream, p);
  }
  return L3CI_OK;
}

}  // namespace l3ci
