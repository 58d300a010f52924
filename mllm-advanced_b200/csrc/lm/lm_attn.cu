// Softmax attention of the language-model engine over keys and values in rows per head (slot caches
// [slot][kv_heads][max_ctx][dim], or keys and values made from latents for one step), with grouped query
// heads, a learned distance bias (a table per layer and head, indexed by min(distance, bias_max)) and an optional sink:
// a key of score 0 without a value, i.e. one more term exp(0) in the denominator.  Keys and values of the step are in
// the caches already.  Scores, weights and sums are fp32; the bf16 kernels multiply bf16 queries and keys exactly into
// fp32 and feed the weights to the value product as a sum of two bf16 numbers.
//   * lm_attn_prefill_kernel: tiles of 64 (token, head) rows that share a kv head, key blocks of 64 through a
//     double-buffered cp.async ring, mma.sync m16n8k16, online softmax in registers, two warps per 16 rows.
//   * lm_attn_decode_kernel + lm_attn_combine_kernel: one token per sequence, the context split over CTAs in chunks of 64
//     or 128 positions, the query heads of a kv head as the rows of one mma tile.
//   * lm_attn_f32_kernel: the 32-bit mode, any step.
#include <algorithm>

#include "../device_common.cuh"
#include "lm_state.h"

namespace mllmb200 {
namespace lm {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kNegInf = -3.402823466e+38f;

// ------------------------------------------------------------------------------------------ fp32, any row
constexpr int kF32Threads = 128;

// NV: value columns per thread
template <int NV>
__global__ void __launch_bounds__(kF32Threads) lm_attn_f32_kernel(AttnShape a, const float* __restrict__ q, int ldq,
                                                                  const int2* __restrict__ row_sp, const float* __restrict__ kc,
                                                                  const float* __restrict__ vc, const float* __restrict__ bias,
                                                                  float* __restrict__ out, int ldo) {
  __shared__ __align__(16) float sq[1024], sp[kF32Threads], red[kF32Threads / 32];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int row = blockIdx.x, h = blockIdx.y, g = h / (a.heads / a.kv_heads), tid = threadIdx.x;
  const int2 s = row_sp[row];
  const size_t base = s.x * a.slot_rows + g * a.head_rows;
  for (int d = tid; d < a.dimp; d += kF32Threads) sq[d] = q[(size_t)row * ldq + h * a.dimp + d];
  float m = a.sink ? 0.0f : kNegInf, l = a.sink ? 1.0f : 0.0f, acc[NV] = {};
  auto block_reduce = [&](float v, bool is_max) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float w = __shfl_xor_sync(0xffffffffu, v, o);
      v = is_max ? fmaxf(v, w) : v + w;
    }
    __syncthreads();
    if ((tid & 31) == 0) red[tid >> 5] = v;
    __syncthreads();
    return is_max ? fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])) : (red[0] + red[1]) + (red[2] + red[3]);
  };
  __syncthreads();
  for (int j0 = 0; j0 <= s.y; j0 += kF32Threads) {
    const int j = j0 + tid;
    float sc = kNegInf;
    if (j <= s.y) {
      const float4* kr = reinterpret_cast<const float4*>(kc + (base + j) * a.dimp);
      float dot = 0.0f;
      for (int d = 0; d < a.dimp / 4; ++d) {
        const float4 kv = kr[d], qv = reinterpret_cast<const float4*>(sq)[d];
        dot = fmaf(kv.x, qv.x, dot), dot = fmaf(kv.y, qv.y, dot), dot = fmaf(kv.z, qv.z, dot), dot = fmaf(kv.w, qv.w, dot);
      }
      sc = dot * a.scale;
      if (a.has_bias) sc += bias[(size_t)h * (a.bias_max + 1) + min(s.y - j, a.bias_max)];
    }
    const float m_new = fmaxf(m, block_reduce(sc, true));
    const float p = j <= s.y ? expf(sc - m_new) : 0.0f, alpha = expf(m - m_new);
    sp[tid] = p;
    l = l * alpha + block_reduce(p, false);  // its barriers publish sp
    m = m_new;
    const int nk = min(kF32Threads, s.y + 1 - j0);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = tid + i * kF32Threads;
      if (d < a.vdimp) {
        float o = acc[i] * alpha;
        for (int t = 0; t < nk; ++t) o = fmaf(sp[t], vc[(base + j0 + t) * a.vdimp + d], o);
        acc[i] = o;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int d = tid + i * kF32Threads;
    if (d < a.vdimp) out[(size_t)row * ldo + h * a.vdimp + d] = acc[i] / l;
  }
}

// ------------------------------------------------------------------------------------------ bf16 prompts
constexpr int kPfRows = 64, kPfKeys = 64, kPfThreads = 256;

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

__device__ __forceinline__ float fast_exp2(float x) {  // results below 2^-126 are 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// entries of a tile's bias window per head: distances of all (token, key) pairs, rounded up to whole 16-byte pieces
__host__ __device__ inline int bias_window(int toks) { return (kPfKeys + toks + 3) / 4 * 4; }

size_t prefill_smem(const AttnShape& a) {
  const int group = a.heads / a.kv_heads, toks = kPfRows / group;
  const size_t kv = (size_t)(2 * kPfKeys) * (a.dimp + 8) * 2 + (size_t)(2 * kPfKeys) * (a.vdimp + 8) * 2;
  return (size_t)kPfRows * (a.dimp + 8) * 2 + std::max(kv, (size_t)kPfRows * a.vdimp * 4) +
         (a.has_bias ? (size_t)2 * group * bias_window(toks) * 4 : 0);
}

// grid (tiles, kv heads); tile = {first row, tokens, slot, position of the first token}.  Eight warps: warp w and warp
// w + 4 own the same 16 rows and one half each of every key block; their online-softmax states meet at the end.
template <int DV>
__global__ void __launch_bounds__(kPfThreads) lm_attn_prefill_kernel(AttnShape a, const __nv_bfloat16* __restrict__ q, int ldq,
                                                                     const __nv_bfloat16* __restrict__ kc,
                                                                     const __nv_bfloat16* __restrict__ vc,
                                                                     const float* __restrict__ bias, const int4* __restrict__ tiles,
                                                                     __nv_bfloat16* __restrict__ out, int ldo) {
  extern __shared__ __align__(16) uint8_t pf_smem[];
  __shared__ float s_m[kPfRows], s_l[kPfRows];
  constexpr int kHalf = kPfKeys / 2;
  const int D = a.dimp, group = a.heads / a.kv_heads, toks = kPfRows / group;
  const int ldk = D + 8, ldv = a.vdimp + 8, win = bias_window(toks);
  // [2][group][win] biases | queries | 2 x keys | 2 x values; the partial outputs of warps 4..7 overlay keys and values
  float* sB = reinterpret_cast<float*>(pf_smem);
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(sB + (a.has_bias ? 2 * group * win : 0));
  __nv_bfloat16* sK = sQ + kPfRows * ldk;
  __nv_bfloat16* sV = sK + 2 * kPfKeys * ldk;
  float* sO = reinterpret_cast<float*>(sK);
  pdl_launch_dependents();
  pdl_wait_prior();
  const int4 tile = tiles[blockIdx.x];
  const int kvh = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, half = warp >> 2, wrow = (warp & 3) * 16;
  const int row0 = tile.x, ntok = tile.y, pos0 = tile.w, last = pos0 + ntok - 1;
  const __nv_bfloat16* kb = kc + (tile.z * a.slot_rows + kvh * a.head_rows) * D;
  const __nv_bfloat16* vb = vc + (tile.z * a.slot_rows + kvh * a.head_rows) * a.vdimp;
  const int dv8 = D / 8, vv8 = a.vdimp / 8;
  // copies: eight threads per row of 16-byte pieces
  const int cr = tid >> 3, cc = tid & 7;
  for (int r = cr; r < kPfRows; r += kPfThreads / 8) {
    const int tok = r / group, hg = r - tok * group;
    const bool ok = tok < ntok && tok < toks;
    const __nv_bfloat16* src = q + (size_t)(row0 + (ok ? tok : 0)) * ldq + (kvh * group + hg) * D;
    for (int c = cc; c < dv8; c += 8) cp_async16(smem_u32(sQ + r * ldk + c * 8), src + c * 8, ok);
  }
  auto fetch = [&](int j0, int buf) {
#pragma unroll
    for (int u = 0; u < kPfKeys / (kPfThreads / 8); ++u) {
      const int r = cr + u * (kPfThreads / 8);
      const bool ok = j0 + r <= last;
      const size_t at = ok ? j0 + r : 0;
      const uint32_t dk = smem_u32(sK + (buf * kPfKeys + r) * ldk), dv = smem_u32(sV + (buf * kPfKeys + r) * ldv);
      for (int c = cc; c < dv8; c += 8) cp_async16(dk + c * 16, kb + at * D + c * 8, ok);
      for (int c = cc; c < vv8; c += 8) cp_async16(dv + c * 16, vb + at * a.vdimp + c * 8, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  // this thread's two rows of the tile (rows past the tile's tokens compute on zeros and are not stored)
  int tok_r[2], hg_r[2], b_at[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = wrow + (lane >> 2) + i * 8;
    tok_r[i] = r / group;
    hg_r[i] = r - tok_r[i] * group;
    b_at[i] = hg_r[i] * win + min(tok_r[i], toks - 1) + kPfKeys - 1 - half * kHalf - (lane & 3) * 2;
  }
  // the mask value is far below every running maximum, so that masked weights come out as 0
  constexpr float kStart = -1e30f;
  float m[2], l[2], o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    m[i] = a.sink ? 0.0f : kStart;
    l[i] = a.sink && half == 0 && (lane & 3) == 0 ? 1.0f : 0.0f;
  }
#pragma unroll
  for (int n = 0; n < DV / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
  const int mat = lane >> 3, ml = lane & 7;
  const uint32_t q_addr = smem_u32(sQ + (wrow + (mat & 1) * 8 + ml) * ldk + (mat >> 1) * 8);
  const uint32_t k_addr = smem_u32(sK + (half * kHalf + (mat >> 1) * 8 + ml) * ldk + (mat & 1) * 8);
  const uint32_t v_addr = smem_u32(sV + (half * kHalf + (mat & 1) * 8 + ml) * ldv + (mat >> 1) * 8);
  const float sc2 = a.scale * kLog2e;

  for (int j0 = 0, blk = 0; j0 <= last; j0 += kPfKeys, ++blk) {
    const int buf = blk & 1;
    float* bw = sB + (size_t)buf * group * win;
    const int n_lo = pos0 - (j0 + kPfKeys - 1);  // distance of the window's first entry
    if (a.has_bias)
      for (int hg = warp; hg < group; hg += kPfThreads / 32) {
        const float* bh = bias + (size_t)(kvh * group + hg) * (a.bias_max + 1);
        for (int i = lane; i < win; i += 32) bw[hg * win + i] = kLog2e * __ldg(bh + min(max(n_lo + i, 0), a.bias_max));
      }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (j0 + kPfKeys <= last) fetch(j0 + kPfKeys, buf ^ 1);
    const int jw = j0 + half * kHalf;  // this warp's first key
    float s[kHalf / 8][4];
#pragma unroll
    for (int n = 0; n < kHalf / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
#pragma unroll 4
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t qa[4];
      ldsm4(qa, q_addr + kk * 2);
#pragma unroll
      for (int n = 0; n < kHalf / 16; ++n) {
        uint32_t b[4];
        ldsm4(b, k_addr + ((buf * kPfKeys + n * 16) * ldk + kk) * 2);
        mma_bf16(s[2 * n], qa, b[0], b[1]);
        mma_bf16(s[2 * n + 1], qa, b[2], b[3]);
      }
    }
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int n = 0; n < kHalf / 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float b = a.has_bias ? bw[b_at[i >> 1] - n * 8 - (i & 1)] : 0.0f;
        s[n][i] = fmaf(s[n][i], sc2, b);
      }
    if (jw + kHalf - 1 > pos0) {  // some keys are later than some rows
#pragma unroll
      for (int n = 0; n < kHalf / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (jw + n * 8 + (lane & 3) * 2 + (i & 1) > pos0 + tok_r[i >> 1]) s[n][i] = kNegInf;
    }
#pragma unroll
    for (int n = 0; n < kHalf / 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      alpha[r] = fast_exp2(m[r] - mx[r]);
      m[r] = mx[r];
      l[r] *= alpha[r];
    }
#pragma unroll
    for (int n = 0; n < kHalf / 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[n][i] = fast_exp2(s[n][i] - m[i >> 1]);
        l[i >> 1] += s[n][i];
      }
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) o[n][0] *= alpha[0], o[n][1] *= alpha[0], o[n][2] *= alpha[1], o[n][3] *= alpha[1];
#pragma unroll
    for (int kk = 0; kk < kHalf / 16; ++kk) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float p0 = s[2 * kk + (i >> 1)][(i & 1) * 2], p1 = s[2 * kk + (i >> 1)][(i & 1) * 2 + 1];
        hi[i] = pack2(p0, p1);
        lo[i] = pack2(p0 - __uint_as_float(hi[i] << 16), p1 - __uint_as_float(hi[i] & 0xffff0000u));
      }
#pragma unroll
      for (int n = 0; n < DV / 16; ++n) {
        if (n * 16 < a.vdimp) {
          uint32_t b[4];
          ldsm4_t(b, v_addr + ((buf * kPfKeys + kk * 16) * ldv + n * 16) * 2);
          mma_bf16(o[2 * n], hi, b[0], b[1]);
          mma_bf16(o[2 * n + 1], hi, b[2], b[3]);
          mma_bf16(o[2 * n], lo, b[0], b[1]);
          mma_bf16(o[2 * n + 1], lo, b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  __syncthreads();  // keys and values are used up
  if (half == 1) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = wrow + (lane >> 2) + r * 8;
      if ((lane & 3) == 0) s_m[row] = m[r], s_l[row] = l[r];
      float* so = sO + (size_t)row * a.vdimp + (lane & 3) * 2;
#pragma unroll
      for (int n = 0; n < DV / 8; ++n)
        if (n * 8 < a.vdimp) *reinterpret_cast<float2*>(so + n * 8) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
    }
  }
  __syncthreads();
  if (half == 1) return;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    if (tok_r[r] >= ntok || tok_r[r] >= toks) continue;
    const int row = wrow + (lane >> 2) + r * 8;
    const float mo = s_m[row], mt = fmaxf(m[r], mo), f0 = fast_exp2(m[r] - mt), f1 = fast_exp2(mo - mt);
    const float inv = 1.0f / (l[r] * f0 + s_l[row] * f1), g0 = f0 * inv, g1 = f1 * inv;
    const float* so = sO + (size_t)row * a.vdimp + (lane & 3) * 2;
    __nv_bfloat16* orow = out + (size_t)(row0 + tok_r[r]) * ldo + (kvh * group + hg_r[r]) * a.vdimp + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
      if (n * 8 < a.vdimp) {
        const float2 w = *reinterpret_cast<const float2*>(so + n * 8);
        *reinterpret_cast<uint32_t*>(orow + n * 8) = pack2(fmaf(o[n][2 * r], g0, w.x * g1), fmaf(o[n][2 * r + 1], g0, w.y * g1));
      }
  }
}

// ------------------------------------------------------------------------------------------ bf16 decode
constexpr int kDecThreads = 128, kDecWarps = 4, kDecRows = 16;  // query heads per CTA: the rows of one mma tile

size_t decode_smem(const AttnShape& a, int chunk) {
  const size_t tiles = (size_t)chunk * (a.dimp + 8 + a.vdimp + 8) * 2, merge = (size_t)kDecWarps * kDecRows * a.vdimp * 4;
  return (size_t)kDecRows * (a.dimp + 8) * 2 + std::max(tiles, merge);
}

// grid (splits, kv heads x blocks of 16 query heads, single rows).  A CTA takes WK x 64 cache positions: all of their
// keys and values are requested at once, each warp multiplies WK x 16 of them with the block's query heads, and the
// warps' online-softmax states meet in shared memory.  One split: the result; else {max, sum} (base 2) and the
// unnormalized output per split.
template <int DV, int WK>
__global__ void __launch_bounds__(kDecThreads) lm_attn_decode_kernel(AttnShape a, const __nv_bfloat16* __restrict__ q, int ldq,
                                                                     const int* __restrict__ single_rows,
                                                                     const int2* __restrict__ row_sp,
                                                                     const __nv_bfloat16* __restrict__ kc,
                                                                     const __nv_bfloat16* __restrict__ vc,
                                                                     const float* __restrict__ bias, __nv_bfloat16* __restrict__ out,
                                                                     int ldo, float* __restrict__ part_o, float2* __restrict__ part_ml) {
  extern __shared__ __align__(16) uint8_t dec_smem[];
  __shared__ float s_m[kDecWarps][kDecRows], s_l[kDecWarps][kDecRows];
  constexpr int kKeys = 64 * WK;
  pdl_launch_dependents();
  pdl_wait_prior();
  const int D = a.dimp, group = a.heads / a.kv_heads, hblocks = (group + kDecRows - 1) / kDecRows;
  const int ldk = D + 8, ldv = a.vdimp + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(dec_smem);
  __nv_bfloat16* sK = sQ + kDecRows * ldk;
  __nv_bfloat16* sV = sK + kKeys * ldk;
  float* sO = reinterpret_cast<float*>(sK);  // [warps][rows][vdimp], once keys and values are used up
  const int split = blockIdx.x, splits = gridDim.x, kvh = blockIdx.y / hblocks, hb0 = (blockIdx.y - kvh * hblocks) * kDecRows;
  const int idx = blockIdx.z, row = single_rows ? single_rows[idx] : idx;
  const int2 sp = row_sp[row];
  const int j0 = split * kKeys, nk = min(kKeys, sp.y + 1 - j0);
  if (nk <= 0) return;
  const int nh = min(kDecRows, group - hb0), h0 = kvh * group + hb0, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const size_t base = sp.x * a.slot_rows + kvh * a.head_rows + j0;
  const int dv8 = D / 8, vv8 = a.vdimp / 8;
  const int cr = tid >> 3, cc = tid & 7;  // copies: eight threads per row of 16-byte pieces
  for (int c = cc; c < dv8; c += 8)
    cp_async16(smem_u32(sQ + cr * ldk + c * 8), q + (size_t)row * ldq + (size_t)(h0 + (cr < nh ? cr : 0)) * D + c * 8, cr < nh);
#pragma unroll
  for (int u = 0; u < kKeys / 16; ++u) {
    const int r = cr + u * 16;
    const __nv_bfloat16* src = kc + (base + (r < nk ? r : 0)) * D;
    for (int c = cc; c < dv8; c += 8) cp_async16(smem_u32(sK + r * ldk + c * 8), src + c * 8, r < nk);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
  for (int u = 0; u < kKeys / 16; ++u) {
    const int r = cr + u * 16;
    const __nv_bfloat16* src = vc + (base + (r < nk ? r : 0)) * a.vdimp;
    for (int c = cc; c < vv8; c += 8) cp_async16(smem_u32(sV + r * ldv + c * 8), src + c * 8, r < nk);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int k0 = warp * 16 * WK, mat = lane >> 3, ml = lane & 7;
  float s[2 * WK][4], m[2] = {kNegInf, kNegInf}, l[2] = {0.0f, 0.0f}, o[DV / 8][4];
#pragma unroll
  for (int n = 0; n < 2 * WK; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {  // the bias (base 2), while the keys are on their way
      const int hr = (lane >> 2) + (i >> 1) * 8, dist = sp.y - (j0 + k0 + n * 8 + (lane & 3) * 2 + (i & 1));
      s[n][i] = a.has_bias && hr < nh && dist >= 0 ? kLog2e * __ldg(bias + (size_t)(h0 + hr) * (a.bias_max + 1) + min(dist, a.bias_max)) : 0.0f;
    }
#pragma unroll
  for (int n = 0; n < DV / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  if (k0 < nk) {
    const uint32_t q_addr = smem_u32(sQ + ((mat & 1) * 8 + ml) * ldk + (mat >> 1) * 8);
    const uint32_t k_addr = smem_u32(sK + (k0 + (mat >> 1) * 8 + ml) * ldk + (mat & 1) * 8);
    float acc[2 * WK][4] = {};
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t qa[4];
      ldsm4(qa, q_addr + kk * 2);
#pragma unroll
      for (int n = 0; n < WK; ++n) {
        uint32_t b[4];
        ldsm4(b, k_addr + (n * 16 * ldk + kk) * 2);
        mma_bf16(acc[2 * n], qa, b[0], b[1]);
        mma_bf16(acc[2 * n + 1], qa, b[2], b[3]);
      }
    }
    const float sc2 = a.scale * kLog2e;
#pragma unroll
    for (int n = 0; n < 2 * WK; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = k0 + n * 8 + (lane & 3) * 2 + (i & 1);
        s[n][i] = c < nk ? fmaf(acc[n][i], sc2, s[n][i]) : kNegInf;
        m[i >> 1] = fmaxf(m[i >> 1], s[n][i]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      m[r] = fmaxf(m[r], __shfl_xor_sync(0xffffffffu, m[r], 1));
      m[r] = fmaxf(m[r], __shfl_xor_sync(0xffffffffu, m[r], 2));
    }
#pragma unroll
    for (int n = 0; n < 2 * WK; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[n][i] = s[n][i] == kNegInf ? 0.0f : exp2f(s[n][i] - m[i >> 1]);
        l[i >> 1] += s[n][i];
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
      l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (k0 < nk) {
    const uint32_t v_addr = smem_u32(sV + (k0 + (mat & 1) * 8 + ml) * ldv + (mat >> 1) * 8);
#pragma unroll
    for (int kk = 0; kk < WK; ++kk) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float p0 = s[2 * kk + (i >> 1)][(i & 1) * 2], p1 = s[2 * kk + (i >> 1)][(i & 1) * 2 + 1];
        hi[i] = pack2(p0, p1);
        lo[i] = pack2(p0 - __uint_as_float(hi[i] << 16), p1 - __uint_as_float(hi[i] & 0xffff0000u));
      }
#pragma unroll
      for (int n = 0; n < DV / 16; ++n)
        if (n * 16 < a.vdimp) {
          uint32_t b[4];
          ldsm4_t(b, v_addr + (kk * 16 * ldv + n * 16) * 2);
          mma_bf16(o[2 * n], hi, b[0], b[1]);
          mma_bf16(o[2 * n], lo, b[0], b[1]);
          mma_bf16(o[2 * n + 1], hi, b[2], b[3]);
          mma_bf16(o[2 * n + 1], lo, b[2], b[3]);
        }
    }
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int hr = (lane >> 2) + r * 8;
    if ((lane & 3) == 0) s_m[warp][hr] = m[r], s_l[warp][hr] = l[r];
    float* so = sO + ((size_t)warp * kDecRows + hr) * a.vdimp + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
      if (n * 8 < a.vdimp) *reinterpret_cast<float2*>(so + n * 8) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
  }
  __syncthreads();
  const bool whole = splits == 1;
  for (int i = tid; i < nh * a.vdimp; i += kDecThreads) {
    const int h = i / a.vdimp;
    float mx = whole && a.sink ? 0.0f : kNegInf, sum, v = 0.0f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) mx = fmaxf(mx, s_m[w][h]);
    sum = whole && a.sink ? exp2f(-mx) : 0.0f;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) {
      const float f = exp2f(s_m[w][h] - mx);
      sum = fmaf(f, s_l[w][h], sum);
      v = fmaf(f, sO[(size_t)w * kDecRows * a.vdimp + i], v);
    }
    if (whole) {
      out[(size_t)row * ldo + h0 * a.vdimp + i] = __float2bfloat16_rn(v / sum);
    } else {
      const size_t at = ((size_t)idx * a.heads + h0 + h) * splits + split;
      part_o[at * a.vdimp + (i - h * a.vdimp)] = v;
      if (i == h * a.vdimp) part_ml[at] = make_float2(mx, sum);
    }
  }
}

// grid (heads, single rows): merges the splits of a row and head, the sink joining here.
__global__ void __launch_bounds__(128) lm_attn_combine_kernel(AttnShape a, int chunk, int splits, const int* __restrict__ single_rows,
                                                              const int2* __restrict__ row_sp, const float* __restrict__ part_o,
                                                              const float2* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                                                              int ldo) {
  extern __shared__ float sw[];  // [splits]
  __shared__ float s_inv;
  pdl_launch_dependents();
  pdl_wait_prior();
  const int h = blockIdx.x, idx = blockIdx.y, row = single_rows ? single_rows[idx] : idx, tid = threadIdx.x;
  const int nact = min(splits, row_sp[row].y / chunk + 1);
  const float2* ml = part_ml + ((size_t)idx * a.heads + h) * splits;
  if (tid < 32) {
    float mx = a.sink ? 0.0f : kNegInf;
    for (int s = tid; s < nact; s += 32) mx = fmaxf(mx, ml[s].x);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float tot = 0.0f;
    for (int s = tid; s < nact; s += 32) {
      const float2 v = ml[s];
      const float f = exp2f(v.x - mx);
      sw[s] = f;
      tot = fmaf(v.y, f, tot);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) tot += __shfl_xor_sync(0xffffffffu, tot, o);
    if (tid == 0) s_inv = 1.0f / (tot + (a.sink ? exp2f(-mx) : 0.0f));
  }
  __syncthreads();
  const float inv = s_inv;
  for (int d = tid; d < a.vdimp; d += blockDim.x) {
    const float* po = part_o + ((size_t)idx * a.heads + h) * splits * a.vdimp + d;
    float o = 0.0f;
    for (int s0 = 0; s0 < nact; s0 += 8) {  // eight partial rows requested together
      float v[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] = po[(size_t)min(s0 + j, nact - 1) * a.vdimp];
#pragma unroll
      for (int j = 0; j < 8; ++j) o = fmaf(s0 + j < nact ? sw[s0 + j] : 0.0f, v[j], o);
    }
    out[(size_t)row * ldo + h * a.vdimp + d] = __float2bfloat16_rn(o * inv);
  }
}

constexpr int kAttnSmemMax = 220 * 1024;

}  // namespace

int attention_tile_rows() { return kPfRows; }

cudaError_t attention_configure() {
  cudaError_t r = cudaSuccess;
  auto set = [&](auto f) {
    if (r == cudaSuccess) r = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, kAttnSmemMax);
  };
  set(lm_attn_prefill_kernel<64>);
  set(lm_attn_prefill_kernel<128>);
  set(lm_attn_prefill_kernel<256>);
  set(lm_attn_decode_kernel<64, 1>);
  set(lm_attn_decode_kernel<64, 2>);
  set(lm_attn_decode_kernel<128, 1>);
  set(lm_attn_decode_kernel<128, 2>);
  set(lm_attn_decode_kernel<256, 1>);
  set(lm_attn_decode_kernel<256, 2>);
  return r;
}

// Rows in `tiles` go through the prompt kernel, `single_rows` (n_single; nullptr = rows 0 .. n_single - 1) through the
// decode kernels; in 32-bit mode all `rows` rows take one kernel.
cudaError_t launch_attention(cudaStream_t s, bool f32, const AttnShape& a, const void* q, int ldq, const int2* row_sp, int rows,
                             const void* kc, const void* vc, const float* bias, void* out, int ldo, const int4* tiles, int n_tiles,
                             const int* single_rows, int n_single, int chunk, int splits, float* part_o, float2* part_ml) {
  if (f32) {
    auto go = [&](auto f) {
      return launch_pdl(f, dim3(rows, a.heads), dim3(kF32Threads), 0, s, a, static_cast<const float*>(q), ldq, row_sp,
                        static_cast<const float*>(kc), static_cast<const float*>(vc), bias, static_cast<float*>(out), ldo);
    };
    return a.vdimp <= 2 * kF32Threads ? go(lm_attn_f32_kernel<2>) : go(lm_attn_f32_kernel<8>);
  }
  const auto* qb = static_cast<const __nv_bfloat16*>(q);
  const auto *kb = static_cast<const __nv_bfloat16*>(kc), *vb = static_cast<const __nv_bfloat16*>(vc);
  auto* ob = static_cast<__nv_bfloat16*>(out);
  cudaError_t r = cudaSuccess;
  if (n_tiles) {
    const dim3 grid(n_tiles, a.kv_heads);
    const size_t smem = prefill_smem(a);
    if (a.vdimp <= 64) r = launch_pdl(lm_attn_prefill_kernel<64>, grid, dim3(kPfThreads), smem, s, a, qb, ldq, kb, vb, bias, tiles, ob, ldo);
    else if (a.vdimp <= 128) r = launch_pdl(lm_attn_prefill_kernel<128>, grid, dim3(kPfThreads), smem, s, a, qb, ldq, kb, vb, bias, tiles, ob, ldo);
    else r = launch_pdl(lm_attn_prefill_kernel<256>, grid, dim3(kPfThreads), smem, s, a, qb, ldq, kb, vb, bias, tiles, ob, ldo);
    if (r != cudaSuccess) return r;
  }
  if (n_single) {
    const int group = a.heads / a.kv_heads;
    const dim3 grid(splits, a.kv_heads * ((group + kDecRows - 1) / kDecRows), n_single);
    const size_t smem = decode_smem(a, chunk);
    auto go = [&](auto f) { return launch_pdl(f, grid, dim3(kDecThreads), smem, s, a, qb, ldq, single_rows, row_sp, kb, vb, bias, ob, ldo, part_o, part_ml); };
    const bool two = chunk == 128;
    r = a.vdimp <= 64    ? (two ? go(lm_attn_decode_kernel<64, 2>) : go(lm_attn_decode_kernel<64, 1>))
        : a.vdimp <= 128 ? (two ? go(lm_attn_decode_kernel<128, 2>) : go(lm_attn_decode_kernel<128, 1>))
                         : (two ? go(lm_attn_decode_kernel<256, 2>) : go(lm_attn_decode_kernel<256, 1>));
    if (r == cudaSuccess && splits > 1)
      r = launch_pdl(lm_attn_combine_kernel, dim3(a.heads, n_single), dim3(128), (size_t)splits * 4, s, a, chunk, splits, single_rows,
                     row_sp, part_o, part_ml, ob, ldo);
  }
  return r;
}

}  // namespace lm
}  // namespace mllmb200
