// Softmax attention of the language-model engine over slot caches [slot][kv_heads][max_ctx][dim], with grouped query
// heads, a learned distance bias (a table per layer and head, indexed by min(distance, bias_max)) and an optional sink:
// a key of score 0 without a value, i.e. one more term exp(0) in the denominator.  Keys and values of the step are in
// the caches already.  Scores, weights and sums are fp32; the bf16 kernels multiply bf16 queries and keys exactly into
// fp32 and feed the weights to the value product as a sum of two bf16 numbers.
//   * lm_attn_prefill_kernel: tiles of 64 (token, head) rows that share a kv head, key blocks of 64 through a
//     double-buffered cp.async ring, mma.sync m16n8k16, online softmax in registers.
//   * lm_attn_decode_kernel + lm_attn_combine_kernel: one token per sequence, the context split over CTAs.
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

__global__ void __launch_bounds__(kF32Threads) lm_attn_f32_kernel(AttnShape a, const float* __restrict__ q, int ldq,
                                                                  const int2* __restrict__ row_sp, const float* __restrict__ kc,
                                                                  const float* __restrict__ vc, const float* __restrict__ bias,
                                                                  float* __restrict__ out, int ldo) {
  __shared__ __align__(16) float sq[256], sp[kF32Threads], red[kF32Threads / 32];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int row = blockIdx.x, h = blockIdx.y, g = h / (a.heads / a.kv_heads), tid = threadIdx.x;
  const int2 s = row_sp[row];
  const size_t base = ((size_t)s.x * a.kv_heads + g) * a.max_ctx;
  for (int d = tid; d < a.dimp; d += kF32Threads) sq[d] = q[(size_t)row * ldq + h * a.dimp + d];
  float m = a.sink ? 0.0f : kNegInf, l = a.sink ? 1.0f : 0.0f, acc[2] = {0.0f, 0.0f};
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
    for (int i = 0; i < 2; ++i) {
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
  for (int i = 0; i < 2; ++i) {
    const int d = tid + i * kF32Threads;
    if (d < a.vdimp) out[(size_t)row * ldo + h * a.vdimp + d] = acc[i] / l;
  }
}

// ------------------------------------------------------------------------------------------ bf16 prompts
constexpr int kPfRows = 64, kPfKeys = 64, kPfThreads = 128;

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

size_t prefill_smem(const AttnShape& a) {
  const int group = a.heads / a.kv_heads, toks = kPfRows / group;
  return (size_t)(3 * kPfKeys) * (a.dimp + 8) * 2 + (size_t)(2 * kPfKeys) * (a.vdimp + 8) * 2 +
         (a.has_bias ? (size_t)2 * group * (kPfKeys + toks) * 4 : 0);
}

// grid (tiles, kv heads); tile = {first row, tokens, slot, position of the first token}
template <int DV>
__global__ void __launch_bounds__(kPfThreads) lm_attn_prefill_kernel(AttnShape a, const __nv_bfloat16* __restrict__ q, int ldq,
                                                                     const __nv_bfloat16* __restrict__ kc,
                                                                     const __nv_bfloat16* __restrict__ vc,
                                                                     const float* __restrict__ bias, const int4* __restrict__ tiles,
                                                                     __nv_bfloat16* __restrict__ out, int ldo) {
  extern __shared__ __align__(16) uint8_t pf_smem[];
  const int D = a.dimp, group = a.heads / a.kv_heads, toks = kPfRows / group;
  const int ldk = D + 8, ldv = a.vdimp + 8, win = kPfKeys + toks;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(pf_smem);
  __nv_bfloat16* sK = sQ + kPfRows * ldk;
  __nv_bfloat16* sV = sK + 2 * kPfKeys * ldk;
  float* sB = reinterpret_cast<float*>(sV + 2 * kPfKeys * ldv);  // [2][group][win]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int4 tile = tiles[blockIdx.x];
  const int kvh = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row0 = tile.x, ntok = tile.y, pos0 = tile.w, last = pos0 + ntok - 1;
  const __nv_bfloat16* kb = kc + ((size_t)tile.z * a.kv_heads + kvh) * a.max_ctx * D;
  const __nv_bfloat16* vb = vc + ((size_t)tile.z * a.kv_heads + kvh) * a.max_ctx * a.vdimp;
  const int dv8 = D / 8, vv8 = a.vdimp / 8;
  for (int i = tid; i < kPfRows * dv8; i += kPfThreads) {
    const int r = i / dv8, c = i - r * dv8, tok = r / group, hg = r - tok * group;
    const bool ok = tok < ntok && tok < toks;
    cp_async16(smem_u32(sQ + r * ldk + c * 8), q + (size_t)(row0 + (ok ? tok : 0)) * ldq + (kvh * group + hg) * D + c * 8, ok);
  }
  auto fetch = [&](int j0, int buf) {
    for (int i = tid; i < kPfKeys * dv8; i += kPfThreads) {
      const int r = i / dv8, c = i - r * dv8;
      const bool ok = j0 + r <= last;
      cp_async16(smem_u32(sK + (buf * kPfKeys + r) * ldk + c * 8), kb + (size_t)(ok ? j0 + r : 0) * D + c * 8, ok);
    }
    for (int i = tid; i < kPfKeys * vv8; i += kPfThreads) {
      const int r = i / vv8, c = i - r * vv8;
      const bool ok = j0 + r <= last;
      cp_async16(smem_u32(sV + (buf * kPfKeys + r) * ldv + c * 8), vb + (size_t)(ok ? j0 + r : 0) * a.vdimp + c * 8, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  // this thread's two rows of the tile
  int tok_r[2], hg_r[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + (lane >> 2) + i * 8;
    tok_r[i] = r / group;
    hg_r[i] = r - tok_r[i] * group;
  }
  float m[2], l[2], o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    m[i] = a.sink ? 0.0f : kNegInf;
    l[i] = a.sink && (lane & 3) == 0 ? 1.0f : 0.0f;
  }
#pragma unroll
  for (int n = 0; n < DV / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;
  const int mat = lane >> 3, ml = lane & 7;
  const uint32_t q_addr = smem_u32(sQ + (warp * 16 + (mat & 1) * 8 + ml) * ldk + (mat >> 1) * 8);
  const uint32_t k_addr = smem_u32(sK + ((mat >> 1) * 8 + ml) * ldk + (mat & 1) * 8);
  const uint32_t v_addr = smem_u32(sV + ((mat & 1) * 8 + ml) * ldv + (mat >> 1) * 8);
  const float sc2 = a.scale * kLog2e;

  for (int j0 = 0, blk = 0; j0 <= last; j0 += kPfKeys, ++blk) {
    const int buf = blk & 1;
    float* bw = sB + (size_t)buf * group * win;
    const int n_lo = pos0 - (j0 + kPfKeys - 1);  // distance of the window's first entry
    if (a.has_bias)
      for (int i = tid; i < group * win; i += kPfThreads) {
        const int hg = i / win, n = n_lo + (i - hg * win);
        bw[i] = kLog2e * __ldg(bias + (size_t)(kvh * group + hg) * (a.bias_max + 1) + min(max(n, 0), a.bias_max));
      }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (j0 + kPfKeys <= last) fetch(j0 + kPfKeys, buf ^ 1);
    float s[kPfKeys / 8][4];
#pragma unroll
    for (int n = 0; n < kPfKeys / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t qa[4];
      ldsm4(qa, q_addr + kk * 2);
#pragma unroll
      for (int n = 0; n < kPfKeys / 16; ++n) {
        uint32_t b[4];
        ldsm4(b, k_addr + ((buf * kPfKeys + n * 16) * ldk + kk) * 2);
        mma_bf16(s[2 * n], qa, b[0], b[1]);
        mma_bf16(s[2 * n + 1], qa, b[2], b[3]);
      }
    }
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int n = 0; n < kPfKeys / 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = i >> 1, c = n * 8 + (lane & 3) * 2 + (i & 1);
        const int dist = pos0 + tok_r[r] - (j0 + c);
        float v = s[n][i] * sc2;
        if (a.has_bias) v += bw[hg_r[r] * win + min(dist - n_lo, win - 1)];
        v = dist >= 0 && tok_r[r] < ntok ? v : kNegInf;
        s[n][i] = v;
        mx[r] = fmaxf(mx[r], v);
      }
    float alpha[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      alpha[r] = exp2f(m[r] - mx[r]);
      m[r] = mx[r];
      l[r] *= alpha[r];
    }
#pragma unroll
    for (int n = 0; n < kPfKeys / 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float p = s[n][i] == kNegInf ? 0.0f : exp2f(s[n][i] - m[i >> 1]);
        s[n][i] = p;
        l[i >> 1] += p;
      }
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) o[n][0] *= alpha[0], o[n][1] *= alpha[0], o[n][2] *= alpha[1], o[n][3] *= alpha[1];
#pragma unroll
    for (int kk = 0; kk < kPfKeys / 16; ++kk) {
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
          mma_bf16(o[2 * n], lo, b[0], b[1]);
          mma_bf16(o[2 * n + 1], hi, b[2], b[3]);
          mma_bf16(o[2 * n + 1], lo, b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (tok_r[r] >= ntok || tok_r[r] >= toks) continue;
    const float inv = 1.0f / l[r];
    __nv_bfloat16* orow = out + (size_t)(row0 + tok_r[r]) * ldo + (kvh * group + hg_r[r]) * a.vdimp + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
      if (n * 8 < a.vdimp) *reinterpret_cast<uint32_t*>(orow + n * 8) = pack2(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
  }
}

// ------------------------------------------------------------------------------------------ bf16 decode
constexpr int kDecThreads = 128, kDecLanes = 8, kDecPass = kDecThreads / kDecLanes, kDecUnroll = 4;

__device__ __forceinline__ void unpack8(const uint4& p, float (&f)[8]) {
  const uint32_t w[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

size_t decode_smem(const AttnShape& a, int hb) {
  const int kg = kDecThreads / (a.vdimp / 8);
  return ((size_t)hb * a.dimp + (size_t)hb * kDecodeKeys + (size_t)kg * hb * a.vdimp) * 4;
}

// grid (splits, kv heads x blocks of HB query heads, single rows).  One chunk of kDecodeKeys cache positions: scores
// (eight lanes per key, 16-byte loads), softmax of the chunk, values (lanes over the value vector, the rest of the CTA
// over keys).  splits == 1: the result; else {max, sum} and the unnormalized output per split.
template <int HB>
__global__ void __launch_bounds__(kDecThreads) lm_attn_decode_kernel(AttnShape a, const __nv_bfloat16* __restrict__ q, int ldq,
                                                                     const int* __restrict__ single_rows,
                                                                     const int2* __restrict__ row_sp,
                                                                     const __nv_bfloat16* __restrict__ kc,
                                                                     const __nv_bfloat16* __restrict__ vc,
                                                                     const float* __restrict__ bias, __nv_bfloat16* __restrict__ out,
                                                                     int ldo, float* __restrict__ part_o, float2* __restrict__ part_ml) {
  extern __shared__ __align__(16) float dec_smem[];
  __shared__ float s_m[HB], s_l[HB];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int D = a.dimp, DV = a.vdimp, group = a.heads / a.kv_heads, hblocks = (group + HB - 1) / HB;
  float* sq = dec_smem;                 // [HB][D]
  float* ss = sq + HB * D;              // [HB][kDecodeKeys]
  float* red = ss + HB * kDecodeKeys;   // [key groups][HB][DV]
  const int split = blockIdx.x, splits = gridDim.x, kvh = blockIdx.y / hblocks, hb0 = (blockIdx.y - kvh * hblocks) * HB;
  const int idx = blockIdx.z, row = single_rows ? single_rows[idx] : idx;
  const int2 sp = row_sp[row];
  const int j0 = split * kDecodeKeys, nk = min(kDecodeKeys, sp.y + 1 - j0);
  if (nk <= 0) return;
  const int nh = min(HB, group - hb0), h0 = kvh * group + hb0, tid = threadIdx.x;
  const size_t base = ((size_t)sp.x * a.kv_heads + kvh) * a.max_ctx + j0;
  for (int i = tid; i < HB * D; i += kDecThreads)
    sq[i] = i / D < nh ? __bfloat162float(q[(size_t)row * ldq + h0 * D + i]) : 0.0f;
  __syncthreads();
  {
    const int kl = tid / kDecLanes, l = tid % kDecLanes, vecs = D / 8;
    for (int k0 = 0; k0 < nk; k0 += kDecPass * kDecUnroll) {
      float acc[kDecUnroll][HB];
#pragma unroll
      for (int u = 0; u < kDecUnroll; ++u)
#pragma unroll
        for (int h = 0; h < HB; ++h) acc[u][h] = 0.0f;
      for (int v = l; v < vecs; v += kDecLanes) {
        uint4 raw[kDecUnroll];
#pragma unroll
        for (int u = 0; u < kDecUnroll; ++u) {
          const int k = k0 + u * kDecPass + kl;
          raw[u] = k < nk ? *reinterpret_cast<const uint4*>(kc + (base + k) * D + v * 8) : make_uint4(0, 0, 0, 0);
        }
        float kf[kDecUnroll][8];
#pragma unroll
        for (int u = 0; u < kDecUnroll; ++u) unpack8(raw[u], kf[u]);
#pragma unroll
        for (int h = 0; h < HB; ++h) {
          const float4 qa = *reinterpret_cast<const float4*>(sq + h * D + v * 8), qb = *reinterpret_cast<const float4*>(sq + h * D + v * 8 + 4);
          const float qv[8] = {qa.x, qa.y, qa.z, qa.w, qb.x, qb.y, qb.z, qb.w};
#pragma unroll
          for (int u = 0; u < kDecUnroll; ++u)
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[u][h] = fmaf(qv[e], kf[u][e], acc[u][h]);
        }
      }
#pragma unroll
      for (int u = 0; u < kDecUnroll; ++u)
#pragma unroll
        for (int h = 0; h < HB; ++h) {
#pragma unroll
          for (int o = kDecLanes / 2; o > 0; o >>= 1) acc[u][h] += __shfl_xor_sync(0xffffffffu, acc[u][h], o);
          const int k = k0 + u * kDecPass + kl;
          if (l == h % kDecLanes && h < nh && k < nk) {
            float s = acc[u][h] * a.scale;
            if (a.has_bias) s += __ldg(bias + (size_t)(h0 + h) * (a.bias_max + 1) + min(sp.y - (j0 + k), a.bias_max));
            ss[h * kDecodeKeys + k] = s;
          }
        }
    }
  }
  __syncthreads();
  for (int h = tid >> 5; h < nh; h += kDecThreads / 32) {
    const int lane = tid & 31;
    float mx = a.sink && splits == 1 ? 0.0f : kNegInf;
    for (int k = lane; k < nk; k += 32) mx = fmaxf(mx, ss[h * kDecodeKeys + k]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.0f;
    for (int k = lane; k < nk; k += 32) {
      const float p = expf(ss[h * kDecodeKeys + k] - mx);
      ss[h * kDecodeKeys + k] = p;
      sum += p;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (lane == 0) {
      s_m[h] = mx;
      s_l[h] = sum + (a.sink && splits == 1 ? expf(-mx) : 0.0f);
    }
  }
  __syncthreads();
  const int vl_n = DV / 8, kg_n = kDecThreads / vl_n, vl = tid % vl_n, kg = tid / vl_n;
  if (kg < kg_n) {
    float acc[HB][8];
#pragma unroll
    for (int h = 0; h < HB; ++h)
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[h][e] = 0.0f;
    for (int k0 = kg; k0 < nk; k0 += kg_n * kDecUnroll) {
      uint4 raw[kDecUnroll];
#pragma unroll
      for (int u = 0; u < kDecUnroll; ++u) {
        const int k = k0 + u * kg_n;
        raw[u] = k < nk ? *reinterpret_cast<const uint4*>(vc + (base + k) * DV + vl * 8) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int u = 0; u < kDecUnroll; ++u) {
        const int k = k0 + u * kg_n;
        if (k >= nk) break;
        float vf[8];
        unpack8(raw[u], vf);
#pragma unroll
        for (int h = 0; h < HB; ++h) {
          const float p = h < nh ? ss[h * kDecodeKeys + k] : 0.0f;
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[h][e] = fmaf(p, vf[e], acc[h][e]);
        }
      }
    }
#pragma unroll
    for (int h = 0; h < HB; ++h) {
      float* r = red + ((size_t)kg * HB + h) * DV + vl * 8;
      *reinterpret_cast<float4*>(r) = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
      *reinterpret_cast<float4*>(r + 4) = make_float4(acc[h][4], acc[h][5], acc[h][6], acc[h][7]);
    }
  }
  __syncthreads();
  for (int i = tid; i < nh * DV; i += kDecThreads) {
    float o = 0.0f;
    for (int g = 0; g < kg_n; ++g) o += red[(size_t)g * HB * DV + i];
    const int h = i / DV;
    if (splits == 1) out[(size_t)row * ldo + h0 * DV + i] = __float2bfloat16_rn(o / s_l[h]);
    else part_o[(((size_t)idx * a.heads + h0 + h) * splits + split) * DV + (i - h * DV)] = o;
  }
  if (splits > 1 && tid < nh) part_ml[((size_t)idx * a.heads + h0 + tid) * splits + split] = make_float2(s_m[tid], s_l[tid]);
}

// grid (heads, single rows): merges the splits of a row and head, the sink joining here.
__global__ void __launch_bounds__(128) lm_attn_combine_kernel(AttnShape a, int splits, const int* __restrict__ single_rows,
                                                              const int2* __restrict__ row_sp, const float* __restrict__ part_o,
                                                              const float2* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                                                              int ldo) {
  extern __shared__ float sw[];  // [splits]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int h = blockIdx.x, idx = blockIdx.y, row = single_rows ? single_rows[idx] : idx, tid = threadIdx.x;
  const int nact = min(splits, row_sp[row].y / kDecodeKeys + 1);
  const float2* ml = part_ml + ((size_t)idx * a.heads + h) * splits;
  float mx = a.sink ? 0.0f : kNegInf;
  for (int s = 0; s < nact; ++s) mx = fmaxf(mx, ml[s].x);
  for (int s = tid; s < nact; s += blockDim.x) sw[s] = expf(ml[s].x - mx);
  __syncthreads();
  float tot = a.sink ? expf(-mx) : 0.0f;
  for (int s = 0; s < nact; ++s) tot = fmaf(ml[s].y, sw[s], tot);
  const float inv = 1.0f / tot;
  for (int d = tid; d < a.vdimp; d += blockDim.x) {
    const float* po = part_o + ((size_t)idx * a.heads + h) * splits * a.vdimp + d;
    float o = 0.0f;
    for (int s = 0; s < nact; ++s) o = fmaf(sw[s], po[(size_t)s * a.vdimp], o);
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
  set(lm_attn_decode_kernel<1>);
  set(lm_attn_decode_kernel<2>);
  set(lm_attn_decode_kernel<4>);
  set(lm_attn_decode_kernel<8>);
  return r;
}

// Rows in `tiles` go through the prompt kernel, `single_rows` (n_single; nullptr = rows 0 .. n_single - 1) through the
// decode kernels; in 32-bit mode all `rows` rows take one kernel.
cudaError_t launch_attention(cudaStream_t s, bool f32, const AttnShape& a, const void* q, int ldq, const int2* row_sp, int rows,
                             const void* kc, const void* vc, const float* bias, void* out, int ldo, const int4* tiles, int n_tiles,
                             const int* single_rows, int n_single, int splits, float* part_o, float2* part_ml) {
  if (f32)
    return launch_pdl(lm_attn_f32_kernel, dim3(rows, a.heads), dim3(kF32Threads), 0, s, a, static_cast<const float*>(q), ldq, row_sp,
                      static_cast<const float*>(kc), static_cast<const float*>(vc), bias, static_cast<float*>(out), ldo);
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
    const int hb = group <= 1 ? 1 : group <= 2 ? 2 : group <= 4 ? 4 : 8;
    const dim3 grid(splits, a.kv_heads * ((group + hb - 1) / hb), n_single);
    const size_t smem = decode_smem(a, hb);
    auto go = [&](auto f) { return launch_pdl(f, grid, dim3(kDecThreads), smem, s, a, qb, ldq, single_rows, row_sp, kb, vb, bias, ob, ldo, part_o, part_ml); };
    r = hb == 1 ? go(lm_attn_decode_kernel<1>) : hb == 2 ? go(lm_attn_decode_kernel<2>) : hb == 4 ? go(lm_attn_decode_kernel<4>) : go(lm_attn_decode_kernel<8>);
    if (r == cudaSuccess && splits > 1)
      r = launch_pdl(lm_attn_combine_kernel, dim3(a.heads, n_single), dim3(128), (size_t)splits * 4, s, a, splits, single_rows, row_sp,
                     part_o, part_ml, ob, ldo);
  }
  return r;
}

}  // namespace lm
}  // namespace mllmb200
