// Latent attention: per position one cached row c of `rank` numbers, shared by all heads; head h has k = U_h c and
// v = V_h c, and no positions.  Two equal ways to attend:
//   * through the latent itself (decoding, short portions of prompts): (U_h^T q_h) . c is the score and V_h applies to the
//     weighted sum of the rows, so that a position costs one read of c whatever the number of heads;
//   * through keys and values made for the step by a linear (long portions), by the kernels of lm_attn.cu.
// Here are the cache's rows (norm and store) and the first way:
//   * lm_head_linear_kernel: a small matrix per head, 16 to 64 rows at a time on mma.sync, the weights straight from memory
//     in fragment order (k is permuted alike on both sides).  It makes the queries U_h^T q_h - some CTAs put the step's
//     latents into the cache meanwhile - and, merging the context splits while it loads, the outputs.
//   * lm_latent_attn_kernel: 16 heads of a row as the rows of one mma tile, blocks of latents through a cp.async ring and
//     used twice, as keys and as values; the warps share the keys for the scores and the columns for the sums.
//   * fp32 forms of both head linears; fp32 attention is that of lm_attn.cu with one head of keys.
// Scores, weights and sums are fp32; the weights enter the second product as a sum of two bf16 numbers.
#include <algorithm>
#include <cmath>
#include <type_traits>

#include "../device_common.cuh"
#include "lm_route.cuh"

namespace mllmb200 {
namespace lm {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kFloor = -1e30f;  // below every score
constexpr int kThreads = 256, kWarps = 8;

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
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
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
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack2(v.x, v.y), pack2(v.z, v.w));
}

// ------------------------------------------------------------------------------------------ the cache
// One warp: row `row` of the step, over its root mean square and times the gains, to its place.  The padding of a row is
// zero in `fresh` and stays zero.
template <class T>
__device__ __forceinline__ void cache_row(const LatentArgs& a, int row, int lane) {
  const float* src = a.fresh + (size_t)row * a.rankp;
  float4 v[kMaxRank / 128];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < kMaxRank / 128; ++i) {
    const int c = lane * 4 + i * 128;
    v[i] = c < a.rankp ? *reinterpret_cast<const float4*>(src + c) : make_float4(0, 0, 0, 0);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.0f / sqrtf(ss / (float)a.rank + a.eps);
  const int2 sp = a.row_sp[row];
  T* dst = static_cast<T*>(a.cache) + ((size_t)sp.x * a.max_ctx + sp.y) * a.rankp;
#pragma unroll
  for (int i = 0; i < kMaxRank / 128; ++i) {
    const int c = lane * 4 + i * 128;
    if (c >= a.rankp) break;
    const float4 g = *reinterpret_cast<const float4*>(a.gain + c);
    store4(dst + c, make_float4(v[i].x * r * g.x, v[i].y * r * g.y, v[i].z * r * g.z, v[i].w * r * g.w));
  }
}

template <class T>
__global__ void __launch_bounds__(kThreads) lm_latent_cache_kernel(LatentArgs a, int rows) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int row = blockIdx.x * kWarps + (threadIdx.x >> 5);
  if (row < rows) cache_row<T>(a, row, threadIdx.x & 31);
}

// ------------------------------------------------------------------------------------------ a matrix per head
// y[i][h] = W_h x[i][h], W_h [N][K] with K a multiple of 16.  Column slices of 64 / KS; KS warps share a slice's K.
// MERGE: x[i][h] is the weighted sum over the context splits of row i.
template <int MT, int KS, bool MERGE>
__global__ void __launch_bounds__(kThreads) lm_head_linear_kernel(LatentArgs a, int N, int K, int slices, int chunk, int splits) {
  extern __shared__ __align__(16) uint8_t hl_smem[];
  __shared__ float red[KS > 1 ? kWarps : 1][16][8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, ks = warp % KS;
  const int row0 = blockIdx.y * 16 * MT, n_here = min(16 * MT, a.n_rows - row0);
  pdl_launch_dependents();
  if (!MERGE && (int)blockIdx.x >= a.heads * slices) {  // the step's latents
    pdl_wait_prior();
    const int r = ((int)blockIdx.x - a.heads * slices) * kWarps + warp;
    if (r < n_here) cache_row<__nv_bfloat16>(a, row0 + r, lane);
    return;
  }
  const int h = blockIdx.x / slices, n0 = (blockIdx.x - h * slices) * (64 / KS) + (warp / KS) * 8;
  const int steps = (K + 31) / 32, per = (steps + KS - 1) / KS, s0 = ks * per, s1 = min(s0 + per, steps);
  const __nv_bfloat16* wp = (MERGE ? a.uv : a.uk_t) + ((size_t)h * N + min(n0 + (lane >> 2), N - 1)) * K + (lane & 3) * 8;
  const bool n_ok = n0 < N;  // N is a multiple of 16: whole tiles of 8 columns
  constexpr int kAhead = 4;
  uint4 wv[kAhead];
  auto fetch = [&](int s) {
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      const bool in = n_ok && s + u < s1 && (s + u) * 32 + (lane & 3) * 8 < K;
      wv[u] = in ? __ldg(reinterpret_cast<const uint4*>(wp + (s + u) * 32)) : make_uint4(0, 0, 0, 0);
    }
  };
  fetch(s0);
  pdl_wait_prior();
  const int ldx = (K + 63) / 64 * 64 + 32;
  __nv_bfloat16* sx = reinterpret_cast<__nv_bfloat16*>(hl_smem);
  float* sw = reinterpret_cast<float*>(sx + 16 * MT * ldx);  // [16 MT][splits]
  if (MERGE) {
    for (int r = warp; r < n_here; r += kWarps) {
      const int row = a.rows ? a.rows[row0 + r] : row0 + r;
      const int nact = min(splits, a.row_sp[row].y / chunk + 1);
      const float2* ml = a.part_ml + ((size_t)(row0 + r) * a.heads + h) * splits;
      float mx = kFloor, tot = 0.0f;
      for (int s = lane; s < nact; s += 32) mx = fmaxf(mx, ml[s].x);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      for (int s = lane; s < splits; s += 32) {
        const float2 v = s < nact ? ml[s] : make_float2(kFloor, 0.0f);
        const float f = s < nact ? exp2f(v.x - mx) : 0.0f;
        sw[r * splits + s] = f;
        tot = fmaf(v.y, f, tot);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) tot += __shfl_xor_sync(0xffffffffu, tot, o);
      __syncwarp();
      for (int s = lane; s < splits; s += 32) sw[r * splits + s] /= tot;
    }
    __syncthreads();
  }
  const int k4 = K / 4, kp4 = ldx / 4;
  if (MERGE) {
    // ITEMS groups of four columns at a time, AT splits of each requested together; splits that do not exist weigh 0
    auto merge = [&](auto items, auto at) {
      constexpr int ITEMS = decltype(items)::value, AT = decltype(at)::value;
      for (int i0 = tid; i0 < 16 * MT * kp4; i0 += kThreads * ITEMS) {
        float4 v[ITEMS];
#pragma unroll
        for (int j = 0; j < ITEMS; ++j) v[j] = make_float4(0, 0, 0, 0);
        const int last = n_here * kp4;  // later places are padding rows
        for (int b = 0; b < splits && i0 < last; b += AT) {
          float4 p[ITEMS][AT];
          float g[ITEMS][AT];
#pragma unroll
          for (int j = 0; j < ITEMS; ++j) {
            const int i = i0 + j * kThreads, r = i / kp4, c = i - r * kp4;
            const bool ok = r < n_here && c < k4;
            const float4* po = reinterpret_cast<const float4*>(a.part_o + ((size_t)(row0 + (ok ? r : 0)) * a.heads + h) * splits * K) + (ok ? c : 0);
#pragma unroll
            for (int u = 0; u < AT; ++u) {
              g[j][u] = ok && b + u < splits ? sw[r * splits + b + u] : 0.0f;
              p[j][u] = g[j][u] != 0.0f ? po[(size_t)(b + u) * k4] : make_float4(0, 0, 0, 0);
            }
          }
#pragma unroll
          for (int j = 0; j < ITEMS; ++j)
#pragma unroll
            for (int u = 0; u < AT; ++u) {
              v[j].x = fmaf(g[j][u], p[j][u].x, v[j].x), v[j].y = fmaf(g[j][u], p[j][u].y, v[j].y);
              v[j].z = fmaf(g[j][u], p[j][u].z, v[j].z), v[j].w = fmaf(g[j][u], p[j][u].w, v[j].w);
            }
        }
#pragma unroll
        for (int j = 0; j < ITEMS; ++j) {
          const int i = i0 + j * kThreads;
          if (i < 16 * MT * kp4) store4(sx + i * 4, v[j]);
        }
      }
    };
    if constexpr (KS > 1) merge(std::integral_constant<int, 1>{}, std::integral_constant<int, 8>{});
    else merge(std::integral_constant<int, 4>{}, std::integral_constant<int, 2>{});
  } else {
    for (int i = tid; i < 16 * MT * kp4; i += kThreads) {
      const int r = i / kp4, c = i - r * kp4;
      uint2 v = make_uint2(0, 0);
      if (r < n_here && c < k4) {
        const int row = a.rows ? a.rows[row0 + r] : row0 + r;
        v = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(a.q) + (size_t)row * a.ldq + (size_t)h * K + c * 4);
      }
      *reinterpret_cast<uint2*>(sx + i * 4) = v;
    }
  }
  __syncthreads();
  float acc[MT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m) acc[m][0] = acc[m][1] = acc[m][2] = acc[m][3] = 0.0f;
  const __nv_bfloat16* xr = sx + (lane >> 2) * ldx + (lane & 3) * 8;
  for (int s = s0; s < s1; s += kAhead) {
    uint4 cw[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) cw[u] = wv[u];
    if (s + kAhead < s1) fetch(s + kAhead);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      if (s + u >= s1) break;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const uint4 lo = *reinterpret_cast<const uint4*>(xr + (m * 16) * ldx + (s + u) * 32);
        const uint4 hi = *reinterpret_cast<const uint4*>(xr + (m * 16 + 8) * ldx + (s + u) * 32);
        mma_bf16(acc[m], lo.x, hi.x, lo.y, hi.y, cw[u].x, cw[u].y);
        mma_bf16(acc[m], lo.z, hi.z, lo.w, hi.w, cw[u].z, cw[u].w);
      }
    }
  }
  if (KS > 1) {  // MT = 1
#pragma unroll
    for (int i = 0; i < 4; ++i) red[warp][(lane >> 2) + (i >> 1) * 8][(lane & 3) * 2 + (i & 1)] = acc[0][i];
    __syncthreads();
    if (ks) return;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float v = 0.0f;
#pragma unroll
      for (int j = 0; j < KS; ++j) v += red[warp + j][(lane >> 2) + (i >> 1) * 8][(lane & 3) * 2 + (i & 1)];
      acc[0][i] = v;
    }
  }
  if (!n_ok) return;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = m * 16 + (lane >> 2) + i * 8;
      if (r >= n_here) continue;
      const size_t at = MERGE ? (size_t)(a.rows ? a.rows[row0 + r] : row0 + r) * a.ldo : (size_t)(row0 + r) * a.heads * N;
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(MERGE ? a.out : a.qa) + at + (size_t)h * N + n0 + (lane & 3) * 2;
      *reinterpret_cast<uint32_t*>(y) = pack2(acc[m][2 * i], acc[m][2 * i + 1]);
    }
}

// fp32: grid (heads, rows); a warp per output column
__global__ void __launch_bounds__(kThreads) lm_head_linear_f32_kernel(const float* __restrict__ x, int ldx, const __nv_bfloat16* __restrict__ w,
                                                                      int N, int K, float* __restrict__ y, int ldy) {
  extern __shared__ __align__(16) float hf_x[];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int h = blockIdx.x, row = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int k = threadIdx.x; k < K; k += kThreads) hf_x[k] = x[(size_t)row * ldx + (size_t)h * K + k];
  __syncthreads();
  for (int n = warp; n < N; n += kWarps) {
    const __nv_bfloat16* wr = w + ((size_t)h * N + n) * K;
    float s = 0.0f;
    for (int k = lane * 8; k < K; k += 256)
      s += dot8(*reinterpret_cast<const uint4*>(wr + k), *reinterpret_cast<const float4*>(hf_x + k), *reinterpret_cast<const float4*>(hf_x + k + 4));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) y[(size_t)row * ldy + (size_t)h * N + n] = s;
  }
}

// ------------------------------------------------------------------------------------------ attention through the latent
constexpr int kHeadRows = 16, kAttnSmemMax = 226 * 1024;

// Shape of a CTA.  NT: tiles of 16 columns per warp; KB: keys per block; ST: blocks in the ring; NW: warps.  Scores: a warp
// takes 8 keys and one of KQ shares of the columns, whose queries it keeps in registers if they fit (HOLD).
template <int NT_, int KB_, int ST_, int NW_, int CTAS_>
struct AttnCta {
  static constexpr int NT = NT_, KB = KB_, ST = ST_, NW = NW_, CTAS = CTAS_;
  static constexpr int kColumns = NT * NW * 16;
  static constexpr int KQ = NW / (KB / 8);
  static constexpr int kSteps = kColumns / 64 / KQ;  // of 64 columns, per warp
  static constexpr bool HOLD = kSteps <= (NW * CTAS <= 8 ? 8 : 4);
  static constexpr int LPR = 2 * NW;                 // lanes that share a row of scores
  static constexpr int kPer = KB / LPR;
  static constexpr int kLdS = KB + 4, kLdP = KB + 8;
  static constexpr size_t smem(int rankp) {
    return (size_t)(kHeadRows + ST * KB) * (rankp + 8) * 2 + (size_t)KQ * kHeadRows * kLdS * 4 + (size_t)2 * kHeadRows * kLdP * 2;
  }
};
using Attn256 = AttnCta<2, 64, 2, 8, 2>;  // two CTAs of eight warps per SM: one computes while the other waits
using Attn512 = AttnCta<4, 64, 2, 8, 1>;
using Attn1024 = AttnCta<4, 32, 2, 16, 1>;

// grid (splits, blocks of 16 heads, rows).  Leaves {max, sum} (base 2) and the unnormalized sum per split.
template <class S>
__global__ void __launch_bounds__(S::NW * 32, S::CTAS) lm_latent_attn_kernel(LatentArgs a, int chunk) {
  extern __shared__ __align__(16) uint8_t la_smem[];
  __shared__ float s_alpha[kHeadRows];
  constexpr int NT = S::NT, KB = S::KB, ST = S::ST, NW = S::NW, KQ = S::KQ, kLdS = S::kLdS, kLdP = S::kLdP;
  const int R = a.rankp, ldc = R + 8, splits = gridDim.x, split = blockIdx.x, idx = blockIdx.z, h0 = blockIdx.y * kHeadRows;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(la_smem);
  __nv_bfloat16* sC = sQ + kHeadRows * ldc;
  __nv_bfloat16* sP = sC + ST * KB * ldc;  // high parts, then low parts
  float* sS = reinterpret_cast<float*>(sP + 2 * kHeadRows * kLdP);  // [KQ][rows]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int row = a.rows ? a.rows[idx] : idx;
  const int2 sp = a.row_sp[row];
  const int j0 = split * chunk, nk = min(chunk, sp.y + 1 - j0);
  if (nk <= 0) return;
  const int nh = min(kHeadRows, a.heads - h0), blocks = (nk + KB - 1) / KB;
  const __nv_bfloat16* cb = static_cast<const __nv_bfloat16*>(a.cache) + ((size_t)sp.x * a.max_ctx + j0) * R;
  const int cr = tid >> 3, cc = (tid & 7) * 8;  // copies: eight threads per row, 128 bytes at a time
  auto fetch = [&](int b) {
    if (b < blocks) {
      __nv_bfloat16* to = sC + (b % ST) * KB * ldc;
      for (int r = cr; r < KB; r += NW * 4) {
        const int j = b * KB + r;
        const __nv_bfloat16* src = cb + (size_t)(j < nk ? j : 0) * R + cc;
        const uint32_t dst = smem_u32(to + r * ldc + cc);
#pragma unroll
        for (int c = 0; c < S::kColumns; c += 64)
          if (c < R) cp_async16(dst + c * 2, src + c, j < nk);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");  // past the last block: an empty group
  };
  if (cr < kHeadRows) {
    const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.qa) + ((size_t)idx * a.heads + h0 + (cr < nh ? cr : 0)) * R;
    for (int c = cc; c < R; c += 64) cp_async16(smem_u32(sQ + cr * ldc + c), src + c, cr < nh);
  }
#pragma unroll
  for (int b = 0; b < ST - 1; ++b) fetch(b);
  const int mat = lane >> 3, ml = lane & 7, part = warp / (KB / 8), key = (warp % (KB / 8)) * 8;
  const uint32_t q_addr = smem_u32(sQ + ((mat & 1) * 8 + ml) * ldc + (mat >> 1) * 8);
  const uint32_t k_addr = smem_u32(sC + (key + ml) * ldc + mat * 8);
  const uint32_t v_addr = smem_u32(sC + ((mat & 1) * 8 + ml) * ldc + warp * NT * 16 + (mat >> 1) * 8);
  const uint32_t p_addr = smem_u32(sP + ((mat & 1) * 8 + ml) * kLdP + (mat >> 1) * 8);
  const float sc2 = a.scale * kLog2e;
  const int srow = tid / S::LPR, scol = (tid % S::LPR) * S::kPer;  // this lane's scores
  uint32_t qf[S::HOLD ? 4 * S::kSteps : 4][4];
  auto load_q = [&](uint32_t(&q)[4], int c) { ldsm4(q, q_addr + c * 2); };
  if (S::HOLD) {
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");  // the first group
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 4 * S::kSteps; ++k) {
      const int c = ((k / 4) * KQ + part) * 64 + (k % 4) * 16;
      qf[k][0] = qf[k][1] = qf[k][2] = qf[k][3] = 0;
      if (c < R) load_q(qf[k], c);
    }
  }
  float m = kFloor, l = 0.0f, o[2 * NT][4];
#pragma unroll
  for (int n = 0; n < 2 * NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.0f;

  for (int b = 0; b < blocks; ++b) {
    const int stage = (b % ST) * KB * ldc * 2;  // bytes
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
    __syncthreads();  // the block has landed; everyone is through with the one before
    fetch(b + ST - 1);
    {
      float acc[4][4] = {};
#pragma unroll
      for (int k = 0; k < S::kSteps; ++k) {
        const int c = (k * KQ + part) * 64;
        if (c < R) {
          uint32_t kf[4], kg[4];
          ldsm4(kf, k_addr + stage + c * 2);
          ldsm4(kg, k_addr + stage + c * 2 + 64);
          if (!S::HOLD)
#pragma unroll
            for (int i = 0; i < 4; ++i) load_q(qf[i], c + i * 16);
          const int q = S::HOLD ? 4 * k : 0;
          mma_bf16(acc[0], qf[q][0], qf[q][1], qf[q][2], qf[q][3], kf[0], kf[1]);
          mma_bf16(acc[1], qf[q + 1][0], qf[q + 1][1], qf[q + 1][2], qf[q + 1][3], kf[2], kf[3]);
          mma_bf16(acc[2], qf[q + 2][0], qf[q + 2][1], qf[q + 2][2], qf[q + 2][3], kg[0], kg[1]);
          mma_bf16(acc[3], qf[q + 3][0], qf[q + 3][1], qf[q + 3][2], qf[q + 3][3], kg[2], kg[3]);
        }
      }
      float* st = sS + (part * kHeadRows + (lane >> 2)) * kLdS + key + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[0][i] += acc[1][i] + (acc[2][i] + acc[3][i]);
      *reinterpret_cast<float2*>(st) = make_float2(acc[0][0], acc[0][1]);
      *reinterpret_cast<float2*>(st + 8 * kLdS) = make_float2(acc[0][2], acc[0][3]);
    }
    __syncthreads();
    {
      float p[S::kPer], mx = m, sum = 0.0f;
#pragma unroll
      for (int i = 0; i < S::kPer; ++i) {
        p[i] = 0.0f;
#pragma unroll
        for (int q = 0; q < KQ; ++q) p[i] += sS[(q * kHeadRows + srow) * kLdS + scol + i];
        p[i] = b * KB + scol + i < nk ? p[i] * sc2 : kFloor;
        mx = fmaxf(mx, p[i]);
      }
#pragma unroll
      for (int d = S::LPR / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
#pragma unroll
      for (int i = 0; i < S::kPer; ++i) {
        p[i] = fast_exp2(p[i] - mx);  // the block has a key: places without one are far below the maximum
        sum += p[i];
      }
      const float alpha = fast_exp2(m - mx);
      m = mx;
      if (tid % S::LPR == 0) s_alpha[srow] = alpha;
      __nv_bfloat16* ph = sP + srow * kLdP + scol;
#pragma unroll
      for (int i = 0; i < S::kPer; ++i) {
        const __nv_bfloat16 hi = __float2bfloat16_rn(p[i]);
        ph[i] = hi;
        ph[kHeadRows * kLdP + i] = __float2bfloat16_rn(p[i] - __bfloat162float(hi));
      }
      l = fmaf(l, alpha, sum);  // of this lane's keys
    }
    __syncthreads();
    const float f0 = s_alpha[lane >> 2], f1 = s_alpha[(lane >> 2) + 8];
    if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {  // a new maximum: seldom after the first blocks
#pragma unroll
      for (int n = 0; n < 2 * NT; ++n) o[n][0] *= f0, o[n][1] *= f0, o[n][2] *= f1, o[n][3] *= f1;
    }
#pragma unroll
    for (int kk = 0; kk < KB / 16; ++kk) {
      uint32_t hi[4], lo[4];
      ldsm4(hi, p_addr + kk * 32);
      ldsm4(lo, p_addr + kHeadRows * kLdP * 2 + kk * 32);
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        if ((warp * NT + t) * 16 < R) {
          uint32_t v[4];
          ldsm4_t(v, v_addr + stage + (kk * 16 * ldc + t * 16) * 2);
          mma_bf16(o[2 * t], hi[0], hi[1], hi[2], hi[3], v[0], v[1]);
          mma_bf16(o[2 * t + 1], hi[0], hi[1], hi[2], hi[3], v[2], v[3]);
          mma_bf16(o[2 * t], lo[0], lo[1], lo[2], lo[3], v[0], v[1]);
          mma_bf16(o[2 * t + 1], lo[0], lo[1], lo[2], lo[3], v[2], v[3]);
        }
      }
    }
  }
#pragma unroll
  for (int d = S::LPR / 2; d > 0; d >>= 1) l += __shfl_xor_sync(0xffffffffu, l, d);
  if (tid % S::LPR == 0 && srow < nh) a.part_ml[((size_t)idx * a.heads + h0 + srow) * splits + split] = make_float2(m, l);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = (lane >> 2) + i * 8;
    if (r >= nh) continue;
    float* po = a.part_o + (((size_t)idx * a.heads + h0 + r) * splits + split) * R + warp * NT * 16 + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < 2 * NT; ++n)
      if (warp * NT * 16 + n * 8 < R) *reinterpret_cast<float2*>(po + n * 8) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
  }
}

// ------------------------------------------------------------------------------------------ launches
struct Split {
  int chunk, splits;
};
// Context per CTA: as many CTAs as fit the GPU at once, but no more splits than pay (a split more costs the merge a
// twenty-fifth of what a block more in a row costs).
Split split_context(const LatentArgs& a) {
  const int kb = a.rankp <= 512 ? Attn512::KB : Attn1024::KB, fit = a.rankp <= 256 ? Attn256::CTAS : 1;
  const int blocks = (a.ctx + kb - 1) / kb, hblocks = (a.heads + kHeadRows - 1) / kHeadRows;
  const int want = std::max(1, std::min((int)std::ceil(5.0 * std::sqrt((double)blocks)), kSms * fit / (a.n_rows * hblocks)));
  const int per = (blocks + want - 1) / want;
  return {per * kb, (blocks + per - 1) / per};
}

size_t head_linear_smem(int mt, int K, int splits) { return (size_t)16 * mt * (((K + 63) / 64 * 64 + 32) * 2 + splits * 4); }

template <bool MERGE>
cudaError_t launch_head_linear(cudaStream_t s, const LatentArgs& a, int N, int K, Split sp, bool cache_rows) {
  const int mt = MERGE || a.n_rows <= 16 ? 1 : a.n_rows <= 32 ? 2 : 4;  // merging is the longer part: more CTAs
  const bool fine = MERGE && a.n_rows <= 8 && K >= 128;  // few rows: more CTAs, K shared by four warps
  const int cols = fine ? 16 : 64, slices = (N + cols - 1) / cols;
  const dim3 grid(a.heads * slices + (cache_rows ? 16 * mt / kWarps : 0), (a.n_rows + 16 * mt - 1) / (16 * mt));
  const size_t smem = head_linear_smem(mt, K, MERGE ? sp.splits : 0);
  auto go = [&](auto f) { return launch_pdl(f, grid, dim3(kThreads), smem, s, a, N, K, slices, sp.chunk, sp.splits); };
  if constexpr (MERGE) {
    return fine ? go(lm_head_linear_kernel<1, 4, true>) : go(lm_head_linear_kernel<1, 1, true>);
  } else {
    return mt == 1 ? go(lm_head_linear_kernel<1, 1, false>) : mt == 2 ? go(lm_head_linear_kernel<2, 1, false>) : go(lm_head_linear_kernel<4, 1, false>);
  }
}

}  // namespace

size_t latent_parts(int rows) { return std::max((size_t)rows, (size_t)2 * kSms); }

cudaError_t latent_configure() {
  cudaError_t r = cudaSuccess;
  auto set = [&](auto f, int most = 200 * 1024) {
    if (r == cudaSuccess) r = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
  };
  set(lm_latent_attn_kernel<Attn256>, kAttnSmemMax);
  set(lm_latent_attn_kernel<Attn512>, kAttnSmemMax);
  set(lm_latent_attn_kernel<Attn1024>, kAttnSmemMax);
  set(lm_head_linear_kernel<1, 1, false>);
  set(lm_head_linear_kernel<2, 1, false>);
  set(lm_head_linear_kernel<4, 1, false>);
  set(lm_head_linear_kernel<1, 4, true>);
  set(lm_head_linear_kernel<1, 1, true>);
  return r;
}

cudaError_t launch_latent_cache(cudaStream_t s, bool f32, const LatentArgs& a, int rows) {
  const dim3 grid((rows + kWarps - 1) / kWarps);
  return f32 ? launch_pdl(lm_latent_cache_kernel<float>, grid, dim3(kThreads), 0, s, a, rows)
             : launch_pdl(lm_latent_cache_kernel<__nv_bfloat16>, grid, dim3(kThreads), 0, s, a, rows);
}

cudaError_t launch_latent_absorbed(cudaStream_t s, bool f32, const LatentArgs& a, bool cache_rows) {
  if (f32) {  // every row of the step
    if (cache_rows) {
      const cudaError_t r = launch_latent_cache(s, true, a, a.n_rows);
      if (r != cudaSuccess) return r;
    }
    const int hr = a.heads * a.rankp;
    cudaError_t r = launch_pdl(lm_head_linear_f32_kernel, dim3(a.heads, a.n_rows), dim3(kThreads), (size_t)a.dimp * 4, s,
                               static_cast<const float*>(a.q), a.ldq, a.uk_t, a.rankp, a.dimp, static_cast<float*>(a.qa), hr);
    if (r != cudaSuccess) return r;
    AttnShape t{};
    t.heads = a.heads;
    t.kv_heads = 1;
    t.dimp = t.vdimp = a.rankp;
    t.slot_rows = t.head_rows = a.max_ctx;
    t.scale = a.scale;
    r = launch_attention(s, true, t, a.qa, hr, a.row_sp, a.n_rows, a.cache, a.cache, nullptr, a.lat, hr, nullptr, 0, nullptr, 0, 0, 0, nullptr, nullptr);
    if (r != cudaSuccess) return r;
    return launch_pdl(lm_head_linear_f32_kernel, dim3(a.heads, a.n_rows), dim3(kThreads), (size_t)a.rankp * 4, s, static_cast<const float*>(a.lat),
                      hr, a.uv, a.vdimp, a.rankp, static_cast<float*>(a.out), a.ldo);
  }
  const Split sp = split_context(a);
  cudaError_t r = launch_head_linear<false>(s, a, a.rankp, a.dimp, sp, cache_rows);
  if (r != cudaSuccess) return r;
  const dim3 grid(sp.splits, (a.heads + kHeadRows - 1) / kHeadRows, a.n_rows);
  auto go = [&](auto shape) {
    using S = decltype(shape);
    return launch_pdl(lm_latent_attn_kernel<S>, grid, dim3(S::NW * 32), S::smem(a.rankp), s, a, sp.chunk);
  };
  r = a.rankp <= 256 ? go(Attn256{}) : a.rankp <= 512 ? go(Attn512{}) : go(Attn1024{});
  if (r != cudaSuccess) return r;
  return launch_head_linear<true>(s, a, a.vdimp, a.rankp, sp, false);
}

}  // namespace lm
}  // namespace mllmb200
