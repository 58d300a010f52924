// bf16-weight linear maps of the language-model engine, y = x W^T, in three kernels that share one epilogue:
//   * lm_gemv_kernel: up to four rows.  Warps stream pairs of weight rows, x waits in shared memory.
//   * lm_gemm_tc_kernel (sm_100a): everything else in bf16.  TMA loads both operands (128-byte swizzle), one elected
//     thread issues tcgen05.mma, the accumulators sit in tensor memory - two of them, so that a persistent CTA's
//     epilogue of one tile overlaps the next tile's K loop.
//   * lm_gemm_f32_kernel: fp32 activations and fp32 FMAs (the 32-bit mode of the engine), more than four rows.
// Each also comes in a form for groups of rows with a weight each (experts), or scattered runs of rows of x: the GEMMs
// then take a table of row tiles, whose length may be known on the device only.
// The epilogue scatters queries, keys and values (keys and values go straight into the caches), applies the gated
// clamped activation to interleaved gate/up columns, or leaves fp32 sums - in several planes when K is split, which
// the consumer (a norm) adds in plane order.
#include "../tcgen05_common.cuh"
#include "lm_state.h"

#include <algorithm>

namespace mllmb200 {
namespace lm {

thread_local long long g_launches = 0;

namespace {

// ------------------------------------------------------------------------------------------ epilogue
template <class T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// All forms are g sigmoid(z(g)) times a form of u: 0.5 (1 + tanh(x)) = sigmoid(2 x).
template <int ACT>
__device__ __forceinline__ float gated_as(float limit, float g, float u) {
  float z = g;
  if (ACT == MLLMB200_LM_ACT_GELU) {
    z = 1.5957691216057308f * fmaf(0.044715f * g * g, g, g);
  } else if (ACT == MLLMB200_LM_ACT_CLAMPED) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit) + 1.0f;
    z = 1.702f * g;
  }
  return g / (1.0f + expf(-z)) * u;
}
__device__ __forceinline__ float gated(const Epi& e, float g, float u) {
  return e.act_kind == MLLMB200_LM_ACT_GELU   ? gated_as<MLLMB200_LM_ACT_GELU>(e.limit, g, u)
         : e.act_kind == MLLMB200_LM_ACT_SILU ? gated_as<MLLMB200_LM_ACT_SILU>(e.limit, g, u)
                                              : gated_as<MLLMB200_LM_ACT_CLAMPED>(e.limit, g, u);
}

// address of column n of row m of a q|k|v product
template <class T>
__device__ __forceinline__ T* qkv_ptr(const Epi& e, int m, int n) {
  if (n < e.q_end) return static_cast<T*>(e.q) + (size_t)m * e.ldq + n;
  const int2 sp = e.row_sp ? e.row_sp[m] : make_int2(0, m);
  const bool is_k = n < e.k_end;
  const int d = is_k ? e.dimp : e.vdimp;
  const int c = n - (is_k ? e.q_end : e.k_end), g = c / d;
  T* base = static_cast<T*>(is_k ? e.kc : e.vc);
  return base + (((size_t)sp.x * e.kv_heads + g) * e.max_ctx + sp.y) * d + (c - g * d);
}

// columns n, n + 1 (n even) of row m
template <class T>
__device__ __forceinline__ void store2(const Epi& e, int m, int n, int N, float v0, float v1, int split) {
  if (e.kind == kEpiPlanes) {
    float* y = e.y + (size_t)split * e.plane + (size_t)m * e.ldy + n;
    y[0] = v0 * e.scale;
    if (n + 1 < N) y[1] = v1 * e.scale;
  } else if (e.kind == kEpiQLatent && n >= e.q_end) {
    float* y = e.y + (size_t)m * e.ldy + (n - e.q_end);
    y[0] = v0;
    y[1] = v1;
  } else if (e.kind != kEpiGate) {
    T* p = qkv_ptr<T>(e, m, n);
    p[0] = from_f32<T>(v0);
    p[1] = from_f32<T>(v1);
  } else {
    static_cast<T*>(e.act)[(size_t)m * e.ld_act + (n >> 1)] = from_f32<T>(gated(e, v0, v1));
  }
}

__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// eight gated pairs, the first of them columns (n, n + 1); pairs past N write zeros into the padding of the row
template <int ACT>
__device__ __forceinline__ void gate8(const Epi& e, int m, int n, int N, const float (&v)[16]) {
  float a[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) a[i] = n + 2 * i < N ? gated_as<ACT>(e.limit, v[2 * i], v[2 * i + 1]) : 0.0f;
  *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(e.act) + (size_t)m * e.ld_act + (n >> 1)) =
      make_uint4(pack_bf16(a[0], a[1]), pack_bf16(a[2], a[3]), pack_bf16(a[4], a[5]), pack_bf16(a[6], a[7]));
}

// columns [n, n + 16) of row m (n a multiple of 16), bf16 outputs; FORM: see form_of
enum Form { kFormPlanes, kFormScatter, kFormGate };
template <int FORM>
__device__ __forceinline__ void store16(const Epi& e, int m, int n, int N, const float (&v)[16], int split) {
  if (FORM == kFormPlanes) {
    float* y = e.y + (size_t)split * e.plane + (size_t)m * e.ldy + n;
    if (n + 16 <= N && (e.ldy & 3) == 0) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        reinterpret_cast<float4*>(y)[i] =
            make_float4(v[4 * i] * e.scale, v[4 * i + 1] * e.scale, v[4 * i + 2] * e.scale, v[4 * i + 3] * e.scale);
    } else {
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (n + i < N) y[i] = v[i] * e.scale;
    }
  } else if (FORM == kFormScatter) {
    if (e.kind == kEpiQLatent && n >= e.q_end) {
      float4* y = reinterpret_cast<float4*>(e.y + (size_t)m * e.ldy + (n - e.q_end));
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
    } else {  // head sizes are multiples of 16: the chunk lies in one head
      uint4* p = reinterpret_cast<uint4*>(qkv_ptr<__nv_bfloat16>(e, m, n));
      p[0] = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
      p[1] = make_uint4(pack_bf16(v[8], v[9]), pack_bf16(v[10], v[11]), pack_bf16(v[12], v[13]), pack_bf16(v[14], v[15]));
    }
  } else if (e.act_kind == MLLMB200_LM_ACT_GELU) {
    gate8<MLLMB200_LM_ACT_GELU>(e, m, n, N, v);
  } else if (e.act_kind == MLLMB200_LM_ACT_SILU) {
    gate8<MLLMB200_LM_ACT_SILU>(e, m, n, N, v);
  } else {
    gate8<MLLMB200_LM_ACT_CLAMPED>(e, m, n, N, v);
  }
}
Form form_of(const Epi& e) { return e.kind == kEpiPlanes ? kFormPlanes : e.kind == kEpiGate ? kFormGate : kFormScatter; }

// ------------------------------------------------------------------------------------------ GEMV
constexpr int kGemvThreads = 256, kGemvWarps = kGemvThreads / 32, kGemvUnroll = 4;

__device__ __forceinline__ void unpack8(const uint4& p, float (&f)[8]) {
  const uint32_t w[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = b.x, f[5] = b.y, f[6] = b.z, f[7] = b.w;
}

// A group of 2^ks_log2 warps owns output columns (2 p, 2 p + 1); its warps split K.  With group_of, CTA row y makes result
// row y from row y / div of x and weight group group_of[y].
template <class T, int MT>
__global__ void __launch_bounds__(kGemvThreads) lm_gemv_kernel(const T* __restrict__ x, const __nv_bfloat16* __restrict__ w,
                                                               int N, int K, int ks_log2, const int* __restrict__ group_of, int div,
                                                               Epi e) {
  extern __shared__ __align__(16) uint8_t gemv_smem[];
  __shared__ float red[kGemvWarps][2 * MT];
  T* xs = reinterpret_cast<T*>(gemv_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int ks_n = 1 << ks_log2, ks = warp & (ks_n - 1);
  const int n0 = 2 * (blockIdx.x * (kGemvWarps >> ks_log2) + (warp >> ks_log2));
  const int iters = (K + 255) >> 8, per = (iters + ks_n - 1) >> ks_log2;
  const int i0 = min(ks * per, iters), i1 = min(i0 + per, iters);
  const __nv_bfloat16 *w0 = w + (size_t)n0 * K, *w1 = w0 + K;
  const bool ok0 = n0 < N, ok1 = n0 + 1 < N;
  uint4 a[kGemvUnroll], b[kGemvUnroll];
  auto fetch = [&](int i) {
#pragma unroll
    for (int u = 0; u < kGemvUnroll; ++u) {
      const int k = (i + u) * 256 + lane * 8;
      const bool in = i + u < i1 && k < K;
      a[u] = in && ok0 ? __ldg(reinterpret_cast<const uint4*>(w0 + k)) : make_uint4(0, 0, 0, 0);
      b[u] = in && ok1 ? __ldg(reinterpret_cast<const uint4*>(w1 + k)) : make_uint4(0, 0, 0, 0);
    }
  };
  pdl_launch_dependents();
  if (!group_of) fetch(i0);  // the weights do not depend on the previous kernel
  pdl_wait_prior();
  const int m0 = group_of ? blockIdx.y : 0;
  if (group_of) {
    w0 += (size_t)group_of[m0] * N * K;
    w1 = w0 + K;
    x += (size_t)(m0 / div) * K;
    fetch(i0);
  }
  constexpr int kVec = 16 / sizeof(T);
  for (int i = tid; i < MT * K / kVec; i += kGemvThreads) reinterpret_cast<uint4*>(xs)[i] = reinterpret_cast<const uint4*>(x)[i];
  __syncthreads();
  float acc[2][MT];
#pragma unroll
  for (int m = 0; m < MT; ++m) acc[0][m] = acc[1][m] = 0.0f;
  for (int i = i0; i < i1; i += kGemvUnroll) {
    uint4 ca[kGemvUnroll], cb[kGemvUnroll];
#pragma unroll
    for (int u = 0; u < kGemvUnroll; ++u) ca[u] = a[u], cb[u] = b[u];
    if (i + kGemvUnroll < i1) fetch(i + kGemvUnroll);
#pragma unroll
    for (int u = 0; u < kGemvUnroll; ++u) {
      const int k = (i + u) * 256 + lane * 8;
      if (i + u >= i1 || k >= K) continue;
      float fa[8], fb[8];
      unpack8(ca[u], fa);
      unpack8(cb[u], fb);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float xv[8];
        load8(xs + m * K + k, xv);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          acc[0][m] = fmaf(fa[j], xv[j], acc[0][m]);
          acc[1][m] = fmaf(fb[j], xv[j], acc[1][m]);
        }
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) acc[r][m] += __shfl_xor_sync(0xffffffffu, acc[r][m], o);
      if (lane == 0) red[warp][r * MT + m] = acc[r][m];
    }
  __syncthreads();
  if (ks == 0 && lane < MT && ok0) {
    float v0 = 0.0f, v1 = 0.0f;
    for (int j = 0; j < ks_n; ++j) {
      v0 += red[warp + j][lane];
      v1 += red[warp + j][MT + lane];
    }
    store2<T>(e, m0 + lane, n0, N, v0, v1, 0);
  }
}

// ------------------------------------------------------------------------------------------ fp32 GEMM
constexpr int kF32Tile = 64, kF32K = 32;

__global__ void __launch_bounds__(256) lm_gemm_f32_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ w, int M,
                                                          int N, int K, const int4* __restrict__ tiles, const int* __restrict__ n_tiles,
                                                          Epi e) {
  __shared__ __align__(16) float xs[kF32K][kF32Tile + 4], ws[kF32K][kF32Tile + 4];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  int m0 = blockIdx.y * kF32Tile, out0 = 0;
  const int n0 = blockIdx.x * kF32Tile;
  if (tiles) {
    if (n_tiles && (int)blockIdx.y >= *n_tiles) return;
    const int4 t = tiles[blockIdx.y];
    w += (size_t)t.x * N * K;
    x += (size_t)t.y * K;
    M = t.z, out0 = t.w, m0 = 0;
  }
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kF32K) {
    for (int i = tid; i < kF32Tile * kF32K / 4; i += 256) {
      const int r = i / (kF32K / 4), c = (i % (kF32K / 4)) * 4;
      float4 v = make_float4(0, 0, 0, 0);
      if (m0 + r < M) v = *reinterpret_cast<const float4*>(x + (size_t)(m0 + r) * K + k0 + c);
      xs[c][r] = v.x, xs[c + 1][r] = v.y, xs[c + 2][r] = v.z, xs[c + 3][r] = v.w;
    }
    {
      const int r = tid >> 2, c = (tid & 3) * 8;
      float f[8] = {};
      if (n0 + r < N) load8(w + (size_t)(n0 + r) * K + k0 + c, f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ws[c + j][r] = f[j];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]), b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      const int n = n0 + tx * 4 + j;
      if (n < N) store2<float>(e, out0 + m, n, N, acc[i][j], acc[i][j + 1], 0);
    }
  }
}

// ------------------------------------------------------------------------------------------ tcgen05 GEMM
constexpr int kTcThreads = 192;  // copy warp, MMA warp, four epilogue warps
constexpr int kTileM = 128, kTileK = 64;
constexpr int kABytes = kTileM * kTileK * 2;

template <int BN>
struct TcShape {
  static constexpr int kStages = BN == 256 ? 4 : (BN == 32 ? 5 : 6);
  static constexpr int kStageBytes = kABytes + BN * kTileK * 2;
  static constexpr int kSmem = kStages * kStageBytes + 1024;
  static constexpr int kTmemCols = 2 * BN;
};

__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(
                   smem_u32(dst)),
               "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
               : "memory");
}
// K-major operand in the 128-byte swizzle: 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t swizzled_desc(uint32_t addr) {
  return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}

// Work items are (K split, weight tile, row tile), row tiles fastest; CTA c takes items c, c + gridDim.x, ...
// GROUPED: the row tiles are those of `tiles`; whole tiles are copied through amap (boxes of 128 rows), the others through
// amap16 (16 rows).  Weight tiles and boxes may reach into the next group: those sums are not stored.
template <int BN, bool GROUPED, int FORM>
__global__ void __launch_bounds__(kTcThreads, 1) lm_gemm_tc_kernel(const __grid_constant__ CUtensorMap amap,
                                                                   const __grid_constant__ CUtensorMap amap16,
                                                                   const __grid_constant__ CUtensorMap wmap, int a_box, int M, int N,
                                                                   int K, int splits, const int4* __restrict__ tiles,
                                                                   const int* __restrict__ n_tiles, int max_tiles, Epi e) {
  using S = TcShape<BN>;
  extern __shared__ uint8_t tc_smem_raw[];
  __shared__ uint64_t full[S::kStages], empty[S::kStages], acc_full[2], acc_empty[2];
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int gave_up;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tc_smem_raw) + 1023) & ~(uintptr_t)1023);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int mt = (M + kTileM - 1) / kTileM;
  const int nt = (N + BN - 1) / BN, kt = K / kTileK;
  int a_rows = M >= kTileM ? kTileM : (M + 15) / 16 * 16;  // rows of x that are loaded at all
  auto grouped_start = [&]() {
    pdl_wait_prior();
    mt = n_tiles ? min(*n_tiles, max_tiles) : max_tiles;
  };
  constexpr int kWBox = BN < 128 ? 32 : 128;
  if (tid == 0) {
    for (int i = 0; i < S::kStages; ++i) mbar_init(&full[i], 1), mbar_init(&empty[i], 1);
    for (int i = 0; i < 2; ++i) mbar_init(&acc_full[i], 1), mbar_init(&acc_empty[i], 4);
    gave_up = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(&tmem_slot, S::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  pdl_launch_dependents();
  auto k_range = [&](int split, int& k0, int& k1) {
    k0 = (int)((long long)kt * split / splits);
    k1 = (int)((long long)kt * (split + 1) / splits);
  };
  if (warp == 0) {
    if (elect_one_sync()) {
      int it = 0, ahead = 0;
      bool ok = true;
      auto stage = [&](int i) { return smem + (size_t)(i % S::kStages) * S::kStageBytes; };
      auto load_w = [&](int i, int k, int w_row) {
        mbar_arrive_expect_tx(&full[i % S::kStages], (uint32_t)(a_rows + BN) * kTileK * 2);
        for (int b = 0; b < BN; b += kWBox)
          tma_load_2d(stage(i) + kABytes + b * kTileK * 2, &wmap, k * kTileK, w_row + b, &full[i % S::kStages]);
      };
      if (GROUPED) {
        grouped_start();
      } else {  // the weights do not depend on the previous kernel, the activations do: fill the ring with weights first
        const int item = blockIdx.x;
        int k0, k1;
        k_range(item / (mt * nt), k0, k1);
        for (; ahead < S::kStages && ahead < k1 - k0; ++ahead) load_w(ahead, k0 + ahead, (item / mt % nt) * BN);
        pdl_wait_prior();
      }
      for (int item = blockIdx.x; item < mt * nt * splits && ok; item += gridDim.x) {
        int x_row = (item % mt) * kTileM, w_row = (item / mt % nt) * BN;
        if (GROUPED) {
          const int4 t = tiles[item % mt];
          x_row = t.y;
          w_row += t.x * N;
          a_box = t.z > kTileM - 16 ? kTileM : 16;
          a_rows = (t.z + 15) / 16 * 16;
        }
        const CUtensorMap* am = !GROUPED || a_box == kTileM ? &amap : &amap16;
        int k0, k1;
        k_range(item / (mt * nt), k0, k1);
        for (int k = k0; k < k1; ++k, ++it) {
          const int st = it % S::kStages;
          if (it >= S::kStages && (gave_up || !mbar_wait_bounded(&empty[st], ((it / S::kStages) & 1) ^ 1))) {
            ok = false;
            break;
          }
          if (it >= ahead) load_w(it, k, w_row);
          for (int b = 0; b < a_rows; b += a_box) tma_load_2d(stage(it) + b * kTileK * 2, am, k * kTileK, x_row + b, &full[st]);
        }
      }
      if (!ok) gave_up = 1;
      // nothing in flight when the CTA leaves: the last copies of every stage have landed
      for (int i = it > S::kStages ? it - S::kStages : 0; !ok && i < it; ++i)
        mbar_wait_bounded(&full[i % S::kStages], (i / S::kStages) & 1);
    }
  } else if (warp == 1) {
    const bool leader = elect_one_sync();
    const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kTileM >> 4) << 24);
    int it = 0, t = 0;
    bool ok = true;
    if (GROUPED) grouped_start();
    for (int item = blockIdx.x; item < mt * nt * splits && ok; item += gridDim.x, ++t) {
      int k0, k1;
      k_range(item / (mt * nt), k0, k1);
      const int buf = t & 1;
      if (t >= 2 && (gave_up || !mbar_wait_bounded(&acc_empty[buf], ((t >> 1) & 1) ^ 1))) ok = false;
      tc_fence_after();
      for (int k = k0; k < k1 && ok; ++k, ++it) {
        const int st = it % S::kStages;
        if (gave_up || !mbar_wait_bounded(&full[st], (it / S::kStages) & 1)) {
          ok = false;
          break;
        }
        tc_fence_after();
        if (leader) {
          const uint32_t a = smem_u32(smem + (size_t)st * S::kStageBytes);
          const uint64_t ad = swizzled_desc(a), bd = swizzled_desc(a + kABytes);
#pragma unroll
          for (int j = 0; j < kTileK / 16; ++j)
            tc_mma_f16(tmem + buf * BN, ad + j * 2, bd + j * 2, idesc, (k > k0 || j > 0) ? 1u : 0u);
          tc_commit(&empty[st]);
        }
        __syncwarp();
      }
      if (ok && leader) tc_commit(&acc_full[buf]);
      __syncwarp();
    }
    if (!ok) gave_up = 1;
  } else {
    if (GROUPED) grouped_start();
    else pdl_wait_prior();  // outputs may still be read by the kernel before
    const int quarter = warp & 3;
    int t = 0;
    for (int item = blockIdx.x; item < mt * nt * splits; item += gridDim.x, ++t) {
      const int buf = t & 1;
      if (gave_up || !mbar_wait_bounded(&acc_full[buf], (t >> 1) & 1)) {
        gave_up = 1;
        break;
      }
      tc_fence_after();
      const int n0 = (item / mt % nt) * BN, split = item / (mt * nt);
      int m0 = (item % mt) * kTileM, m_end = M;
      if (GROUPED) {
        const int4 tile = tiles[item % mt];
        m0 = tile.w;
        m_end = tile.w + tile.z;
      }
      const int m = m0 + quarter * 32 + lane;
      if (m0 + quarter * 32 < m_end) {
        const uint32_t base = tmem + ((uint32_t)(quarter * 32) << 16) + buf * BN;
#pragma unroll 1  // a kernel starts with a cold instruction cache: short code
        for (int c = 0; c < BN; c += 32) {
          if (n0 + c >= N) break;
          uint32_t r0[16], r1[16];
          tmem_ld16(base + c, r0);
          tmem_ld16(base + c + 16, r1);
          tmem_ld_wait();
          float v[16];
          if (m < m_end) {
#pragma unroll
            for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r0[i]);
            store16<FORM>(e, m, n0 + c, N, v, split);
            if (n0 + c + 16 < N) {
#pragma unroll
              for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r1[i]);
              store16<FORM>(e, m, n0 + c + 16, N, v, split);
            }
          }
          __syncwarp();
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&acc_empty[buf]);
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (warp == 1) tmem_dealloc(tmem, S::kTmemCols);
}

// ------------------------------------------------------------------------------------------ packing
__global__ void lm_pack_rows_kernel(const __nv_bfloat16* __restrict__ src, int n, int k, __nv_bfloat16* __restrict__ dst, int ldk,
                                    int row_block, int row_block_pad, int row_mul, int row_off, int col_block, int col_block_pad) {
  for (int r = blockIdx.x; r < n; r += gridDim.x) {
    const size_t dr = (size_t)((r / row_block) * row_block_pad + r % row_block) * row_mul + row_off;
    for (int c = threadIdx.x; c < k; c += blockDim.x)
      dst[dr * ldk + (c / col_block) * col_block_pad + c % col_block] = src[(size_t)r * k + c];
  }
}

__global__ void lm_pack_heads_transposed_kernel(const __nv_bfloat16* __restrict__ src, int heads, int dim, int rank,
                                                __nv_bfloat16* __restrict__ dst, int rankp, int dimp) {
  for (int r = blockIdx.x; r < heads * rank; r += gridDim.x) {
    const int h = r / rank, c = r - h * rank;
    for (int d = threadIdx.x; d < dim; d += blockDim.x)
      dst[((size_t)h * rankp + c) * dimp + d] = src[((size_t)h * dim + d) * rank + c];
  }
}

using EncodeFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                              const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                              CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

int encode(CUtensorMap* map, const void* base, int rows, int k, int box_rows) {
  static EncodeFn fn = nullptr;
  if (!fn) {
    cudaDriverEntryPointQueryResult q;
    void* p = nullptr;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || !p) return MLLMB200_CUDA_ERROR;
    fn = reinterpret_cast<EncodeFn>(p);
  }
  const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)k * 2};
  const cuuint32_t box[2] = {(cuuint32_t)kTileK, (cuuint32_t)box_rows}, one[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
             ? MLLMB200_OK
             : MLLMB200_CUDA_ERROR;
}

// Tile width and K splits with the smallest estimated time: waves x (K tiles x cycles per K tile + fixed cost).
void choose_tile(int M, int mt, int a_rows, int N, int K, int max_splits, int* bn_out, int* splits_out) {
  const int kt = K / kTileK;
  double best = 1e30;
  for (int bn : {256, 128, 64, 32}) {
    const int nt = (N + bn - 1) / bn;
    for (int s = 1; s <= max_splits && s <= kt; ++s) {
      const long long items = (long long)mt * nt * s;
      const double waves = (double)((items + kSms - 1) / kSms);
      const double per_k = std::max(2.0 * bn, (a_rows + bn) * 128.0 / 40.0);
      // more planes are written here and read by the consumer: about 2600 bytes per cycle
      const double t = waves * (((kt + s - 1) / s) * per_k + 600.0 + 6.0 * bn) + 900.0 + (s - 1) * (150.0 + 8.0 * M * N / 2600.0);
      if (t < best) best = t, *bn_out = bn, *splits_out = s;
    }
  }
}

template <int BN, int FORM>
cudaError_t launch_tc_form(cudaStream_t s, const Linear& w, const ActMap& am, int M, int splits, const Groups* g, const Epi& e) {
  const int nt = (w.n + BN - 1) / BN;
  const CUtensorMap& wmap = BN < 128 ? w.map32 : w.map128;
  if (g)
    return launch_pdl(lm_gemm_tc_kernel<BN, true, FORM>, dim3(std::min(g->max_tiles * nt * splits, kSms)), dim3(kTcThreads), TcShape<BN>::kSmem,
                      s, am.map128, am.map16, wmap, 128, M, w.n, w.k, splits, g->tiles, g->n_tiles, g->max_tiles, e);
  const int mt = (M + kTileM - 1) / kTileM;
  return launch_pdl(lm_gemm_tc_kernel<BN, false, FORM>, dim3(std::min(mt * nt * splits, kSms)), dim3(kTcThreads), TcShape<BN>::kSmem, s,
                    M >= kTileM ? am.map128 : am.map16, am.map16, wmap, M >= kTileM ? 128 : 16, M, w.n, w.k, splits, nullptr, nullptr, 0, e);
}
template <int BN>
cudaError_t launch_tc(cudaStream_t s, const Linear& w, const ActMap& am, int M, int splits, const Groups* g, const Epi& e) {
  const Form f = form_of(e);
  return f == kFormPlanes ? launch_tc_form<BN, kFormPlanes>(s, w, am, M, splits, g, e)
         : f == kFormGate ? launch_tc_form<BN, kFormGate>(s, w, am, M, splits, g, e)
                          : launch_tc_form<BN, kFormScatter>(s, w, am, M, splits, g, e);
}
template <int BN, int FORM>
cudaError_t configure_tc() {
  const cudaError_t r = cudaFuncSetAttribute(lm_gemm_tc_kernel<BN, false, FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcShape<BN>::kSmem);
  return r != cudaSuccess ? r : cudaFuncSetAttribute(lm_gemm_tc_kernel<BN, true, FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcShape<BN>::kSmem);
}
template <int BN>
cudaError_t configure_tc_forms() {
  cudaError_t r = configure_tc<BN, kFormPlanes>();
  if (r == cudaSuccess) r = configure_tc<BN, kFormScatter>();
  return r != cudaSuccess ? r : configure_tc<BN, kFormGate>();
}

template <class T, int MT>
cudaError_t launch_gemv_mt(cudaStream_t s, const Linear& w, const void* x, const Groups* g, const Epi& e) {
  int ks = 0;
  const int pairs = (w.n + 1) / 2, ys = g ? g->rows : 1;
  while (ks < 3 && ((long long)pairs * ys << ks) / kGemvWarps < 2 * kSms && (w.k >> (8 + ks)) >= 2) ++ks;
  const int per_cta = kGemvWarps >> ks;
  return launch_pdl(lm_gemv_kernel<T, MT>, dim3((pairs + per_cta - 1) / per_cta, ys), dim3(kGemvThreads), (size_t)MT * w.k * sizeof(T), s,
                    static_cast<const T*>(x), w.w, w.n, w.k, ks, g ? g->group_of : nullptr, g ? g->div : 1, e);
}
template <class T>
cudaError_t launch_gemv(cudaStream_t s, const Linear& w, const void* x, int M, const Epi& e) {
  switch (M) {
    case 1: return launch_gemv_mt<T, 1>(s, w, x, nullptr, e);
    case 2: return launch_gemv_mt<T, 2>(s, w, x, nullptr, e);
    case 3: return launch_gemv_mt<T, 3>(s, w, x, nullptr, e);
    default: return launch_gemv_mt<T, 4>(s, w, x, nullptr, e);
  }
}
constexpr size_t kGemvSmemMax = 200 * 1024;
template <class T>
cudaError_t configure_gemv() {
  cudaError_t r = cudaSuccess;
  auto set = [&](auto f) {
    if (r == cudaSuccess) r = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGemvSmemMax);
  };
  set(lm_gemv_kernel<T, 1>);
  set(lm_gemv_kernel<T, 2>);
  set(lm_gemv_kernel<T, 3>);
  set(lm_gemv_kernel<T, 4>);
  return r;
}

}  // namespace

cudaError_t linear_configure() {
  cudaError_t r = configure_tc_forms<256>();
  if (r == cudaSuccess) r = configure_tc_forms<128>();
  if (r == cudaSuccess) r = configure_tc_forms<64>();
  if (r == cudaSuccess) r = configure_tc_forms<32>();
  if (r == cudaSuccess) r = configure_gemv<float>();
  if (r == cudaSuccess) r = configure_gemv<__nv_bfloat16>();
  return r;
}

int make_act_map(ActMap* m, const void* buf, int rows, int k) {
  const int st = encode(&m->map16, buf, rows, k, 16);
  return st != MLLMB200_OK ? st : encode(&m->map128, buf, rows, k, 128);
}
int make_linear_maps(Linear* l) {
  const int st = encode(&l->map32, l->w, l->n * l->groups, l->k, 32);
  return st != MLLMB200_OK ? st : encode(&l->map128, l->w, l->n * l->groups, l->k, 128);
}

namespace {
cudaError_t launch_tc_any(cudaStream_t s, int bn, const Linear& w, const ActMap& am, int M, int splits, const Groups* g, const Epi& e) {
  return bn == 256   ? launch_tc<256>(s, w, am, M, splits, g, e)
         : bn == 128 ? launch_tc<128>(s, w, am, M, splits, g, e)
         : bn == 64  ? launch_tc<64>(s, w, am, M, splits, g, e)
                     : launch_tc<32>(s, w, am, M, splits, g, e);
}
}  // namespace

int group_tile_rows(bool f32) { return f32 ? kF32Tile : kTileM; }

int launch_linear(cudaStream_t s, bool f32, const Linear& w, const ActMap& am, const void* x, int M, const Epi& e, int max_splits) {
  cudaError_t r;
  int splits = 1;
  const size_t elt = f32 ? 4 : 2;
  if (M <= kGemvRows && (size_t)M * w.k * elt <= kGemvSmemMax) {
    r = f32 ? launch_gemv<float>(s, w, x, M, e) : launch_gemv<__nv_bfloat16>(s, w, x, M, e);
  } else if (f32) {
    r = launch_pdl(lm_gemm_f32_kernel, dim3((w.n + kF32Tile - 1) / kF32Tile, (M + kF32Tile - 1) / kF32Tile), dim3(256), 0, s,
                   static_cast<const float*>(x), w.w, M, w.n, w.k, nullptr, nullptr, e);
  } else {
    int bn = 32;
    choose_tile(M, (M + kTileM - 1) / kTileM, M >= kTileM ? kTileM : pad_to(M, 16), w.n, w.k, e.kind == kEpiPlanes ? max_splits : 1, &bn, &splits);
    r = launch_tc_any(s, bn, w, am, M, splits, nullptr, e);
  }
  return r == cudaSuccess ? splits : -1;
}

int launch_linear_groups(cudaStream_t s, bool f32, const Linear& w, const ActMap& am, const void* x, const Groups& g, const Epi& e, int max_splits) {
  cudaError_t r;
  int splits = 1;
  if (g.group_of) {
    r = f32 ? launch_gemv_mt<float, 1>(s, w, x, &g, e) : launch_gemv_mt<__nv_bfloat16, 1>(s, w, x, &g, e);
  } else if (f32) {
    r = launch_pdl(lm_gemm_f32_kernel, dim3((w.n + kF32Tile - 1) / kF32Tile, g.max_tiles), dim3(256), 0, s, static_cast<const float*>(x), w.w, 0,
                   w.n, w.k, g.tiles, g.n_tiles, e);
  } else {
    int bn = 32;
    const int per = (g.rows + g.likely_tiles - 1) / g.likely_tiles;
    choose_tile(g.rows, g.likely_tiles, std::min(kTileM, pad_to(per, 16)), w.n, w.k, e.kind == kEpiPlanes ? max_splits : 1, &bn, &splits);
    r = launch_tc_any(s, bn, w, am, g.rows, splits, &g, e);
  }
  return r == cudaSuccess ? splits : -1;
}

cudaError_t launch_pack_heads_transposed(cudaStream_t s, const __nv_bfloat16* src, int heads, int dim, int rank, __nv_bfloat16* dst,
                                         int rankp, int dimp) {
  lm_pack_heads_transposed_kernel<<<std::min(heads * rank, 148 * 16), 256, 0, s>>>(src, heads, dim, rank, dst, rankp, dimp);
  return cudaGetLastError();
}
cudaError_t launch_pack_rows(cudaStream_t s, const __nv_bfloat16* src, int n, int k, __nv_bfloat16* dst, int ldk, int row_block,
                             int row_block_pad, int row_mul, int row_off, int col_block, int col_block_pad) {
  lm_pack_rows_kernel<<<std::min(n, 148 * 16), 256, 0, s>>>(src, n, k, dst, ldk, row_block, row_block_pad, row_mul, row_off, col_block,
                                                          col_block_pad);
  return cudaGetLastError();
}

}  // namespace lm
}  // namespace mllmb200
