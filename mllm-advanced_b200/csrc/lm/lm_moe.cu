// Mixture of experts: the choice from router logits, and the rows in expert order.  A pair is (row, k-th choice).
#include <algorithm>

#include "../device_common.cuh"
#include "lm_route.cuh"

namespace mllmb200 {
namespace lm {
namespace {

constexpr int kTopkWarps = 8;

// a warp per row; logits [planes][rows][ldl] without the bias
__global__ void __launch_bounds__(kTopkWarps * 32) lm_topk_kernel(RouterArgs a, const float* __restrict__ logits, int ldl, int planes,
                                                                  size_t plane, int rows) {
  extern __shared__ float z_all[];  // [warps][experts]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * kTopkWarps + warp;
  if (row >= rows) return;
  float* z = z_all + (size_t)warp * a.experts;
  const float* src = logits + (size_t)row * ldl;
  for (int e = lane; e < a.experts; e += 32) {
    float p[kMaxSplits], v = a.b[e];
#pragma unroll
    for (int i = 0; i < kMaxSplits; ++i) p[i] = i < planes ? src[i * plane + e] : 0.0f;
#pragma unroll
    for (int i = 0; i < kMaxSplits; ++i) v += p[i];
    z[e] = v;
  }
  __syncwarp();
  choose_experts(z, a, row, lane);
}

constexpr int kPermThreads = 256, kPermWarps = kPermThreads / 32;

// Expert e's rows start at the sum of the counts before it; a pair's row follows from its rank.  A warp copies a pair's
// row; the first CTA also writes the row tiles of the grouped linears.
__global__ void __launch_bounds__(kPermThreads) lm_moe_permute_kernel(RouterArgs a, const uint4* __restrict__ x, int row16, int rows,
                                                                      int tile_rows, uint4* __restrict__ out, int* __restrict__ pair_row,
                                                                      int4* __restrict__ tiles, int* __restrict__ n_tiles) {
  __shared__ int s_first[kMaxExperts], s_tile[kMaxExperts];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (warp == 0) {
    int at = 0, tile = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
      const int e = e0 + lane, n = e < a.experts ? a.count[e] : 0, nt = (n + tile_rows - 1) / tile_rows;
      int sn = n, st = nt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, sn, o), v = __shfl_up_sync(0xffffffffu, st, o);
        if (lane >= o) sn += u, st += v;
      }
      if (e < a.experts) s_first[e] = at + sn - n, s_tile[e] = tile + st - nt;
      at += __shfl_sync(0xffffffffu, sn, 31);
      tile += __shfl_sync(0xffffffffu, st, 31);
    }
    if (blockIdx.x == 0 && lane == 0) *n_tiles = tile;
  }
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = tid; e < a.experts; e += kPermThreads) {
      const int n = a.count[e];
      for (int j = 0, t = s_tile[e]; j < n; j += tile_rows, ++t)
        tiles[t] = make_int4(e, s_first[e] + j, min(tile_rows, n - j), s_first[e] + j);
    }
  const int pairs = rows * a.top;
  for (int p = blockIdx.x * kPermWarps + warp; p < pairs; p += gridDim.x * kPermWarps) {
    const int dst = s_first[a.sel[p]] + a.rank[p];
    if (lane == 0) pair_row[p] = dst;
    const uint4* src = x + (size_t)(p / a.top) * row16;
    uint4* to = out + (size_t)dst * row16;
    for (int c = lane; c < row16; c += 32) to[c] = src[c];
  }
}

}  // namespace

cudaError_t launch_topk(cudaStream_t s, const RouterArgs& a, const float* logits, int ldl, int planes, size_t plane, int rows) {
  return launch_pdl(lm_topk_kernel, dim3((rows + kTopkWarps - 1) / kTopkWarps), dim3(kTopkWarps * 32), (size_t)kTopkWarps * a.experts * 4, s, a,
                    logits, ldl, planes, plane, rows);
}

cudaError_t launch_moe_permute(cudaStream_t s, bool f32, const RouterArgs& a, const void* x, int ldx, int rows, void* out, int* pair_row,
                               int4* tiles, int* n_tiles) {
  const int grid = std::min((rows * a.top + kPermWarps - 1) / kPermWarps, 8 * kSms);
  return launch_pdl(lm_moe_permute_kernel, dim3(grid), dim3(kPermThreads), 0, s, a, static_cast<const uint4*>(x), ldx * (f32 ? 4 : 2) / 16, rows,
                    group_tile_rows(f32), static_cast<uint4*>(out), pair_row, tiles, n_tiles);
}

}  // namespace lm
}  // namespace mllmb200
