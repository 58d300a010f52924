// Row operators of the language-model engine: embedding, sandwich norm with residual and causal input convolution, norm
// behind the residual sum (with the choice of experts), the bookkeeping of a decode step, and the argmax candidates of greedy sampling.
#include <cooperative_groups.h>

#include <algorithm>

#include "../device_common.cuh"
#include "lm_route.cuh"

namespace mllmb200 {
namespace lm {
namespace {

constexpr int kNormThreads = 256;

__device__ __forceinline__ float block_sum(float v, float* scratch) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float t = lane < (int)(blockDim.x >> 5) ? scratch[lane] : 0.0f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) t += __shfl_xor_sync(0xffffffffu, t, o);
  return t;
}

__device__ __forceinline__ float4 fma4(float s, const float4& a, const float4& b) {
  return make_float4(fmaf(s, a.x, b.x), fmaf(s, a.y, b.y), fmaf(s, a.z, b.z), fmaf(s, a.w, b.w));
}
__device__ __forceinline__ float dot4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// columns [c, c + 4) of a row of the sublayer output
__device__ __forceinline__ float4 load_delta(const Delta& d, int row, int c) {
  if (!d.mix_w) {
    const float* p = d.p + (size_t)row * d.ldx + c;
    float4 v = *reinterpret_cast<const float4*>(p);
    for (int i = 1; i < d.planes; ++i) v = fma4(1.0f, *reinterpret_cast<const float4*>(p + i * d.plane), v);
    return v;
  }
  float4 v = make_float4(0, 0, 0, 0);
  for (int k = 0; k < d.top; ++k) {
    const int pair = row * d.top + k;
    const float* p = d.p + (size_t)(d.mix_row ? d.mix_row[pair] : pair) * d.ldx + c;
    float4 y = *reinterpret_cast<const float4*>(p);
    for (int i = 1; i < d.planes; ++i) y = fma4(1.0f, *reinterpret_cast<const float4*>(p + i * d.plane), y);
    v = fma4(d.mix_w[pair], y, v);
  }
  return v;
}

// x' = x + rms_unit(delta) * g_post;  h = rms_unit(x') * g_pre;  out = h + conv(h).
// The gains are one number per norm.  A CTA walks `rows_per_cta` rows in order and keeps the last taps rows of h in
// shared memory; the taps - 1 rows in front of its first one are recomputed (x_in is not overwritten: x_out is another
// buffer), or come from the sequence's tail when they belong to an earlier step.  A thread owns the same columns of
// every row, so the ring needs no synchronization.  The CTA with a sequence's last row writes the new tail, into the
// other of the sequence's two tail buffers (another CTA may still read the old one).
template <class T, int NV>
__global__ void __launch_bounds__(kNormThreads) lm_norm_kernel(NormArgs a) {
  extern __shared__ __align__(16) float ring[];  // [taps][ldx]
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int tid = threadIdx.x, nv = a.ldx >> 2;
  const float g_pre = *a.g_pre, g_post = a.delta.p ? *a.g_post : 0.0f, inv_w = 1.0f / (float)a.width;
  const int r_begin = blockIdx.x * a.rows_per_cta, r_end = min(r_begin + a.rows_per_cta, a.rows);
  int t0 = r_begin;
  if (a.taps > 1) t0 = max(r_begin - (a.taps - 1), a.entries[a.row_entry[r_begin]].row0);
  for (int t = t0; t < r_end; ++t) {
    const int src = a.gather ? a.gather[t] : t;
    const float* xr = a.x_in + (size_t)src * a.ldx;
    float4 x[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = tid + i * kNormThreads;
      x[i] = c < nv ? reinterpret_cast<const float4*>(xr)[c] : make_float4(0, 0, 0, 0);
    }
    if (a.delta.p) {
      float4 d[NV];
      float ss = 0.0f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = tid + i * kNormThreads;
        d[i] = make_float4(0, 0, 0, 0);
        if (c < nv) {
          d[i] = load_delta(a.delta, src, c * 4);
          ss += dot4(d[i]);
        }
      }
      const float r = g_post / sqrtf(block_sum(ss, scratch) * inv_w + a.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i) x[i] = fma4(r, d[i], x[i]);
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += dot4(x[i]);
    const float r = g_pre / sqrtf(block_sum(ss, scratch) * inv_w + a.eps);
    const bool own = t >= r_begin;
    if (own && a.x_out) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = tid + i * kNormThreads;
        if (c < nv) store4(a.x_out + (size_t)t * a.ldx + c * 4, x[i]);
      }
    }
    T* out = static_cast<T*>(a.out) + (size_t)t * a.ldx;
    if (a.taps == 0) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = tid + i * kNormThreads;
        if (c < nv) store4(out + c * 4, fma4(r, x[i], make_float4(0, 0, 0, 0)));
      }
      continue;
    }
    const Entry e = a.entries[a.row_entry[t]];
    const int off = t - e.row0, keep = a.taps - 1;
    const float* old_tail = a.tail + ((size_t)e.slot * 2 + e.tail) * keep * a.ldx;
    float* new_tail = a.tail + ((size_t)e.slot * 2 + (e.tail ^ 1)) * keep * a.ldx;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = tid + i * kNormThreads;
      if (c >= nv) continue;
      const float4 h = fma4(r, x[i], make_float4(0, 0, 0, 0));
      store4(ring + (size_t)(t % a.taps) * a.ldx + c * 4, h);
      if (!own) continue;
      float4 y = h;
      for (int s = 0; s < a.taps; ++s) {
        float4 hs;
        if (s <= off) hs = *reinterpret_cast<const float4*>(ring + (size_t)((t - s) % a.taps) * a.ldx + c * 4);
        else if (s <= e.pos0 + off) hs = *reinterpret_cast<const float4*>(old_tail + (size_t)(keep - (s - off)) * a.ldx + c * 4);
        else break;  // before the start of the sequence
        const float4 w = *reinterpret_cast<const float4*>(a.conv_w + (size_t)(keep - s) * a.ldx + c * 4);
        y = make_float4(fmaf(w.x, hs.x, y.x), fmaf(w.y, hs.y, y.y), fmaf(w.z, hs.z, y.z), fmaf(w.w, hs.w, y.w));
      }
      store4(out + c * 4, y);
      const int at = keep - (e.count - off);
      if (at >= 0) store4(new_tail + (size_t)at * a.ldx + c * 4, h);
      if (off == e.count - 1)  // a short step: older rows move down
        for (int j = 0; j + e.count < keep; ++j)
          store4(new_tail + (size_t)j * a.ldx + c * 4, *reinterpret_cast<const float4*>(old_tail + (size_t)(j + e.count) * a.ldx + c * 4));
    }
  }
}

// A row of the sublayer output, column lane + 32 i of float4s in x[i].
template <int NVW>
__device__ __forceinline__ void warp_delta(const Delta& d, int row, int lane, int nv, float4 (&x)[NVW]) {
  const int n_src = d.mix_w ? d.top : 1;
#pragma unroll
  for (int i = 0; i < NVW; ++i) x[i] = make_float4(0, 0, 0, 0);
  for (int k = 0; k < n_src; ++k) {
    const int pair = row * n_src + k;
    const float g = d.mix_w ? d.mix_w[pair] : 1.0f;
    const float* src = d.p + (size_t)(d.mix_w && d.mix_row ? d.mix_row[pair] : pair) * d.ldx;
    for (int p = 0; p < d.planes; ++p)
#pragma unroll
      for (int i = 0; i < NVW; ++i) {
        const int c = lane + i * 32;
        if (c < nv) x[i] = fma4(g, *reinterpret_cast<const float4*>(src + p * d.plane + c * 4), x[i]);
      }
  }
}

// The same for many rows: a warp per row for the sums (no block barrier inside), then - with a convolution - the threads
// sweep the CTA's rows column by column with the last TW - 1 rows of h in registers.  x' of the CTA's own rows is read
// back from x_out (or x_in when there is nothing to fold in), that of the rows in front of them from shared memory.
constexpr int kRowsThreads = 384, kRowsWarps = kRowsThreads / 32;  // rows a CTA handles at once, the recomputed ones included

template <class T, int NVW, int TW>
__global__ void __launch_bounds__(kRowsThreads) lm_norm_rows_kernel(NormArgs a) {
  extern __shared__ __align__(16) float halo[];  // [TW - 1][ldx]
  __shared__ float s_r[2 * kRowsWarps];
  __shared__ Entry s_e[2 * kRowsWarps];
  pdl_launch_dependents();
  pdl_wait_prior();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nv = a.ldx >> 2;
  const float g_pre = *a.g_pre, g_post = a.delta.p ? *a.g_post : 0.0f, inv_w = 1.0f / (float)a.width;
  const int r_begin = blockIdx.x * a.rows_per_cta, r_end = min(r_begin + a.rows_per_cta, a.rows);
  int t0 = r_begin;
  if (TW > 1) t0 = max(r_begin - (a.taps - 1), a.entries[a.row_entry[r_begin]].row0);
  auto warp_sum = [](float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
  };
  if (TW > 1 && tid < r_end - t0) s_e[tid] = a.entries[a.row_entry[t0 + tid]];
  for (int t = t0 + warp; t < r_end; t += kRowsWarps) {
    const float4* xr = reinterpret_cast<const float4*>(a.x_in + (size_t)t * a.ldx);
    float4 x[NVW];
    float ss = 0.0f;
    if (a.delta.p) {
      warp_delta<NVW>(a.delta, t, lane, nv, x);
#pragma unroll
      for (int i = 0; i < NVW; ++i) ss += dot4(x[i]);
      const float r = g_post / sqrtf(warp_sum(ss) * inv_w + a.eps);
      ss = 0.0f;
#pragma unroll
      for (int i = 0; i < NVW; ++i) {
        const int c = lane + i * 32;
        if (c < nv) x[i] = fma4(r, x[i], xr[c]);
        ss += dot4(x[i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < NVW; ++i) {
        const int c = lane + i * 32;
        x[i] = c < nv ? xr[c] : make_float4(0, 0, 0, 0);
        ss += dot4(x[i]);
      }
    }
    const float r = g_pre / sqrtf(warp_sum(ss) * inv_w + a.eps);
    float* keep = t < r_begin ? halo + (size_t)(t - t0) * a.ldx : (a.x_out ? a.x_out + (size_t)t * a.ldx : nullptr);
    T* out = static_cast<T*>(a.out) + (size_t)t * a.ldx;
    if (lane == 0) s_r[t - t0] = r;
#pragma unroll
    for (int i = 0; i < NVW; ++i) {
      const int c = lane + i * 32;
      if (c >= nv) continue;
      if (keep) store4(keep + c * 4, x[i]);
      if (TW == 1) store4(out + c * 4, fma4(r, x[i], make_float4(0, 0, 0, 0)));
    }
  }
  if (TW == 1) return;
  __syncthreads();
  const int keep = a.taps - 1;
  const float* own_x = a.delta.p ? a.x_out : a.x_in;
  for (int c = tid * 4; c < a.ldx; c += kRowsThreads * 4) {
    float4 w[TW], hist[TW];  // hist[s]: h of s rows ago
#pragma unroll
    for (int s = 0; s < TW; ++s) {
      w[s] = s <= keep ? *reinterpret_cast<const float4*>(a.conv_w + (size_t)(keep - s) * a.ldx + c) : make_float4(0, 0, 0, 0);
      hist[s] = make_float4(0, 0, 0, 0);
    }
    for (int tb = t0; tb < r_end; tb += kRowsWarps) {
      float4 x[kRowsWarps];
#pragma unroll
      for (int u = 0; u < kRowsWarps; ++u) {
        const int t = tb + u;
        if (t < r_end) x[u] = *reinterpret_cast<const float4*>(t >= r_begin ? own_x + (size_t)t * a.ldx + c : halo + (size_t)(t - t0) * a.ldx + c);
      }
#pragma unroll
      for (int u = 0; u < kRowsWarps; ++u) {
        const int t = tb + u;
        if (t >= r_end) break;
        const Entry e = s_e[t - t0];
        const int off = t - e.row0;
        if (off == 0) {  // a sequence's share starts: the rows before it come from its tail, or are zero
          const float* old_tail = a.tail + ((size_t)e.slot * 2 + e.tail) * keep * a.ldx + c;
#pragma unroll
          for (int s = 1; s < TW; ++s)
            hist[s] = s <= keep && s <= e.pos0 ? *reinterpret_cast<const float4*>(old_tail + (size_t)(keep - s) * a.ldx) : make_float4(0, 0, 0, 0);
        }
        hist[0] = fma4(s_r[t - t0], x[u], make_float4(0, 0, 0, 0));
        if (t >= r_begin) {
          float4 y = hist[0];
#pragma unroll
          for (int s = 0; s < TW; ++s)
            y = make_float4(fmaf(w[s].x, hist[s].x, y.x), fmaf(w[s].y, hist[s].y, y.y), fmaf(w[s].z, hist[s].z, y.z), fmaf(w[s].w, hist[s].w, y.w));
          store4(static_cast<T*>(a.out) + (size_t)t * a.ldx + c, y);
          const int at = keep - (e.count - off);
          if (at >= 0) {  // among the last rows of its sequence's share: the new tail
            const float* old_tail = a.tail + ((size_t)e.slot * 2 + e.tail) * keep * a.ldx + c;
            float* new_tail = a.tail + ((size_t)e.slot * 2 + (e.tail ^ 1)) * keep * a.ldx + c;
            store4(new_tail + (size_t)at * a.ldx, hist[0]);
            if (off == e.count - 1)  // a short step: older rows move down
              for (int j = 0; j + e.count < keep; ++j)
                store4(new_tail + (size_t)j * a.ldx, *reinterpret_cast<const float4*>(old_tail + (size_t)(j + e.count) * a.ldx));
          }
        }
#pragma unroll
        for (int s = TW - 1; s > 0; --s) hist[s] = hist[s - 1];
      }
    }
  }
}

template <class T, int NVW>
cudaError_t launch_norm_rows(cudaStream_t s, NormArgs a) {
  const int halo = a.taps ? a.taps - 1 : 0;
  a.rows_per_cta = (a.rows >= 4 * kSms * kRowsWarps ? 2 : 1) * kRowsWarps - halo;
  const dim3 grid((a.rows + a.rows_per_cta - 1) / a.rows_per_cta);
  if (a.taps == 0) return launch_pdl(lm_norm_rows_kernel<T, NVW, 1>, grid, dim3(kRowsThreads), 0, s, a);
  const size_t smem = (size_t)halo * a.ldx * sizeof(float);
  if (smem > 40 * 1024) {
    const cudaError_t r = cudaFuncSetAttribute(lm_norm_rows_kernel<T, NVW, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (r != cudaSuccess) return r;
  }
  return launch_pdl(lm_norm_rows_kernel<T, NVW, 4>, grid, dim3(kRowsThreads), smem, s, a);
}

template <class T, int NV>
cudaError_t launch_norm_nv(cudaStream_t s, const NormArgs& a) {
  const size_t smem = (size_t)a.taps * a.ldx * sizeof(float);
  if (smem > 48 * 1024) {
    const cudaError_t r = cudaFuncSetAttribute(lm_norm_kernel<T, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (r != cudaSuccess) return r;
  }
  return launch_pdl(lm_norm_kernel<T, NV>, dim3((a.rows + a.rows_per_cta - 1) / a.rows_per_cta), dim3(kNormThreads), smem, s, a);
}
template <class T>
cudaError_t launch_norm_t(cudaStream_t s, const NormArgs& a) {
  // enough rows for a warp each, and a convolution (if any) that fits the register window
  if (a.rows >= 2 * kSms && !a.gather && (a.taps == 0 || (a.taps >= 2 && a.taps <= 4)) && a.ldx <= 4096) {
    const int w = (a.ldx / 4 + 31) / 32;
    if (w <= 8) return launch_norm_rows<T, 8>(s, a);
    if (w <= 16) return launch_norm_rows<T, 16>(s, a);
    return launch_norm_rows<T, 32>(s, a);
  }
  const int per = (a.ldx / 4 + kNormThreads - 1) / kNormThreads;
  if (per <= 1) return launch_norm_nv<T, 1>(s, a);
  if (per <= 2) return launch_norm_nv<T, 2>(s, a);
  if (per <= 4) return launch_norm_nv<T, 4>(s, a);
  if (per <= 8) return launch_norm_nv<T, 8>(s, a);
  return cudaErrorInvalidValue;
}

// x' = rms_unit(alpha x + delta) * gain, a CTA per row.  With a router a cluster of CTAs per row: each makes the row and
// the logits of its share of the experts, the first one keeps the row and chooses.
template <class T, int NV, bool ROUTER>
__global__ void __launch_bounds__(kNormThreads) lm_post_norm_kernel(PostNormArgs a) {
  extern __shared__ __align__(16) float row_x[];  // [ldx], then [experts]; with a router only
  __shared__ float scratch[32];
  const int tid = threadIdx.x, nv = a.ldx >> 2, t = blockIdx.x, part = ROUTER ? blockIdx.y : 0, parts = ROUTER ? gridDim.y : 1;
  pdl_launch_dependents();
  if (ROUTER)  // the router's weights do not depend on the previous kernel: into L2, a share per row and CTA
    for (size_t at = ((size_t)(t * parts + part) * kNormThreads + tid) * 64, step = (size_t)gridDim.x * parts * kNormThreads * 64;
         at < (size_t)a.router.experts * a.router.ldw; at += step)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(a.router.w + at));
  float4 g[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = tid + i * kNormThreads;
    g[i] = c < nv ? __ldg(reinterpret_cast<const float4*>(a.gain) + c) : make_float4(0, 0, 0, 0);
  }
  pdl_wait_prior();
  const int src = a.gather ? a.gather[t] : t;
  float4 x[NV];
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = tid + i * kNormThreads;
    x[i] = make_float4(0, 0, 0, 0);
    if (c < nv) {
      const float4 d = a.delta.p ? load_delta(a.delta, src, c * 4) : x[i];
      x[i] = fma4(a.alpha, *reinterpret_cast<const float4*>(a.x_in + (size_t)src * a.ldx + c * 4), d);
    }
    ss += dot4(x[i]);
  }
  const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)a.width + a.eps);
  auto keep_row = [&]() {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = tid + i * kNormThreads;
      if (c >= nv) continue;
      if (a.x_out) store4(a.x_out + (size_t)t * a.ldx + c * 4, x[i]);
      store4(static_cast<T*>(a.out) + (size_t)t * a.ldx + c * 4, x[i]);
    }
  };
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    x[i] = make_float4(x[i].x * r * g[i].x, x[i].y * r * g[i].y, x[i].z * r * g[i].z, x[i].w * r * g[i].w);
    const int c = tid + i * kNormThreads;
    if (ROUTER && c < nv) store4(row_x + c * 4, x[i]);
  }
  if (!ROUTER) {
    keep_row();
    return;
  }
  __syncthreads();
  auto cluster = cooperative_groups::this_cluster();
  float* z = cluster.map_shared_rank(row_x + a.ldx, 0);  // the logits meet in the first CTA
  const int warp = tid >> 5, lane = tid & 31, step = parts * (kNormThreads / 32);
  constexpr int kAtOnce = 4;
  for (int e0 = part * (kNormThreads / 32) + warp; e0 < a.router.experts; e0 += step * kAtOnce) {
    float s[kAtOnce] = {};
#pragma unroll 4
    for (int c = lane * 8; c < a.ldx; c += 256) {
      const float4 u = *reinterpret_cast<const float4*>(row_x + c), v = *reinterpret_cast<const float4*>(row_x + c + 4);
#pragma unroll
      for (int j = 0; j < kAtOnce; ++j) {
        const int e = min(e0 + j * step, a.router.experts - 1);
        s[j] += dot8(__ldg(reinterpret_cast<const uint4*>(a.router.w + (size_t)e * a.router.ldw + c)), u, v);
      }
    }
#pragma unroll
    for (int j = 0; j < kAtOnce; ++j) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s[j] += __shfl_xor_sync(0xffffffffu, s[j], o);
      const int e = e0 + j * step;
      if (lane == 0 && e < a.router.experts) z[e] = s[j] + a.router.b[e];
    }
  }
  cluster.sync();  // also: every CTA has read the row, which x_out may overwrite
  if (part) return;
  keep_row();
  if (warp == 0) choose_experts(row_x + a.ldx, a.router, t, lane);
}

// The same for many rows, a warp per row.
template <class T, int NVW>
__global__ void __launch_bounds__(kNormThreads) lm_post_norm_rows_kernel(PostNormArgs a) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int lane = threadIdx.x & 31, nv = a.ldx >> 2, t = blockIdx.x * (kNormThreads / 32) + (threadIdx.x >> 5);
  if (t >= a.rows) return;
  float4 x[NVW];
  if (a.delta.p) {
    warp_delta<NVW>(a.delta, t, lane, nv, x);
  } else {
#pragma unroll
    for (int i = 0; i < NVW; ++i) x[i] = make_float4(0, 0, 0, 0);
  }
  const float4* xr = reinterpret_cast<const float4*>(a.x_in + (size_t)t * a.ldx);
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NVW; ++i) {
    const int c = lane + i * 32;
    if (c < nv) x[i] = fma4(a.alpha, xr[c], x[i]);
    ss += dot4(x[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float r = 1.0f / sqrtf(ss / (float)a.width + a.eps);
#pragma unroll
  for (int i = 0; i < NVW; ++i) {
    const int c = lane + i * 32;
    if (c >= nv) continue;
    const float4 g = __ldg(reinterpret_cast<const float4*>(a.gain) + c);
    const float4 y = make_float4(x[i].x * r * g.x, x[i].y * r * g.y, x[i].z * r * g.z, x[i].w * r * g.w);
    if (a.x_out) store4(a.x_out + (size_t)t * a.ldx + c * 4, y);
    store4(static_cast<T*>(a.out) + (size_t)t * a.ldx + c * 4, y);
  }
}

constexpr int kFusedRouterRows = 2 * kSms;

template <class T, int NV>
cudaError_t launch_post_norm_nv(cudaStream_t s, const PostNormArgs& a) {
  if (!a.router.w) return launch_pdl(lm_post_norm_kernel<T, NV, false>, dim3(a.rows), dim3(kNormThreads), 0, s, a);
  int parts = 8;
  while (parts > 1 && (a.rows * parts > 2 * kSms || a.router.experts < parts * (kNormThreads / 32))) parts /= 2;
  const size_t smem = (size_t)(a.ldx + a.router.experts) * sizeof(float);
  return launch_pdl_cluster(lm_post_norm_kernel<T, NV, true>, dim3(a.rows, parts), dim3(kNormThreads), dim3(1, parts, 1), smem, s, a);
}
template <class T>
cudaError_t launch_post_norm_t(cudaStream_t s, const PostNormArgs& a) {
  if (a.rows > 16 * kSms && !a.gather && !a.router.w && a.ldx <= 4096) {
    const int w = (a.ldx / 4 + 31) / 32;
    const dim3 grid((a.rows + kNormThreads / 32 - 1) / (kNormThreads / 32));
    if (w <= 8) return launch_pdl(lm_post_norm_rows_kernel<T, 8>, grid, dim3(kNormThreads), 0, s, a);
    if (w <= 16) return launch_pdl(lm_post_norm_rows_kernel<T, 16>, grid, dim3(kNormThreads), 0, s, a);
    return launch_pdl(lm_post_norm_rows_kernel<T, 32>, grid, dim3(kNormThreads), 0, s, a);
  }
  const int per = (a.ldx / 4 + kNormThreads - 1) / kNormThreads;
  if (per <= 1) return launch_post_norm_nv<T, 1>(s, a);
  if (per <= 2) return launch_post_norm_nv<T, 2>(s, a);
  if (per <= 4) return launch_post_norm_nv<T, 4>(s, a);
  if (per <= 8) return launch_post_norm_nv<T, 8>(s, a);
  return cudaErrorInvalidValue;
}

template <class T>
__global__ void lm_embed_kernel(const int* __restrict__ tokens, const __nv_bfloat16* __restrict__ table, int width, int ldx,
                                float* __restrict__ x, T* __restrict__ h, int* __restrict__ zero, int n_zero) {
  pdl_launch_dependents();
  pdl_wait_prior();
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n_zero; i += gridDim.x * blockDim.x) zero[i] = 0;
  const __nv_bfloat16* src = table + (size_t)tokens[blockIdx.x] * width;
  float* dst = x + (size_t)blockIdx.x * ldx;
  T* hd = h ? h + (size_t)blockIdx.x * ldx : nullptr;
  int k0 = 0;
  if ((width & 7) == 0) {
    k0 = width;
    for (int k = threadIdx.x * 8; k < width; k += blockDim.x * 8) {
      const uint4 p = *reinterpret_cast<const uint4*>(src + k);
      const uint32_t w[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float4 v = make_float4(__uint_as_float(w[2 * i] << 16), __uint_as_float(w[2 * i] & 0xffff0000u),
                                     __uint_as_float(w[2 * i + 1] << 16), __uint_as_float(w[2 * i + 1] & 0xffff0000u));
        store4(dst + k + 4 * i, v);
        if (hd) store4(hd + k + 4 * i, v);
      }
    }
  }
  for (int k = k0 + threadIdx.x; k < ldx; k += blockDim.x) {
    const float v = k < width ? __bfloat162float(src[k]) : 0.0f;
    dst[k] = v;
    if (hd) hd[k] = static_cast<T>(v);  // exact: the table is bf16
  }
}

// Rows of a decode step: one token per slot, from the slots' own state.
__global__ void lm_decode_prep_kernel(int n, const int* __restrict__ slots, const int* __restrict__ pos, const int* __restrict__ token,
                                      const int* __restrict__ flip, int2* __restrict__ row_sp, int* __restrict__ row_token,
                                      Entry* __restrict__ entries, int* __restrict__ row_entry) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= n) return;
  const int slot = slots[b], p = pos[slot];
  row_sp[b] = make_int2(slot, p);
  row_token[b] = token[slot];
  entries[b] = Entry{slot, p, b, 1, flip[slot]};
  row_entry[b] = b;
}

// The largest logit of each of gridDim.x ranges of the vocabulary (lowest index on ties); gridDim.y rows.
__global__ void __launch_bounds__(256) lm_argmax_kernel(const float* __restrict__ logits, int vocab, float2* __restrict__ best) {
  __shared__ float sv[8];
  __shared__ int si[8];
  pdl_launch_dependents();
  pdl_wait_prior();
  const float* row = logits + (size_t)blockIdx.y * vocab;
  float bv = -3.402823466e+38f;
  int bi = 0x7fffffff;
  for (int i = blockIdx.x * 256 + threadIdx.x; i < vocab; i += gridDim.x * 256)
    if (row[i] > bv) bv = row[i], bi = i;
  auto merge = [&](float ov, int oi) {
    if (ov > bv || (ov == bv && oi < bi)) bv = ov, bi = oi;
  };
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    merge(ov, oi);
  }
  if ((threadIdx.x & 31) == 0) sv[threadIdx.x >> 5] = bv, si[threadIdx.x >> 5] = bi;
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int i = 1; i < 8; ++i) merge(sv[i], si[i]);
    best[(size_t)blockIdx.y * gridDim.x + blockIdx.x] = make_float2(bv, __int_as_float(bi));
  }
}

}  // namespace

cudaError_t launch_norm(cudaStream_t s, bool f32, const NormArgs& a) {
  return f32 ? launch_norm_t<float>(s, a) : launch_norm_t<__nv_bfloat16>(s, a);
}
bool fused_router(int rows) { return rows <= kFusedRouterRows; }
cudaError_t launch_post_norm(cudaStream_t s, bool f32, const PostNormArgs& a) {
  return f32 ? launch_post_norm_t<float>(s, a) : launch_post_norm_t<__nv_bfloat16>(s, a);
}
cudaError_t launch_embed(cudaStream_t s, bool f32, const int* tokens, const __nv_bfloat16* table, int width, int ldx, int rows, float* x,
                         void* h, int* zero, int n_zero) {
  if (f32) return launch_pdl(lm_embed_kernel<float>, dim3(rows), dim3(256), 0, s, tokens, table, width, ldx, x, static_cast<float*>(h), zero, n_zero);
  return launch_pdl(lm_embed_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, s, tokens, table, width, ldx, x, static_cast<__nv_bfloat16*>(h), zero,
                    n_zero);
}
cudaError_t launch_decode_prep(cudaStream_t s, int n, const int* slots, const int* pos, const int* token, const int* flip,
                               int2* row_sp, int* row_token, Entry* entries, int* row_entry) {
  return launch_pdl(lm_decode_prep_kernel, dim3((n + 127) / 128), dim3(128), 0, s, n, slots, pos, token, flip, row_sp, row_token,
                    entries, row_entry);
}
cudaError_t launch_argmax(cudaStream_t s, const float* logits, int rows, int vocab, int blocks, float2* best) {
  return launch_pdl(lm_argmax_kernel, dim3(blocks, rows), dim3(256), 0, s, logits, vocab, best);
}

}  // namespace lm
}  // namespace mllmb200
