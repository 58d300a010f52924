// Retention: linear attention with a fixed decay per head, S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, each head's
// o over its root mean square, times silu of a gate.  q and k are rotated (half-split layout, first rot_dims
// coordinates) and k is multiplied by dim^-1/2.  Everything after the projections is fp32: the rotated q and k, the
// states, the decays (powers tabulated in double precision and rounded once) and all products.
//   * one token per sequence: lm_ret_decode_kernel updates the state in place.
//   * prompts and portions: chunks of kChunk tokens, cut from the portion's own start.  lm_ret_chunk_kernel forms every
//     chunk's own contribution to the state, lm_ret_scan_kernel chains them (leaving the state in front of every chunk),
//     lm_ret_output_kernel combines the part inside the chunk with the state in front of it, and applies norm and gate.
//     Both rotate as they load.
#include <algorithm>

#include "../device_common.cuh"
#include "lm_state.h"

namespace mllmb200 {
namespace lm {
namespace {

constexpr int kThreads = 256, kPad = kChunk + 4, kStateRows = 16;
constexpr int kRows = 8, kTileThreads = kChunk / kRows * 16;  // of the tiled products: rows per thread, threads per 64 rows

template <class T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// angles in double precision, one rounding of cos and sin
__global__ void lm_rope_table_kernel(float* cos_t, float* sin_t, int max_pos, int half, double base) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= max_pos * half) return;
  const int p = i / half, d = i - p * half;
  const double a = (double)p * pow(base, -(double)d / (double)half);
  double s, c;
  sincos(a, &s, &c);
  cos_t[i] = (float)c;
  sin_t[i] = (float)s;
}

// coordinate d of a rotated head at position pos; x points at the head
__device__ __forceinline__ float rotated(const float* x, int d, int rot_dims, const float* cos_r, const float* sin_r) {
  if (d >= rot_dims) return x[d];
  const int half = rot_dims >> 1;
  const int i = d < half ? d : d - half;
  const float u = x[i], v = x[i + half], c = cos_r[i], s = sin_r[i];
  return d < half ? u * c - v * s : v * c + u * s;
}

template <class T>
__global__ void __launch_bounds__(kThreads) lm_ret_decode_kernel(RetentionArgs a) {
  extern __shared__ __align__(16) float dec_smem[];
  __shared__ float wsum[kThreads / 32];
  float *sq = dec_smem, *sk = sq + a.dimp, *sv = sk + a.dimp, *red = sv + a.vdimp;
  pdl_launch_dependents();
  pdl_wait_prior();
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
  const int2 sp = a.row_sp[row];
  const float* qr = a.qkvg + (size_t)row * a.ld + h * a.dimp;
  const float* kr = qr + a.heads * a.dimp;
  const float* vr = a.qkvg + (size_t)row * a.ld + 2 * a.heads * a.dimp + h * a.vdimp;
  const float* gr = vr + a.heads * a.vdimp;
  const int half = a.rot_dims >> 1;
  const float *cr = a.cos_t + (size_t)sp.y * half, *sr = a.sin_t + (size_t)sp.y * half;
  const float decay = a.decay[h * (kChunk + 1) + 1], kscale = 1.0f / sqrtf((float)a.dim);
  const int vl_n = a.vdimp >> 2, rg_n = kThreads / vl_n, vl = tid % vl_n, rg = tid / vl_n;
  float* st = a.state + ((size_t)sp.x * a.heads + h) * a.dimp * a.vdimp + vl * 4;
  const bool fresh = sp.y == 0;
  for (int d = tid; d < a.dimp; d += kThreads) {
    sq[d] = rotated(qr, d, a.rot_dims, cr, sr);
    sk[d] = rotated(kr, d, a.rot_dims, cr, sr) * kscale;
  }
  for (int d = tid; d < a.vdimp; d += kThreads) sv[d] = vr[d];
  __syncthreads();
  if (rg < rg_n) {
    const float4 v = *reinterpret_cast<const float4*>(sv + vl * 4);
    float4 o = make_float4(0, 0, 0, 0);
    constexpr int U = 8;
    for (int r0 = rg; r0 < a.dim; r0 += U * rg_n) {
      float4 s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * rg_n;
        s[u] = !fresh && r < a.dim ? *reinterpret_cast<const float4*>(st + (size_t)r * a.vdimp) : make_float4(0, 0, 0, 0);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * rg_n;
        if (r >= a.dim) break;
        const float k = sk[r], q = sq[r];
        s[u] = make_float4(fmaf(decay, s[u].x, k * v.x), fmaf(decay, s[u].y, k * v.y), fmaf(decay, s[u].z, k * v.z),
                           fmaf(decay, s[u].w, k * v.w));
        *reinterpret_cast<float4*>(st + (size_t)r * a.vdimp) = s[u];
        o = make_float4(fmaf(q, s[u].x, o.x), fmaf(q, s[u].y, o.y), fmaf(q, s[u].z, o.z), fmaf(q, s[u].w, o.w));
      }
    }
    *reinterpret_cast<float4*>(red + (size_t)rg * a.vdimp + vl * 4) = o;
  }
  __syncthreads();
  float o = 0.0f;
  if (tid < a.vdimp)
    for (int g = 0; g < rg_n; ++g) o += red[(size_t)g * a.vdimp + tid];
  float ss = o * o;
#pragma unroll
  for (int i = 16; i > 0; i >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, i);
  if ((tid & 31) == 0) wsum[tid >> 5] = ss;
  __syncthreads();
  ss = 0.0f;
  for (int i = 0; i < kThreads / 32; ++i) ss += wsum[i];
  if (tid < a.vdimp)
    static_cast<T*>(a.out)[(size_t)row * a.ldo + h * a.vdimp + tid] =
        from_f32<T>(o / sqrtf(ss / (float)a.vdim + a.eps) * silu(gr[tid]));
}

// coordinates d .. d + 3 of a rotated head (rot_dims / 2 a multiple of 4)
__device__ __forceinline__ float4 rotated4(const float* x, int d, int rot_dims, const float* cos_r, const float* sin_r) {
  const float4 own = *reinterpret_cast<const float4*>(x + d);
  if (d >= rot_dims) return own;
  const int half = rot_dims >> 1, i = d < half ? d : d - half;
  const float4 other = *reinterpret_cast<const float4*>(x + (d < half ? d + half : i));
  const float4 c = *reinterpret_cast<const float4*>(cos_r + i), sn = *reinterpret_cast<const float4*>(sin_r + i);
  const float sg = d < half ? -1.0f : 1.0f;
  return make_float4(own.x * c.x + sg * (other.x * sn.x), own.y * c.y + sg * (other.y * sn.y), own.z * c.z + sg * (other.z * sn.z),
                     own.w * c.w + sg * (other.w * sn.w));
}

// the same for any rot_dims; coordinates past dim are the padding (zero)
__device__ __forceinline__ float4 rotated_any(const float* x, int d, const RetentionArgs& a, int pos) {
  const int half = a.rot_dims >> 1;
  const float *cr = a.cos_t + (size_t)pos * half, *sr = a.sin_t + (size_t)pos * half;
  if ((a.rot_dims & 7) == 0) return rotated4(x, d, a.rot_dims, cr, sr);
  return make_float4(rotated(x, d, a.rot_dims, cr, sr), rotated(x, d + 1, a.rot_dims, cr, sr), rotated(x, d + 2, a.rot_dims, cr, sr),
                     rotated(x, d + 3, a.rot_dims, cr, sr));
}

// Two fp32 products and sums per instruction.
__device__ __forceinline__ void fma2(uint64_t& acc, uint64_t a, uint64_t b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(acc) : "l"(a), "l"(b));
}
__device__ __forceinline__ uint64_t both(float v) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ float2 halves(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}

// A kRows x (4 NC) tile per thread: rows kRows ty .., columns 4 tx + 64 i .. + 3, two columns per accumulator.
template <int NC>
struct Tile {
  uint64_t v[kRows][2 * NC];
  __device__ __forceinline__ void clear() {
#pragma unroll
    for (int r = 0; r < kRows; ++r)
#pragma unroll
      for (int i = 0; i < 2 * NC; ++i) v[r][i] = 0;
  }
  // += sum over k of a(k, row) * B[k][column], in shared memory; a(k, row) = A[row][k] (KMAJOR; n a multiple of 4) or
  // A[k][row].  Columns past `cols` repeat column 0: they hold something, and nobody stores it.
  template <bool KMAJOR>
  __device__ __forceinline__ void fma(const float* A, int lda, const float* B, int ldb, int n, int ty, int tx, int cols) {
    constexpr int kStep = KMAJOR ? 4 : 1;
    A += ty * kRows * (KMAJOR ? lda : 1);
    const float* b[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) b[i] = B + (tx * 4 + i * 64 < cols ? tx * 4 + i * 64 : 0);
#pragma unroll 2
    for (int k0 = 0; k0 < n; k0 += kStep) {
      float av[kRows][kStep];
      if (KMAJOR) {
#pragma unroll
        for (int r = 0; r < kRows; ++r) *reinterpret_cast<float4*>(av[r]) = *reinterpret_cast<const float4*>(A + r * lda + k0);
      } else {
#pragma unroll
        for (int r = 0; r < kRows; r += 4) {
          const float4 t = *reinterpret_cast<const float4*>(A + k0 * lda + r);
          av[r][0] = t.x, av[r + 1][0] = t.y, av[r + 2][0] = t.z, av[r + 3][0] = t.w;
        }
      }
#pragma unroll
      for (int kk = 0; kk < kStep; ++kk)
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const ulonglong2 bv = *reinterpret_cast<const ulonglong2*>(b[i] + (k0 + kk) * ldb);
#pragma unroll
          for (int r = 0; r < kRows; ++r) {
            fma2(v[r][2 * i], both(av[r][kk]), bv.x);
            fma2(v[r][2 * i + 1], both(av[r][kk]), bv.y);
          }
        }
    }
  }
  __device__ __forceinline__ void scale_row(int r, float f) {
#pragma unroll
    for (int i = 0; i < 2 * NC; ++i) {
      const float2 h = halves(v[r][i]);
      asm("mov.b64 %0, {%1, %2};" : "=l"(v[r][i]) : "f"(h.x * f), "f"(h.y * f));
    }
  }
  __device__ __forceinline__ float4 get(int r, int i) const {
    const float2 a = halves(v[r][2 * i]), b = halves(v[r][2 * i + 1]);
    return make_float4(a.x, a.y, b.x, b.y);
  }
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

struct ChunkPos {
  int row0, len, pos;  // first row, tokens, position of the first token
};
__device__ __forceinline__ ChunkPos chunk_pos(const RetentionArgs& a, int chunk) {
  const int2 c = a.chunks[chunk];
  const Entry e = a.entries[c.x];
  return {e.row0 + c.y, min(kChunk, e.count - c.y), e.pos0 + c.y};
}

// grid (chunks, heads, blocks of 64 state rows): sum over the chunk of decay^(len-1-j) k_j v_j^T
template <int NC>
__global__ void __launch_bounds__(kTileThreads) lm_ret_chunk_kernel(RetentionArgs a) {
  extern __shared__ __align__(16) float ck_smem[];
  float *sK = ck_smem, *sV = sK + kChunk * 64;  // [kChunk][64], [kChunk][vdimp]
  pdl_launch_dependents();
  pdl_wait_prior();
  const int chunk = blockIdx.x, h = blockIdx.y, d0 = blockIdx.z * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const ChunkPos p = chunk_pos(a, chunk);
  const float* pw = a.decay + h * (kChunk + 1);
  const float* kb = a.qkvg + (size_t)p.row0 * a.ld + (a.heads + h) * a.dimp;
  const float* vb = a.qkvg + (size_t)p.row0 * a.ld + 2 * a.heads * a.dimp + h * a.vdimp;
  const int nd = min(64, a.dimp - d0), v4 = a.vdimp / 4;
  const float kscale = 1.0f / sqrtf((float)a.dim);
  for (int i = tid; i < p.len * 16; i += kTileThreads) {
    const int j = i >> 4, c = (i & 15) * 4;
    float4 k = make_float4(0, 0, 0, 0);
    if (c < nd) k = rotated_any(kb + (size_t)j * a.ld, d0 + c, a, p.pos + j);
    const float f = pw[p.len - 1 - j] * kscale;
    *reinterpret_cast<float4*>(sK + j * 64 + c) = make_float4(k.x * f, k.y * f, k.z * f, k.w * f);
  }
  for (int i = tid; i < p.len * v4; i += kTileThreads) {
    const int j = i / v4, c = (i - j * v4) * 4;
    *reinterpret_cast<float4*>(sV + j * a.vdimp + c) = *reinterpret_cast<const float4*>(vb + (size_t)j * a.ld + c);
  }
  __syncthreads();
  Tile<NC> acc;
  acc.clear();
  acc.template fma<false>(sK, 64, sV, a.vdimp, p.len, ty, tx, a.vdimp);
  float* dst = a.chunk_state + ((size_t)chunk * a.heads + h) * a.dimp * a.vdimp;
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int d = d0 + ty * kRows + r;
    if (d >= a.dimp) break;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = tx * 4 + i * 64;
      if (c < a.vdimp) *reinterpret_cast<float4*>(dst + (size_t)d * a.vdimp + c) = acc.get(r, i);
    }
  }
}

// grid (blocks of 256 float4 of a state, heads, entries): chunk_state becomes the state in front of each chunk
__global__ void __launch_bounds__(kThreads) lm_ret_scan_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int i = blockIdx.x * kThreads + threadIdx.x, h = blockIdx.y;
  const size_t n4 = (size_t)a.dimp * a.vdimp / 4;
  if (i >= (int)n4) return;
  const Entry e = a.entries[blockIdx.z];
  const int2 ec = a.entry_chunks[blockIdx.z];
  float4* st = reinterpret_cast<float4*>(a.state) + ((size_t)e.slot * a.heads + h) * n4 + i;
  float4 s = e.pos0 == 0 ? make_float4(0, 0, 0, 0) : *st;
  float4* cs = reinterpret_cast<float4*>(a.chunk_state) + ((size_t)ec.x * a.heads + h) * n4 + i;
  const size_t step = (size_t)a.heads * n4;
  for (int c0 = 0; c0 < ec.y; c0 += 8) {
    float4 u[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < ec.y) u[j] = cs[(size_t)(c0 + j) * step];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j >= ec.y) break;
      const float f = a.decay[h * (kChunk + 1) + min(kChunk, e.count - (c0 + j) * kChunk)];
      cs[(size_t)(c0 + j) * step] = s;
      s = make_float4(fmaf(f, s.x, u[j].x), fmaf(f, s.y, u[j].y), fmaf(f, s.z, u[j].z), fmaf(f, s.w, u[j].w));
    }
  }
  *st = s;
}

size_t output_smem(const RetentionArgs& a) {
  const size_t rows = (size_t)kChunk * (a.dimp + 4);
  const size_t shared_part = std::max(rows, (size_t)kChunk * kPad + (size_t)2 * kStateRows * a.vdimp);
  return (rows + shared_part + (size_t)kChunk * a.vdimp) * 4;
}

// grid (chunks, heads)
template <class T, int NC>
__global__ void __launch_bounds__(kTileThreads, NC == 4 ? 1 : 2) lm_ret_output_kernel(RetentionArgs a) {
  extern __shared__ __align__(16) float out_smem[];
  const int ldq = a.dimp + 4;
  float* sQ = out_smem;                        // [kChunk][ldq]
  float* sV = sQ + (size_t)kChunk * ldq;       // [kChunk][vdimp]
  float* sK = sV + (size_t)kChunk * a.vdimp;   // [kChunk][ldq]; afterwards
  float* sA = sK;                              //   [kChunk][kPad]: decayed scores
  float* sS = sA + (size_t)kChunk * kPad;      //   [2][kStateRows][vdimp]: rows of the state
  pdl_launch_dependents();
  pdl_wait_prior();
  const int chunk = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const ChunkPos p = chunk_pos(a, chunk);
  const float* pw = a.decay + h * (kChunk + 1);
  const float* qb = a.qkvg + (size_t)p.row0 * a.ld + h * a.dimp;
  const float* kb = qb + a.heads * a.dimp;
  const float* vb = a.qkvg + (size_t)p.row0 * a.ld + 2 * a.heads * a.dimp + h * a.vdimp;
  const float* gb = vb + a.heads * a.vdimp;
  const int d4 = a.dimp / 4, v4 = a.vdimp / 4;
  const float kscale = 1.0f / sqrtf((float)a.dim);
  for (int i = tid; i < kChunk * v4; i += kTileThreads) {
    const int j = i / v4, c = (i - j * v4) * 4;
    if (j < p.len) cp_async16(sV + j * a.vdimp + c, vb + (size_t)j * a.ld + c);
    else *reinterpret_cast<float4*>(sV + j * a.vdimp + c) = make_float4(0, 0, 0, 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll 4
  for (int i = tid; i < kChunk * d4; i += kTileThreads) {
    const int j = i / d4, d = (i - j * d4) * 4;
    float4 q = make_float4(0, 0, 0, 0), k = q;
    if (j < p.len) {
      q = rotated_any(qb + (size_t)j * a.ld, d, a, p.pos + j);
      k = rotated_any(kb + (size_t)j * a.ld, d, a, p.pos + j);
    }
    *reinterpret_cast<float4*>(sQ + j * ldq + d) = q;
    *reinterpret_cast<float4*>(sK + j * ldq + d) = make_float4(k.x * kscale, k.y * kscale, k.z * kscale, k.w * kscale);
  }
  __syncthreads();
  const float* S = a.chunk_state + ((size_t)chunk * a.heads + h) * a.dimp * a.vdimp;
  auto fetch = [&](int d0) {  // kStateRows rows of the state; dimp is a multiple of them
    float* dst = sS + (size_t)((d0 / kStateRows) & 1) * kStateRows * a.vdimp;
    for (int i = tid; i < kStateRows * v4; i += kTileThreads) cp_async16(dst + 4 * i, S + (size_t)d0 * a.vdimp + 4 * i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  {  // scores of rows kRows ty .. and keys tx, tx + 16, ..; even and odd coordinates are summed side by side
    uint64_t s[kRows][4];
#pragma unroll
    for (int r = 0; r < kRows; ++r) s[r][0] = s[r][1] = s[r][2] = s[r][3] = 0;
#pragma unroll 2
    for (int d = 0; d < a.dimp; d += 4) {
      ulonglong2 kv[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) kv[c] = *reinterpret_cast<const ulonglong2*>(sK + (tx + 16 * c) * ldq + d);
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        const ulonglong2 qv = *reinterpret_cast<const ulonglong2*>(sQ + (ty * kRows + r) * ldq + d);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          fma2(s[r][c], qv.x, kv[c].x);
          fma2(s[r][c], qv.y, kv[c].y);
        }
      }
    }
    __syncthreads();  // k is no longer needed
    fetch(0);
#pragma unroll
    for (int r = 0; r < kRows; ++r)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int i = ty * kRows + r, j = tx + 16 * c;
        const float2 h = halves(s[r][c]);
        sA[i * kPad + j] = j <= i ? (h.x + h.y) * pw[i - j] : 0.0f;
      }
  }
  Tile<NC> acc;
  acc.clear();
  for (int d0 = 0; d0 < a.dimp; d0 += kStateRows) {
    if (d0 + kStateRows < a.dimp) {
      fetch(d0 + kStateRows);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    acc.template fma<true>(sQ + d0, ldq, sS + (size_t)((d0 / kStateRows) & 1) * kStateRows * a.vdimp, a.vdimp, kStateRows, ty, tx, a.vdimp);
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < kRows; ++r) acc.scale_row(r, pw[ty * kRows + r + 1]);
  acc.template fma<true>(sA, kPad, sV, a.vdimp, (ty / 2 + 1) * 2 * kRows, ty, tx, a.vdimp);
  T* out = static_cast<T*>(a.out);
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      if (tx * 4 + i * 64 >= a.vdimp) break;
      const float4 v = acc.get(r, i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const int j = ty * kRows + r;
    if (j >= p.len) continue;
    const float inv = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = tx * 4 + i * 64;
      if (c < a.vdimp) {
        const float4 g = *reinterpret_cast<const float4*>(gb + (size_t)j * a.ld + c), v = acc.get(r, i);
        store4(out + (size_t)(p.row0 + j) * a.ldo + h * a.vdimp + c,
               make_float4(v.x * inv * silu(g.x), v.y * inv * silu(g.y), v.z * inv * silu(g.z), v.w * inv * silu(g.w)));
      }
    }
  }
}

template <class T, int NC>
cudaError_t prefill_nc(cudaStream_t s, const RetentionArgs& a) {
  cudaError_t r = launch_pdl(lm_ret_chunk_kernel<NC>, dim3(a.n_chunks, a.heads, (a.dimp + 63) / 64), dim3(kTileThreads), (size_t)kChunk * (64 + a.vdimp) * 4, s, a);
  if (r == cudaSuccess) {
    const int n4 = a.dimp * a.vdimp / 4;
    r = launch_pdl(lm_ret_scan_kernel, dim3((n4 + kThreads - 1) / kThreads, a.heads, a.n_entries), dim3(kThreads), 0, s, a);
  }
  if (r == cudaSuccess) r = launch_pdl(lm_ret_output_kernel<T, NC>, dim3(a.n_chunks, a.heads), dim3(kTileThreads), output_smem(a), s, a);
  return r;
}
template <class T>
cudaError_t prefill_t(cudaStream_t s, const RetentionArgs& a) {
  return a.vdimp <= 64 ? prefill_nc<T, 1>(s, a) : a.vdimp <= 128 ? prefill_nc<T, 2>(s, a) : prefill_nc<T, 4>(s, a);
}

constexpr int kRetSmemMax = 220 * 1024;

}  // namespace

cudaError_t retention_configure() {
  cudaError_t r = cudaSuccess;
  auto set = [&](auto f) {
    if (r == cudaSuccess) r = cudaFuncSetAttribute(f, cudaFuncAttributeMaxDynamicSharedMemorySize, kRetSmemMax);
  };
  set(lm_ret_chunk_kernel<1>);
  set(lm_ret_chunk_kernel<2>);
  set(lm_ret_chunk_kernel<4>);
  set(lm_ret_output_kernel<float, 1>);
  set(lm_ret_output_kernel<float, 2>);
  set(lm_ret_output_kernel<float, 4>);
  set(lm_ret_output_kernel<__nv_bfloat16, 1>);
  set(lm_ret_output_kernel<__nv_bfloat16, 2>);
  set(lm_ret_output_kernel<__nv_bfloat16, 4>);
  return r;
}

cudaError_t launch_rope_table(cudaStream_t s, float* cos_t, float* sin_t, int max_pos, int dims, double base) {
  const int n = max_pos * (dims / 2);
  if (n > 0) lm_rope_table_kernel<<<(n + 255) / 256, 256, 0, s>>>(cos_t, sin_t, max_pos, dims / 2, base);
  return cudaGetLastError();
}

cudaError_t launch_retention_decode(cudaStream_t s, bool f32, const RetentionArgs& a) {
  const int rg = kThreads / (a.vdimp / 4);
  const size_t smem = ((size_t)2 * a.dimp + a.vdimp + (size_t)rg * a.vdimp) * 4;
  const dim3 grid(a.heads, a.rows);
  return f32 ? launch_pdl(lm_ret_decode_kernel<float>, grid, dim3(kThreads), smem, s, a)
             : launch_pdl(lm_ret_decode_kernel<__nv_bfloat16>, grid, dim3(kThreads), smem, s, a);
}
cudaError_t launch_retention_prefill(cudaStream_t s, bool f32, const RetentionArgs& a) {
  return f32 ? prefill_t<float>(s, a) : prefill_t<__nv_bfloat16>(s, a);
}

}  // namespace lm
}  // namespace mllmb200
