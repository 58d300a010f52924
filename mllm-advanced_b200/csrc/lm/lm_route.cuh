// The choice of experts from a row's router logits, shared by the norm that makes them itself and the kernel behind a
// router linear.
#pragma once
#include "lm_state.h"

namespace mllmb200 {
namespace lm {

// eight bf16 weights times eight fp32 numbers
__device__ __forceinline__ float dot8(const uint4& p, const float4& u, const float4& v) {
  float s = __uint_as_float(p.x << 16) * u.x;
  s = fmaf(__uint_as_float(p.x & 0xffff0000u), u.y, s);
  s = fmaf(__uint_as_float(p.y << 16), u.z, s);
  s = fmaf(__uint_as_float(p.y & 0xffff0000u), u.w, s);
  s = fmaf(__uint_as_float(p.z << 16), v.x, s);
  s = fmaf(__uint_as_float(p.z & 0xffff0000u), v.y, s);
  s = fmaf(__uint_as_float(p.w << 16), v.z, s);
  return fmaf(__uint_as_float(p.w & 0xffff0000u), v.w, s);
}

// One warp: the `top` largest of z[0, experts) in shared memory (lowest index on ties; z is used up), softmax over them.
__device__ __forceinline__ void choose_experts(float* z, const RouterArgs& a, int row, int lane) {
  constexpr float kUsed = -3.402823466e+38f;
  float mine = 0.0f, first = 0.0f;
  int mine_e = 0;
  // a lane's own candidate is looked for again only after it was chosen
  float own = kUsed;
  int own_e = 0x7fffffff;
  auto look = [&]() {
    own = kUsed;
    own_e = 0x7fffffff;
    for (int e = lane; e < a.experts; e += 32)
      if (z[e] > own) own = z[e], own_e = e;
  };
  look();
  for (int k = 0; k < a.top; ++k) {
    float bv = own;
    int be = own_e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) bv = ov, be = oe;
    }
    be = min(be, a.experts - 1);  // logits that are not numbers
    if (k == 0) first = bv;
    if (lane == k) mine = bv, mine_e = be;
    if (be == own_e) {
      z[be] = kUsed;
      look();
    }
  }
  const float p = lane < a.top ? expf(mine - first) : 0.0f;
  float sum = p;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  if (lane < a.top) {
    const size_t at = (size_t)row * a.top + lane;
    a.sel[at] = mine_e;
    a.weight[at] = p / sum;
    if (a.rank) a.rank[at] = atomicAdd(a.count + mine_e, 1);
  }
}

}  // namespace lm
}  // namespace mllmb200
