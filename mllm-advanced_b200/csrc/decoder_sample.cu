// Greedy sampling, shared by the decoders.
#include "device_common.cuh"

namespace mllmb200 {

// Greedy sampling from the per-CTA candidates of lm_head_f16_kernel, then the bookkeeping of a
// step (greedy = AutoLLM.hpp:70-105 of the reference project: scan in order, strict comparison, so the
// lowest index wins ties): the sampled token becomes the next input and is appended to the history (entry p = the
// token sampled after position p); the position advances.  One warp.
__global__ void sample_advance_kernel(const float2* __restrict__ best, int count, int* __restrict__ pos,
                                      int* __restrict__ token, int* __restrict__ next, int* __restrict__ history,
                                      int max_hist) {
  float bv = -3.402823466e+38f;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < count; i += 32) {
    const float2 c = best[i];
    const int ci = __float_as_int(c.y);
    if (c.x > bv || (c.x == bv && ci < bi)) {
      bv = c.x;
      bi = ci;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) {
      bv = ov;
      bi = oi;
    }
  }
  if (threadIdx.x == 0) {
    const int p = *pos;
    *next = bi;
    *token = bi;
    if (p < max_hist) history[p] = bi;
    *pos = p + 1;
  }
}

// Greedy sampling and bookkeeping of a step for every sequence (one warp each): sample_advance_kernel per row.
// slot_of: the sequence a row belongs to (nullptr: row r = sequence r); flip: a bit per sequence toggled by the step.
__global__ void sample_advance_batched_kernel(const float2* __restrict__ best, int count, int* __restrict__ pos,
                                              int* __restrict__ token, int* __restrict__ history, int max_hist,
                                              const int* __restrict__ slot_of, int* __restrict__ flip) {
  pdl_launch_dependents();
  pdl_wait_prior();
  const int seq = slot_of ? slot_of[blockIdx.x] : blockIdx.x;
  best += (size_t)blockIdx.x * count;
  float bv = -3.402823466e+38f;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < count; i += 32) {
    const float2 c = best[i];
    const int ci = __float_as_int(c.y);
    if (c.x > bv || (c.x == bv && ci < bi)) {
      bv = c.x;
      bi = ci;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > bv || (ov == bv && oi < bi)) {
      bv = ov;
      bi = oi;
    }
  }
  if (threadIdx.x == 0) {
    const int p = pos[seq];
    token[seq] = bi;
    if (p < max_hist) history[(size_t)seq * max_hist + p] = bi;
    pos[seq] = p + 1;
    if (flip) flip[seq] ^= 1;
  }
}

}  // namespace mllmb200
