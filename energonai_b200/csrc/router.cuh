// The selection step of a mixture-of-experts router, by one warp.
#pragma once

#include <cfloat>

#include "common.cuh"

namespace eb {

constexpr int kMaxExperts = 4096;

// z[experts] (shared memory, overwritten): router logits of one token.  The scores are the
// softmax over ALL experts in fp32; the `top` largest are chosen (the lowest index among equals)
// and keep their scores as they are (not renormalised).  With `counts`, every choice also takes a
// ticket of its expert: ranks[k] = its place among the rows the expert gets.
__device__ __forceinline__ void route_warp(float *z, int experts, int top, int *idx, float *weights, int *counts, int *ranks) {
  const int lane = threadIdx.x & 31;
  float m = -FLT_MAX;
  for (int e = lane; e < experts; e += 32) m = fmaxf(m, z[e]);
  m = warp_max(m);
  float s = 0.f;
  for (int e = lane; e < experts; e += 32) s += expf(z[e] - m);
  const float inv = 1.f / warp_sum(s);
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < experts; e += 32) {
      const float v = z[e];
      if (v > best) { best = v; bi = e; }          // a lane walks its experts in rising order
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if (bi >= experts) bi = 0;                     // logits that are not numbers: any valid expert
    if (lane == 0) {
      idx[k] = bi;
      weights[k] = expf(best - m) * inv;
      z[bi] = -INFINITY;
      if (counts) ranks[k] = atomicAdd(counts + bi, 1);
    }
    __syncwarp();
  }
}

}  // namespace eb
