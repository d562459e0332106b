// The selection step of a mixture-of-experts router, by one warp.
#pragma once

#include <cfloat>

#include "common.cuh"

namespace eb {

constexpr int kMaxExperts = 4096;
constexpr int kCountStride = 32;       // ints between two experts' counters: tickets of one cache line are handed out one after the other

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
  for (int k0 = 0; k0 < top; k0 += 32) {
    int mine = 0;                                    // lane k: choice k0 + k
    float score = 0.f;
    const int n = min(32, top - k0);
    for (int k = 0; k < n; ++k) {
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
      if (lane == k) { mine = bi; score = expf(best - m) * inv; }
      if (lane == 0) z[bi] = -INFINITY;
      __syncwarp();
    }
    if (lane < n) {                                  // all choices' tickets and stores together
      idx[k0 + lane] = mine;
      weights[k0 + lane] = score;
      if (counts) ranks[k0 + lane] = atomicAdd(counts + mine * kCountStride, 1);
    }
  }
}

}  // namespace eb
