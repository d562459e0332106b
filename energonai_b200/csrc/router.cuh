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

constexpr int kRankChoices = 128;

// How a router chooses beyond the plain softmax scores.
struct RouterRule {
  const float *correction = nullptr;   // [choices] added to the scores for the choice alone, or null
  int groups = 1, keep = 1;            // equal groups of neighbours; only the best `keep` (by their largest choice score) are open
  int real = 0;                        // choices below this are experts with rows, the others stand for the input itself
};

__host__ __device__ inline int rule_floats(int choices, const RouterRule &r) { return 2 * choices + 2 * r.groups; }

inline int make_rule(const char *name, int choices, int experts, int top, const float *correction, int groups, int keep, RouterRule *r) {
  if (choices <= 0 || choices > kMaxExperts || experts < 0 || experts > choices) return fail(EB_EINVAL, "%s: bad router (%d choices, %d experts)", name, choices, experts);
  if (groups <= 0 || keep <= 0 || keep > groups || choices % groups != 0) return fail(EB_EINVAL, "%s: %d choices in %d groups of which %d are kept", name, choices, groups, keep);
  if (top <= 0 || top > choices / groups * keep) return fail(EB_EINVAL, "%s: top %d of %d open choices", name, top, choices / groups * keep);
  r->correction = correction;
  r->groups = groups;
  r->keep = keep;
  r->real = experts;
  return EB_OK;
}

// The largest of v[0..n) that is above -inf, and its index (the lowest among equals; n or more if there is none).
__device__ __forceinline__ void warp_argmax(const float *v, int n, float &best, int &bi) {
  best = -INFINITY;
  bi = 0x7fffffff;
  for (int e = threadIdx.x & 31; e < n; e += 32) {
    const float x = v[e];
    if (x > best) { best = x; bi = e; }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
  }
}

// route_warp with a rule; z has room for rule_floats() numbers.  The `top` choices with the largest
// score + correction among the open groups are taken; their weights are their scores, divided by
// their sum (+ 1e-20).  RANKS: up to kRankChoices choices each one's rank is counted, which takes a warp by itself less
// time than picking one after the other (and many warps together more).
template <bool RANKS>
__device__ __forceinline__ void route_warp_rule(float *z, int choices, int top, const RouterRule &rule, int *idx, float *weights, int *counts, int *ranks) {
  const int lane = threadIdx.x & 31;
  float *c = z + choices, *gs = c + choices, *open = gs + rule.groups;
  float m = -FLT_MAX;
  for (int e = lane; e < choices; e += 32) m = fmaxf(m, z[e]);
  m = warp_max(m);
  float s = 0.f;
  for (int e = lane; e < choices; e += 32) s += expf(z[e] - m);
  const float inv = 1.f / warp_sum(s);
  for (int e = lane; e < choices; e += 32) {
    const float sc = expf(z[e] - m) * inv;
    z[e] = sc;
    c[e] = sc + (rule.correction ? rule.correction[e] : 0.f);
  }
  __syncwarp();
  if (rule.keep < rule.groups) {
    const int per = choices / rule.groups;
    if (rule.groups <= 32) {                         // lane = group: its rank among them
      float mine = -INFINITY;
      if (lane < rule.groups)
        for (int e = 0; e < per; ++e) mine = fmaxf(mine, c[lane * per + e]);
      int before = 0;
      for (int g = 0; g < rule.groups; ++g) {
        const float other = __shfl_sync(0xffffffffu, mine, g);
        before += other > mine || (other == mine && g < lane);
      }
      if (lane < rule.groups) open[lane] = before < rule.keep ? 1.f : 0.f;
      __syncwarp();
    } else {
      for (int g = lane; g < rule.groups; g += 32) {
        float b = -INFINITY;
        for (int e = 0; e < per; ++e) b = fmaxf(b, c[g * per + e]);
        gs[g] = b;
        open[g] = 0.f;
      }
      __syncwarp();
      for (int k = 0; k < rule.keep; ++k) {
        float best;
        int bi;
        warp_argmax(gs, rule.groups, best, bi);
        if (lane == 0 && bi < rule.groups) { gs[bi] = -INFINITY; open[bi] = 1.f; }
        __syncwarp();
      }
    }
    for (int e = lane; e < choices; e += 32)
      if (open[e / per] == 0.f) c[e] = -INFINITY;
    __syncwarp();
  }
  float total = 0.f;
  if (RANKS && choices <= kRankChoices) {
    // every choice's rank among all; the first `top` are taken.  (Logits that are not numbers leave places of the list
    // untaken: any valid choices stand there.)
    for (int k = lane; k < top; k += 32) {
      idx[k] = k;
      weights[k] = 0.f;
      if (counts) ranks[k] = -1;
    }
    __syncwarp();
    float mine[kRankChoices / 32];
    int before[kRankChoices / 32];
#pragma unroll
    for (int i = 0; i < kRankChoices / 32; ++i) {
      mine[i] = lane + 32 * i < choices ? c[lane + 32 * i] : -INFINITY;
      before[i] = 0;
    }
    for (int e = 0; e < choices; ++e) {
      const float other = c[e];
#pragma unroll
      for (int i = 0; i < kRankChoices / 32; ++i)
        if (32 * i < choices) before[i] += other > mine[i] || (other == mine[i] && e < lane + 32 * i);
    }
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < kRankChoices / 32; ++i)
      if (lane + 32 * i < choices && before[i] < top) sum += z[lane + 32 * i];
    total = warp_sum(sum) + 1e-20f;
#pragma unroll
    for (int i = 0; i < kRankChoices / 32; ++i) {
      const int e = lane + 32 * i, k = before[i];
      if (e >= choices || k >= top) continue;
      idx[k] = e;
      weights[k] = z[e] / total;
      if (counts) ranks[k] = e < rule.real ? atomicAdd(counts + e * kCountStride, 1) : -1;
    }
    return;
  }
  for (int k0 = 0; k0 < top; k0 += 32) {
    int mine = 0;                                    // lane k: choice k0 + k
    float score = 0.f;
    const int n = min(32, top - k0);
    for (int k = 0; k < n; ++k) {
      float best;
      int bi;
      warp_argmax(c, choices, best, bi);
      if (bi >= choices) bi = 0;                     // logits that are not numbers: any valid choice
      if (lane == k) { mine = bi; score = z[bi]; }
      __syncwarp();
      if (lane == 0) c[bi] = -INFINITY;
      __syncwarp();
    }
    total += warp_sum(score);
    if (lane < n) {
      idx[k0 + lane] = mine;
      weights[k0 + lane] = score;
      if (counts) ranks[k0 + lane] = mine < rule.real ? atomicAdd(counts + mine * kCountStride, 1) : -1;
    }
  }
  for (int k = lane; k < top; k += 32) weights[k] = weights[k] / (total + 1e-20f);       // (this lane's own entries)
}

}  // namespace eb
