// Gates of the decaying memories (decay_memory.cu, decay_memory_tc.cu), in fp32 with the accurate
// functions (these files are compiled without fast math).
#pragma once

namespace eb {

// log(1 + e) for 0 <= e <= 1 as 2 artanh(e / (2 + e)): the argument is at most 1/3, seven terms of the series leave 2e-9
__device__ __forceinline__ float log1p_unit(float e) {
  const float s = __fdividef(e, 2.f + e), s2 = s * s;
  float r = 1.f / 13.f;
  r = fmaf(r, s2, 1.f / 11.f);
  r = fmaf(r, s2, 1.f / 9.f);
  r = fmaf(r, s2, 1.f / 7.f);
  r = fmaf(r, s2, 1.f / 5.f);
  r = fmaf(r, s2, 1.f / 3.f);
  return 2.f * fmaf(r * s2, s, s);
}
// log(1 + exp(x)) for any x
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1p_unit(expf(-fabsf(x))); }
// logarithm of the decay of a state-space head whose step is dt
__device__ __forceinline__ float log_decay_ssm(float a_log, float dt) { return -expf(a_log) * dt; }
// logarithm of sigmoid(z)^(1 / tau)
__device__ __forceinline__ float log_decay_gla(float z, float inv_tau) { return -softplus(-z) * inv_tau; }

}  // namespace eb
