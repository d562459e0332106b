// Gates of the decaying memories (decay_memory.cu, decay_memory_tc.cu), in fp32 with the accurate
// functions (these files are compiled without fast math).
#pragma once

namespace eb {

// log(1 + exp(x)) for any x
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// logarithm of the decay of a state-space head whose step is dt
__device__ __forceinline__ float log_decay_ssm(float a_log, float dt) { return -expf(a_log) * dt; }
// logarithm of sigmoid(z)^(1 / tau)
__device__ __forceinline__ float log_decay_gla(float z, float inv_tau) { return -softplus(-z) * inv_tau; }

}  // namespace eb
