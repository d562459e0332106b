// Gates of the matrix memory (matrix_memory.cu, matrix_memory_tc.cu), in fp32 with the accurate
// functions (these files are compiled without fast math).
#pragma once

namespace eb {

__device__ __forceinline__ float soft_cap(float a, float cap) { return cap * tanhf(a / cap); }
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_input_gate(float a, float bias, float cap) { return soft_cap(a + bias, cap); }
__device__ __forceinline__ float log_forget_gate(float a, float bias, float cap) { return log_sigmoid(soft_cap(a + bias, cap)); }

constexpr float kMemoryDenomEps = 1e-6f;

}  // namespace eb
