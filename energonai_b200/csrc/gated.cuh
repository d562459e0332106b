// Units of a feed-forward, in fp32 (EB_UNIT_*):
//   clamped   g = min(gate, limit), u = clamp(up, -limit, limit);  g * sigmoid(alpha * g) * (u + 1)
//   geglu     gelu_tanh(gate) * up
//   gelu      gelu(up), the erf form (no gate)
#pragma once

namespace eb {

__device__ __forceinline__ float gated_value(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
// 0.5 z (1 + tanh(t)) = z / (1 + exp(-2 t)): no cancellation where tanh is near -1
__device__ __forceinline__ float gelu_tanh_value(float z) {
  const float t = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
  return z / (1.f + expf(-2.f * t));
}
__device__ __forceinline__ float gelu_erf_value(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
__device__ __forceinline__ float unit_value(int unit, float gate, float up, float limit, float alpha) {
  return unit == EB_UNIT_GEGLU ? gelu_tanh_value(gate) * up : gated_value(gate, up, limit, alpha);
}

}  // namespace eb
