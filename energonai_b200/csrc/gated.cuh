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
// The same for 16-bit results, with the rational approximation of erfc by Hastings (Abramowitz and Stegun 7.1.26, error at
// most 1.5e-7): erfc(x) = t (a1 + t (a2 + t (a3 + t (a4 + t a5)))) exp(-x^2), t = 1 / (1 + p x), x >= 0.
// The left tail is erfc itself, so nothing cancels there.
__device__ __forceinline__ float gelu_erf_fast(float z) {
  const float x = fabsf(z) * 0.70710678118654752f, t = __fdividef(1.f, fmaf(0.3275911f, x, 1.f));
  const float poly = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.061405429f, -1.453152027f), 1.421413741f), -0.284496736f), 0.254829592f);
  const float tail = 0.5f * z * poly * __expf(-x * x);
  return z > 0.f ? z - tail : tail;
}
__device__ __forceinline__ float unit_value(int unit, float gate, float up, float limit, float alpha) {
  return unit == EB_UNIT_GEGLU ? gelu_tanh_value(gate) * up : gated_value(gate, up, limit, alpha);
}

}  // namespace eb
