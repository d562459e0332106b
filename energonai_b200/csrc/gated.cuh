// The clamped gated unit of an expert, in fp32:
//   g = min(gate, limit), u = clamp(up, -limit, limit);  value = g * sigmoid(alpha * g) * (u + 1)
#pragma once

namespace eb {

__device__ __forceinline__ float gated_value(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

}  // namespace eb
