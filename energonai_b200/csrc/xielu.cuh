// The xIELU activation, in fp32:
//   z > 0:  up * z^2 + z/2          z <= 0:  down * (exp(z) - 1 - z) + z/2
// with up = softplus(p) and down = 1/2 + softplus(q) of the layer's two numbers.
#pragma once

namespace eb {

// for 16-bit results (the cancellation in exp(z) - 1 near zero is below their resolution); no branch:
// each half vanishes on the other side of zero
__device__ __forceinline__ float xielu_fast(float z, float up, float down) {
  const float pos = fmaxf(z, 0.f), neg = fminf(z, 0.f);
  return fmaf(up * pos, pos, fmaf(down, (__expf(neg) - 1.f) - neg, 0.5f * z));
}
__device__ __forceinline__ float xielu_exact(float z, float up, float down) {
  return 0.5f * z + (z > 0.f ? up * z * z : down * (expm1f(fminf(z, 0.f)) - z));
}

}  // namespace eb
