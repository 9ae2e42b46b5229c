// xIELU: for z > 0, ap z^2 + z / 2; for z <= 0, an (e^z - 1 - z) + z / 2. ap = softplus(p) and
// an = 1/2 + softplus(q) are computed once per layer on the host.
#pragma once

namespace rb {

__device__ __forceinline__ float xielu(float z, float ap, float an) {
  const float neg = fminf(z, 0.f);
  return 0.5f * z + (z > 0.f ? ap * z * z : an * (expm1f(neg) - neg));
}

// The same with the hardware exponential, for epilogues that round the result to bf16: the absolute
// error of e^z - 1 is about 1e-7, far below half a bf16 step of the result except where the result
// itself is of that size.
__device__ __forceinline__ float xielu_fast(float z, float ap, float an) {
  const float neg = fminf(z, 0.f);
  return 0.5f * z + (z > 0.f ? ap * z * z : an * (__expf(neg) - 1.f - neg));
}

}  // namespace rb
