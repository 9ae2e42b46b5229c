// Activations of gated feed-forwards, a function of the gate's and the up projection's value:
//   limit == 0   SwiGLU: silu(g) u
//   limit  > 0   clamped gate: g' = min(g, limit), u' = clamp(u, -limit, limit),
//                g' sigmoid(1.702 g') (u' + 1)
#pragma once

namespace rb {

constexpr float kClampedGateSlope = 1.702f;

__device__ __forceinline__ float gated_act(float g, float u, float limit) {
  if (limit > 0.f) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-kClampedGateSlope * g)) * (u + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}
// The same with the hardware exponential and division, for results that are rounded to bf16.
__device__ __forceinline__ float gated_act_fast(float g, float u, float limit) {
  if (limit > 0.f) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.f + __expf(fminf(-kClampedGateSlope * g, 80.f))) * (u + 1.f);
  }
  return __fdividef(g, 1.f + __expf(fminf(-g, 80.f))) * u;
}

}  // namespace rb
