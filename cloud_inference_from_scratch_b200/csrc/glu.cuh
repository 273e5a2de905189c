// The gated activation of an expert, and what multiplies its input.
#pragma once

namespace cie {

// clamped == 0: SiLU(g) * u.  clamped == 1: g = min(g, limit), u = clamp(u, -limit, limit),
// g * sigmoid(slope * g) * (u + shift).  weights (or nullptr): gate and up of (token, choice) pair p are multiplied by
// weights[p] first, which is what multiplying the expert's input by it does.
struct GluAct {
  int clamped;
  float limit, slope, shift;
  const float* weights;
};

__device__ __forceinline__ float glu(const GluAct& a, float g, float u, float weight) {
  g *= weight;
  u *= weight;
  if (a.clamped) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    return g / (1.f + expf(-a.slope * g)) * (u + a.shift);
  }
  return g / (1.f + expf(-g)) * u;
}

}  // namespace cie
