// Gated feed-forward activations: g and u are the two halves of the input product.
#pragma once
#include <math.h>

namespace axb {

enum GateKind { kGateSilu = 0, kGateGeluTanh = 1, kGateClamped = 2 };

template <int kKind>
__device__ __forceinline__ float gate_value(float g, float u, float limit, float alpha) {
  if (kKind == kGateSilu) return g / (1.f + expf(-g)) * u;
  if (kKind == kGateGeluTanh) {
    // 0.5 (1 + tanh(t)) = 1 / (1 + exp(-2 t)), t = sqrt(2 / pi) (g + 0.044715 g^3)
    const float t = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return g / (1.f + expf(-2.f * t)) * u;
  }
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

}  // namespace axb
