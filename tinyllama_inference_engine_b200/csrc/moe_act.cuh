// How the two halves of an expert's first product meet, the same in every kernel of routed experts.
#pragma once

#include "common.cuh"

namespace tlie {

// kind 0: silu(gate) * up.  1: gelu (tanh form) of the gate times up.  2: the square of relu, for experts without a gate.  3: with g = min(gate, limit) and
// u = clamp(up, -limit, limit), g * sigmoid(alpha * g) * (u + shift).
template <int KIND>
__device__ __forceinline__ float expert_gate(float g, float u, float limit, float alpha, float shift) {
  if (KIND == 3) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + shift);
  }
  if (KIND == 2) {
    const float r = fmaxf(g, 0.0f);
    return r * r * u;
  }
  if (KIND == 1) return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  return g / (1.0f + expf(-g)) * u;
}

struct ExpertGate {
  int kind;
  float limit, alpha, shift;   // kind 3
  __device__ __forceinline__ float operator()(float g, float u) const {
    switch (kind) {
      case 3: return expert_gate<3>(g, u, limit, alpha, shift);
      case 2: return expert_gate<2>(g, u, limit, alpha, shift);
      case 1: return expert_gate<1>(g, u, limit, alpha, shift);
    }
    return expert_gate<0>(g, u, limit, alpha, shift);
  }
  __device__ __forceinline__ float ungated(float z) const { return (*this)(z, 1.0f); }
};

}  // namespace tlie
