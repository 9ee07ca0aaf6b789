// The activations of gated feed-forwards, f(gate, up), that the matrix products carry in their epilogues.
#pragma once
#include "common.cuh"

namespace atom {

constexpr int kGateSilu = 1;       // silu(g) * u
constexpr int kGateGelu = 2;       // gelu_tanh(g) * u
constexpr int kGateClamped = 3;    // g = min(g, limit), u = clamp(u, -limit, limit): g * sigmoid(1.702 g) * (u + 1)

constexpr float kClampedSlope = 1.702f;

__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-kClampedSlope * g)) * (u + 1.f);
}

// silu or the clamped form (act is one of the codes above).
__device__ __forceinline__ float gated_act(int act, float g, float u, float limit) {
  return act == kGateClamped ? clamped_gate(g, u, limit) : g / (1.f + expf(-g)) * u;
}

}  // namespace atom
