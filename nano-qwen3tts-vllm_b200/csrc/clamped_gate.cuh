// clamped_gate.cuh - the activation of clamped gated feed-forwards, shared by the epilogues of the dense and the grouped
// GEMM and by the stand-alone kernel:
//
//   g = min(gate, limit),  u = clamp(up, -limit, limit):      g * sigmoid(alpha g) * (u + 1)
#pragma once

#include "common.cuh"

namespace b2 {

__device__ __forceinline__ float clamped_gate(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}

}  // namespace b2
