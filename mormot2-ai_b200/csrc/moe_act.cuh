// The activations of the experts' first product, shared by the routed products' kernels.
#pragma once
#include "common.cuh"

// act(gate) * up. 0: SiLU; 1: the tanh form of GELU; 2: the clamped form
// g' = min(g, limit), u' = clamp(u, -limit, limit), g' sigmoid(1.702 g') (u' + 1).
__device__ __forceinline__ float moe_gated(float z, float u, int act, float limit) {
  if (act == 2) {
    z = fminf(z, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return z / (1.0f + expf(-1.702f * z)) * (u + 1.0f);
  }
  if (act == 1)
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * u;
  return z / (1.0f + expf(-z)) * u;
}

// An activation of one input, for experts without a gate (the codes of the elementwise kernels).
// 0: SiLU; 1: the tanh form of GELU; 3: the square of relu.
__device__ __forceinline__ float moe_plain(float z, int act) {
  if (act == 3) {
    z = fmaxf(z, 0.f);
    return z * z;
  }
  if (act == 1)
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  return z / (1.0f + expf(-z));
}

// What a product of the experts is: the second one, the first with gate and up rows, or the first
// of experts without a gate (W [E][N][K]).
enum { MOE_DOWN = 0, MOE_GATED_UP = 1, MOE_PLAIN_UP = 2 };

template <int MODE>
__device__ __forceinline__ float moe_act(float z, float u, int act, float limit) {
  return MODE == MOE_GATED_UP ? moe_gated(z, u, act, limit) : moe_plain(z, act);
}
