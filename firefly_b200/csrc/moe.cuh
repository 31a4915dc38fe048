// What the grouped products over experts share: the kinds of product and the activations between the two of them.
#pragma once
#include "common.cuh"

namespace ff {

// MOE_GATEUP: two B matrices (gate and up), gathered A rows, out = activation(gate, up) in the activation type.
// MOE_UP: one B matrix, gathered A rows, out = relu(up)^2.  MOE_DOWN: A rows in place, out 32-bit.
enum { MOE_DOWN = 0, MOE_GATEUP = 1, MOE_UP = 2 };

// act 1: silu(g) * u, no clamps.  act 0: g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = clamp(u, -limit, limit).
__device__ __forceinline__ float clamped_glu(float g, float u, float limit, int act = 0) {
    if (act == 1) return g / (1.0f + expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}

// The same on the fast exponential and division, for results that are rounded to bfloat16.
__device__ __forceinline__ float clamped_glu_fast(float g, float u, float limit, int act) {
    if (act == 1) return __fdividef(g, 1.0f + __expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-1.702f * g)) * (u + 1.0f);
}

constexpr int GROUPED_TC_ROWS = 128;      // rows of a row tile of the tensor-core product

__device__ __forceinline__ float relu2(float z) { z = fmaxf(z, 0.f); return z * z; }

}  // namespace ff
