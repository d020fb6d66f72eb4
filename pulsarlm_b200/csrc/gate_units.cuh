// Gated units that several kernels form between two projections.
#pragma once

#include <cuda_runtime.h>

// g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1). EXACT: the library's exponential and
// division (the float32 engine); else the hardware's approximate ones, far below the bfloat16 step the result is
// rounded to.
template <bool EXACT>
__device__ __forceinline__ float pl_clamped_unit(float gate, float up, float limit) {
    const float g = fminf(gate, limit);
    const float u = fminf(fmaxf(up, -limit), limit);
    return (EXACT ? g / (1.0f + expf(-1.702f * g)) : __fdividef(g, 1.0f + __expf(-1.702f * g))) * (u + 1.0f);
}

// The exact GELU: z Phi(z), Phi the normal distribution's, through the complementary error function (accurate for
// negative z, where 1 + erf would cancel).
__device__ __forceinline__ float pl_gelu(float z) { return 0.5f * z * erfcf(-0.70710678118654752f * z); }

// Activations of a plain projection by code: 1 the square of relu, 2 tanh, 3 the exact GELU, else none.
__device__ __forceinline__ float pl_plain_activation(float z, int act) {
    if (act == 1) {
        return z > 0.0f ? z * z : 0.0f;
    }
    return act == 2 ? tanhf(z) : act == 3 ? pl_gelu(z) : z;
}
