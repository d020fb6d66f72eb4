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
