// Gated units that several kernels form between two projections.
#pragma once

#include <cuda_runtime.h>

// g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(1.702 g) (u + 1).
__device__ __forceinline__ float pl_clamped_unit(float gate, float up, float limit) {
    const float g = fminf(gate, limit);
    const float u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}
