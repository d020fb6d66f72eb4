// Pieces of a row: PER neighbouring elements as one load or store (16 bytes' worth, or one element for sizes and
// addresses that do not allow more), kept as they are stored until a kernel wants floats.
#pragma once

#include "common.cuh"

template <typename scalar_t, int PER>
struct RowPiece;

template <typename scalar_t>
struct RowPiece<scalar_t, 1> {
    using Raw = scalar_t;
    __device__ static __forceinline__ Raw get(const scalar_t* p) { return *p; }
    __device__ static __forceinline__ void put(scalar_t* p, Raw raw) { *p = raw; }
    __device__ static __forceinline__ void floats(Raw raw, float (&o)[1]) { o[0] = pl_load(&raw); }
    __device__ static __forceinline__ Raw pack(const float (&v)[1]) {
        scalar_t r;
        pl_store(&r, v[0]);
        return r;
    }
};
template <>
struct RowPiece<float, 4> {
    using Raw = float4;
    __device__ static __forceinline__ Raw get(const float* p) { return *reinterpret_cast<const float4*>(p); }
    __device__ static __forceinline__ void put(float* p, Raw raw) { *reinterpret_cast<float4*>(p) = raw; }
    __device__ static __forceinline__ void floats(Raw raw, float (&o)[4]) {
        o[0] = raw.x;
        o[1] = raw.y;
        o[2] = raw.z;
        o[3] = raw.w;
    }
    __device__ static __forceinline__ Raw pack(const float (&v)[4]) { return make_float4(v[0], v[1], v[2], v[3]); }
};
template <>
struct RowPiece<__nv_bfloat16, 8> {
    using Raw = uint4;
    __device__ static __forceinline__ Raw get(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
    __device__ static __forceinline__ void put(__nv_bfloat16* p, Raw raw) { *reinterpret_cast<uint4*>(p) = raw; }
    __device__ static __forceinline__ void floats(Raw raw, float (&o)[8]) {
        // (a bfloat16 is the upper half of a float)
        const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[2 * i] = __uint_as_float(words[i] << 16);
            o[2 * i + 1] = __uint_as_float(words[i] & 0xffff0000u);
        }
    }
    __device__ static __forceinline__ Raw pack(const float (&v)[8]) {
        uint4 raw;
        uint32_t* words = reinterpret_cast<uint32_t*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 pair = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
            words[i] = *reinterpret_cast<const uint32_t*>(&pair);
        }
        return raw;
    }
};

// PER floats from an fp32 array (16-byte aligned when PER is a multiple of 4).
template <int PER>
__device__ __forceinline__ void pl_floats(const float* p, float (&o)[PER]) {
    if constexpr (PER % 4 == 0) {
#pragma unroll
        for (int i = 0; i < PER; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(p + i);
            o[i] = v.x;
            o[i + 1] = v.y;
            o[i + 2] = v.z;
            o[i + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            o[i] = p[i];
        }
    }
}
