// The residual add of a layer whose mixer is two sublayers side by side, each output normed on its way in, beside a
// feed-forward that read the same input:
//
//   v = x + factor * (u1 / rms(u1) * w1 + u2 / rms(u2) * w2) + y3        u1 = y1 + b1, u2 = y2 + b2
//
// fused with what the next reader wants, one of
//
//   out = v / rms(v) * w                         the next layer's norm (or the model's last one over chosen rows)
//   out = [v, entered]                           two rows side by side: the input of a projection that joins the
//                                                stream with what entered the first layer
//   nothing                                      (out == nullptr) the stream alone is updated
//
// rms(u) = sqrt(mean(u^2) + eps). Every term may be absent (y1 and y2 together). One block per row, statistics and
// sums in fp32 in an order that the width alone decides, one rounding on each store.
#include "row_piece.cuh"

namespace {

template <typename scalar_t>
struct SideNormParams {
    float* x;
    const scalar_t* y1;
    const float* b1;
    const float* w1;
    const scalar_t* y2;
    const float* b2;
    const float* w2;
    float factor, eps_y;
    const scalar_t* y3;
    const float* w;  // the next norm (nullptr: none)
    float eps;
    const float* entered;  // (join) fp32 [T, hidden]
    scalar_t* out;         // [rows, hidden], or (join) [rows, 2 * hidden]
    const int32_t* rows;
    int hidden;
};

// Two sums over the block at once.
__device__ __forceinline__ float2 block_sums(float2 v, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v.x = pl_warp_sum(v.x);
    v.y = pl_warp_sum(v.y);
    __syncthreads();
    if (lane == 0) {
        scratch[warp] = v;
    }
    __syncthreads();
    const int warps = (blockDim.x + 31) >> 5;
    const float2 total = lane < warps ? scratch[lane] : make_float2(0.0f, 0.0f);
    return make_float2(pl_warp_sum(total.x), pl_warp_sum(total.y));
}

// The row in registers, VECS groups of four a thread.
template <typename scalar_t, int VECS>
__global__ void __launch_bounds__(512) side_norm_reg_kernel(const SideNormParams<scalar_t> p) {
    pl_grid_trigger();
    __shared__ float2 scratch[32];
    const int n_vec = p.hidden / 4;
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 g1[VECS], g2[VECS], gw[VECS];  // (weights: read before the wait on earlier kernels)
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        const bool in = c < n_vec;
        g1[i] = in && p.y1 != nullptr ? pl_load4(p.w1 + 4 * c) : zero;
        g2[i] = in && p.y1 != nullptr ? pl_load4(p.w2 + 4 * c) : zero;
        gw[i] = in && p.w != nullptr ? pl_load4(p.w + 4 * c) : zero;
    }
    pl_grid_wait();
    const int r = blockIdx.x;
    const int64_t s = p.rows != nullptr ? p.rows[r] : r;
    const int64_t at = s * p.hidden;
    float4 u1[VECS], u2[VECS], v[VECS];
    float2 squares = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        u1[i] = u2[i] = v[i] = zero;
        if (c < n_vec) {
            v[i] = pl_load4(p.x + at + 4 * c);
            if (p.y1 != nullptr) {
                u1[i] = pl_load4(p.y1 + at + 4 * c);
                u2[i] = pl_load4(p.y2 + at + 4 * c);
            }
            if (p.y3 != nullptr) {
                const float4 y = pl_load4(p.y3 + at + 4 * c);
                v[i].x += y.x;
                v[i].y += y.y;
                v[i].z += y.z;
                v[i].w += y.w;
            }
            if (p.b1 != nullptr) {
                const float4 b = pl_load4(p.b1 + 4 * c);
                u1[i].x += b.x;
                u1[i].y += b.y;
                u1[i].z += b.z;
                u1[i].w += b.w;
            }
            if (p.b2 != nullptr) {
                const float4 b = pl_load4(p.b2 + 4 * c);
                u2[i].x += b.x;
                u2[i].y += b.y;
                u2[i].z += b.z;
                u2[i].w += b.w;
            }
            squares.x += u1[i].x * u1[i].x + u1[i].y * u1[i].y + u1[i].z * u1[i].z + u1[i].w * u1[i].w;
            squares.y += u2[i].x * u2[i].x + u2[i].y * u2[i].y + u2[i].z * u2[i].z + u2[i].w * u2[i].w;
        }
    }
    const float n = static_cast<float>(p.hidden);
    float f1 = 0.0f, f2 = 0.0f;
    if (p.y1 != nullptr) {
        const float2 total = block_sums(squares, scratch);
        f1 = p.factor / sqrtf(total.x / n + p.eps_y);
        f2 = p.factor / sqrtf(total.y / n + p.eps_y);
    }
    const bool write_back = p.rows == nullptr && (p.y1 != nullptr || p.y3 != nullptr);
    float local = 0.0f;
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n_vec) {
            v[i].x += u1[i].x * f1 * g1[i].x + u2[i].x * f2 * g2[i].x;
            v[i].y += u1[i].y * f1 * g1[i].y + u2[i].y * f2 * g2[i].y;
            v[i].z += u1[i].z * f1 * g1[i].z + u2[i].z * f2 * g2[i].z;
            v[i].w += u1[i].w * f1 * g1[i].w + u2[i].w * f2 * g2[i].w;
            if (write_back) {
                pl_store4(p.x + at + 4 * c, v[i]);
            }
            local += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
    }
    if (p.out == nullptr) {
        return;
    }
    if (p.entered != nullptr) {
        scalar_t* out = p.out + static_cast<int64_t>(r) * 2 * p.hidden;
#pragma unroll
        for (int i = 0; i < VECS; ++i) {
            const int c = threadIdx.x + i * blockDim.x;
            if (c < n_vec) {
                pl_store4(out + 4 * c, v[i]);
                pl_store4(out + p.hidden + 4 * c, pl_load4(p.entered + at + 4 * c));
            }
        }
        return;
    }
    const float inv = 1.0f / sqrtf(block_sums(make_float2(local, 0.0f), scratch).x / n + p.eps);
#pragma unroll
    for (int i = 0; i < VECS; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < n_vec) {
            pl_store4(p.out + static_cast<int64_t>(r) * p.hidden + 4 * c,
                      make_float4(v[i].x * inv * gw[i].x, v[i].y * inv * gw[i].y, v[i].z * inv * gw[i].z,
                                  v[i].w * inv * gw[i].w));
        }
    }
}

// Any width: the row in shared memory, element by element.
template <typename scalar_t>
__global__ void side_norm_kernel(const SideNormParams<scalar_t> p) {
    pl_grid_trigger();
    pl_grid_wait();
    extern __shared__ float row[];  // [hidden]
    __shared__ float2 scratch[32];
    const int r = blockIdx.x;
    const int64_t s = p.rows != nullptr ? p.rows[r] : r;
    const int64_t at = s * p.hidden;
    auto side = [&](const scalar_t* y, const float* b, int i) { return pl_load(y + at + i) + (b != nullptr ? b[i] : 0.0f); };
    float2 squares = make_float2(0.0f, 0.0f);
    if (p.y1 != nullptr) {
        for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
            const float a = side(p.y1, p.b1, i), b = side(p.y2, p.b2, i);
            squares.x += a * a;
            squares.y += b * b;
        }
    }
    const float n = static_cast<float>(p.hidden);
    float f1 = 0.0f, f2 = 0.0f;
    if (p.y1 != nullptr) {
        const float2 total = block_sums(squares, scratch);
        f1 = p.factor / sqrtf(total.x / n + p.eps_y);
        f2 = p.factor / sqrtf(total.y / n + p.eps_y);
    }
    const bool write_back = p.rows == nullptr && (p.y1 != nullptr || p.y3 != nullptr);
    float local = 0.0f;
    for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
        float v = p.x[at + i];
        if (p.y3 != nullptr) {
            v += pl_load(p.y3 + at + i);
        }
        if (p.y1 != nullptr) {
            v += side(p.y1, p.b1, i) * f1 * p.w1[i] + side(p.y2, p.b2, i) * f2 * p.w2[i];
        }
        if (write_back) {
            p.x[at + i] = v;
        }
        row[i] = v;
        local += v * v;
    }
    if (p.out == nullptr) {
        return;
    }
    if (p.entered != nullptr) {
        scalar_t* out = p.out + static_cast<int64_t>(r) * 2 * p.hidden;
        for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
            pl_store(out + i, row[i]);  // (a thread reads back what it wrote)
            pl_store(out + p.hidden + i, p.entered[at + i]);
        }
        return;
    }
    const float inv = 1.0f / sqrtf(block_sums(make_float2(local, 0.0f), scratch).x / n + p.eps);
    for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
        pl_store(p.out + static_cast<int64_t>(r) * p.hidden + i, row[i] * inv * p.w[i]);
    }
}

template <typename scalar_t>
int launch(const SideNormParams<scalar_t>& p, int n_rows, cudaStream_t stream) {
    const int hidden = p.hidden;
    const bool vectors = hidden % 4 == 0 &&
        ((reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.y1) | reinterpret_cast<uintptr_t>(p.y2) |
          reinterpret_cast<uintptr_t>(p.y3) | reinterpret_cast<uintptr_t>(p.b1) | reinterpret_cast<uintptr_t>(p.b2) |
          reinterpret_cast<uintptr_t>(p.w1) | reinterpret_cast<uintptr_t>(p.w2) | reinterpret_cast<uintptr_t>(p.w) |
          reinterpret_cast<uintptr_t>(p.entered) | reinterpret_cast<uintptr_t>(p.out)) & 15) == 0;
    int threads = ((hidden + 3) / 4 + 31) / 32 * 32;
    threads = threads < 64 ? 64 : threads > 512 ? 512 : threads;
    if (vectors && hidden <= 4 * 4 * threads) {
        const int vecs = (hidden / 4 + threads - 1) / threads;
        if (vecs == 1) {
            pl_launch_overlapped(side_norm_reg_kernel<scalar_t, 1>, dim3(n_rows), dim3(threads), 0, stream, p);
        } else if (vecs == 2) {
            pl_launch_overlapped(side_norm_reg_kernel<scalar_t, 2>, dim3(n_rows), dim3(threads), 0, stream, p);
        } else {
            pl_launch_overlapped(side_norm_reg_kernel<scalar_t, 4>, dim3(n_rows), dim3(threads), 0, stream, p);
        }
    } else {
        const size_t smem = static_cast<size_t>(hidden) * sizeof(float);
        if (smem > 48 * 1024) {
            cudaFuncSetAttribute(side_norm_kernel<scalar_t>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 static_cast<int>(smem));
        }
        pl_launch_overlapped(side_norm_kernel<scalar_t>, dim3(n_rows), dim3(threads), smem, stream, p);
    }
    PL_CHECK_LAUNCH("side_norm");
    return 0;
}

}  // namespace

// x fp32 [T, hidden]; y1, y2, y3 [T, hidden] in the engine's dtype (y1 and y2 together or neither; y3 may be nullptr);
// b1, b2 (each may be nullptr), w1, w2, w fp32 [hidden]. rows == nullptr: every row, x updated in place; rows given:
// output row r is made from source row rows[r] and x is left as it was. entered (fp32 [T, hidden]) with out [rows, 2 *
// hidden]: the stream and `entered` side by side; else out [rows, hidden] is the stream's RMS norm with weight w;
// out == nullptr: the stream alone.
PL_API int pl_side_norm(float* x, const void* y1, const float* b1, const float* w1, const void* y2, const float* b2,
                        const float* w2, float factor, float eps_y, const void* y3, const float* w, float eps,
                        const float* entered, void* out, const int32_t* rows, int n_rows, int hidden, int dtype,
                        cudaStream_t stream) {
    PL_REQUIRE(n_rows >= 0 && hidden > 0, "side_norm: bad sizes rows=%d hidden=%d", n_rows, hidden);
    PL_REQUIRE((y1 == nullptr) == (y2 == nullptr) && (y1 == nullptr || (w1 != nullptr && w2 != nullptr)),
               "side_norm: both sides come with their norms' weights, or neither");
    PL_REQUIRE(out == nullptr || entered != nullptr || w != nullptr, "side_norm: a normed output needs its weight");
    PL_REQUIRE(hidden * sizeof(float) <= 160 * 1024, "side_norm: width %d is too large", hidden);
    if (n_rows == 0) {
        return 0;
    }
    PL_DISPATCH_DTYPE(dtype, "side_norm", {
        SideNormParams<scalar_t> p;
        p.x = x;
        p.y1 = static_cast<const scalar_t*>(y1);
        p.b1 = y1 != nullptr ? b1 : nullptr;
        p.w1 = w1;
        p.y2 = static_cast<const scalar_t*>(y2);
        p.b2 = y2 != nullptr ? b2 : nullptr;
        p.w2 = w2;
        p.factor = factor;
        p.eps_y = eps_y;
        p.y3 = static_cast<const scalar_t*>(y3);
        p.w = w;
        p.eps = eps;
        p.entered = entered;
        p.out = static_cast<scalar_t*>(out);
        p.rows = rows;
        p.hidden = hidden;
        return launch<scalar_t>(p, n_rows, stream);
    });
    return 0;
}
