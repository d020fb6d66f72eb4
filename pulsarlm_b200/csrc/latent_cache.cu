// Rows RMS-normed and stored into a paged cache: what a mixer that caches one low-rank
// latent per token (instead of keys and values per head) writes each step.
//
//   c[t] = z[t] * rsqrt(mean(z[t]^2) + eps) * weight          fp32, one rounding on store
//   pool[table[entry[t]][pos[t] / page], pos[t] % page] = c[t]
//
// One warp per token; the sum of squares is added in an order fixed by the rank.
#include "common.cuh"

namespace {

template <typename scalar_t>
__global__ void norm_write_paged_kernel(const scalar_t* __restrict__ z, int64_t row_stride,
                                        const float* __restrict__ weight, float eps,
                                        const int32_t* __restrict__ pos, const int32_t* __restrict__ entry,
                                        const int32_t* __restrict__ table, int table_width,
                                        scalar_t* __restrict__ pool, int64_t page_stride, int page_size, int n_pages,
                                        int rank, int n_tokens, int32_t* status) {
    pl_grid_trigger();
    pl_grid_wait();
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (t >= n_tokens) {
        return;
    }
    const scalar_t* row = z + t * row_stride;
    float square = 0.0f;
    for (int d = lane; d < rank; d += 32) {
        const float value = pl_load(row + d);
        square += value * value;
    }
    const float inv = 1.0f / sqrtf(pl_warp_sum(square) / static_cast<float>(rank) + eps);
    const int p = pos[t];
    const int page = table[static_cast<int64_t>(entry[t]) * table_width + p / page_size];
    if (page < 0 || page >= n_pages) {
        if (lane == 0 && status != nullptr) {
            atomicOr(status, 2);
        }
        return;
    }
    scalar_t* dst = pool + page * page_stride + static_cast<int64_t>(p % page_size) * rank;
    for (int d = lane; d < rank; d += 32) {
        pl_store(dst + d, pl_load(row + d) * inv * weight[d]);
    }
}

// Two latents of a token at once: block row 0 norms the queries' latent into a dense row, block row 1 (where the layer
// caches) the latent that is cached into its page. A warp per row; four elements a lane and turn where VEC is 4. The
// order of additions is fixed by the rank.
struct LatentNorm {
    const void* z;
    int64_t row_stride;
    const float* weight;
    int rank;
};

template <typename scalar_t, int VEC>
__device__ __forceinline__ void norm_row(const scalar_t* __restrict__ row, const float* __restrict__ weight, int rank,
                                         float eps, scalar_t* __restrict__ dst, int lane) {
    float square = 0.0f;
    if constexpr (VEC == 4) {
        for (int d = lane * 4; d < rank; d += 128) {
            const float4 x = pl_load4(row + d);
            square = fmaf(x.x, x.x, square);
            square = fmaf(x.y, x.y, square);
            square = fmaf(x.z, x.z, square);
            square = fmaf(x.w, x.w, square);
        }
    } else {
        for (int d = lane; d < rank; d += 32) {
            const float x = pl_load(row + d);
            square = fmaf(x, x, square);
        }
    }
    const float inv = 1.0f / sqrtf(pl_warp_sum(square) / static_cast<float>(rank) + eps);
    if constexpr (VEC == 4) {
        for (int d = lane * 4; d < rank; d += 128) {
            const float4 x = pl_load4(row + d), w = *reinterpret_cast<const float4*>(weight + d);
            pl_store4(dst + d, make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w));
        }
    } else {
        for (int d = lane; d < rank; d += 32) {
            pl_store(dst + d, pl_load(row + d) * inv * weight[d]);
        }
    }
}

template <typename scalar_t, int VEC>
__global__ void latent_norms_kernel(const LatentNorm query, scalar_t* __restrict__ query_out, const LatentNorm cached,
                                    float eps, const int32_t* __restrict__ pos, const int32_t* __restrict__ entry,
                                    const int32_t* __restrict__ table, int table_width, scalar_t* __restrict__ pool,
                                    int64_t page_stride, int page_size, int n_pages, int n_tokens, int32_t* status) {
    pl_grid_trigger();
    pl_grid_wait();
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (t >= n_tokens) {
        return;
    }
    const LatentNorm& n = blockIdx.y == 0 ? query : cached;
    const scalar_t* row = static_cast<const scalar_t*>(n.z) + t * n.row_stride;
    scalar_t* dst = query_out + static_cast<int64_t>(t) * query.rank;
    if (blockIdx.y == 1) {
        const int p = pos[t];
        const int page = table[static_cast<int64_t>(entry[t]) * table_width + p / page_size];
        if (page < 0 || page >= n_pages) {
            if (lane == 0 && status != nullptr) {
                atomicOr(status, 2);
            }
            return;
        }
        dst = pool + page * page_stride + static_cast<int64_t>(p % page_size) * n.rank;
    }
    norm_row<scalar_t, VEC>(row, n.weight, n.rank, eps, dst, lane);
}

}  // namespace

// z [T, rank] with row_stride elements between rows and pool [pages, 1, page_size, rank]
// (page_stride elements between pages) in the engine's dtype; weight fp32 [rank].
PL_API int pl_norm_write_paged(const void* z, int64_t row_stride, const float* weight, float eps, const int32_t* pos,
                               const int32_t* entry, const int32_t* table, int table_width, void* pool,
                               int64_t page_stride, int page_size, int n_pages, int rank, int n_tokens, int dtype,
                               int32_t* status, cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && rank > 0 && page_size > 0 && table_width > 0, "norm_write_paged: bad sizes tokens=%d "
               "rank=%d page=%d", n_tokens, rank, page_size);
    if (n_tokens == 0) {
        return 0;
    }
    const int warps = 4;
    PL_DISPATCH_DTYPE(dtype, "norm_write_paged", {
        pl_launch_overlapped(norm_write_paged_kernel<scalar_t>, dim3((n_tokens + warps - 1) / warps), dim3(warps * 32), 0,
                             stream, static_cast<const scalar_t*>(z), row_stride, weight, eps, pos, entry, table,
                             table_width, static_cast<scalar_t*>(pool), page_stride, page_size, n_pages, rank,
                             n_tokens, status);
    });
    PL_CHECK_LAUNCH("norm_write_paged");
    return 0;
}

// query_out [T, query_rank] = rmsnorm(query_z) * query_weight, dense; and, where z is not nullptr, pl_norm_write_paged of z
// in the same launch. Rows of query_z and z may be columns of one wider matrix.
PL_API int pl_latent_norms(const void* query_z, int64_t query_stride, const float* query_weight, int query_rank,
                           void* query_out, const void* z, int64_t row_stride, const float* weight, int rank, float eps,
                           const int32_t* pos, const int32_t* entry, const int32_t* table, int table_width, void* pool,
                           int64_t page_stride, int page_size, int n_pages, int n_tokens, int dtype, int32_t* status,
                           cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && query_rank > 0 && (z == nullptr || (rank > 0 && page_size > 0 && table_width > 0)),
               "latent_norms: bad sizes tokens=%d ranks=%d, %d", n_tokens, query_rank, rank);
    if (n_tokens == 0) {
        return 0;
    }
    const int warps = 4;
    const dim3 grid((n_tokens + warps - 1) / warps, z != nullptr ? 2 : 1);
    PL_DISPATCH_DTYPE(dtype, "latent_norms", {
        auto whole = [](const void* ptr) { return reinterpret_cast<uintptr_t>(ptr) % (4 * sizeof(scalar_t)) == 0; };
        bool vectors = query_rank % 4 == 0 && query_stride % 4 == 0 && whole(query_z) && whole(query_out) &&
            reinterpret_cast<uintptr_t>(query_weight) % 16 == 0;
        if (z != nullptr) {
            vectors = vectors && rank % 4 == 0 && row_stride % 4 == 0 && page_stride % 4 == 0 && whole(z) && whole(pool) &&
                reinterpret_cast<uintptr_t>(weight) % 16 == 0;
        }
        const LatentNorm query = {query_z, query_stride, query_weight, query_rank};
        const LatentNorm cached = {z, row_stride, weight, rank};
        pl_launch_overlapped(vectors ? latent_norms_kernel<scalar_t, 4> : latent_norms_kernel<scalar_t, 1>, grid,
                             dim3(warps * 32), 0, stream, query, static_cast<scalar_t*>(query_out), cached, eps, pos, entry,
                             table, table_width, static_cast<scalar_t*>(pool), page_stride, page_size, n_pages, n_tokens,
                             status);
    });
    PL_CHECK_LAUNCH("latent_norms");
    return 0;
}
