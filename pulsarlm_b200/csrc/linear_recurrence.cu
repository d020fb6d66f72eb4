// A gated linear recurrence per channel (an RG-LRU) behind a short convolution over time:
//
//   u[t]  = conv_bias + sum_j w[j] * (x[t - (taps - 1) + j] + x_bias)        zeros before position 0; rounded as stored
//   r, i  = sigmoid(Ra_b u_b + ra_bias), sigmoid(Ri_b u_b + ri_bias)          per block b of `block` neighbouring channels
//   log a = decay * r            (decay = -8 softplus(lambda) per channel, at most 0)
//   S     = a * S + sqrt(1 - a^2) * i * u                                      from S = 0
//   out   = S * gelu(y + y_bias)                                               the tanh form
//
// The state S (fp32) and the convolution's last inputs belong to a request's slot. The inputs are kept as a ring of
// `taps` rows indexed by position (position p in row p mod taps, as the projection wrote it, without the bias): a
// token reads rows p - 1 ... p - taps + 1 and writes row p mod taps, which none of them is, so blocks that share a
// token's inputs need not agree on when the ring moves on.
//
// Steps with prompt portions run three kernels: ring_conv (u), the block-diagonal products (elsewhere: [blocks, T,
// 2 * block] in fp32), and the scan over each portion. Steps of single tokens in bfloat16 run `step`,
// one launch for all of it. Gates, decays, the state and its products are fp32.
#include "cluster_helpers.cuh"
#include "row_piece.cuh"

namespace {

// sqrt(1 - a^2) needs 1 - exp(z) for z = 2 log a: where z is near zero the difference of two near-equal numbers would
// lose it, so there the series z (1 + z/2 (1 + z/3 (1 + ...))) stands in (relative error below 3e-7 on [-1/2, 0]).
__device__ __forceinline__ float one_minus_exp(float z, float exp_z) {
    float s = fmaf(z, 1.0f / 8.0f, 1.0f);
    s = fmaf(z * (1.0f / 7.0f), s, 1.0f);
    s = fmaf(z * (1.0f / 6.0f), s, 1.0f);
    s = fmaf(z * (1.0f / 5.0f), s, 1.0f);
    s = fmaf(z * (1.0f / 4.0f), s, 1.0f);
    s = fmaf(z * (1.0f / 3.0f), s, 1.0f);
    s = fmaf(z * (1.0f / 2.0f), s, 1.0f);
    return z > -0.5f ? -z * s : 1.0f - exp_z;
}

// EXACT: the library's exponentials and divisions (the float32 engine); else the hardware's approximate ones, whose
// error is of the order of fp32's own rounding.
template <bool EXACT>
__device__ __forceinline__ float sigmoid_of(float z) {
    return EXACT ? 1.0f / (1.0f + expf(-z)) : __fdividef(1.0f, 1.0f + __expf(-z));
}
template <bool EXACT>
__device__ __forceinline__ void recurrence_terms(float r_pre, float i_pre, float decay, float u, float& a, float& b) {
    const float log_a = decay * sigmoid_of<EXACT>(r_pre);
    a = EXACT ? expf(log_a) : __expf(log_a);
    const float m = one_minus_exp(2.0f * log_a, a * a);
    b = (EXACT ? sqrtf(m) : __fsqrt_rn(m)) * (sigmoid_of<EXACT>(i_pre) * u);
}
// 0.5 z (1 + tanh(q)) = z sigmoid(2 q), q = sqrt(2 / pi) (z + 0.044715 z^3)
template <bool EXACT>
__device__ __forceinline__ float gelu_of(float z) {
    const float q = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z * sigmoid_of<EXACT>(2.0f * q);
}

// ------------------------------------------------------------------------------------------------ convolution
template <typename scalar_t, int PER>
__global__ void __launch_bounds__(128) ring_conv_kernel(
        const scalar_t* __restrict__ x, int64_t x_stride, const float* __restrict__ x_bias,
        const float* __restrict__ weight, const float* __restrict__ conv_bias, int taps,
        const scalar_t* __restrict__ ring, const int32_t* __restrict__ first, const int32_t* __restrict__ entry,
        const int32_t* __restrict__ slots, const int32_t* __restrict__ pos, scalar_t* __restrict__ u, int n_tokens,
        int width, int tokens_per_block) {
    using Piece = RowPiece<scalar_t, PER>;
    pl_grid_trigger();
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * PER;
    if (c >= width) {
        return;
    }
    float xb[PER], cb[PER];
    pl_floats<PER>(x_bias + c, xb);
    pl_floats<PER>(conv_bias + c, cb);
    pl_grid_wait();
    const int t1 = min((static_cast<int>(blockIdx.x) + 1) * tokens_per_block, n_tokens);
    for (int t = blockIdx.x * tokens_per_block; t < t1; ++t) {
        const int e = entry[t], p = pos[t];
        const int inside = t - first[e];  // rows of this portion before this one
        const scalar_t* mine = ring + static_cast<int64_t>(slots[e]) * taps * width + c;
        float y[PER];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            y[i] = 0.0f;
        }
        for (int j = max(0, taps - 1 - p); j < taps; ++j) {
            const int back = taps - 1 - j;
            const typename Piece::Raw raw =
                back <= inside ? Piece::get(x + static_cast<int64_t>(t - back) * x_stride + c)
                               : Piece::get(mine + static_cast<int64_t>((p - back) % taps) * width);
            float v[PER], w[PER];
            Piece::floats(raw, v);
            pl_floats<PER>(weight + static_cast<int64_t>(j) * width + c, w);
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                y[i] = fmaf(w[i], v[i] + xb[i], y[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            y[i] += cb[i];
        }
        Piece::put(u + static_cast<int64_t>(t) * width + c, Piece::pack(y));
    }
}

// ------------------------------------------------------------------------------------------------ scan
// A cluster of CTAs takes 64 channels of one entry's portion, each CTA the next kSpan tokens in turn. Two forms:
//
// * walked (float32): all threads form (a, b) of the CTA's tokens in shared memory at once; then the CTAs walk their
//   tokens one after the other, a thread per channel, and hand the state on through distributed shared memory; then
//   all threads multiply by the other branch and store. The walk is the plain recurrence in token order, whatever the
//   cluster's size: a portion's cut changes no bit.
// * composed (bfloat16): a thread takes kSub neighbouring tokens of a channel, (a, b) and the other branch in
//   registers, and composes them into one step S -> A S + B; a CTA's threads' steps compose into the CTA's, which goes to
//   every CTA's shared memory. One barrier of the cluster makes the steps visible, every thread folds those before its
//   own into its start, and walks its tokens from there. The fp32 sums differ from the walked form's in their last
//   bits only.
constexpr int kChannels = 64;
constexpr int kSpan = 128;
constexpr int kScanThreads = 256;
constexpr int kScanShared = 2 * kSpan * kChannels * static_cast<int>(sizeof(float));
constexpr int kSubs = kScanThreads / kChannels;
constexpr int kSub = kSpan / kSubs;
constexpr int kMaxCluster = 8;

__device__ __forceinline__ void cluster_store1(uint32_t remote, float v) {
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
}
__device__ __forceinline__ void cluster_store2(uint32_t remote, float2 v) {
    asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(remote), "f"(v.x), "f"(v.y) : "memory");
}

struct ScanParams {
    const float* pre;  // [blocks, T, 2 * block]
    const float* ra_bias;
    const float* ri_bias;
    const float* decay;
    const void* u;  // [T, width]
    const void* y;
    int64_t y_stride;
    const float* y_bias;
    const void* x;
    int64_t x_stride;
    void* ring;  // [slots, taps, width]
    int taps;
    float* states;  // [slots, width]
    const int32_t* first;
    const int32_t* count;
    const int32_t* slots;
    const int32_t* pos;
    void* out;  // [T, width]
    int n_tokens, width, block, cluster;
};

// The ring after an entry's portion (the convolution's kernel, which read it, has finished).
template <typename scalar_t>
__device__ __forceinline__ void move_ring_on(const ScanParams& p, int c, int64_t slot, int64_t start, int n_all, int j0, int step) {
    const scalar_t* x = static_cast<const scalar_t*>(p.x);
    scalar_t* ring = static_cast<scalar_t*>(p.ring);
    for (int j = j0; j < min(p.taps - 1, n_all); j += step) {
        const int64_t t = start + n_all - 1 - j;
        ring[(slot * p.taps + p.pos[t] % p.taps) * p.width + c] = x[t * p.x_stride + c];
    }
}

__global__ void __launch_bounds__(kScanThreads) linear_scan_walked_kernel(const ScanParams p) {
    extern __shared__ __align__(16) float terms[];  // [kSpan][kChannels] a, then the same of b (then S)
    float* a_s = terms;
    float* b_s = terms + kSpan * kChannels;
    __shared__ float carry[kChannels];
    pl_grid_trigger();
    const int cluster = p.cluster, rank = blockIdx.x % cluster;
    const int lane = threadIdx.x % kChannels, row0 = threadIdx.x / kChannels;
    const int c = (blockIdx.x / cluster) * kChannels + lane;
    const bool live = c < p.width;
    const float* u = static_cast<const float*>(p.u);
    const float* y = static_cast<const float*>(p.y);
    float* out = static_cast<float*>(p.out);
    float rb = 0.0f, ib = 0.0f, dc = 0.0f, yb = 0.0f;
    if (live) {
        rb = p.ra_bias[c];
        ib = p.ri_bias[c];
        dc = p.decay[c];
        yb = p.y_bias[c];
    }
    const int blk = live ? c / p.block : 0;
    const float* pre_r = p.pre + static_cast<int64_t>(blk) * p.n_tokens * 2 * p.block + (c - blk * p.block);
    if (cluster > 1) {
        cluster_arrive_all();  // "this CTA runs": waited for before the first hand-over
    }
    pl_grid_wait();
    const int e = blockIdx.y;
    const int start = p.first[e], n_all = p.count[e];
    const int64_t slot = p.slots[e];
    if (cluster > 1) {
        cluster_wait_all();
    }
    for (int base = 0; base < n_all; base += cluster * kSpan) {
        const int t0 = base + rank * kSpan;
        const int n = max(0, min(n_all - t0, kSpan));
        if (live) {
            for (int r = row0; r < n; r += kSubs) {
                const int64_t t = start + t0 + r;
                float a, b;
                recurrence_terms<true>(pre_r[t * 2 * p.block] + rb, pre_r[t * 2 * p.block + p.block] + ib, dc,
                                       u[t * p.width + c], a, b);
                a_s[r * kChannels + lane] = a;
                b_s[r * kChannels + lane] = b;
            }
        }
        __syncthreads();
        for (int turn = 0; turn < cluster; ++turn) {
            if (turn == rank && threadIdx.x < kChannels) {
                float s = base == 0 && rank == 0 ? (live ? p.states[slot * p.width + c] : 0.0f) : carry[lane];
                for (int r = 0; r < n; ++r) {
                    s = fmaf(a_s[r * kChannels + lane], s, b_s[r * kChannels + lane]);
                    b_s[r * kChannels + lane] = s;
                }
                if (cluster > 1) {
                    cluster_store1(cluster_map(&carry[lane], (rank + 1) % cluster), s);
                } else {
                    carry[lane] = s;
                }
            }
            if (cluster > 1) {
                __syncwarp();
                cluster_arrive_all();
                cluster_wait_all();
            } else {
                __syncthreads();
            }
        }
        if (live) {
            for (int r = row0; r < n; r += kSubs) {
                const int64_t t = start + t0 + r;
                out[t * p.width + c] = b_s[r * kChannels + lane] * gelu_of<true>(y[t * p.y_stride + c] + yb);
            }
        }
        __syncthreads();
    }
    // (the first CTA was handed the state after the last token)
    if (rank == 0 && live && n_all > 0) {
        if (row0 == 0) {
            p.states[slot * p.width + c] = carry[lane];
        }
        move_ring_on<float>(p, c, slot, start, n_all, row0, kSubs);
    }
}

__global__ void __launch_bounds__(kScanThreads, 2) linear_scan_composed_kernel(const ScanParams p) {
    __shared__ float2 own_steps[kSubs][kChannels];          // this CTA's threads' steps, in token order
    __shared__ float2 steps[2][kMaxCluster][kChannels];     // [round's parity] the CTAs' steps, in token order
    pl_grid_trigger();
    const int cluster = p.cluster, rank = blockIdx.x % cluster;
    const int lane = threadIdx.x % kChannels, sub = threadIdx.x / kChannels;
    const int c_true = (blockIdx.x / cluster) * kChannels + lane;
    const bool live = c_true < p.width;
    const int c = live ? c_true : p.width - 1;  // (threads past the width repeat its last channel and store nothing)
    const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(p.u);
    const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(p.y);
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
    const float rb = p.ra_bias[c], ib = p.ri_bias[c], dc = p.decay[c], yb = p.y_bias[c];
    const int blk = c / p.block;
    const float* pre_r = p.pre + static_cast<int64_t>(blk) * p.n_tokens * 2 * p.block + (c - blk * p.block);
    if (cluster > 1) {
        cluster_arrive_all();  // "this CTA runs": waited for before the first store into a peer
    }
    pl_grid_wait();
    const int e = blockIdx.y;
    const int start = p.first[e], n_all = p.count[e];
    const int64_t slot = p.slots[e];
    float s_base = p.states[slot * p.width + c];  // the state where the round at hand begins
    if (cluster > 1) {
        cluster_wait_all();
    }
    int round = 0;
    for (int base = 0; base < n_all; base += cluster * kSpan, ++round) {
        const int t0 = base + rank * kSpan + sub * kSub;
        const int n = max(0, min(n_all - t0, kSub));
        float a[kSub], b[kSub];
        __nv_bfloat16 other[kSub];
        // Loads first, a batch at a time (places past the portion's end read its last token and count for nothing).
        constexpr int kBatch = 8;
#pragma unroll
        for (int i0 = 0; i0 < kSub; i0 += kBatch) {
            if (i0 < n) {
                float r_pre[kBatch], i_pre[kBatch];
                __nv_bfloat16 u_in[kBatch];
#pragma unroll
                for (int i = 0; i < kBatch; ++i) {
                    const int64_t t = start + min(t0 + i0 + i, n_all - 1);
                    r_pre[i] = pre_r[t * 2 * p.block];
                    i_pre[i] = pre_r[t * 2 * p.block + p.block];
                    u_in[i] = u[t * p.width + c];
                }
#pragma unroll
                for (int i = 0; i < kBatch; ++i) {
                    recurrence_terms<false>(r_pre[i] + rb, i_pre[i] + ib, dc, __bfloat162float(u_in[i]), a[i0 + i], b[i0 + i]);
                    if (i0 + i >= n) {
                        a[i0 + i] = 1.0f;
                        b[i0 + i] = 0.0f;
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < kBatch; ++i) {
                    a[i0 + i] = 1.0f;
                    b[i0 + i] = 0.0f;
                }
            }
        }
        // (the other branch's values are asked for here, ahead of the barrier, where the terms' registers are free again)
#pragma unroll
        for (int i = 0; i < kSub; ++i) {
            other[i] = y[(start + static_cast<int64_t>(min(t0 + i, n_all - 1))) * p.y_stride + c];
        }
        float big_a = 1.0f, big_b = 0.0f;
#pragma unroll
        for (int i = 0; i < kSub; ++i) {
            big_b = fmaf(a[i], big_b, b[i]);
            big_a *= a[i];
        }
        own_steps[sub][lane] = make_float2(big_a, big_b);
        __syncthreads();
        if (sub == 0) {
            float2 all = own_steps[0][lane];
            for (int k = 1; k < kSubs; ++k) {
                const float2 step = own_steps[k][lane];
                all = make_float2(step.x * all.x, fmaf(step.x, all.y, step.y));
            }
            for (int k = 0; k < cluster; ++k) {
                cluster_store2(cluster_map(&steps[round & 1][rank][lane], k), all);
            }
        }
        __syncwarp();
        cluster_arrive_all();  // (a CTA without peers is a cluster of one)
        cluster_wait_all();
        float s = s_base;
        for (int k = 0; k < cluster; ++k) {
            s = k == rank ? s_base : s;
            const float2 step = steps[round & 1][k][lane];
            s_base = fmaf(step.x, s_base, step.y);
        }
        for (int k = 0; k < sub; ++k) {
            const float2 step = own_steps[k][lane];
            s = fmaf(step.x, s, step.y);
        }
#pragma unroll
        for (int i = 0; i < kSub; ++i) {
            s = fmaf(a[i], s, b[i]);
            if (i < n && live) {
                out[(start + static_cast<int64_t>(t0) + i) * p.width + c] =
                    __float2bfloat16_rn(s * gelu_of<false>(__bfloat162float(other[i]) + yb));
            }
        }
        __syncthreads();  // own_steps is written again (a peer writes this parity's steps again only after another barrier)
    }
    if (rank == 0 && live && n_all > 0) {
        if (sub == 0) {
            p.states[slot * p.width + c] = s_base;
        }
        move_ring_on<__nv_bfloat16>(p, c, slot, start, n_all, sub, kSubs);
    }
}

// ------------------------------------------------------------------------------------------------ single tokens
// A step in which every entry brings one token, bfloat16: block (gate block and 16 of its channels, 8 tokens). All of
// the gate block's convolved inputs go to shared memory (each CTA of the gate block makes them anew: a few taps), a
// warp takes the rows of both gates for four channels, and after a transposing sum over the warp every lane holds
// one (channel, token) pair's two products and does its recurrence.
constexpr int kStepTokens = 8;
constexpr int kStepChannels = 16;
constexpr int kStepThreads = 128;

template <int PER>
__global__ void __launch_bounds__(kStepThreads) linear_step_kernel(
        const __nv_bfloat16* __restrict__ x, int64_t x_stride, const float* __restrict__ x_bias,
        const float* __restrict__ weight, const float* __restrict__ conv_bias, int taps, __nv_bfloat16* __restrict__ ring,
        const __nv_bfloat16* __restrict__ gates, const float* __restrict__ ra_bias, const float* __restrict__ ri_bias,
        const float* __restrict__ decay, const __nv_bfloat16* __restrict__ y, int64_t y_stride,
        const float* __restrict__ y_bias, float* __restrict__ states, const int32_t* __restrict__ entry,
        const int32_t* __restrict__ slots, const int32_t* __restrict__ pos, __nv_bfloat16* __restrict__ out, int n_tokens,
        int width, int block) {
    using Piece = RowPiece<__nv_bfloat16, PER>;
    extern __shared__ __align__(16) float u_s[];  // [kStepTokens][block]
    __shared__ int at_s[kStepTokens], slot_s[kStepTokens];
    pl_grid_trigger();
    const int tiles = (block + kStepChannels - 1) / kStepChannels;
    const int blk = blockIdx.x / tiles, o0 = (blockIdx.x - blk * tiles) * kStepChannels;
    const int t0 = blockIdx.y * kStepTokens, here = min(kStepTokens, n_tokens - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int ow = o0 + warp * 4;  // this warp's four channels
    const int c0 = blk * block;
    // The first pieces of the warp's eight rows (ra of its channels, then ri): weights, asked for before the wait.
    const __nv_bfloat16* rows[8];
#pragma unroll
    for (int q = 0; q < 8; ++q) {
        const int o = min(ow + (q & 3), block - 1) + (q >= 4 ? block : 0);
        rows[q] = gates + (static_cast<int64_t>(blk) * 2 * block + o) * block;
    }
    typename Piece::Raw ahead[8];
    const bool first_in = lane * PER < block;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
        ahead[q] = Piece::get(rows[q] + (first_in ? lane * PER : 0));
    }
    pl_grid_wait();
    if (threadIdx.x < kStepTokens) {
        const int t = t0 + min(static_cast<int>(threadIdx.x), here - 1);
        at_s[threadIdx.x] = pos[t];
        slot_s[threadIdx.x] = slots[entry[t]];
    }
    __syncthreads();
    const int pieces = block / PER;
    for (int idx = threadIdx.x; idx < here * pieces; idx += kStepThreads) {
        const int tt = idx / pieces, i0 = (idx - tt * pieces) * PER, c = c0 + i0;
        const int p = at_s[tt];
        __nv_bfloat16* mine = ring + static_cast<int64_t>(slot_s[tt]) * taps * width + c;
        const typename Piece::Raw own = Piece::get(x + static_cast<int64_t>(t0 + tt) * x_stride + c);
        float acc[PER], v[PER], w[PER], xb[PER], cb[PER];
        pl_floats<PER>(x_bias + c, xb);
        pl_floats<PER>(conv_bias + c, cb);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            acc[i] = 0.0f;
        }
        for (int j = max(0, taps - 1 - p); j < taps; ++j) {
            const int back = taps - 1 - j;
            Piece::floats(back == 0 ? own : Piece::get(mine + static_cast<int64_t>((p - back) % taps) * width), v);
            pl_floats<PER>(weight + static_cast<int64_t>(j) * width + c, w);
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                acc[i] = fmaf(w[i], v[i] + xb[i], acc[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            acc[i] += cb[i];
        }
        Piece::floats(Piece::pack(acc), acc);  // (rounded as the kernel of longer steps stores it)
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            u_s[tt * block + i0 + i] = acc[i];
        }
        // The ring's next row, by the CTA whose channels these are (none of the rows read here by any CTA).
        if (taps > 1 && i0 + PER > o0 && i0 < o0 + kStepChannels) {
            if constexpr (kStepChannels % PER == 0) {
                Piece::put(mine + static_cast<int64_t>(p % taps) * width, own);
            }
        }
    }
    __syncthreads();
    float sums[2][4 * kStepTokens];  // [ra, ri][channel * kStepTokens + token]
#pragma unroll
    for (int m = 0; m < 4 * kStepTokens; ++m) {
        sums[0][m] = sums[1][m] = 0.0f;
    }
    if (ow < block) {
        for (int i0 = lane * PER; i0 < block; i0 += 32 * PER) {
            if (i0 != lane * PER) {
#pragma unroll
                for (int q = 0; q < 8; ++q) {
                    ahead[q] = Piece::get(rows[q] + i0);
                }
            }
            float w[8][PER];
#pragma unroll
            for (int q = 0; q < 8; ++q) {
                Piece::floats(ahead[q], w[q]);
            }
#pragma unroll
            for (int tt = 0; tt < kStepTokens; ++tt) {
                if (tt < here) {
                    float v[PER];
                    pl_floats<PER>(u_s + tt * block + i0, v);
#pragma unroll
                    for (int q = 0; q < 8; ++q) {
#pragma unroll
                        for (int i = 0; i < PER; ++i) {
                            sums[q >> 2][(q & 3) * kStepTokens + tt] = fmaf(w[q][i], v[i], sums[q >> 2][(q & 3) * kStepTokens + tt]);
                        }
                    }
                }
            }
        }
    }
    // Sums over the lanes, each lane left with the pair m = lane: halves are exchanged, then quarters, ...
#pragma unroll
    for (int g = 0; g < 2; ++g) {
#pragma unroll
        for (int half = 16; half > 0; half >>= 1) {
            const bool upper = (lane & half) != 0;
#pragma unroll
            for (int m = 0; m < half; ++m) {
                const float keep = upper ? sums[g][m + half] : sums[g][m];
                const float send = upper ? sums[g][m] : sums[g][m + half];
                sums[g][m] = keep + __shfl_xor_sync(0xffffffffu, send, half);
            }
        }
    }
    const int o = ow + lane / kStepTokens, tt = lane % kStepTokens;
    if (o < block && tt < here) {
        const int c = c0 + o;
        const int64_t t = t0 + tt;
        float a, b;
        recurrence_terms<false>(sums[0][0] + ra_bias[c], sums[1][0] + ri_bias[c], decay[c], u_s[tt * block + o], a, b);
        float* state = states + static_cast<int64_t>(slot_s[tt]) * width + c;
        const float s = fmaf(a, *state, b);
        *state = s;
        pl_store(out + t * width + c, s * gelu_of<false>(pl_load(y + t * y_stride + c) + y_bias[c]));
    }
}

}  // namespace

// x [T, width] (x_stride elements between rows), ring [slots, taps, width], u [T, width] dense, in the engine's dtype;
// x_bias, conv_bias fp32 [width]; weight fp32 [taps, width] (the last row the current token's); first int32 [entries]
// the row of each entry's first token; entry, pos int32 [T]; slots int32 [entries]. The ring is read, not written.
PL_API int pl_ring_conv(const void* x, int64_t x_stride, const float* x_bias, const float* weight, const float* conv_bias,
                        int taps, const void* ring, const int32_t* first, const int32_t* entry, const int32_t* slots,
                        const int32_t* pos, void* u, int n_tokens, int width, int dtype, cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && width > 0 && taps >= 1 && x_stride >= width, "ring_conv: bad sizes tokens=%d width=%d "
               "taps=%d", n_tokens, width, taps);
    if (n_tokens == 0) {
        return 0;
    }
    auto whole = [](const void* ptr) { return reinterpret_cast<uintptr_t>(ptr) % 16 == 0; };
    const int per = dtype == PL_F32 ? 4 : 8;
    const bool pieces = width % per == 0 && x_stride % per == 0 && whole(x) && whole(x_bias) && whole(weight) &&
        whole(conv_bias) && whole(ring) && whole(u);
    const int tokens_per_block = n_tokens > 256 ? 4 : 1;
    const int lanes = pieces ? width / per : width;
    const dim3 grid((n_tokens + tokens_per_block - 1) / tokens_per_block, (lanes + 127) / 128);
#define PL_RING_CONV(S, PER)                                                                                          \
    pl_launch_overlapped(ring_conv_kernel<S, PER>, grid, dim3(128), 0, stream, static_cast<const S*>(x), x_stride,    \
                         x_bias, weight, conv_bias, taps, static_cast<const S*>(ring), first, entry, slots, pos,      \
                         static_cast<S*>(u), n_tokens, width, tokens_per_block)
    if (dtype == PL_F32) {
        if (pieces) { PL_RING_CONV(float, 4); } else { PL_RING_CONV(float, 1); }
    } else if (dtype == PL_BF16) {
        if (pieces) { PL_RING_CONV(__nv_bfloat16, 8); } else { PL_RING_CONV(__nv_bfloat16, 1); }
    } else {
        return pl_fail(2, "ring_conv: unknown dtype code %d", dtype);
    }
#undef PL_RING_CONV
    PL_CHECK_LAUNCH("ring_conv");
    return 0;
}

// pre fp32 [width / block, T, 2 * block]: each gate block's products Ra u, then Ri u; ra_bias, ri_bias, decay, y_bias
// fp32 [width]; u, out [T, width] dense, y and x [T, width] with row strides, ring [slots, taps, width] in the engine's
// dtype; states fp32 [slots, width]; first, count, slots int32 [entries]; pos int32 [T]; longest: the most tokens an
// entry brings. Every entry's rows are consecutive; its state and its ring move on.
PL_API int pl_linear_scan(const float* pre, const float* ra_bias, const float* ri_bias, const float* decay, const void* u,
                          const void* y, int64_t y_stride, const float* y_bias, const void* x, int64_t x_stride,
                          void* ring, int taps, float* states, const int32_t* first, const int32_t* count,
                          const int32_t* slots, const int32_t* pos, void* out, int n_tokens, int n_entries, int longest,
                          int width, int block, int dtype, cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && n_entries >= 0 && n_entries <= 65535 && width > 0 && block > 0 && width % block == 0 &&
                   taps >= 1 && longest >= 0,
               "linear_scan: bad sizes tokens=%d entries=%d width=%d block=%d taps=%d", n_tokens, n_entries, width, block,
               taps);
    if (n_tokens == 0 || n_entries == 0) {
        return 0;
    }
    PL_REQUIRE(dtype == PL_F32 || dtype == PL_BF16, "linear_scan: unknown dtype code %d", dtype);
    int cluster = 1;
    while (cluster < kMaxCluster && cluster * kSpan < longest) {
        cluster *= 2;
    }
    const ScanParams p = {pre, ra_bias, ri_bias, decay, u, y, y_stride, y_bias, x, x_stride, ring, taps, states,
                          first, count, slots, pos, out, n_tokens, width, block, cluster};
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3((width + kChannels - 1) / kChannels * cluster, n_entries);
    config.blockDim = dim3(kScanThreads);
    config.dynamicSmemBytes = dtype == PL_F32 ? kScanShared : 0;
    config.stream = stream;
    cudaLaunchAttribute attributes[2];
    attributes[0].id = cudaLaunchAttributeClusterDimension;
    attributes[0].val.clusterDim.x = cluster;
    attributes[0].val.clusterDim.y = 1;
    attributes[0].val.clusterDim.z = 1;
    attributes[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[1].val.programmaticStreamSerializationAllowed = 1;
    config.attrs = attributes;
    config.numAttrs = pl_overlap_enabled() ? 2 : 1;
    cudaError_t err = cudaSuccess;
    if (dtype == PL_F32) {
        err = cudaFuncSetAttribute(linear_scan_walked_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kScanShared);
        if (err == cudaSuccess) {
            err = cudaLaunchKernelEx(&config, linear_scan_walked_kernel, p);
        }
    } else {
        err = cudaLaunchKernelEx(&config, linear_scan_composed_kernel, p);
    }
    if (err != cudaSuccess) {
        return pl_fail(3, "linear_scan: launch failed: %s", cudaGetErrorString(err));
    }
    return 0;
}

// A step in which every entry brings one token, bfloat16: convolution, gates, recurrence, output and both states in
// one launch. gates [width / block, 2 * block, block] (a gate block's rows of Ra, then of Ri); the rest as above.
PL_API int pl_linear_step(const void* x, int64_t x_stride, const float* x_bias, const float* weight,
                          const float* conv_bias, int taps, void* ring, const void* gates, const float* ra_bias,
                          const float* ri_bias, const float* decay, const void* y, int64_t y_stride, const float* y_bias,
                          float* states, const int32_t* entry, const int32_t* slots, const int32_t* pos, void* out,
                          int n_tokens, int width, int block, cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && width > 0 && block > 0 && width % block == 0 && taps >= 1 && x_stride >= width &&
                   y_stride >= width,
               "linear_step: bad sizes tokens=%d width=%d block=%d taps=%d", n_tokens, width, block, taps);
    const size_t smem = static_cast<size_t>(kStepTokens) * block * sizeof(float);
    PL_REQUIRE(smem <= 200 * 1024, "linear_step: gate blocks of %d channels are too wide", block);
    if (n_tokens == 0) {
        return 0;
    }
    auto whole = [](const void* ptr) { return reinterpret_cast<uintptr_t>(ptr) % 16 == 0; };
    const bool pieces = block % 8 == 0 && x_stride % 8 == 0 && whole(x) && whole(x_bias) && whole(weight) &&
        whole(conv_bias) && whole(ring) && whole(gates);
    const dim3 grid(width / block * ((block + kStepChannels - 1) / kStepChannels),
                    (n_tokens + kStepTokens - 1) / kStepTokens);
    PL_REQUIRE(grid.y <= 65535, "linear_step: %d tokens exceed the grid limit", n_tokens);
#define PL_STEP(PER)                                                                                                     \
    if (smem > 48 * 1024) {                                                                                              \
        cudaFuncSetAttribute(linear_step_kernel<PER>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)); \
    }                                                                                                                    \
    pl_launch_overlapped(linear_step_kernel<PER>, grid, dim3(kStepThreads), smem, stream,                                \
                         static_cast<const __nv_bfloat16*>(x), x_stride, x_bias, weight, conv_bias, taps,                \
                         static_cast<__nv_bfloat16*>(ring), static_cast<const __nv_bfloat16*>(gates), ra_bias, ri_bias,  \
                         decay, static_cast<const __nv_bfloat16*>(y), y_stride, y_bias, states, entry, slots, pos,       \
                         static_cast<__nv_bfloat16*>(out), n_tokens, width, block)
    if (pieces) {
        PL_STEP(8);
    } else {
        PL_STEP(1);
    }
#undef PL_STEP
    PL_CHECK_LAUNCH("linear_step");
    return 0;
}
