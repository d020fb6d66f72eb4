// A matrix memory with exponential gates (the mLSTM recurrence), per head a state S [dim, vdim], a normaliser n [dim]
// and the stabiliser m, all zero at a sequence's start:
//
//   i = cap tanh((i_logit + i_bias) / cap),  f = logsigmoid(cap tanh((f_logit + f_bias) / cap))
//   m' = max(f + m, i);  S = exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone;  m = m'
//   o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)          q times `q_scale`
//   out = o / sqrt(mean(o^2) + eps) * norm * sigmoid(g)       the mean over the head's vdim
//
// A request's slot holds, head by head, [S | n | m | padding to a multiple of four] in fp32 (`head_floats`). Gates,
// exponentials, state, denominators and the per-head norm are fp32. Three ways through a step:
//
// * walk (every shape, both dtypes; the float32 engine's only one): a CTA per (block of columns, head, entry) walks the
//   entry's tokens one by one, a column of the state in the registers of four neighbouring lanes; n is one more column
//   (its values are all 1) and its product with q is the denominator's. A second kernel norms, gates and stores, and moves
//   m on (every CTA of the walk reads the old one). The order of additions is fixed by the sizes: a cut changes no bit.
// * chunks (bfloat16 prompt portions): 64 tokens at a time. With b_t the running sum of f inside a chunk and m_0, S_0, n_0
//   what enters it: m_t = b_t + max(m_0, max_{s <= t} (i_s - b_s)) and
//       S_t = exp(b_t + m_0 - m_t) S_0 + sum_{s <= t} exp(b_t - b_s + i_s - m_t) k_s v_s^T.
//   sums: every chunk's own sum at its end, relative to its own largest exponent; chain: an element of [S | n] per thread
//   goes through the chunks in order and leaves what enters each chunk in the place of its sum; outputs: scores q k^T,
//   their weights, the product with the values and with S_0, the norm and the gate. Products run on bfloat16 tensor cores
//   with fp32 accumulators; a factor that is fp32 by nature (the state, weighted values, weighted scores) goes in as
//   three bfloat16 terms, whose sum carries all 24 bits of it.
// * step (bfloat16, one token per entry): one launch; a cluster of CTAs shares a (token, head) by columns, forms the gate
//   logits itself in fp32 (rows of the two gate projections), reads and writes the state once and norms across the cluster.
#include "cluster_helpers.cuh"
#include "mma_helpers.cuh"

namespace {

__host__ __device__ __forceinline__ int64_t head_floats(int dim, int vdim) {
    return (static_cast<int64_t>(dim) * vdim + dim + 1 + 3) / 4 * 4;
}

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }

struct MemoryParams {
    const void* q;  // q, k [T, heads * dim], v and g [T, heads * vdim]: columns of one matrix, rows row_stride elements apart
    const void* k;
    const void* v;
    const void* g;
    int64_t row_stride;
    const float* logits;  // [T, 2 * heads]: input gates, then forget gates, without biases
    const float* i_bias;  // [heads]
    const float* f_bias;
    float cap;
    const float* norm;    // [heads * vdim]
    float eps;
    float q_scale;
    float* states;        // [slots][heads][head_floats]
    const int32_t* first;  // per entry: its first row and how many rows it brings
    const int32_t* count;
    const int32_t* slots;
    int heads, dim, vdim;
};

__device__ __forceinline__ float* head_state(const MemoryParams& p, int slot, int head) {
    return p.states + (static_cast<int64_t>(slot) * p.heads + head) * head_floats(p.dim, p.vdim);
}

// ------------------------------------------------------------------------------------------------ walk
constexpr int kWalkTokens = 16;   // tokens staged at a time
constexpr int kWalkColumns = 32;  // columns of [S | n] per CTA, four lanes each
constexpr int kWalkThreads = 4 * kWalkColumns;

// ROWS rows of its column per lane (dim <= 4 * ROWS). raw [T, heads, vdim + 1]: S^T q and, last, n . q; top [T, heads]: m.
template <typename scalar_t, int ROWS>
__global__ void __launch_bounds__(kWalkThreads) matrix_memory_walk_kernel(const MemoryParams p, float* __restrict__ raw,
                                                                          float* __restrict__ top) {
    extern __shared__ __align__(16) float shared[];
    constexpr int kDim = 4 * ROWS;
    float* q_s = shared;                          // [kWalkTokens][kDim], zeros past dim
    float* k_s = q_s + kWalkTokens * kDim;
    float* v_s = k_s + kWalkTokens * kDim;        // [kWalkTokens][kWalkColumns]
    __shared__ float keep_s[kWalkTokens], add_s[kWalkTokens], i_s[kWalkTokens], f_s[kWalkTokens], m_s[kWalkTokens];
    pl_grid_trigger();
    pl_grid_wait();
    const int head = blockIdx.y, e = blockIdx.z;
    const int c0 = blockIdx.x * kWalkColumns;
    const int column = c0 + (threadIdx.x >> 2), part = threadIdx.x & 3;
    const int first = p.first[e], count = p.count[e];
    float* state = head_state(p, p.slots[e], head);
    const int n_at = p.dim * p.vdim;
    const bool is_n = column == p.vdim, live = column <= p.vdim;
    auto row_of = [&](int r) { return (r >> 2) * 16 + part * 4 + (r & 3); };
    float s[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int d = row_of(r);
        s[r] = live && d < p.dim ? (is_n ? state[n_at + d] : state[static_cast<int64_t>(d) * p.vdim + column]) : 0.0f;
    }
    float m = state[n_at + p.dim];  // (thread 0 walks it)
    const scalar_t* q = static_cast<const scalar_t*>(p.q) + static_cast<int64_t>(head) * p.dim;
    const scalar_t* k = static_cast<const scalar_t*>(p.k) + static_cast<int64_t>(head) * p.dim;
    const scalar_t* v = static_cast<const scalar_t*>(p.v) + static_cast<int64_t>(head) * p.vdim;
    for (int base = 0; base < count; base += kWalkTokens) {
        const int here = min(kWalkTokens, count - base);
        __syncthreads();
        for (int i = threadIdx.x; i < here * kDim; i += kWalkThreads) {
            const int t = i / kDim, d = i % kDim;
            const int64_t at = (first + base + t) * p.row_stride + d;
            q_s[i] = d < p.dim ? pl_load(q + at) * p.q_scale : 0.0f;
            k_s[i] = d < p.dim ? pl_load(k + at) : 0.0f;
        }
        for (int i = threadIdx.x; i < here * kWalkColumns; i += kWalkThreads) {
            const int t = i / kWalkColumns, c = c0 + i % kWalkColumns;
            v_s[i] = c < p.vdim ? pl_load(v + (first + base + t) * p.row_stride + c) : (c == p.vdim ? 1.0f : 0.0f);
        }
        if (threadIdx.x < here) {
            const float* logit = p.logits + static_cast<int64_t>(first + base + threadIdx.x) * 2 * p.heads + head;
            i_s[threadIdx.x] = capped(logit[0] + p.i_bias[head], p.cap);
            f_s[threadIdx.x] = log_sigmoid(capped(logit[p.heads] + p.f_bias[head], p.cap));
        }
        __syncthreads();
        if (threadIdx.x == 0) {
            for (int t = 0; t < here; ++t) {
                const float carried = f_s[t] + m;
                m = fmaxf(carried, i_s[t]);
                keep_s[t] = expf(carried - m);
                add_s[t] = expf(i_s[t] - m);
                m_s[t] = m;
            }
        }
        __syncthreads();
        for (int t = 0; t < here; ++t) {
            const float keep = keep_s[t], add = add_s[t] * v_s[t * kWalkColumns + (threadIdx.x >> 2)];
            float o = 0.0f;
#pragma unroll
            for (int r = 0; r < ROWS; r += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(k_s + t * kDim + row_of(r));
                const float4 q4 = *reinterpret_cast<const float4*>(q_s + t * kDim + row_of(r));
                s[r] = fmaf(add, k4.x, keep * s[r]);
                s[r + 1] = fmaf(add, k4.y, keep * s[r + 1]);
                s[r + 2] = fmaf(add, k4.z, keep * s[r + 2]);
                s[r + 3] = fmaf(add, k4.w, keep * s[r + 3]);
                o = fmaf(q4.x, s[r], o);
                o = fmaf(q4.y, s[r + 1], o);
                o = fmaf(q4.z, s[r + 2], o);
                o = fmaf(q4.w, s[r + 3], o);
            }
            o += __shfl_xor_sync(0xffffffffu, o, 1);
            o += __shfl_xor_sync(0xffffffffu, o, 2);
            if (part == 0 && live) {
                const int64_t at = static_cast<int64_t>(first + base + t) * p.heads + head;
                raw[at * (p.vdim + 1) + column] = o;
                if (is_n) {
                    top[at] = m_s[t];
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
        const int d = row_of(r);
        if (live && d < p.dim) {
            (is_n ? state[n_at + d] : state[static_cast<int64_t>(d) * p.vdim + column]) = s[r];
        }
    }
}

// A warp per (token, head): o, its norm and its gate; the entry's last token moves m on.
template <typename scalar_t>
__global__ void __launch_bounds__(128) matrix_memory_finish_kernel(const MemoryParams p, const float* __restrict__ raw,
                                                                   const float* __restrict__ top,
                                                                   const int32_t* __restrict__ entry,
                                                                   scalar_t* __restrict__ out, int n_tokens) {
    pl_grid_trigger();
    pl_grid_wait();
    const int lane = threadIdx.x & 31;
    const int64_t item = blockIdx.x * 4ll + (threadIdx.x >> 5);
    if (item >= static_cast<int64_t>(n_tokens) * p.heads) {
        return;
    }
    const int t = static_cast<int>(item / p.heads), head = static_cast<int>(item % p.heads);
    const float* row = raw + item * (p.vdim + 1);
    const float m = top[item];
    const float scale = 1.0f / (fmaxf(fabsf(row[p.vdim]), expf(-m)) + 1e-6f);
    float squares = 0.0f;
    for (int c = lane; c < p.vdim; c += 32) {
        const float o = row[c] * scale;
        squares = fmaf(o, o, squares);
    }
    const float inv = 1.0f / sqrtf(pl_warp_sum(squares) / p.vdim + p.eps);
    const scalar_t* g = static_cast<const scalar_t*>(p.g) + t * p.row_stride + static_cast<int64_t>(head) * p.vdim;
    for (int c = lane; c < p.vdim; c += 32) {
        pl_store(out + item * p.vdim + c, row[c] * scale * inv * p.norm[head * p.vdim + c] * sigmoid_f32(pl_load(g + c)));
    }
    const int e = entry[t];
    if (lane == 0 && t == p.first[e] + p.count[e] - 1) {
        head_state(p, p.slots[e], head)[p.dim * p.vdim + p.dim] = m;
    }
}

// ------------------------------------------------------------------------------------------------ chunks
constexpr int kChunk = 64;    // tokens of a chunk
constexpr int kBlock = 64;    // columns of the values per CTA
constexpr int kChunkThreads = 128;
constexpr int kTileBytes = kChunk * 128;  // [64][64] bfloat16
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkParams {
    MemoryParams m;
    const int4* chunks;  // {first row, rows, entry, 1 on the entry's last chunk}
    const int4* spans;   // {first chunk, chunks, entry, 0}
    float* sums;         // [chunks][heads][head_floats]: a chunk's own sum, then what enters it
    float2* ends;        // [chunks][heads]: (sum of f over the chunk, its largest exponent)
    float* starts;       // [chunks][heads]: m at the chunk's start
    __nv_bfloat16* out;  // [T, heads * vdim]
};

// A chunk's gates in shared memory: b[t] the running sum of f, a[t] = i_t - b_t (-inf past the rows). One warp, two
// tokens a lane. Returns the sum of f over the chunk.
__device__ __forceinline__ float chunk_gates(const MemoryParams& p, int row0, int rows, int head, float* b, float* a) {
    const int lane = threadIdx.x & 31;
    float f[2], i[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int t = 2 * lane + u;
        f[u] = 0.0f;
        i[u] = -INFINITY;
        if (t < rows) {
            const float* logit = p.logits + static_cast<int64_t>(row0 + t) * 2 * p.heads + head;
            i[u] = capped(logit[0] + p.i_bias[head], p.cap);
            f[u] = log_sigmoid(capped(logit[p.heads] + p.f_bias[head], p.cap));
        }
    }
    float run = f[0] + f[1];
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
        const float other = __shfl_up_sync(0xffffffffu, run, d);
        run += lane >= d ? other : 0.0f;
    }
    const float b0 = run - f[1];
    b[2 * lane] = b0;
    b[2 * lane + 1] = run;
    a[2 * lane] = i[0] - b0;
    a[2 * lane + 1] = i[1] - run;
    return __shfl_sync(0xffffffffu, run, 31);
}

// x as three bfloat16 numbers whose sum is x to fp32's 24 bits.
__device__ __forceinline__ void three_terms(float x, float& hi, float& mid, float& lo) {
    hi = bf16_round(x);
    const float rest = x - hi;
    mid = bf16_round(rest);
    lo = rest - mid;
}

// Rows [0, rows) of a [64][dim] tile of q or k into shared memory by 16-byte copies (zeros past the rows).
__device__ __forceinline__ void copy_rows(unsigned char* dst, const __nv_bfloat16* src, int64_t row_stride, int rows,
                                          int dim, int row_bytes) {
    const int chunks = dim / 8;
    for (int c = threadIdx.x; c < kChunk * chunks; c += kChunkThreads) {
        const int r = c / chunks, ch = c - r * chunks;
        cp_async_16_or_zero(dst + swizzled(r, ch, row_bytes), src + static_cast<int64_t>(min(r, rows - 1)) * row_stride + ch * 8,
                            r < rows);
    }
}

// Eight values x * w as three bfloat16 terms into chunk `ch` of row r of three [64][64] tiles.
__device__ __forceinline__ void store_terms(unsigned char* tiles, int tile_bytes, int at, const float (&x)[8]) {
    uint32_t hi[4], mid[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        float h0, m0, l0, h1, m1, l1;
        three_terms(x[2 * j], h0, m0, l0);
        three_terms(x[2 * j + 1], h1, m1, l1);
        hi[j] = pack_bf16(h0, h1);
        mid[j] = pack_bf16(m0, m1);
        lo[j] = pack_bf16(l0, l1);
    }
    *reinterpret_cast<uint4*>(tiles + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(tiles + tile_bytes + at) = make_uint4(mid[0], mid[1], mid[2], mid[3]);
    *reinterpret_cast<uint4*>(tiles + 2 * tile_bytes + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
}

__device__ __forceinline__ void unpack8(uint4 raw, float (&x)[8]) {
    const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        x[2 * j] = __uint_as_float(words[j] << 16);
        x[2 * j + 1] = __uint_as_float(words[j] & 0xffff0000u);
    }
}

// Grid (column block, chunk, head): sum_s exp(b_L - b_s + i_s - top) k_s v_s^T over the chunk's rows, top the largest of
// those exponents; column block 0 also sums the keys alone.
__global__ void __launch_bounds__(kChunkThreads) matrix_memory_sums_kernel(const ChunkParams c) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ float b_s[kChunk], a_s[kChunk], w_s[kChunk];
    __shared__ float end_s[2];
    pl_grid_trigger();
    pl_grid_wait();
    const MemoryParams& p = c.m;
    const int4 chunk = c.chunks[blockIdx.y];
    const int row0 = chunk.x, rows = chunk.y, head = blockIdx.z, e0 = blockIdx.x * kBlock;
    const int row_bytes = padded_row_bytes(p.dim);
    unsigned char* k_s = smem;                               // [64][dim]
    unsigned char* v_s = smem + kChunk * row_bytes;          // three [64][64]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    copy_rows(k_s, static_cast<const __nv_bfloat16*>(p.k) + row0 * p.row_stride + static_cast<int64_t>(head) * p.dim,
              p.row_stride, rows, p.dim, row_bytes);
    cp_async_commit();
    const int columns = min(kBlock, p.vdim - e0);
    // this thread's pieces of the values: (row, 16-byte piece) pairs, asked for before the gates are known
    constexpr int kPieces = kChunk * (kBlock / 8) / kChunkThreads;
    uint4 v_raw[kPieces];
#pragma unroll
    for (int u = 0; u < kPieces; ++u) {
        const int idx = threadIdx.x + u * kChunkThreads, r = idx >> 3, ch = idx & 7;
        v_raw[u] = r < rows && ch * 8 < columns
            ? *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.v) + (row0 + r) * p.row_stride +
                                              static_cast<int64_t>(head) * p.vdim + e0 + ch * 8)
            : make_uint4(0u, 0u, 0u, 0u);
    }
    if (warp == 0) {
        const float total = chunk_gates(p, row0, rows, head, b_s, a_s);
        __syncwarp();
        const float top = total + pl_warp_max(fmaxf(a_s[2 * lane], a_s[2 * lane + 1]));
        w_s[2 * lane] = exp2f((total + a_s[2 * lane] - top) * kLog2e);
        w_s[2 * lane + 1] = exp2f((total + a_s[2 * lane + 1] - top) * kLog2e);
        if (lane == 0) {
            end_s[0] = total;
            end_s[1] = top;
        }
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < kPieces; ++u) {
        const int idx = threadIdx.x + u * kChunkThreads, r = idx >> 3, ch = idx & 7;
        float x[8];
        unpack8(v_raw[u], x);
        const float w = w_s[r];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            x[j] *= w;
        }
        store_terms(v_s, kTileBytes, swizzled(r, ch, 128), x);
    }
    cp_async_wait<0>();
    __syncthreads();
    float* sums = c.sums + (static_cast<int64_t>(blockIdx.y) * p.heads + head) * head_floats(p.dim, p.vdim);
    const int mi = lane >> 3, r8 = lane & 7, g = lane >> 2, tig = lane & 3;
    const int n_tiles = p.dim / 16 * 2;  // 16 rows of S x 32 columns
    for (int tile = warp; tile < n_tiles; tile += kChunkThreads / 32) {
        const int d0 = (tile >> 1) * 16, n0 = (tile & 1) * 32;
        if (n0 >= columns) {
            continue;
        }
        float acc[4][4] = {};
#pragma unroll
        for (int ks = 0; ks < kChunk / 16; ++ks) {
            uint32_t ka[4];
            ldmatrix_x4_trans(ka, k_s + swizzled(ks * 16 + (mi >> 1) * 8 + r8, d0 / 8 + (mi & 1), row_bytes));
#pragma unroll
            for (int term = 0; term < 3; ++term) {
#pragma unroll
                for (int np = 0; np < 2; ++np) {
                    uint32_t vb[4];
                    ldmatrix_x4_trans(vb, v_s + term * kTileBytes +
                                              swizzled(ks * 16 + (mi & 1) * 8 + r8, n0 / 8 + 2 * np + (mi >> 1), 128));
                    mma_bf16(acc[2 * np], ka, vb[0], vb[1]);
                    mma_bf16(acc[2 * np + 1], ka, vb[2], vb[3]);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            const int e = n0 + 8 * n + 2 * tig;
            if (e < columns) {
                float* at = sums + static_cast<int64_t>(d0 + g) * p.vdim + e0 + e;
                *reinterpret_cast<float2*>(at) = make_float2(acc[n][0], acc[n][1]);
                *reinterpret_cast<float2*>(at + 8ll * p.vdim) = make_float2(acc[n][2], acc[n][3]);
            }
        }
    }
    if (blockIdx.x == 0) {
        for (int d = threadIdx.x; d < p.dim; d += kChunkThreads) {
            float n = 0.0f;
#pragma unroll 8
            for (int s = 0; s < rows; ++s) {
                n = fmaf(w_s[s], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(
                                     k_s + swizzled(s, d >> 3, row_bytes) + (d & 7) * 2)), n);
            }
            sums[p.dim * p.vdim + d] = n;
        }
        if (threadIdx.x == 0) {
            c.ends[static_cast<int64_t>(blockIdx.y) * p.heads + head] = make_float2(end_s[0], end_s[1]);
        }
    }
}

constexpr int kChainThreads = 128;
constexpr int kChainAhead = 8;

// Grid (four-element pieces of [S | n], head, span): the state through the span's chunks in order. What enters a chunk
// takes the place of its sum; the state after the last chunk goes to the slot (all but m, which every block reads here:
// the outputs' kernel moves it on).
__global__ void __launch_bounds__(kChainThreads) matrix_memory_chain_kernel(const ChunkParams c) {
    pl_grid_trigger();
    pl_grid_wait();
    const MemoryParams& p = c.m;
    const int4 span = c.spans[blockIdx.z];
    const int head = blockIdx.y;
    const int64_t per_head = head_floats(p.dim, p.vdim);
    const int elements = p.dim * p.vdim + p.dim;  // (a multiple of four)
    const int at = (blockIdx.x * kChainThreads + threadIdx.x) * 4;
    float* state = head_state(p, p.slots[span.z], head);
    float m = state[elements];
    const bool live = at < elements;
    float4 s = live ? *reinterpret_cast<const float4*>(state + at) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    for (int base = 0; base < span.y; base += kChainAhead) {
        float4 u[kChainAhead];
        float2 end[kChainAhead];
#pragma unroll
        for (int j = 0; j < kChainAhead; ++j) {
            const int64_t item = static_cast<int64_t>(span.x + min(base + j, span.y - 1)) * p.heads + head;
            u[j] = live ? *reinterpret_cast<const float4*>(c.sums + item * per_head + at) : s;
            end[j] = c.ends[item];
        }
#pragma unroll
        for (int j = 0; j < kChainAhead; ++j) {
            if (base + j < span.y) {
                const int64_t item = static_cast<int64_t>(span.x + base + j) * p.heads + head;
                if (live) {
                    *reinterpret_cast<float4*>(c.sums + item * per_head + at) = s;
                }
                if (at == 0) {
                    c.starts[item] = m;
                }
                const float carried = end[j].x + m;
                m = fmaxf(carried, end[j].y);
                const float keep = expf(carried - m), add = expf(end[j].y - m);
                s.x = fmaf(keep, s.x, add * u[j].x);
                s.y = fmaf(keep, s.y, add * u[j].y);
                s.z = fmaf(keep, s.z, add * u[j].z);
                s.w = fmaf(keep, s.w, add * u[j].w);
            }
        }
    }
    if (live) {
        *reinterpret_cast<float4*>(state + at) = s;
    }
}

// Grid (column block, chunk, head), a cluster over the column blocks (they share the norm): the chunk's outputs.
__global__ void __launch_bounds__(kChunkThreads) matrix_memory_outputs_kernel(const ChunkParams c) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ float b_s[kChunk], a_s[kChunk], m_s[kChunk], qn_s[kChunk];
    __shared__ __align__(16) float n_s[256];  // n_0
    __shared__ float square_s[8][kChunk];  // [rank][row]
    if (gridDim.x > 1) {
        cluster_arrive_all();  // "this CTA runs": waited for before anything is stored into a peer
    }
    pl_grid_trigger();
    pl_grid_wait();
    const MemoryParams& p = c.m;
    const int4 chunk = c.chunks[blockIdx.y];
    const int row0 = chunk.x, rows = chunk.y, head = blockIdx.z, rank = blockIdx.x, ranks = gridDim.x;
    const int e0 = rank * kBlock, columns = min(kBlock, p.vdim - e0);
    const int row_bytes = padded_row_bytes(p.dim);
    const int s_bytes = p.dim * 128;                    // [dim][64] bfloat16
    unsigned char* q_s = smem;                          // [64][dim]
    unsigned char* k_s = q_s + kChunk * row_bytes;
    unsigned char* v_s = k_s + kChunk * row_bytes;      // [64][64]
    unsigned char* st_s = v_s + kTileBytes;             // three [dim][64]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int mi = lane >> 3, r8 = lane & 7, g = lane >> 2, tig = lane & 3;
    const int64_t item = static_cast<int64_t>(blockIdx.y) * p.heads + head;
    const int64_t from = row0 * p.row_stride + static_cast<int64_t>(head) * p.dim;
    copy_rows(q_s, static_cast<const __nv_bfloat16*>(p.q) + from, p.row_stride, rows, p.dim, row_bytes);
    copy_rows(k_s, static_cast<const __nv_bfloat16*>(p.k) + from, p.row_stride, rows, p.dim, row_bytes);
    const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(p.v) + row0 * p.row_stride +
        static_cast<int64_t>(head) * p.vdim + e0;
    for (int i = threadIdx.x; i < kChunk * 8; i += kChunkThreads) {
        const int r = i >> 3, ch = i & 7;
        const bool valid = r < rows && ch * 8 < columns;
        cp_async_16_or_zero(v_s + swizzled(r, ch, 128), valid ? v + r * p.row_stride + ch * 8 : v, valid);
    }
    cp_async_commit();
    // the entering state, as three bfloat16 terms
    const float* entering = c.sums + item * head_floats(p.dim, p.vdim);
    const float m0 = c.starts[item];
    if (warp == 0) {
        const float total = chunk_gates(p, row0, rows, head, b_s, a_s);
        __syncwarp();
        // m_t = b_t + max(m_0, max over s <= t of a_s)
        const float first = a_s[2 * lane];
        float best = fmaxf(first, a_s[2 * lane + 1]);
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const float other = __shfl_up_sync(0xffffffffu, best, d);
            best = lane >= d ? fmaxf(best, other) : best;
        }
        const float before = __shfl_up_sync(0xffffffffu, best, 1);
        m_s[2 * lane] = b_s[2 * lane] + fmaxf(m0, lane > 0 ? fmaxf(before, first) : first);
        m_s[2 * lane + 1] = b_s[2 * lane + 1] + fmaxf(m0, best);
        if (lane == 31 && rank == 0 && chunk.w) {
            // (rows past the end count f = 0 and nothing else: the last m is the entry's)
            head_state(p, p.slots[chunk.z], head)[p.dim * p.vdim + p.dim] = total + fmaxf(m0, best);
        }
    }
    for (int d = threadIdx.x * 4; d < p.dim; d += kChunkThreads * 4) {
        *reinterpret_cast<float4*>(n_s + d) = *reinterpret_cast<const float4*>(entering + p.dim * p.vdim + d);
    }
#pragma unroll 4
    for (int i = threadIdx.x; i < p.dim * 8; i += kChunkThreads) {
        const int d = i >> 3, ch = i & 7;
        float x[8] = {};
        if (ch * 8 < columns) {
            const float* src = entering + static_cast<int64_t>(d) * p.vdim + e0 + ch * 8;
            const float4 lo = *reinterpret_cast<const float4*>(src), hi = *reinterpret_cast<const float4*>(src + 4);
            x[0] = lo.x; x[1] = lo.y; x[2] = lo.z; x[3] = lo.w;
            x[4] = hi.x; x[5] = hi.y; x[6] = hi.z; x[7] = hi.w;
        }
        store_terms(st_s, s_bytes, swizzled(d, ch, 128), x);
    }
    cp_async_wait<0>();
    __syncthreads();
    {
        // q . n_0: two threads a row, each every second 16-byte piece
        const int r = threadIdx.x >> 1, half = threadIdx.x & 1;
        float dot = 0.0f;
        for (int ch = half; ch < p.dim / 8; ch += 2) {
            float x[8];
            unpack8(*reinterpret_cast<const uint4*>(q_s + swizzled(r, ch, row_bytes)), x);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                dot = fmaf(x[j], n_s[ch * 8 + j], dot);
            }
        }
        dot += __shfl_xor_sync(0xffffffffu, dot, 1);
        if (half == 0) {
            qn_s[r] = dot;
        }
    }
    __syncthreads();
    const int t_lo = warp * 16 + g, t_hi = t_lo + 8;
    const float r_lo = (b_s[t_lo] - m_s[t_lo]) * kLog2e, r_hi = (b_s[t_hi] - m_s[t_hi]) * kLog2e;
    const float in_lo = exp2f(fmaf(m0, kLog2e, r_lo)) * p.q_scale, in_hi = exp2f(fmaf(m0, kLog2e, r_hi)) * p.q_scale;
    float o[kBlock / 8][4] = {};
    float s[kChunk / 8][4] = {};
    const int dim_steps = p.dim / 16;
    for (int kk = 0; kk < dim_steps; ++kk) {
        uint32_t qa[4];
        ldmatrix_x4(qa, q_s + swizzled(warp * 16 + (mi & 1) * 8 + r8, 2 * kk + (mi >> 1), row_bytes));
        // scores against the keys up to the warp's last row
#pragma unroll
        for (int np = 0; np < kChunk / 16; ++np) {
            if (np <= warp) {
                uint32_t kb[4];
                ldmatrix_x4(kb, k_s + swizzled(np * 16 + (mi >> 1) * 8 + r8, 2 * kk + (mi & 1), row_bytes));
                mma_bf16(s[2 * np], qa, kb[0], kb[1]);
                mma_bf16(s[2 * np + 1], qa, kb[2], kb[3]);
            }
        }
#pragma unroll
        for (int term = 0; term < 3; ++term) {
#pragma unroll
            for (int np = 0; np < kBlock / 16; ++np) {
                uint32_t sb[4];
                ldmatrix_x4_trans(sb, st_s + term * s_bytes +
                                          swizzled(kk * 16 + (mi & 1) * 8 + r8, 2 * np + (mi >> 1), 128));
                mma_bf16(o[2 * np], qa, sb[0], sb[1]);
                mma_bf16(o[2 * np + 1], qa, sb[2], sb[3]);
            }
        }
    }
#pragma unroll
    for (int n = 0; n < kBlock / 8; ++n) {
        o[n][0] *= in_lo;
        o[n][1] *= in_lo;
        o[n][2] *= in_hi;
        o[n][3] *= in_hi;
    }
    // the scores' weights: exp(b_t - m_t + i_s - b_s) for s <= t
    float sum_lo = 0.0f, sum_hi = 0.0f;
#pragma unroll
    for (int n = 0; n < kChunk / 8; ++n) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int key = 8 * n + 2 * tig + j;
            const float a = a_s[key];
            s[n][j] = key <= t_lo ? s[n][j] * (p.q_scale * exp2f(fmaf(a, kLog2e, r_lo))) : 0.0f;
            s[n][2 + j] = key <= t_hi ? s[n][2 + j] * (p.q_scale * exp2f(fmaf(a, kLog2e, r_hi))) : 0.0f;
            sum_lo += s[n][j];
            sum_hi += s[n][2 + j];
        }
    }
    sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 1);
    sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, 2);
    sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 1);
    sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, 2);
#pragma unroll
    for (int ks = 0; ks < kChunk / 16; ++ks) {
        if (ks <= warp) {
            uint32_t pa[3][4];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
#pragma unroll
                for (int pair = 0; pair < 2; ++pair) {
                    float h0, m0_, l0, h1, m1, l1;
                    three_terms(s[2 * ks + half][2 * pair], h0, m0_, l0);
                    three_terms(s[2 * ks + half][2 * pair + 1], h1, m1, l1);
                    pa[0][2 * half + pair] = pack_bf16(h0, h1);
                    pa[1][2 * half + pair] = pack_bf16(m0_, m1);
                    pa[2][2 * half + pair] = pack_bf16(l0, l1);
                }
            }
#pragma unroll
            for (int np = 0; np < kBlock / 16; ++np) {
                uint32_t vb[4];
                ldmatrix_x4_trans(vb, v_s + swizzled(ks * 16 + (mi & 1) * 8 + r8, 2 * np + (mi >> 1), 128));
#pragma unroll
                for (int term = 0; term < 3; ++term) {
                    mma_bf16(o[2 * np], pa[term], vb[0], vb[1]);
                    mma_bf16(o[2 * np + 1], pa[term], vb[2], vb[3]);
                }
            }
        }
    }
    const float inv_lo = 1.0f / (fmaxf(fabsf(fmaf(qn_s[t_lo], in_lo, sum_lo)), expf(-m_s[t_lo])) + 1e-6f);
    const float inv_hi = 1.0f / (fmaxf(fabsf(fmaf(qn_s[t_hi], in_hi, sum_hi)), expf(-m_s[t_hi])) + 1e-6f);
    float sq_lo = 0.0f, sq_hi = 0.0f;
#pragma unroll
    for (int n = 0; n < kBlock / 8; ++n) {
        o[n][0] *= inv_lo;
        o[n][1] *= inv_lo;
        o[n][2] *= inv_hi;
        o[n][3] *= inv_hi;
        sq_lo = fmaf(o[n][0], o[n][0], fmaf(o[n][1], o[n][1], sq_lo));
        sq_hi = fmaf(o[n][2], o[n][2], fmaf(o[n][3], o[n][3], sq_hi));
    }
    sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 1);
    sq_lo += __shfl_xor_sync(0xffffffffu, sq_lo, 2);
    sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 1);
    sq_hi += __shfl_xor_sync(0xffffffffu, sq_hi, 2);
    if (ranks > 1) {
        cluster_wait_all();
        if (tig == 0) {
            for (int peer = 0; peer < ranks; ++peer) {
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(cluster_map(&square_s[rank][t_lo], peer)), "f"(sq_lo)
                             : "memory");
                asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(cluster_map(&square_s[rank][t_hi], peer)), "f"(sq_hi)
                             : "memory");
            }
        }
        cluster_arrive_all();
        cluster_wait_all();
        sq_lo = sq_hi = 0.0f;
        for (int peer = 0; peer < ranks; ++peer) {
            sq_lo += square_s[peer][t_lo];
            sq_hi += square_s[peer][t_hi];
        }
    }
    const float norm_lo = 1.0f / sqrtf(sq_lo / p.vdim + p.eps), norm_hi = 1.0f / sqrtf(sq_hi / p.vdim + p.eps);
    const int64_t out_stride = static_cast<int64_t>(p.heads) * p.vdim;
#pragma unroll
    for (int n = 0; n < kBlock / 8; ++n) {
        const int e = 8 * n + 2 * tig;
        if (e < columns) {
            const int64_t channel = static_cast<int64_t>(head) * p.vdim + e0 + e;
            const float w0 = p.norm[channel], w1 = p.norm[channel + 1];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = half ? t_hi : t_lo;
                if (t < rows) {
                    const __nv_bfloat162 gate = *reinterpret_cast<const __nv_bfloat162*>(
                        static_cast<const __nv_bfloat16*>(p.g) + (row0 + t) * p.row_stride + channel);
                    const float scale = half ? norm_hi : norm_lo;
                    *reinterpret_cast<uint32_t*>(c.out + (row0 + t) * out_stride + channel) =
                        pack_bf16(o[n][2 * half] * scale * w0 * sigmoid_f32(__low2float(gate)),
                                  o[n][2 * half + 1] * scale * w1 * sigmoid_f32(__high2float(gate)));
                }
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ step
constexpr int kStepThreads = 256;

// Grid (column block, head, token), a cluster over the column blocks. `block` columns each (a multiple of four).
__global__ void __launch_bounds__(kStepThreads) matrix_memory_step_kernel(
        const MemoryParams p, const __nv_bfloat16* __restrict__ h, int64_t h_stride, int hidden,
        const __nv_bfloat16* __restrict__ gates, const int32_t* __restrict__ entry, __nv_bfloat16* __restrict__ out,
        int block) {
    extern __shared__ __align__(16) float shared[];
    float* q_s = shared;             // [dim]
    float* k_s = q_s + p.dim;        // [dim]
    float4* part_s = reinterpret_cast<float4*>(shared + (2 * p.dim + 3) / 4 * 4);  // [kStepThreads]
    __shared__ float logit_s[kStepThreads / 32], dot_s[kStepThreads / 32];
    __shared__ float square_s[8];
    if (gridDim.x > 1) {
        cluster_arrive_all();  // "this CTA runs"
    }
    pl_grid_trigger();
    const int rank = blockIdx.x, ranks = gridDim.x, head = blockIdx.y, t = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int e0 = rank * block, columns = min(block, p.vdim - e0);
    // this warp's share of a gate's row: the first pieces are asked for before the wait (weights)
    const __nv_bfloat16* gate_row = gates + static_cast<int64_t>(warp < 4 ? head : p.heads + head) * hidden;
    constexpr int kAhead = 2;
    uint4 ahead[kAhead];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
        const int i = ((warp & 3) + 4 * u) * 256 + lane * 8;
        ahead[u] = i < hidden ? *reinterpret_cast<const uint4*>(gate_row + i) : make_uint4(0u, 0u, 0u, 0u);
    }
    pl_grid_wait();
    float* state = head_state(p, p.slots[entry[t]], head);
    const int groups = (columns + 3) / 4;          // four columns a thread,
    const int row_step = kStepThreads / (block / 4);  // and this many rows of S side by side
    const int group = threadIdx.x % (block / 4), row = threadIdx.x / (block / 4);
    const bool live = group < groups && row < row_step;
    // this thread's first rows of the state
    constexpr int kRows = 8;
    float4 first[kRows];
#pragma unroll
    for (int u = 0; u < kRows; ++u) {
        const int d = row + u * row_step;
        first[u] = live && d < p.dim
            ? *reinterpret_cast<const float4*>(state + static_cast<int64_t>(d) * p.vdim + e0 + group * 4)
            : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    const float m_old = state[p.dim * p.vdim + p.dim];
    const int64_t at = t * p.row_stride + static_cast<int64_t>(head) * p.dim;
    for (int d = threadIdx.x; d < p.dim; d += kStepThreads) {
        q_s[d] = __bfloat162float(static_cast<const __nv_bfloat16*>(p.q)[at + d]) * p.q_scale;
        k_s[d] = __bfloat162float(static_cast<const __nv_bfloat16*>(p.k)[at + d]);
    }
    {
        float dot = 0.0f;
        const __nv_bfloat16* x = h + t * h_stride;
#pragma unroll
        for (int u = 0; u < kAhead; ++u) {
            const int i = ((warp & 3) + 4 * u) * 256 + lane * 8;
            if (i < hidden) {
                float a[8], b[8];
                unpack8(ahead[u], a);
                unpack8(*reinterpret_cast<const uint4*>(x + i), b);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    dot = fmaf(a[j], b[j], dot);
                }
            }
        }
        for (int i = ((warp & 3) + 4 * kAhead) * 256 + lane * 8; i < hidden; i += 1024) {
            float a[8], b[8];
            unpack8(*reinterpret_cast<const uint4*>(gate_row + i), a);
            unpack8(*reinterpret_cast<const uint4*>(x + i), b);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                dot = fmaf(a[j], b[j], dot);
            }
        }
        dot = pl_warp_sum(dot);
        if (lane == 0) {
            logit_s[warp] = dot;
        }
    }
    __syncthreads();
    const float i = capped(logit_s[0] + logit_s[1] + logit_s[2] + logit_s[3] + p.i_bias[head], p.cap);
    const float f = log_sigmoid(capped(logit_s[4] + logit_s[5] + logit_s[6] + logit_s[7] + p.f_bias[head], p.cap));
    const float m = fmaxf(f + m_old, i);
    const float keep = expf(f + m_old - m), add = expf(i - m);
    // n . q, every CTA of the cluster for itself; the first writes n and m once all have read them
    float n_new[2];
    float dot = 0.0f;
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int d = threadIdx.x + u * kStepThreads;
        if (d < p.dim) {
            n_new[u] = fmaf(add, k_s[d], keep * state[p.dim * p.vdim + d]);
            dot = fmaf(n_new[u], q_s[d], dot);
        }
    }
    dot = pl_warp_sum(dot);
    if (lane == 0) {
        dot_s[warp] = dot;
    }
    float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (live) {
        float4 v;
        {
            const float4 raw = pl_load4(static_cast<const __nv_bfloat16*>(p.v) + t * p.row_stride +
                                        static_cast<int64_t>(head) * p.vdim + e0 + group * 4);
            v = make_float4(add * raw.x, add * raw.y, add * raw.z, add * raw.w);
        }
        auto advance = [&](int d, float4 s) {
            const float k = k_s[d], q = q_s[d];
            s.x = fmaf(k, v.x, keep * s.x);
            s.y = fmaf(k, v.y, keep * s.y);
            s.z = fmaf(k, v.z, keep * s.z);
            s.w = fmaf(k, v.w, keep * s.w);
            *reinterpret_cast<float4*>(state + static_cast<int64_t>(d) * p.vdim + e0 + group * 4) = s;
            o.x = fmaf(q, s.x, o.x);
            o.y = fmaf(q, s.y, o.y);
            o.z = fmaf(q, s.z, o.z);
            o.w = fmaf(q, s.w, o.w);
        };
#pragma unroll
        for (int u = 0; u < kRows; ++u) {
            const int d = row + u * row_step;
            if (d < p.dim) {
                advance(d, first[u]);
            }
        }
        for (int d0 = row + kRows * row_step; d0 < p.dim; d0 += kRows * row_step) {
            float4 s[kRows];
#pragma unroll
            for (int u = 0; u < kRows; ++u) {
                const int d = d0 + u * row_step;
                s[u] = d < p.dim ? *reinterpret_cast<const float4*>(state + static_cast<int64_t>(d) * p.vdim + e0 + group * 4)
                                 : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
#pragma unroll
            for (int u = 0; u < kRows; ++u) {
                const int d = d0 + u * row_step;
                if (d < p.dim) {
                    advance(d, s[u]);
                }
            }
        }
    }
    part_s[threadIdx.x] = o;
    __syncthreads();
    float squares = 0.0f;
    const bool mine = threadIdx.x < groups;  // (one thread a group adds up its rows' shares)
    if (mine) {
        float nq = 0.0f;
#pragma unroll
        for (int w = 0; w < kStepThreads / 32; ++w) {
            nq += dot_s[w];
        }
        const float scale = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
        o = part_s[threadIdx.x];
        for (int r = 1; r < row_step; ++r) {
            const float4 part = part_s[r * (block / 4) + threadIdx.x];
            o.x += part.x;
            o.y += part.y;
            o.z += part.z;
            o.w += part.w;
        }
        o.x *= scale;
        o.y *= scale;
        o.z *= scale;
        o.w *= scale;
        squares = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w)));
    }
    squares = pl_warp_sum(squares);
    __syncthreads();
    if (lane == 0) {
        dot_s[warp] = squares;
    }
    __syncthreads();
    squares = 0.0f;
#pragma unroll
    for (int w = 0; w < kStepThreads / 32; ++w) {
        squares += dot_s[w];
    }
    if (ranks > 1) {
        cluster_wait_all();
        if (threadIdx.x < ranks) {
            asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(cluster_map(&square_s[rank], threadIdx.x)), "f"(squares)
                         : "memory");
        }
        cluster_arrive_all();
        cluster_wait_all();
        squares = 0.0f;
        for (int peer = 0; peer < ranks; ++peer) {
            squares += square_s[peer];
        }
    }
    if (mine) {
        const float inv = 1.0f / sqrtf(squares / p.vdim + p.eps);
        const int64_t channel = static_cast<int64_t>(head) * p.vdim + e0 + threadIdx.x * 4;
        const float4 g = pl_load4(static_cast<const __nv_bfloat16*>(p.g) + t * p.row_stride + channel);
        const float4 w = make_float4(p.norm[channel], p.norm[channel + 1], p.norm[channel + 2], p.norm[channel + 3]);
        pl_store4(out + static_cast<int64_t>(t) * p.heads * p.vdim + channel,
                  make_float4(o.x * inv * w.x * sigmoid_f32(g.x), o.y * inv * w.y * sigmoid_f32(g.y),
                              o.z * inv * w.z * sigmoid_f32(g.z), o.w * inv * w.w * sigmoid_f32(g.w)));
    }
    if (rank == 0) {
        // (past the cluster's barrier: every CTA has read n and m)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int d = threadIdx.x + u * kStepThreads;
            if (d < p.dim) {
                state[p.dim * p.vdim + d] = n_new[u];
            }
        }
        if (threadIdx.x == 0) {
            state[p.dim * p.vdim + p.dim] = m;
        }
    }
}

template <typename scalar_t, int ROWS>
int launch_walk(const MemoryParams& p, float* raw, float* top, int n_entries, cudaStream_t stream) {
    constexpr int smem = (2 * kWalkTokens * 4 * ROWS + kWalkTokens * kWalkColumns) * 4;
    if (smem > 48 * 1024) {
        cudaFuncSetAttribute(matrix_memory_walk_kernel<scalar_t, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    }
    const dim3 grid((p.vdim + 1 + kWalkColumns - 1) / kWalkColumns, p.heads, n_entries);
    pl_launch_overlapped(matrix_memory_walk_kernel<scalar_t, ROWS>, grid, dim3(kWalkThreads), smem, stream, p, raw, top);
    PL_CHECK_LAUNCH("matrix_memory_walk");
    return 0;
}

int chunk_smem_sums(int dim) { return kChunk * padded_row_bytes(dim) + 3 * kTileBytes; }
int chunk_smem_outputs(int dim) { return 2 * kChunk * padded_row_bytes(dim) + kTileBytes + 3 * dim * 128; }

template <typename... Params, typename... Args>
cudaError_t launch_cluster(void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, int cluster, cudaStream_t stream,
                           Args... args) {
    cudaLaunchConfig_t config = {};
    config.gridDim = grid;
    config.blockDim = block;
    config.dynamicSmemBytes = smem;
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
    return cudaLaunchKernelEx(&config, kernel, static_cast<Params>(args)...);
}

}  // namespace

// Floats a head keeps per request: [S | n | m | padding].
PL_API int64_t pl_matrix_memory_head_floats(int dim, int vdim) { return head_floats(dim, vdim); }

// Tokens of a chunk, for the caller's chunk lists.
PL_API int pl_matrix_memory_chunk_tokens() { return kChunk; }

// 1 when the chunked form takes bfloat16 portions of this shape (the projections' columns start on 16 bytes each).
PL_API int pl_matrix_memory_chunks_supports(int dim, int vdim, int dtype) {
    return dtype == PL_BF16 && dim % 16 == 0 && dim <= 256 && vdim % 8 == 0 && vdim <= 8 * kBlock;
}

// 1 when the single-token form takes this shape.
PL_API int pl_matrix_memory_step_supports(int dim, int vdim, int hidden, int dtype) {
    return dtype == PL_BF16 && dim <= 2 * kStepThreads && vdim % 4 == 0 && vdim <= 1024 && hidden % 8 == 0;
}

namespace {
int check_sizes(int n_tokens, int heads, int dim, int vdim, float cap) {
    PL_REQUIRE(n_tokens >= 0 && heads > 0 && heads <= 65535 && dim > 0 && vdim > 0 && cap > 0.0f,
               "matrix_memory: bad sizes tokens=%d heads=%d dim=%d vdim=%d cap=%g", n_tokens, heads, dim, vdim,
               static_cast<double>(cap));
    PL_REQUIRE(dim <= 512, "matrix_memory: a key size of %d exceeds 512", dim);
    return 0;
}
}  // namespace

// Walks each entry's rows in order (any shape up to dim 512). q, k, v, g: columns of one matrix with row_stride elements
// between rows; logits fp32 [T, 2 * heads]; states fp32 [slots][heads][head_floats]; raw fp32 [T, heads, vdim + 1] and top
// fp32 [T, heads] are scratch; out [T, heads * vdim].
PL_API int pl_matrix_memory_walk(const void* q, const void* k, const void* v, const void* g, int64_t row_stride,
                                 const float* logits, const float* i_bias, const float* f_bias, float cap,
                                 const float* norm, float eps, float q_scale, float* states, const int32_t* first,
                                 const int32_t* count, const int32_t* slots, const int32_t* entry, float* raw, float* top,
                                 void* out, int n_tokens, int n_entries, int heads, int dim, int vdim, int dtype,
                                 cudaStream_t stream) {
    if (const int code = check_sizes(n_tokens, heads, dim, vdim, cap)) {
        return code;
    }
    PL_REQUIRE(n_entries <= 65535, "matrix_memory: %d entries exceed the grid limit", n_entries);
    if (n_tokens == 0 || n_entries == 0) {
        return 0;
    }
    const MemoryParams p = {q, k, v, g, row_stride, logits, i_bias, f_bias, cap, norm, eps, q_scale, states, first, count,
                            slots, heads, dim, vdim};
    PL_DISPATCH_DTYPE(dtype, "matrix_memory", {
        int code;
        if (dim <= 32) {
            code = launch_walk<scalar_t, 8>(p, raw, top, n_entries, stream);
        } else if (dim <= 64) {
            code = launch_walk<scalar_t, 16>(p, raw, top, n_entries, stream);
        } else if (dim <= 128) {
            code = launch_walk<scalar_t, 32>(p, raw, top, n_entries, stream);
        } else if (dim <= 256) {
            code = launch_walk<scalar_t, 64>(p, raw, top, n_entries, stream);
        } else {
            code = launch_walk<scalar_t, 128>(p, raw, top, n_entries, stream);
        }
        if (code != 0) {
            return code;
        }
        const int64_t warps = static_cast<int64_t>(n_tokens) * heads;
        pl_launch_overlapped(matrix_memory_finish_kernel<scalar_t>, dim3(static_cast<unsigned>((warps + 3) / 4)), dim3(128), 0,
                             stream, p, raw, top, entry, static_cast<scalar_t*>(out), n_tokens);
    });
    PL_CHECK_LAUNCH("matrix_memory_finish");
    return 0;
}

// bfloat16 portions in chunks. chunks: int32 [n_chunks, 4] = {first row, rows (1..64), entry, 1 on the entry's last};
// spans: int32 [n_spans, 4] = {first chunk, chunks, entry, 0}; sums fp32 [n_chunks][heads][head_floats], ends fp32
// [n_chunks][heads][2], starts fp32 [n_chunks][heads]: scratch. Rows no chunk lists are left alone.
PL_API int pl_matrix_memory_chunks(const void* q, const void* k, const void* v, const void* g, int64_t row_stride,
                                   const float* logits, const float* i_bias, const float* f_bias, float cap,
                                   const float* norm, float eps, float q_scale, float* states, const int32_t* slots,
                                   const int32_t* chunks, int n_chunks, const int32_t* spans, int n_spans, float* sums,
                                   float* ends, float* starts, void* out, int heads, int dim, int vdim,
                                   cudaStream_t stream) {
    if (const int code = check_sizes(n_chunks, heads, dim, vdim, cap)) {
        return code;
    }
    PL_REQUIRE(pl_matrix_memory_chunks_supports(dim, vdim, PL_BF16), "matrix_memory_chunks: unsupported shape dim=%d vdim=%d",
               dim, vdim);
    PL_REQUIRE(((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) |
                 reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(chunks) | reinterpret_cast<uintptr_t>(spans) |
                 reinterpret_cast<uintptr_t>(sums) | reinterpret_cast<uintptr_t>(states)) & 15) == 0 && row_stride % 8 == 0,
               "matrix_memory_chunks: operands must start on 16 bytes, rows a multiple of 8 elements apart");
    PL_REQUIRE(n_chunks <= 65535 && n_spans <= 65535, "matrix_memory_chunks: %d chunks exceed the grid limit", n_chunks);
    if (n_chunks == 0 || n_spans == 0) {
        return 0;
    }
    ChunkParams c;
    c.m = {q, k, v, g, row_stride, logits, i_bias, f_bias, cap, norm, eps, q_scale, states, nullptr, nullptr, slots, heads,
           dim, vdim};
    c.chunks = reinterpret_cast<const int4*>(chunks);
    c.spans = reinterpret_cast<const int4*>(spans);
    c.sums = sums;
    c.ends = reinterpret_cast<float2*>(ends);
    c.starts = starts;
    c.out = static_cast<__nv_bfloat16*>(out);
    static bool configured = false;
    if (!configured) {
        cudaFuncSetAttribute(matrix_memory_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem_sums(256));
        cudaFuncSetAttribute(matrix_memory_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             chunk_smem_outputs(256));
        configured = true;
    }
    const int blocks = (vdim + kBlock - 1) / kBlock;
    pl_launch_overlapped(matrix_memory_sums_kernel, dim3(blocks, n_chunks, heads), dim3(kChunkThreads), chunk_smem_sums(dim),
                         stream, c);
    PL_CHECK_LAUNCH("matrix_memory_sums");
    const int pieces = (dim * vdim + dim) / 4;
    pl_launch_overlapped(matrix_memory_chain_kernel, dim3((pieces + kChainThreads - 1) / kChainThreads, heads, n_spans),
                         dim3(kChainThreads), 0, stream, c);
    PL_CHECK_LAUNCH("matrix_memory_chain");
    const cudaError_t err = launch_cluster(matrix_memory_outputs_kernel, dim3(blocks, n_chunks, heads), dim3(kChunkThreads),
                                           chunk_smem_outputs(dim), blocks, stream, c);
    if (err != cudaSuccess) {
        return pl_fail(3, "matrix_memory_outputs: launch failed: %s", cudaGetErrorString(err));
    }
    return 0;
}

// bfloat16, one token per entry, tokens 0 .. n_tokens - 1. h [T, hidden] (rows h_stride apart) and gates [2 * heads, hidden]
// (the input gates' rows, then the forget gates'): the gate logits are formed here.
PL_API int pl_matrix_memory_step(const void* q, const void* k, const void* v, const void* g, int64_t row_stride,
                                 const void* h, int64_t h_stride, int hidden, const void* gates, const float* i_bias,
                                 const float* f_bias, float cap, const float* norm, float eps, float q_scale, float* states,
                                 const int32_t* slots, const int32_t* entry, void* out, int n_tokens, int heads, int dim,
                                 int vdim, cudaStream_t stream) {
    if (const int code = check_sizes(n_tokens, heads, dim, vdim, cap)) {
        return code;
    }
    PL_REQUIRE(pl_matrix_memory_step_supports(dim, vdim, hidden, PL_BF16) && n_tokens <= 65535,
               "matrix_memory_step: unsupported shape tokens=%d dim=%d vdim=%d hidden=%d", n_tokens, dim, vdim, hidden);
    PL_REQUIRE(((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(gates) | reinterpret_cast<uintptr_t>(states)) &
                15) == 0 && h_stride % 8 == 0 &&
                   ((reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(g) | reinterpret_cast<uintptr_t>(out)) & 7) ==
                       0 && row_stride % 4 == 0,
               "matrix_memory_step: operands must be aligned (h, gates and states 16 bytes, v, g and out 8)");
    if (n_tokens == 0) {
        return 0;
    }
    const MemoryParams p = {q, k, v, g, row_stride, nullptr, i_bias, f_bias, cap, norm, eps, q_scale, states, nullptr,
                            nullptr, slots, heads, dim, vdim};
    // About 32 KB of the state per CTA (or as many CTAs as fill the device), at most eight to a (token, head), a block of
    // columns a power of two times four.
    int block = 4;
    while (block < vdim && block < 1024) {
        block *= 2;
    }
    while (block > 32 && (static_cast<int64_t>(block) * dim * 4 > 32 * 1024 || n_tokens * heads * ((vdim + block - 1) / block) < 148) &&
           (vdim + block / 2 - 1) / (block / 2) <= 8) {
        block /= 2;
    }
    const int ranks = (vdim + block - 1) / block;
    const size_t smem = (static_cast<size_t>(2 * dim + 3) / 4 * 4 + 4 * kStepThreads) * sizeof(float);
    const cudaError_t err = launch_cluster(matrix_memory_step_kernel, dim3(ranks, heads, n_tokens), dim3(kStepThreads), smem,
                                           ranks, stream, p, static_cast<const __nv_bfloat16*>(h), h_stride, hidden,
                                           static_cast<const __nv_bfloat16*>(gates), entry, static_cast<__nv_bfloat16*>(out),
                                           block);
    if (err != cudaSuccess) {
        return pl_fail(3, "matrix_memory_step: launch failed: %s", cudaGetErrorString(err));
    }
    return 0;
}
