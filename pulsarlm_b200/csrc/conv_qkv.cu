// What lies between the q/k/v projection and paged attention in a mixer that filters all three over time:
//
//   u[t] = proj[t] + bias                                          q, k and v channels
//   y[t] = sum_j w[j, :] * u[t - (taps - 1) + j]                    per channel; zeros before position 0
//   q    = y_q * (1 + coef * ln(floor((pos + 1) / every) + 1))      the query's temperature (coef 0: none)
//   q_out[t, head] <- q,   K page <- y_k,   V page <- y_v           rows of a common size, zeros past their own columns
//
// Key and value sizes may differ: all three are written as rows of one size (at least the larger), which is what the
// paged attention kernels know; a product with a zero adds nothing. Earlier inputs of a sequence come from the step's
// own rows where the portion has them and from the request's state slot where not (the slot holds the last taps - 1
// projected rows, without the bias, as the product wrote them). In a step whose entries bring one token each the slot
// moves on in the same launch (every channel belongs to one thread); otherwise a second kernel moves it on afterwards
// (pl_filter_state). Everything is fp32 with one rounding on each store, the taps in order from the oldest.
//
// A thread takes a piece of a row (16 bytes where sizes and addresses allow, else one element) for a few
// neighbouring tokens; with few taps (known to the compiler) the earlier inputs stay in registers from token to token.
#include "row_piece.cuh"

namespace {

struct ConvQkvParams {
    const void* proj;
    int64_t row_stride;
    const float* bias;    // [channels] or nullptr
    const float* weight;  // [taps, channels]
    void* state;          // [slots, taps - 1, channels]
    const int32_t* slots;
    int taps;
    int channels;  // columns of proj that the state keeps (q, k, v and what pads them apart)
    int update_state;
    float temp_coef;
    int temp_every;
    const int32_t* pos;
    const int32_t* entry;
    const int32_t* table;
    int table_width;
    void* q_out;
    void* k_pool;
    void* v_pool;
    int64_t page_stride, head_stride;
    int page_size, n_pages;
    int n_tokens, n_heads, n_kv, dim, vdim, row;
    int k_col, v_col;  // first column of k and of v
    int tokens_per_block;
    int32_t* status;
};

constexpr int kThreads = 128;

// TAPS > 0: that many taps, known to the compiler; 0: p.taps.
template <typename scalar_t, int PER, int TAPS>
__global__ void __launch_bounds__(kThreads) conv_qkv_write_kernel(const ConvQkvParams p) {
    using Piece = RowPiece<scalar_t, PER>;
    constexpr int kReach = TAPS > 1 ? TAPS - 1 : 1;
    pl_grid_trigger();
    const int taps = TAPS > 0 ? TAPS : p.taps, reach = taps - 1;
    const int per_row = p.row / PER;
    const int piece = blockIdx.y * kThreads + threadIdx.x;
    const int slot = piece / per_row, d = (piece - slot * per_row) * PER;
    if (slot >= p.n_heads + 2 * p.n_kv) {
        return;
    }
    const bool is_q = slot < p.n_heads, is_v = slot >= p.n_heads + p.n_kv;
    const int head = is_q ? slot : is_v ? slot - p.n_heads - p.n_kv : slot - p.n_heads;
    const int size = is_v ? p.vdim : p.dim;
    const bool live = d < size;  // (else a piece of the row's zeros)
    const int col = (is_q ? 0 : is_v ? p.v_col : p.k_col) + head * size + d;
    const scalar_t* proj = static_cast<const scalar_t*>(p.proj);
    float b[PER], w[TAPS > 0 ? TAPS : 1][PER];  // (weights: read before the wait on earlier kernels)
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        b[i] = 0.0f;
    }
    if (live) {
        if (p.bias != nullptr) {
            pl_floats<PER>(p.bias + col, b);
        }
        if constexpr (TAPS > 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                pl_floats<PER>(p.weight + static_cast<int64_t>(j) * p.channels + col, w[j]);
            }
        }
    }
    pl_grid_wait();
    const int t0 = blockIdx.x * p.tokens_per_block, t1 = min(t0 + p.tokens_per_block, p.n_tokens);
    float window[kReach][PER];  // (TAPS > 0) the inputs before the token at hand, oldest first, with the bias
    int last_entry = -1;
    for (int t = t0; t < t1; ++t) {
        const int e = p.entry[t], at = p.pos[t];
        float y[PER];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            y[i] = 0.0f;
        }
        if (live) {
            const typename Piece::Raw own = Piece::get(proj + static_cast<int64_t>(t) * p.row_stride + col);
            scalar_t* old = static_cast<scalar_t*>(p.state) + static_cast<int64_t>(p.slots[e]) * reach * p.channels + col;
            const bool fresh = TAPS == 0 || e != last_entry;  // nothing of this sequence in registers
            int inside = 0;  // rows before this one that belong to the same sequence (up to `reach`)
            if (fresh) {
                while (inside < reach && t - inside - 1 >= 0 && p.entry[t - inside - 1] == e) {
                    ++inside;
                }
            }
            auto earlier = [&](int back) {
                return back <= inside ? Piece::get(proj + static_cast<int64_t>(t - back) * p.row_stride + col)
                                      : Piece::get(old + static_cast<int64_t>(reach - (back - inside)) * p.channels);
            };
            float v[PER];
            if constexpr (TAPS > 0) {
                if (fresh) {
                    typename Piece::Raw raw[kReach];
#pragma unroll
                    for (int j = 0; j < TAPS - 1; ++j) {
                        raw[j] = earlier(TAPS - 1 - j);
                    }
#pragma unroll
                    for (int j = 0; j < TAPS - 1; ++j) {
                        Piece::floats(raw[j], v);
#pragma unroll
                        for (int i = 0; i < PER; ++i) {
                            window[j][i] = at - (TAPS - 1 - j) >= 0 ? v[i] + b[i] : 0.0f;
                        }
                    }
                    if (p.update_state) {
#pragma unroll
                        for (int j = 0; j < TAPS - 1; ++j) {
                            Piece::put(old + static_cast<int64_t>(j) * p.channels, j + 1 < TAPS - 1 ? raw[j + 1] : own);
                        }
                    }
                }
                Piece::floats(own, v);
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    v[i] += b[i];
#pragma unroll
                    for (int j = 0; j < TAPS - 1; ++j) {
                        y[i] = fmaf(w[j][i], window[j][i], y[i]);
                    }
                    y[i] = fmaf(w[TAPS - 1][i], v[i], y[i]);
#pragma unroll
                    for (int j = 0; j + 1 < TAPS - 1; ++j) {
                        window[j][i] = window[j + 1][i];
                    }
                    window[kReach - 1][i] = v[i];
                }
            } else {
                for (int j = 0; j < taps; ++j) {
                    const int back = reach - j;
                    const typename Piece::Raw raw = back == 0 ? own : earlier(back);
                    if (at - back >= 0) {
                        float wj[PER];
                        pl_floats<PER>(p.weight + static_cast<int64_t>(j) * p.channels + col, wj);
                        Piece::floats(raw, v);
#pragma unroll
                        for (int i = 0; i < PER; ++i) {
                            y[i] = fmaf(wj[i], v[i] + b[i], y[i]);
                        }
                    }
                    if (p.update_state && j > 0) {
                        // (one token per entry: every earlier input is a slot's row, read before it is written)
                        Piece::put(old + static_cast<int64_t>(j - 1) * p.channels, raw);
                    }
                }
            }
            last_entry = e;
        }
        if (is_q) {
            if (p.temp_coef != 0.0f) {
                const float steps = static_cast<float>((at + 1) / p.temp_every);
                const float factor = 1.0f + p.temp_coef * logf(steps + 1.0f);
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    y[i] *= factor;
                }
            }
            Piece::put(static_cast<scalar_t*>(p.q_out) + (static_cast<int64_t>(t) * p.n_heads + head) * p.row + d,
                       Piece::pack(y));
            continue;
        }
        const int page = p.table[static_cast<int64_t>(e) * p.table_width + at / p.page_size];
        if (page < 0 || page >= p.n_pages) {
            if (d == 0 && p.status != nullptr) {
                atomicOr(p.status, 2);
            }
            continue;
        }
        scalar_t* pool = static_cast<scalar_t*>(is_v ? p.v_pool : p.k_pool);
        Piece::put(pool + page * p.page_stride + head * p.head_stride + static_cast<int64_t>(at % p.page_size) * p.row + d,
                   Piece::pack(y));
    }
}

// The slots after the step, one block row per entry: row j becomes the input `taps - 1 - j` places before the next token,
// from the step's rows or, for a portion shorter than that, moved up inside the slot (a thread owns a piece of every
// row and walks them upwards, so it reads a row before it writes it).
template <typename scalar_t, int PER>
__global__ void __launch_bounds__(kThreads) filter_state_kernel(
        const scalar_t* __restrict__ proj, int64_t row_stride, const int32_t* __restrict__ first,
        const int32_t* __restrict__ count, const int32_t* __restrict__ slots, scalar_t* __restrict__ state, int reach,
        int channels) {
    using Piece = RowPiece<scalar_t, PER>;
    pl_grid_trigger();
    pl_grid_wait();
    const int c = (blockIdx.x * kThreads + threadIdx.x) * PER;
    if (c >= channels) {
        return;
    }
    const int e = blockIdx.y, n = count[e];
    scalar_t* mine = state + static_cast<int64_t>(slots[e]) * reach * channels + c;
    const scalar_t* rows = proj + static_cast<int64_t>(first[e]) * row_stride + c;
    for (int j = 0; j < reach; ++j) {
        const int at = n - reach + j;  // among the portion's rows
        Piece::put(mine + static_cast<int64_t>(j) * channels,
                   at >= 0 ? Piece::get(rows + at * row_stride) : Piece::get(mine + static_cast<int64_t>(n + j) * channels));
    }
}

template <typename scalar_t, int PER>
void launch(const ConvQkvParams& p, cudaStream_t stream) {
    const int pieces = (p.n_heads + 2 * p.n_kv) * (p.row / PER);
    const dim3 grid((p.n_tokens + p.tokens_per_block - 1) / p.tokens_per_block, (pieces + kThreads - 1) / kThreads);
    switch (p.taps) {
        case 1: pl_launch_overlapped(conv_qkv_write_kernel<scalar_t, PER, 1>, grid, dim3(kThreads), 0, stream, p); break;
        case 2: pl_launch_overlapped(conv_qkv_write_kernel<scalar_t, PER, 2>, grid, dim3(kThreads), 0, stream, p); break;
        case 3: pl_launch_overlapped(conv_qkv_write_kernel<scalar_t, PER, 3>, grid, dim3(kThreads), 0, stream, p); break;
        case 4: pl_launch_overlapped(conv_qkv_write_kernel<scalar_t, PER, 4>, grid, dim3(kThreads), 0, stream, p); break;
        default: pl_launch_overlapped(conv_qkv_write_kernel<scalar_t, PER, 0>, grid, dim3(kThreads), 0, stream, p); break;
    }
}

}  // namespace

// proj [T, >= channels] (row_stride elements between rows): q [n_heads * dim] from column 0, k [n_kv * dim] from
// column k_col, v [n_kv * vdim] from column v_col, all below `channels`; bias fp32 [channels] (may be nullptr); weight
// fp32 [taps, channels] (the last row the current token's); state [slots, taps - 1, channels]; q_out [T, n_heads, row]
// dense; pools [pages, n_kv, page_size, row]; row >= dim, vdim. update_state != 0: every entry brings one token and
// its slot moves on here. temp_coef, temp_every: see above.
PL_API int pl_conv_qkv_write(const void* proj, int64_t row_stride, const float* bias, const float* weight, int taps,
                             void* state, const int32_t* slots, int channels, int update_state, float temp_coef,
                             int temp_every, const int32_t* pos, const int32_t* entry, const int32_t* table,
                             int table_width, void* q_out, void* k_pool, void* v_pool, int64_t page_stride,
                             int64_t head_stride, int page_size, int n_pages, int n_tokens, int n_heads, int n_kv, int dim,
                             int vdim, int row, int k_col, int v_col, int dtype, int32_t* status, cudaStream_t stream) {
    PL_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv > 0 && dim > 0 && vdim > 0 && page_size > 0 && row >= dim && row >= vdim,
               "conv_qkv_write: bad sizes tokens=%d heads=%d kv_heads=%d dim=%d vdim=%d row=%d page=%d", n_tokens, n_heads,
               n_kv, dim, vdim, row, page_size);
    PL_REQUIRE(taps >= 1 && taps <= 16 && weight != nullptr && slots != nullptr && (taps == 1 || state != nullptr),
               "conv_qkv_write: %d taps (1 to 16) need their weights and state", taps);
    PL_REQUIRE(k_col >= n_heads * dim && v_col >= k_col + n_kv * dim && channels >= v_col + n_kv * vdim &&
                   row_stride >= channels,
               "conv_qkv_write: columns k=%d v=%d of %d do not hold the heads", k_col, v_col, channels);
    PL_REQUIRE(temp_coef == 0.0f || temp_every > 0, "conv_qkv_write: a temperature needs a positive step, not %d", temp_every);
    if (n_tokens == 0) {
        return 0;
    }
    ConvQkvParams p;
    p.proj = proj;
    p.row_stride = row_stride;
    p.bias = bias;
    p.weight = weight;
    p.state = state;
    p.slots = slots;
    p.taps = taps;
    p.channels = channels;
    p.update_state = update_state;
    p.temp_coef = temp_coef;
    p.temp_every = temp_every > 0 ? temp_every : 1;
    p.pos = pos;
    p.entry = entry;
    p.table = table;
    p.table_width = table_width;
    p.q_out = q_out;
    p.k_pool = k_pool;
    p.v_pool = v_pool;
    p.page_stride = page_stride;
    p.head_stride = head_stride;
    p.page_size = page_size;
    p.n_pages = n_pages;
    p.n_tokens = n_tokens;
    p.n_heads = n_heads;
    p.n_kv = n_kv;
    p.dim = dim;
    p.vdim = vdim;
    p.row = row;
    p.k_col = k_col;
    p.v_col = v_col;
    p.tokens_per_block = n_tokens > 256 ? 8 : 1;
    p.status = status;
    auto whole = [](const void* ptr) { return reinterpret_cast<uintptr_t>(ptr) % 16 == 0; };
    const int per = dtype == PL_F32 ? 4 : 8;
    const bool pieces = dim % per == 0 && vdim % per == 0 && row % per == 0 && k_col % per == 0 && v_col % per == 0 &&
        channels % per == 0 && row_stride % per == 0 && page_stride % per == 0 && head_stride % per == 0 && whole(proj) &&
        whole(bias) && whole(weight) && whole(state) && whole(q_out) && whole(k_pool) && whole(v_pool);
    if (dtype == PL_F32) {
        pieces ? launch<float, 4>(p, stream) : launch<float, 1>(p, stream);
    } else if (dtype == PL_BF16) {
        pieces ? launch<__nv_bfloat16, 8>(p, stream) : launch<__nv_bfloat16, 1>(p, stream);
    } else {
        return pl_fail(2, "conv_qkv_write: unknown dtype code %d", dtype);
    }
    PL_CHECK_LAUNCH("conv_qkv_write");
    return 0;
}

// Brings every entry's slot of the state [slots, taps - 1, channels] up to date with the step's rows (run after
// pl_conv_qkv_write has read the old slots): first, count int32 [entries], the row of each entry's first token and how
// many it brings.
PL_API int pl_filter_state(const void* proj, int64_t row_stride, const int32_t* first, const int32_t* count,
                           const int32_t* slots, void* state, int n_entries, int channels, int taps, int dtype,
                           cudaStream_t stream) {
    PL_REQUIRE(n_entries >= 0 && n_entries <= 65535 && channels > 0 && taps >= 1 && row_stride >= channels,
               "filter_state: bad sizes entries=%d channels=%d taps=%d", n_entries, channels, taps);
    if (n_entries == 0 || taps == 1) {
        return 0;
    }
    const int per = dtype == PL_F32 ? 4 : 8;
    const bool pieces = channels % per == 0 && row_stride % per == 0 &&
        ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(state)) & 15) == 0;
    const int lanes = pieces ? channels / per : channels;
    const dim3 grid((lanes + kThreads - 1) / kThreads, n_entries);
#define PL_FILTER_STATE(S, PER)                                                                                       \
    pl_launch_overlapped(filter_state_kernel<S, PER>, grid, dim3(kThreads), 0, stream, static_cast<const S*>(proj),   \
                         row_stride, first, count, slots, static_cast<S*>(state), taps - 1, channels)
    if (dtype == PL_F32) {
        if (pieces) { PL_FILTER_STATE(float, 4); } else { PL_FILTER_STATE(float, 1); }
    } else if (dtype == PL_BF16) {
        if (pieces) { PL_FILTER_STATE(__nv_bfloat16, 8); } else { PL_FILTER_STATE(__nv_bfloat16, 1); }
    } else {
        return pl_fail(2, "filter_state: unknown dtype code %d", dtype);
    }
#undef PL_FILTER_STATE
    PL_CHECK_LAUNCH("filter_state");
    return 0;
}
