// What stands between a mixer's input projection and its attention or recurrence when a short causal convolution over time
// runs on every projected channel:
//     y_t[c] = sum_j taps[j][c] * u_(t - n + 1 + j)[c],     u = projection (+ bias), zero before the sequence's start.
//
//   attention inputs    convolution, RMS norm over all queries' (keys') channels together, rotation of adjacent pairs by
//                       position, then the queries to rows and the keys and values to the paged cache and / or to packed rows
//   recurrence inputs   convolution and silu; the inverse length of every query's and key's head beside them
//   state               the last n - 1 projected rows of each sequence, as projected (the bias is added when they are read)
//
// A step's rows: token t belongs to sequence sequence_of[t], which owns rows [first, first + fresh) and had `context` tokens
// before.  A sequence with fresh == 0 has one idle row: nothing is kept of it.  Sequences with one new token have their state
// brought up to date by the same threads that read it; for the others the state kernel follows.
// Arithmetic is f32.
#include "row_pack.cuh"

namespace singe {
namespace {

constexpr int kConvThreads = 256;
constexpr int kMaxTaps = 16;

struct ConvRows {
    const void *projected;  // [rows, stride]; the convolved columns are the first `span`
    long long stride;
    int span;
    const void *bias;       // [span] or nullptr
    const void *taps;       // [count, span]
    int count;
    void *state;            // [sequences, count - 1, span]
    const int32_t *sequence_of, *first, *fresh, *context;
    int sequences;
};

// Where the taps of one token find their rows (null before the sequence's start) and its sequence's state; false for an idle row.
template <typename T>
__device__ __forceinline__ bool locate_taps(const ConvRows &p, int token, const T **rows, T *&state, int &fresh) {
    const int sequence = p.sequence_of[token];
    state = nullptr;
    fresh = 0;
    if (sequence < 0 || sequence >= p.sequences) return false;
    fresh = p.fresh[sequence];
    if (fresh <= 0) return false;
    const int at = token - p.first[sequence], context = p.context[sequence];
    state = static_cast<T *>(p.state) + static_cast<size_t>(sequence) * (p.count - 1) * p.span;
    for (int j = threadIdx.x; j < p.count; j += blockDim.x) {
        const int from = at - (p.count - 1) + j;  // index among the step's tokens of the sequence
        const T *row = nullptr;
        if (from >= 0) {
            row = static_cast<const T *>(p.projected) + static_cast<long long>(token - (at - from)) * p.stride;
        } else if (context + from >= 0) {
            row = state + static_cast<size_t>(p.count - 1 + from) * p.span;
        }
        rows[j] = row;
    }
    return true;
}

// Columns c .. c + VEC - 1 of the convolution; `shift` moves the sequence's state on by one token.
template <typename T, int VEC>
__device__ __forceinline__ Pack<VEC> convolve(const ConvRows &p, const T *const *rows, T *state, bool shift, int c) {
    Pack<VEC> y, bias;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        y.v[i] = 0.0f;
        bias.v[i] = 0.0f;
    }
    if (p.bias != nullptr) bias = load_pack<VEC>(static_cast<const T *>(p.bias) + c);
    for (int j = 0; j < p.count; ++j) {
        if (rows[j] == nullptr) continue;
        const Pack<VEC> x = load_pack<VEC>(rows[j] + c);
        const Pack<VEC> tap = load_pack<VEC>(static_cast<const T *>(p.taps) + static_cast<size_t>(j) * p.span + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) y.v[i] = fmaf(tap.v[i], x.v[i] + bias.v[i], y.v[i]);
        // slot j - 1 has been read (it is the tap before) and takes what tap j holds
        if (shift && j > 0) store_pack<VEC>(state + static_cast<size_t>(j - 1) * p.span + c, x);
    }
    return y;
}

struct AttentionInputs {
    ConvRows rows;
    int key_at, value_at;                  // columns of the projected row
    int heads, kv_heads, dim, vdim;
    int key_size, value_size;              // of a head in the outputs, padded with zeros
    const void *query_norm, *key_norm;     // [heads * dim], [kv_heads * dim]
    float eps;
    const long long *positions;
    const double *frequencies;             // [pairs]
    int pairs;
    float rotation_scale;
    void *query;                           // [rows, query_stride]
    long long query_stride;
    void *key_cache, *value_cache;         // [pages, page_size, kv_heads, size]
    const long long *write_pages, *write_slots;
    long long pages, page_size;
    const uint8_t *cached;                 // nullptr: every token; else 0 keeps the token out of the cache
    void *packed_keys, *packed_values;     // [packed_count, kv_heads, size], or nullptr
    const int32_t *packed_rows;            // row of each token, negative: none
    long long packed_count;
    uint32_t *status;
};

// One head-padded output row: `size` columns per head, of which `dim` come from `values`.
template <typename T, int VEC, typename Element>
__device__ __forceinline__ void store_heads(T *first, T *second, int heads, int dim, int size, Element element) {
    const int total = heads * size;
    for (int at = threadIdx.x * VEC; at < total; at += blockDim.x * VEC) {
        const int head = at / size, d = at - head * size;
        Pack<VEC> out;
#pragma unroll
        for (int i = 0; i < VEC; ++i) out.v[i] = d + i < dim ? element(head * dim + d + i, d + i) : 0.0f;
        if (first != nullptr) store_pack<VEC>(first + at, out);
        if (second != nullptr) store_pack<VEC>(second + at, out);
    }
}

template <typename T, int VEC, int OUT>
__global__ void __launch_bounds__(kConvThreads) attention_inputs_kernel(const AttentionInputs p) {
    grid_launch_dependents();
    grid_dependency_wait();
    extern __shared__ float shared[];
    float *values = shared;                       // [span]
    float *cosine = values + p.rows.span;         // [pairs]
    float *sine = cosine + p.pairs;
    __shared__ const T *taps[kMaxTaps];
    __shared__ float scratch[32];
    const int token = blockIdx.x;
    T *query = static_cast<T *>(p.query) + token * p.query_stride;
    T *state;
    int fresh;
    if (!locate_taps<T>(p.rows, token, taps, state, fresh)) {
        for (int at = threadIdx.x * OUT; at < p.heads * p.key_size; at += blockDim.x * OUT) {
            Pack<OUT> zero = {};
            store_pack<OUT>(query + at, zero);
        }
        return;
    }
    for (int i = threadIdx.x; i < p.pairs; i += blockDim.x) {
        // the angle modulo a turn in double, so that far positions keep the precision of near ones
        const double angle = static_cast<double>(p.positions[token]) * p.frequencies[i];
        float s, c;
        sincosf(static_cast<float>(angle - 6.283185307179586 * rint(angle * 0.15915494309189535)), &s, &c);
        cosine[i] = c * p.rotation_scale;
        sine[i] = s * p.rotation_scale;
    }
    __syncthreads();
    float square_q = 0.0f, square_k = 0.0f;
    const int queries = p.heads * p.dim, keys = p.kv_heads * p.dim;
    for (int c = threadIdx.x * VEC; c < p.rows.span; c += blockDim.x * VEC) {
        const Pack<VEC> y = convolve<T, VEC>(p.rows, taps, state, fresh == 1, c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const int at = c + i;
            values[at] = y.v[i];
            if (at < queries) square_q = square_chain(square_q, y.v[i]);
            if (at >= p.key_at && at < p.key_at + keys) square_k = square_chain(square_k, y.v[i]);
        }
    }
    const float scale_q = 1.0f / sqrtf(cta_sum(square_q, scratch) / static_cast<float>(queries) + p.eps);
    const float scale_k = 1.0f / sqrtf(cta_sum(square_k, scratch) / static_cast<float>(keys) + p.eps);
    const T *query_norm = static_cast<const T *>(p.query_norm), *key_norm = static_cast<const T *>(p.key_norm);
    auto rotated = [&](const float *x, const T *gain, float scale, int c, int d) -> float {
        const float own = x[c] * scale * to_float<T>(gain[c]);
        if (d >= 2 * p.pairs) return own;
        const int partner = c + ((d & 1) ? -1 : 1), pair = d >> 1;
        const float other = x[partner] * scale * to_float<T>(gain[partner]);
        return (d & 1) ? fmaf(own, cosine[pair], other * sine[pair]) : fmaf(own, cosine[pair], -(other * sine[pair]));
    };
    store_heads<T, OUT>(query, static_cast<T *>(nullptr), p.heads, p.dim, p.key_size,
                        [&](int c, int d) { return rotated(values, query_norm, scale_q, c, d); });
    long long page = p.write_pages[token], slot = p.write_slots[token];
    if (page < 0) page += p.pages;
    if (slot < 0) slot += p.page_size;
    const bool inside = page >= 0 && page < p.pages && slot >= 0 && slot < p.page_size;
    if (!inside && threadIdx.x == 0) report_status(p.status, kStatusIndexOutOfBounds);
    const bool keep = inside && (p.cached == nullptr || p.cached[token] != 0);
    const long long packed = p.packed_rows == nullptr ? -1 : p.packed_rows[token];
    const bool pack = packed >= 0 && packed < p.packed_count;
    const size_t key_width = static_cast<size_t>(p.kv_heads) * p.key_size, value_width = static_cast<size_t>(p.kv_heads) * p.value_size;
    const size_t cell = keep ? static_cast<size_t>(page * p.page_size + slot) : 0;
    store_heads<T, OUT>(keep ? static_cast<T *>(p.key_cache) + cell * key_width : nullptr,
                        pack ? static_cast<T *>(p.packed_keys) + packed * key_width : nullptr, p.kv_heads, p.dim, p.key_size,
                        [&](int c, int d) { return rotated(values + p.key_at, key_norm, scale_k, c, d); });
    store_heads<T, OUT>(keep ? static_cast<T *>(p.value_cache) + cell * value_width : nullptr,
                        pack ? static_cast<T *>(p.packed_values) + packed * value_width : nullptr, p.kv_heads, p.vdim, p.value_size,
                        [&](int c, int) { return values[p.value_at + c]; });
}

struct RecurrenceInputs {
    ConvRows rows;
    int unit_heads, dim;      // the first unit_heads pieces of `dim` columns, ...
    int second_at;            // ... and as many from this column on, get an inverse length
    float eps;
    void *mixed;              // [rows, mixed_stride]: silu of the convolution
    long long mixed_stride;
    float *inverse;           // [rows, 2 * unit_heads]
};

template <typename T, int VEC>
__global__ void __launch_bounds__(kConvThreads) recurrence_inputs_kernel(const RecurrenceInputs p) {
    grid_launch_dependents();
    grid_dependency_wait();
    extern __shared__ float values[];  // [span]
    __shared__ const T *taps[kMaxTaps];
    const int token = blockIdx.x;
    T *mixed = static_cast<T *>(p.mixed) + token * p.mixed_stride;
    float *inverse = p.inverse + static_cast<size_t>(token) * 2 * p.unit_heads;
    T *state;
    int fresh;
    if (!locate_taps<T>(p.rows, token, taps, state, fresh)) {
        // nothing uses an idle row, but a box of neighbouring rows may take it along: it has to be finite
        for (int c = threadIdx.x * VEC; c < p.rows.span; c += blockDim.x * VEC) {
            Pack<VEC> zero = {};
            store_pack<VEC>(mixed + c, zero);
        }
        return;
    }
    __syncthreads();
    for (int c = threadIdx.x * VEC; c < p.rows.span; c += blockDim.x * VEC) {
        Pack<VEC> y = convolve<T, VEC>(p.rows, taps, state, fresh == 1, c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const T rounded = from_float<T>(y.v[i] / (1.0f + expf(-y.v[i])));
            y.v[i] = to_float<T>(rounded);
            values[c + i] = y.v[i];
        }
        store_pack<VEC>(mixed + c, y);
    }
    __syncthreads();
    const int lane = threadIdx.x & 31;
    for (int unit = threadIdx.x >> 5; unit < 2 * p.unit_heads; unit += kConvThreads / 32) {
        const float *x = values + (unit < p.unit_heads ? unit * p.dim : p.second_at + (unit - p.unit_heads) * p.dim);
        float square = 0.0f;
        for (int d = lane; d < p.dim; d += 32) square = square_chain(square, x[d]);
        square = warp_sum(square);
        if (lane == 0) inverse[unit] = 1.0f / sqrtf(square + p.eps);
    }
}

// The state of the sequences with more than one new token: one CTA column per sequence.
template <typename T, int VEC>
__global__ void __launch_bounds__(kConvThreads) conv_state_kernel(const ConvRows p) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int sequence = blockIdx.y;
    const int fresh = p.fresh[sequence];
    if (fresh <= 1) return;
    const int c = (blockIdx.x * kConvThreads + threadIdx.x) * VEC;
    if (c >= p.span) return;
    const T *rows = static_cast<const T *>(p.projected) + static_cast<long long>(p.first[sequence]) * p.stride + c;
    T *state = static_cast<T *>(p.state) + static_cast<size_t>(sequence) * (p.count - 1) * p.span + c;
    for (int j = 0; j < p.count - 1; ++j) {
        const int from = fresh - (p.count - 1) + j;  // negative: an earlier token's slot, still ahead of slot j
        const Pack<VEC> x = from >= 0 ? load_pack<VEC>(rows + from * p.stride)
                                      : load_pack<VEC>(state + static_cast<size_t>(p.count - 1 + from) * p.span);
        store_pack<VEC>(state + static_cast<size_t>(j) * p.span, x);
    }
}

// ---- bf16 in packs of eight columns: what the sizes of real models take ----
//
// A thread owns eight adjacent columns and walks `tile` neighbouring tokens with the taps' rows in registers, so that a row is
// read once however many taps there are.

constexpr int kWideTaps = 4;
constexpr int kTileTokens = 8;

struct Eight {
    float v[8];
};

__device__ __forceinline__ Eight widen(const uint4 &raw) {
    Eight x;
    const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        x.v[2 * i] = __uint_as_float(words[i] << 16);
        x.v[2 * i + 1] = __uint_as_float(words[i] & 0xffff0000u);
    }
    return x;
}

__device__ __forceinline__ uint4 narrow(const Eight &x) {
    return make_uint4(pack2<__nv_bfloat16>(x.v[0], x.v[1]), pack2<__nv_bfloat16>(x.v[2], x.v[3]), pack2<__nv_bfloat16>(x.v[4], x.v[5]),
                      pack2<__nv_bfloat16>(x.v[6], x.v[7]));
}

__device__ __forceinline__ uint4 load_eight(const void *base, long long element) {
    return *reinterpret_cast<const uint4 *>(static_cast<const __nv_bfloat16 *>(base) + element);
}

// The convolution's moving window over one thread's columns.
template <int N>
struct TapWindow {
    uint4 taps[N], bias;
    uint4 past[N > 1 ? N - 1 : 1];  // past[j]: the row j + 1 tokens back
    bool there[N > 1 ? N - 1 : 1];  // false: before the sequence's start
    uint4 ahead;                    // the next row, on its way while this one is worked on
    bool follows;                   // the window stands just before the next token of its sequence

    __device__ __forceinline__ void start(const ConvRows &p, int c) {
#pragma unroll
        for (int j = 0; j < N; ++j) taps[j] = load_eight(p.taps, static_cast<long long>(j) * p.span + c);
        bias = p.bias != nullptr ? load_eight(p.bias, c) : make_uint4(0u, 0u, 0u, 0u);
        follows = false;
    }

    __device__ __forceinline__ void fetch(const ConvRows &p, int c, int token) { ahead = load_eight(p.projected, token * p.stride + c); }

    // The convolution at `token`, a sequence's new token number `at`, whose row is `now`; moves the window on, and with `shift` the
    // sequence's state.
    __device__ __forceinline__ Eight step(const ConvRows &p, int c, const uint4 &now, int token, int sequence, int at, int context,
                                          bool shift) {
        __nv_bfloat16 *state = static_cast<__nv_bfloat16 *>(p.state) + static_cast<size_t>(sequence) * (N - 1) * p.span + c;
        if (!follows || at == 0) {
#pragma unroll
            for (int j = 0; j < N - 1; ++j) {
                const int from = at - 1 - j;
                there[j] = context + from >= 0;
                past[j] = make_uint4(0u, 0u, 0u, 0u);
                if (from >= 0) {
                    past[j] = load_eight(p.projected, (token - 1 - j) * p.stride + c);
                } else if (there[j]) {
                    past[j] = *reinterpret_cast<const uint4 *>(state + static_cast<size_t>(N - 1 + from) * p.span);
                }
            }
        }
        const Eight b = widen(bias);
        Eight y;
        {
            const Eight x = widen(now), w = widen(taps[N - 1]);
#pragma unroll
            for (int i = 0; i < 8; ++i) y.v[i] = w.v[i] * (x.v[i] + b.v[i]);
        }
#pragma unroll
        for (int j = 0; j < N - 1; ++j) {
            if (!there[j]) continue;
            const Eight x = widen(past[j]), w = widen(taps[N - 2 - j]);
#pragma unroll
            for (int i = 0; i < 8; ++i) y.v[i] = fmaf(w.v[i], x.v[i] + b.v[i], y.v[i]);
        }
        if (shift) {
#pragma unroll
            for (int j = 0; j < N - 1; ++j) {
                uint4 *slot = reinterpret_cast<uint4 *>(state + static_cast<size_t>(N - 2 - j) * p.span);
                if (j == 0) {
                    *slot = now;
                } else if (there[j - 1]) {
                    *slot = past[j - 1];
                }
            }
        }
#pragma unroll
        for (int j = N - 2; j > 0; --j) {
            past[j] = past[j - 1];
            there[j] = there[j - 1];
        }
        if (N > 1) {
            past[0] = now;
            there[0] = true;
        }
        follows = true;
        return y;
    }
};

// What a tile's tokens need to know, looked up once for all threads.
struct TileToken {
    int sequence, at, context, fresh;
};

__device__ __forceinline__ void look_up_tile(const ConvRows &p, TileToken *tokens, int token0, int tile, int rows) {
    for (int i = threadIdx.x; i < tile && token0 + i < rows; i += blockDim.x) {
        TileToken t = {p.sequence_of[token0 + i], 0, 0, 0};
        if (t.sequence >= 0 && t.sequence < p.sequences) {
            t.at = token0 + i - p.first[t.sequence];
            t.context = p.context[t.sequence];
            t.fresh = p.fresh[t.sequence];
        }
        tokens[i] = t;
    }
}

// One thread per eight columns of the whole row, so that the norms over all queries and keys meet in the CTA.
template <int N, int THREADS>
__global__ void __launch_bounds__(THREADS, THREADS <= 384 ? 2 : 1) attention_inputs_wide_kernel(const AttentionInputs p, int rows, int tile) {
    using T = __nv_bfloat16;
    grid_launch_dependents();
    __shared__ float2 scratch[2][32];
    __shared__ TileToken tokens[kTileTokens];
    __shared__ long long cells[kTileTokens], packs[kTileTokens];  // rows of the cache and of the packed arrays, or negative
    extern __shared__ float2 turns[];                             // [tile][pairs]: cosine, sine
    const int c = threadIdx.x * 8, warps = (blockDim.x + 31) >> 5;
    const int token0 = blockIdx.x * tile;
    const bool live = c < p.rows.span;
    TapWindow<N> window;
    if (live) window.start(p.rows, c);  // weights: they do not wait for the kernel before
    grid_dependency_wait();
    if (live) window.fetch(p.rows, c, token0);
    look_up_tile(p.rows, tokens, token0, tile, rows);
    for (int i = threadIdx.x; i < tile && token0 + i < rows; i += blockDim.x) {
        long long page = p.write_pages[token0 + i], slot = p.write_slots[token0 + i];
        if (page < 0) page += p.pages;
        if (slot < 0) slot += p.page_size;
        const bool inside = page >= 0 && page < p.pages && slot >= 0 && slot < p.page_size;
        if (!inside) report_status(p.status, kStatusIndexOutOfBounds);
        cells[i] = inside && (p.cached == nullptr || p.cached[token0 + i] != 0) ? page * p.page_size + slot : -1;
        const long long packed = p.packed_rows == nullptr ? -1 : p.packed_rows[token0 + i];
        packs[i] = packed < p.packed_count ? packed : -1;
    }
    for (int i = threadIdx.x; i < tile * p.pairs; i += blockDim.x) {
        const int token = token0 + i / p.pairs;
        if (token >= rows) break;
        // the angle modulo a turn in double, so that far positions keep the precision of near ones
        const double angle = static_cast<double>(p.positions[token]) * p.frequencies[i % p.pairs];
        float sine, cosine;
        sincosf(static_cast<float>(angle - 6.283185307179586 * rint(angle * 0.15915494309189535)), &sine, &cosine);
        turns[i] = make_float2(cosine * p.rotation_scale, sine * p.rotation_scale);
    }
    const int queries = p.heads * p.dim, keys = p.kv_heads * p.dim;
    const bool is_query = c < queries, is_key = c >= p.key_at && c < p.key_at + keys;
    const bool is_value = live && c >= p.value_at;
    // where the columns go within a head-padded row
    const int within = is_query ? c : is_key ? c - p.key_at : c - p.value_at;
    const int head_dim = is_value ? p.vdim : p.dim, size = is_value ? p.value_size : p.key_size;
    const int head = within / head_dim, d = within - head * head_dim;
    const int target = head * size + d;
    Eight gain = {};
    if (is_query) gain = widen(load_eight(p.query_norm, within));
    if (is_key) gain = widen(load_eight(p.key_norm, within));
    const bool normed = is_query || is_key;
    const size_t key_width = static_cast<size_t>(p.kv_heads) * p.key_size, value_width = static_cast<size_t>(p.kv_heads) * p.value_size;
    __syncthreads();
    int parity = 0;
    for (int i = 0; i < tile && token0 + i < rows; ++i) {
        const int token = token0 + i;
        const TileToken now = tokens[i];
        const uint4 row = window.ahead;
        if (live && i + 1 < tile && token + 1 < rows) window.fetch(p.rows, c, token + 1);
        T *query = static_cast<T *>(p.query) + token * p.query_stride;
        if (now.fresh <= 0) {
            for (int at = c; at < p.heads * p.key_size; at += blockDim.x * 8) {
                *reinterpret_cast<uint4 *>(query + at) = make_uint4(0u, 0u, 0u, 0u);
            }
            window.follows = false;
            continue;
        }
        Eight y = {};
        if (live) y = window.step(p.rows, c, row, token, now.sequence, now.at, now.context, now.fresh == 1);
        float square = 0.0f;
#pragma unroll
        for (int e = 0; e < 8; ++e) square = square_chain(square, y.v[e]);
        // sums of the queries' and of the keys' squares
        const float own_q = warp_sum(is_query ? square : 0.0f), own_k = warp_sum(is_key ? square : 0.0f);
        float2 *sums = scratch[parity];  // last used two barriers ago
        parity ^= 1;
        if ((threadIdx.x & 31) == 0) sums[threadIdx.x >> 5] = make_float2(own_q, own_k);
        __syncthreads();
        const float2 part = (threadIdx.x & 31) < warps ? sums[threadIdx.x & 31] : make_float2(0.0f, 0.0f);
        const float total_q = warp_sum(part.x), total_k = warp_sum(part.y);
        const float scale = is_query ? 1.0f / sqrtf(total_q / static_cast<float>(queries) + p.eps)
                                     : 1.0f / sqrtf(total_k / static_cast<float>(keys) + p.eps);
        if (normed) {
#pragma unroll
            for (int e = 0; e < 8; e += 2) {
                float u = y.v[e] * scale * gain.v[e], v = y.v[e + 1] * scale * gain.v[e + 1];
                const int pair = (d + e) >> 1;
                if (pair < p.pairs) {
                    const float2 turn = turns[i * p.pairs + pair];
                    const float turned = fmaf(u, turn.x, -(v * turn.y));
                    v = fmaf(v, turn.x, u * turn.y);
                    u = turned;
                }
                y.v[e] = u;
                y.v[e + 1] = v;
            }
        }
        const uint4 out = narrow(y);
        const bool keep = cells[i] >= 0, pack = packs[i] >= 0;
        const size_t cell = keep ? static_cast<size_t>(cells[i]) : 0, packed = pack ? static_cast<size_t>(packs[i]) : 0;
        T *cached_keys = static_cast<T *>(p.key_cache) + cell * key_width, *cached_values = static_cast<T *>(p.value_cache) + cell * value_width;
        T *packed_keys = static_cast<T *>(p.packed_keys) + packed * key_width;
        T *packed_values = static_cast<T *>(p.packed_values) + packed * value_width;
        if (is_query) *reinterpret_cast<uint4 *>(query + target) = out;
        if (keep && is_key) *reinterpret_cast<uint4 *>(cached_keys + target) = out;
        if (keep && is_value) *reinterpret_cast<uint4 *>(cached_values + target) = out;
        if (pack && is_key) *reinterpret_cast<uint4 *>(packed_keys + target) = out;
        if (pack && is_value) *reinterpret_cast<uint4 *>(packed_values + target) = out;
        // heads narrower than their rows: the rest is zero
        const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
        const int key_rest = (p.key_size - p.dim) / 8, value_rest = (p.value_size - p.vdim) / 8;
        for (int at = threadIdx.x; at < (p.heads + p.kv_heads) * key_rest; at += blockDim.x) {
            const int h = at / key_rest, rest = p.dim + (at - h * key_rest) * 8;
            if (h < p.heads) {
                *reinterpret_cast<uint4 *>(query + h * p.key_size + rest) = zero;
            } else {
                const int place = (h - p.heads) * p.key_size + rest;
                if (keep) *reinterpret_cast<uint4 *>(cached_keys + place) = zero;
                if (pack) *reinterpret_cast<uint4 *>(packed_keys + place) = zero;
            }
        }
        for (int at = threadIdx.x; at < p.kv_heads * value_rest; at += blockDim.x) {
            const int h = at / value_rest, place = h * p.value_size + p.vdim + (at - h * value_rest) * 8;
            if (keep) *reinterpret_cast<uint4 *>(cached_values + place) = zero;
            if (pack) *reinterpret_cast<uint4 *>(packed_values + place) = zero;
        }
    }
}

// blockIdx.y takes a slice of the columns; the lanes of a head are neighbours, a power of two of them.
template <int N>
__global__ void __launch_bounds__(kConvThreads, 4) recurrence_inputs_wide_kernel(const RecurrenceInputs p, int rows, int tile) {
    grid_launch_dependents();
    __shared__ TileToken tokens[kTileTokens];
    const int c = (blockIdx.y * kConvThreads + threadIdx.x) * 8;
    const int token0 = blockIdx.x * tile;
    const bool live = c < p.rows.span;
    TapWindow<N> window;
    if (live) window.start(p.rows, c);
    grid_dependency_wait();
    if (live) window.fetch(p.rows, c, token0);
    look_up_tile(p.rows, tokens, token0, tile, rows);
    __syncthreads();
    const int units = p.unit_heads * p.dim, lanes = p.dim / 8;
    const bool first = c < units, second = c >= p.second_at && c < p.second_at + units;
    const int unit = first ? c / p.dim : p.unit_heads + (c - p.second_at) / p.dim;
    for (int i = 0; i < tile && token0 + i < rows; ++i) {
        const int token = token0 + i;
        const TileToken now = tokens[i];
        const uint4 row = window.ahead;
        if (live && i + 1 < tile && token + 1 < rows) window.fetch(p.rows, c, token + 1);
        uint4 out = make_uint4(0u, 0u, 0u, 0u);
        float square = 0.0f;
        if (now.fresh <= 0) {
            window.follows = false;
        } else if (live) {
            Eight y = window.step(p.rows, c, row, token, now.sequence, now.at, now.context, now.fresh == 1);
#pragma unroll
            for (int e = 0; e < 8; ++e) y.v[e] = __fdividef(y.v[e], 1.0f + __expf(-y.v[e]));
            out = narrow(y);
            const Eight kept = widen(out);
#pragma unroll
            for (int e = 0; e < 8; ++e) square = square_chain(square, kept.v[e]);
        }
        if (live) *reinterpret_cast<uint4 *>(static_cast<__nv_bfloat16 *>(p.mixed) + token * p.mixed_stride + c) = out;
        for (int offset = lanes >> 1; offset > 0; offset >>= 1) square += __shfl_xor_sync(0xffffffffu, square, offset);
        if ((first || second) && now.fresh > 0 && (threadIdx.x & (lanes - 1)) == 0) {
            p.inverse[static_cast<size_t>(token) * 2 * p.unit_heads + unit] = 1.0f / sqrtf(square + p.eps);
        }
    }
}

// Tokens of a tile: one where there are few rows (a decode batch), else enough to read each row once.
int conv_tile(size_t rows, size_t slices) { return rows * slices >= 4 * static_cast<size_t>(device_sm_count()) * kTileTokens ? kTileTokens : 1; }

bool conv_eights(const ConvRows &p) {
    return p.count <= kWideTaps && p.span % 8 == 0 && p.stride % 8 == 0 && aligned_to(p.projected, 16) && aligned_to(p.bias, 16) &&
           aligned_to(p.taps, 16) && aligned_to(p.state, 16);
}

template <int N>
auto attention_inputs_kernel_for(unsigned threads) {
    return threads <= 384 ? attention_inputs_wide_kernel<N, 384>
                          : threads <= 768 ? attention_inputs_wide_kernel<N, 768> : attention_inputs_wide_kernel<N, 1024>;
}

template <int N>
auto recurrence_inputs_kernel_for(unsigned) {
    return recurrence_inputs_wide_kernel<N>;
}

#define SINGE_WIDE_CONV(CHOOSE, GRID, THREADS, SHARED)                                                                     \
    do {                                                                                                                   \
        auto kernel = CHOOSE<1>(THREADS);                                                                                  \
        if (p.rows.count == 2) kernel = CHOOSE<2>(THREADS);                                                                \
        if (p.rows.count == 3) kernel = CHOOSE<3>(THREADS);                                                                \
        if (p.rows.count == 4) kernel = CHOOSE<4>(THREADS);                                                                \
        SINGE_CUDA_TRY(launch_dependent(kernel, GRID, dim3(THREADS), SHARED, static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p, \
                                        static_cast<int>(rows), tile));                                                    \
        return launch_status();                                                                                            \
    } while (0)

int validate(const ConvRows &p, size_t rows) {
    if (rows == 0 || p.span <= 0 || p.count <= 0 || p.sequences <= 0 || p.stride < p.span) return SINGE_ERR_INVALID_LENGTH;
    if (p.count > kMaxTaps) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    if (!fits_i32(rows)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (p.projected == nullptr || p.taps == nullptr || (p.count > 1 && p.state == nullptr) || p.sequence_of == nullptr ||
        p.first == nullptr || p.fresh == nullptr || p.context == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    return SINGE_OK;
}

template <typename T>
bool conv_wide(const ConvRows &p) {
    const size_t bytes = 4 * sizeof(T);
    return p.span % 4 == 0 && p.stride % 4 == 0 && aligned_to(p.projected, bytes) && aligned_to(p.bias, bytes) &&
           aligned_to(p.taps, bytes) && aligned_to(p.state, bytes);
}

ConvRows conv_rows(const void *projected, size_t stride, size_t span, const void *bias, const void *taps, size_t count,
                   void *state, const int32_t *sequence_of, const int32_t *first, const int32_t *fresh,
                   const int32_t *context, size_t sequences) {
    ConvRows p = {};
    p.projected = projected;
    p.stride = static_cast<long long>(stride);
    p.span = static_cast<int>(span);
    p.bias = bias;
    p.taps = taps;
    p.count = static_cast<int>(count);
    p.state = state;
    p.sequence_of = sequence_of;
    p.first = first;
    p.fresh = fresh;
    p.context = context;
    p.sequences = static_cast<int>(sequences);
    return p;
}

template <typename T>
int attention_inputs(singe_stream_t stream, const AttentionInputs &p, size_t rows) {
    SINGE_TRY(validate(p.rows, rows));
    if (p.heads <= 0 || p.kv_heads <= 0 || p.dim <= 0 || p.vdim <= 0 || p.key_size < p.dim || p.value_size < p.vdim ||
        p.pairs < 0 || 2 * p.pairs > p.dim || p.key_at < p.heads * p.dim || p.value_at < p.key_at + p.kv_heads * p.dim ||
        p.rows.span < p.value_at + p.kv_heads * p.vdim || p.query_stride < static_cast<long long>(p.heads) * p.key_size ||
        p.pages <= 0 || p.page_size <= 0) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (p.query_norm == nullptr || p.key_norm == nullptr || p.positions == nullptr || p.query == nullptr ||
        p.key_cache == nullptr || p.value_cache == nullptr || p.write_pages == nullptr || p.write_slots == nullptr ||
        (p.pairs > 0 && p.frequencies == nullptr) ||
        (p.packed_rows != nullptr && (p.packed_keys == nullptr || p.packed_values == nullptr))) {
        return SINGE_ERR_NULL_POINTER;
    }
    if (sizeof(T) == 2 && conv_eights(p.rows) && p.dim % 8 == 0 && p.vdim % 8 == 0 && p.key_at % 8 == 0 && p.value_at % 8 == 0 &&
        p.key_size % 8 == 0 && p.value_size % 8 == 0 && p.query_stride % 8 == 0 && p.rows.span <= 8192 && p.pairs <= 256 &&
        p.key_at == p.heads * p.dim && p.value_at == p.key_at + p.kv_heads * p.dim && p.rows.span == p.value_at + p.kv_heads * p.vdim &&
        aligned_to(p.query, 16) && aligned_to(p.key_cache, 16) && aligned_to(p.value_cache, 16) && aligned_to(p.packed_keys, 16) &&
        aligned_to(p.packed_values, 16) && aligned_to(p.query_norm, 16) && aligned_to(p.key_norm, 16)) {
        const int tile = conv_tile(rows, 1);
        const unsigned threads = static_cast<unsigned>((p.rows.span / 8 + 31) / 32 * 32);
        const dim3 grid(static_cast<unsigned>((rows + tile - 1) / tile));
        SINGE_WIDE_CONV(attention_inputs_kernel_for, grid, threads, static_cast<size_t>(tile) * p.pairs * sizeof(float2));
    }
    const size_t bytes = 4 * sizeof(T);
    const bool out_wide = p.key_size % 4 == 0 && p.value_size % 4 == 0 && p.query_stride % 4 == 0 && aligned_to(p.query, bytes) &&
                          aligned_to(p.key_cache, bytes) && aligned_to(p.value_cache, bytes) &&
                          aligned_to(p.packed_keys, bytes) && aligned_to(p.packed_values, bytes);
    const bool wide = conv_wide<T>(p.rows) && out_wide;
    auto kernel = wide ? attention_inputs_kernel<T, 4, 4> : attention_inputs_kernel<T, 1, 1>;
    static int configured_wide[kMaxDevices] = {0}, configured[kMaxDevices] = {0};
    const size_t shared = (static_cast<size_t>(p.rows.span) + 2 * p.pairs) * sizeof(float);
    if (shared > 220 * 1024) return SINGE_ERR_UNSUPPORTED_WIDTH;
    SINGE_CUDA_TRY(ensure_dynamic_shared(kernel, static_cast<int>(shared), wide ? configured_wide : configured));
    SINGE_CUDA_TRY(launch_dependent(kernel, dim3(static_cast<unsigned>(rows)), dim3(kConvThreads), shared,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p));
    return launch_status();
}

template <typename T>
int recurrence_inputs(singe_stream_t stream, const RecurrenceInputs &p, size_t rows) {
    SINGE_TRY(validate(p.rows, rows));
    if (p.unit_heads <= 0 || p.dim <= 0 || p.second_at < p.unit_heads * p.dim ||
        p.rows.span < p.second_at + p.unit_heads * p.dim || p.mixed_stride < p.rows.span) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (p.mixed == nullptr || p.inverse == nullptr) return SINGE_ERR_NULL_POINTER;
    const int lanes = p.dim / 8;
    if (sizeof(T) == 2 && conv_eights(p.rows) && p.dim % 8 == 0 && lanes <= 32 && (lanes & (lanes - 1)) == 0 &&
        p.second_at == p.unit_heads * p.dim && p.mixed_stride % 8 == 0 && aligned_to(p.mixed, 16)) {
        const size_t slices = (static_cast<size_t>(p.rows.span) / 8 + kConvThreads - 1) / kConvThreads;
        const int tile = conv_tile(rows, slices);
        const dim3 grid(static_cast<unsigned>((rows + tile - 1) / tile), static_cast<unsigned>(slices));
        SINGE_WIDE_CONV(recurrence_inputs_kernel_for, grid, kConvThreads, 0);
    }
    const bool wide = conv_wide<T>(p.rows) && p.mixed_stride % 4 == 0 && aligned_to(p.mixed, 4 * sizeof(T));
    auto kernel = wide ? recurrence_inputs_kernel<T, 4> : recurrence_inputs_kernel<T, 1>;
    static int configured_wide[kMaxDevices] = {0}, configured[kMaxDevices] = {0};
    const size_t shared = static_cast<size_t>(p.rows.span) * sizeof(float);
    if (shared > 220 * 1024) return SINGE_ERR_UNSUPPORTED_WIDTH;
    SINGE_CUDA_TRY(ensure_dynamic_shared(kernel, static_cast<int>(shared), wide ? configured_wide : configured));
    SINGE_CUDA_TRY(launch_dependent(kernel, dim3(static_cast<unsigned>(rows)), dim3(kConvThreads), shared,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p));
    return launch_status();
}

template <typename T>
int conv_state(singe_stream_t stream, const ConvRows &p, size_t rows) {
    SINGE_TRY(validate(p, rows));
    if (p.count == 1) return SINGE_OK;
    if (p.sequences > 65535) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    const bool wide = conv_wide<T>(p);
    const int columns = kConvThreads * (wide ? 4 : 1);
    SINGE_CUDA_TRY(launch_dependent(wide ? conv_state_kernel<T, 4> : conv_state_kernel<T, 1>,
                                    dim3(static_cast<unsigned>((p.span + columns - 1) / columns), static_cast<unsigned>(p.sequences)),
                                    dim3(kConvThreads), 0, static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p));
    return launch_status();
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

#define SINGE_CONV_ENTRIES(SUFFIX, T)                                                                                     \
    int singe_conv_attention_inputs_##SUFFIX(                                                                             \
        singe_stream_t stream, void *query, size_t query_stride, void *key_cache, void *value_cache, void *packed_keys,    \
        void *packed_values, const void *projected, size_t projected_stride, const void *bias, const void *taps,          \
        void *state, const void *query_norm, const void *key_norm, const double *frequencies, size_t pairs,               \
        float rotation_scale, const int64_t *positions, const int32_t *sequence_of, const int32_t *first,                 \
        const int32_t *fresh, const int32_t *context, const int64_t *write_pages, const int64_t *write_slots,             \
        const uint8_t *cached, const int32_t *packed_rows, size_t packed_count, size_t rows, size_t sequences,            \
        size_t tap_count, size_t heads, size_t kv_heads, size_t dim, size_t vdim, size_t key_size, size_t value_size,     \
        size_t key_at, size_t value_at, size_t span, size_t pages, size_t page_size, float eps, uint32_t *status) {       \
        if (!fits_i32(span) || !fits_i32(heads * key_size) || !fits_i32(kv_heads * value_size) || !fits_i32(sequences)) { \
            return SINGE_ERR_LENGTH_EXCEEDS_I32;                                                                          \
        }                                                                                                                 \
        AttentionInputs p = {};                                                                                           \
        p.rows = conv_rows(projected, projected_stride, span, bias, taps, tap_count, state, sequence_of, first, fresh,    \
                           context, sequences);                                                                           \
        p.key_at = static_cast<int>(key_at);                                                                              \
        p.value_at = static_cast<int>(value_at);                                                                          \
        p.heads = static_cast<int>(heads);                                                                                \
        p.kv_heads = static_cast<int>(kv_heads);                                                                          \
        p.dim = static_cast<int>(dim);                                                                                    \
        p.vdim = static_cast<int>(vdim);                                                                                  \
        p.key_size = static_cast<int>(key_size);                                                                          \
        p.value_size = static_cast<int>(value_size);                                                                      \
        p.query_norm = query_norm;                                                                                        \
        p.key_norm = key_norm;                                                                                            \
        p.eps = eps;                                                                                                      \
        p.positions = reinterpret_cast<const long long *>(positions);                                                     \
        p.frequencies = frequencies;                                                                                      \
        p.pairs = static_cast<int>(pairs);                                                                                \
        p.rotation_scale = rotation_scale;                                                                                \
        p.query = query;                                                                                                  \
        p.query_stride = static_cast<long long>(query_stride);                                                            \
        p.key_cache = key_cache;                                                                                          \
        p.value_cache = value_cache;                                                                                      \
        p.write_pages = reinterpret_cast<const long long *>(write_pages);                                                 \
        p.write_slots = reinterpret_cast<const long long *>(write_slots);                                                 \
        p.pages = static_cast<long long>(pages);                                                                          \
        p.page_size = static_cast<long long>(page_size);                                                                  \
        p.cached = cached;                                                                                                \
        p.packed_keys = packed_keys;                                                                                      \
        p.packed_values = packed_values;                                                                                  \
        p.packed_rows = packed_rows;                                                                                      \
        p.packed_count = static_cast<long long>(packed_count);                                                            \
        p.status = status;                                                                                                \
        return attention_inputs<T>(stream, p, rows);                                                                      \
    }                                                                                                                     \
    int singe_conv_recurrence_inputs_##SUFFIX(                                                                            \
        singe_stream_t stream, void *mixed, size_t mixed_stride, float *inverse, const void *projected,                   \
        size_t projected_stride, const void *taps, void *state, const int32_t *sequence_of, const int32_t *first,         \
        const int32_t *fresh, const int32_t *context, size_t rows, size_t sequences, size_t tap_count, size_t unit_heads, \
        size_t dim, size_t second_at, size_t span, float eps) {                                                           \
        if (!fits_i32(span) || !fits_i32(unit_heads * dim) || !fits_i32(sequences)) return SINGE_ERR_LENGTH_EXCEEDS_I32;  \
        RecurrenceInputs p = {};                                                                                          \
        p.rows = conv_rows(projected, projected_stride, span, nullptr, taps, tap_count, state, sequence_of, first, fresh, \
                           context, sequences);                                                                           \
        p.unit_heads = static_cast<int>(unit_heads);                                                                      \
        p.dim = static_cast<int>(dim);                                                                                    \
        p.second_at = static_cast<int>(second_at);                                                                        \
        p.eps = eps;                                                                                                      \
        p.mixed = mixed;                                                                                                  \
        p.mixed_stride = static_cast<long long>(mixed_stride);                                                            \
        p.inverse = inverse;                                                                                              \
        return recurrence_inputs<T>(stream, p, rows);                                                                     \
    }                                                                                                                     \
    int singe_conv_state_##SUFFIX(singe_stream_t stream, const void *projected, size_t projected_stride, void *state,     \
                                  const int32_t *first, const int32_t *fresh, size_t rows, size_t sequences,              \
                                  size_t tap_count, size_t span) {                                                        \
        if (!fits_i32(span) || !fits_i32(sequences)) return SINGE_ERR_LENGTH_EXCEEDS_I32;                                 \
        const ConvRows p = conv_rows(projected, projected_stride, span, nullptr, projected, tap_count, state, first,      \
                                     first, fresh, fresh, sequences);                                                     \
        return conv_state<T>(stream, p, rows);                                                                            \
    }

SINGE_CONV_ENTRIES(bf16, __nv_bfloat16)
SINGE_CONV_ENTRIES(f32, float)
#undef SINGE_CONV_ENTRIES

}  // extern "C"
