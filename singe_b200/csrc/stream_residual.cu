// The residual of decoders that carry several streams instead of one: a sublayer reads one blend of them, and its output and
// a blend of the old streams make the new ones,
//     u = sum_s in[s] x_s,     x'_t = sum_s mix[s, t] x_s + out[t] y.
// One launch between two sublayers takes the output y of the one before into the streams and hands rms_norm(u) * weight to the
// one after; the first launch of a step fills the streams from the embedding table instead.
//
// y may be the scaled sum of two outputs side by side in one row, each RMS-normed over the width with a weight of its own:
// y = scale * (rms_norm(left) * w_left + rms_norm(right) * w_right), in f32 from the projections on.
//
// Streams, blends and norms are f32; T is the type of the sublayers' outputs, the norm weights, the table and the normed row.
// One CTA per row; the streams are read and written once.
#include "row_pack.cuh"

namespace singe {
namespace {

constexpr int kMaxStreams = 16;

struct StreamStep {
    float *streams;          // [rows, count, width]
    const void *delta;       // nullptr: nothing is taken in
    long long delta_stride;
    int parts;               // 1: delta is y; 2: delta holds two outputs side by side, ...
    int second_at;           // ... the second from this column on
    const void *part_weights[2];
    float part_scale;
    const float *mix, *out;  // [count, count] (from, to), [count]: of the sublayer whose output is taken in
    const float *in;         // [count]: of the sublayer that reads next
    int count;
    int store;               // 0: the new streams are not needed any more
    const void *table;       // nullptr, or the streams start as rows ids[row] of the table [vocab, width]
    const long long *ids;
    long long vocab;
    void *normed;            // nullptr: only the streams are brought up to date
    long long normed_stride;
    const void *weight;
    float normed_scale;
    int width;
    float eps;
    uint32_t *status;
};

// S > 0: that many streams, held in registers; S == 0: any number up to kMaxStreams.  The blend the next sublayer reads waits in
// shared memory between the pass over the streams and the norm.
template <typename T, int VEC, int S>
__global__ void __launch_bounds__(kNormThreads, 1) stream_step_kernel(const StreamStep p) {
    grid_launch_dependents();
    constexpr int kRoom = S > 0 ? S : kMaxStreams;
    extern __shared__ __align__(16) float blend[];  // [width]
    __shared__ float scratch[32];
    __shared__ float factors[kMaxStreams * kMaxStreams + 2 * kMaxStreams];
    const int count = S > 0 ? S : p.count;
    float *mix = factors, *out = factors + count * count, *in = out + count;
    // the blends are weights: they do not wait for the kernel before
    for (int i = threadIdx.x; i < count * count; i += blockDim.x) mix[i] = p.delta != nullptr ? p.mix[i] : 0.0f;
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
        out[i] = p.delta != nullptr ? p.out[i] : 0.0f;
        in[i] = p.in != nullptr ? p.in[i] : 1.0f;
    }
    grid_dependency_wait();
    __syncthreads();
    const size_t row = blockIdx.x;
    const int stride = blockDim.x * VEC;
    const T *delta = p.delta == nullptr ? nullptr : static_cast<const T *>(p.delta) + row * p.delta_stride;
    float part_scale[2] = {1.0f, 1.0f};
    if (delta != nullptr && p.parts == 2) {
        float square[2] = {0.0f, 0.0f};
#pragma unroll 4
        for (int c = threadIdx.x * VEC; c < p.width; c += stride) {
#pragma unroll
            for (int side = 0; side < 2; ++side) {
                const Pack<VEC> x = load_pack<VEC>(delta + side * p.second_at + c);
#pragma unroll
                for (int i = 0; i < VEC; ++i) square[side] = square_chain(square[side], x.v[i]);
            }
        }
#pragma unroll
        for (int side = 0; side < 2; ++side) {
            part_scale[side] = p.part_scale / sqrtf(cta_sum(square[side], scratch) / static_cast<float>(p.width) + p.eps);
        }
    }
    const T *source = nullptr;
    if (p.table != nullptr) {
        long long id = p.ids[row];
        if (id < 0) id += p.vocab;
        const bool valid = id >= 0 && id < p.vocab;
        if (!valid && threadIdx.x == 0) report_status(p.status, kStatusIndexOutOfBounds);
        source = static_cast<const T *>(p.table) + static_cast<size_t>(valid ? id : 0) * p.width;
    }
    float *streams = p.streams + row * count * p.width;
    float square = 0.0f;
#pragma unroll 1
    for (int c = threadIdx.x * VEC; c < p.width; c += stride) {
        Pack<VEC> x[kRoom];
        if (source != nullptr) {
            const Pack<VEC> start = load_pack<VEC>(source + c);
            if constexpr (S > 0) {
#pragma unroll
                for (int s = 0; s < S; ++s) x[s] = start;
            } else {
                for (int s = 0; s < count; ++s) x[s] = start;
            }
        } else if constexpr (S > 0) {
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = load_pack<VEC>(streams + static_cast<size_t>(s) * p.width + c);
        } else {
            for (int s = 0; s < count; ++s) x[s] = load_pack<VEC>(streams + static_cast<size_t>(s) * p.width + c);
        }
        Pack<VEC> y = {}, u = {};
        if (delta != nullptr) {
            y = load_pack<VEC>(delta + c);
            if (p.parts == 2) {
                const Pack<VEC> other = load_pack<VEC>(delta + p.second_at + c);
                const Pack<VEC> gain0 = load_pack<VEC>(static_cast<const T *>(p.part_weights[0]) + c);
                const Pack<VEC> gain1 = load_pack<VEC>(static_cast<const T *>(p.part_weights[1]) + c);
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    y.v[i] = fmaf(y.v[i] * part_scale[0], gain0.v[i], other.v[i] * part_scale[1] * gain1.v[i]);
                }
            }
        }
        auto advance = [&](int t) {
            Pack<VEC> next = x[t];
            if (delta != nullptr) {
#pragma unroll
                for (int i = 0; i < VEC; ++i) next.v[i] = out[t] * y.v[i];
                auto add = [&](int s) {
                    const float factor = mix[s * count + t];
#pragma unroll
                    for (int i = 0; i < VEC; ++i) next.v[i] = fmaf(factor, x[s].v[i], next.v[i]);
                };
                if constexpr (S > 0) {
#pragma unroll
                    for (int s = 0; s < S; ++s) add(s);
                } else {
#pragma unroll 1
                    for (int s = 0; s < count; ++s) add(s);
                }
            }
            if (p.store) store_pack<VEC>(streams + static_cast<size_t>(t) * p.width + c, next);
#pragma unroll
            for (int i = 0; i < VEC; ++i) u.v[i] = fmaf(in[t], next.v[i], u.v[i]);
        };
        if constexpr (S > 0) {
#pragma unroll
            for (int t = 0; t < S; ++t) advance(t);
        } else {
#pragma unroll 1
            for (int t = 0; t < count; ++t) advance(t);
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) square = square_chain(square, u.v[i]);
        store_pack<VEC>(blend + c, u);
    }
    if (p.normed == nullptr) return;
    const float scale = 1.0f / sqrtf(cta_sum(square, scratch) / static_cast<float>(p.width) + p.eps);
    T *target = static_cast<T *>(p.normed) + row * p.normed_stride;
    for (int c = threadIdx.x * VEC; c < p.width; c += stride) {
        Pack<VEC> u = load_pack<VEC>(blend + c);
        const Pack<VEC> gain = load_pack<VEC>(static_cast<const T *>(p.weight) + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) u.v[i] = u.v[i] * scale * gain.v[i] * p.normed_scale;
        store_pack<VEC>(target + c, u);
    }
}

template <typename T>
int stream_step(singe_stream_t stream, const StreamStep &p, size_t rows) {
    if (rows == 0 || p.width <= 0 || p.count <= 0 || (p.parts != 1 && p.parts != 2)) return SINGE_ERR_INVALID_LENGTH;
    if (p.delta != nullptr && p.delta_stride < static_cast<long long>(p.width) + (p.parts == 2 ? p.second_at : 0)) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (p.parts == 2 && p.second_at < p.width) return SINGE_ERR_INVALID_LENGTH;
    if (p.normed != nullptr && p.normed_stride < p.width) return SINGE_ERR_INVALID_LENGTH;
    if (p.table != nullptr && (p.vocab <= 0 || p.delta != nullptr)) return SINGE_ERR_INVALID_ARGUMENT;
    if (!fits_i32(rows)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (p.streams == nullptr || (p.table != nullptr && p.ids == nullptr) || (p.normed != nullptr && p.weight == nullptr) ||
        (p.delta != nullptr && (p.mix == nullptr || p.out == nullptr)) ||
        (p.delta != nullptr && p.parts == 2 && (p.part_weights[0] == nullptr || p.part_weights[1] == nullptr))) {
        return SINGE_ERR_NULL_POINTER;
    }
    if (p.count > kMaxStreams) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    const size_t bytes = 4 * sizeof(T);
    const bool wide = p.width % 4 == 0 && p.delta_stride % 4 == 0 && p.second_at % 4 == 0 && p.normed_stride % 4 == 0 &&
                      aligned_to(p.streams, 16) &&
                      aligned_to(p.delta, bytes) && aligned_to(p.normed, bytes) && aligned_to(p.weight, bytes) &&
                      aligned_to(p.table, bytes) && aligned_to(p.part_weights[0], bytes) && aligned_to(p.part_weights[1], bytes);
    const size_t shared = static_cast<size_t>(p.width) * sizeof(float);
    if (shared > 200 * 1024) return SINGE_ERR_UNSUPPORTED_WIDTH;
    auto kernel = wide ? stream_step_kernel<T, 4, 0> : stream_step_kernel<T, 1, 0>;
    int which = wide ? 0 : 1;
#define SINGE_STREAMS(S_)                       \
    if (wide && p.count == S_) {                \
        kernel = stream_step_kernel<T, 4, S_>;  \
        which = 1 + S_;                         \
    }
    SINGE_STREAMS(1)
    SINGE_STREAMS(2)
    SINGE_STREAMS(3)
    SINGE_STREAMS(4)
    SINGE_STREAMS(8)
#undef SINGE_STREAMS
    static int configured[10][kMaxDevices] = {};
    SINGE_CUDA_TRY(ensure_dynamic_shared(kernel, static_cast<int>(shared), configured[which]));
    SINGE_CUDA_TRY(launch_dependent(kernel, dim3(static_cast<unsigned>(rows)),
                                    dim3(norm_threads(static_cast<size_t>(p.width), wide ? 4 : 1)), shared,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p));
    return launch_status();
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

#define SINGE_STREAM_ENTRIES(SUFFIX, T)                                                                                  \
    int singe_stream_embedding_norm_##SUFFIX(singe_stream_t stream, float *streams, const void *table, const int64_t *ids, \
                                             const float *in, void *normed, size_t normed_stride, const void *weight,    \
                                             size_t rows, size_t count, size_t width, size_t vocab, float eps,           \
                                             uint32_t *status) {                                                         \
        if (!fits_i32(width) || !fits_i32(count) || table == nullptr) return SINGE_ERR_INVALID_LENGTH;                   \
        StreamStep p = {};                                                                                               \
        p.streams = streams;                                                                                             \
        p.parts = 1;                                                                                                     \
        p.in = in;                                                                                                       \
        p.count = static_cast<int>(count);                                                                               \
        p.store = 1;                                                                                                     \
        p.table = table;                                                                                                 \
        p.ids = reinterpret_cast<const long long *>(ids);                                                                \
        p.vocab = static_cast<long long>(vocab);                                                                         \
        p.normed = normed;                                                                                               \
        p.normed_stride = static_cast<long long>(normed_stride);                                                         \
        p.weight = weight;                                                                                               \
        p.normed_scale = 1.0f;                                                                                           \
        p.width = static_cast<int>(width);                                                                               \
        p.eps = eps;                                                                                                     \
        p.status = status;                                                                                               \
        return stream_step<T>(stream, p, rows);                                                                          \
    }                                                                                                                    \
    int singe_stream_step_norm_##SUFFIX(                                                                                 \
        singe_stream_t stream, float *streams, const void *delta, size_t delta_stride, int parts, size_t second_at,      \
        const void *left_weight, const void *right_weight, float part_scale, const float *mix, const float *out,         \
        const float *in, int store, void *normed, size_t normed_stride, const void *weight, float normed_scale,          \
        size_t rows, size_t count, size_t width, float eps) {                                                            \
        if (!fits_i32(width) || !fits_i32(count) || !fits_i32(second_at)) return SINGE_ERR_LENGTH_EXCEEDS_I32;                                   \
        if (delta == nullptr) return SINGE_ERR_NULL_POINTER;                                                             \
        StreamStep p = {};                                                                                               \
        p.streams = streams;                                                                                             \
        p.delta = delta;                                                                                                 \
        p.delta_stride = static_cast<long long>(delta_stride);                                                           \
        p.parts = parts;                                                                                                 \
        p.second_at = static_cast<int>(second_at);                                                                       \
        p.part_weights[0] = left_weight;                                                                                 \
        p.part_weights[1] = right_weight;                                                                                \
        p.part_scale = part_scale;                                                                                       \
        p.mix = mix;                                                                                                     \
        p.out = out;                                                                                                     \
        p.in = in;                                                                                                       \
        p.count = static_cast<int>(count);                                                                               \
        p.store = store;                                                                                                 \
        p.normed = normed;                                                                                               \
        p.normed_stride = static_cast<long long>(normed_stride);                                                         \
        p.weight = weight;                                                                                               \
        p.normed_scale = normed_scale;                                                                                   \
        p.width = static_cast<int>(width);                                                                               \
        p.eps = eps;                                                                                                     \
        return stream_step<T>(stream, p, rows);                                                                          \
    }

SINGE_STREAM_ENTRIES(bf16, __nv_bfloat16)
SINGE_STREAM_ENTRIES(f32, float)
#undef SINGE_STREAM_ENTRIES

}  // extern "C"
