// Glue of decoders that keep their residual stream in f32: layer norm with the residual add, embedding lookup with its
// norm, the two RMS norms of a latent projection with the write of the latent into its paged cache, a row gather out
// of that cache, and the argmax over f32 logits.
//
// T is the activation and weight type (bf16, or f32 for a decoder run entirely in 32-bit); arithmetic is f32.
//   layer_norm(x) = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w        (deviations squared, not x^2 - mean^2)
//   rms_norm(x)   = x / sqrt(mean(x^2) + eps) * w
// One CTA per row; a row is read once and kept in registers between the passes.
#include "row_pack.cuh"

namespace singe {
namespace {

// The layer norm of the row held in `x` (kHeldPacks packs per thread), in place.
template <typename T, int VEC>
__device__ __forceinline__ void normalise_held(Pack<VEC> (&x)[kHeldPacks], const T *weight, int width, float eps,
                                               float *scratch) {
    const int stride = blockDim.x * VEC;
    float sum = 0.0f;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        if (threadIdx.x * VEC + h * stride < width) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum += x[h].v[i];
        }
    }
    const float mean = cta_sum(sum, scratch) / static_cast<float>(width);
    float square = 0.0f;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        if (threadIdx.x * VEC + h * stride < width) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                x[h].v[i] -= mean;
                square = square_chain(square, x[h].v[i]);
            }
        }
    }
    const float scale = 1.0f / sqrtf(cta_sum(square, scratch) / static_cast<float>(width) + eps);
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        const int c = threadIdx.x * VEC + h * stride;
        if (c < width) {
            const Pack<VEC> gain = load_pack<VEC>(weight + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) x[h].v[i] = x[h].v[i] * scale * gain.v[i];
        }
    }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kNormThreads)
    embedding_layer_norm_kernel(float *residual, const T *table, const long long *ids, const T *weight, int width,
                                long long vocab, float eps, uint32_t *status) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float scratch[32];
    long long id = ids[blockIdx.x];
    if (id < 0) id += vocab;
    const bool valid = id >= 0 && id < vocab;
    if (!valid && threadIdx.x == 0) report_status(status, kStatusIndexOutOfBounds);
    const T *source = table + static_cast<size_t>(valid ? id : 0) * width;
    Pack<VEC> x[kHeldPacks];
    const int stride = blockDim.x * VEC;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        const int c = threadIdx.x * VEC + h * stride;
        if (c < width) x[h] = load_pack<VEC>(source + c);
    }
    normalise_held<T, VEC>(x, weight, width, eps, scratch);
    float *target = residual + static_cast<size_t>(blockIdx.x) * width;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        const int c = threadIdx.x * VEC + h * stride;
        if (c < width) store_pack<VEC>(target + c, x[h]);
    }
}

// residual += delta (when given), then normed = layer_norm(residual) (when given).
template <typename T, int VEC>
__global__ void __launch_bounds__(kNormThreads)
    add_layer_norm_kernel(float *residual, const T *delta, long long delta_stride, T *normed, long long normed_stride,
                          const T *weight, int width, float eps) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float scratch[32];
    float *row = residual + static_cast<size_t>(blockIdx.x) * width;
    const T *change = delta == nullptr ? nullptr : delta + blockIdx.x * delta_stride;
    Pack<VEC> x[kHeldPacks];
    const int stride = blockDim.x * VEC;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        const int c = threadIdx.x * VEC + h * stride;
        if (c < width) {
            x[h] = load_pack<VEC>(row + c);
            if (change != nullptr) {
                const Pack<VEC> other = load_pack<VEC>(change + c);
#pragma unroll
                for (int i = 0; i < VEC; ++i) x[h].v[i] += other.v[i];
                store_pack<VEC>(row + c, x[h]);
            }
        }
    }
    if (normed == nullptr) return;
    normalise_held<T, VEC>(x, weight, width, eps, scratch);
    T *target = normed + blockIdx.x * normed_stride;
#pragma unroll
    for (int h = 0; h < kHeldPacks; ++h) {
        const int c = threadIdx.x * VEC + h * stride;
        if (c < width) store_pack<VEC>(target + c, x[h]);
    }
}

// A projected row holds [query latent (q_rank) | key/value latent (kv_rank) | ...].  Both are RMS-normed; the first goes
// to q_out, the second into the cache row (write_pages[t], write_slots[t]), zero-padded to cache_width.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
    latent_norm_cache_write_kernel(T *q_out, long long q_stride, T *cache, int cache_width, const T *projected,
                                   long long projected_stride, const T *q_weight, int q_rank, const T *kv_weight,
                                   int kv_rank, const long long *write_pages, const long long *write_slots,
                                   long long pages, long long page_size, float eps, uint32_t *status) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float scratch[32];
    const int token = blockIdx.x;
    const T *row = projected + token * projected_stride;
    float square_q = 0.0f, square_kv = 0.0f;
    for (int c = threadIdx.x * VEC; c < q_rank; c += blockDim.x * VEC) {
        const Pack<VEC> x = load_pack<VEC>(row + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) square_q = square_chain(square_q, x.v[i]);
    }
    for (int c = threadIdx.x * VEC; c < kv_rank; c += blockDim.x * VEC) {
        const Pack<VEC> x = load_pack<VEC>(row + q_rank + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) square_kv = square_chain(square_kv, x.v[i]);
    }
    const float scale_q = 1.0f / sqrtf(cta_sum(square_q, scratch) / static_cast<float>(q_rank) + eps);
    const float scale_kv = 1.0f / sqrtf(cta_sum(square_kv, scratch) / static_cast<float>(kv_rank) + eps);
    for (int c = threadIdx.x * VEC; c < q_rank; c += blockDim.x * VEC) {
        Pack<VEC> x = load_pack<VEC>(row + c);
        const Pack<VEC> gain = load_pack<VEC>(q_weight + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) x.v[i] = x.v[i] * scale_q * gain.v[i];
        store_pack<VEC>(q_out + token * q_stride + c, x);
    }
    long long page = write_pages[token];
    long long slot = write_slots[token];
    if (page < 0) page += pages;
    if (slot < 0) slot += page_size;
    if (page < 0 || page >= pages || slot < 0 || slot >= page_size) {
        if (threadIdx.x == 0) report_status(status, kStatusIndexOutOfBounds);
        return;
    }
    T *target = cache + static_cast<size_t>(page * page_size + slot) * cache_width;
    for (int c = threadIdx.x * VEC; c < cache_width; c += blockDim.x * VEC) {
        Pack<VEC> x;
#pragma unroll
        for (int i = 0; i < VEC; ++i) x.v[i] = 0.0f;
        if (c < kv_rank) {
            x = load_pack<VEC>(row + q_rank + c);
            const Pack<VEC> gain = load_pack<VEC>(kv_weight + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) x.v[i] = x.v[i] * scale_kv * gain.v[i];
        }
        store_pack<VEC>(target + c, x);
    }
}

// out[targets[i], :] = source[rows[i], :] in 16-byte pieces (targets == nullptr: out[i, :]).
__global__ void __launch_bounds__(256)
    gather_rows_kernel(uint4 *out, const uint4 *source, const int32_t *rows, const int32_t *targets, long long count, int pieces,
                       long long source_rows, long long out_rows, uint32_t *status) {
    grid_launch_dependents();
    grid_dependency_wait();
    const long long total = count * pieces;
    for (long long index = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; index < total;
         index += static_cast<long long>(gridDim.x) * blockDim.x) {
        const long long row = index / pieces;
        const long long from = rows[row];
        const long long piece = index - row * pieces;
        const long long to = targets == nullptr ? row : targets[row];
        if (to < 0 || to >= out_rows) {
            report_status(status, kStatusIndexOutOfBounds);
            continue;
        }
        if (from < 0 || from >= source_rows) {
            report_status(status, kStatusIndexOutOfBounds);
            out[to * pieces + piece] = make_uint4(0u, 0u, 0u, 0u);
            continue;
        }
        out[to * pieces + piece] = source[from * pieces + piece];
    }
}

// Row-wise argmax over f32 logits; ties go to the lowest index, NaN never wins.
__global__ void __launch_bounds__(1024)
    argmax_f32_kernel(float *best_value, long long *best_index, const float *logits, long long stride, int width,
                      long long index_offset) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float values[32];
    __shared__ int indices[32];
    const float *row = logits + blockIdx.x * stride;
    float best = -INFINITY;
    int where = 0x7fffffff;
    auto look = [&](float value, int c) {  // in ascending order: a later equal value never replaces an earlier one
        if (value > best) {
            best = value;
            where = c;
        }
    };
    int c = 0;
    if ((reinterpret_cast<uintptr_t>(row) & 15u) == 0) {
        constexpr int kAhead = 4;  // independent loads of a thread
        for (; c + 4096 * kAhead <= width; c += 4096 * kAhead) {
            float4 x[kAhead];
#pragma unroll
            for (int u = 0; u < kAhead; ++u) x[u] = *reinterpret_cast<const float4 *>(row + c + u * 4096 + threadIdx.x * 4);
#pragma unroll
            for (int u = 0; u < kAhead; ++u) {
                const int at = c + u * 4096 + threadIdx.x * 4;
                look(x[u].x, at);
                look(x[u].y, at + 1);
                look(x[u].z, at + 2);
                look(x[u].w, at + 3);
            }
        }
    }
    for (c += threadIdx.x; c < width; c += 1024) look(row[c], c);
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) {
        const float other = __shfl_xor_sync(0xffffffffu, best, offset);
        const int other_where = __shfl_xor_sync(0xffffffffu, where, offset);
        if (other > best || (other == best && other_where < where)) {
            best = other;
            where = other_where;
        }
    }
    if ((threadIdx.x & 31) == 0) {
        values[threadIdx.x >> 5] = best;
        indices[threadIdx.x >> 5] = where;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int i = 1; i < static_cast<int>(blockDim.x >> 5); ++i) {
            if (values[i] > best || (values[i] == best && indices[i] < where)) {
                best = values[i];
                where = indices[i];
            }
        }
        best_value[blockIdx.x] = best;
        best_index[blockIdx.x] = static_cast<long long>(where) + index_offset;
    }
}

template <typename T>
int embedding_layer_norm(singe_stream_t stream, float *residual, const void *table, const int64_t *ids,
                         const void *weight, size_t tokens, size_t width, size_t vocab, float eps, uint32_t *status) {
    if (tokens == 0 || width == 0 || vocab == 0) return SINGE_ERR_INVALID_LENGTH;
    if (!fits_i32(tokens) || !fits_i32(width) || !fits_i32(vocab)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (residual == nullptr || table == nullptr || ids == nullptr || weight == nullptr) return SINGE_ERR_NULL_POINTER;
    const bool wide = width % 4 == 0 && aligned_to(residual, 16) && aligned_to(table, 4 * sizeof(T)) &&
                      aligned_to(weight, 4 * sizeof(T));
    if (!row_fits(width, wide ? 4 : 1)) return SINGE_ERR_UNSUPPORTED_WIDTH;
    auto kernel = wide ? embedding_layer_norm_kernel<T, 4> : embedding_layer_norm_kernel<T, 1>;
    SINGE_CUDA_TRY(launch_dependent(kernel, dim3(static_cast<unsigned>(tokens)), dim3(norm_threads(width, wide ? 4 : 1)), 0,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, residual,
                                    static_cast<const T *>(table), reinterpret_cast<const long long *>(ids),
                                    static_cast<const T *>(weight), static_cast<int>(width),
                                    static_cast<long long>(vocab), eps, status));
    return launch_status();
}

template <typename T>
int add_layer_norm(singe_stream_t stream, float *residual, const void *delta, size_t delta_stride, void *normed,
                   size_t normed_stride, const void *weight, size_t rows, size_t width, float eps) {
    if (rows == 0 || width == 0 || (delta != nullptr && delta_stride < width) ||
        (normed != nullptr && normed_stride < width)) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(rows) || !fits_i32(width)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (residual == nullptr || (normed != nullptr && weight == nullptr) || (normed == nullptr && delta == nullptr)) {
        return SINGE_ERR_NULL_POINTER;
    }
    const bool wide = width % 4 == 0 && delta_stride % 4 == 0 && normed_stride % 4 == 0 && aligned_to(residual, 16) &&
                      aligned_to(delta, 4 * sizeof(T)) && aligned_to(normed, 4 * sizeof(T)) &&
                      aligned_to(weight, 4 * sizeof(T));
    if (!row_fits(width, wide ? 4 : 1)) return SINGE_ERR_UNSUPPORTED_WIDTH;
    auto kernel = wide ? add_layer_norm_kernel<T, 4> : add_layer_norm_kernel<T, 1>;
    SINGE_CUDA_TRY(launch_dependent(kernel, dim3(static_cast<unsigned>(rows)), dim3(norm_threads(width, wide ? 4 : 1)), 0,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, residual,
                                    static_cast<const T *>(delta), static_cast<long long>(delta_stride),
                                    static_cast<T *>(normed), static_cast<long long>(normed_stride),
                                    static_cast<const T *>(weight), static_cast<int>(width), eps));
    return launch_status();
}

template <typename T>
int latent_norm_cache_write(singe_stream_t stream, void *q_out, size_t q_stride, void *cache, size_t cache_width,
                            const void *projected, size_t projected_stride, const void *q_weight, size_t q_rank,
                            const void *kv_weight, size_t kv_rank, const int64_t *write_pages, const int64_t *write_slots,
                            size_t tokens, size_t pages, size_t page_size, float eps, uint32_t *status) {
    if (tokens == 0 || q_rank == 0 || kv_rank == 0 || cache_width < kv_rank || q_stride < q_rank ||
        projected_stride < q_rank + kv_rank || pages == 0 || page_size == 0) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(tokens) || !fits_i32(projected_stride) || !fits_i32(cache_width)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (q_out == nullptr || cache == nullptr || projected == nullptr || q_weight == nullptr || kv_weight == nullptr ||
        write_pages == nullptr || write_slots == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    const size_t bytes = 4 * sizeof(T);
    const bool wide = q_rank % 4 == 0 && kv_rank % 4 == 0 && cache_width % 4 == 0 && projected_stride % 4 == 0 &&
                      q_stride % 4 == 0 && aligned_to(q_out, bytes) && aligned_to(cache, bytes) &&
                      aligned_to(projected, bytes) && aligned_to(q_weight, bytes) && aligned_to(kv_weight, bytes);
    auto kernel = wide ? latent_norm_cache_write_kernel<T, 4> : latent_norm_cache_write_kernel<T, 1>;
    SINGE_CUDA_TRY(launch_dependent(
        kernel, dim3(static_cast<unsigned>(tokens)), dim3(256), 0, static_cast<cudaStream_t>(stream), kLaunchGlue, 1,
        static_cast<T *>(q_out), static_cast<long long>(q_stride), static_cast<T *>(cache), static_cast<int>(cache_width),
        static_cast<const T *>(projected), static_cast<long long>(projected_stride), static_cast<const T *>(q_weight),
        static_cast<int>(q_rank), static_cast<const T *>(kv_weight), static_cast<int>(kv_rank),
        reinterpret_cast<const long long *>(write_pages), reinterpret_cast<const long long *>(write_slots),
        static_cast<long long>(pages), static_cast<long long>(page_size), eps, status));
    return launch_status();
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

#define SINGE_RESIDUAL_NORM_ENTRIES(SUFFIX, T)                                                                          \
    int singe_embedding_layer_norm_##SUFFIX(singe_stream_t stream, float *residual, const void *table,                  \
                                            const int64_t *ids, const void *weight, size_t tokens, size_t width,        \
                                            size_t vocab, float eps, uint32_t *status) {                                \
        return embedding_layer_norm<T>(stream, residual, table, ids, weight, tokens, width, vocab, eps, status);        \
    }                                                                                                                   \
    int singe_add_layer_norm_##SUFFIX(singe_stream_t stream, float *residual, const void *delta, size_t delta_stride,   \
                                      void *normed, size_t normed_stride, const void *weight, size_t rows,              \
                                      size_t width, float eps) {                                                        \
        return add_layer_norm<T>(stream, residual, delta, delta_stride, normed, normed_stride, weight, rows, width,     \
                                 eps);                                                                                  \
    }                                                                                                                   \
    int singe_latent_norm_cache_write_##SUFFIX(                                                                         \
        singe_stream_t stream, void *q_out, size_t q_stride, void *cache, size_t cache_width, const void *projected,    \
        size_t projected_stride, const void *q_weight, size_t q_rank, const void *kv_weight, size_t kv_rank,            \
        const int64_t *write_pages, const int64_t *write_slots, size_t tokens, size_t pages, size_t page_size,          \
        float eps, uint32_t *status) {                                                                                  \
        return latent_norm_cache_write<T>(stream, q_out, q_stride, cache, cache_width, projected, projected_stride,     \
                                          q_weight, q_rank, kv_weight, kv_rank, write_pages, write_slots, tokens,       \
                                          pages, page_size, eps, status);                                               \
    }

SINGE_RESIDUAL_NORM_ENTRIES(bf16, __nv_bfloat16)
SINGE_RESIDUAL_NORM_ENTRIES(f32, float)
#undef SINGE_RESIDUAL_NORM_ENTRIES

static int gather_rows(singe_stream_t stream, void *out, const void *source, const int32_t *rows, const int32_t *targets,
                       size_t count, size_t row_bytes, size_t source_rows, size_t out_rows, uint32_t *status) {
    if (count == 0 || row_bytes == 0 || source_rows == 0 || out_rows == 0) return SINGE_ERR_INVALID_LENGTH;
    if (out == nullptr || source == nullptr || rows == nullptr) return SINGE_ERR_NULL_POINTER;
    if (row_bytes % 16 != 0 || !aligned_to(out, 16) || !aligned_to(source, 16)) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    if (!fits_i32(row_bytes) || !fits_i32(count)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    const size_t pieces = row_bytes / 16;
    size_t blocks = (count * pieces + 255) / 256;
    const size_t most = static_cast<size_t>(device_sm_count()) * 16;
    if (blocks > most) blocks = most;
    SINGE_CUDA_TRY(launch_dependent(gather_rows_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, static_cast<uint4 *>(out),
                                    static_cast<const uint4 *>(source), rows, targets, static_cast<long long>(count),
                                    static_cast<int>(pieces), static_cast<long long>(source_rows),
                                    static_cast<long long>(out_rows), status));
    return launch_status();
}

int singe_gather_rows(singe_stream_t stream, void *out, const void *source, const int32_t *rows, size_t count,
                      size_t row_bytes, size_t source_rows, uint32_t *status) {
    return gather_rows(stream, out, source, rows, nullptr, count, row_bytes, source_rows, count, status);
}

int singe_move_rows(singe_stream_t stream, void *out, const void *source, const int32_t *rows, const int32_t *targets,
                    size_t count, size_t row_bytes, size_t source_rows, size_t out_rows, uint32_t *status) {
    if (targets == nullptr) return SINGE_ERR_NULL_POINTER;
    return gather_rows(stream, out, source, rows, targets, count, row_bytes, source_rows, out_rows, status);
}

int singe_argmax_f32(singe_stream_t stream, float *best_value, int64_t *best_index, const float *logits,
                     size_t row_stride, size_t rows, size_t width, int64_t index_offset) {
    if (rows == 0 || width == 0 || row_stride < width) return SINGE_ERR_INVALID_LENGTH;
    if (!fits_i32(rows) || !fits_i32(width)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (best_value == nullptr || best_index == nullptr || logits == nullptr) return SINGE_ERR_NULL_POINTER;
    SINGE_CUDA_TRY(launch_dependent(argmax_f32_kernel, dim3(static_cast<unsigned>(rows)), dim3(1024), 0,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, best_value,
                                    reinterpret_cast<long long *>(best_index), logits, static_cast<long long>(row_stride),
                                    static_cast<int>(width), static_cast<long long>(index_offset)));
    return launch_status();
}

}  // extern "C"
