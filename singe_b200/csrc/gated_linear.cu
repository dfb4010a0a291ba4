// Gated linear attention: a recurrence over a state S [dim, vdim] per head with one decay per key channel,
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t,     alpha_t = sigmoid(z_t)^(1 / tau),
// z_t = W_a2 a_t + b from a low-rank projection a_t.  Each head's o is RMS-normed over vdim, multiplied by silu(g) and
// handed to the output projection.
//
// A projected row holds [q (H x dim) | k (H x dim) | v (H x vdim) | g (H x vdim) | a (rank)]; the state of sequence s is
// state[s] of an f32 array [sequences, H, dim, vdim].  Everything between the projections and the output is f32:
// q, k, v, g and a come as the activation type T, decays, state, outputs and the norm do not leave f32.
//
// Sequence s owns rows [first[s], first[s] + count[s]) of the step; context[s] tokens came before (0: the state starts at
// zero, whatever its slot held before).  A sequence without tokens keeps its state; its idle row is written as zeros.
#include "common.cuh"

namespace singe {
namespace {

struct GatedLinear {
    void *out;                // [rows, out_stride], heads side by side
    long long out_stride;
    const void *projected;    // [rows, stride]
    long long stride;
    const void *decay_weight; // [H * dim, rank]
    const void *decay_bias;   // [H * dim]
    const void *norm_weight;  // [vdim]
    float *state;
    const int32_t *first, *count, *context;
    int heads, dim, vdim, rank;
    float inverse_tau, query_scale, eps;
    int longest;              // the step kernel serves sequences of up to this many tokens, the chunk kernels the others
};

// log(sigmoid(z)) without cancellation for either sign
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

constexpr int kStepThreads = 256;
constexpr int kStepBatch = 8;  // state packs a thread keeps in flight

template <int VEC>
struct StatePack;
template <>
struct StatePack<4> {
    using type = float4;
};
template <>
struct StatePack<1> {
    using type = float;
};

template <int VEC>
__device__ __forceinline__ float &part(typename StatePack<VEC>::type &x, int i) {
    return reinterpret_cast<float *>(&x)[i];
}

// One CTA per (head, sequence): token by token, the state streamed from global memory (a decode step reads and writes it
// once).  A thread owns VEC adjacent columns and every `groups`-th key channel, so it only ever touches its own elements.
template <typename T, int VEC>
__global__ void __launch_bounds__(kStepThreads, 4) gated_linear_step_kernel(const GatedLinear p) {
    using Pack = typename StatePack<VEC>::type;
    grid_launch_dependents();
    const int head = blockIdx.x, sequence = blockIdx.y;
    float *state = p.state + (static_cast<size_t>(sequence) * p.heads + head) * p.dim * p.vdim;
    if (VEC == 4 && threadIdx.x < 32) {
        // the state crosses HBM while the projection is still running (a hint: nothing is read before the wait)
        const int bytes = p.dim * p.vdim * 4;
        for (int at = threadIdx.x * 4096; at < bytes; at += 32 * 4096) {
            asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(reinterpret_cast<const char *>(state) + at),
                         "r"(min(4096, bytes - at))
                         : "memory");
        }
    }
    grid_dependency_wait();
    const int tokens = p.count[sequence];
    const int row0 = p.first[sequence];
    const int tid = threadIdx.x;
    T *out = static_cast<T *>(p.out) + row0 * p.out_stride + head * p.vdim;
    if (tokens <= 0) {
        for (int v = tid; v < p.vdim; v += kStepThreads) out[v] = from_float<T>(0.0f);
        return;
    }
    if (tokens > p.longest) return;
    extern __shared__ float shared[];
    float *alpha = shared;               // [dim]
    float *query = alpha + p.dim;        // [dim]
    float *key = query + p.dim;          // [dim]
    float *output = key + p.dim;         // [vdim]
    float *low = output + p.vdim;        // [rank]
    float *partial = low + p.rank;       // [kStepThreads * VEC]
    __shared__ float scratch[32];
    const int packs = p.vdim / VEC;                       // column packs of the head
    const int columns = packs < 64 ? packs : 64;          // ... handled at a time
    const int groups = kStepThreads / columns;
    const int column = tid % columns, group = tid / columns;
    const bool active = group < groups;
    const int key_at = p.heads * p.dim, value_at = 2 * p.heads * p.dim, gate_at = value_at + p.heads * p.vdim;
    const int low_at = gate_at + p.heads * p.vdim;
    bool fresh = p.context[sequence] == 0;
    const bool in_batch = p.dim <= groups * kStepBatch && packs <= columns;  // a thread's whole share is one batch of packs
    for (int t = 0; t < tokens; ++t, fresh = false) {
        // the share of the state is on its way while the decays are computed
        Pack held[kStepBatch];
        if (in_batch && active) {
#pragma unroll
            for (int u = 0; u < kStepBatch; ++u) {
                const int c = group + u * groups;
#pragma unroll
                for (int i = 0; i < VEC; ++i) part<VEC>(held[u], i) = 0.0f;
                if (c < p.dim && !fresh) held[u] = (reinterpret_cast<Pack *>(state) + column)[static_cast<size_t>(c) * packs];
            }
        }
        const T *row = static_cast<const T *>(p.projected) + (row0 + t) * p.stride;
        for (int r = tid; r < p.rank; r += kStepThreads) low[r] = to_float<T>(row[low_at + r]);
        __syncthreads();
        for (int c = tid; c < p.dim; c += kStepThreads) {
            const int channel = head * p.dim + c;
            const T *weight = static_cast<const T *>(p.decay_weight) + static_cast<size_t>(channel) * p.rank;
            query[c] = to_float<T>(row[channel]) * p.query_scale;
            key[c] = to_float<T>(row[key_at + channel]);
            float z = to_float<T>(static_cast<const T *>(p.decay_bias)[channel]);
#pragma unroll 16
            for (int r = 0; r < p.rank; ++r) z = fmaf(to_float<T>(weight[r]), low[r], z);
            alpha[c] = expf(log_sigmoid(z) * p.inverse_tau);
        }
        __syncthreads();
        for (int base = 0; base < packs; base += columns) {
            const int pack = base + column;
            const bool live = active && pack < packs;
            Pack sum;
#pragma unroll
            for (int i = 0; i < VEC; ++i) part<VEC>(sum, i) = 0.0f;
            if (live) {
                Pack value;
#pragma unroll
                for (int i = 0; i < VEC; ++i) {
                    part<VEC>(value, i) = to_float<T>(row[value_at + head * p.vdim + pack * VEC + i]);
                }
                Pack *cell = reinterpret_cast<Pack *>(state) + pack;
                for (int c0 = group; c0 < p.dim; c0 += groups * kStepBatch) {
                    if (!in_batch) {
#pragma unroll
                        for (int u = 0; u < kStepBatch; ++u) {
                            const int c = c0 + u * groups;
#pragma unroll
                            for (int i = 0; i < VEC; ++i) part<VEC>(held[u], i) = 0.0f;
                            if (c < p.dim && !fresh) held[u] = cell[static_cast<size_t>(c) * packs];
                        }
                    }
#pragma unroll
                    for (int u = 0; u < kStepBatch; ++u) {
                        const int c = c0 + u * groups;
                        if (c < p.dim) {
#pragma unroll
                            for (int i = 0; i < VEC; ++i) {
                                float &s = part<VEC>(held[u], i);
                                s = fmaf(alpha[c], s, key[c] * part<VEC>(value, i));
                                part<VEC>(sum, i) = fmaf(query[c], s, part<VEC>(sum, i));
                            }
                            cell[static_cast<size_t>(c) * packs] = held[u];
                        }
                    }
                }
            }
            reinterpret_cast<Pack *>(partial)[tid] = sum;
            __syncthreads();
            for (int v = tid; v < columns * VEC; v += kStepThreads) {
                if (base * VEC + v < p.vdim) {
                    float total = 0.0f;
                    for (int g = 0; g < groups; ++g) total += partial[g * columns * VEC + v];
                    output[base * VEC + v] = total;
                }
            }
            __syncthreads();
        }
        float square = 0.0f;
        for (int v = tid; v < p.vdim; v += kStepThreads) square = square_chain(square, output[v]);
        square = warp_sum(square);
        if ((tid & 31) == 0) scratch[tid >> 5] = square;
        __syncthreads();
        float total = 0.0f;
#pragma unroll
        for (int i = 0; i < kStepThreads / 32; ++i) total += scratch[i];
        const float scale = 1.0f / sqrtf(total / static_cast<float>(p.vdim) + p.eps);
        for (int v = tid; v < p.vdim; v += kStepThreads) {
            const float gate = to_float<T>(row[gate_at + head * p.vdim + v]);
            const float normed = output[v] * scale * to_float<T>(static_cast<const T *>(p.norm_weight)[v]);
            out[t * p.out_stride + v] = from_float<T>(normed * (gate / (1.0f + expf(-gate))));
        }
        __syncthreads();
    }
}

int validate(const GatedLinear &p, size_t rows, size_t sequences) {
    if (rows == 0 || sequences == 0 || p.heads <= 0 || p.dim <= 0 || p.vdim <= 0 || p.rank <= 0) return SINGE_ERR_INVALID_LENGTH;
    const long long inner = static_cast<long long>(p.heads) * p.vdim;
    if (p.stride < 2ll * p.heads * p.dim + 2 * inner + p.rank || p.out_stride < inner) return SINGE_ERR_INVALID_LENGTH;
    if (sequences > 65535 || !fits_i32(rows)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (p.out == nullptr || p.projected == nullptr || p.decay_weight == nullptr || p.decay_bias == nullptr ||
        p.norm_weight == nullptr || p.state == nullptr || p.first == nullptr || p.count == nullptr || p.context == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    return SINGE_OK;
}

template <typename T, int VEC>
int launch_step(cudaStream_t stream, const GatedLinear &p, size_t sequences) {
    const size_t shared = (3 * static_cast<size_t>(p.dim) + p.vdim + p.rank + kStepThreads * VEC + 4) * sizeof(float);
    if (shared > 200 * 1024) return SINGE_ERR_UNSUPPORTED_WIDTH;
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_step_kernel<T, VEC>, static_cast<int>(shared), configured));
    SINGE_CUDA_TRY(launch_dependent(gated_linear_step_kernel<T, VEC>,
                                    dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(sequences)), dim3(kStepThreads),
                                    shared, stream, kLaunchGlue, 1, p));
    return launch_status();
}

GatedLinear describe(void *out, size_t out_stride, const void *projected, size_t stride, const void *decay_weight,
                     const void *decay_bias, const void *norm_weight, float *state, const int32_t *first,
                     const int32_t *count, const int32_t *context, size_t heads, size_t dim, size_t vdim, size_t rank,
                     float tau, float query_scale, float eps, size_t longest) {
    GatedLinear p;
    p.out = out;
    p.out_stride = static_cast<long long>(out_stride);
    p.projected = projected;
    p.stride = static_cast<long long>(stride);
    p.decay_weight = decay_weight;
    p.decay_bias = decay_bias;
    p.norm_weight = norm_weight;
    p.state = state;
    p.first = first;
    p.count = count;
    p.context = context;
    p.heads = static_cast<int>(heads);
    p.dim = static_cast<int>(dim);
    p.vdim = static_cast<int>(vdim);
    p.rank = static_cast<int>(rank);
    p.inverse_tau = 1.0f / tau;
    p.query_scale = query_scale;
    p.eps = eps;
    p.longest = longest > 0x7fffffff ? 0x7fffffff : static_cast<int>(longest);
    return p;
}

template <typename T>
int gated_linear_step(singe_stream_t stream, const GatedLinear &p, size_t rows, size_t sequences) {
    SINGE_TRY(validate(p, rows, sequences));
    // columns in fours where a head's rows of the state and the shared-memory layout keep 16-byte alignment
    const bool wide = p.vdim % 4 == 0 && (3 * p.dim + p.vdim + p.rank) % 4 == 0 &&
                      (reinterpret_cast<uintptr_t>(p.state) & 15u) == 0;
    return wide ? launch_step<T, 4>(static_cast<cudaStream_t>(stream), p, sequences)
                : launch_step<T, 1>(static_cast<cudaStream_t>(stream), p, sequences);
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

#define SINGE_GATED_LINEAR_STEP(SUFFIX, T)                                                                               \
    int singe_gated_linear_step_##SUFFIX(                                                                                \
        singe_stream_t stream, void *out, size_t out_stride, const void *projected, size_t projected_stride,             \
        const void *decay_weight, const void *decay_bias, const void *norm_weight, float *state, const int32_t *first,   \
        const int32_t *count, const int32_t *context, size_t rows, size_t sequences, size_t heads, size_t dim,           \
        size_t vdim, size_t rank, float tau, float query_scale, float eps, size_t longest) {                             \
        return gated_linear_step<T>(stream,                                                                              \
                                    describe(out, out_stride, projected, projected_stride, decay_weight, decay_bias,     \
                                             norm_weight, state, first, count, context, heads, dim, vdim, rank, tau,     \
                                             query_scale, eps, longest),                                                 \
                                    rows, sequences);                                                                    \
    }

SINGE_GATED_LINEAR_STEP(bf16, __nv_bfloat16)
SINGE_GATED_LINEAR_STEP(f32, float)
#undef SINGE_GATED_LINEAR_STEP

}  // extern "C"
