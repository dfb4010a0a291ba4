// Gated delta rule: a recurrence over a state S [dim, vdim] per head with one decay per key channel,
//     S <- diag(g_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t,
//     g_t = exp(-exp(A) softplus(z_t + bias)),   beta_t = sigmoid(b_t),
// with q and k unit vectors.  Each head's o is RMS-normed over vdim, multiplied by sigmoid(gate) and handed to the output
// projection.  Query / key head h / (heads / kv_heads) serves head h.
//
// A mixed row holds [q (G x dim) | k (G x dim) at key_at | v (H x vdim) at value_at], as the convolution left them; the inverse
// lengths of its 2 G queries and keys are f32 beside it.  The state of sequence s is state[s] of an f32 array [sequences, H,
// dim, vdim].  Unit vectors, decays, write strengths, gates, the state and the norm are f32.
//
// Sequence s owns rows [first[s], first[s] + count[s]) of the step; context[s] tokens came before (0: the state starts at
// zero, whatever its slot held before).  A sequence without tokens keeps its state; its idle row is written as zeros.
#include "row_pack.cuh"

namespace singe {
namespace {

constexpr int kStepThreads = 256;

struct GatedDelta {
    void *out;              // [rows, out_stride], heads side by side
    long long out_stride;
    const void *mixed;      // [rows, mixed_stride]
    long long mixed_stride;
    const float *inverse;   // [rows, 2 * kv_heads]
    const void *strength;   // [rows, strength_stride]: b
    long long strength_stride;
    const void *decay;      // [rows, decay_stride]: z (H x dim), and from gate_at on the gates (H x vdim)
    long long decay_stride;
    int gate_at;
    const float *rate;      // [heads]: A
    const float *bias;      // [heads * dim]
    const void *norm_weight;  // [vdim]
    float *state;
    const int32_t *first, *count, *context;
    int heads, kv_heads, dim, vdim, key_at, value_at;
    float eps;
    int longest;            // sequences of more new tokens are left alone
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// One CTA per (head, sequence), token by token.  A thread owns VEC adjacent columns and every `groups`-th key channel, so it
// only ever touches its own elements of the state.  BATCH > 0: its share is at most BATCH packs and stays in registers from
// the first token to the last; BATCH == 0: any size, the state goes through global memory twice a token.
template <typename T, int VEC, int BATCH>
__global__ void __launch_bounds__(kStepThreads, 2) gated_delta_step_kernel(const GatedDelta p) {
    grid_launch_dependents();
    const int head = blockIdx.x, sequence = blockIdx.y;
    float *state = p.state + (static_cast<size_t>(sequence) * p.heads + head) * p.dim * p.vdim;
    if (VEC == 4 && threadIdx.x < 32) {
        // the state crosses HBM while the kernels before are still running (a hint: nothing is read before the wait)
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
    float *partial = shared;                        // [kStepThreads * VEC]
    float *written = partial + kStepThreads * VEC;  // [vdim]
    float *output = written + p.vdim;               // [vdim]
    float *keep = output + p.vdim;                  // [dim]
    float *query = keep + p.dim;                    // [dim]
    float *key = query + p.dim;                     // [dim]
    __shared__ float scratch[32];
    const int packs = p.vdim / VEC;
    const int columns = packs < 64 ? packs : 64;
    const int groups = kStepThreads / columns;
    const int column = tid % columns, group = tid / columns;
    const bool active = group < groups;
    const int source = head / (p.heads / p.kv_heads);
    const float query_scale = 1.0f / sqrtf(static_cast<float>(p.dim));
    const float rate = expf(p.rate[head]);
    bool fresh = p.context[sequence] == 0;

    Pack<VEC> held[BATCH > 0 ? BATCH : 1];
    if (BATCH > 0 && active) {
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const int c = group + u * groups;
#pragma unroll
            for (int i = 0; i < VEC; ++i) held[u].v[i] = 0.0f;
            if (c < p.dim && !fresh) held[u] = load_pack<VEC>(state + static_cast<size_t>(c) * p.vdim + column * VEC);
        }
    }
    for (int t = 0; t < tokens; ++t) {
        const long long row = row0 + t;
        const T *mixed = static_cast<const T *>(p.mixed) + row * p.mixed_stride;
        const T *decay = static_cast<const T *>(p.decay) + row * p.decay_stride;
        const float unit_q = p.inverse[row * 2 * p.kv_heads + source] * query_scale;
        const float unit_k = p.inverse[row * 2 * p.kv_heads + p.kv_heads + source];
        const float b = to_float<T>(static_cast<const T *>(p.strength)[row * p.strength_stride + head]);
        const float beta = 1.0f / (1.0f + expf(-b));
        for (int c = tid; c < p.dim; c += kStepThreads) {
            const int channel = head * p.dim + c;
            query[c] = to_float<T>(mixed[source * p.dim + c]) * unit_q;
            key[c] = to_float<T>(mixed[p.key_at + source * p.dim + c]) * unit_k;
            keep[c] = expf(-rate * softplus(to_float<T>(decay[channel]) + p.bias[channel]));
        }
        __syncthreads();
        for (int base = 0; base < packs; base += columns) {
            const int pack = base + column;
            const bool live = active && pack < packs;
            float *cell = state + static_cast<size_t>(pack) * VEC;
            // ---- what the decayed state recalls for the key ----
            Pack<VEC> sum = {};
            if (BATCH > 0) {
                if (live) {
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        const int c = group + u * groups;
                        if (c < p.dim) {
                            const float g = keep[c], k = key[c];
#pragma unroll
                            for (int i = 0; i < VEC; ++i) {
                                held[u].v[i] *= g;
                                sum.v[i] = fmaf(k, held[u].v[i], sum.v[i]);
                            }
                        }
                    }
                }
            } else if (live && !fresh) {
                for (int c = group; c < p.dim; c += groups) {
                    const Pack<VEC> x = load_pack<VEC>(cell + static_cast<size_t>(c) * p.vdim);
#pragma unroll
                    for (int i = 0; i < VEC; ++i) sum.v[i] = fmaf(key[c], keep[c] * x.v[i], sum.v[i]);
                }
            }
            store_pack<VEC>(partial + tid * VEC, sum);
            __syncthreads();
            for (int v = tid; v < columns * VEC; v += kStepThreads) {
                const int at = base * VEC + v;
                if (at < p.vdim) {
                    float total = 0.0f;
                    for (int g = 0; g < groups; ++g) total += partial[g * columns * VEC + v];
                    written[at] = beta * (to_float<T>(mixed[p.value_at + head * p.vdim + at]) - total);
                }
            }
            __syncthreads();
            // ---- the write, and the read-out after it ----
#pragma unroll
            for (int i = 0; i < VEC; ++i) sum.v[i] = 0.0f;
            if (live) {
                const Pack<VEC> w = load_pack<VEC>(written + pack * VEC);
                if (BATCH > 0) {
#pragma unroll
                    for (int u = 0; u < BATCH; ++u) {
                        const int c = group + u * groups;
                        if (c < p.dim) {
                            const float k = key[c], q = query[c];
#pragma unroll
                            for (int i = 0; i < VEC; ++i) {
                                held[u].v[i] = fmaf(k, w.v[i], held[u].v[i]);
                                sum.v[i] = fmaf(q, held[u].v[i], sum.v[i]);
                            }
                        }
                    }
                } else {
                    for (int c = group; c < p.dim; c += groups) {
                        Pack<VEC> x = {};
                        if (!fresh) x = load_pack<VEC>(cell + static_cast<size_t>(c) * p.vdim);
#pragma unroll
                        for (int i = 0; i < VEC; ++i) {
                            x.v[i] = fmaf(key[c], w.v[i], keep[c] * x.v[i]);
                            sum.v[i] = fmaf(query[c], x.v[i], sum.v[i]);
                        }
                        store_pack<VEC>(cell + static_cast<size_t>(c) * p.vdim, x);
                    }
                }
            }
            store_pack<VEC>(partial + tid * VEC, sum);
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
        const float scale = 1.0f / sqrtf(cta_sum(square, scratch) / static_cast<float>(p.vdim) + p.eps);
        for (int v = tid; v < p.vdim; v += kStepThreads) {
            const float gate = to_float<T>(decay[p.gate_at + head * p.vdim + v]);
            const float normed = output[v] * scale * to_float<T>(static_cast<const T *>(p.norm_weight)[v]);
            out[t * p.out_stride + v] = from_float<T>(normed / (1.0f + expf(-gate)));
        }
        fresh = false;
    }
    if (BATCH > 0 && active) {
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const int c = group + u * groups;
            if (c < p.dim) store_pack<VEC>(state + static_cast<size_t>(c) * p.vdim + column * VEC, held[u]);
        }
    }
}

template <typename T, int VEC, int BATCH>
int launch_step(cudaStream_t stream, const GatedDelta &p, size_t sequences) {
    const size_t shared = (3 * static_cast<size_t>(p.dim) + 2 * p.vdim + kStepThreads * VEC) * sizeof(float);
    if (shared > 200 * 1024) return SINGE_ERR_UNSUPPORTED_WIDTH;
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_delta_step_kernel<T, VEC, BATCH>, static_cast<int>(shared), configured));
    SINGE_CUDA_TRY(launch_dependent(gated_delta_step_kernel<T, VEC, BATCH>,
                                    dim3(static_cast<unsigned>(p.heads), static_cast<unsigned>(sequences)), dim3(kStepThreads),
                                    shared, stream, kLaunchGlue, 1, p));
    return launch_status();
}

template <typename T>
int gated_delta_step(singe_stream_t stream, const GatedDelta &p, size_t rows, size_t sequences) {
    if (rows == 0 || sequences == 0 || p.heads <= 0 || p.kv_heads <= 0 || p.heads % p.kv_heads != 0 || p.dim <= 0 || p.vdim <= 0) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    const long long inner = static_cast<long long>(p.heads) * p.vdim;
    if (p.key_at < p.kv_heads * p.dim || p.value_at < p.key_at + p.kv_heads * p.dim || p.mixed_stride < p.value_at + inner ||
        p.gate_at < p.heads * p.dim || p.decay_stride < p.gate_at + inner || p.strength_stride < p.heads || p.out_stride < inner) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (sequences > 65535 || !fits_i32(rows)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (p.out == nullptr || p.mixed == nullptr || p.inverse == nullptr || p.strength == nullptr || p.decay == nullptr ||
        p.rate == nullptr || p.bias == nullptr || p.norm_weight == nullptr || p.state == nullptr || p.first == nullptr ||
        p.count == nullptr || p.context == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (p.vdim % 4 != 0 || !aligned_to(p.state, 16)) return launch_step<T, 1, 0>(s, p, sequences);
    const int packs = p.vdim / 4, columns = packs < 64 ? packs : 64;
    const int share = (p.dim + kStepThreads / columns - 1) / (kStepThreads / columns);
    if (packs > columns || share > 16) return launch_step<T, 4, 0>(s, p, sequences);
    if (share > 8) return launch_step<T, 4, 16>(s, p, sequences);
    if (share > 4) return launch_step<T, 4, 8>(s, p, sequences);
    return launch_step<T, 4, 4>(s, p, sequences);
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

#define SINGE_GATED_DELTA_STEP(SUFFIX, T)                                                                                 \
    int singe_gated_delta_step_##SUFFIX(                                                                                  \
        singe_stream_t stream, void *out, size_t out_stride, const void *mixed, size_t mixed_stride, const float *inverse, \
        const void *strength, size_t strength_stride, const void *decay, size_t decay_stride, const float *rate,          \
        const float *bias, const void *norm_weight, float *state, const int32_t *first, const int32_t *count,             \
        const int32_t *context, size_t rows, size_t sequences, size_t heads, size_t kv_heads, size_t dim, size_t vdim,    \
        size_t key_at, size_t value_at, size_t gate_at, float eps, size_t longest) {                                      \
        if (!fits_i32(heads * dim) || !fits_i32(heads * vdim) || !fits_i32(value_at) || !fits_i32(gate_at)) {             \
            return SINGE_ERR_LENGTH_EXCEEDS_I32;                                                                          \
        }                                                                                                                 \
        GatedDelta p = {};                                                                                                \
        p.out = out;                                                                                                      \
        p.out_stride = static_cast<long long>(out_stride);                                                                \
        p.mixed = mixed;                                                                                                  \
        p.mixed_stride = static_cast<long long>(mixed_stride);                                                            \
        p.inverse = inverse;                                                                                              \
        p.strength = strength;                                                                                            \
        p.strength_stride = static_cast<long long>(strength_stride);                                                      \
        p.decay = decay;                                                                                                  \
        p.decay_stride = static_cast<long long>(decay_stride);                                                            \
        p.gate_at = static_cast<int>(gate_at);                                                                            \
        p.rate = rate;                                                                                                    \
        p.bias = bias;                                                                                                    \
        p.norm_weight = norm_weight;                                                                                      \
        p.state = state;                                                                                                  \
        p.first = first;                                                                                                  \
        p.count = count;                                                                                                  \
        p.context = context;                                                                                              \
        p.heads = static_cast<int>(heads);                                                                                \
        p.kv_heads = static_cast<int>(kv_heads);                                                                          \
        p.dim = static_cast<int>(dim);                                                                                    \
        p.vdim = static_cast<int>(vdim);                                                                                  \
        p.key_at = static_cast<int>(key_at);                                                                              \
        p.value_at = static_cast<int>(value_at);                                                                          \
        p.eps = eps;                                                                                                      \
        p.longest = longest > 0x7fffffff ? 0x7fffffff : static_cast<int>(longest);                                        \
        return gated_delta_step<T>(stream, p, rows, sequences);                                                           \
    }

SINGE_GATED_DELTA_STEP(bf16, __nv_bfloat16)
SINGE_GATED_DELTA_STEP(f32, float)
#undef SINGE_GATED_DELTA_STEP

}  // extern "C"
