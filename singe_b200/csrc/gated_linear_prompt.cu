// Gated linear attention over prompts: the recurrence of gated_linear.cu (same operands, same meaning), block by block on
// the tensor core.
//
// In a block of 16 tokens let a_t be the running sum of log alpha per key channel (a_0 the first token's, A the last one's).
// With S the state before the block,
//     o_t = (q_t exp(a_t))^T S + sum_(j <= t) P_tj v_j,     P_tj = sum_c q_tc k_jc exp(a_tc - a_jc),
//     S'  = exp(A) S + sum_j (k_j exp(A - a_j)) v_j^T.
// Every exponent that reaches a product is <= 0 except in the factored form of P (below), which is only used where the
// block's whole decay stays above e^-60.
//
// 32-bit without 32-bit tensor cores: the operands that are f32 by nature (decayed q and k, P, the state) enter the bf16 MMA
// as two terms hi + lo, x = hi + lo up to 2^-17 |x|; v is bf16 from its projection and enters as it is.  Products of two
// split operands keep hi hi + hi lo + lo hi.  Accumulators, and the state between the blocks, are f32.
//
//   prepare   one CTA per (block, head): decays, the split operands and P, to scratch
//   advance   one CTA per (segment, head): the blocks of a segment in order, the state in registers as S^T [vdim, dim], whose
//             accumulator layout is the A-operand layout of the next product.  A warp owns 16 (or 32) value rows.
//             A long sequence is cut into segments that run side by side: a first pass (STATE_ONLY) takes every segment
//             but the last from a zero state (the first one from the sequence's state) to its end, and in the second
//             pass a segment starts from the fold of its predecessors' end states.
#include "common.cuh"

namespace singe {
namespace {

constexpr int kBlock = 16;             // tokens
constexpr int kPrepareThreads = 128;
constexpr int kStages = 3;
constexpr float kFactoredLimit = -60.0f;

struct PromptShape {
    int heads, dim, vdim, rank;
    int dim_pad;        // 16, 32, 64, 128 or 256
    int vdim_pad;       // 16 x value tiles per warp x warps
};

struct PromptParams {
    PromptShape shape;
    __nv_bfloat16 *out;
    long long out_stride;
    const __nv_bfloat16 *projected;
    long long stride;
    const __nv_bfloat16 *decay_weight, *decay_bias, *norm_weight;
    float *state;
    const int32_t *context;
    const int32_t *block_row, *block_tokens;  // first packed row and tokens of each block
    const int32_t *segments;                  // [n][4]: sequence, first block, blocks, segments of the sequence before this
    const int32_t *segment_last;              // [n]: 1 for a sequence's last segment
    uint8_t *operands;                        // [blocks, heads] packs of operand_bytes
    float *segment_state;                     // [segments, heads, vdim_pad, dim_pad]: end state of a segment
    float *segment_start;                     // the same shape: the state a sequence's first segment starts from
    float *segment_decay;                     // [segments, heads, dim_pad]
    float inverse_tau, query_scale, eps;
};

__host__ __device__ constexpr int operand_bytes(int dim_pad) { return 4 * kBlock * dim_pad * 2 + 2 * kBlock * kBlock * 2 + dim_pad * 4; }

__device__ __forceinline__ float log_sigmoid_f32(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// x = hi + lo
__device__ __forceinline__ void split_bf16(float x, __nv_bfloat16 &hi, __nv_bfloat16 &lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}

// The same for a pair, packed as an MMA register.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &hi, uint32_t &lo) {
    hi = pack2<__nv_bfloat16>(x, y);
    lo = pack2<__nv_bfloat16>(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}

__device__ __forceinline__ void load_async_16(uint32_t target, const void *source, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(target), "l"(source), "r"(valid ? 16 : 0) : "memory");
}

__global__ void __launch_bounds__(kPrepareThreads) gated_linear_prepare_kernel(const PromptParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    const PromptShape &s = p.shape;
    const int block = blockIdx.x, head = blockIdx.y;
    const int row0 = p.block_row[block], tokens = p.block_tokens[block];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pitch = s.dim_pad + 8;  // bf16 elements of a padded operand row in shared memory
    extern __shared__ __align__(16) float prepare_shared[];
    float *low = prepare_shared;                       // [16][rank]
    float *query = low + kBlock * s.rank;              // [16][dim_pad]: q, scaled
    float *key = query + kBlock * s.dim_pad;           // [16][dim_pad]
    float *alpha = key + kBlock * s.dim_pad;           // [16][dim_pad]
    // factored operands of P, split: q exp(a_t) and k exp(-a_j)
    __nv_bfloat16 *fq = reinterpret_cast<__nv_bfloat16 *>(alpha + kBlock * s.dim_pad);  // hi, lo [16][pitch] each
    __nv_bfloat16 *fk = fq + 2 * kBlock * pitch;
    uint8_t *pack = p.operands + (static_cast<size_t>(block) * s.heads + head) * operand_bytes(s.dim_pad);
    __nv_bfloat16 *q_hi = reinterpret_cast<__nv_bfloat16 *>(pack);
    __nv_bfloat16 *q_lo = q_hi + kBlock * s.dim_pad, *k_hi = q_lo + kBlock * s.dim_pad, *k_lo = k_hi + kBlock * s.dim_pad;
    __nv_bfloat16 *p_hi = k_lo + kBlock * s.dim_pad, *p_lo = p_hi + kBlock * kBlock;
    float *decay = reinterpret_cast<float *>(p_lo + kBlock * kBlock);

    const int low_at = 2 * s.heads * (s.dim + s.vdim);
    for (int i = tid; i < kBlock * s.rank; i += kPrepareThreads) {
        const int t = i / s.rank;
        low[i] = t < tokens ? __bfloat162float(p.projected[(row0 + t) * p.stride + low_at + i - t * s.rank]) : 0.0f;
    }
    __syncthreads();
    bool strong = false;
    for (int c = tid; c < s.dim_pad; c += kPrepareThreads) {
        const bool real = c < s.dim;
        const int channel = head * s.dim + (real ? c : 0);
        float z[kBlock] = {};
        if (real) {
            const __nv_bfloat16 *weight = p.decay_weight + static_cast<size_t>(channel) * s.rank;
            for (int r = 0; r < s.rank; ++r) {
                const float w = __bfloat162float(weight[r]);
#pragma unroll
                for (int t = 0; t < kBlock; ++t) z[t] = fmaf(w, low[t * s.rank + r], z[t]);
            }
        }
        const float bias = real ? __bfloat162float(p.decay_bias[channel]) : 0.0f;
        float running = 0.0f;
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            const float step = real && t < tokens ? log_sigmoid_f32(z[t] + bias) * p.inverse_tau : 0.0f;
            alpha[t * s.dim_pad + c] = expf(step);
            running += step;
            z[t] = running;
        }
        strong = strong || running < kFactoredLimit;
        decay[c] = expf(running);
        const __nv_bfloat16 *source = p.projected + row0 * p.stride + channel;
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            const bool live = real && t < tokens;
            const float q = live ? __bfloat162float(source[t * p.stride]) * p.query_scale : 0.0f;
            const float k = live ? __bfloat162float(source[t * p.stride + s.heads * s.dim]) : 0.0f;
            query[t * s.dim_pad + c] = q;
            key[t * s.dim_pad + c] = k;
            const float decayed = q * expf(z[t]);
            __nv_bfloat16 hi, lo;
            split_bf16(decayed, hi, lo);
            q_hi[t * s.dim_pad + c] = hi;
            q_lo[t * s.dim_pad + c] = lo;
            fq[t * pitch + c] = hi;
            fq[(kBlock + t) * pitch + c] = lo;
            split_bf16(k * expf(running - z[t]), hi, lo);
            k_hi[t * s.dim_pad + c] = hi;
            k_lo[t * s.dim_pad + c] = lo;
            split_bf16(k * expf(fminf(-z[t], -kFactoredLimit)), hi, lo);
            fk[t * pitch + c] = hi;
            fk[(kBlock + t) * pitch + c] = lo;
        }
    }
    if (__syncthreads_or(strong ? 1 : 0) == 0) {
        // P = (q exp(a)) (k exp(-a))^T, one 16 x 16 product of split operands
        if (warp == 0) {
            float acc[2][4] = {};
            for (int k0 = 0; k0 < s.dim_pad; k0 += 16) {
                uint32_t a[2][4], b[2][4];
#pragma unroll
                for (int part = 0; part < 2; ++part) {
                    ldmatrix_x4(smem_u32(fq + (part * kBlock + (lane & 15)) * pitch + k0 + (lane >> 4) * 8), a[part][0], a[part][1],
                                a[part][2], a[part][3]);
                    ldmatrix_x4(smem_u32(fk + (part * kBlock + (lane & 7) + ((lane >> 4) << 3)) * pitch + k0 + ((lane >> 3) & 1) * 8),
                                b[part][0], b[part][1], b[part][2], b[part][3]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    mma_m16n8k16<__nv_bfloat16>(acc[n], a[0][0], a[0][1], a[0][2], a[0][3], b[0][2 * n], b[0][2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(acc[n], a[0][0], a[0][1], a[0][2], a[0][3], b[1][2 * n], b[1][2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(acc[n], a[1][0], a[1][1], a[1][2], a[1][3], b[0][2 * n], b[0][2 * n + 1]);
                }
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int t = (lane >> 2) + half * 8, j = n * 8 + (lane & 3) * 2;
                    const float x = j <= t ? acc[n][2 * half] : 0.0f, y = j + 1 <= t ? acc[n][2 * half + 1] : 0.0f;
                    uint32_t hi, lo;
                    split_pair(x, y, hi, lo);
                    *reinterpret_cast<uint32_t *>(p_hi + t * kBlock + j) = hi;
                    *reinterpret_cast<uint32_t *>(p_lo + t * kBlock + j) = lo;
                }
            }
        }
    } else {
        // Decays too strong to factor: k_j is carried to the later tokens by the decays themselves, one multiplication a
        // token.  A warp takes four columns j, its lanes the channels; lane pair l ends up with the sum of row t = l.
        for (int j = warp; j < kBlock; j += kPrepareThreads / 32) {
            float sum[kBlock] = {};
            for (int c = lane; c < s.dim_pad; c += 32) {
                float carried = key[j * s.dim_pad + c];
#pragma unroll
                for (int t = 0; t < kBlock; ++t) {
                    if (t > j) carried *= alpha[t * s.dim_pad + c];
                    if (t >= j) sum[t] = fmaf(query[t * s.dim_pad + c], carried, sum[t]);
                }
            }
#pragma unroll
            for (int half = 8; half >= 1; half >>= 1) {
                const bool upper = (lane & (2 * half)) != 0;
#pragma unroll
                for (int i = 0; i < half; ++i) {
                    const float sent = upper ? sum[i] : sum[i + half];
                    const float kept = upper ? sum[i + half] : sum[i];
                    sum[i] = kept + __shfl_xor_sync(0xffffffffu, sent, 2 * half);
                }
            }
            const float value = sum[0] + __shfl_xor_sync(0xffffffffu, sum[0], 1);
            if ((lane & 1) == 0) {
                const int t = lane >> 1;
                __nv_bfloat16 hi, lo;
                split_bf16(t >= j ? value : 0.0f, hi, lo);
                p_hi[t * kBlock + j] = hi;
                p_lo[t * kBlock + j] = lo;
            }
        }
    }
}

// Shared-memory stage of the advance kernel (bytes): q hi, q lo, k hi, k lo, P hi, P lo, decay, v, g with padded rows.
struct StageLayout {
    int pitch_k, pitch_v;  // bytes of a row
    int k_hi, p_hi, decay, v, g, bytes;
};

constexpr int kPitchP = kBlock * 2 + 16;

__host__ __device__ inline StageLayout stage_layout(int dim_pad, int vdim_pad) {
    StageLayout l;
    l.pitch_k = dim_pad * 2 + 16;
    l.pitch_v = vdim_pad * 2 + 16;
    l.k_hi = 2 * kBlock * l.pitch_k;
    l.p_hi = 4 * kBlock * l.pitch_k;
    l.decay = l.p_hi + 2 * kBlock * kPitchP;
    l.v = l.decay + dim_pad * 4;
    l.g = l.v + kBlock * l.pitch_v;
    l.bytes = l.g + kBlock * l.pitch_v;
    return l;
}

// KT = dim_pad / 16; MT = 16-row value tiles of a warp.
template <int KT, int MT, bool STATE_ONLY>
__global__ void __launch_bounds__(KT <= 4 ? 512 : 256) gated_linear_advance_kernel(const PromptParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    constexpr int kDim = KT * 16;
    const PromptShape &s = p.shape;
    const int segment = blockIdx.x, head = blockIdx.y;
    const int sequence = p.segments[4 * segment], first_block = p.segments[4 * segment + 1];
    const int blocks = p.segments[4 * segment + 2], before = p.segments[4 * segment + 3];
    const bool last = p.segment_last[segment] != 0;
    if (STATE_ONLY && last) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const int g = lane >> 2, q2 = (lane & 3) * 2;
    const StageLayout layout = stage_layout(kDim, s.vdim_pad);
    extern __shared__ __align__(128) uint8_t advance_shared[];
    float *squares = reinterpret_cast<float *>(advance_shared + kStages * layout.bytes);  // [warps][16]
    const size_t state_size = static_cast<size_t>(s.vdim_pad) * kDim;
    const size_t slot = static_cast<size_t>(segment) * s.heads + head;
    const int value0 = warp * MT * 16;

    // ---- the state before the segment, S^T: rows v, columns k ----
    float state[MT][2 * KT][4];
    float *home = p.state + (static_cast<size_t>(sequence) * s.heads + head) * s.dim * s.vdim;
    if (before == 0) {
        const bool fresh = p.context[sequence] == 0;
        const bool parked = !STATE_ONLY && !last;  // the first pass keeps a copy: the last segment overwrites the original
        float *start = p.segment_start + slot * state_size;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
#pragma unroll
            for (int n = 0; n < 2 * KT; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int v = value0 + m * 16 + g + (i >> 1) * 8, k = n * 8 + q2 + (i & 1);
                    if (parked) {
                        state[m][n][i] = start[static_cast<size_t>(v) * kDim + k];
                    } else {
                        state[m][n][i] = !fresh && v < s.vdim && k < s.dim ? home[static_cast<size_t>(k) * s.vdim + v] : 0.0f;
                        if (STATE_ONLY) start[static_cast<size_t>(v) * kDim + k] = state[m][n][i];
                    }
                }
            }
        }
    } else {
#pragma unroll
        for (int m = 0; m < MT; ++m) {
#pragma unroll
            for (int n = 0; n < 2 * KT; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) state[m][n][i] = 0.0f;
            }
        }
        if (!STATE_ONLY) {
            for (int earlier = segment - before; earlier < segment; ++earlier) {
                const size_t at = static_cast<size_t>(earlier) * s.heads + head;
                const float *end = p.segment_state + at * state_size;
                const float *kept = p.segment_decay + at * kDim;
#pragma unroll
                for (int n = 0; n < 2 * KT; ++n) {
                    const float2 d = *reinterpret_cast<const float2 *>(kept + n * 8 + q2);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
#pragma unroll
                        for (int half = 0; half < 2; ++half) {
                            const int v = value0 + m * 16 + g + half * 8;
                            const float2 x = *reinterpret_cast<const float2 *>(end + static_cast<size_t>(v) * kDim + n * 8 + q2);
                            state[m][n][2 * half] = fmaf(state[m][n][2 * half], d.x, x.x);
                            state[m][n][2 * half + 1] = fmaf(state[m][n][2 * half + 1], d.y, x.y);
                        }
                    }
                }
            }
        }
    }

    auto load_block = [&](int index) {
        const int block = first_block + index;
        const uint32_t stage = smem_u32(advance_shared) + (index % kStages) * layout.bytes;
        const uint8_t *pack = p.operands + (static_cast<size_t>(block) * s.heads + head) * operand_bytes(kDim);
        constexpr int kPieces = kDim / 8;
        // the state-only pass needs no queries
        for (int i = tid + (STATE_ONLY ? 2 * kBlock * kPieces : 0); i < 4 * kBlock * kPieces; i += blockDim.x) {
            load_async_16(stage + (i / kPieces) * layout.pitch_k + (i % kPieces) * 16, pack + i * 16, true);
        }
        const uint8_t *tail = pack + 4 * kBlock * kDim * 2;
        if (!STATE_ONLY) {
            for (int i = tid; i < 2 * kBlock * 2; i += blockDim.x) {
                load_async_16(stage + layout.p_hi + (i >> 1) * kPitchP + (i & 1) * 16, tail + i * 16, true);
            }
        }
        for (int i = tid; i < kDim / 4; i += blockDim.x) {
            load_async_16(stage + layout.decay + i * 16, tail + 2 * kBlock * kBlock * 2 + i * 16, true);
        }
        const int row0 = p.block_row[block], tokens = p.block_tokens[block];
        const int value_pieces = s.vdim_pad / 8;
        const __nv_bfloat16 *values = p.projected + 2 * s.heads * s.dim + head * s.vdim;
        for (int i = tid; i < kBlock * value_pieces; i += blockDim.x) {
            const int t = i / value_pieces, piece = i - t * value_pieces;
            const bool valid = t < tokens && piece * 8 < s.vdim;
            const __nv_bfloat16 *source = values + (row0 + (valid ? t : 0)) * p.stride + (valid ? piece * 8 : 0);
            load_async_16(stage + layout.v + t * layout.pitch_v + piece * 16, source, valid);
            if (!STATE_ONLY) {
                load_async_16(stage + layout.g + t * layout.pitch_v + piece * 16, source + s.heads * s.vdim, valid);
            }
        }
    };
    for (int i = 0; i < kStages - 1; ++i) {
        if (i < blocks) load_block(i);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    float kept[2 * KT][2];  // product of the segment's decays (STATE_ONLY)
    if (STATE_ONLY) {
#pragma unroll
        for (int n = 0; n < 2 * KT; ++n) kept[n][0] = kept[n][1] = 1.0f;
    }

    for (int index = 0; index < blocks; ++index) {
        asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
        __syncthreads();  // the block has arrived for every thread, and everyone is done with the stage loaded next
        if (index + kStages - 1 < blocks) load_block(index + kStages - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        uint8_t *here = advance_shared + (index % kStages) * layout.bytes;
        const uint32_t stage = smem_u32(here);

        uint32_t value[MT][4];  // v^T of this warp: rows v, columns tokens
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int t = (lane & 7) + ((lane >> 4) << 3);
            ldmatrix_x4_trans(stage + layout.v + t * layout.pitch_v + (value0 + m * 16 + ((lane >> 3) & 1) * 8) * 2, value[m][0],
                              value[m][1], value[m][2], value[m][3]);
        }
        float o[MT][2][4] = {};
        if (!STATE_ONLY) {
            // ---- o^T = S^T (q exp(a))^T ----
            const int t = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
            for (int kt = 0; kt < KT; ++kt) {
                const uint32_t at = stage + t * layout.pitch_k + (kt * 16 + ((lane >> 3) & 1) * 8) * 2;
                uint32_t hi[4], lo[4];
                ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kBlock * layout.pitch_k, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    uint32_t sh[4], sl[4];
                    split_pair(state[m][2 * kt][0], state[m][2 * kt][1], sh[0], sl[0]);
                    split_pair(state[m][2 * kt][2], state[m][2 * kt][3], sh[1], sl[1]);
                    split_pair(state[m][2 * kt + 1][0], state[m][2 * kt + 1][1], sh[2], sl[2]);
                    split_pair(state[m][2 * kt + 1][2], state[m][2 * kt + 1][3], sh[3], sl[3]);
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], sh[0], sh[1], sh[2], sh[3], hi[2 * n], hi[2 * n + 1]);
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], sh[0], sh[1], sh[2], sh[3], lo[2 * n], lo[2 * n + 1]);
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], sl[0], sl[1], sl[2], sl[3], hi[2 * n], hi[2 * n + 1]);
                    }
                }
            }
            // ---- o^T += v^T P^T ----
            {
                const uint32_t at = stage + layout.p_hi + t * kPitchP + ((lane >> 3) & 1) * 16;
                uint32_t hi[4], lo[4];
                ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kBlock * kPitchP, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], value[m][0], value[m][1], value[m][2], value[m][3], hi[2 * n], hi[2 * n + 1]);
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], value[m][0], value[m][1], value[m][2], value[m][3], lo[2 * n], lo[2 * n + 1]);
                    }
                }
            }
        }
        // ---- S^T = S^T exp(A) + v^T (k exp(A - a)) ----
#pragma unroll
        for (int kt = 0; kt < KT; ++kt) {
            const uint32_t at = stage + layout.k_hi + (lane & 15) * layout.pitch_k + (kt * 16 + (lane >> 4) * 8) * 2;
            uint32_t hi[4], lo[4];
            ldmatrix_x4_trans(at, hi[0], hi[1], hi[2], hi[3]);
            ldmatrix_x4_trans(at + kBlock * layout.pitch_k, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float2 d = *reinterpret_cast<const float2 *>(here + layout.decay + (kt * 16 + n * 8 + q2) * 4);
                if (STATE_ONLY) {
                    kept[2 * kt + n][0] *= d.x;
                    kept[2 * kt + n][1] *= d.y;
                }
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    float(&x)[4] = state[m][2 * kt + n];
                    x[0] *= d.x;
                    x[1] *= d.y;
                    x[2] *= d.x;
                    x[3] *= d.y;
                    mma_m16n8k16<__nv_bfloat16>(x, value[m][0], value[m][1], value[m][2], value[m][3], hi[2 * n], hi[2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(x, value[m][0], value[m][1], value[m][2], value[m][3], lo[2 * n], lo[2 * n + 1]);
                }
            }
        }
        if (!STATE_ONLY) {
            // ---- RMS norm over the head's values, gate, store ----
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float square = 0.0f;
#pragma unroll
                    for (int m = 0; m < MT; ++m) square += o[m][n][i] * o[m][n][i] + o[m][n][2 + i] * o[m][n][2 + i];
                    square += __shfl_xor_sync(0xffffffffu, square, 4);
                    square += __shfl_xor_sync(0xffffffffu, square, 8);
                    square += __shfl_xor_sync(0xffffffffu, square, 16);
                    if (g == 0) squares[warp * kBlock + n * 8 + q2 + i] = square;
                }
            }
            __syncthreads();
            float scale[2][2];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float total = 0.0f;
                    for (int w = 0; w < warps; ++w) total += squares[w * kBlock + n * 8 + q2 + i];
                    scale[n][i] = 1.0f / sqrtf(total / static_cast<float>(s.vdim) + p.eps);
                }
            }
            __nv_bfloat16 *gates = reinterpret_cast<__nv_bfloat16 *>(here + layout.g);  // overwritten by the result
            const int pitch = layout.pitch_v / 2;
#pragma unroll
            for (int m = 0; m < MT; ++m) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int v = value0 + m * 16 + g + half * 8;
                    const float weight = v < s.vdim ? __bfloat162float(p.norm_weight[v]) : 0.0f;
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
#pragma unroll
                        for (int i = 0; i < 2; ++i) {
                            __nv_bfloat16 *cell = gates + (n * 8 + q2 + i) * pitch + v;
                            const float gate = __bfloat162float(*cell);
                            *cell = __float2bfloat16_rn(o[m][n][2 * half + i] * scale[n][i] * weight * silu_fast(gate));
                        }
                    }
                }
            }
            __syncthreads();
            const int block = first_block + index;
            const int row0 = p.block_row[block], tokens = p.block_tokens[block];
            const int pieces = s.vdim / 8;
            for (int i = tid; i < tokens * pieces; i += blockDim.x) {
                const int t = i / pieces, piece = i - t * pieces;
                *reinterpret_cast<uint4 *>(p.out + (row0 + t) * p.out_stride + head * s.vdim + piece * 8) =
                    *reinterpret_cast<const uint4 *>(gates + t * pitch + piece * 8);
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");

    if (STATE_ONLY) {
        float *end = p.segment_state + slot * state_size;
#pragma unroll
        for (int n = 0; n < 2 * KT; ++n) {
#pragma unroll
            for (int m = 0; m < MT; ++m) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int v = value0 + m * 16 + g + half * 8;
                    *reinterpret_cast<float2 *>(end + static_cast<size_t>(v) * kDim + n * 8 + q2) =
                        make_float2(state[m][n][2 * half], state[m][n][2 * half + 1]);
                }
            }
            // the first segment's end state already holds what the sequence came with
            if (warp == 0 && g == 0) {
                *reinterpret_cast<float2 *>(p.segment_decay + slot * kDim + n * 8 + q2) = make_float2(kept[n][0], kept[n][1]);
            }
        }
    } else if (last) {
#pragma unroll
        for (int m = 0; m < MT; ++m) {
#pragma unroll
            for (int n = 0; n < 2 * KT; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int v = value0 + m * 16 + g + (i >> 1) * 8, k = n * 8 + q2 + (i & 1);
                    if (v < s.vdim && k < s.dim) home[static_cast<size_t>(k) * s.vdim + v] = state[m][n][i];
                }
            }
        }
    }
}

template <int KT, int MT>
int launch_advance(cudaStream_t stream, const PromptParams &p, size_t segments, bool cut, int warps) {
    const StageLayout layout = stage_layout(KT * 16, p.shape.vdim_pad);
    const int bytes = kStages * layout.bytes + warps * kBlock * 4;
    if (bytes > 227 * 1024) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    static int configured[kMaxDevices] = {0};
    static int configured_state[kMaxDevices] = {0};
    const dim3 grid(static_cast<unsigned>(segments), static_cast<unsigned>(p.shape.heads));
    if (cut) {
        SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_advance_kernel<KT, MT, true>, bytes, configured_state));
        SINGE_CUDA_TRY(launch_dependent(gated_linear_advance_kernel<KT, MT, true>, grid, dim3(warps * 32), bytes, stream,
                                        kLaunchGlue, 1, p));
    }
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_advance_kernel<KT, MT, false>, bytes, configured));
    SINGE_CUDA_TRY(launch_dependent(gated_linear_advance_kernel<KT, MT, false>, grid, dim3(warps * 32), bytes, stream,
                                    kLaunchGlue, 1, p));
    return launch_status();
}

// Padded sizes, or false when the state of a head does not fit the registers of a CTA.
bool prompt_tiling(size_t dim, size_t vdim, int &dim_pad, int &value_tiles, int &warps) {
    if (dim == 0 || vdim == 0 || dim > 256 || dim % 8 != 0 || vdim % 8 != 0) return false;
    dim_pad = 16;
    while (static_cast<size_t>(dim_pad) < dim) dim_pad *= 2;
    const int tiles = static_cast<int>((vdim + 15) / 16);
    const int most = dim_pad <= 64 ? 16 : 8;  // warps: 32 (64) state registers a thread at one (two) tiles leave room for 512 threads
    value_tiles = tiles <= most ? 1 : 2;
    warps = (tiles + value_tiles - 1) / value_tiles;
    return warps <= most && !(dim_pad == 256 && value_tiles == 2);
}

size_t align256(size_t bytes) { return (bytes + 255) / 256 * 256; }

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

size_t singe_gated_linear_prompt_scratch(size_t heads, size_t dim, size_t vdim, size_t blocks, size_t segments) {
    int dim_pad, value_tiles, warps;
    if (!prompt_tiling(dim, vdim, dim_pad, value_tiles, warps)) return 0;
    const size_t state = static_cast<size_t>(dim_pad) * value_tiles * 16 * warps * sizeof(float);
    return align256(blocks * heads * operand_bytes(dim_pad)) + 2 * align256(segments * heads * state) +
           align256(segments * heads * dim_pad * sizeof(float));
}

int singe_gated_linear_prompt_bf16(singe_stream_t stream, void *out, size_t out_stride, const void *projected,
                                   size_t projected_stride, const void *decay_weight, const void *decay_bias,
                                   const void *norm_weight, float *state, const int32_t *context, size_t heads, size_t dim,
                                   size_t vdim, size_t rank, float tau, float query_scale, float eps,
                                   const int32_t *block_row, const int32_t *block_tokens, size_t blocks,
                                   const int32_t *segments, const int32_t *segment_last, size_t segment_count, int cut,
                                   void *scratch) {
    if (heads == 0 || rank == 0 || blocks == 0 || segment_count == 0 || out_stride < heads * vdim ||
        projected_stride < 2 * heads * (dim + vdim) + rank) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(blocks) || !fits_i32(segment_count) || !fits_i32(projected_stride) || heads > 65535) {
        return SINGE_ERR_LENGTH_EXCEEDS_I32;
    }
    if (out == nullptr || projected == nullptr || decay_weight == nullptr || decay_bias == nullptr || norm_weight == nullptr ||
        state == nullptr || context == nullptr || block_row == nullptr || block_tokens == nullptr || segments == nullptr ||
        segment_last == nullptr || scratch == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    int dim_pad, value_tiles, warps;
    if (!prompt_tiling(dim, vdim, dim_pad, value_tiles, warps) || projected_stride % 8 != 0 || out_stride % 8 != 0 ||
        ((reinterpret_cast<uintptr_t>(projected) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(scratch)) & 15u) != 0) {
        return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    }
    PromptParams p = {};
    p.shape.heads = static_cast<int>(heads);
    p.shape.dim = static_cast<int>(dim);
    p.shape.vdim = static_cast<int>(vdim);
    p.shape.rank = static_cast<int>(rank);
    p.shape.dim_pad = dim_pad;
    p.shape.vdim_pad = value_tiles * 16 * warps;
    p.out = static_cast<__nv_bfloat16 *>(out);
    p.out_stride = static_cast<long long>(out_stride);
    p.projected = static_cast<const __nv_bfloat16 *>(projected);
    p.stride = static_cast<long long>(projected_stride);
    p.decay_weight = static_cast<const __nv_bfloat16 *>(decay_weight);
    p.decay_bias = static_cast<const __nv_bfloat16 *>(decay_bias);
    p.norm_weight = static_cast<const __nv_bfloat16 *>(norm_weight);
    p.state = state;
    p.context = context;
    p.block_row = block_row;
    p.block_tokens = block_tokens;
    p.segments = segments;
    p.segment_last = segment_last;
    p.operands = static_cast<uint8_t *>(scratch);
    const size_t state_bytes = static_cast<size_t>(dim_pad) * p.shape.vdim_pad * sizeof(float);
    uint8_t *at = p.operands + align256(blocks * heads * operand_bytes(dim_pad));
    p.segment_state = reinterpret_cast<float *>(at);
    at += align256(segment_count * heads * state_bytes);
    p.segment_start = reinterpret_cast<float *>(at);
    at += align256(segment_count * heads * state_bytes);
    p.segment_decay = reinterpret_cast<float *>(at);
    p.inverse_tau = 1.0f / tau;
    p.query_scale = query_scale;
    p.eps = eps;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    const size_t shared = (kBlock * rank + 3 * kBlock * dim_pad) * sizeof(float) + 4 * kBlock * (dim_pad + 8) * 2;
    if (shared > 227 * 1024) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_prepare_kernel, static_cast<int>(shared), configured));
    SINGE_CUDA_TRY(launch_dependent(gated_linear_prepare_kernel,
                                    dim3(static_cast<unsigned>(blocks), static_cast<unsigned>(heads)), dim3(kPrepareThreads),
                                    shared, s, kLaunchGlue, 1, p));
    const bool segmented = cut != 0;
#define SINGE_ADVANCE(KT_, MT_) \
    if (dim_pad == KT_ * 16 && value_tiles == MT_) return launch_advance<KT_, MT_>(s, p, segment_count, segmented, warps);
    SINGE_ADVANCE(1, 1)
    SINGE_ADVANCE(1, 2)
    SINGE_ADVANCE(2, 1)
    SINGE_ADVANCE(2, 2)
    SINGE_ADVANCE(4, 1)
    SINGE_ADVANCE(4, 2)
    SINGE_ADVANCE(8, 1)
    SINGE_ADVANCE(8, 2)
    SINGE_ADVANCE(16, 1)
#undef SINGE_ADVANCE
    return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
}

}  // extern "C"
