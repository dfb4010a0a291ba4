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
//   prepare   one warp per (block, head): decays, the split operands and P, to scratch, laid out as the next kernel's
//             shared memory wants them (rows padded against bank conflicts), so that a block arrives in one bulk copy
//   advance   one CTA per (segment, head): the blocks of a segment in order, the state in registers as S^T [vdim, dim], whose
//             accumulator layout is the A-operand layout of the next product.  A warp owns 16 (or 32) value rows.
//             A long sequence is cut into segments that run side by side: a first pass (STATE_ONLY) takes every segment
//             but the last from a zero state (the first one from the sequence's state) to its end, and in the second
//             pass a segment starts from the fold of its predecessors' end states.
#include "split_bf16.cuh"

namespace singe {
namespace {

constexpr int kPrepareWarps = 4;
constexpr int kMaxStages = 6;
constexpr float kFactoredLimit = -60.0f;
constexpr int kPitchP = kBlock * 2 + 16;  // bytes of a padded row of P

// The operands of one (block, head), bytes: q hi, q lo, P hi, P lo, and from `state_part` on what the state needs: k hi,
// k lo, decay.
struct OperandLayout {
    int pitch;  // bytes of a padded row of q or k
    int p_hi, state_part, decay, bytes;
};

__host__ __device__ constexpr OperandLayout operand_layout(int dim_pad) {
    OperandLayout l = {};
    l.pitch = dim_pad * 2 + 16;
    l.p_hi = 2 * kBlock * l.pitch;
    l.state_part = l.p_hi + 2 * kBlock * kPitchP;
    l.decay = l.state_part + 2 * kBlock * l.pitch;
    l.bytes = l.decay + dim_pad * 4;
    return l;
}

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
    uint32_t *error;
    int stages;  // blocks on their way to a CTA, plus the one in use
};

__host__ __device__ constexpr int operand_bytes(int dim_pad) { return operand_layout(dim_pad).bytes; }

// Shared memory of one warp of the prepare kernel, in bytes: the factored operands of P (q hi, lo, k hi, lo) and the
// logarithms of the decays.
__host__ __device__ constexpr int prepare_warp_bytes(int dim_pad) {
    return 4 * kBlock * (dim_pad * 2 + 16) + kBlock * dim_pad * 4;
}

__global__ void __launch_bounds__(kPrepareWarps * 32) gated_linear_prepare_kernel(const PromptParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    const PromptShape &s = p.shape;
    const int block = blockIdx.x;
    const int row0 = p.block_row[block], tokens = p.block_tokens[block];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const OperandLayout layout = operand_layout(s.dim_pad);
    extern __shared__ __align__(16) uint8_t prepare_shared[];
    float *low = reinterpret_cast<float *>(prepare_shared);  // [rank][16]
    uint8_t *own = prepare_shared + kBlock * s.rank * 4 + warp * prepare_warp_bytes(s.dim_pad);
    uint8_t *fq = own, *fk = own + 2 * kBlock * layout.pitch;
    float *steps = reinterpret_cast<float *>(own + 4 * kBlock * layout.pitch);  // [16][dim_pad]

    const int low_at = 2 * s.heads * (s.dim + s.vdim);
    for (int i = threadIdx.x; i < kBlock * s.rank; i += blockDim.x) {
        const int t = i / s.rank, r = i - t * s.rank;
        low[r * kBlock + t] = t < tokens ? __bfloat162float(p.projected[(row0 + t) * p.stride + low_at + r]) : 0.0f;
    }
    __syncthreads();
    const int head = blockIdx.y * kPrepareWarps + warp;
    if (head >= s.heads) return;
    uint8_t *pack = p.operands + (static_cast<size_t>(block) * s.heads + head) * layout.bytes;
    uint8_t *q_out = pack, *k_out = pack + layout.state_part;
    float *decay = reinterpret_cast<float *>(pack + layout.decay);

    bool strong = false;
    for (int c = 2 * lane; c < s.dim_pad; c += 64) {  // a lane takes two adjacent channels
        const bool real = c < s.dim;                   // dim is a multiple of eight
        const int channel = head * s.dim + (real ? c : 0);
        uint32_t q_raw[kBlock], k_raw[kBlock];
        const __nv_bfloat16 *source = p.projected + row0 * p.stride + channel;
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            const bool live = real && t < tokens;
            q_raw[t] = live ? *reinterpret_cast<const uint32_t *>(source + t * p.stride) : 0u;
            k_raw[t] = live ? *reinterpret_cast<const uint32_t *>(source + t * p.stride + s.heads * s.dim) : 0u;
        }
        float z[2][kBlock] = {};
        if (real) {
            const __nv_bfloat16 *weight = p.decay_weight + static_cast<size_t>(channel) * s.rank;
#pragma unroll 4
            for (int r = 0; r < s.rank; ++r) {
                const float w0 = __bfloat162float(weight[r]), w1 = __bfloat162float(weight[s.rank + r]);
#pragma unroll
                for (int t = 0; t < kBlock; t += 4) {
                    const float4 x = *reinterpret_cast<const float4 *>(low + r * kBlock + t);
                    z[0][t] = fmaf(w0, x.x, z[0][t]);
                    z[0][t + 1] = fmaf(w0, x.y, z[0][t + 1]);
                    z[0][t + 2] = fmaf(w0, x.z, z[0][t + 2]);
                    z[0][t + 3] = fmaf(w0, x.w, z[0][t + 3]);
                    z[1][t] = fmaf(w1, x.x, z[1][t]);
                    z[1][t + 1] = fmaf(w1, x.y, z[1][t + 1]);
                    z[1][t + 2] = fmaf(w1, x.z, z[1][t + 2]);
                    z[1][t + 3] = fmaf(w1, x.w, z[1][t + 3]);
                }
            }
        }
        float total[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float bias = real ? __bfloat162float(p.decay_bias[channel + i]) : 0.0f;
            float running = 0.0f;
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                const float x = z[i][t] + bias;
                // log(sigmoid(x)) / tau, without cancellation for either sign
                const float step = real && t < tokens ? (fminf(x, 0.0f) - log1pf(__expf(-fabsf(x)))) * p.inverse_tau : 0.0f;
                steps[t * s.dim_pad + c + i] = step;
                running += step;
                z[i][t] = running;
            }
            total[i] = running;
        }
        const bool factors = fminf(total[0], total[1]) >= kFactoredLimit;
        strong = strong || !factors;
        const float whole[2] = {__expf(total[0]), __expf(total[1])};
        *reinterpret_cast<float2 *>(decay + c) = make_float2(whole[0], whole[1]);
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            float before[2], after[2], back[2];  // exp(a_t), exp(A - a_t), exp(-a_t)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                before[i] = __expf(z[i][t]);
                if (factors) {
                    back[i] = __expf(-z[i][t]);
                    after[i] = whole[i] * back[i];
                } else {
                    back[i] = __expf(fminf(-z[i][t], -kFactoredLimit));
                    after[i] = __expf(total[i] - z[i][t]);
                }
            }
            const float q0 = __uint_as_float(q_raw[t] << 16) * p.query_scale, q1 = __uint_as_float(q_raw[t] & 0xffff0000u) * p.query_scale;
            const float k0 = __uint_as_float(k_raw[t] << 16), k1 = __uint_as_float(k_raw[t] & 0xffff0000u);
            const int at = t * layout.pitch + c * 2, low_half = kBlock * layout.pitch;
            uint32_t hi, lo;
            split_pair(q0 * before[0], q1 * before[1], hi, lo);
            *reinterpret_cast<uint32_t *>(q_out + at) = hi;
            *reinterpret_cast<uint32_t *>(q_out + low_half + at) = lo;
            *reinterpret_cast<uint32_t *>(fq + at) = hi;
            *reinterpret_cast<uint32_t *>(fq + low_half + at) = lo;
            split_pair(k0 * after[0], k1 * after[1], hi, lo);
            *reinterpret_cast<uint32_t *>(k_out + at) = hi;
            *reinterpret_cast<uint32_t *>(k_out + low_half + at) = lo;
            split_pair(k0 * back[0], k1 * back[1], hi, lo);
            *reinterpret_cast<uint32_t *>(fk + at) = hi;
            *reinterpret_cast<uint32_t *>(fk + low_half + at) = lo;
        }
    }
    __syncwarp();
    uint8_t *p_hi = pack + layout.p_hi, *p_lo = p_hi + kBlock * kPitchP;
    if (!__any_sync(0xffffffffu, strong)) {
        // P = (q exp(a)) (k exp(-a))^T, one 16 x 16 product of split operands
        float acc[2][4] = {};
        const uint32_t a_at = smem_u32(fq) + (lane & 15) * layout.pitch + (lane >> 4) * 16;
        const uint32_t b_at = smem_u32(fk) + ((lane & 7) + ((lane >> 4) << 3)) * layout.pitch + ((lane >> 3) & 1) * 16;
        for (int k0 = 0; k0 < s.dim_pad; k0 += 16) {
            uint32_t a[2][4], b[2][4];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const uint32_t offset = half * kBlock * layout.pitch + k0 * 2;
                ldmatrix_x4(a_at + offset, a[half][0], a[half][1], a[half][2], a[half][3]);
                ldmatrix_x4(b_at + offset, b[half][0], b[half][1], b[half][2], b[half][3]);
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
                *reinterpret_cast<uint32_t *>(p_hi + t * kPitchP + j * 2) = hi;
                *reinterpret_cast<uint32_t *>(p_lo + t * kPitchP + j * 2) = lo;
            }
        }
        return;
    }
    // Decays too strong to factor: k_j is carried to the later tokens by the decays themselves, one multiplication a token.
    // The lanes are the channels; lane pair l ends up with the sum of row t = l.
    const __nv_bfloat16 *queries = p.projected + row0 * p.stride + head * s.dim, *keys = queries + s.heads * s.dim;
    for (int j = 0; j < kBlock; ++j) {
        float sum[kBlock] = {};
        for (int c = lane; c < s.dim && j < tokens; c += 32) {
            float carried = __bfloat162float(keys[j * p.stride + c]) * p.query_scale;
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                if (t > j) carried *= __expf(steps[t * s.dim_pad + c]);
                if (t >= j && t < tokens) sum[t] = fmaf(__bfloat162float(queries[t * p.stride + c]), carried, sum[t]);
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
            *reinterpret_cast<__nv_bfloat16 *>(p_hi + t * kPitchP + j * 2) = hi;
            *reinterpret_cast<__nv_bfloat16 *>(p_lo + t * kPitchP + j * 2) = lo;
        }
    }
}

// Shared-memory stage of the advance kernel (bytes): the operands as prepared, then v and g as TMA boxes of 16 tokens x 64
// columns, SWIZZLE_128B.
struct StageLayout {
    int v, g, bytes;
};

__host__ __device__ inline StageLayout stage_layout(int dim_pad, int vdim_pad) {
    const int boxes = (vdim_pad + 63) / 64;
    StageLayout l;
    l.v = (operand_bytes(dim_pad) + 1023) / 1024 * 1024;
    l.g = l.v + boxes * kValueBox;
    l.bytes = l.g + boxes * kValueBox;
    return l;
}

// KT = dim_pad / 16; MT = 16-row value tiles of a warp.
// THREADS bounds the CTA; small states leave registers for three CTAs of an SM, whose latencies then hide one another.
template <int KT, int MT, int THREADS, bool STATE_ONLY>
__global__ void __launch_bounds__(THREADS, KT <= 4 && THREADS <= 256 / MT ? 3 : 1) gated_linear_advance_kernel(
    const __grid_constant__ CUtensorMap value_map, const PromptParams p) {
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
    constexpr OperandLayout kOperands = operand_layout(kDim);
    const StageLayout layout = stage_layout(kDim, s.vdim_pad);
    const int stages = p.stages;
    extern __shared__ uint8_t advance_raw[];
    uint8_t *advance_shared = advance_raw + ((1024u - (smem_u32(advance_raw) & 1023u)) & 1023u);
    float *squares = reinterpret_cast<float *>(advance_shared + stages * layout.bytes);  // [8 or more][16]
    const uint32_t bars = smem_u32(squares + max(warps, 8) * kBlock);
    for (int i = tid; i < max(warps, 8) * kBlock; i += blockDim.x) squares[i] = 0.0f;
    if (tid == 0) {
        for (int i = 0; i < stages; ++i) mbar_init(bars + 8 * i, 1);
        mbar_init_fence();
    }
    __syncthreads();
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

    // One warp brings a block in: the operands in one bulk copy, v and g in boxes.  What a box holds past a short block or
    // past the head's columns belongs to other rows or columns; it meets zeros in k and P, or is never stored.
    const int value_boxes = (s.vdim_pad + 63) / 64;
    auto load_block = [&](int index) {
        if (warp != 0) return;
        const int block = first_block + index;
        const uint32_t bar = bars + 8 * (index % stages);
        const uint32_t stage = smem_u32(advance_shared) + (index % stages) * layout.bytes;
        constexpr uint32_t kFrom = STATE_ONLY ? kOperands.state_part : 0, kBytes = kOperands.bytes - kFrom;
        const int boxes = value_boxes * (STATE_ONLY ? 1 : 2);
        if (lane == 0) {
            mbar_expect_tx(bar, kBytes + boxes * kValueBox);
            bulk_load(stage + kFrom, p.operands + (static_cast<size_t>(block) * s.heads + head) * kOperands.bytes + kFrom, kBytes, bar);
        }
        __syncwarp();
        if (lane < boxes) {
            const int gate = lane < value_boxes ? 0 : 1, box = lane - gate * value_boxes;
            tma_load_2d(stage + (gate ? layout.g : layout.v) + box * kValueBox, &value_map, bar,
                        2 * s.heads * s.dim + gate * s.heads * s.vdim + head * s.vdim + box * 64, p.block_row[block]);
        }
    };
    for (int i = 0; i < stages - 1 && i < blocks; ++i) load_block(i);
    bool failed = false;
    float kept[2 * KT][2];  // product of the segment's decays (STATE_ONLY)
    if (STATE_ONLY) {
#pragma unroll
        for (int n = 0; n < 2 * KT; ++n) kept[n][0] = kept[n][1] = 1.0f;
    }

    const float inverse_vdim = 1.0f / static_cast<float>(s.vdim);
    float weight[MT][2];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int v = value0 + m * 16 + g + half * 8;
            weight[m][half] = v < s.vdim ? __bfloat162float(p.norm_weight[v]) : 0.0f;
        }
    }

    // the rows and the 16-byte piece of the output this thread stores (threads past whole rows store none)
    const int pieces = s.vdim / 8, store_rows = max(static_cast<int>(blockDim.x) / pieces, 1);
    const int store_piece = tid % pieces, store_row = tid / pieces < store_rows ? tid / pieces : kBlock;

    for (int index = 0; index < blocks; ++index) {
        const int row0 = p.block_row[first_block + index], tokens = p.block_tokens[first_block + index];
        const bool arrived = mbar_wait(bars + 8 * (index % stages), (index / stages) & 1);
        fence_proxy_async_shared();
        // the block has arrived for every thread, and everyone is done with the stage loaded next
        if (__syncthreads_or(arrived ? 0 : 1) != 0) {
            failed = true;
            break;
        }
        if (index + stages - 1 < blocks) load_block(index + stages - 1);
        uint8_t *here = advance_shared + (index % stages) * layout.bytes;
        const uint32_t stage = smem_u32(here);

        uint32_t value[MT][4];  // v^T of this warp: rows v, columns tokens
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int t = (lane & 7) + ((lane >> 4) << 3);
            ldmatrix_x4_trans(stage + layout.v + value_at(t, value0 + m * 16 + ((lane >> 3) & 1) * 8), value[m][0],
                              value[m][1], value[m][2], value[m][3]);
        }
        float o[MT][2][4] = {};
        if (!STATE_ONLY) {
            float cross[MT][2][4] = {};  // the small terms, a dependency chain of their own
            // ---- o^T = S^T (q exp(a))^T ----
            const int t = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
            for (int kt = 0; kt < KT; ++kt) {
                const uint32_t at = stage + t * kOperands.pitch + (kt * 16 + ((lane >> 3) & 1) * 8) * 2;
                uint32_t hi[4], lo[4];
                ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kBlock * kOperands.pitch, lo[0], lo[1], lo[2], lo[3]);
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
                        mma_m16n8k16<__nv_bfloat16>(cross[m][n], sh[0], sh[1], sh[2], sh[3], lo[2 * n], lo[2 * n + 1]);
                        mma_m16n8k16<__nv_bfloat16>(cross[m][n], sl[0], sl[1], sl[2], sl[3], hi[2 * n], hi[2 * n + 1]);
                    }
                }
            }
            // ---- o^T += v^T P^T ----
            {
                const uint32_t at = stage + kOperands.p_hi + t * kPitchP + ((lane >> 3) & 1) * 16;
                uint32_t hi[4], lo[4];
                ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kBlock * kPitchP, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        mma_m16n8k16<__nv_bfloat16>(o[m][n], value[m][0], value[m][1], value[m][2], value[m][3], hi[2 * n], hi[2 * n + 1]);
                        mma_m16n8k16<__nv_bfloat16>(cross[m][n], value[m][0], value[m][1], value[m][2], value[m][3], lo[2 * n], lo[2 * n + 1]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < MT; ++m) {
#pragma unroll
                for (int n = 0; n < 2; ++n) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) o[m][n][i] += cross[m][n][i];
                }
            }
        }
        // ---- S^T = S^T exp(A) + v^T (k exp(A - a)) ----
#pragma unroll
        for (int kt = 0; kt < KT; ++kt) {
            const uint32_t at = stage + kOperands.state_part + (lane & 15) * kOperands.pitch + (kt * 16 + (lane >> 4) * 8) * 2;
            uint32_t hi[4], lo[4];
            ldmatrix_x4_trans(at, hi[0], hi[1], hi[2], hi[3]);
            ldmatrix_x4_trans(at + kBlock * kOperands.pitch, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float2 d = *reinterpret_cast<const float2 *>(here + kOperands.decay + (kt * 16 + n * 8 + q2) * 4);
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
                    for (int m = 0; m < MT; ++m) {
                        const int v = value0 + m * 16 + g;  // rows past vdim hold what is not this head's
                        square += v < s.vdim ? o[m][n][i] * o[m][n][i] : 0.0f;
                        square += v + 8 < s.vdim ? o[m][n][2 + i] * o[m][n][2 + i] : 0.0f;
                    }
                    square += __shfl_xor_sync(0xffffffffu, square, 4);
                    square += __shfl_xor_sync(0xffffffffu, square, 8);
                    square += __shfl_xor_sync(0xffffffffu, square, 16);
                    if (g == 0) squares[warp * kBlock + n * 8 + q2 + i] = square;
                }
            }
            __syncthreads();
            // every lane adds up one warp's (or two warps') squares of its four tokens, then the eight lanes of a column meet
            float scale[2][2];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float2 total = *reinterpret_cast<const float2 *>(squares + g * kBlock + n * 8 + q2);
                if (warps > 8 && g + 8 < warps) {
                    const float2 more = *reinterpret_cast<const float2 *>(squares + (g + 8) * kBlock + n * 8 + q2);
                    total.x += more.x;
                    total.y += more.y;
                }
#pragma unroll
                for (int d = 4; d <= 16; d <<= 1) {
                    total.x += __shfl_xor_sync(0xffffffffu, total.x, d);
                    total.y += __shfl_xor_sync(0xffffffffu, total.y, d);
                }
                scale[n][0] = rsqrtf(total.x * inverse_vdim + p.eps);
                scale[n][1] = rsqrtf(total.y * inverse_vdim + p.eps);
            }
            // the gates come out of shared memory in the layout of o^T, and the result goes back to where they were
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const uint32_t at = stage + layout.g + value_at((lane & 7) + ((lane >> 4) << 3), value0 + m * 16 + ((lane >> 3) & 1) * 8);
                uint32_t gate[4];
                ldmatrix_x4_trans(at, gate[0], gate[1], gate[2], gate[3]);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const uint32_t pair = gate[2 * n + half];
                        const float x = o[m][n][2 * half] * scale[n][0] * weight[m][half] * silu_fast(__uint_as_float(pair << 16));
                        const float y = o[m][n][2 * half + 1] * scale[n][1] * weight[m][half] * silu_fast(__uint_as_float(pair & 0xffff0000u));
                        gate[2 * n + half] = pack2<__nv_bfloat16>(x, y);
                    }
                }
                stmatrix_x4_trans(at, gate[0], gate[1], gate[2], gate[3]);
            }
            __syncthreads();
            for (int t = store_row; t < tokens; t += store_rows) {
                *reinterpret_cast<uint4 *>(p.out + (row0 + t) * p.out_stride + head * s.vdim + store_piece * 8) =
                    *reinterpret_cast<const uint4 *>(here + layout.g + value_at(t, store_piece * 8));
            }
        }
    }
    if (failed) {
        if (tid == 0) report_status(p.error, kStatusWaitTimeout);
        linger_after_timeout();
        return;
    }
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

template <int KT, int MT, int THREADS>
int launch_advance(cudaStream_t stream, const CUtensorMap &value_map, PromptParams p, size_t segments, bool cut, int warps) {
    const StageLayout layout = stage_layout(KT * 16, p.shape.vdim_pad);
    const auto shared_bytes = [&](int stages) { return stages * layout.bytes + (warps > 8 ? warps : 8) * kBlock * 4 + kMaxStages * 8 + 1024; };
    p.stages = kMaxStages;  // as many as leave room for two more CTAs, three at least
    while (p.stages > 3 && shared_bytes(p.stages) > 75 * 1024) --p.stages;
    const int bytes = shared_bytes(p.stages);
    if (bytes > 227 * 1024) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    static int configured[kMaxDevices] = {0};
    static int configured_state[kMaxDevices] = {0};
    const dim3 grid(static_cast<unsigned>(segments), static_cast<unsigned>(p.shape.heads));
    if (cut) {
        SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_advance_kernel<KT, MT, THREADS, true>, bytes, configured_state));
        SINGE_CUDA_TRY(launch_dependent(gated_linear_advance_kernel<KT, MT, THREADS, true>, grid, dim3(warps * 32), bytes, stream,
                                        kLaunchGlue, 1, value_map, p));
    }
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_advance_kernel<KT, MT, THREADS, false>, bytes, configured));
    SINGE_CUDA_TRY(launch_dependent(gated_linear_advance_kernel<KT, MT, THREADS, false>, grid, dim3(warps * 32), bytes, stream,
                                    kLaunchGlue, 1, value_map, p));
    return launch_status();
}

// Padded sizes, or false when the state of a head does not fit the registers of a CTA.
bool prompt_tiling(size_t dim, size_t vdim, int &dim_pad, int &value_tiles, int &warps) {
    if (dim == 0 || vdim == 0 || dim > 256 || dim % 8 != 0 || vdim % 8 != 0) return false;
    dim_pad = 16;
    while (static_cast<size_t>(dim_pad) < dim) dim_pad *= 2;
    const int tiles = static_cast<int>((vdim + 15) / 16);
    const int most = dim_pad <= 64 ? 16 : 8;  // warps: 32 (64) state registers a thread at one (two) tiles leave room for 512 threads
    // two value tiles a warp share the operands it reads, where they leave the registers for it
    value_tiles = tiles <= most && (tiles % 2 != 0 || dim_pad > 64) ? 1 : 2;
    warps = (tiles + value_tiles - 1) / value_tiles;
    return warps <= most && !(dim_pad == 256 && value_tiles == 2);
}

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
                                   const void *norm_weight, float *state, const int32_t *context, size_t rows, size_t heads, size_t dim,
                                   size_t vdim, size_t rank, float tau, float query_scale, float eps,
                                   const int32_t *block_row, const int32_t *block_tokens, size_t blocks,
                                   const int32_t *segments, const int32_t *segment_last, size_t segment_count, int cut,
                                   void *scratch) {
    if (rows == 0 || heads == 0 || rank == 0 || blocks == 0 || segment_count == 0 || out_stride < heads * vdim ||
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
    p.error = device_error_word();
    const size_t shared = kBlock * rank * sizeof(float) + kPrepareWarps * prepare_warp_bytes(dim_pad);
    if (shared > 227 * 1024) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_linear_prepare_kernel, static_cast<int>(shared), configured));
    SINGE_CUDA_TRY(launch_dependent(gated_linear_prepare_kernel,
                                    dim3(static_cast<unsigned>(blocks), static_cast<unsigned>((heads + kPrepareWarps - 1) / kPrepareWarps)),
                                    dim3(kPrepareWarps * 32), shared, s, kLaunchGlue, 1, p));
    CUtensorMap value_map;
    {
        const uint64_t dims[2] = {2 * heads * (dim + vdim) + rank, rows};
        const uint64_t strides[1] = {projected_stride * 2};
        const uint32_t box[2] = {64, kBlock};
        SINGE_TRY(encode_tensor_map(&value_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, projected, dims, strides, box,
                                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B));
    }
    const bool segmented = cut != 0;
#define SINGE_ADVANCE(KT_, MT_, THREADS_)                                          \
    if (dim_pad == KT_ * 16 && value_tiles == MT_ && warps * 32 <= THREADS_) {      \
        return launch_advance<KT_, MT_, THREADS_>(s, value_map, p, segment_count, segmented, warps); \
    }
    SINGE_ADVANCE(1, 1, 256)
    SINGE_ADVANCE(1, 1, 512)
    SINGE_ADVANCE(1, 2, 128)
    SINGE_ADVANCE(1, 2, 512)
    SINGE_ADVANCE(2, 1, 256)
    SINGE_ADVANCE(2, 1, 512)
    SINGE_ADVANCE(2, 2, 128)
    SINGE_ADVANCE(2, 2, 512)
    SINGE_ADVANCE(4, 1, 256)
    SINGE_ADVANCE(4, 1, 512)
    SINGE_ADVANCE(4, 2, 128)
    SINGE_ADVANCE(4, 2, 512)
    SINGE_ADVANCE(8, 1, 256)
    SINGE_ADVANCE(8, 2, 256)
    SINGE_ADVANCE(16, 1, 256)
#undef SINGE_ADVANCE
    return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
}

}  // extern "C"
