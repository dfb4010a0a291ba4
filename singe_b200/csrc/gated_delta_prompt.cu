// Gated delta rule over prompts: the recurrence of gated_delta.cu (same operands, same meaning), block by block on the tensor
// core.
//
// In a block of 16 tokens let a_t be the running sum of log g per key channel (A the last one's) and S the state before the
// block.  The written rows u_t solve a unit lower-triangular system,
//     (I + M) u = beta (v - (k exp(a))^T S),     M_tj = beta_t sum_c k_tc k_jc exp(a_tc - a_jc)  for j < t,
// so that with T = (I + M)^-1 diag(beta) and W = T (k exp(a)),
//     u   = T v - W S,
//     o_t = (q_t exp(a_t))^T S + sum_(j <= t) P_tj u_j,     P_tj = sum_c q_tc k_jc exp(a_tc - a_jc),
//     S'  = exp(A) S + sum_j (k_j exp(A - a_j)) u_j^T.
// Every exponent that reaches a product is <= 0 except in the factored form of M and P, which is only used where the block's
// whole decay stays above e^-60.
//
// 32-bit without 32-bit tensor cores: operands that are f32 by nature enter the bf16 MMA as two terms hi + lo (2^-17 of the
// value is lost) and their products keep hi hi + hi lo + lo hi; v is bf16 from its convolution and enters as it is.
// Accumulators, and the state between the blocks, are f32.
//
//   prepare   one CTA per (block, head): decays, M and its inverse, P and the split operands, to scratch, laid out as the next
//             kernel's shared memory wants them, so that a block arrives in one bulk copy
//   advance   one CTA per (sequence, head, slice of the values): the blocks in order, the state in registers as S^T [vdim, dim],
//             whose accumulator layout is the A-operand layout of the next product.  The columns of the state do not meet, so
//             slices run side by side.
//   finish    RMS norm over a head's values, gate, store
#include "row_pack.cuh"
#include "split_bf16.cuh"

namespace singe {
namespace {

constexpr int kMaxStages = 6;
constexpr float kFactoredLimit = -60.0f;
constexpr int kPitchP = kBlock * 2 + 16;  // bytes of a padded row of P or T

// The operands of one (block, head), bytes: q exp(a) hi, lo; W hi, lo; k exp(A - a) hi, lo; P hi, lo; T hi, lo; exp(A).
struct DeltaLayout {
    int pitch;  // bytes of a padded row of q, W or k
    int w, k, p, t, decay, bytes;
};

__host__ __device__ constexpr DeltaLayout delta_layout(int dim_pad) {
    DeltaLayout l = {};
    l.pitch = dim_pad * 2 + 16;
    l.w = 2 * kBlock * l.pitch;
    l.k = 2 * l.w;
    l.p = 3 * l.w;
    l.t = l.p + 2 * kBlock * kPitchP;
    l.decay = l.t + 2 * kBlock * kPitchP;
    l.bytes = l.decay + dim_pad * 4;
    return l;
}

struct DeltaParams {
    int heads, kv_heads, dim, vdim, key_at, value_at, gate_at;
    int dim_pad, slice;       // slice: value columns of an advance CTA, 16 per warp
    __nv_bfloat16 *out;
    long long out_stride;
    const __nv_bfloat16 *mixed;
    long long mixed_stride;
    const float *inverse;
    const __nv_bfloat16 *strength;
    long long strength_stride;
    const __nv_bfloat16 *decay;
    long long decay_stride;
    const float *rate, *bias;
    const __nv_bfloat16 *norm_weight;
    float *state;
    const int32_t *context;
    const int32_t *block_row, *block_tokens;  // first packed row and tokens of each block
    const int32_t *runs;                      // [n][3]: sequence, first block, blocks
    int blocks;
    uint8_t *operands;                        // [blocks, heads] packs
    float *attended;                          // [rows, heads * vdim]: o before its norm
    float eps;
    uint32_t *error;
    int stages;
};

// Shared memory of the prepare kernel: the operands as they will go out, (k exp(-a)) hi and lo, a 16 x 17 matrix, three numbers a
// token, and the decay of either half of the block per channel.
__host__ __device__ constexpr int prepare_bytes(int dim_pad) {
    return delta_layout(dim_pad).bytes + 2 * kBlock * (dim_pad * 2 + 16) + kBlock * 17 * 4 + 3 * kBlock * 4 + dim_pad * 8;
}

// acc (two n tiles of 8) += A[16, 16 rows at a] . B[16 rows at b, same columns]^T over `columns`, split operands.
__device__ __forceinline__ void product_rows(float (&acc)[2][4], uint32_t a_at, uint32_t b_at, int pitch, int columns) {
    for (int k0 = 0; k0 < columns; k0 += 16) {
        uint32_t a[2][4], b[2][4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const uint32_t offset = half * kBlock * pitch + k0 * 2;
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
}

__device__ __forceinline__ float low_half(uint32_t pair) { return __uint_as_float(pair << 16); }
__device__ __forceinline__ float high_half(uint32_t pair) { return __uint_as_float(pair & 0xffff0000u); }

// One CTA per (block, head); a thread takes two adjacent channels of one half of the block's tokens.
__global__ void __launch_bounds__(256) gated_delta_prepare_kernel(const DeltaParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    constexpr int kHalf = kBlock / 2;
    const int block = blockIdx.x, head = blockIdx.y;
    const int row0 = p.block_row[block], tokens = p.block_tokens[block];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
    const DeltaLayout layout = delta_layout(p.dim_pad);
    extern __shared__ __align__(128) uint8_t prepare_shared[];
    const int half_bytes = kBlock * layout.pitch;  // from the hi to the lo part
    uint8_t *pack = prepare_shared;
    uint8_t *fq = pack, *fa = pack + layout.w;  // k exp(a) is where W goes, column tile by column tile
    uint8_t *fk = pack + layout.bytes;
    float *matrix = reinterpret_cast<float *>(fk + 2 * half_bytes);  // [16][17]
    float *betas = matrix + kBlock * 17, *units_q = betas + kBlock, *units_k = units_q + kBlock;
    float2 *totals = reinterpret_cast<float2 *>(units_k + kBlock);   // [2 halves][dim_pad / 2]
    const int source = head / (p.heads / p.kv_heads);
    const float rate = expf(p.rate[head]);

    if (tid < kBlock) {
        float beta = 0.0f, unit_q = 0.0f, unit_k = 0.0f;
        if (tid < tokens) {
            const long long row = row0 + tid;
            unit_q = p.inverse[row * 2 * p.kv_heads + source] / sqrtf(static_cast<float>(p.dim));
            unit_k = p.inverse[row * 2 * p.kv_heads + p.kv_heads + source];
            beta = 1.0f / (1.0f + expf(-__bfloat162float(p.strength[row * p.strength_stride + head])));
        }
        betas[tid] = beta;
        units_q[tid] = unit_q;
        units_k[tid] = unit_k;
    }
    const int pairs = p.dim_pad / 2;
    const int c = 2 * (tid % pairs), half = tid / pairs;
    const bool inside = half < 2, real = inside && c < p.dim;  // dim is a multiple of eight
    const int t0 = half * kHalf, channel = head * p.dim + (real ? c : 0);
    uint32_t q_raw[kHalf], k_raw[kHalf], z_raw[kHalf];
    {
        const __nv_bfloat16 *rows = p.mixed + (row0 + t0) * p.mixed_stride + source * p.dim + (real ? c : 0);
        const __nv_bfloat16 *decays = p.decay + (row0 + t0) * p.decay_stride + channel;
#pragma unroll
        for (int i = 0; i < kHalf; ++i) {
            const bool live = real && t0 + i < tokens;
            z_raw[i] = live ? *reinterpret_cast<const uint32_t *>(decays + i * p.decay_stride) : 0u;
            q_raw[i] = live ? *reinterpret_cast<const uint32_t *>(rows + i * p.mixed_stride) : 0u;
            k_raw[i] = live ? *reinterpret_cast<const uint32_t *>(rows + i * p.mixed_stride + p.key_at) : 0u;
        }
    }
    // running sums of the log decays, over this half and then over the block
    float2 sum[kHalf];
    {
        const float2 bias = real ? *reinterpret_cast<const float2 *>(p.bias + channel) : make_float2(0.0f, 0.0f);
        float2 running = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int i = 0; i < kHalf; ++i) {
            if (real && t0 + i < tokens) {
                const float x = low_half(z_raw[i]) + bias.x, y = high_half(z_raw[i]) + bias.y;
                running.x -= rate * (fmaxf(x, 0.0f) + log1pf(__expf(-fabsf(x))));
                running.y -= rate * (fmaxf(y, 0.0f) + log1pf(__expf(-fabsf(y))));
            }
            sum[i] = running;
        }
        if (inside) totals[half * pairs + c / 2] = running;
    }
    __syncthreads();
    bool strong = false;
    if (inside) {
        const float2 first = totals[c / 2], second = totals[pairs + c / 2];
        const float2 total = make_float2(first.x + second.x, first.y + second.y);
        if (half == 1) {
#pragma unroll
            for (int i = 0; i < kHalf; ++i) sum[i] = make_float2(sum[i].x + first.x, sum[i].y + first.y);
        }
        const bool factors = fminf(total.x, total.y) >= kFactoredLimit;
        strong = !factors;
        const float2 whole = make_float2(__expf(total.x), __expf(total.y));
        if (half == 0) *reinterpret_cast<float2 *>(pack + layout.decay + c * 4) = whole;
#pragma unroll
        for (int i = 0; i < kHalf; ++i) {
            const float uq = units_q[t0 + i], uk = units_k[t0 + i];
            // exp(a_t), exp(A - a_t), exp(-a_t)
            const float2 before = make_float2(__expf(sum[i].x), __expf(sum[i].y));
            float2 after, back = make_float2(0.0f, 0.0f);
            if (factors) {
                back = make_float2(__expf(-sum[i].x), __expf(-sum[i].y));
                after = make_float2(whole.x * back.x, whole.y * back.y);
            } else {
                after = make_float2(__expf(total.x - sum[i].x), __expf(total.y - sum[i].y));
            }
            const float q0 = low_half(q_raw[i]) * uq, q1 = high_half(q_raw[i]) * uq;
            const float k0 = low_half(k_raw[i]) * uk, k1 = high_half(k_raw[i]) * uk;
            const int at = (t0 + i) * layout.pitch + c * 2;
            uint32_t hi, lo;
            split_pair(q0 * before.x, q1 * before.y, hi, lo);
            *reinterpret_cast<uint32_t *>(fq + at) = hi;
            *reinterpret_cast<uint32_t *>(fq + half_bytes + at) = lo;
            split_pair(k0 * after.x, k1 * after.y, hi, lo);
            *reinterpret_cast<uint32_t *>(pack + layout.k + at) = hi;
            *reinterpret_cast<uint32_t *>(pack + layout.k + half_bytes + at) = lo;
            split_pair(k0 * back.x, k1 * back.y, hi, lo);
            *reinterpret_cast<uint32_t *>(fk + at) = hi;
            *reinterpret_cast<uint32_t *>(fk + half_bytes + at) = lo;
            split_pair(k0 * before.x, k1 * before.y, hi, lo);
            *reinterpret_cast<uint32_t *>(fa + at) = hi;
            *reinterpret_cast<uint32_t *>(fa + half_bytes + at) = lo;
        }
    }
    // ---- P, and M (not yet times beta) ----
    uint8_t *p_hi = pack + layout.p, *p_lo = p_hi + kBlock * kPitchP;
    uint8_t *t_hi = pack + layout.t, *t_lo = t_hi + kBlock * kPitchP;
    if (__syncthreads_or(strong ? 1 : 0) == 0) {
        const int a_offset = (lane & 15) * layout.pitch + (lane >> 4) * 16;
        const int b_offset = ((lane & 7) + ((lane >> 4) << 3)) * layout.pitch + ((lane >> 3) & 1) * 16;
        if (warp == 0) {
            float scores[2][4] = {};
            product_rows(scores, smem_u32(fq) + a_offset, smem_u32(fk) + b_offset, layout.pitch, p.dim_pad);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int t = (lane >> 2) + i * 8, j = n * 8 + (lane & 3) * 2;
                    uint32_t hi, lo;
                    split_pair(j <= t ? scores[n][2 * i] : 0.0f, j + 1 <= t ? scores[n][2 * i + 1] : 0.0f, hi, lo);
                    *reinterpret_cast<uint32_t *>(p_hi + t * kPitchP + j * 2) = hi;
                    *reinterpret_cast<uint32_t *>(p_lo + t * kPitchP + j * 2) = lo;
                }
            }
        }
        if (warp == warps - 1) {
            float keys[2][4] = {};
            product_rows(keys, smem_u32(fa) + a_offset, smem_u32(fk) + b_offset, layout.pitch, p.dim_pad);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int t = (lane >> 2) + (i >> 1) * 8, j = n * 8 + (lane & 3) * 2 + (i & 1);
                    matrix[t * 17 + j] = j < t ? keys[n][i] : 0.0f;
                }
            }
        }
    } else {
        // Decays too strong to factor: every pair's decay is taken as one exponential.  The running sums go where k exp(-a)
        // was; the lanes are the channels, the warps take the pairs in turn.
        float *sums = reinterpret_cast<float *>(fk);  // [16][dim_pad]
        if (inside) {
#pragma unroll
            for (int i = 0; i < kHalf; ++i) *reinterpret_cast<float2 *>(sums + (t0 + i) * p.dim_pad + c) = sum[i];
        }
        __syncthreads();
        const __nv_bfloat16 *queries = p.mixed + row0 * p.mixed_stride + source * p.dim, *keys = queries + p.key_at;
        for (int item = warp; item < kBlock * kBlock; item += warps) {
            const int t = item / kBlock, j = item % kBlock;
            float score = 0.0f, dot = 0.0f;
            if (j <= t && t < tokens) {
                for (int d = lane; d < p.dim; d += 32) {
                    const float carried = __bfloat162float(keys[j * p.mixed_stride + d]) * units_k[j] *
                                          __expf(sums[t * p.dim_pad + d] - sums[j * p.dim_pad + d]);
                    score = fmaf(__bfloat162float(queries[t * p.mixed_stride + d]) * units_q[t], carried, score);
                    dot = fmaf(__bfloat162float(keys[t * p.mixed_stride + d]) * units_k[t], carried, dot);
                }
                score = warp_sum(score);
                dot = warp_sum(dot);
            }
            if (lane == 0) {
                __nv_bfloat16 hi, lo;
                split_bf16(score, hi, lo);
                *reinterpret_cast<__nv_bfloat16 *>(p_hi + t * kPitchP + j * 2) = hi;
                *reinterpret_cast<__nv_bfloat16 *>(p_lo + t * kPitchP + j * 2) = lo;
                matrix[t * 17 + j] = j < t ? dot : 0.0f;
            }
        }
    }
    __syncthreads();
    // ---- T = (I + diag(beta) M)^-1 diag(beta): a lane solves for one column ----
    if (warp == 0) {
        float x[kBlock];
        const int j = lane & 15;
#pragma unroll
        for (int t = 0; t < kBlock; ++t) {
            float known = 0.0f;
#pragma unroll
            for (int i = 0; i < t; ++i) known = fmaf(matrix[t * 17 + i], x[i], known);
            x[t] = (t == j ? 1.0f : 0.0f) - betas[t] * known;
        }
        __syncwarp();
        const float beta = betas[j];
        if (lane < kBlock) {
#pragma unroll
            for (int t = 0; t < kBlock; ++t) {
                const float value = x[t] * beta;
                matrix[t * 17 + j] = value;
                __nv_bfloat16 hi, lo;
                split_bf16(value, hi, lo);
                *reinterpret_cast<__nv_bfloat16 *>(t_hi + t * kPitchP + j * 2) = hi;
                *reinterpret_cast<__nv_bfloat16 *>(t_lo + t * kPitchP + j * 2) = lo;
            }
        }
    }
    __syncthreads();
    // ---- W = T (k exp(a)) ----
    uint32_t sh[4], sl[4];  // T as A operand
    {
        const int t = lane >> 2, j = (lane & 3) * 2;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float *cell = matrix + (t + (i & 1) * 8) * 17 + j + (i >> 1) * 8;
            split_pair(cell[0], cell[1], sh[i], sl[i]);
        }
    }
    const uint32_t w_at = smem_u32(fa) + (lane & 15) * layout.pitch + (lane >> 4) * 16;
    for (int c0 = warp * 16; c0 < p.dim_pad; c0 += warps * 16) {
        uint32_t hi[4], lo[4];
        ldmatrix_x4_trans(w_at + c0 * 2, hi[0], hi[1], hi[2], hi[3]);
        ldmatrix_x4_trans(w_at + half_bytes + c0 * 2, lo[0], lo[1], lo[2], lo[3]);
        __syncwarp();  // the tile has been read by all lanes
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            float acc[4] = {};
            mma_m16n8k16<__nv_bfloat16>(acc, sh[0], sh[1], sh[2], sh[3], hi[2 * n], hi[2 * n + 1]);
            mma_m16n8k16<__nv_bfloat16>(acc, sh[0], sh[1], sh[2], sh[3], lo[2 * n], lo[2 * n + 1]);
            mma_m16n8k16<__nv_bfloat16>(acc, sl[0], sl[1], sl[2], sl[3], hi[2 * n], hi[2 * n + 1]);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int at = ((lane >> 2) + i * 8) * layout.pitch + (c0 + n * 8 + (lane & 3) * 2) * 2;
                uint32_t x, y;
                split_pair(acc[2 * i], acc[2 * i + 1], x, y);
                *reinterpret_cast<uint32_t *>(pack + layout.w + at) = x;
                *reinterpret_cast<uint32_t *>(pack + layout.w + half_bytes + at) = y;
            }
        }
    }
    // ---- out in one bulk copy ----
    fence_proxy_async_shared();
    __syncthreads();
    if (tid == 0) {
        bulk_store(p.operands + (static_cast<size_t>(block) * p.heads + head) * layout.bytes, smem_u32(pack), layout.bytes);
        tma_store_commit();
        tma_store_wait<0>();
    }
}

// Stage of the advance kernel (bytes): the operands as prepared, then the slice's values in TMA boxes.
__host__ __device__ inline int delta_values_at(int dim_pad) { return (delta_layout(dim_pad).bytes + 1023) / 1024 * 1024; }
__host__ __device__ inline int delta_stage_bytes(int dim_pad, int slice) {
    return delta_values_at(dim_pad) + (slice + 63) / 64 * kValueBox;
}

// KT = dim_pad / 16.  16 value rows of the slice belong to KS warps, each with KT / KS of the key tiles: with few (sequence, head)
// pairs one warp's products are what a block waits for, and sharing them pays for bringing the sums together.
template <int KT, int KS>
__global__ void __launch_bounds__(256, KT / KS <= 8 ? 2 : 1) gated_delta_advance_kernel(const __grid_constant__ CUtensorMap value_map,
                                                                                       const DeltaParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    constexpr int kDim = KT * 16, kTiles = KT / KS;
    constexpr DeltaLayout kLayout = delta_layout(kDim);
    constexpr int kHalf = kBlock * kLayout.pitch;
    const int run = blockIdx.x, head = blockIdx.y, slice0 = blockIdx.z * p.slice;
    const int sequence = p.runs[3 * run], first_block = p.runs[3 * run + 1], blocks = p.runs[3 * run + 2];
    // a run's rows are adjacent, and only its last block may be short
    const int first_row = p.block_row[first_block], last_tokens = p.block_tokens[first_block + blocks - 1];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, q2 = (lane & 3) * 2;
    const int share = warp % KS, tile0 = share * kTiles;  // this warp's key tiles
    const int stages = p.stages;
    const int stage_bytes = delta_stage_bytes(kDim, p.slice), values_at = delta_values_at(kDim);
    extern __shared__ uint8_t advance_raw[];
    uint8_t *advance_shared = advance_raw + ((1024u - (smem_u32(advance_raw) & 1023u)) & 1023u);
    float4 *sums = reinterpret_cast<float4 *>(advance_shared + stages * stage_bytes);  // [warps][4][32], KS > 1
    const uint32_t bars = smem_u32(sums + (KS > 1 ? blockDim.x * 4 : 0));
    if (tid == 0) {
        for (int i = 0; i < stages; ++i) mbar_init(bars + 8 * i, 1);
        mbar_init_fence();
    }
    __syncthreads();

    const int value0 = warp / KS * 16;  // within the slice
    float state[2 * kTiles][4];         // S^T: rows v, columns k
    float *home = p.state + (static_cast<size_t>(sequence) * p.heads + head) * p.dim * p.vdim;
    const bool fresh = p.context[sequence] == 0;
#pragma unroll
    for (int n = 0; n < 2 * kTiles; ++n) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int v = slice0 + value0 + g + (i >> 1) * 8, k = tile0 * 16 + n * 8 + q2 + (i & 1);
            state[n][i] = !fresh && v < p.vdim && k < p.dim ? home[static_cast<size_t>(k) * p.vdim + v] : 0.0f;
        }
    }

    // One warp brings a block in.  What a box holds past a short block or past the head's columns belongs to other rows or
    // columns (finite values): it meets zeros in T, or is never stored.
    const int boxes = (p.slice + 63) / 64;
    auto load_block = [&](int index, int slot) {
        if (warp != 0) return;
        const uint32_t bar = bars + 8 * slot;
        const uint32_t stage = smem_u32(advance_shared) + slot * stage_bytes;
        if (lane == 0) {
            mbar_expect_tx(bar, kLayout.bytes + boxes * kValueBox);
            bulk_load(stage, p.operands + (static_cast<size_t>(first_block + index) * p.heads + head) * kLayout.bytes, kLayout.bytes, bar);
        }
        __syncwarp();
        if (lane < boxes) {
            tma_load_2d(stage + values_at + lane * kValueBox, &value_map, bar,
                        p.value_at + head * p.vdim + slice0 + lane * 64, first_row + index * kBlock);
        }
    };
    for (int i = 0; i < stages - 1 && i < blocks; ++i) load_block(i, i);
    bool failed = false;
    int slot = 0, round = 0;

    for (int index = 0; index < blocks; ++index, round ^= slot == 0) {
        const int here_slot = slot, next_slot = slot == 0 ? stages - 1 : slot - 1;
        const int parity = round;
        slot = slot + 1 == stages ? 0 : slot + 1;
        const int row0 = first_row + index * kBlock, tokens = index + 1 < blocks ? kBlock : last_tokens;
        const bool arrived = mbar_wait(bars + 8 * here_slot, parity);
        fence_proxy_async_shared();
        // the block has arrived for every thread, and everyone is done with the stage loaded next and with the sums
        if (__syncthreads_or(arrived ? 0 : 1) != 0) {
            failed = true;
            break;
        }
        if (index + stages - 1 < blocks) load_block(index + stages - 1, next_slot);
        uint8_t *here = advance_shared + here_slot * stage_bytes;
        const uint32_t stage = smem_u32(here);
        const int t = (lane & 7) + ((lane >> 4) << 3);

        uint32_t value[4];  // v^T of this warp: rows v, columns tokens
        ldmatrix_x4_trans(stage + values_at + value_at(t, value0 + ((lane >> 3) & 1) * 8), value[0], value[1], value[2], value[3]);
        // ---- S^T W^T and S^T (q exp(a))^T; the small terms are dependency chains of their own ----
        float o[2][4] = {}, u[2][4] = {};
        {
            float o_low[2][4] = {}, u_low[2][4] = {};
#pragma unroll
            for (int kt = 0; kt < kTiles; ++kt) {
                const uint32_t at = stage + t * kLayout.pitch + ((tile0 + kt) * 16 + ((lane >> 3) & 1) * 8) * 2;
                uint32_t sh[4], sl[4], hi[4], lo[4];
                split_pair(state[2 * kt][0], state[2 * kt][1], sh[0], sl[0]);
                split_pair(state[2 * kt][2], state[2 * kt][3], sh[1], sl[1]);
                split_pair(state[2 * kt + 1][0], state[2 * kt + 1][1], sh[2], sl[2]);
                split_pair(state[2 * kt + 1][2], state[2 * kt + 1][3], sh[3], sl[3]);
                ldmatrix_x4(at + kLayout.w, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kLayout.w + kHalf, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    mma_m16n8k16<__nv_bfloat16>(u[n], sh[0], sh[1], sh[2], sh[3], hi[2 * n], hi[2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(u_low[n], sh[0], sh[1], sh[2], sh[3], lo[2 * n], lo[2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(u_low[n], sl[0], sl[1], sl[2], sl[3], hi[2 * n], hi[2 * n + 1]);
                }
                ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
                ldmatrix_x4(at + kHalf, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    mma_m16n8k16<__nv_bfloat16>(o[n], sh[0], sh[1], sh[2], sh[3], hi[2 * n], hi[2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(o_low[n], sh[0], sh[1], sh[2], sh[3], lo[2 * n], lo[2 * n + 1]);
                    mma_m16n8k16<__nv_bfloat16>(o_low[n], sl[0], sl[1], sl[2], sl[3], hi[2 * n], hi[2 * n + 1]);
                }
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    o[n][i] += o_low[n][i];
                    u[n][i] += u_low[n][i];
                }
            }
        }
        if (KS > 1) {
            float4 *mine = sums + warp * 128 + lane;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                mine[n * 32] = make_float4(u[n][0], u[n][1], u[n][2], u[n][3]);
                mine[(2 + n) * 32] = make_float4(o[n][0], o[n][1], o[n][2], o[n][3]);
            }
            __syncthreads();
            const float4 *all = sums + (warp - share) * 128 + lane;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
#pragma unroll
                for (int i = 0; i < 4; ++i) u[n][i] = o[n][i] = 0.0f;
#pragma unroll
                for (int other = 0; other < KS; ++other) {
                    const float4 x = all[other * 128 + n * 32];
                    u[n][0] += x.x;
                    u[n][1] += x.y;
                    u[n][2] += x.z;
                    u[n][3] += x.w;
                    if (share == 0) {
                        const float4 y = all[other * 128 + (2 + n) * 32];
                        o[n][0] += y.x;
                        o[n][1] += y.y;
                        o[n][2] += y.z;
                        o[n][3] += y.w;
                    }
                }
            }
        }
        // ---- u^T = v^T T^T - S^T W^T ----
        uint32_t uh[4], ul[4];
        {
            const uint32_t at = stage + kLayout.t + t * kPitchP + ((lane >> 3) & 1) * 16;
            uint32_t hi[4], lo[4];
            ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
            ldmatrix_x4(at + kBlock * kPitchP, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                float direct[4] = {};
                mma_m16n8k16<__nv_bfloat16>(direct, value[0], value[1], value[2], value[3], hi[2 * n], hi[2 * n + 1]);
                mma_m16n8k16<__nv_bfloat16>(direct, value[0], value[1], value[2], value[3], lo[2 * n], lo[2 * n + 1]);
#pragma unroll
                for (int i = 0; i < 4; ++i) u[n][i] = direct[i] - u[n][i];
                split_pair(u[n][0], u[n][1], uh[2 * n], ul[2 * n]);
                split_pair(u[n][2], u[n][3], uh[2 * n + 1], ul[2 * n + 1]);
            }
        }
        // ---- S^T = S^T exp(A) + u^T (k exp(A - a)) ----
#pragma unroll
        for (int kt = 0; kt < kTiles; ++kt) {
            const uint32_t at = stage + kLayout.k + (lane & 15) * kLayout.pitch + ((tile0 + kt) * 16 + (lane >> 4) * 8) * 2;
            uint32_t hi[4], lo[4];
            ldmatrix_x4_trans(at, hi[0], hi[1], hi[2], hi[3]);
            ldmatrix_x4_trans(at + kHalf, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float2 d = *reinterpret_cast<const float2 *>(here + kLayout.decay + ((tile0 + kt) * 16 + n * 8 + q2) * 4);
                float(&x)[4] = state[2 * kt + n];
                x[0] *= d.x;
                x[1] *= d.y;
                x[2] *= d.x;
                x[3] *= d.y;
                mma_m16n8k16<__nv_bfloat16>(x, uh[0], uh[1], uh[2], uh[3], hi[2 * n], hi[2 * n + 1]);
                mma_m16n8k16<__nv_bfloat16>(x, uh[0], uh[1], uh[2], uh[3], lo[2 * n], lo[2 * n + 1]);
                mma_m16n8k16<__nv_bfloat16>(x, ul[0], ul[1], ul[2], ul[3], hi[2 * n], hi[2 * n + 1]);
            }
        }
        // ---- o^T += u^T P^T; eight lanes hold eight adjacent values of a token ----
        if (share == 0) {
            const uint32_t at = stage + kLayout.p + t * kPitchP + ((lane >> 3) & 1) * 16;
            uint32_t hi[4], lo[4];
            ldmatrix_x4(at, hi[0], hi[1], hi[2], hi[3]);
            ldmatrix_x4(at + kBlock * kPitchP, lo[0], lo[1], lo[2], lo[3]);
            float *target = p.attended + static_cast<size_t>(row0) * p.heads * p.vdim + head * p.vdim + slice0 + value0;
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                mma_m16n8k16<__nv_bfloat16>(o[n], uh[0], uh[1], uh[2], uh[3], hi[2 * n], hi[2 * n + 1]);
                mma_m16n8k16<__nv_bfloat16>(o[n], uh[0], uh[1], uh[2], uh[3], lo[2 * n], lo[2 * n + 1]);
                mma_m16n8k16<__nv_bfloat16>(o[n], ul[0], ul[1], ul[2], ul[3], hi[2 * n], hi[2 * n + 1]);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int token = n * 8 + q2 + (i & 1), v = g + (i >> 1) * 8;
                    if (token < tokens && slice0 + value0 + v < p.vdim) target[static_cast<size_t>(token) * p.heads * p.vdim + v] = o[n][i];
                }
            }
        }
    }
    if (failed) {
        if (tid == 0) report_status(p.error, kStatusWaitTimeout);
        linger_after_timeout();
        return;
    }
#pragma unroll
    for (int n = 0; n < 2 * kTiles; ++n) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int v = slice0 + value0 + g + (i >> 1) * 8, k = tile0 * 16 + n * 8 + q2 + (i & 1);
            if (v < p.vdim && k < p.dim) home[static_cast<size_t>(k) * p.vdim + v] = state[n][i];
        }
    }
}

// One warp per (token, head), four in turn: out = rms_norm(o) * weight * sigmoid(gate).  HELD: a head's values are at most one pack a
// lane, and everything is asked for before the sums.
template <bool HELD>
__global__ void __launch_bounds__(256) gated_delta_finish_kernel(const DeltaParams p) {
    grid_launch_dependents();
    grid_dependency_wait();
    constexpr int kTurns = 4;
    const int block = blockIdx.x;
    const int row0 = p.block_row[block], tokens = p.block_tokens[block];
    const int lane = threadIdx.x & 31, packs = p.vdim / 4, items = tokens * p.heads;
    const float inverse_vdim = 1.0f / static_cast<float>(p.vdim);
    auto store = [&](Pack<4> x, const Pack<4> &gate, const Pack<4> &weight, float scale, __nv_bfloat16 *out) {
#pragma unroll
        for (int j = 0; j < 4; ++j) x.v[j] = x.v[j] * scale * weight.v[j] * __fdividef(1.0f, 1.0f + __expf(-gate.v[j]));
        store_pack<4>(out, x);
    };
    Pack<4> held_weight = {};
    if (HELD && lane < packs) held_weight = load_pack<4>(p.norm_weight + lane * 4);
    for (int item0 = (blockIdx.y * 8 + (threadIdx.x >> 5)) * kTurns; item0 < items; item0 += gridDim.y * 8 * kTurns) {
        if (HELD) {
            Pack<4> x[kTurns], gate[kTurns];
            __nv_bfloat16 *out[kTurns];
#pragma unroll
            for (int turn = 0; turn < kTurns; ++turn) {
                const int item = item0 + turn, token = item / p.heads, head = item - token * p.heads;
                const size_t row = row0 + token;
                x[turn] = {};
                out[turn] = p.out + row * p.out_stride + head * p.vdim + lane * 4;
                if (item < items && lane < packs) {
                    x[turn] = load_pack<4>(p.attended + row * p.heads * p.vdim + head * p.vdim + lane * 4);
                    gate[turn] = load_pack<4>(p.decay + row * p.decay_stride + p.gate_at + head * p.vdim + lane * 4);
                }
            }
#pragma unroll
            for (int turn = 0; turn < kTurns; ++turn) {
                float square = 0.0f;
#pragma unroll
                for (int j = 0; j < 4; ++j) square = square_chain(square, x[turn].v[j]);
                const float scale = 1.0f / sqrtf(warp_sum(square) * inverse_vdim + p.eps);
                if (item0 + turn < items && lane < packs) store(x[turn], gate[turn], held_weight, scale, out[turn]);
            }
        } else {
            for (int item = item0; item < min(item0 + kTurns, items); ++item) {
                const int token = item / p.heads, head = item - token * p.heads;
                const size_t row = row0 + token;
                const float *o = p.attended + row * p.heads * p.vdim + head * p.vdim;
                float square = 0.0f;
                for (int i = lane; i < packs; i += 32) {
                    const Pack<4> x = load_pack<4>(o + i * 4);
#pragma unroll
                    for (int j = 0; j < 4; ++j) square = square_chain(square, x.v[j]);
                }
                const float scale = 1.0f / sqrtf(warp_sum(square) * inverse_vdim + p.eps);
                for (int i = lane; i < packs; i += 32) {
                    store(load_pack<4>(o + i * 4), load_pack<4>(p.decay + row * p.decay_stride + p.gate_at + head * p.vdim + i * 4),
                          load_pack<4>(p.norm_weight + i * 4), scale, p.out + row * p.out_stride + head * p.vdim + i * 4);
                }
            }
        }
    }
}

template <int KT, int KS>
int launch_advance(cudaStream_t stream, const CUtensorMap &value_map, DeltaParams p, size_t runs) {
    const int threads = p.slice * 2 * KS;
    const auto bytes_of = [&](int stages) {
        return stages * delta_stage_bytes(KT * 16, p.slice) + (KS > 1 ? threads * 64 : 0) + kMaxStages * 8 + 1024;
    };
    p.stages = kMaxStages;  // as many as leave room for a second CTA, three at least
    while (p.stages > 3 && bytes_of(p.stages) > 112 * 1024) --p.stages;
    if (bytes_of(p.stages) > 227 * 1024) return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    const dim3 grid(static_cast<unsigned>(runs), static_cast<unsigned>(p.heads),
                    static_cast<unsigned>((p.vdim + p.slice - 1) / p.slice));
    // A grid that leaves SMs idle must not put two CTAs on one: those that launch while the kernel before drains would.  More than
    // half of an SM's shared memory keeps them apart.
    int bytes = bytes_of(p.stages);
    const size_t ctas = static_cast<size_t>(grid.x) * grid.y * grid.z;
    if (ctas <= static_cast<size_t>(device_sm_count()) && bytes < 120 * 1024) bytes = 120 * 1024;
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_delta_advance_kernel<KT, KS>, bytes, configured));
    SINGE_CUDA_TRY(launch_dependent(gated_delta_advance_kernel<KT, KS>, grid, dim3(threads), bytes, stream, kLaunchGlue, 1, value_map, p));
    return launch_status();
}

// The padded key size, or 0 for sizes the block form does not take.
int delta_dim_pad(size_t dim, size_t vdim) {
    if (dim == 0 || vdim == 0 || dim > 256 || dim % 8 != 0 || vdim % 8 != 0) return 0;
    int pad = 16;
    while (static_cast<size_t>(pad) < dim) pad *= 2;
    return pad;
}

// Value columns of a CTA: all of a head's up to 128, fewer while (run, head, slice) triples leave SMs idle.  `shared_keys`: so few
// that the key tiles are shared out among four warps as well.
int delta_slice(size_t runs, size_t heads, size_t vdim, int dim_pad, bool &shared_keys) {
    const size_t sms = static_cast<size_t>(device_sm_count());
    shared_keys = dim_pad >= 64 && runs * heads * ((vdim + 15) / 16) < 2 * sms;
    if (shared_keys) return runs * heads * ((vdim + 15) / 16) <= sms ? 16 : 32;
    int slice = 16;
    while (slice < 128 && static_cast<size_t>(slice) < vdim) slice *= 2;
    while (slice > 16 && runs * heads * ((vdim + slice - 1) / slice) < sms) slice /= 2;
    return slice;
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

size_t singe_gated_delta_prompt_scratch(size_t heads, size_t dim, size_t vdim, size_t rows, size_t blocks) {
    const int dim_pad = delta_dim_pad(dim, vdim);
    if (dim_pad == 0) return 0;
    return align256(blocks * heads * delta_layout(dim_pad).bytes) + align256(rows * heads * vdim * sizeof(float));
}

int singe_gated_delta_prompt_bf16(singe_stream_t stream, void *out, size_t out_stride, const void *mixed, size_t mixed_stride,
                                  const float *inverse, const void *strength, size_t strength_stride, const void *decay,
                                  size_t decay_stride, const float *rate, const float *bias, const void *norm_weight, float *state,
                                  const int32_t *context, size_t rows, size_t heads, size_t kv_heads, size_t dim, size_t vdim,
                                  size_t key_at, size_t value_at, size_t gate_at, float eps, const int32_t *block_row,
                                  const int32_t *block_tokens, size_t blocks, const int32_t *runs, size_t run_count, void *scratch) {
    if (rows == 0 || heads == 0 || kv_heads == 0 || heads % kv_heads != 0 || blocks == 0 || run_count == 0 ||
        key_at < kv_heads * dim || value_at < key_at + kv_heads * dim || mixed_stride < value_at + heads * vdim ||
        gate_at < heads * dim || decay_stride < gate_at + heads * vdim || strength_stride < heads || out_stride < heads * vdim) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(rows) || !fits_i32(blocks) || !fits_i32(run_count) || !fits_i32(mixed_stride) || !fits_i32(decay_stride) ||
        heads > 65535) {
        return SINGE_ERR_LENGTH_EXCEEDS_I32;
    }
    if (out == nullptr || mixed == nullptr || inverse == nullptr || strength == nullptr || decay == nullptr || rate == nullptr ||
        bias == nullptr || norm_weight == nullptr || state == nullptr || context == nullptr || block_row == nullptr ||
        block_tokens == nullptr || runs == nullptr || scratch == nullptr) {
        return SINGE_ERR_NULL_POINTER;
    }
    const int dim_pad = delta_dim_pad(dim, vdim);
    if (dim_pad == 0 || mixed_stride % 8 != 0 || decay_stride % 8 != 0 || out_stride % 8 != 0 || key_at % 8 != 0 ||
        value_at % 8 != 0 || gate_at % 8 != 0 || !aligned_to(mixed, 16) || !aligned_to(decay, 16) || !aligned_to(out, 16) ||
        !aligned_to(norm_weight, 8) || !aligned_to(bias, 8) || !aligned_to(scratch, 16)) {
        return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    }
    DeltaParams p = {};
    p.heads = static_cast<int>(heads);
    p.kv_heads = static_cast<int>(kv_heads);
    p.dim = static_cast<int>(dim);
    p.vdim = static_cast<int>(vdim);
    p.key_at = static_cast<int>(key_at);
    p.value_at = static_cast<int>(value_at);
    p.gate_at = static_cast<int>(gate_at);
    p.dim_pad = dim_pad;
    bool shared_keys = false;
    p.slice = delta_slice(run_count, heads, vdim, dim_pad, shared_keys);
    p.out = static_cast<__nv_bfloat16 *>(out);
    p.out_stride = static_cast<long long>(out_stride);
    p.mixed = static_cast<const __nv_bfloat16 *>(mixed);
    p.mixed_stride = static_cast<long long>(mixed_stride);
    p.inverse = inverse;
    p.strength = static_cast<const __nv_bfloat16 *>(strength);
    p.strength_stride = static_cast<long long>(strength_stride);
    p.decay = static_cast<const __nv_bfloat16 *>(decay);
    p.decay_stride = static_cast<long long>(decay_stride);
    p.rate = rate;
    p.bias = bias;
    p.norm_weight = static_cast<const __nv_bfloat16 *>(norm_weight);
    p.state = state;
    p.context = context;
    p.block_row = block_row;
    p.block_tokens = block_tokens;
    p.runs = runs;
    p.blocks = static_cast<int>(blocks);
    p.operands = static_cast<uint8_t *>(scratch);
    p.attended = reinterpret_cast<float *>(p.operands + align256(blocks * heads * delta_layout(dim_pad).bytes));
    p.eps = eps;
    p.error = device_error_word();
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(gated_delta_prepare_kernel, prepare_bytes(dim_pad), configured));
    SINGE_CUDA_TRY(launch_dependent(gated_delta_prepare_kernel, dim3(static_cast<unsigned>(blocks), static_cast<unsigned>(heads)),
                                    dim3(dim_pad < 32 ? 32 : dim_pad), prepare_bytes(dim_pad), s, kLaunchGlue, 1, p));
    CUtensorMap value_map;
    {
        const uint64_t dims[2] = {value_at + heads * vdim, rows};
        const uint64_t strides[1] = {mixed_stride * 2};
        const uint32_t box[2] = {64, kBlock};
        SINGE_TRY(encode_tensor_map(&value_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, mixed, dims, strides, box,
                                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B));
    }
    int launched = SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    if (dim_pad == 16) launched = launch_advance<1, 1>(s, value_map, p, run_count);
    if (dim_pad == 32) launched = launch_advance<2, 1>(s, value_map, p, run_count);
    if (dim_pad == 64) {
        launched = shared_keys ? launch_advance<4, 4>(s, value_map, p, run_count) : launch_advance<4, 1>(s, value_map, p, run_count);
    }
    if (dim_pad == 128) {
        launched = shared_keys ? launch_advance<8, 4>(s, value_map, p, run_count) : launch_advance<8, 1>(s, value_map, p, run_count);
    }
    if (dim_pad == 256) {
        launched = shared_keys ? launch_advance<16, 4>(s, value_map, p, run_count) : launch_advance<16, 1>(s, value_map, p, run_count);
    }
    SINGE_TRY(launched);
    const unsigned groups = static_cast<unsigned>((heads * kBlock + 127) / 128);  // four (token, head) pairs, four times, a warp
    SINGE_CUDA_TRY(launch_dependent(vdim <= 128 ? gated_delta_finish_kernel<true> : gated_delta_finish_kernel<false>,
                                    dim3(static_cast<unsigned>(blocks), groups), dim3(256), 0, s, kLaunchGlue, 1, p));
    return launch_status();
}

}  // extern "C"
