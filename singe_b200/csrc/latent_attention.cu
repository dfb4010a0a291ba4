// Attention of few query rows (a decode step) over a paged latent cache: one cached row of `latent` bf16 per token serves
// every head as key and as value,
//     score[h, j] = scale * q[h] . c[j],   out[h] = sum_j softmax(score[h])_j c[j],
// with q already multiplied into the latent space.  A sliding window bounds the keys of a query.
//
// The cache is the traffic: a tile of 64 cached rows is read from HBM once for up to 32 heads and used twice, as keys and
// as values.  Two kernels:
//   latent_decode_tcgen05_kernel  pages of 8, 16, 32 or a multiple of 64 tokens: tiles by TMA, both products on the fifth-
//                                 generation tensor core with the heads as the N side, scores and outputs in tensor memory
//   latent_decode_kernel          any page size: cp.async and mma.sync
// With more than one split the normalised partial and its log-sum-exp (base 2) go to scratch and a third kernel folds them.
#include "common.cuh"
#include "tcgen05.cuh"

namespace singe {
namespace {

constexpr int kTileKeys = 64;
constexpr int kSlice = 64;                        // latent columns of one warp
constexpr int kSliceBytes = kTileKeys * kSlice * 2;
constexpr int kScoreStride = kTileKeys + 8;       // floats; spreads the fragment stores over the banks
constexpr int kWeightStride = kTileKeys + 8;      // bf16
constexpr int kLatentStages = 2;
constexpr int kMaxLatent = 512;

struct LatentDecode {
    __nv_bfloat16 *out;
    float *attn;  // [queries, splits, heads, latent]
    float *lse;   // [queries, splits, heads]
    const __nv_bfloat16 *query;
    const __nv_bfloat16 *cache;
    const int32_t *sequence_of, *lens, *table;
    int heads, latent, page_size, pages, sequences, table_stride, window, splits;
    float scale_log2;
    uint32_t *status;
    uint32_t *error;
};

__device__ __forceinline__ void copy_async_16(uint32_t target, const void *source, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(target), "l"(source), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Byte offset of 16-byte piece `piece` of key row `key` in a slice: pieces are permuted within a row so that eight rows
// read at one piece position touch all banks.
__device__ __forceinline__ uint32_t slice_at(int key, int piece) {
    return static_cast<uint32_t>(key * 128 + ((piece ^ (key & 7)) << 4));
}

int latent_shared_bytes(int warps, int head_tiles) {
    return kLatentStages * warps * kSliceBytes + warps * head_tiles * 16 * kScoreStride * 4 +
           head_tiles * 16 * kWeightStride * 2 + 3 * head_tiles * 16 * 4;
}

// ---- any page size ----
// One CTA per (query, split of its keys, 32 heads), one warp per 64 columns of the latent:
//   load      a warp copies its own 64-column slice of the tile (cp.async, two tiles in flight) and is the only reader of it
//   scores    its share of q . c over its 64 columns (q stays in registers), f32 partials to shared memory
//   softmax   partials of all warps summed, f32 online softmax, weights to shared memory as bf16
//   values    weights x its slice into f32 accumulators [heads, 64]
template <int MT>  // 16-head tiles of a CTA
__global__ void __launch_bounds__(256, 1) latent_decode_kernel(const LatentDecode p) {
    constexpr int kHeads = MT * 16;
    grid_launch_dependents();
    grid_dependency_wait();
    extern __shared__ __align__(128) uint8_t shared[];
    const int warps = blockDim.x >> 5;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, q2 = (lane & 3) * 2;  // fragment row and column pair
    uint8_t *tiles = shared;
    float *scores = reinterpret_cast<float *>(shared + kLatentStages * warps * kSliceBytes);  // [warps][kHeads][stride]
    __nv_bfloat16 *weights = reinterpret_cast<__nv_bfloat16 *>(scores + warps * kHeads * kScoreStride);
    float *row_max = reinterpret_cast<float *>(weights + kHeads * kWeightStride);
    float *row_sum = row_max + kHeads;
    float *row_factor = row_sum + kHeads;

    const int query = blockIdx.x, split = blockIdx.y, head0 = blockIdx.z * kHeads;
    const int sequence = p.sequence_of[query];
    const bool known = sequence >= 0 && sequence < p.sequences;
    if (!known && threadIdx.x == 0) report_status(p.status, kStatusIndexOutOfBounds);
    const int end_all = known ? min(p.lens[query], p.table_stride * p.page_size) : 0;
    const int start_all = p.window > 0 ? max(end_all - p.window, 0) : 0;
    const int per_split = ((max(end_all - start_all, 0) + p.splits - 1) / p.splits + kTileKeys - 1) / kTileKeys * kTileKeys;
    const int start = start_all + split * per_split;
    const int end = min(start + per_split, end_all);
    const int tile_count = end > start ? (end - start + kTileKeys - 1) / kTileKeys : 0;
    const int column0 = warp * kSlice;

    if (tile_count == 0) {
        for (int r = threadIdx.x; r < kHeads; r += blockDim.x) {
            if (p.splits > 1 && head0 + r < p.heads) {
                p.lse[(static_cast<size_t>(query) * p.splits + split) * p.heads + head0 + r] = -INFINITY;
            }
        }
        if (p.splits == 1) {
            for (int i = threadIdx.x; i < kHeads * p.latent; i += blockDim.x) {
                const int head = head0 + i / p.latent;
                if (head < p.heads) {
                    p.out[(static_cast<size_t>(query) * p.heads + head) * p.latent + i % p.latent] = __float2bfloat16_rn(0.0f);
                }
            }
        }
        return;
    }

    const int32_t *table = p.table + static_cast<size_t>(sequence) * p.table_stride;
    const uint32_t slice = smem_u32(tiles) + warp * kSliceBytes;
    const int stage_bytes = warps * kSliceBytes;
    auto load_tile = [&](int tile) {
        // lanes look up the cache rows of two keys each, then all copy four keys at a time, eight 16-byte pieces each
        int row[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int key = start + tile * kTileKeys + lane + 32 * i;
            row[i] = -1;
            if (key < end) {
                const int page = table[key / p.page_size];
                if (page >= 0 && page < p.pages) {
                    row[i] = page * p.page_size + key % p.page_size;
                } else {
                    report_status(p.status, kStatusIndexOutOfBounds);
                }
            }
        }
        const uint32_t target = slice + (tile % kLatentStages) * stage_bytes;
        const int piece = lane & 7;
#pragma unroll
        for (int i = 0; i < kTileKeys / 4; ++i) {
            const int key = (lane >> 3) + 4 * i;
            const int at = __shfl_sync(0xffffffffu, row[i / 8], key & 31);
            const __nv_bfloat16 *source = p.cache + static_cast<size_t>(max(at, 0)) * p.latent + column0 + piece * 8;
            copy_async_16(target + slice_at(key, piece), source, at >= 0);
        }
    };
    load_tile(0);
    copy_async_commit();
    if (tile_count > 1) load_tile(1);
    copy_async_commit();

    // q fragments of this warp's columns, for the whole kernel
    uint32_t qf[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int head = head0 + m * 16 + g + (i & 1) * 8;
                const int column = column0 + ks * 16 + q2 + (i >> 1) * 8;
                qf[m][ks][i] = head < p.heads ? *reinterpret_cast<const uint32_t *>(
                                                    p.query + (static_cast<size_t>(query) * p.heads + head) * p.latent + column)
                                              : 0u;
            }
        }
    }
    for (int r = threadIdx.x; r < kHeads; r += blockDim.x) {
        row_max[r] = -INFINITY;
        row_sum[r] = 0.0f;
    }
    float acc[MT][8][4] = {};
    __syncthreads();

    for (int tile = 0; tile < tile_count; ++tile) {
        copy_async_wait<kLatentStages - 1>();
        __syncwarp();
        const uint32_t here = slice + (tile % kLatentStages) * stage_bytes;
        {
            float s[MT][8][4] = {};
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
#pragma unroll
                for (int pair = 0; pair < 4; ++pair) {  // two 8-key tiles at a time
                    uint32_t b0, b1, b2, b3;
                    const int key = pair * 16 + (lane & 7) + ((lane >> 4) << 3);
                    ldmatrix_x4(here + slice_at(key, ks * 2 + ((lane >> 3) & 1)), b0, b1, b2, b3);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        mma_m16n8k16<__nv_bfloat16>(s[m][2 * pair], qf[m][ks][0], qf[m][ks][1], qf[m][ks][2], qf[m][ks][3], b0, b1);
                        mma_m16n8k16<__nv_bfloat16>(s[m][2 * pair + 1], qf[m][ks][0], qf[m][ks][1], qf[m][ks][2], qf[m][ks][3], b2, b3);
                    }
                }
            }
            float *mine = scores + warp * kHeads * kScoreStride;
#pragma unroll
            for (int m = 0; m < MT; ++m) {
#pragma unroll
                for (int n = 0; n < 8; ++n) {
                    *reinterpret_cast<float2 *>(mine + (m * 16 + g) * kScoreStride + n * 8 + q2) = make_float2(s[m][n][0], s[m][n][1]);
                    *reinterpret_cast<float2 *>(mine + (m * 16 + g + 8) * kScoreStride + n * 8 + q2) = make_float2(s[m][n][2], s[m][n][3]);
                }
            }
        }
        __syncthreads();
        const int visible = end - start - tile * kTileKeys;  // keys of this tile
        for (int r = warp; r < kHeads; r += warps) {
            float a = 0.0f, b = 0.0f;
            for (int w = 0; w < warps; ++w) {
                a += scores[(w * kHeads + r) * kScoreStride + lane];
                b += scores[(w * kHeads + r) * kScoreStride + lane + 32];
            }
            a = lane < visible ? a * p.scale_log2 : -INFINITY;
            b = lane + 32 < visible ? b * p.scale_log2 : -INFINITY;
            const float before = row_max[r];
            const float now = fmaxf(before, warp_max(fmaxf(a, b)));  // finite: the tile has at least one key
            a = exp2f(a - now);
            b = exp2f(b - now);
            const float sum = warp_sum(a + b);
            weights[r * kWeightStride + lane] = __float2bfloat16_rn(a);
            weights[r * kWeightStride + lane + 32] = __float2bfloat16_rn(b);
            __syncwarp();
            if (lane == 0) {
                const float factor = exp2f(before - now);
                row_factor[r] = factor;
                row_max[r] = now;
                row_sum[r] = row_sum[r] * factor + sum;
            }
        }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const float f0 = row_factor[m * 16 + g], f1 = row_factor[m * 16 + g + 8];
#pragma unroll
            for (int n = 0; n < 8; ++n) {
                acc[m][n][0] *= f0;
                acc[m][n][1] *= f0;
                acc[m][n][2] *= f1;
                acc[m][n][3] *= f1;
            }
        }
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            uint32_t a[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const __nv_bfloat16 *at = weights + (m * 16 + (lane & 15)) * kWeightStride + ks * 16 + (lane >> 4) * 8;
                ldmatrix_x4(smem_u32(at), a[m][0], a[m][1], a[m][2], a[m][3]);
            }
#pragma unroll
            for (int pair = 0; pair < 4; ++pair) {  // two 8-column tiles at a time
                uint32_t b0, b1, b2, b3;
                const int key = ks * 16 + (lane & 15);
                ldmatrix_x4_trans(here + slice_at(key, pair * 2 + (lane >> 4)), b0, b1, b2, b3);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    mma_m16n8k16<__nv_bfloat16>(acc[m][2 * pair], a[m][0], a[m][1], a[m][2], a[m][3], b0, b1);
                    mma_m16n8k16<__nv_bfloat16>(acc[m][2 * pair + 1], a[m][0], a[m][1], a[m][2], a[m][3], b2, b3);
                }
            }
        }
        __syncwarp();
        if (tile + kLatentStages < tile_count) load_tile(tile + kLatentStages);
        copy_async_commit();
    }
    copy_async_wait<0>();

#pragma unroll
    for (int m = 0; m < MT; ++m) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int r = m * 16 + g + half * 8;
            const int head = head0 + r;
            if (head >= p.heads) continue;
            const float inverse = 1.0f / row_sum[r];
#pragma unroll
            for (int n = 0; n < 8; ++n) {
                const int column = column0 + n * 8 + q2;
                const float x = acc[m][n][2 * half] * inverse, y = acc[m][n][2 * half + 1] * inverse;
                if (p.splits == 1) {
                    *reinterpret_cast<uint32_t *>(p.out + (static_cast<size_t>(query) * p.heads + head) * p.latent + column) =
                        pack2<__nv_bfloat16>(x, y);
                } else {
                    *reinterpret_cast<float2 *>(
                        p.attn + ((static_cast<size_t>(query) * p.splits + split) * p.heads + head) * p.latent + column) =
                        make_float2(x, y);
                }
            }
            if (p.splits > 1 && warp == 0 && q2 == 0) {
                p.lse[(static_cast<size_t>(query) * p.splits + split) * p.heads + head] = row_max[r] + log2f(row_sum[r]);
            }
        }
    }
}

// ---- tcgen05 ----
// One CTA per (query, split of its keys, 32 heads); heads past the last one are zero rows of q.
//   warp 0     TMA producer: q once, then tiles of 64 keys, SWIZZLE_128B, stored as [64-column chunk][64 keys][128 bytes].
//              Pages of 64 tokens arrive in one box a tile; smaller pages take one box per page and chunk, which the TMA
//              unit works off at about 12 bytes a clock, a quarter of the large boxes' rate.
//   warp 1     MMA issuer and owner of tensor memory:
//                S^T [keys, heads] = C q^T: A = the tile, K-major, M = 64: key k lands in tensor-memory lane
//                32 * (k / 16) + k % 16.
//                O^T [latent, heads] += C^T P^T: A = the same tile, MN-major, 128 latent columns a product; B = P from
//                shared memory.
//              Neighbouring products go to different accumulators: with 32 columns a product is all latency.
//              QK(t + 1) is issued before PV(t) when its tile is there, so that the tensor core works while the softmax of
//              tile t runs; a tile that is still on its way does not hold PV(t), whose end frees the stage after it.
//   warps 2-5  softmax and epilogue.  A thread of a warp's first half is a key: its lane holds the key's scores of all
//              heads.  Weights are taken relative to a base per head, on which the result does not depend; when a score
//              exceeds its head's base by more than 2^8, the tile's maxima (a butterfly across the lanes) give new bases,
//              and O and the sums are scaled.
// Tensor memory: S of even tiles [0, 64), of odd tiles [64, 128), two accumulators each, whose sum is the score; O^T from
// 128 on, 32 columns per 128 latent columns.
// Every wait is bounded.
constexpr int kTcHeads = 32;
constexpr int kTcThreads = 192;
constexpr int kTcMaxStages = 4;
constexpr int kChunkBytes = kTileKeys * 128;       // 64 keys x 64 columns
constexpr int kQueryChunkBytes = kTcHeads * 128;
constexpr int kWeightBytes = kTcHeads * 128;       // P: 32 heads x 64 keys
constexpr float kRebase = 8.0f;                    // log2 units

struct LatentTcShape {
    int chunks, stages;
    int page_rows, box_chunks;  // rows and 64-column chunks of a TMA box
};

__host__ __device__ inline int latent_tc_bytes(int chunks, int stages) {
    // tiles, then q (also what the over-reading product of an odd last chunk touches), P twice, exchange area, barriers
    const int query = chunks * kQueryChunkBytes > 2 * kChunkBytes ? chunks * kQueryChunkBytes : 2 * kChunkBytes;
    return stages * chunks * kChunkBytes + query + 2 * kWeightBytes + 5 * kTcHeads * 4 + 16 + 8 * (2 * kTcMaxStages + 8) + 1024;
}

// Lane h ends up with op over all lanes of x[h].
template <typename Op>
__device__ __forceinline__ float transpose_reduce(float (&x)[32], int lane, Op op) {
#pragma unroll
    for (int half = 16; half >= 1; half >>= 1) {
        const bool upper = (lane & half) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float sent = upper ? x[i] : x[i + half];
            const float kept = upper ? x[i + half] : x[i];
            x[i] = op(kept, __shfl_xor_sync(0xffffffffu, sent, half));
        }
    }
    return x[0];
}

__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

__global__ void __launch_bounds__(kTcThreads, 2)
    latent_decode_tcgen05_kernel(const __grid_constant__ CUtensorMap cache_map, const __grid_constant__ CUtensorMap query_map,
                                 const LatentDecode p, const LatentTcShape shape) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    const int chunks = shape.chunks, stages = shape.stages;
    const uint32_t stage_bytes = chunks * kChunkBytes;
    const uint32_t query_at = base + stages * stage_bytes;
    const uint32_t weights_at = query_at + max(chunks * kQueryChunkBytes, 2 * kChunkBytes);
    const uint32_t exchange_at = weights_at + 2 * kWeightBytes;
    float *exchange = reinterpret_cast<float *>(smem_raw + (exchange_at - raw));  // [5][32]: one row per softmax warp, then the bases
    const uint32_t bars = exchange_at + 5 * kTcHeads * 4 + 16;
    const uint32_t bar_full = bars, bar_empty = bars + 8 * kTcMaxStages;
    const uint32_t bar_query = bars + 16 * kTcMaxStages;
    const uint32_t bar_scores = bar_query + 8;    // [2]
    const uint32_t bar_weights = bar_query + 24;  // [2], one arrival per softmax warp
    const uint32_t bar_values = bar_query + 40;   // PV of a tile has retired
    const uint32_t holder = bar_query + 48;
    volatile uint32_t *holder_ptr = reinterpret_cast<volatile uint32_t *>(smem_raw + (holder - raw));

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int i = 0; i < stages; ++i) {
            mbar_init(bar_full + 8 * i, 1);
            mbar_init(bar_empty + 8 * i, 1);
        }
        mbar_init(bar_query, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(bar_scores + 8 * i, 1);
            mbar_init(bar_weights + 8 * i, 4);
        }
        mbar_init(bar_values, 1);
        mbar_init_fence();
    }
    if (warp == 1) {
        tmem_alloc(holder, 256);
        tmem_relinquish();
    }
    tcgen05_fence_before();
    __syncthreads();
    tcgen05_fence_after();
    const uint32_t tmem = *holder_ptr;
    grid_dependency_wait();  // the set-up above ran beside the kernels before

    const int query = blockIdx.x, split = blockIdx.y, head0 = blockIdx.z * kTcHeads;
    const int sequence = p.sequence_of[query];
    const bool known = sequence >= 0 && sequence < p.sequences;
    if (!known && threadIdx.x == 0) report_status(p.status, kStatusIndexOutOfBounds);
    const int end_all = known ? min(p.lens[query], p.table_stride * p.page_size) : 0;
    const int visible_from = p.window > 0 ? max(end_all - p.window, 0) : 0;
    // tiles start on box boundaries; keys before the window are masked
    const int start_all = visible_from / shape.page_rows * shape.page_rows;
    const int per_split = ((max(end_all - start_all, 0) + p.splits - 1) / p.splits + kTileKeys - 1) / kTileKeys * kTileKeys;
    const int start = start_all + split * per_split;
    const int end = min(start + per_split, end_all);
    const int tile_count = end > start ? (end - start + kTileKeys - 1) / kTileKeys : 0;

    if (tile_count == 0) {
        if (p.splits > 1) {
            for (int r = threadIdx.x; r < kTcHeads; r += blockDim.x) {
                if (head0 + r < p.heads) p.lse[(static_cast<size_t>(query) * p.splits + split) * p.heads + head0 + r] = -INFINITY;
            }
        } else {
            for (int i = threadIdx.x; i < kTcHeads * p.latent; i += blockDim.x) {
                const int head = head0 + i / p.latent;
                if (head < p.heads) {
                    p.out[(static_cast<size_t>(query) * p.heads + head) * p.latent + i % p.latent] = __float2bfloat16_rn(0.0f);
                }
            }
        }
    }

    bool failed = false;

    if (tile_count == 0) {
        // nothing to attend to
    } else if (warp == 0) {
        // ---------------- TMA producer ----------------
        if (lane == 0) {
            prefetch_tensor_map(&cache_map);
            prefetch_tensor_map(&query_map);
            mbar_expect_tx(bar_query, chunks * kQueryChunkBytes);
            for (int c = 0; c < chunks; ++c) tma_load_3d(query_at + c * kQueryChunkBytes, &query_map, bar_query, c * 64, head0, query);
        }
        const int32_t *table = p.table + static_cast<size_t>(sequence) * p.table_stride;
        const int boxes = kTileKeys / shape.page_rows;  // boxes of one chunk: 1, 2, 4 or 8
        const int box_bits = 31 - __clz(boxes);
        const int columns = chunks / shape.box_chunks;  // boxes side by side
        for (int tile = 0; tile < tile_count; ++tile) {
            const int stage = tile % stages;
            // lane b looks up box b's first cache row; boxes past the end repeat the tile's first box (masked)
            int row = 0;
            if (lane < boxes) {
                int key = start + tile * kTileKeys + lane * shape.page_rows;
                if (key >= end) key = start + tile * kTileKeys;
                int page = table[key / p.page_size];
                if (page < 0 || page >= p.pages) {
                    report_status(p.status, kStatusIndexOutOfBounds);
                    page = 0;
                }
                row = page * p.page_size + key % p.page_size;
            }
            int ok = 1;
            if (lane == 0 && tile >= stages) ok = mbar_wait(bar_empty + 8 * stage, (tile / stages - 1) & 1) ? 1 : 0;
            if (__shfl_sync(0xffffffffu, ok, 0) == 0) {
                failed = true;
                break;
            }
            if (lane == 0) mbar_expect_tx(bar_full + 8 * stage, stage_bytes);
            __syncwarp();
            for (int i = lane; i - lane < boxes * columns; i += 32) {
                const int box = i & (boxes - 1), chunk = (i >> box_bits) * shape.box_chunks;
                const int from = __shfl_sync(0xffffffffu, row, box);
                if (i < boxes * columns) {
                    tma_load_3d(base + stage * stage_bytes + chunk * kChunkBytes + box * shape.page_rows * 128, &cache_map,
                                bar_full + 8 * stage, 0, from, chunk);
                }
            }
        }
    } else if (warp == 1) {
        // ---------------- MMA issuer ----------------
        constexpr uint32_t kIdescScores = make_instr_desc(kTileKeys, kTcHeads, true, 0, 0);
        constexpr uint32_t kIdescValues = make_instr_desc(128, kTcHeads, true, 1, 0);  // A = C^T, MN-major
        auto wait_all = [&](uint32_t bar, uint32_t parity) -> bool {
            return __all_sync(0xffffffffu, mbar_wait(bar, parity) ? 1 : 0) != 0;
        };
        // Descriptors advance by adding to their address field (16-byte units).
        auto issue_scores = [&](int tile) {
            if (elect_one()) {
                uint64_t a = make_smem_desc(base + (tile % stages) * stage_bytes, 16, 1024);
                uint64_t b = make_smem_desc(query_at, 16, 1024);
                const uint32_t target = tmem + (tile & 1) * 2 * kTcHeads;
                uint32_t accumulate = 0;
#pragma unroll 2
                for (int c = 0; c < chunks; ++c) {
                    umma_ss(target, a, b, kIdescScores, accumulate);
                    umma_ss(target + kTcHeads, a + 2, b + 2, kIdescScores, accumulate);
                    umma_ss(target, a + 4, b + 4, kIdescScores, 1u);
                    umma_ss(target + kTcHeads, a + 6, b + 6, kIdescScores, 1u);
                    accumulate = 1;
                    a += kChunkBytes >> 4;
                    b += kQueryChunkBytes >> 4;
                }
                tcgen05_commit(bar_scores + 8 * (tile & 1));
            }
            __syncwarp();
        };
        auto issue_values = [&](int tile) -> bool {
            if (!wait_all(bar_weights + 8 * (tile & 1), (tile >> 1) & 1)) return false;
            tcgen05_fence_after();
            if (elect_one()) {
                const uint64_t a = make_smem_desc(base + (tile % stages) * stage_bytes, kChunkBytes, 1024);
                const uint64_t b = make_smem_desc(weights_at + (tile & 1) * kWeightBytes, 16, 1024);
                uint32_t accumulate = tile > 0 ? 1u : 0u;
#pragma unroll
                for (int ks = 0; ks < kTileKeys / 16; ++ks) {
#pragma unroll 4
                    for (int m = 0; m < (chunks + 1) / 2; ++m) {
                        umma_ss(tmem + 4 * kTcHeads + m * kTcHeads, a + m * ((2 * kChunkBytes) >> 4) + 128 * ks, b + 2 * ks,
                                kIdescValues, accumulate);
                    }
                    accumulate = 1;
                }
                tcgen05_commit(bar_empty + 8 * (tile % stages));
                tcgen05_commit(bar_values);
            }
            __syncwarp();
            return true;
        };
        if (!wait_all(bar_query, 0)) failed = true;
        int scored = 0;  // tiles whose scores have been issued
        for (int tile = 0; tile < tile_count && !failed; ++tile) {
            // scores of this tile if they are still to come, and of the next one if its keys have arrived
            for (int ahead = tile; ahead < tile + 2 && ahead < tile_count && !failed; ++ahead) {
                if (ahead < scored) continue;
                const uint32_t bar = bar_full + 8 * (ahead % stages), parity = (ahead / stages) & 1;
                if (ahead > tile) {
                    if (__shfl_sync(0xffffffffu, mbar_test_wait(bar, parity) ? 1 : 0, 0) == 0) break;
                }
                if (!wait_all(bar, parity)) {
                    failed = true;
                    break;
                }
                tcgen05_fence_after();
                issue_scores(ahead);
                scored = ahead + 1;
            }
            if (!failed && !issue_values(tile)) failed = true;
        }
    } else {
        // ---------------- softmax, epilogue ----------------
        const int quarter = warp & 3;  // tensor-memory lanes 32 * quarter ..
        const uint32_t lanes = static_cast<uint32_t>(quarter * 32) << 16;
        const bool has_key = lane < 16;
        const int my_key = quarter * 16 + (lane & 15);
        float base_log2 = -INFINITY;       // of head `lane`; the same in all four warps
        float sum[kTcHeads];               // of this thread's key
#pragma unroll
        for (int h = 0; h < kTcHeads; ++h) sum[h] = 0.0f;
        float *bases = exchange + 4 * kTcHeads;                                  // the base in use per head
        volatile int *grown = reinterpret_cast<volatile int *>(bases + kTcHeads);  // [4]: a warp saw a score beyond its base
        auto maximum = [](float a, float b) { return fmaxf(a, b); };
        auto addition = [](float a, float b) { return a + b; };
        for (int tile = 0; tile < tile_count; ++tile) {
            uint32_t scores[32];
            const int key = start + tile * kTileKeys + my_key;
            const bool visible = has_key && key >= visible_from && key < end;
            if (!failed && !__all_sync(0xffffffffu, mbar_wait(bar_scores + 8 * (tile & 1), (tile >> 1) & 1) ? 1 : 0)) failed = true;
            tcgen05_fence_after();
            if (!failed) {
                uint32_t other[32];
                tmem_ld_x32(tmem + lanes + (tile & 1) * 2 * kTcHeads, scores);
                tmem_ld_x32(tmem + lanes + (tile & 1) * 2 * kTcHeads + kTcHeads, other);
                tmem_wait_ld_into(scores);
                tmem_wait_ld_into(other);
                float excess = tile == 0 ? INFINITY : -INFINITY;
#pragma unroll
                for (int h = 0; h < 32; h += 4) {
                    const float4 b = *reinterpret_cast<const float4 *>(bases + h);
                    const float subtracted[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float both = __uint_as_float(scores[h + i]) + __uint_as_float(other[h + i]);
                        const float x = visible ? both * p.scale_log2 : -INFINITY;
                        scores[h + i] = __float_as_uint(x);
                        if (tile > 0) excess = fmaxf(excess, x - subtracted[i]);
                    }
                }
                const bool beyond = __any_sync(0xffffffffu, excess > kRebase);
                if (lane == 0) grown[quarter] = beyond ? 1 : 0;
            }
            softmax_barrier();
            if ((grown[0] | grown[1] | grown[2] | grown[3]) != 0) {  // the same answer in all four warps
                float top[32];
#pragma unroll
                for (int h = 0; h < 32; ++h) top[h] = __uint_as_float(scores[h]);
                exchange[quarter * kTcHeads + lane] = transpose_reduce(top, lane, maximum);
                softmax_barrier();
                const float tile_top = fmaxf(fmaxf(exchange[lane], exchange[kTcHeads + lane]),
                                             fmaxf(exchange[2 * kTcHeads + lane], exchange[3 * kTcHeads + lane]));
                const float next = fmaxf(base_log2, tile_top);
                const float factor = base_log2 == -INFINITY ? 0.0f : exp2f(base_log2 - next);
                if (tile > 0) {
                    // O holds P V up to the tile before
                    if (!failed && !__all_sync(0xffffffffu, mbar_wait(bar_values, (tile - 1) & 1) ? 1 : 0)) failed = true;
                    tcgen05_fence_after();
                    for (int m = 0; m < (chunks + 1) / 2 && !failed; ++m) {
                        uint32_t o[32];
                        tmem_ld_x32(tmem + lanes + 4 * kTcHeads + m * kTcHeads, o);
                        tmem_wait_ld_into(o);
#pragma unroll
                        for (int h = 0; h < 32; ++h) {
                            o[h] = __float_as_uint(__uint_as_float(o[h]) * __shfl_sync(0xffffffffu, factor, h));
                        }
                        tmem_st_x32(tmem + lanes + 4 * kTcHeads + m * kTcHeads, o);
                    }
                    tmem_wait_st();
                }
                base_log2 = next;
#pragma unroll
                for (int h = 0; h < 32; ++h) sum[h] *= __shfl_sync(0xffffffffu, factor, h);
                if (quarter == 0) bases[lane] = next == -INFINITY ? 0.0f : next;
                softmax_barrier();
            }
            if (has_key && !failed) {
                // P[head, key], 128-byte rows with the 16-byte pieces permuted as SWIZZLE_128B has them
                uint8_t *weights = smem_raw + (weights_at - raw) + (tile & 1) * kWeightBytes;
                const int piece = my_key >> 3, within = (my_key & 7) * 2;
#pragma unroll
                for (int h0 = 0; h0 < 32; h0 += 8) {  // eight heads at a time, so that their latencies overlap
                    const float4 low = *reinterpret_cast<const float4 *>(bases + h0);
                    const float4 high = *reinterpret_cast<const float4 *>(bases + h0 + 4);
                    const float subtracted[8] = {low.x, low.y, low.z, low.w, high.x, high.y, high.z, high.w};
                    float x[8];
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        x[i] = exp2_fast(__uint_as_float(scores[h0 + i]) - subtracted[i]);  // a hidden key's score is -inf
                        sum[h0 + i] += x[i];
                    }
#pragma unroll
                    for (int i = 0; i < 8; ++i) {
                        *reinterpret_cast<__nv_bfloat16 *>(weights + (h0 + i) * 128 + ((piece ^ i) << 4) + within) =
                            __float2bfloat16_rn(x[i]);
                    }
                }
                fence_proxy_async_shared();
            }
            tcgen05_fence_before();
            softmax_barrier();  // also: everyone has read the exchange area
            if (lane == 0) mbar_arrive(bar_weights + 8 * (tile & 1));
        }
        grid_launch_dependents();  // late: the fold's many small CTAs would take the slots of CTAs still to come
        // ---- O^T / sum ----
        // A parity wait tells neighbouring phases apart, not more: the last scores imply the values up to the third-last
        // tile, so the second-last tile is waited for before the last.
        for (int tile = max(tile_count - 2, 0); tile < tile_count && !failed; ++tile) {
            if (!__all_sync(0xffffffffu, mbar_wait(bar_values, tile & 1) ? 1 : 0)) failed = true;
        }
        tcgen05_fence_after();
        exchange[quarter * kTcHeads + lane] = transpose_reduce(sum, lane, addition);
        softmax_barrier();
        const float total = (exchange[lane] + exchange[kTcHeads + lane]) + (exchange[2 * kTcHeads + lane] + exchange[3 * kTcHeads + lane]);
        const float inverse = total > 0.0f ? 1.0f / total : 0.0f;
        if (p.splits > 1 && quarter == 0 && head0 + lane < p.heads) {
            p.lse[(static_cast<size_t>(query) * p.splits + split) * p.heads + head0 + lane] =
                total > 0.0f ? base_log2 + log2f(total) : -INFINITY;
        }
        for (int m = 0; m < (chunks + 1) / 2 && !failed; ++m) {
            uint32_t o[32];
            tmem_ld_x32(tmem + lanes + 4 * kTcHeads + m * kTcHeads, o);
            tmem_wait_ld_into(o);
            const int column = m * 128 + quarter * 32 + lane;
            if (p.splits == 1) {
                __nv_bfloat16 *out = p.out + (static_cast<size_t>(query) * p.heads + head0) * p.latent + column;
#pragma unroll
                for (int h = 0; h < 32; ++h) {
                    const float x = __uint_as_float(o[h]) * __shfl_sync(0xffffffffu, inverse, h);
                    if (head0 + h < p.heads && column < p.latent) out[h * p.latent] = __float2bfloat16_rn(x);
                }
            } else {
                float *out = p.attn + ((static_cast<size_t>(query) * p.splits + split) * p.heads + head0) * p.latent + column;
#pragma unroll
                for (int h = 0; h < 32; ++h) {
                    const float x = __uint_as_float(o[h]) * __shfl_sync(0xffffffffu, inverse, h);
                    if (head0 + h < p.heads && column < p.latent) out[h * p.latent] = x;
                }
            }
        }
    }
    if (failed && lane == 0) report_status(p.error, kStatusWaitTimeout);
    if (failed) linger_after_timeout();
    tcgen05_fence_before();
    __syncthreads();
    if (warp == 1) {
        tcgen05_fence_after();
        tmem_dealloc(tmem, 256);
    }
}

// out[query, head] = sum over the splits of exp2(lse_s - max) * attn_s, normalised.
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentDecode p) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int query = blockIdx.x, head = blockIdx.y;
    const float *lse = p.lse + static_cast<size_t>(query) * p.splits * p.heads + head;
    float top = -INFINITY;
    for (int s = 0; s < p.splits; ++s) top = fmaxf(top, lse[s * p.heads]);
    float total = 0.0f;
    for (int s = 0; s < p.splits; ++s) total += top == -INFINITY ? 0.0f : exp2f(lse[s * p.heads] - top);
    const float inverse = total > 0.0f ? 1.0f / total : 0.0f;
    for (int c = threadIdx.x * 4; c < p.latent; c += blockDim.x * 4) {
        float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        for (int s = 0; s < p.splits; ++s) {
            const float value = lse[s * p.heads];
            if (value == -INFINITY) continue;  // a split without keys wrote nothing
            const float weight = exp2f(value - top) * inverse;
            const float4 x = *reinterpret_cast<const float4 *>(
                p.attn + ((static_cast<size_t>(query) * p.splits + s) * p.heads + head) * p.latent + c);
            sum.x = fmaf(weight, x.x, sum.x);
            sum.y = fmaf(weight, x.y, sum.y);
            sum.z = fmaf(weight, x.z, sum.z);
            sum.w = fmaf(weight, x.w, sum.w);
        }
        *reinterpret_cast<uint2 *>(p.out + (static_cast<size_t>(query) * p.heads + head) * p.latent + c) =
            make_uint2(pack2<__nv_bfloat16>(sum.x, sum.y), pack2<__nv_bfloat16>(sum.z, sum.w));
    }
}

// Rows of a TMA box for a page size, or 0 for sizes the tcgen05 kernel does not take.
int latent_box_rows(size_t page_size) {
    if (page_size == 8 || page_size == 16 || page_size == 32) return static_cast<int>(page_size);
    return page_size % 64 == 0 ? 64 : 0;
}

// Two CTAs share an SM where their tiles fit it twice.
int latent_tc_stages(int chunks) {
    int stages = kTcMaxStages;
    const int limit = latent_tc_bytes(chunks, 2) <= 113 * 1024 ? 113 * 1024 : 227 * 1024;
    while (stages > 2 && latent_tc_bytes(chunks, stages) > limit) --stages;
    return stages;
}

int launch_fold(cudaStream_t stream, const LatentDecode &p, size_t queries) {
    if (p.splits > 1) {
        const int threads = (p.latent / 4 + 31) / 32 * 32;
        SINGE_CUDA_TRY(launch_dependent(latent_combine_kernel, dim3(static_cast<unsigned>(queries), static_cast<unsigned>(p.heads)),
                                        dim3(threads), 0, stream, kLaunchCombine, 1, p));
    }
    return launch_status();
}

int launch_latent_tcgen05(cudaStream_t stream, const LatentDecode &p, size_t queries, int box_rows) {
    LatentTcShape shape;
    shape.chunks = p.latent / 64;
    shape.page_rows = box_rows;
    shape.box_chunks = box_rows == kTileKeys ? shape.chunks : 1;
    shape.stages = latent_tc_stages(shape.chunks);
    const int bytes = latent_tc_bytes(shape.chunks, shape.stages);
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(latent_decode_tcgen05_kernel, bytes, configured));
    CUtensorMap cache_map, query_map;
    {
        // the latent's 64-column chunks as the outer dimension, so that a box lands chunk by chunk
        const uint64_t dims[3] = {64, static_cast<uint64_t>(p.pages) * p.page_size, static_cast<uint64_t>(shape.chunks)};
        const uint64_t strides[2] = {static_cast<uint64_t>(p.latent) * 2, 128};
        const uint32_t box[3] = {64, static_cast<uint32_t>(box_rows), static_cast<uint32_t>(shape.box_chunks)};
        SINGE_TRY(encode_tensor_map(&cache_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, p.cache, dims, strides, box,
                                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B));
    }
    {
        const uint64_t dims[3] = {static_cast<uint64_t>(p.latent), static_cast<uint64_t>(p.heads), queries};
        const uint64_t strides[2] = {static_cast<uint64_t>(p.latent) * 2, static_cast<uint64_t>(p.latent) * p.heads * 2};
        const uint32_t box[3] = {64, kTcHeads, 1};
        SINGE_TRY(encode_tensor_map(&query_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, p.query, dims, strides, box,
                                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B));
    }
    const dim3 grid(static_cast<unsigned>(queries), static_cast<unsigned>(p.splits),
                    static_cast<unsigned>((p.heads + kTcHeads - 1) / kTcHeads));
    SINGE_CUDA_TRY(launch_dependent(latent_decode_tcgen05_kernel, grid, dim3(kTcThreads), bytes, stream, kLaunchDecode, 1,
                                    cache_map, query_map, p, shape));
    return launch_fold(stream, p, queries);
}

template <int MT>
int launch_latent_decode(cudaStream_t stream, const LatentDecode &p, size_t queries) {
    const int warps = p.latent / kSlice;
    const int bytes = latent_shared_bytes(warps, MT);
    static int configured[kMaxDevices] = {0};
    SINGE_CUDA_TRY(ensure_dynamic_shared(latent_decode_kernel<MT>, bytes, configured));
    const dim3 grid(static_cast<unsigned>(queries), static_cast<unsigned>(p.splits),
                    static_cast<unsigned>((p.heads + MT * 16 - 1) / (MT * 16)));
    SINGE_CUDA_TRY(launch_dependent(latent_decode_kernel<MT>, grid, dim3(warps * 32), bytes, stream, kLaunchDecode, 1, p));
    return launch_fold(stream, p, queries);
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

size_t singe_latent_decode_splits(size_t queries, size_t heads, size_t latent, size_t key_bound) {
    // CTAs run in waves; one costs a fixed ramp and a time per key (its share of what HBM gives an SM); each split adds to
    // the fold.
    const int chunks = static_cast<int>((latent + 63) / 64);
    const double per_sm = latent_tc_bytes(chunks, 2) <= 113 * 1024 ? 2.0 : 1.0;
    const double slots = device_sm_count() * per_sm;
    const double groups = static_cast<double>((heads + kTcHeads - 1) / kTcHeads);
    const double key_us = static_cast<double>(latent) * 2.0 * per_sm / 36e3;
    const size_t finest = key_bound / (2 * kTileKeys) > 0 ? key_bound / (2 * kTileKeys) : 1;
    size_t best = 1;
    double best_time = 1e30;
    for (size_t splits = 1; splits <= finest && splits <= 64; ++splits) {
        const double ctas = static_cast<double>(queries) * groups * static_cast<double>(splits);
        const double waves = static_cast<double>(static_cast<long long>((ctas + slots - 1) / slots));
        const double keys = static_cast<double>((key_bound + splits - 1) / splits);
        const double time = waves * (4.0 + key_us * keys) + (splits > 1 ? 2.0 + 0.3 * static_cast<double>(splits) : 0.0);
        if (time < best_time) {
            best_time = time;
            best = splits;
        }
    }
    return best;
}

int singe_latent_decode_bf16(singe_stream_t stream, void *out, float *attn_scratch, float *lse_scratch, const void *query,
                             const void *cache, const int32_t *sequence_of, const int32_t *lens,
                             const int32_t *block_table, size_t queries, size_t heads, size_t latent, size_t page_size,
                             size_t pages, size_t sequences, size_t table_stride, size_t window, size_t splits,
                             float scale, uint32_t *status) {
    if (queries == 0 || heads == 0 || latent == 0 || page_size == 0 || pages == 0 || sequences == 0 || table_stride == 0 ||
        splits == 0 || !(scale == scale)) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(queries) || !fits_i32(heads) || !fits_i32(pages * page_size) || !fits_i32(table_stride * page_size) ||
        !fits_i32(window)) {
        return SINGE_ERR_LENGTH_EXCEEDS_I32;
    }
    if (out == nullptr || query == nullptr || cache == nullptr || sequence_of == nullptr || lens == nullptr ||
        block_table == nullptr || (splits > 1 && (attn_scratch == nullptr || lse_scratch == nullptr))) {
        return SINGE_ERR_NULL_POINTER;
    }
    if (latent % kSlice != 0 || latent > kMaxLatent || splits > 65535 || heads > 65535 ||
        ((reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(query) | reinterpret_cast<uintptr_t>(out) |
          reinterpret_cast<uintptr_t>(attn_scratch)) & 15u) != 0) {
        return SINGE_ERR_UNSUPPORTED_CONFIGURATION;
    }
    LatentDecode p;
    p.out = static_cast<__nv_bfloat16 *>(out);
    p.attn = attn_scratch;
    p.lse = lse_scratch;
    p.query = static_cast<const __nv_bfloat16 *>(query);
    p.cache = static_cast<const __nv_bfloat16 *>(cache);
    p.sequence_of = sequence_of;
    p.lens = lens;
    p.table = block_table;
    p.heads = static_cast<int>(heads);
    p.latent = static_cast<int>(latent);
    p.page_size = static_cast<int>(page_size);
    p.pages = static_cast<int>(pages);
    p.sequences = static_cast<int>(sequences);
    p.table_stride = static_cast<int>(table_stride);
    p.window = static_cast<int>(window);
    p.splits = static_cast<int>(splits);
    p.scale_log2 = scale * 1.4426950408889634f;
    p.status = status;
    p.error = device_error_word();
    const int box_rows = latent_box_rows(page_size);
    if (box_rows > 0) return launch_latent_tcgen05(static_cast<cudaStream_t>(stream), p, queries, box_rows);
    return heads <= 16 ? launch_latent_decode<1>(static_cast<cudaStream_t>(stream), p, queries)
                       : launch_latent_decode<2>(static_cast<cudaStream_t>(stream), p, queries);
}

}  // extern "C"
