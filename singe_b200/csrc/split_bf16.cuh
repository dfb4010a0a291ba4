// What the block forms of the recurrences share: f32 operands as two bf16 terms for the tensor core, bulk copies of prepared
// operands, and the shared-memory layout of a block's values.
#pragma once

#include "common.cuh"

namespace singe {

constexpr int kBlock = 16;                // tokens of a block
constexpr int kValueBox = kBlock * 128;   // bytes of a TMA box of 16 tokens x 64 columns, SWIZZLE_128B

inline size_t align256(size_t bytes) { return (bytes + 255) / 256 * 256; }

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

// Bulk copy global -> shared, completing `bytes` on the mbarrier (16-byte aligned addresses and size).
__device__ __forceinline__ void bulk_load(uint32_t target, const void *source, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(target),
                 "l"(source), "r"(bytes), "r"(bar)
                 : "memory");
}

// Bulk copy shared -> global as part of the thread's current bulk group (16-byte aligned addresses and size).
__device__ __forceinline__ void bulk_store(void *target, uint32_t source, uint32_t bytes) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(target), "r"(source), "r"(bytes) : "memory");
}

// ldmatrix_x4_trans's inverse: four 8x8 matrices out of MMA fragments, transposed.
__device__ __forceinline__ void stmatrix_x4_trans(uint32_t address, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
    asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(address), "r"(r0), "r"(r1),
                 "r"(r2), "r"(r3)
                 : "memory");
}

// Byte offset of columns v .. v + 7 (v a multiple of eight) of token t in the boxes of v or g.
__device__ __forceinline__ uint32_t value_at(int t, int v) {
    return static_cast<uint32_t>((v >> 6) * kValueBox + t * 128 + ((((v >> 3) & 7) ^ (t & 7)) << 4));
}

}  // namespace singe
