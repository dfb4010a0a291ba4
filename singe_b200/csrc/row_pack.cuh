// Rows handled by one CTA each and kept in registers between passes: packs of VEC adjacent values, the sum over a CTA, and
// the thread count for a row.
#pragma once

#include "common.cuh"

namespace singe {

inline bool aligned_to(const void *pointer, size_t bytes) { return (reinterpret_cast<uintptr_t>(pointer) & (bytes - 1)) == 0; }

// Sum over the CTA, the same value in every thread.  `scratch` holds 32 floats; usable back to back.
__device__ __forceinline__ float cta_sum(float value, float *scratch) {
    value = warp_sum(value);
    const int warps = (blockDim.x + 31) >> 5;
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = value;
    __syncthreads();
    float total = 0.0f;
    for (int i = 0; i < warps; ++i) total += scratch[i];
    __syncthreads();
    return total;
}

template <int VEC>
struct Pack {
    float v[VEC];
};

template <int VEC>
__device__ __forceinline__ Pack<VEC> load_pack(const float *p) {
    Pack<VEC> out;
    if constexpr (VEC == 4) {
        const float4 raw = *reinterpret_cast<const float4 *>(p);
        out.v[0] = raw.x;
        out.v[1] = raw.y;
        out.v[2] = raw.z;
        out.v[3] = raw.w;
    } else {
        out.v[0] = *p;
    }
    return out;
}

template <int VEC>
__device__ __forceinline__ Pack<VEC> load_pack(const __nv_bfloat16 *p) {
    Pack<VEC> out;
    if constexpr (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2 *>(p);
        out.v[0] = __uint_as_float(raw.x << 16);
        out.v[1] = __uint_as_float(raw.x & 0xffff0000u);
        out.v[2] = __uint_as_float(raw.y << 16);
        out.v[3] = __uint_as_float(raw.y & 0xffff0000u);
    } else {
        out.v[0] = __bfloat162float(*p);
    }
    return out;
}

template <int VEC>
__device__ __forceinline__ void store_pack(float *p, const Pack<VEC> &x) {
    if constexpr (VEC == 4) {
        *reinterpret_cast<float4 *>(p) = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    } else {
        *p = x.v[0];
    }
}

template <int VEC>
__device__ __forceinline__ void store_pack(__nv_bfloat16 *p, const Pack<VEC> &x) {
    if constexpr (VEC == 4) {
        *reinterpret_cast<uint2 *>(p) = make_uint2(pack2<__nv_bfloat16>(x.v[0], x.v[1]), pack2<__nv_bfloat16>(x.v[2], x.v[3]));
    } else {
        *p = __float2bfloat16_rn(x.v[0]);
    }
}

constexpr int kHeldPacks = 8;      // packs a thread keeps of its row
constexpr int kNormThreads = 512;  // at most: rows up to 512 * 8 * VEC wide

inline unsigned norm_threads(size_t width, int vec) {
    // four packs a thread: fewer warps to bring together than with one, and loads enough in flight
    const size_t packs = (width + vec - 1) / vec;
    size_t threads = ((packs + 3) / 4 + 31) / 32 * 32;
    if (threads > kNormThreads) threads = kNormThreads;
    return static_cast<unsigned>(threads);
}

inline bool row_fits(size_t width, int vec) { return width <= static_cast<size_t>(kNormThreads) * kHeldPacks * vec; }

}  // namespace singe
