// Linear layers in true 32-bit: out[M, N] = x[M, K] . weight[N, K]^T with f32 operands, f32 products and f32 sums (no
// TF32).  It serves decoders run entirely in f32, where exactness is the point; the tensor-core GEMM serves bf16.
//
// 64 x 64 tiles of 256 threads, 4 x 4 outputs each, K in slices of 16 through shared memory.  blockIdx.z is the problem
// of a batched call (one product per attention head).  Every extent may be ragged.
#include "common.cuh"

namespace singe {
namespace {

constexpr int kTileF32 = 64;
constexpr int kSliceF32 = 16;

struct LinearF32 {
    float *out;
    const float *x;
    const float *weight;
    const float *gate;  // nullptr, or row m of problem b is multiplied by sigmoid(gate[m * gate_stride + b])
    int m, n, k;
    long long ldx, ldw, ldo, gate_stride;
    long long x_batch, w_batch, out_batch;  // element offsets between problems
    int squared_relu;
};

__global__ void __launch_bounds__(256) linear_f32_kernel(const LinearF32 p) {
    grid_launch_dependents();
    grid_dependency_wait();
    __shared__ float xs[kSliceF32][kTileF32 + 4];
    __shared__ float ws[kSliceF32][kTileF32 + 4];
    const int problem = blockIdx.z;
    const float *x = p.x + problem * p.x_batch;
    const float *w = p.weight + problem * p.w_batch;
    const int m0 = blockIdx.y * kTileF32;
    const int n0 = blockIdx.x * kTileF32;
    const int tm = threadIdx.x / 16, tn = threadIdx.x % 16;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.k; k0 += kSliceF32) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int index = threadIdx.x + i * 256;
            const int row = index / kSliceF32, column = index % kSliceF32;
            const bool in_k = k0 + column < p.k;
            xs[column][row] = in_k && m0 + row < p.m ? x[(m0 + row) * p.ldx + k0 + column] : 0.0f;
            ws[column][row] = in_k && n0 + row < p.n ? w[(n0 + row) * p.ldw + k0 + column] : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kSliceF32; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = xs[k][tm + 16 * i];
                b[i] = ws[k][tn + 16 * i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int row = m0 + tm + 16 * i;
        if (row >= p.m) continue;
        float factor = 1.0f;
        if (p.gate != nullptr) factor = 1.0f / (1.0f + expf(-p.gate[row * p.gate_stride + problem]));
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int column = n0 + tn + 16 * j;
            if (column >= p.n) continue;
            float value = acc[i][j] * factor;
            if (p.squared_relu) {
                value = fmaxf(value, 0.0f);
                value *= value;
            }
            p.out[row * p.ldo + problem * p.out_batch + column] = value;
        }
    }
}

int launch_linear_f32(singe_stream_t stream, const LinearF32 &p, size_t batch) {
    const size_t blocks_m = (static_cast<size_t>(p.m) + kTileF32 - 1) / kTileF32;
    if (blocks_m > 65535 || batch > 65535) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    const dim3 grid(static_cast<unsigned>((p.n + kTileF32 - 1) / kTileF32), static_cast<unsigned>(blocks_m),
                    static_cast<unsigned>(batch));
    SINGE_CUDA_TRY(launch_dependent(linear_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), kLaunchGlue, 1, p));
    return launch_status();
}

__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }

// out = silu(gate) * up, elementwise.
__global__ void __launch_bounds__(256) silu_mul_f32_kernel(float *out, long long out_stride, const float *gate, const float *up,
                                                           long long in_stride, int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    const long long row = blockIdx.x;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        out[row * out_stride + c] = silu_exact(gate[row * in_stride + c]) * up[row * in_stride + c];
    }
}

}  // namespace
}  // namespace singe

using namespace singe;

extern "C" {

int singe_linear_f32(singe_stream_t stream, float *out, const float *x, const float *weight, size_t rows, size_t columns,
                     size_t reduction, size_t x_row_stride, size_t weight_row_stride, size_t output_row_stride,
                     int activation) {
    if (rows == 0 || columns == 0 || reduction == 0 || x_row_stride < reduction || weight_row_stride < reduction ||
        output_row_stride < columns) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (activation != 0 && activation != 2) return SINGE_ERR_INVALID_ARGUMENT;
    if (!fits_i32(rows) || !fits_i32(columns) || !fits_i32(reduction)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (out == nullptr || x == nullptr || weight == nullptr) return SINGE_ERR_NULL_POINTER;
    LinearF32 p = {};
    p.out = out;
    p.x = x;
    p.weight = weight;
    p.m = static_cast<int>(rows);
    p.n = static_cast<int>(columns);
    p.k = static_cast<int>(reduction);
    p.ldx = static_cast<long long>(x_row_stride);
    p.ldw = static_cast<long long>(weight_row_stride);
    p.ldo = static_cast<long long>(output_row_stride);
    p.squared_relu = activation == 2 ? 1 : 0;
    return launch_linear_f32(stream, p, 1);
}

int singe_silu_mul_f32(singe_stream_t stream, float *out, size_t output_row_stride, const float *gate, const float *up,
                       size_t input_row_stride, size_t rows, size_t width) {
    if (rows == 0 || width == 0 || input_row_stride < width || output_row_stride < width) return SINGE_ERR_INVALID_LENGTH;
    if (!fits_i32(rows) || !fits_i32(width)) return SINGE_ERR_LENGTH_EXCEEDS_I32;
    if (out == nullptr || gate == nullptr || up == nullptr) return SINGE_ERR_NULL_POINTER;
    SINGE_CUDA_TRY(launch_dependent(silu_mul_f32_kernel, dim3(static_cast<unsigned>(rows)), dim3(256), 0,
                                    static_cast<cudaStream_t>(stream), kLaunchGlue, 1, out,
                                    static_cast<long long>(output_row_stride), gate, up, static_cast<long long>(input_row_stride),
                                    static_cast<int>(width)));
    return launch_status();
}

int singe_head_linear_f32(singe_stream_t stream, float *out, const float *x, const float *weight, size_t rows,
                          size_t heads, size_t columns, size_t reduction, size_t x_row_stride, size_t x_head_stride,
                          size_t weight_row_stride, size_t weight_head_rows, size_t out_row_stride,
                          size_t out_head_stride, const float *gate, size_t gate_row_stride) {
    if (rows == 0 || heads == 0 || columns == 0 || reduction == 0 || weight_row_stride < reduction ||
        weight_head_rows < columns || x_head_stride < reduction || out_head_stride < columns ||
        x_row_stride < (heads - 1) * x_head_stride + reduction ||
        out_row_stride < (heads - 1) * out_head_stride + columns || (gate != nullptr && gate_row_stride < heads)) {
        return SINGE_ERR_INVALID_LENGTH;
    }
    if (!fits_i32(rows) || !fits_i32(heads) || !fits_i32(columns) || !fits_i32(reduction)) {
        return SINGE_ERR_LENGTH_EXCEEDS_I32;
    }
    if (out == nullptr || x == nullptr || weight == nullptr) return SINGE_ERR_NULL_POINTER;
    LinearF32 p = {};
    p.out = out;
    p.x = x;
    p.weight = weight;
    p.gate = gate;
    p.m = static_cast<int>(rows);
    p.n = static_cast<int>(columns);
    p.k = static_cast<int>(reduction);
    p.ldx = static_cast<long long>(x_row_stride);
    p.ldw = static_cast<long long>(weight_row_stride);
    p.ldo = static_cast<long long>(out_row_stride);
    p.gate_stride = static_cast<long long>(gate_row_stride);
    p.x_batch = static_cast<long long>(x_head_stride);
    p.w_batch = static_cast<long long>(weight_head_rows * weight_row_stride);
    p.out_batch = static_cast<long long>(out_head_stride);
    return launch_linear_f32(stream, p, heads);
}

}  // extern "C"
