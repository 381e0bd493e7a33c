// Small kernels around composite mixers and repeated walks over a run of layers.
//
//   scaled_sum       out[i] = a * x[i] + b * y[i] (float32 arithmetic, one rounding on store): two mixers side by side whose
//                    outputs join with a weight each.  x and y are of one dtype, out of its own.
//   normed_sum       out[n] = a * x[n] / rms(x[n]) * wx + b * y[n] / rms(y[n]) * wy, rms over the row with eps inside the root, wx and
//                    wy float32 [width]: the same where each output is normed before they join.  x and y are float32 rows.
//   concat_streams   out[n] = [ residual[n] (+ delta[n]) | origin[n] ] in the activation dtype: the operand of the product that
//                    opens a walk, x <- W [x ; x0].  residual and origin are float32 [N, width]; delta (optional) is what the
//                    layer before left pending.
#include "common.cuh"

namespace {

using namespace pb;

template <typename TIn, typename T>
__global__ void scaled_sum_kernel(const TIn* __restrict__ x, const TIn* __restrict__ y, T* __restrict__ out, float a, float b, size_t total) {
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
        out[i] = from_float<T>(fmaf(a, to_float(x[i]), b * to_float(y[i])));
}

template <typename T>
__global__ void concat_streams_kernel(const float* __restrict__ residual, const T* __restrict__ delta, const float* __restrict__ origin,
                                      T* __restrict__ out, int width, size_t total) {
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t row = i / width, col = i % width;
        const float x = residual[i] + (delta != nullptr ? to_float(delta[i]) : 0.0f);
        out[row * 2 * width + col] = from_float<T>(x);
        out[row * 2 * width + width + col] = from_float<T>(origin[i]);
    }
}

// One block per row, ITEMS quads of neighbouring elements of each row a thread; one pair of barriers for both sums of squares.
template <typename T, int ITEMS>
__global__ void __launch_bounds__(512) normed_sum_quads_kernel(const float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ wx,
                                        const float* __restrict__ wy, T* __restrict__ out, float a, float b, int width, float eps) {
    pdl_wait();
    __shared__ float sums[2][16];
    const size_t at = (size_t)blockIdx.x * width;
    float xv[ITEMS][4], yv[ITEMS][4];
    float sx = 0.0f, sy = 0.0f;
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i < width) {
            load_quad(x + at + i, xv[k]);
            load_quad(y + at + i, yv[k]);
#pragma unroll
            for (int e = 0; e < 4; ++e) { sx = fmaf(xv[k][e], xv[k][e], sx); sy = fmaf(yv[k][e], yv[k][e], sy); }
        }
    }
    sx = warp_sum(sx);
    sy = warp_sum(sy);
    if ((threadIdx.x & 31) == 0) { sums[0][threadIdx.x >> 5] = sx; sums[1][threadIdx.x >> 5] = sy; }
    __syncthreads();
    sx = sy = 0.0f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) { sx += sums[0][w]; sy += sums[1][w]; }
    const float fx = a * rsqrtf(sx / (float)width + eps), fy = b * rsqrtf(sy / (float)width + eps);
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i < width) {
            float u[4], v[4];
            load_quad(wx + i, u);
            load_quad(wy + i, v);
#pragma unroll
            for (int e = 0; e < 4; ++e) u[e] = fmaf(fx * xv[k][e], u[e], fy * yv[k][e] * v[e]);
            store_quad(out + at + i, u);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) normed_sum_kernel(const float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ wx,
                                  const float* __restrict__ wy, T* __restrict__ out, float a, float b, int width, float eps) {
    pdl_wait();
    __shared__ float scratch[32];
    const size_t at = (size_t)blockIdx.x * width;
    float sx = 0.0f, sy = 0.0f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) { sx = fmaf(x[at + i], x[at + i], sx); sy = fmaf(y[at + i], y[at + i], sy); }
    const float fx = a * rsqrtf(block_sum(sx, scratch) / (float)width + eps), fy = b * rsqrtf(block_sum(sy, scratch) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) out[at + i] = from_float<T>(fmaf(fx * x[at + i], wx[i], fy * y[at + i] * wy[i]));
}

unsigned blocks_for(size_t total) {
    size_t blocks = (total + 255) / 256;
    return (unsigned)(blocks > 148 * 16 ? 148 * 16 : blocks);
}

}  // namespace

PB_EXPORT int pb_scaled_sum(int in_dtype, int dtype, const void* x, const void* y, void* out, float a, float b, long long total,
                            cudaStream_t stream) {
    if (total <= 0) return 0;
#define PB_SUM(TI, T) return launch_pdl(scaled_sum_kernel<TI, T>, dim3(blocks_for(total)), dim3(256), 0, stream, (const TI*)x, \
                                        (const TI*)y, (T*)out, a, b, (size_t)total)
    if (in_dtype == PB_F32 && dtype == PB_F32) PB_SUM(float, float);
    if (in_dtype == PB_F32 && dtype == PB_BF16) PB_SUM(float, __nv_bfloat16);
    if (in_dtype == PB_BF16 && dtype == PB_BF16) PB_SUM(__nv_bfloat16, __nv_bfloat16);
    if (in_dtype == PB_BF16 && dtype == PB_F32) PB_SUM(__nv_bfloat16, float);
#undef PB_SUM
    return PB_ERR_BAD_DTYPE;
}

PB_EXPORT int pb_normed_sum(int dtype, const float* x, const float* y, const float* wx, const float* wy, void* out, float a, float b, int n,
                            int width, float eps, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (width <= 0) return PB_ERR_BAD_SIZE;
    if (dtype != PB_F32 && dtype != PB_BF16) return PB_ERR_BAD_DTYPE;
    const bool aligned = (((uintptr_t)x | (uintptr_t)y | (uintptr_t)wx | (uintptr_t)wy | (uintptr_t)out) & 15) == 0;
    if (width % 4 == 0 && aligned && width <= 512 * 16) {
        const int quads = width / 4;
        const int items = quads <= 512 ? 1 : quads <= 1024 ? 2 : 4;
        const int threads = ((quads + items - 1) / items + 31) / 32 * 32;
#define PB_NS(T, I) return launch_pdl(normed_sum_quads_kernel<T, I>, dim3(n), dim3(threads), 0, stream, x, y, wx, wy, (T*)out, a, b, width, eps)
        if (dtype == PB_F32) { if (items == 1) PB_NS(float, 1); if (items == 2) PB_NS(float, 2); PB_NS(float, 4); }
        if (items == 1) PB_NS(__nv_bfloat16, 1);
        if (items == 2) PB_NS(__nv_bfloat16, 2);
        PB_NS(__nv_bfloat16, 4);
#undef PB_NS
    }
    if (dtype == PB_F32) return launch_pdl(normed_sum_kernel<float>, dim3(n), dim3(256), 0, stream, x, y, wx, wy, (float*)out, a, b, width, eps);
    return launch_pdl(normed_sum_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, stream, x, y, wx, wy, (__nv_bfloat16*)out, a, b, width, eps);
}

PB_EXPORT int pb_concat_streams(int dtype, const float* residual, const void* delta, const float* origin, void* out, int n, int width,
                                cudaStream_t stream) {
    if (n <= 0) return 0;
    if (width <= 0) return PB_ERR_BAD_SIZE;
    const size_t total = (size_t)n * width;
    if (dtype == PB_F32)
        return launch_pdl(concat_streams_kernel<float>, dim3(blocks_for(total)), dim3(256), 0, stream, residual, (const float*)delta, origin,
                          (float*)out, width, total);
    if (dtype == PB_BF16)
        return launch_pdl(concat_streams_kernel<__nv_bfloat16>, dim3(blocks_for(total)), dim3(256), 0, stream, residual,
                          (const __nv_bfloat16*)delta, origin, (__nv_bfloat16*)out, width, total);
    return PB_ERR_BAD_DTYPE;
}
