// What stands between the fused q | k (| gate) projection and the general attention kernels when the heads are
// rotated and normed without a weight, and what stands behind those kernels when the heads are gated.
//
//   qk_prepare     per (token, head) of a projection row [q: Hq*D | k: Hkv*D | ...] (float32 or T, row stride given):
//                    x = row + bias                                     (bias float32, optional)
//                    weighted norm (pre_eps >= 0): x / sqrt(mean(x^2) + pre_eps) * w, w float32 [D], one for the query
//                    heads and one for the key heads, before the rotation
//                    key heads with values_from_keys: x, as it is now, goes to the value pool
//                    the first `rotary` dimensions turn in the rotate-half layout: element i pairs with element
//                    i + rotary/2, (u, v) -> (u cos - v sin, v cos + u sin), cos/sin [N, rotary/2] float32
//                    unit norm (eps >= 0): x / sqrt(mean(x^2) + eps) over the head, no weight
//                  queries to float32 [N, Hq, D], keys to the key pool (T).  All arithmetic is float32; the pools
//                  take one rounding.  Hv > 0: Hv value heads of Dv behind the key heads in the row go to the value
//                  pool as they are.
//   qk_prepare_whole   the same place where q and k are normed over their whole projections: per token the RMS norm runs over
//                  all Hq*D query elements (and over all Hkv*D key elements) at once with a weight for each, the heads then
//                  turn (pairs of neighbours or rotate-half), and the value heads may turn too, over `v_rotary` of their Dv
//                  dimensions with a table of their own.  One block per (token, section q | k | v); the section's row sits in
//                  registers, four neighbouring elements at a time, where the sizes allow it, else in shared memory.
//   add_bias       x[n, c] += bias[c] (bias float32): a projection's bias where no kernel behind the product takes it along.
//   sigmoid_gate_strided   x[n, c] *= sigmoid(gate[n, c / group]) with float32 arithmetic; gate float32 or T, a column slice
//                  of a wider row; `group` columns of x share a gate column (a gate per head).
#include "common.cuh"

namespace {

using namespace pb;

constexpr int kMaxPerLane = 16;          // head sizes up to 512

template <typename TIn, typename T>
__global__ void qk_prepare_kernel(const TIn* __restrict__ rows, long row_stride, const float* __restrict__ q_bias,
                                  const float* __restrict__ k_bias, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                  float* __restrict__ q_out, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                  const int* __restrict__ slots, int Hq, int Hkv, int D, int rotary, float eps, int unit_norm,
                                  int values_from_keys, int page_size, const float* __restrict__ q_norm_w,
                                  const float* __restrict__ k_norm_w, float pre_eps, int Hv, int Dv, const PoolBounds bounds) {
    pdl_wait();
    extern __shared__ float smem[];                      // [warps][D]
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int head = blockIdx.y * (blockDim.x >> 5) + warp;
    if (head >= Hq + Hkv + Hv) return;
    if (head >= Hq + Hkv) {                              // a value head: copied to its page
        const int hv = head - Hq - Hkv;
        const int slot = slots[t];
        if (slot < 0 || !slot_ok(slot, page_size, bounds)) return;
        const TIn* src = rows + (size_t)t * row_stride + (size_t)(Hq + Hkv) * D + (size_t)hv * Dv;
        T* dst = v_pool + (((size_t)(slot / page_size) * Hv + hv) * page_size + slot % page_size) * Dv;
        for (int i = lane; i < Dv; i += 32) dst[i] = from_float<T>(to_float(src[i]));
        return;
    }
    float* x = smem + (size_t)warp * D;
    const bool is_q = head < Hq;
    const TIn* src = rows + (size_t)t * row_stride + (size_t)head * D;       // key heads follow the query heads
    const float* bias = is_q ? (q_bias ? q_bias + (size_t)head * D : nullptr) : (k_bias ? k_bias + (size_t)(head - Hq) * D : nullptr);
    for (int i = lane; i < D; i += 32) x[i] = to_float(src[i]) + (bias ? bias[i] : 0.0f);
    __syncwarp();
    int slot = -1;
    size_t at = 0;
    if (!is_q) {
        slot = slots[t];
        if (slot < 0 || !slot_ok(slot, page_size, bounds)) return;           // uniform over the warp
        at = (((size_t)(slot / page_size) * Hkv + (head - Hq)) * page_size + slot % page_size) * D;
        if (values_from_keys)
            for (int i = lane; i < D; i += 32) v_pool[at + i] = from_float<T>(x[i]);
    }
    const float* pre_w = is_q ? q_norm_w : k_norm_w;
    if (pre_w != nullptr) {
        float ss = 0.0f;
        for (int i = lane; i < D; i += 32) ss += x[i] * x[i];
        const float r = rsqrtf(warp_sum(ss) / (float)D + pre_eps);
        for (int i = lane; i < D; i += 32) x[i] = x[i] * r * pre_w[i];
        __syncwarp();
    }
    const int half = rotary >> 1;
    const float* c = cos_t + (size_t)t * half;
    const float* s = sin_t + (size_t)t * half;
    for (int i = lane; i < half; i += 32) {
        const float u = x[i], v = x[i + half];
        x[i] = u * c[i] - v * s[i];
        x[i + half] = v * c[i] + u * s[i];
    }
    __syncwarp();
    float inv = 1.0f;
    if (unit_norm) {
        float ss = 0.0f;
        for (int i = lane; i < D; i += 32) ss += x[i] * x[i];
        inv = rsqrtf(warp_sum(ss) / (float)D + eps);
    }
    if (is_q) {
        float* dst = q_out + ((size_t)t * Hq + head) * D;
        for (int i = lane; i < D; i += 32) dst[i] = x[i] * inv;
    } else {
        for (int i = lane; i < D; i += 32) k_pool[at + i] = from_float<T>(x[i] * inv);
    }
}

struct WholeShape {
    int Hq, Hkv, Hv, D, Dv, rotary, v_rotary, neighbours, page_size;
    float eps;
};

template <typename T>
__device__ __forceinline__ void put(T* dst, size_t at, float v) { dst[at] = from_float<T>(v); }

template <typename TIn, typename T>
__global__ void qk_prepare_whole_kernel(const TIn* __restrict__ rows, long row_stride, const float* __restrict__ q_norm_w,
                                        const float* __restrict__ k_norm_w, const float* __restrict__ cos_t,
                                        const float* __restrict__ sin_t, const float* __restrict__ v_cos, const float* __restrict__ v_sin,
                                        float* __restrict__ q_out, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                        const int* __restrict__ slots, const WholeShape sh, const PoolBounds bounds) {
    pdl_wait();
    extern __shared__ __align__(16) float x[];           // the section's row
    __shared__ float scratch[32];
    const int t = blockIdx.x, section = blockIdx.y;      // 0: queries, 1: keys, 2: values
    const int heads = section == 0 ? sh.Hq : section == 1 ? sh.Hkv : sh.Hv, D = section == 2 ? sh.Dv : sh.D;
    const int n = heads * D;
    const size_t first = section == 0 ? 0 : (size_t)sh.Hq * sh.D + (section == 2 ? (size_t)sh.Hkv * sh.D : 0);
    int slot = 0;
    if (section != 0) {
        slot = slots[t];
        if (slot < 0 || !slot_ok(slot, sh.page_size, bounds)) return;        // uniform over the block
    }
    const TIn* src = rows + (size_t)t * row_stride + first;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = to_float(src[i]); x[i] = v; ss += v * v; }
    const float* w = section == 0 ? q_norm_w : section == 1 ? k_norm_w : nullptr;
    float r = 1.0f;
    if (w != nullptr) r = rsqrtf(block_sum(ss, scratch) / (float)n + sh.eps);
    __syncthreads();
    const int rotary = section == 2 ? sh.v_rotary : sh.rotary, turning = rotary >> 1, half = (D + 1) >> 1;
    const float* c = (section == 2 ? v_cos : cos_t) + (size_t)t * turning;
    const float* s = (section == 2 ? v_sin : sin_t) + (size_t)t * turning;
    const size_t page = (size_t)(slot / sh.page_size), in_page = slot % sh.page_size;
    for (int i = threadIdx.x; i < heads * half; i += blockDim.x) {           // two elements of a head at a time
        const int head = i / half, j = i - head * half;
        const bool turns = j < turning;
        int a, b;                                                            // the pair's places in the head
        if (sh.neighbours || !turns) { a = 2 * j; b = a + 1; }
        else { a = j; b = j + turning; }
        const bool both = b < D;                                             // an odd head's last element stands alone
        const int ia = head * D + a, ib = head * D + b;
        float u = x[ia], v = both ? x[ib] : 0.0f;
        if (w != nullptr) { u = u * r * w[ia]; v = both ? v * r * w[ib] : 0.0f; }
        if (turns) {
            const float u0 = u;
            u = u0 * c[j] - v * s[j];
            v = v * c[j] + u0 * s[j];
        }
        if (section == 0) {
            const size_t at = (size_t)t * n;
            q_out[at + ia] = u;
            if (both) q_out[at + ib] = v;
        } else {
            const size_t at = ((page * heads + head) * sh.page_size + in_page) * D;
            T* dst = section == 1 ? k_pool : v_pool;
            put(dst, at + a, u);
            if (both) put(dst, at + b, v);
        }
    }
}

// The same for sizes and rows in fours (pairs of neighbours): a thread holds ITERS quads of the section's row in registers.
template <typename TIn, typename T, int ITERS>
__global__ void qk_prepare_whole_quads_kernel(const TIn* __restrict__ rows, long row_stride, const float* __restrict__ q_norm_w,
                                              const float* __restrict__ k_norm_w, const float* __restrict__ cos_t,
                                              const float* __restrict__ sin_t, const float* __restrict__ v_cos,
                                              const float* __restrict__ v_sin, float* __restrict__ q_out, T* __restrict__ k_pool,
                                              T* __restrict__ v_pool, const int* __restrict__ slots, const WholeShape sh,
                                              const PoolBounds bounds) {
    pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x, section = blockIdx.y;      // 0: queries, 1: keys, 2: values
    const int heads = section == 0 ? sh.Hq : section == 1 ? sh.Hkv : sh.Hv, D = section == 2 ? sh.Dv : sh.D;
    const int n = heads * D;
    const size_t first = section == 0 ? 0 : (size_t)sh.Hq * sh.D + (section == 2 ? (size_t)sh.Hkv * sh.D : 0);
    int slot = 0;
    if (section != 0) {
        slot = slots[t];
        if (slot < 0 || !slot_ok(slot, sh.page_size, bounds)) return;        // uniform over the block
    }
    const TIn* src = rows + (size_t)t * row_stride + first;
    float x[ITERS][4];
    float ss = 0.0f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int i = (threadIdx.x + it * blockDim.x) * 4;
        if (i < n) {
            load_quad(src + i, x[it]);
#pragma unroll
            for (int e = 0; e < 4; ++e) ss += x[it][e] * x[it][e];
        }
    }
    const float* w = section == 0 ? q_norm_w : section == 1 ? k_norm_w : nullptr;
    float r = 1.0f;
    if (w != nullptr) r = rsqrtf(block_sum(ss, scratch) / (float)n + sh.eps);
    const int rotary = section == 2 ? sh.v_rotary : sh.rotary, turning = rotary >> 1;
    const float* c = (section == 2 ? v_cos : cos_t) + (size_t)t * turning;
    const float* s = (section == 2 ? v_sin : sin_t) + (size_t)t * turning;
    const size_t page = (size_t)(slot / sh.page_size), in_page = slot % sh.page_size;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int i = (threadIdx.x + it * blockDim.x) * 4;
        if (i >= n) continue;
        const int head = i / D, at = i - head * D;
        float y[4] = {x[it][0], x[it][1], x[it][2], x[it][3]};
        if (w != nullptr) {
            float wv[4];
            load_quad(w + i, wv);
#pragma unroll
            for (int e = 0; e < 4; ++e) y[e] = y[e] * r * wv[e];
        }
        if (at < rotary) {                               // both pairs of the quad turn (rotary is a multiple of 4)
            const float2 cc = *reinterpret_cast<const float2*>(c + (at >> 1)), sn = *reinterpret_cast<const float2*>(s + (at >> 1));
            const float u0 = y[0], u1 = y[2];
            y[0] = u0 * cc.x - y[1] * sn.x;
            y[1] = y[1] * cc.x + u0 * sn.x;
            y[2] = u1 * cc.y - y[3] * sn.y;
            y[3] = y[3] * cc.y + u1 * sn.y;
        }
        if (section == 0) store_quad(q_out + (size_t)t * n + i, y);
        else store_quad((section == 1 ? k_pool : v_pool) + ((page * heads + head) * sh.page_size + in_page) * D + at, y);
    }
}

template <typename TIn, typename T>
int launch_whole(const void* rows, long row_stride, const float* q_norm_w, const float* k_norm_w, const float* cos_t, const float* sin_t,
                 const float* v_cos, const float* v_sin, float* q_out, void* k_pool, void* v_pool, const int* slots, int n,
                 const WholeShape& sh, cudaStream_t stream) {
    int widest = sh.Hq * sh.D;
    if (sh.Hkv * sh.D > widest) widest = sh.Hkv * sh.D;
    if (sh.Hv * sh.Dv > widest) widest = sh.Hv * sh.Dv;
    auto aligned = [](const void* p, size_t bytes) { return ((uintptr_t)p % bytes) == 0; };
    const bool quads = sh.neighbours && sh.D % 4 == 0 && sh.Dv % 4 == 0 && sh.rotary % 4 == 0 && sh.v_rotary % 4 == 0 && row_stride % 4 == 0 &&
                       aligned(rows, 4 * sizeof(TIn)) && aligned(q_out, 16) && aligned(k_pool, 4 * sizeof(T)) && aligned(v_pool, 4 * sizeof(T)) &&
                       aligned(q_norm_w, 16) && aligned(k_norm_w, 16) && aligned(cos_t, 8) && aligned(sin_t, 8) && aligned(v_cos, 8) && aligned(v_sin, 8);
    if (quads && widest <= 4 * 4 * 1024) {
        const int n_quads = widest / 4, iters = n_quads > 2048 ? 4 : n_quads > 256 ? 2 : 1;
        const int threads_q = ((n_quads + iters - 1) / iters + 31) / 32 * 32;
#define PB_QUADS(ITERS) return launch_pdl(qk_prepare_whole_quads_kernel<TIn, T, ITERS>, dim3(n, sh.Hkv > 0 ? 3 : 1), dim3(threads_q), 0, stream,     \
                                          (const TIn*)rows, row_stride, q_norm_w, k_norm_w, cos_t, sin_t, v_cos, v_sin, q_out, (T*)k_pool, \
                                          (T*)v_pool, slots, sh, pool_bounds_now())
        if (iters == 1) PB_QUADS(1);
        if (iters == 2) PB_QUADS(2);
        PB_QUADS(4);
#undef PB_QUADS
    }
    const size_t smem = sizeof(float) * (size_t)widest;
    if (smem > 200 * 1024) return PB_ERR_TOO_LARGE;
    static size_t allowed = 48 * 1024;                     // per instantiation
    if (smem > allowed) {
        const cudaError_t e = cudaFuncSetAttribute(qk_prepare_whole_kernel<TIn, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        allowed = smem;
    }
    int threads = 64;
    while (threads < 512 && threads * 8 < widest) threads <<= 1;
    return launch_pdl(qk_prepare_whole_kernel<TIn, T>, dim3(n, sh.Hkv > 0 ? 3 : 1), dim3(threads), smem, stream, (const TIn*)rows,
                      row_stride, q_norm_w, k_norm_w, cos_t, sin_t, v_cos, v_sin, q_out, (T*)k_pool, (T*)v_pool, slots, sh,
                      pool_bounds_now());
}

template <typename T, typename TG>
__global__ void sigmoid_gate_strided_kernel(T* __restrict__ x, const TG* __restrict__ gate, long gate_stride, int width, int group,
                                            size_t total) {
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t row = i / width, col = i % width;
        const float g = to_float(gate[row * gate_stride + col / group]);
        x[i] = from_float<T>(to_float(x[i]) / (1.0f + expf(-g)));
    }
}

template <typename T>
__global__ void add_bias_kernel(T* __restrict__ x, const float* __restrict__ bias, int width, size_t total) {
    pdl_wait();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
        x[i] = from_float<T>(to_float(x[i]) + bias[i % width]);
}

template <typename TIn, typename T>
int launch_prepare(const void* rows, long row_stride, const float* q_bias, const float* k_bias, const float* cos_t, const float* sin_t,
                   float* q_out, void* k_pool, void* v_pool, const int* slots, int n, int Hq, int Hkv, int D, int rotary, float eps,
                   int unit_norm, int values_from_keys, int page_size, const float* q_norm_w, const float* k_norm_w, float pre_eps,
                   int Hv, int Dv, cudaStream_t stream) {
    const int warps = 4;
    dim3 grid(n, (Hq + Hkv + Hv + warps - 1) / warps);
    return launch_pdl(qk_prepare_kernel<TIn, T>, grid, dim3(warps * 32), sizeof(float) * warps * D, stream, (const TIn*)rows, row_stride,
                      q_bias, k_bias, cos_t, sin_t, q_out, (T*)k_pool, (T*)v_pool, slots, Hq, Hkv, D, rotary, eps, unit_norm,
                      values_from_keys, page_size, q_norm_w, k_norm_w, pre_eps, Hv, Dv, pool_bounds_now());
}

}  // namespace

// rows [n, row_stride] of dtype in_dtype (query heads, then key heads, D wide each); pools of dtype `dtype`
// [pages, Hkv, page_size, D]; q_out float32 [n, Hq, D]; cos/sin float32 [n, rotary / 2]; eps < 0: no unit norm.
// Hkv 0: the rows hold queries only (pools and slots unused).  pre_eps >= 0: the weighted norm before the rotation with
// q_norm_w / k_norm_w float32 [D].  Hv > 0: value heads of Dv behind the key heads; v_pool is [pages, Hv, page_size, Dv].
PB_EXPORT int pb_qk_prepare(int in_dtype, int dtype, const void* rows, long row_stride, const float* q_bias, const float* k_bias,
                            const float* cos_t, const float* sin_t, float* q_out, void* k_pool, void* v_pool, const int* slots,
                            int n, int Hq, int Hkv, int D, int rotary, float eps, int values_from_keys, int page_size,
                            const float* q_norm_w, const float* k_norm_w, float pre_eps, int Hv, int Dv, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (Hv < 0 || (Hv > 0 && (Dv <= 0 || v_pool == nullptr || slots == nullptr || values_from_keys)) ||
        row_stride < (long)(Hq + Hkv) * D + (long)Hv * Dv || (pre_eps >= 0.0f && q_norm_w == nullptr) ||
        (pre_eps >= 0.0f && Hkv > 0 && k_norm_w == nullptr))
        return PB_ERR_BAD_SIZE;
    if (pre_eps < 0.0f) q_norm_w = k_norm_w = nullptr;
    if (Hq <= 0 || Hkv < 0 || D <= 0 || D > 32 * kMaxPerLane * 4 || rotary < 0 || rotary > D || rotary % 2 || page_size <= 0 ||
        row_stride < (long)(Hq + Hkv) * D || (Hkv > 0 && (k_pool == nullptr || slots == nullptr)) ||
        (values_from_keys && Hkv > 0 && v_pool == nullptr) || (rotary > 0 && (cos_t == nullptr || sin_t == nullptr)))
        return PB_ERR_BAD_SIZE;
    if ((Hq + Hkv + Hv + 3) / 4 > 65535) return PB_ERR_TOO_LARGE;
    const int unit = eps >= 0.0f ? 1 : 0;
#define PB_PREP(TI, T) return launch_prepare<TI, T>(rows, row_stride, q_bias, k_bias, cos_t, sin_t, q_out, k_pool, v_pool, slots, n, Hq, \
                                                    Hkv, D, rotary, eps, unit, values_from_keys, page_size, q_norm_w, k_norm_w, pre_eps, Hv, Dv, stream)
    if (in_dtype == PB_F32 && dtype == PB_F32) PB_PREP(float, float);
    if (in_dtype == PB_F32 && dtype == PB_BF16) PB_PREP(float, __nv_bfloat16);
    if (in_dtype == PB_BF16 && dtype == PB_BF16) PB_PREP(__nv_bfloat16, __nv_bfloat16);
    if (in_dtype == PB_BF16 && dtype == PB_F32) PB_PREP(__nv_bfloat16, float);
#undef PB_PREP
    return PB_ERR_BAD_DTYPE;
}

// rows [n, row_stride] of dtype in_dtype: query heads, key heads (D each), value heads (Dv each).  q_norm_w float32 [Hq*D],
// k_norm_w [Hkv*D] (null: no norm).  cos/sin float32 [n, rotary / 2], v_cos/v_sin [n, v_rotary / 2]; neighbours: elements 2j
// and 2j + 1 are a pair (else rotate-half).  Queries to q_out float32 [n, Hq, D], keys to k_pool [pages, Hkv, page_size, D], values to
// v_pool [pages, Hv, page_size, Dv] (dtype).  Hkv 0: the rows hold queries only.
PB_EXPORT int pb_qk_prepare_whole(int in_dtype, int dtype, const void* rows, long row_stride, const float* q_norm_w, const float* k_norm_w,
                                  float eps, const float* cos_t, const float* sin_t, const float* v_cos, const float* v_sin,
                                  float* q_out, void* k_pool, void* v_pool, const int* slots, int n, int Hq, int Hkv, int D, int Hv, int Dv,
                                  int rotary, int v_rotary, int neighbours, int page_size, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (Hq <= 0 || Hkv < 0 || D <= 0 || rotary < 0 || rotary > D || rotary % 2 || page_size <= 0 || !(eps >= 0.0f) ||
        (rotary > 0 && (cos_t == nullptr || sin_t == nullptr)))
        return PB_ERR_BAD_SIZE;
    if (Hkv > 0 && (Hv <= 0 || Dv <= 0 || v_rotary < 0 || v_rotary > Dv || v_rotary % 2 || k_pool == nullptr ||
                    v_pool == nullptr || slots == nullptr || (v_rotary > 0 && (v_cos == nullptr || v_sin == nullptr))))
        return PB_ERR_BAD_SIZE;
    if (Hkv == 0) Hv = Dv = v_rotary = 0;
    if (row_stride < (long)(Hq + Hkv) * D + (long)Hv * Dv) return PB_ERR_BAD_SIZE;
    const WholeShape sh{Hq, Hkv, Hv, D, Dv, rotary, v_rotary, neighbours != 0, page_size, eps};
#define PB_WHOLE(TI, T) return launch_whole<TI, T>(rows, row_stride, q_norm_w, k_norm_w, cos_t, sin_t, v_cos, v_sin, q_out, k_pool, v_pool, slots, n, sh, stream)
    if (in_dtype == PB_F32 && dtype == PB_F32) PB_WHOLE(float, float);
    if (in_dtype == PB_F32 && dtype == PB_BF16) PB_WHOLE(float, __nv_bfloat16);
    if (in_dtype == PB_BF16 && dtype == PB_BF16) PB_WHOLE(__nv_bfloat16, __nv_bfloat16);
#undef PB_WHOLE
    return PB_ERR_BAD_DTYPE;
}

// x [n, width] (dtype) *= sigmoid(gate[n, c / group]) where gate rows are gate_stride elements apart (gate_dtype): `group`
// neighbouring columns of x share one gate column (1: a gate per element; a head's width: a gate per head).
PB_EXPORT int pb_sigmoid_gate_strided(int dtype, int gate_dtype, void* x, const void* gate, long gate_stride, int n, int width,
                                      int group, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (width <= 0 || group <= 0 || width % group || gate_stride < width / group) return PB_ERR_BAD_SIZE;
    const size_t total = (size_t)n * width;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
#define PB_GATE(T, TG) return launch_pdl(sigmoid_gate_strided_kernel<T, TG>, dim3((unsigned)blocks), dim3(256), 0, stream, (T*)x, \
                                         (const TG*)gate, gate_stride, width, group, total)
    if (dtype == PB_F32 && gate_dtype == PB_F32) PB_GATE(float, float);
    if (dtype == PB_BF16 && gate_dtype == PB_F32) PB_GATE(__nv_bfloat16, float);
    if (dtype == PB_BF16 && gate_dtype == PB_BF16) PB_GATE(__nv_bfloat16, __nv_bfloat16);
    if (dtype == PB_F32 && gate_dtype == PB_BF16) PB_GATE(float, __nv_bfloat16);
#undef PB_GATE
    return PB_ERR_BAD_DTYPE;
}

// x [n, width] (dtype) += bias [width] (float32).
PB_EXPORT int pb_add_bias(int dtype, void* x, const float* bias, int n, int width, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (width <= 0 || bias == nullptr) return PB_ERR_BAD_SIZE;
    const size_t total = (size_t)n * width;
    size_t blocks = (total + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    if (dtype == PB_F32) return launch_pdl(add_bias_kernel<float>, dim3((unsigned)blocks), dim3(256), 0, stream, (float*)x, bias, width, total);
    if (dtype == PB_BF16)
        return launch_pdl(add_bias_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(256), 0, stream, (__nv_bfloat16*)x, bias, width, total);
    return PB_ERR_BAD_DTYPE;
}
