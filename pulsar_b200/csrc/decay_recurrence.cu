// Linear recurrences whose matrix state decays by one factor per (token, head), and the two mixers built on them.
//
//   S_t = a_t S_(t-1) + b_t k_t v_t^T        S [D, V] float32, kept per sequence in a state slot, zero at the start
//   r_t = S_t^T q_t                          [V]
//
//   matrix memory (exponential gates)   i = cap tanh((i' + i_bias) / cap), f = logsigmoid(cap tanh((f' + f_bias) / cap)) per
//       head; the running maximum m_t = max(f + m_(t-1), i) (zero at the start) keeps a_t = exp(f + m_(t-1) - m_t) and
//       b_t = exp(i - m_t) small; n_t follows S_t with k alone; o = r / (max(|n . q|, exp(-m)) + denom_eps); then per head
//       o / rms(o) * weight * sigmoid(g).
//   state space with a scalar decay     x, B and C (channels of one row) pass a short causal convolution and silu; dt =
//       softplus(dt' + dt_bias), a_t = exp(-exp(A_log) dt), b_t = dt, k = B, q = C (shared by the heads of a group), v = x;
//       y = r + D x; then y * silu(z), normed in equal parts of the row, * weight.
//
// Both arrive as float32 rows [N, stride] of one projection.  Three forms:
//
//   recurrence_step        token by token: a block per (head, sequence, tile of columns); thread (column, slice) holds its rows of a
//                          column of S in registers, so a token costs one pass over the state.  Decoding, short portions, and
//                          the float32 engine.  Where one block holds a head of the matrix memory it does the gates, the
//                          denominator, the norm and the output gate as well; the state space's convolution and step size
//                          are done in the block too.
//   recurrence_chunk_*     portions in chunks of kChunk tokens, parallel over chunks, on the tensor cores (bfloat16 engine):
//                            state   U_c = sum_j (decay behind j) b_j k_j v_j^T over the chunk's tokens        (per chunk, head)
//                            fold    S_in(c) = state entering chunk c; S <- decay(c) S + U_c along a sequence  (per element)
//                            out     r_i = sum_(j<=i) decay(j..i) b_j (q_i . k_j) v_j + decay(..i) S_in^T q_i
//                          q, k and v are rounded to bfloat16 once (as projections may be); everything of the recurrence
//                          that meets a tensor core (weighted values, weighted scores, the entering state) is split into two
//                          bfloat16 numbers, hi + lo (16 bits of mantissa together), and enters two MMAs with the same
//                          float32 accumulator.  The normaliser n and its products are float32 on CUDA cores.
//   gates, gated_norm      what stands before the chunks (log decays and input weights per token and head; for the matrix memory
//                          a scan over the tokens, m is max-plus linear) and behind the forms that leave raw rows.
#include "mma_common.cuh"

namespace {

using namespace pb;

constexpr int kChunk = 64;              // tokens of a chunk
constexpr int kCols = 64;               // value columns of a block in the chunked form
constexpr int kPad = 8;                 // bfloat16 elements behind a shared-memory row: rows fall on different banks
constexpr float kLeastLogDecay = -104.0f;      // exp of it is below the smallest float32: nothing of a state survives it

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float log_sigmoid_f(float v) { return fminf(v, 0.0f) - log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float capped(float v, float cap) { return cap * tanhf(v / cap); }

__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 hf = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - hf.x, y - hf.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Where a step's sequences and their state live.
struct Step {
    const int *cu_q, *state_slots;
    float* state;
    long state_stride;
    int n, n_seqs;
};

// The convolution in front of the state space: `channels` columns of the rows from `off` on.
struct Conv {
    const float *taps, *bias;           // [channels, n_taps], [channels]
    int off, channels, n_taps;
    long tail_off;                      // in a slot: [channels, n_taps - 1], the last inputs of the sequence
};

// ------------------------------------------------------------------------------------------------ token by token
enum StepMode { kMemoryWhole = 0, kGiven = 1, kStateSpace = 2 };

struct StepArgs {
    Step st;
    const float* rows;
    long stride;
    int H, D, V;
    int cols, tile, slices;             // columns of the state (the normaliser is one more), columns of a block, slices of D
    int q_off, k_off, v_off;            // in a row; the state space: C, B and x inside the convolution's channels
    int share;                          // heads that read the same q and k
    float q_scale;
    // matrix memory
    int g_off, i_off, f_off;
    const float *i_bias, *f_bias, *norm_w;
    float cap, denom_eps, eps;
    const float *ld, *wt;               // kGiven: log decays and input weights [N, H]
    float* den;                         // kGiven: n . q [N, H]
    // state space
    Conv conv;
    int dt_off;
    const float *dt_bias, *a_log, *d_skip;
    float* raw;                         // [N, H, V]
};

__device__ __forceinline__ float conv_silu_at(const StepArgs& a, const float* tail, int t, int i, int c) {
    float acc = a.conv.bias[c];
    const int T = a.conv.n_taps;
    for (int tau = 0; tau < T; ++tau) {
        const int back = T - 1 - tau;
        const float v = i >= back ? a.rows[(size_t)(t - back) * a.stride + a.conv.off + c] : tail[(size_t)c * (T - 1) + T - 1 + i - back];
        acc = fmaf(a.conv.taps[(size_t)c * T + tau], v, acc);
    }
    return silu_f(acc);
}

template <typename T, int PER, int THREADS, int MODE>
__global__ void __launch_bounds__(THREADS) recurrence_step_kernel(const StepArgs a, T* __restrict__ y) {
    pdl_wait();
    extern __shared__ __align__(16) float smem[];
    const int Dp = a.slices * PER;
    const int buf_size = 2 * Dp + ((a.tile + 3) & ~3) + 4;
    float* red = smem + 2 * buf_size;                     // [32], behind two of: q [Dp], k [Dp], v [tile], scalars [4]
    float* part = red + 32;                               // [slices][tile]
    const int h = blockIdx.x, s = blockIdx.y, c0 = blockIdx.z * a.tile, tid = threadIdx.x;
    const int c = tid % a.tile, ds = tid / a.tile, col = c0 + c;
    const int cols_here = min(a.tile, a.cols - c0);
    const bool on = ds < a.slices && c < cols_here;
    const int d0 = ds * PER;
    const int t0 = a.st.cu_q[s], t1 = a.st.cu_q[s + 1];
    float* slot = a.st.state + (size_t)a.st.state_slots[s] * a.st.state_stride;
    const size_t HDV = (size_t)a.H * a.D * a.V;
    float* kept = col < a.V ? slot + (size_t)h * a.D * a.V + col : slot + HDV + (size_t)h * a.D;     // the normaliser: D numbers
    const size_t kept_step = col < a.V ? a.V : 1;
    float* kept_m = slot + HDV + (size_t)a.H * a.D + h;
    const float* tail = MODE == kStateSpace ? slot + a.conv.tail_off : nullptr;
    kept += (size_t)d0 * kept_step;
    const int rows_here = on ? min(PER, a.D - d0) : 0;
    float S[PER];
    {
        const float* p = kept;
#pragma unroll
        for (int i = 0; i < PER; ++i, p += kept_step) S[i] = i < rows_here ? *p : 0.0f;
    }
    float m = (MODE == kMemoryWhole && tid == 0) ? *kept_m : 0.0f;
    const int qh = h / a.share;
    for (int t = t0; t < t1; ++t) {
        float* qs = smem + ((t - t0) & 1) * buf_size;
        float* ks = qs + Dp;
        float* sc = ks + Dp;
        float* vs = sc + 4;
        const float* row = a.rows + (size_t)t * a.stride;
        if (MODE == kStateSpace) {
            // (one loop over the three rows, so that a block's loads are in flight together)
            for (int i = tid; i < 2 * Dp + cols_here; i += blockDim.x) {
                const int which = i < Dp ? 0 : i < 2 * Dp ? 1 : 2;
                const int d = which == 0 ? i : which == 1 ? i - Dp : i - 2 * Dp;
                float v = 0.0f;
                if (which == 2 || d < a.D) {
                    const int ch = which == 0 ? a.q_off + qh * a.D + d : which == 1 ? a.k_off + qh * a.D + d : a.v_off + h * a.V + c0 + d;
                    v = conv_silu_at(a, tail, t, t - t0, ch);
                }
                (which == 0 ? qs : which == 1 ? ks : vs)[d] = v;
            }
        } else {
            for (int i = tid; i < Dp; i += blockDim.x) {
                const bool in = i < a.D;
                qs[i] = in ? row[a.q_off + qh * a.D + i] * a.q_scale : 0.0f;
                ks[i] = in ? row[a.k_off + qh * a.D + i] : 0.0f;
            }
            for (int i = tid; i < cols_here; i += blockDim.x) vs[i] = c0 + i < a.V ? row[a.v_off + h * a.V + c0 + i] : 1.0f;
        }
        if (tid == 0) {
            if (MODE == kMemoryWhole) {
                const float gi = capped(row[a.i_off + h] + a.i_bias[h], a.cap);
                const float gf = log_sigmoid_f(capped(row[a.f_off + h] + a.f_bias[h], a.cap));
                const float next = fmaxf(gf + m, gi);
                sc[0] = expf(gf + m - next);
                sc[1] = expf(gi - next);
                sc[2] = expf(-next);
                m = next;
            } else if (MODE == kGiven) {
                sc[0] = expf(a.ld[(size_t)t * a.H + h]);
                sc[1] = a.wt[(size_t)t * a.H + h];
            } else {
                const float dt = softplus_f(row[a.dt_off + h] + a.dt_bias[h]);
                sc[0] = expf(-expf(a.a_log[h]) * dt);
                sc[1] = dt;
            }
        }
        __syncthreads();
        const float keep = sc[0], vb = on ? sc[1] * vs[c] : 0.0f;
        if (on) {
            float acc = 0.0f;
#pragma unroll
            for (int i = 0; i < PER; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4*>(ks + d0 + i), q4 = *reinterpret_cast<const float4*>(qs + d0 + i);
                S[i] = fmaf(keep, S[i], k4.x * vb);
                S[i + 1] = fmaf(keep, S[i + 1], k4.y * vb);
                S[i + 2] = fmaf(keep, S[i + 2], k4.z * vb);
                S[i + 3] = fmaf(keep, S[i + 3], k4.w * vb);
                acc = fmaf(S[i], q4.x, acc);
                acc = fmaf(S[i + 1], q4.y, acc);
                acc = fmaf(S[i + 2], q4.z, acc);
                acc = fmaf(S[i + 3], q4.w, acc);
            }
            part[ds * a.tile + c] = acc;
        }
        __syncthreads();
        float o = 0.0f;
        const bool mine = on && ds == 0;
        if (mine)
            for (int k = 0; k < a.slices; ++k) o += part[k * a.tile + c];
        if (MODE == kMemoryWhole) {
            float size = 0.0f;
            for (int k = 0; k < a.slices; ++k) size += part[k * a.tile + a.V];          // one tile: the normaliser is its last column
            o = (mine && col < a.V) ? o / (fmaxf(fabsf(size), sc[2]) + a.denom_eps) : 0.0f;
            const float ss = block_sum(o * o, red);
            if (mine && col < a.V) {
                const float g = row[a.g_off + h * a.V + col];
                y[((size_t)t * a.H + h) * a.V + col] =
                    from_float<T>(o * rsqrtf(ss / (float)a.V + a.eps) * a.norm_w[h * a.V + col] * sigmoid_f(g));
            }
        } else if (mine) {
            if (col < a.V) a.raw[((size_t)t * a.H + h) * a.V + col] = MODE == kStateSpace ? fmaf(a.d_skip[h], vs[c], o) : o;
            else a.den[(size_t)t * a.H + h] = o;
        }
    }
    {
        float* p = kept;
#pragma unroll
        for (int i = 0; i < PER; ++i, p += kept_step)
            if (i < rows_here) *p = S[i];
    }
    if (MODE == kMemoryWhole && tid == 0) *kept_m = m;
}

// ------------------------------------------------------------------------------------------------ gates
// Log decays, input weights and floors of the matrix memory, [N, H]: a block per (head, sequence) walks the tokens blockDim at a
// time.  A token maps m to max(f + m, i); maps compose as (F, M) then (f, i) = (F + f, max(f + M, i)), so the block scans them.
__global__ void __launch_bounds__(1024) memory_gates_kernel(const float* __restrict__ rows, long stride, int i_off, int f_off, const float* __restrict__ i_bias,
                                    const float* __restrict__ f_bias, float cap, const Step st, long m_off, int H,
                                    float* __restrict__ ld, float* __restrict__ wt, float* __restrict__ floor_out) {
    pdl_wait();
    __shared__ float wf[32], wm[32], last;
    const int h = blockIdx.x, s = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int t0 = st.cu_q[s], t1 = st.cu_q[s + 1];
    float* kept_m = st.state + (size_t)st.state_slots[s] * st.state_stride + m_off + h;
    float m_in = *kept_m;
    const float bi = i_bias[h], bf = f_bias[h];
    float pre_i = 0.0f, pre_f = 0.0f;                     // the next round's pre-activations, fetched a round ahead
    if (t0 + (int)threadIdx.x < t1) {
        pre_i = rows[(size_t)(t0 + threadIdx.x) * stride + i_off + h];
        pre_f = rows[(size_t)(t0 + threadIdx.x) * stride + f_off + h];
    }
    for (int base = t0; base < t1; base += blockDim.x) {
        const int t = base + threadIdx.x;
        const bool in = t < t1;
        float gi = -INFINITY, gf = 0.0f;                  // behind the end: a map that changes nothing
        if (in) {
            gi = capped(pre_i + bi, cap);
            gf = log_sigmoid_f(capped(pre_f + bf, cap));
        }
        if (t + (int)blockDim.x < t1) {
            pre_i = rows[(size_t)(t + blockDim.x) * stride + i_off + h];
            pre_f = rows[(size_t)(t + blockDim.x) * stride + f_off + h];
        }
        float F = gf, M = gi;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) { M = fmaxf(F + Mp, M); F += Fp; }
        }
        if (lane == 31) { wf[warp] = F; wm[warp] = M; }
        __syncthreads();
        float m = m_in;                                   // the maximum that enters this warp's tokens
        for (int w = 0; w < warp; ++w) m = fmaxf(wf[w] + m, wm[w]);
        const float now = fmaxf(F + m, M);
        float before = __shfl_up_sync(0xffffffffu, now, 1);
        if (lane == 0) before = m;
        if (in) {
            ld[(size_t)t * H + h] = gf + before - now;
            wt[(size_t)t * H + h] = expf(gi - now);
            floor_out[(size_t)t * H + h] = expf(-now);
        }
        if (warp == warps - 1 && lane == 31) last = now;
        __syncthreads();
        m_in = last;
        __syncthreads();
    }
    if (threadIdx.x == 0) *kept_m = m_in;
}

// The state space's: ld = -exp(A_log) dt, wt = dt.
__global__ void space_gates_kernel(const float* __restrict__ rows, long stride, int dt_off, const float* __restrict__ dt_bias,
                                   const float* __restrict__ a_log, int H, int total, float* __restrict__ ld, float* __restrict__ wt) {
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= total) return;
    const int t = e / H, h = e - t * H;
    const float dt = softplus_f(rows[(size_t)t * stride + dt_off + h] + dt_bias[h]);
    ld[e] = -expf(a_log[h]) * dt;
    wt[e] = dt;
}

// ------------------------------------------------------------------------------------------------ chunks
// The chunk `chunk` of a step whose sequence s has ceil(q_len / kChunk) chunks: its sequence and tokens [t0, t1).
__device__ __forceinline__ bool find_chunk(const int* cu_q, int n_seqs, int chunk, int& s, int& t0, int& t1) {
    int base = 0;
    for (s = 0; s < n_seqs; ++s) {
        const int q0 = cu_q[s], len = cu_q[s + 1] - q0;
        const int nc = (len + kChunk - 1) / kChunk;
        if (chunk < base + nc) {
            t0 = q0 + (chunk - base) * kChunk;
            t1 = min(t0 + kChunk, q0 + len);
            return true;
        }
        base += nc;
    }
    return false;
}

// Rows of q, k and v: element d of head h of token t at base + t * tok + (h / share) * D + d.
template <typename T> struct Source {
    const T *q, *k, *v;
    long tok;
    int share;
};

// A chunk's state of a head in memory: [D, V] filled up to whole tiles of 16 rows and 8 columns (Dp, Vp; zeros), tile by tile
// (rows of tiles first) in the order in which the lanes of a warp take a B operand of m16n8k16: lane l holds column l / 4 and
// rows 2 (l % 4), 2 (l % 4) + 1 and the same + 8, four numbers of 16 bytes.  The normaliser's D numbers follow.
struct ChunkShape {
    const int* cu_q;
    int n_seqs, H, D, V, normaliser;
    int Dp, Vp;
    long per;                // words of U per (chunk, head): Dp * Vp, then D for the normaliser, rounded up to a multiple of four
    float q_scale;
    int heads;               // heads of a block; they read the same q and k
};

// What warp 0 leaves for a head: cum[j], the sum of the chunk's log decays up to and including token j (zero log decay behind the end;
// two tokens a lane), and weight[j] = the token's input weight, times (kBehind) the decay behind it.  Returns the whole sum.
template <bool kBehind>
__device__ __forceinline__ float chunk_decays(const float* __restrict__ ld, const float* __restrict__ wt, int H, int h, int t0, int n, float* cum,
                                              float* weight) {
    const int lane = threadIdx.x, j = 2 * lane;
    const bool in_a = j < n, in_b = j + 1 < n;
    const size_t at = (size_t)(t0 + j) * H + h;
    const float a = in_a ? fmaxf(ld[at], kLeastLogDecay) : 0.0f, b = in_b ? fmaxf(ld[at + H], kLeastLogDecay) : 0.0f;
    float wa = in_a ? wt[at] : 0.0f, wb = in_b ? wt[at + H] : 0.0f;
    float sum = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float p = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += p;
    }
    const float all = __shfl_sync(0xffffffffu, sum, 31);
    if (kBehind) { wa *= expf(all - (sum - b)); wb *= expf(all - sum); }
    cum[j] = sum - b;
    cum[j + 1] = sum;
    weight[j] = wa;
    weight[j + 1] = wb;
    return all;
}

template <typename T> __device__ __forceinline__ void load4(const T* src, bool vec, int left, float (&v)[4]) {
    if (vec) {
        load_quad(src, v);
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = e < left ? to_float(src[e]) : 0.0f;
    }
}

template <typename T> __device__ __forceinline__ bool quads_aligned(const T* src, long tok, int limit) {
    return (limit & 3) == 0 && (((uintptr_t)src | (uintptr_t)(tok * (long)sizeof(T))) & (4 * sizeof(T) - 1)) == 0;
}

// How 128 threads walk rows of `parts` vectors: a power of two of neighbouring threads per row, the rest over the rows.
struct Lanes {
    int lanes, lane, row, rows;
    __device__ __forceinline__ explicit Lanes(int parts) {
        const int bits = parts >= 128 ? 7 : parts <= 1 ? 0 : 32 - __clz(parts - 1);
        lanes = 1 << bits;
        lane = threadIdx.x & (lanes - 1);
        row = threadIdx.x >> bits;
        rows = 128 >> bits;
    }
};

// Columns [0, limit) of n rows -> kChunk shared rows of bfloat16, `width` columns (stride ld_s); zeros behind the limit and the n rows.
template <typename T>
__device__ __forceinline__ void stage_rows(const T* __restrict__ src, long tok, int n, int limit, int width, bf16* dst, int ld_s) {
    if (sizeof(T) == 2 && (limit & 7) == 0 && (((uintptr_t)src | (uintptr_t)(tok * 2)) & 15) == 0) {      // bfloat16 rows as they are
        const Lanes at(width >> 3);
        for (int d = at.lane << 3; d < width; d += at.lanes << 3)
#pragma unroll 8
            for (int j = at.row; j < kChunk; j += at.rows) {
                const bool in = j < n && d < limit;
                cp_async16(smem_u32(dst + j * ld_s + d), in ? src + (size_t)j * tok + d : src, in);
            }
        cp_async_commit();
        cp_async_wait<0>();
        return;
    }
    const Lanes at(width >> 2);
    const bool vec = quads_aligned(src, tok, limit);
    for (int d = at.lane << 2; d < width; d += at.lanes << 2) {
        if (vec && n == kChunk && d < limit) {            // whole rows: the loads of eight of them in flight together
            for (int j0 = at.row; j0 < kChunk; j0 += 8 * at.rows) {
                float v[8][4];
#pragma unroll
                for (int k = 0; k < 8; ++k)
                    if (j0 + k * at.rows < kChunk) load_quad(src + (size_t)(j0 + k * at.rows) * tok + d, v[k]);
#pragma unroll
                for (int k = 0; k < 8; ++k)
                    if (j0 + k * at.rows < kChunk) store_quad(dst + (j0 + k * at.rows) * ld_s + d, v[k]);
            }
            continue;
        }
        for (int j = at.row; j < kChunk; j += at.rows) {
            float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            if (j < n && d < limit) load4(src + (size_t)j * tok + d, vec, limit - d, v);
            store_quad(dst + j * ld_s + d, v);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(128) recurrence_chunk_state_kernel(const Source<T> in, const float* __restrict__ ld, const float* __restrict__ wt,
                                                                     const ChunkShape sh, float* __restrict__ U, float* __restrict__ total) {
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw_smem[];
    __shared__ float cum[kChunk], coef[kChunk];
    const int ldk = sh.Dp + kPad, ldv = kCols + kPad;
    bf16* ks = reinterpret_cast<bf16*>(raw_smem);         // [kChunk][ldk]
    bf16* vh = ks + kChunk * ldk;                         // [kChunk][ldv] weighted values, high halves
    bf16* vl = vh + kChunk * ldv;                         // low halves
    const int chunk = blockIdx.x, h0 = blockIdx.y * sh.heads, v0 = blockIdx.z * kCols;
    int s, t0, t1;
    if (!find_chunk(sh.cu_q, sh.n_seqs, chunk, s, t0, t1)) return;
    const int n = t1 - t0, cols = min(sh.V - v0, kCols);
    const int NT = sh.Vp >> 3, nt0 = v0 >> 3, tiles = min(NT - nt0, kCols / 8);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tq = lane & 3;
    const int k_steps = (n + 15) >> 4;
    stage_rows(in.k + (size_t)t0 * in.tok + (size_t)(h0 / in.share) * sh.D, in.tok, n, sh.D, sh.Dp, ks, ldk);
    for (int h = h0; h < h0 + sh.heads; ++h) {
        __syncthreads();                                  // the head before has been read
        if (warp == 0) {
            const float all = chunk_decays<true>(ld, wt, sh.H, h, t0, n, cum, coef);
            if (lane == 0 && v0 == 0) total[(size_t)chunk * sh.H + h] = all;
        }
        __syncthreads();
        {
            const T* src = in.v + (size_t)t0 * in.tok + (size_t)h * sh.V + v0;
            const bool vec = quads_aligned(src, in.tok, cols);
            const int v = (threadIdx.x & (kCols / 4 - 1)) << 2, row = threadIdx.x / (kCols / 4);
            constexpr int kRows = 128 / (kCols / 4);
            float xs[kChunk / kRows][4];
#pragma unroll
            for (int k = 0; k < kChunk / kRows; ++k) {
                xs[k][0] = xs[k][1] = xs[k][2] = xs[k][3] = 0.0f;
                if (row + k * kRows < n && v < cols) load4(src + (size_t)(row + k * kRows) * in.tok + v, vec, cols - v, xs[k]);
            }
#pragma unroll
            for (int k = 0; k < kChunk / kRows; ++k) {
                const int j = row + k * kRows;
                const float (&x)[4] = xs[k];
                const float w = coef[j];
                uint2 hi, lo;
                split_bf16(x[0] * w, x[1] * w, hi.x, lo.x);
                split_bf16(x[2] * w, x[3] * w, hi.y, lo.y);
                *reinterpret_cast<uint2*>(vh + j * ldv + v) = hi;
                *reinterpret_cast<uint2*>(vl + j * ldv + v) = lo;
            }
        }
        __syncthreads();
        float* out = U + ((size_t)chunk * sh.H + h) * sh.per;
        if (sh.normaliser && v0 == 0)
            for (int d = threadIdx.x; d < sh.D; d += 128) {
                float sum = 0.0f;
                for (int j = 0; j < n; ++j) sum = fmaf(coef[j], __bfloat162float(ks[j * ldk + d]), sum);
                out[(size_t)sh.Dp * sh.Vp + d] = sum;
            }
        for (int mt = warp; mt < sh.Dp / 16; mt += 4) {
            float acc[kCols / 8][4];
#pragma unroll
            for (int i = 0; i < kCols / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
            for (int kk = 0; kk < k_steps; ++kk) {
                uint32_t a[4];
                ldmatrix_x4_trans(a, smem_u32(ks + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + mt * 16 + ((lane >> 3) & 1) * 8));
                const int at = (kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ldv + (lane >> 4) * 8;
#pragma unroll
                for (int i = 0; i < kCols / 16; ++i) {
                    if (2 * i < tiles) {
                        uint32_t bh[4], bl[4];
                        ldmatrix_x4_trans(bh, smem_u32(vh + at + i * 16));
                        ldmatrix_x4_trans(bl, smem_u32(vl + at + i * 16));
                        mma_bf16(acc[2 * i], a, bh[0], bh[1]);
                        mma_bf16(acc[2 * i + 1], a, bh[2], bh[3]);
                        mma_bf16(acc[2 * i], a, bl[0], bl[1]);
                        mma_bf16(acc[2 * i + 1], a, bl[2], bl[3]);
                    }
                }
            }
            // rows g of neighbouring lanes (g even and odd) change places, so that a lane holds four numbers of the layout
#pragma unroll
            for (int i = 0; i < kCols / 8; ++i) {
                if (i < tiles) {                          // uniform over the block
                    const bool odd = g & 1;
                    const float r0 = __shfl_xor_sync(0xffffffffu, odd ? acc[i][0] : acc[i][1], 4);
                    const float r1 = __shfl_xor_sync(0xffffffffu, odd ? acc[i][2] : acc[i][3], 4);
                    const float4 four = odd ? make_float4(r0, acc[i][1], r1, acc[i][3]) : make_float4(acc[i][0], r0, acc[i][2], r1);
                    const int at = 8 * tq + (odd ? 4 : 0) + (g >> 1);
                    *reinterpret_cast<float4*>(out + ((size_t)(mt * NT + nt0 + i) * 32 + at) * 4) = four;
                }
            }
        }
    }
}

// Along a sequence's chunks: U_c is replaced by the state that enters chunk c (each number as two bfloat16, high and low half of its
// word; the normaliser's stay float32); the state behind the last chunk is kept.
__global__ void recurrence_fold_kernel(float* __restrict__ U, const float* __restrict__ total, const Step st, const ChunkShape sh) {
    pdl_wait();
    const int e = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y, s = blockIdx.z;
    const int DVp = sh.Dp * sh.Vp, DV = sh.D * sh.V;
    if (e >= DVp + (sh.normaliser ? sh.D : 0)) return;
    int first = 0;
    for (int i = 0; i < s; ++i) first += (sh.cu_q[i + 1] - sh.cu_q[i] + kChunk - 1) / kChunk;
    const int nc = (sh.cu_q[s + 1] - sh.cu_q[s] + kChunk - 1) / kChunk;
    float* slot = st.state + (size_t)st.state_slots[s] * st.state_stride;
    const bool matrix = e < DVp;
    float* kept = nullptr;
    if (matrix) {
        const int j = e & 3, ln = (e >> 2) & 31, tile = e >> 7, NT = sh.Vp >> 3;
        const int kk = tile / NT, d = kk * 16 + ((ln & 3) << 1) + (j & 1) + ((j & 2) << 2), v = (tile - kk * NT) * 8 + (ln >> 2);
        if (d < sh.D && v < sh.V) kept = slot + (size_t)h * DV + (size_t)d * sh.V + v;
    } else {
        kept = slot + (size_t)sh.H * DV + (size_t)h * sh.D + (e - DVp);
    }
    float S = kept != nullptr ? *kept : 0.0f;
    float* u0 = U + ((size_t)first * sh.H + h) * sh.per + e;
    const float* tot = total + (size_t)first * sh.H + h;
    const size_t step = (size_t)sh.H * sh.per;
    constexpr int kAhead = 8;                // chunks whose own parts are in flight together: they do not depend on the fold
    for (int c0 = 0; c0 < nc; c0 += kAhead) {
        float own[kAhead], dec[kAhead];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            own[k] = c0 + k < nc ? u0[(size_t)(c0 + k) * step] : 0.0f;
            dec[k] = c0 + k < nc ? tot[(size_t)(c0 + k) * sh.H] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            if (c0 + k < nc) {
                float w = S;
                if (matrix) {
                    const bf16 hi = __float2bfloat16_rn(S), lo = __float2bfloat16_rn(S - __bfloat162float(hi));
                    w = __uint_as_float((uint32_t)__bfloat16_as_ushort(hi) << 16 | __bfloat16_as_ushort(lo));
                }
                u0[(size_t)(c0 + k) * step] = w;
                S = fmaf(expf(dec[k]), S, own[k]);
            }
        }
    }
    if (kept != nullptr) *kept = S;
}

// Four warps, 16 tokens each; kCols columns of the values.  The scores q . k are computed once for the block's heads.
template <typename T>
__global__ void __launch_bounds__(128, 4) recurrence_chunk_out_kernel(const Source<T> in, const float* __restrict__ ld, const float* __restrict__ wt,
                                                                      const ChunkShape sh, const float* __restrict__ S_in,
                                                                      const float* __restrict__ d_skip, float* __restrict__ out,
                                                                      float* __restrict__ den) {
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw_smem[];
    __shared__ float cum[kChunk], weight[kChunk];
    const int ldk = sh.Dp + kPad, ldv = kCols + kPad;
    bf16* qs = reinterpret_cast<bf16*>(raw_smem);         // [kChunk][ldk]
    bf16* ks = qs + kChunk * ldk;                         // [kChunk][ldk]
    bf16* vs = ks + kChunk * ldk;                         // [kChunk][ldv]
    const int chunk = blockIdx.x, h0 = blockIdx.y * sh.heads, v0 = blockIdx.z * kCols;
    int s, t0, t1;
    if (!find_chunk(sh.cu_q, sh.n_seqs, chunk, s, t0, t1)) return;
    const int n = t1 - t0, cols = min(sh.V - v0, kCols);
    const int NT = sh.Vp >> 3, nt0 = v0 >> 3, tiles = min(NT - nt0, kCols / 8);
    const size_t qk_at = (size_t)t0 * in.tok + (size_t)(h0 / in.share) * sh.D;
    stage_rows(in.q + qk_at, in.tok, n, sh.D, sh.Dp, qs, ldk);
    stage_rows(in.k + qk_at, in.tok, n, sh.D, sh.Dp, ks, ldk);
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, tq = lane & 3;
    const bool active = warp * 16 < n;
    const int i0 = warp * 16 + g, i1 = i0 + 8;
    const bf16* q_at = qs + (warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ldk + (lane >> 4) * 8;
    float sc[kChunk / 8][4];
#pragma unroll
    for (int i = 0; i < kChunk / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.0f;
    if (active) {
        for (int kk = 0; kk < sh.Dp / 16; ++kk) {
            uint32_t qa[4];
            ldmatrix_x4(qa, smem_u32(q_at + kk * 16));
#pragma unroll
            for (int nn = 0; nn < kChunk / 16; ++nn) {
                if (nn <= warp) {                         // keys behind the warp's last token are not seen
                    uint32_t kb[4];
                    ldmatrix_x4(kb, smem_u32(ks + (nn * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + kk * 16 + ((lane >> 3) & 1) * 8));
                    mma_bf16(sc[2 * nn], qa, kb[0], kb[1]);
                    mma_bf16(sc[2 * nn + 1], qa, kb[2], kb[3]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < kChunk / 8; ++i) { sc[i][0] *= sh.q_scale; sc[i][1] *= sh.q_scale; sc[i][2] *= sh.q_scale; sc[i][3] *= sh.q_scale; }
    }
    for (int h = h0; h < h0 + sh.heads; ++h) {
        if (h > h0) __syncthreads();                      // the head before has been read
        if (warp == 0) chunk_decays<false>(ld, wt, sh.H, h, t0, n, cum, weight);
        stage_rows(in.v + (size_t)t0 * in.tok + (size_t)h * sh.V + v0, in.tok, n, cols, kCols, vs, ldv);
        const float* Sc = S_in + ((size_t)chunk * sh.H + h) * sh.per;
        float acc[kCols / 8][4];
#pragma unroll
        for (int i = 0; i < kCols / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.0f;
        if (active) {
            // the entering state comes from memory in the operand's order: 16 bytes a lane and tile, high and low halves in a word
            const uint4* Sw = reinterpret_cast<const uint4*>(Sc) + (size_t)nt0 * 32 + lane;
            for (int kk = 0; kk < sh.Dp / 16; ++kk) {
                uint4 b[kCols / 8];
#pragma unroll
                for (int i = 0; i < kCols / 8; ++i) b[i] = i < tiles ? Sw[((size_t)kk * NT + i) * 32] : make_uint4(0, 0, 0, 0);
                uint32_t qa[4];
                ldmatrix_x4(qa, smem_u32(q_at + kk * 16));
#pragma unroll
                for (int i = 0; i < kCols / 8; ++i)
                    if (i < tiles) mma_bf16(acc[i], qa, __byte_perm(b[i].x, b[i].y, 0x7632), __byte_perm(b[i].z, b[i].w, 0x7632));
#pragma unroll
                for (int i = 0; i < kCols / 8; ++i)
                    if (i < tiles) mma_bf16(acc[i], qa, __byte_perm(b[i].x, b[i].y, 0x5410), __byte_perm(b[i].z, b[i].w, 0x5410));
            }
        }
        __syncthreads();                                  // the head's decays and values are in shared memory
        if (!active) continue;
        const float cum0 = cum[i0], cum1 = cum[i1];
        const float carry0 = expf(cum0) * sh.q_scale, carry1 = expf(cum1) * sh.q_scale;
#pragma unroll
        for (int i = 0; i < kCols / 8; ++i) { acc[i][0] *= carry0; acc[i][1] *= carry0; acc[i][2] *= carry1; acc[i][3] *= carry1; }
        float size[2] = {0.0f, 0.0f};
#pragma unroll
        for (int nn = 0; nn < kChunk / 16; ++nn) {
            if (nn > warp) continue;
            float p[2][4];
#pragma unroll
            for (int x = 0; x < 2; ++x)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int j = nn * 16 + x * 8 + 2 * tq + (e & 1), i = (e >> 1) ? i1 : i0;
                    const float d = (e >> 1) ? cum1 - cum[j] : cum0 - cum[j];
                    p[x][e] = (nn < warp || j <= i) ? sc[2 * nn + x][e] * (__expf(d) * weight[j]) : 0.0f;
                    size[e >> 1] += p[x][e];
                }
            uint32_t ph[4], pl[4];
            split_bf16(p[0][0], p[0][1], ph[0], pl[0]);
            split_bf16(p[0][2], p[0][3], ph[1], pl[1]);
            split_bf16(p[1][0], p[1][1], ph[2], pl[2]);
            split_bf16(p[1][2], p[1][3], ph[3], pl[3]);
            const int vr = nn * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int i = 0; i < kCols / 16; ++i) {
                if (2 * i < tiles) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, smem_u32(vs + vr * ldv + i * 16 + (lane >> 4) * 8));
                    mma_bf16(acc[2 * i], ph, b[0], b[1]);
                    mma_bf16(acc[2 * i + 1], ph, b[2], b[3]);
                    mma_bf16(acc[2 * i], pl, b[0], b[1]);
                    mma_bf16(acc[2 * i + 1], pl, b[2], b[3]);
                }
            }
        }
        if (sh.normaliser && v0 == 0) {
            const float* n_in = Sc + (size_t)sh.Dp * sh.Vp;
            float part[2] = {0.0f, 0.0f};
            for (int d = tq; d < sh.D; d += 4) {
                const float x = n_in[d];
                part[0] = fmaf(__bfloat162float(qs[i0 * ldk + d]), x, part[0]);
                part[1] = fmaf(__bfloat162float(qs[i1 * ldk + d]), x, part[1]);
            }
            size[0] = fmaf(carry0, part[0], size[0]);
            size[1] = fmaf(carry1, part[1], size[1]);
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                size[r] += __shfl_xor_sync(0xffffffffu, size[r], 1);
                size[r] += __shfl_xor_sync(0xffffffffu, size[r], 2);
            }
            if (tq == 0) {
                if (i0 < n) den[(size_t)(t0 + i0) * sh.H + h] = size[0];
                if (i1 < n) den[(size_t)(t0 + i1) * sh.H + h] = size[1];
            }
        }
        const float skip = d_skip ? d_skip[h] : 0.0f;
        const bool pairs = (sh.V & 1) == 0, full = n == kChunk && cols == kCols && pairs;
        float* first = out + ((size_t)(t0 + i0) * sh.H + h) * sh.V + v0 + 2 * tq;
        const size_t eight_rows = (size_t)8 * sh.H * sh.V;
#pragma unroll
        for (int i = 0; i < kCols / 8; ++i) {
            const int v = i * 8 + 2 * tq;
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int row = r ? i1 : i0;
                if (!full && (row >= n || v >= cols)) continue;
                float x0 = acc[i][2 * r], x1 = acc[i][2 * r + 1];
                if (d_skip != nullptr) {
                    x0 = fmaf(skip, __bfloat162float(vs[row * ldv + v]), x0);
                    x1 = fmaf(skip, __bfloat162float(vs[row * ldv + v + 1]), x1);
                }
                float* at = first + r * eight_rows + i * 8;
                if (pairs) *reinterpret_cast<float2*>(at) = make_float2(x0, x1);
                else {
                    at[0] = x0;
                    if (v + 1 < cols) at[1] = x1;
                }
            }
        }
    }
}

// ------------------------------------------------------------------------------------------------ behind the raw rows
struct NormArgs {
    const float* raw;                    // [N, width]
    const float* gate;                   // rows of gate_stride floats
    long gate_stride;
    const float* weight;                 // [width]
    int width, parts, per_part;
    float eps;
    const float *den, *floor;            // [N, parts] or null: a part is divided by max(|den|, floor) + denom_eps first
    float denom_eps;
    int gate_first;                      // 1: silu gate, norm, weight; 0: norm, weight, sigmoid gate
    // the convolution's tails (conv.channels 0: none): moved on by the blocks behind the n rows' ones
    const float* rows;
    long stride;
    Conv conv;
    Step st;
    int row_blocks, tail_blocks;
};

// The tail of a sequence moves on: its entry k becomes the input at index q_len - (T-1) + k of this portion, or, where the portion is
// shorter than the tail, the old entry k + q_len (read before anything at or above it is written).
__device__ __forceinline__ void move_tail(const NormArgs& a, int b) {
    const int s = b / a.tail_blocks, c = (b - s * a.tail_blocks) * blockDim.x + threadIdx.x;
    if (c >= a.conv.channels) return;
    const int q0 = a.st.cu_q[s], q_len = a.st.cu_q[s + 1] - q0, keep = a.conv.n_taps - 1;
    float* tail = a.st.state + (size_t)a.st.state_slots[s] * a.st.state_stride + a.conv.tail_off + (size_t)c * keep;
    for (int k = 0; k < keep; ++k) {
        const int j = q_len - keep + k;
        tail[k] = j >= 0 ? a.rows[(size_t)(q0 + j) * a.stride + a.conv.off + c] : tail[k + q_len];
    }
}

// One (token, part) per group of `lanes` threads (a power of two from 32 to 256), ITEMS quads of neighbouring elements a thread.
template <typename T, int ITEMS>
__global__ void __launch_bounds__(256) gated_norm_quads_kernel(const NormArgs a, T* __restrict__ out, int lanes) {
    pdl_wait();
    if ((int)blockIdx.x >= a.row_blocks) { move_tail(a, blockIdx.x - a.row_blocks); return; }
    __shared__ float sums[8];
    const int groups = blockDim.x / lanes, group = threadIdx.x / lanes, l = threadIdx.x - group * lanes;
    const long unit = (long)blockIdx.x * groups + group;
    const bool live = unit < (long)a.st.n * a.parts;
    const int t = live ? (int)(unit / a.parts) : 0, p = live ? (int)(unit - (long)t * a.parts) : 0;
    const float* src = a.raw + (size_t)t * a.width + (size_t)p * a.per_part;
    const float* gate = a.gate + (size_t)t * a.gate_stride + (size_t)p * a.per_part;
    const float scale = (live && a.den != nullptr) ? 1.0f / (fmaxf(fabsf(a.den[unit]), a.floor[unit]) + a.denom_eps) : 1.0f;
    float x[ITEMS][4], gv[ITEMS][4];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = (l + k * lanes) * 4;
        if (live && i < a.per_part) {
            load_quad(src + i, x[k]);
            load_quad(gate + i, gv[k]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                x[k][e] = a.gate_first ? x[k][e] * silu_f(gv[k][e]) : x[k][e] * scale;
                ss = fmaf(x[k][e], x[k][e], ss);
            }
        }
    }
    ss = warp_sum(ss);
    if (lanes > 32) {                                     // uniform over the block
        if ((threadIdx.x & 31) == 0) sums[threadIdx.x >> 5] = ss;
        __syncthreads();
        const int w0 = group * (lanes >> 5);
        ss = 0.0f;
        for (int w = 0; w < lanes >> 5; ++w) ss += sums[w0 + w];
    }
    if (!live) return;
    const float inv = rsqrtf(ss / (float)a.per_part + a.eps);
    T* dst = out + (size_t)t * a.width + (size_t)p * a.per_part;
    const float* weight = a.weight + (size_t)p * a.per_part;
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
        const int i = (l + k * lanes) * 4;
        if (i < a.per_part) {
            float w[4], y[4];
            load_quad(weight + i, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                y[e] = x[k][e] * inv * w[e];
                if (!a.gate_first) y[e] *= sigmoid_f(gv[k][e]);
            }
            store_quad(dst + i, y);
        }
    }
}

// The same for any size: a block per (token, part), two passes over the part.
template <typename T>
__global__ void __launch_bounds__(128) gated_norm_kernel(const NormArgs a, T* __restrict__ out) {
    pdl_wait();
    if ((int)blockIdx.x >= a.row_blocks) { move_tail(a, blockIdx.x - a.row_blocks); return; }
    __shared__ float scratch[32];
    const int t = blockIdx.x / a.parts, p = blockIdx.x - t * a.parts;
    const float* src = a.raw + (size_t)t * a.width + (size_t)p * a.per_part;
    const float* gate = a.gate + (size_t)t * a.gate_stride + (size_t)p * a.per_part;
    const float scale = a.den != nullptr ? 1.0f / (fmaxf(fabsf(a.den[blockIdx.x]), a.floor[blockIdx.x]) + a.denom_eps) : 1.0f;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < a.per_part; i += blockDim.x) {
        const float v = a.gate_first ? src[i] * silu_f(gate[i]) : src[i] * scale;
        ss = fmaf(v, v, ss);
    }
    const float inv = rsqrtf(block_sum(ss, scratch) / (float)a.per_part + a.eps);
    for (int i = threadIdx.x; i < a.per_part; i += blockDim.x) {
        const float v = a.gate_first ? src[i] * silu_f(gate[i]) : src[i] * scale;
        const float y = v * inv * a.weight[(size_t)p * a.per_part + i];
        out[(size_t)t * a.width + (size_t)p * a.per_part + i] = from_float<T>(a.gate_first ? y : y * sigmoid_f(gate[i]));
    }
}

// ------------------------------------------------------------------------------------------------ host side
template <typename K>
int allow_smem(K kernel, size_t smem) {
    if (smem <= 48 * 1024) return 0;
    if (smem > 200 * 1024) return PB_ERR_TOO_LARGE;
    return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

int launch_norm(int dtype, NormArgs a, void* y, cudaStream_t stream) {
    a.per_part = a.width / a.parts;
    const bool aligned = (((uintptr_t)a.raw | (uintptr_t)a.gate | (uintptr_t)a.weight | (uintptr_t)y) & 15) == 0;
    const bool quads = a.per_part % 4 == 0 && a.gate_stride % 4 == 0 && aligned && a.per_part <= 8192;
    const int threads = quads ? 256 : 128;
    a.tail_blocks = a.conv.channels > 0 && a.conv.n_taps > 1 ? (a.conv.channels + threads - 1) / threads : 0;
    const long units = (long)a.st.n * a.parts;
    if (quads) {
        int lanes = 32;
        while (lanes < 256 && lanes * 4 < a.per_part) lanes <<= 1;
        const int items = (a.per_part / 4 + lanes - 1) / lanes;
        const long blocks = (units + 256 / lanes - 1) / (256 / lanes);
        if (blocks > 0x7fffff00L) return PB_ERR_TOO_LARGE;
        a.row_blocks = (int)blocks;
        const dim3 grid((unsigned)(blocks + (long)a.tail_blocks * a.st.n_seqs));
#define PB_NORM(T, I) return launch_pdl(gated_norm_quads_kernel<T, I>, grid, dim3(256), 0, stream, a, (T*)y, lanes)
#define PB_NORM_T(T)                \
    do {                            \
        if (items <= 1) PB_NORM(T, 1); \
        if (items <= 2) PB_NORM(T, 2); \
        if (items <= 4) PB_NORM(T, 4); \
        PB_NORM(T, 8);              \
    } while (0)
        if (dtype == PB_F32) PB_NORM_T(float);
        PB_NORM_T(__nv_bfloat16);
#undef PB_NORM_T
#undef PB_NORM
    }
    if (units > 0x7fffff00L) return PB_ERR_TOO_LARGE;
    a.row_blocks = (int)units;
    const dim3 grid((unsigned)(units + (long)a.tail_blocks * a.st.n_seqs));
    if (dtype == PB_F32) return launch_pdl(gated_norm_kernel<float>, grid, dim3(128), 0, stream, a, (float*)y);
    return launch_pdl(gated_norm_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, a, (__nv_bfloat16*)y);
}

// The least rows per thread with which a block of `tile` columns holds D rows: 8, 16 or 32 with up to 544 threads, 64 with up to
// 288 (a block's registers are 64 K); 0: none.
int step_rows(int D, int tile) {
    for (int per = 8; per <= 32; per <<= 1)
        if (tile * ((D + per - 1) / per) <= 544) return per;
    return tile * ((D + 63) / 64) <= 288 ? 64 : 0;
}

// The widest tile of columns that step_rows takes, at most `most`; 0: none.
int step_tile(int D, int cols, int most) {
    int tile = cols < most ? cols : most;
    while (tile > 0 && step_rows(D, tile) == 0) tile = tile > 8 ? tile / 2 : 0;
    return tile;
}

template <typename T, int MODE>
int launch_step(StepArgs a, void* y, int tile, cudaStream_t stream) {
    const int per = step_rows(a.D, tile);
    if (per == 0) return PB_ERR_TOO_LARGE;
    a.tile = tile;
    a.slices = (a.D + per - 1) / per;
    const dim3 grid(a.H, a.st.n_seqs, (a.cols + tile - 1) / tile);
    const dim3 block((tile * a.slices + 31) / 32 * 32);
    const size_t smem = sizeof(float) * ((size_t)a.slices * tile + 32 + 2 * (2 * (size_t)a.slices * per + ((tile + 3) & ~3) + 4));
#define PB_STEP(PER, THREADS)                                                                  \
    do {                                                                                       \
        const int rc = allow_smem(recurrence_step_kernel<T, PER, THREADS, MODE>, smem);         \
        if (rc != 0) return rc;                                                                \
        return launch_pdl(recurrence_step_kernel<T, PER, THREADS, MODE>, grid, block, smem, stream, a, (T*)y); \
    } while (0)
    if (per == 8) PB_STEP(8, 544);
    if (per == 16) PB_STEP(16, 544);
    if (per == 32) PB_STEP(32, 544);
    PB_STEP(64, 288);
#undef PB_STEP
}

size_t smem_state(int D) {
    const size_t Dp = (D + 15) & ~15;
    return 2 * ((size_t)kChunk * (Dp + kPad) + (size_t)2 * kChunk * (kCols + kPad));
}
size_t smem_out(int D) {
    const size_t Dp = (D + 15) & ~15;
    return 2 * ((size_t)2 * kChunk * (Dp + kPad) + (size_t)kChunk * (kCols + kPad));
}
bool chunks_fit(int D) { return smem_out(D) <= 200 * 1024 && smem_state(D) <= 200 * 1024; }

long chunk_words(int D, int V, int normaliser) {
    return ((long)((D + 15) & ~15) * ((V + 7) & ~7) + (normaliser ? D : 0) + 3) / 4 * 4;
}

template <typename T>
int launch_chunks(const Source<T>& in, const float* ld, const float* wt, ChunkShape sh, const Step& st, float* U, float* total,
                  int max_chunks, const float* d_skip, float* raw, float* den, cudaStream_t stream) {
    const int tiles = (sh.V + kCols - 1) / kCols;
    if (tiles > 65535 || sh.H > 65535 || st.n_seqs > 65535) return PB_ERR_TOO_LARGE;
    sh.Dp = (sh.D + 15) & ~15;
    sh.Vp = (sh.V + 7) & ~7;
    sh.per = chunk_words(sh.D, sh.V, sh.normaliser);
    // neighbouring heads that read the same q and k share a block (their keys are staged and their scores computed once), as long
    // as there are blocks for every SM
    sh.heads = 1;
    while (sh.heads < 4 && in.share % (2 * sh.heads) == 0 && (long)max_chunks * tiles * sh.H / (2 * sh.heads) >= 2 * 148) sh.heads *= 2;
    int rc = allow_smem(recurrence_chunk_state_kernel<T>, smem_state(sh.D));
    if (rc == 0) rc = allow_smem(recurrence_chunk_out_kernel<T>, smem_out(sh.D));
    if (rc != 0) return rc;
    const dim3 grid(max_chunks, sh.H / sh.heads, tiles);
    rc = launch_pdl(recurrence_chunk_state_kernel<T>, grid, dim3(128), smem_state(sh.D), stream, in, ld, wt, sh, U, total);
    if (rc != 0) return rc;
    const int own = sh.Dp * sh.Vp + (sh.normaliser ? sh.D : 0);
    rc = launch_pdl(recurrence_fold_kernel, dim3((own + 255) / 256, sh.H, st.n_seqs), dim3(256), 0, stream, U, (const float*)total, st, sh);
    if (rc != 0) return rc;
    return launch_pdl(recurrence_chunk_out_kernel<T>, grid, dim3(128), smem_out(sh.D), stream, in, ld, wt, sh, (const float*)U, d_skip, raw, den);
}

}  // namespace

PB_EXPORT int pb_recurrence_chunk() { return kChunk; }

// Whether the forms take these sizes: bit 0 the token-by-token form, bit 1 the form in chunks, bit 2 (the matrix memory) one block
// that does everything for a head.
PB_EXPORT int pb_recurrence_supported(int D, int V) {
    if (D <= 0 || V <= 0) return 0;
    return (step_tile(D, V + 1, 128) > 0 ? 1 : 0) | (chunks_fit(D) ? 2 : 0) | (step_rows(D, V + 1) > 0 ? 4 : 0);
}

// Floats of workspace: per token and head the log decays, weights, floors and denominators [4, n, H], the raw rows [n, H, V], the
// chunks' totals [max_chunks, H] and their states.
PB_EXPORT long pb_recurrence_workspace(int n, int H, int D, int V, int max_chunks, int normaliser) {
    const long raw = ((long)n * H * V + 3) / 4 * 4, scalars = ((long)4 * n * H + 3) / 4 * 4, totals = ((long)max_chunks * H + 3) / 4 * 4;
    return raw + scalars + totals + (long)max_chunks * H * chunk_words(D, V, normaliser);
}

// rows float32 [n, stride]: q (H*D) | k (H*D) | v (H*V) | g (H*V) | i (H) | f (H); biases float32 [H]; norm_w float32 [H*V]; state:
// float32 rows of state_stride elements per slot, the first H*D*V + H*D + H are this mixer's S [H, D, V], n [H, D], m [H];
// y [n, H*V] in `dtype`.  max_chunks > 0: the form in chunks (bfloat16 y), max_chunks >= the sum over the step's sequences of
// ceil(q_len / pb_recurrence_chunk()).  work: pb_recurrence_workspace floats (unused where one block does a head).
PB_EXPORT int pb_matrix_memory(int dtype, const float* rows, long stride, const float* i_bias, const float* f_bias, float cap,
                               const float* norm_w, float eps, float q_scale, float denom_eps, float* state, long state_stride,
                               const int* cu_q, const int* state_slots, void* y, int n, int n_seqs, int H, int D, int V, int whole,
                               int max_chunks, float* work, cudaStream_t stream) {
    if (n <= 0 || n_seqs <= 0) return 0;
    const long HDV = (long)H * D * V;
    if (H <= 0 || D <= 0 || V <= 0 || !(cap > 0.0f) || stride < (long)2 * H * (D + V) + 2 * H || state_stride < HDV + (long)H * D + H)
        return PB_ERR_BAD_SIZE;
    if (dtype != PB_F32 && dtype != PB_BF16) return PB_ERR_BAD_DTYPE;
    if (n_seqs > 65535 || HDV > 0x7fffffffL) return PB_ERR_TOO_LARGE;
    const Step st{cu_q, state_slots, state, state_stride, n, n_seqs};
    StepArgs a{};
    a.st = st;
    a.rows = rows;
    a.stride = stride;
    a.H = H; a.D = D; a.V = V;
    a.cols = V + 1;
    a.q_off = 0; a.k_off = H * D; a.v_off = 2 * H * D; a.g_off = 2 * H * D + H * V;
    a.i_off = a.g_off + H * V; a.f_off = a.i_off + H;
    a.share = 1;
    a.q_scale = q_scale;
    a.i_bias = i_bias; a.f_bias = f_bias; a.norm_w = norm_w;
    a.cap = cap; a.denom_eps = denom_eps; a.eps = eps;
    if (max_chunks <= 0 && whole) {
        if (step_rows(D, V + 1) == 0) return PB_ERR_TOO_LARGE;
        if (dtype == PB_F32) return launch_step<float, kMemoryWhole>(a, y, V + 1, stream);
        return launch_step<__nv_bfloat16, kMemoryWhole>(a, y, V + 1, stream);
    }
    if (work == nullptr) return PB_ERR_BAD_SIZE;
    float* raw = work;
    float* ld = raw + ((long)n * H * V + 3) / 4 * 4;
    float *wt = ld + (long)n * H, *floor = wt + (long)n * H, *den = floor + (long)n * H;
    float* total = ld + ((long)4 * n * H + 3) / 4 * 4;
    float* U = total + ((long)(max_chunks > 0 ? max_chunks : 0) * H + 3) / 4 * 4;
    const int threads = n >= 512 * n_seqs ? 1024 : n >= 128 * n_seqs ? 512 : 128;
    int rc = launch_pdl(memory_gates_kernel, dim3(H, n_seqs), dim3(threads), 0, stream, rows, stride, a.i_off, a.f_off, i_bias, f_bias, cap, st,
                        HDV + (long)H * D, H, ld, wt, floor);
    if (rc != 0) return rc;
    if (max_chunks > 0) {
        if (dtype != PB_BF16 || !chunks_fit(D)) return PB_ERR_TOO_LARGE;
        const Source<float> in{rows, rows + a.k_off, rows + a.v_off, stride, 1};
        const ChunkShape sh{cu_q, n_seqs, H, D, V, 1, 0, 0, 0, q_scale, 1};
        rc = launch_chunks<float>(in, ld, wt, sh, st, U, total, max_chunks, nullptr, raw, den, stream);
    } else {
        const int tile = step_tile(D, V + 1, 128);
        if (tile == 0) return PB_ERR_TOO_LARGE;
        a.ld = ld; a.wt = wt; a.den = den; a.raw = raw;
        rc = launch_step<float, kGiven>(a, nullptr, tile, stream);
    }
    if (rc != 0) return rc;
    NormArgs na{};
    na.raw = raw;
    na.gate = rows + a.g_off;
    na.gate_stride = stride;
    na.weight = norm_w;
    na.width = H * V;
    na.parts = H;
    na.eps = eps;
    na.den = den; na.floor = floor; na.denom_eps = denom_eps;
    na.st = st;
    return launch_norm(dtype, na, y, stream);
}

// rows float32 [n, stride]: z (H*V) | x (H*V) | B (G*D) | C (G*D) | dt (H); taps float32 [H*V + 2 G*D, n_taps], conv_bias likewise; dt_bias,
// a_log, d_skip float32 [H]; norm_w float32 [H*V]; state: rows of state_stride floats per slot, the first H*D*V + (H*V + 2 G*D) *
// (n_taps - 1) are this mixer's S [H, D, V] and convolution tail; y [n, H*V] in `dtype`.  xbc: the convolution's output
// [n, H*V + 2 G*D] in `dtype` (pb_causal_conv_silu) for the form in chunks (max_chunks > 0; bfloat16), else unused: the token-by-token
// form does the convolution itself.  work: pb_recurrence_workspace floats.
PB_EXPORT int pb_state_space(int dtype, const float* rows, long stride, const float* taps, const float* conv_bias, int n_taps,
                             const float* dt_bias, const float* a_log, const float* d_skip, const float* norm_w, int norm_parts, float eps,
                             float* state, long state_stride, const int* cu_q, const int* state_slots, const void* xbc, void* y, int n,
                             int n_seqs, int H, int D, int V, int G, int max_chunks, float* work, cudaStream_t stream) {
    if (n <= 0 || n_seqs <= 0) return 0;
    const long HDV = (long)H * D * V;
    const int inner = H * V, channels = inner + 2 * G * D;
    if (H <= 0 || D <= 0 || V <= 0 || G <= 0 || H % G || n_taps < 1 || norm_parts <= 0 || inner % norm_parts ||
        stride < (long)inner + channels + H || state_stride < HDV + (long)channels * (n_taps - 1) || work == nullptr)
        return PB_ERR_BAD_SIZE;
    if (dtype != PB_F32 && dtype != PB_BF16) return PB_ERR_BAD_DTYPE;
    if (n_seqs > 65535 || HDV > 0x7fffffffL) return PB_ERR_TOO_LARGE;
    const Step st{cu_q, state_slots, state, state_stride, n, n_seqs};
    const Conv conv{taps, conv_bias, inner, channels, n_taps, HDV};
    float* raw = work;
    float* ld = raw + ((long)n * H * V + 3) / 4 * 4;
    float* wt = ld + (long)n * H;
    float* total = ld + ((long)4 * n * H + 3) / 4 * 4;
    float* U = total + ((long)(max_chunks > 0 ? max_chunks : 0) * H + 3) / 4 * 4;
    int rc;
    if (max_chunks > 0) {
        if (dtype != PB_BF16 || !chunks_fit(D)) return PB_ERR_TOO_LARGE;
        if (xbc == nullptr || (long)n * H > 0x7fffffffL) return PB_ERR_BAD_SIZE;
        const int entries = n * H;
        rc = launch_pdl(space_gates_kernel, dim3((entries + 255) / 256), dim3(256), 0, stream, rows, stride, inner + channels, dt_bias, a_log, H,
                        entries, ld, wt);
        if (rc != 0) return rc;
        const bf16* x = (const bf16*)xbc;
        const Source<bf16> in{x + inner + G * D, x + inner, x, channels, H / G};
        const ChunkShape sh{cu_q, n_seqs, H, D, V, 0, 0, 0, 0, 1.0f, 1};
        rc = launch_chunks<bf16>(in, ld, wt, sh, st, U, total, max_chunks, d_skip, raw, nullptr, stream);
    } else {
        StepArgs a{};
        a.st = st;
        a.rows = rows;
        a.stride = stride;
        a.H = H; a.D = D; a.V = V;
        a.cols = V;
        a.v_off = 0; a.k_off = inner; a.q_off = inner + G * D;
        a.share = H / G;
        a.q_scale = 1.0f;
        a.conv = conv;
        a.dt_off = inner + channels;
        a.dt_bias = dt_bias; a.a_log = a_log; a.d_skip = d_skip;
        a.raw = raw;
        const int tile = step_tile(D, V, 128);
        if (tile == 0) return PB_ERR_TOO_LARGE;
        rc = launch_step<float, kStateSpace>(a, nullptr, tile, stream);
    }
    if (rc != 0) return rc;
    NormArgs na{};
    na.raw = raw;
    na.gate = rows;
    na.gate_stride = stride;
    na.weight = norm_w;
    na.width = inner;
    na.parts = norm_parts;
    na.eps = eps;
    na.gate_first = 1;
    na.rows = rows;
    na.stride = stride;
    na.conv = conv;
    na.st = st;
    return launch_norm(dtype, na, y, stream);
}
