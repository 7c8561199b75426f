// RMSNorm over the last dimension, fused with the residual add that precedes it.
//
//   v   = x[row] (+ delta[row])                      32-bit sum: the residual stream is float32
//   out = v * rsqrt(mean(v^2) + eps) * w             sum of squares, rsqrt and products in 32-bit
//
// One block per output row.  `rows` (optional) picks which rows of x/delta are read, so the
// final norm can run only at the positions whose logits are wanted.  With `write_sum` the sum
// v is written back into x (the layer's residual update), which needs rows == nullptr.
// Formula and product order (x*inv)*w: src/layers/rms_norm.cu:77-93; the reference runs the
// add as its own kernel (src/ops/add.cu:16-27).
#include "common.cuh"

template <typename TX, typename TD, typename TO>
__global__ void rmsnorm_kernel(TX* __restrict__ x, const TD* __restrict__ delta,
                               const float* __restrict__ w, TO* __restrict__ out,
                               const int32_t* __restrict__ rows, int hidden, float eps,
                               int write_sum, int vec, int delta_parts, long long delta_part_stride) {
    // The norm weights are read before the wait for the kernel that produces x / delta.
    float g0[8];
    const bool one_trip = vec && hidden <= static_cast<int>(blockDim.x) * 8;
    if (one_trip && static_cast<int>(threadIdx.x) * 8 < hidden) load8(w + threadIdx.x * 8, g0);
    pdl_begin();
    extern __shared__ __align__(16) float smem[];   // hidden floats (padded to 8) + 33 for the reduction
    float* v = smem;
    float* scratch = smem + ((hidden + 7) & ~7);
    const size_t src = rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
    TX* xr = x + src * hidden;
    const TD* dr = delta ? delta + src * hidden : nullptr;
    TO* orow = out + static_cast<size_t>(blockIdx.x) * hidden;
    float ss = 0.0f;
    if (vec) {                                      // 8 elements per thread per trip, 16-byte accesses
        for (int h = threadIdx.x * 8; h < hidden; h += blockDim.x * 8) {
            float a[8];
            load8(xr + h, a);
            if (dr) {
                for (int part = 0; part < delta_parts; ++part) {    // delta may come as the k-splits of a product
                    float b[8];
                    load8(dr + part * delta_part_stride + h, b);
#pragma unroll
                    for (int i = 0; i < 8; ++i) a[i] += b[i];
                }
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) ss += a[i] * a[i];
            store8(v + h, a);
            if (write_sum) store8(xr + h, a);
        }
    } else {
        for (int h = threadIdx.x; h < hidden; h += blockDim.x) {
            float a = to_f32(xr[h]);
            if (dr)
                for (int part = 0; part < delta_parts; ++part) a += to_f32(dr[part * delta_part_stride + h]);
            v[h] = a;
            ss += a * a;
            if (write_sum) xr[h] = from_f32<TX>(a);
        }
    }
    const float total = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(total / static_cast<float>(hidden) + eps);
    if (one_trip) {
        const int h = threadIdx.x * 8;
        if (h < hidden) {
            float a[8];
            load8(v + h, a);
#pragma unroll
            for (int i = 0; i < 8; ++i) a[i] = a[i] * inv * g0[i];
            store8(orow + h, a);
        }
    } else if (vec) {
        for (int h = threadIdx.x * 8; h < hidden; h += blockDim.x * 8) {
            float a[8], g[8];
            load8(v + h, a);
            load8(w + h, g);
#pragma unroll
            for (int i = 0; i < 8; ++i) a[i] = a[i] * inv * g[i];
            store8(orow + h, a);
        }
    } else {
        for (int h = threadIdx.x; h < hidden; h += blockDim.x) orow[h] = from_f32<TO>(v[h] * inv * w[h]);
    }
}

template <typename TX, typename TD, typename TO>
static int launch_rmsnorm(void* x, const void* delta, const float* w, void* out, const int32_t* rows,
                          int num_rows, int hidden, float eps, int write_sum, int delta_parts,
                          long long delta_part_stride, cudaStream_t s) {
    const size_t smem = (static_cast<size_t>((hidden + 7) & ~7) + 33) * sizeof(float);
    const int vec = (hidden % 8 == 0) && aligned16(x) && aligned16(out) && aligned16(w) && (!delta || aligned16(delta));
    if (smem > 200 * 1024) return LLM_REFUSED_SIZE;
    auto kern = rmsnorm_kernel<TX, TD, TO>;
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                   static_cast<int>(smem));
        if (e != cudaSuccess) return static_cast<int>(e);
    }
    const int threads = hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128);
    launch_pdl(kern, dim3(num_rows), dim3(threads), smem, s, static_cast<TX*>(x), static_cast<const TD*>(delta), w,
                                         static_cast<TO*>(out), rows, hidden, eps, write_sum, vec, delta_parts, delta_part_stride);
    return launch_status();
}

// x: [*, hidden] (x_dtype), delta: same shape or null (delta_dtype), w: float32 [hidden],
// out: [num_rows, hidden] (out_dtype), rows: int32 [num_rows] or null.  delta may be given as
// delta_parts tensors of x's shape, delta_part_stride elements apart, that are added up on the fly.
extern "C" int llm_rmsnorm(void* x, int x_dtype, const void* delta, int delta_dtype, const float* w,
                           void* out, int out_dtype, const int32_t* rows, int num_rows, int hidden,
                           float eps, int write_sum, int delta_parts, long long delta_part_stride,
                           uintptr_t stream) {
    if (num_rows <= 0) return LLM_OK;
    if (hidden <= 0) return LLM_REFUSED_SIZE;
    if (write_sum && rows) return LLM_REFUSED_SIZE;
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    if (!delta) delta_dtype = x_dtype;
    const int key = x_dtype * 4 + delta_dtype * 2 + out_dtype;
#define CASE(k, TX, TD, TO)                                                                     \
    case k:                                                                                       \
        return launch_rmsnorm<TX, TD, TO>(x, delta, w, out, rows, num_rows, hidden, eps, write_sum,       \
                                          delta_parts < 1 ? 1 : delta_parts, delta_part_stride, s);
    switch (key) {
        CASE(0, float, float, float)
        CASE(1, float, float, bf16)
        CASE(2, float, bf16, float)
        CASE(3, float, bf16, bf16)
        CASE(4, bf16, float, float)
        CASE(5, bf16, float, bf16)
        CASE(6, bf16, bf16, float)
        CASE(7, bf16, bf16, bf16)
    }
#undef CASE
    return LLM_REFUSED_DTYPE;
}

// A norm on a sublayer's OUTPUT, fused with the residual add that follows it:
//     h[row] += y[row] * rsqrt(mean(y[row]^2) + eps) * w          (32-bit throughout; h is float32)
// and, optionally, `copy[row]` = the new h[row] in the compute dtype: what the next sublayer of a
// design reads whose sublayers take the stream itself (no norm in front of them).
// One block per row; y is float32 or bfloat16, `y_stride` elements from row to row.  y may come as the
// `parts` k-splits of a product, `part_stride` elements apart, which are added up in order as they are read.
template <typename TY, typename TC>
__global__ void rmsnorm_add_kernel(float* __restrict__ h, const TY* __restrict__ y, long long y_stride,
                                   const float* __restrict__ w, TC* __restrict__ copy, int hidden, float eps, int vec,
                                   int parts, long long part_stride) {
    pdl_begin();
    extern __shared__ __align__(16) float smem[];
    float* v = smem;
    float* scratch = smem + ((hidden + 7) & ~7);
    const TY* yr = y + static_cast<size_t>(blockIdx.x) * y_stride;
    float* hr = h + static_cast<size_t>(blockIdx.x) * hidden;
    TC* cr = copy ? copy + static_cast<size_t>(blockIdx.x) * hidden : nullptr;
    float ss = 0.0f;
    if (vec) {                                      // 8 elements per thread per trip, 16-byte accesses
        for (int i = threadIdx.x * 8; i < hidden; i += blockDim.x * 8) {
            float a[8];
            load8(yr + i, a);
            for (int part = 1; part < parts; ++part) {
                float b[8];
                load8(yr + part * part_stride + i, b);
#pragma unroll
                for (int u = 0; u < 8; ++u) a[u] += b[u];
            }
#pragma unroll
            for (int u = 0; u < 8; ++u) ss += a[u] * a[u];
            store8(v + i, a);
        }
    } else {
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            float a = to_f32(yr[i]);
            for (int part = 1; part < parts; ++part) a += to_f32(yr[part * part_stride + i]);
            v[i] = a;
            ss += a * a;
        }
    }
    const float total = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(total / static_cast<float>(hidden) + eps);
    if (vec) {
        for (int i = threadIdx.x * 8; i < hidden; i += blockDim.x * 8) {
            float a[8], b[8], g[8];
            load8(v + i, a);
            load8(hr + i, b);
            load8(w + i, g);
#pragma unroll
            for (int u = 0; u < 8; ++u) b[u] += a[u] * inv * g[u];
            store8(hr + i, b);
            if (cr) store8(cr + i, b);
        }
    } else {
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float a = hr[i] + v[i] * inv * w[i];
            hr[i] = a;
            if (cr) cr[i] = from_f32<TC>(a);
        }
    }
}

extern "C" int llm_rmsnorm_add(float* h, const void* y, int y_dtype, long long y_stride, const float* w, void* copy,
                               int copy_dtype, int num_rows, int hidden, float eps, int parts, long long part_stride,
                               uintptr_t stream) {
    if (num_rows <= 0) return LLM_OK;
    if (hidden <= 0 || y_stride < hidden || parts < 1) return LLM_REFUSED_SIZE;
    const size_t smem = (static_cast<size_t>((hidden + 7) & ~7) + 33) * sizeof(float);
    if (smem > 200 * 1024) return LLM_REFUSED_SIZE;
    const int threads = hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128);
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    if (!copy) copy_dtype = LLM_DT_F32;
    const int vec = (hidden % 8 == 0) && (y_stride % 8 == 0) && (part_stride % 8 == 0) && aligned16(h) && aligned16(y) &&
                    aligned16(w) && (!copy || aligned16(copy));
#define LAUNCH(TY, TC)                                                                                           \
    do {                                                                                                         \
        auto kern = rmsnorm_add_kernel<TY, TC>;                                                                  \
        if (smem > 48 * 1024) {                                                                                  \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,        \
                                                       static_cast<int>(smem));                                  \
            if (e != cudaSuccess) return static_cast<int>(e);                                                    \
        }                                                                                                        \
        launch_pdl(kern, dim3(num_rows), dim3(threads), smem, s, h, static_cast<const TY*>(y), y_stride, w,      \
                   static_cast<TC*>(copy), hidden, eps, vec, parts, part_stride);                                \
    } while (0)
    if (y_dtype == LLM_DT_F32 && copy_dtype == LLM_DT_F32) LAUNCH(float, float);
    else if (y_dtype == LLM_DT_F32 && copy_dtype == LLM_DT_BF16) LAUNCH(float, bf16);
    else if (y_dtype == LLM_DT_BF16 && copy_dtype == LLM_DT_F32) LAUNCH(bf16, float);
    else if (y_dtype == LLM_DT_BF16 && copy_dtype == LLM_DT_BF16) LAUNCH(bf16, bf16);
    else return LLM_REFUSED_DTYPE;
#undef LAUNCH
    return launch_status();
}

// block_sum with one barrier: every warp adds the warps' sums up itself.  `scratch` (32 floats) serves one call only.
__device__ __forceinline__ float block_sum_once(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    v = warp_sum(v);
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    return warp_sum(lane < static_cast<int>((blockDim.x + 31) >> 5) ? scratch[lane] : 0.0f);
}

// The step between two sublayers of a design that norms a sublayer's input AND its output, in 32-bit throughout:
//     v      = h[row] + n(y[row]) * w_post (+ join[row])        n(a) = a * rsqrt(mean(a^2) + eps)
//     h[row] = v                                                (with write_h; the stream is float32)
//     out    = n(v) * w_pre                                     stored in the compute dtype
// Without w_post, y joins as it is; y may be absent; y may come as the `parts` k-splits of a product, `part_stride`
// elements apart, added in order as they are read.  `join` (optional, float32 like h) is one more summand: what a
// design adds to the stream in front of a sublayer.  `w_post` carries whatever constant factors the sum has per
// channel.  `rows` (optional) picks which rows are read, so a model's final norm runs only where logits are wanted
// (h is then left alone).
// One block per row.  REG: the row fits the block with eight neighbouring elements a thread (blockDim * 8 >= hidden),
// which stay in registers between the two reductions, and everything the row needs is asked for before the first of
// them.  Otherwise the row passes through shared memory.
template <typename TY, typename TO, bool REG>
__global__ void __launch_bounds__(1024) rmsnorm_sandwich_kernel(float* __restrict__ h, const TY* __restrict__ y, long long y_stride, int parts,
                                        long long part_stride, const float* __restrict__ w_post, float eps_post,
                                        const float* __restrict__ join, const float* __restrict__ w_pre, float eps_pre,
                                        TO* __restrict__ out, const int32_t* __restrict__ rows, int hidden, int write_h) {
    __shared__ float scratch[2][32];
    if constexpr (REG) {
        const int i = threadIdx.x * 8;
        const bool mine = i < hidden;
        // the weights are the model's: on their way before the wait, but in no registers until they are used (more blocks
        // of a long step fit an SM)
        if (mine && w_post) asm volatile("prefetch.global.L1 [%0];\n" ::"l"(w_post + i));
        if (mine) asm volatile("prefetch.global.L1 [%0];\n" ::"l"(w_pre + i));
        pdl_begin();
        const size_t src = rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
        float* hr = h + src * hidden;
        float v[8] = {0, 0, 0, 0, 0, 0, 0, 0}, a[8] = {0, 0, 0, 0, 0, 0, 0, 0};
        if (mine) {
            load8(hr + i, v);
            if (join) {
                float b[8];
                load8(join + src * hidden + i, b);
#pragma unroll
                for (int u = 0; u < 8; ++u) v[u] += b[u];
            }
            if (y) {
                const TY* yr = y + src * y_stride + i;
                load8(yr, a);
#pragma unroll 4
                for (int part = 1; part < parts; ++part) {
                    float b[8];
                    load8(yr + part * part_stride, b);
#pragma unroll
                    for (int u = 0; u < 8; ++u) a[u] += b[u];
                }
            }
        }
        if (y) {
            float inv = 1.0f;
            if (w_post) {
                float ss = 0.0f;
#pragma unroll
                for (int u = 0; u < 8; ++u) ss += a[u] * a[u];
                inv = 1.0f / sqrtf(block_sum_once(ss, scratch[0]) / static_cast<float>(hidden) + eps_post);
            }
            float wp[8] = {1, 1, 1, 1, 1, 1, 1, 1};
            if (mine && w_post) load8(w_post + i, wp);
#pragma unroll
            for (int u = 0; u < 8; ++u) v[u] += a[u] * inv * wp[u];       // a thread without elements holds zeros
        }
        if (write_h && mine) store8(hr + i, v);
        float ss = 0.0f;
#pragma unroll
        for (int u = 0; u < 8; ++u) ss += v[u] * v[u];
        const float inv = 1.0f / sqrtf(block_sum_once(ss, scratch[1]) / static_cast<float>(hidden) + eps_pre);
        if (mine) {
            float wn[8];
            load8(w_pre + i, wn);
#pragma unroll
            for (int u = 0; u < 8; ++u) v[u] = v[u] * inv * wn[u];
            store8(out + static_cast<size_t>(blockIdx.x) * hidden + i, v);
        }
    } else {
        pdl_begin();
        extern __shared__ __align__(16) float row_s[];
        const size_t src = rows ? static_cast<size_t>(rows[blockIdx.x]) : blockIdx.x;
        float* hr = h + src * hidden;
        const float* jr = join ? join + src * hidden : nullptr;
        const TY* yr = y ? y + src * y_stride : nullptr;
        float inv = 1.0f;
        if (yr) {
            float ss = 0.0f;
            for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
                float a = to_f32(yr[i]);
                for (int part = 1; part < parts; ++part) a += to_f32(yr[part * part_stride + i]);
                row_s[i] = a;
                ss += a * a;
            }
            if (w_post) inv = 1.0f / sqrtf(block_sum_once(ss, scratch[0]) / static_cast<float>(hidden) + eps_post);
        }
        float ss = 0.0f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {       // each thread meets the elements it wrote itself
            float v = hr[i];
            if (jr) v += jr[i];
            if (yr) v += w_post ? row_s[i] * inv * w_post[i] : row_s[i];
            row_s[i] = v;
            if (write_h) hr[i] = v;
            ss += v * v;
        }
        inv = 1.0f / sqrtf(block_sum_once(ss, scratch[1]) / static_cast<float>(hidden) + eps_pre);
        TO* orow = out + static_cast<size_t>(blockIdx.x) * hidden;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) orow[i] = from_f32<TO>(row_s[i] * inv * w_pre[i]);
    }
}

// h: float32 [*, hidden]; y: [*, hidden] with `y_stride` elements a row, or null; w_post: float32 [hidden] or null; join:
// float32 like h, or null; w_pre: float32 [hidden]; out: [num_rows, hidden]; rows: int32 [num_rows] or null.
extern "C" int llm_rmsnorm_sandwich(float* h, const void* y, int y_dtype, long long y_stride, int parts, long long part_stride,
                                    const float* w_post, float eps_post, const float* join, const float* w_pre, float eps_pre,
                                    void* out, int out_dtype, const int32_t* rows, int num_rows, int hidden,
                                    uintptr_t stream) {
    if (num_rows <= 0) return LLM_OK;
    if (hidden <= 0 || parts < 1 || (y && y_stride < hidden) || !w_pre || !out) return LLM_REFUSED_SIZE;
    const size_t smem = static_cast<size_t>(hidden) * sizeof(float);
    if (smem > 200 * 1024) return LLM_REFUSED_SIZE;
    if (!y) y_dtype = LLM_DT_F32;
    const int write_h = (y || join) && !rows;
    const bool reg = hidden % 8 == 0 && hidden <= 8192 && aligned16(h) && aligned16(out) && aligned16(w_pre) &&
                     (!y || (aligned16(y) && y_stride % 8 == 0 && part_stride % 8 == 0)) && (!w_post || aligned16(w_post)) &&
                     (!join || aligned16(join));
    const int threads = reg ? (hidden / 8 + 31) / 32 * 32 : (hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128));
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define LAUNCH(TY, TO)                                                                                                   \
    do {                                                                                                                 \
        auto kern = reg ? rmsnorm_sandwich_kernel<TY, TO, true> : rmsnorm_sandwich_kernel<TY, TO, false>;                \
        if (!reg && smem > 48 * 1024) {                                                                                  \
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize,                \
                                                       static_cast<int>(smem));                                          \
            if (e != cudaSuccess) return static_cast<int>(e);                                                            \
        }                                                                                                                \
        launch_pdl(kern, dim3(num_rows), dim3(threads), reg ? 0 : smem, s, h, static_cast<const TY*>(y), y_stride, parts, \
                   part_stride, w_post, eps_post, join, w_pre, eps_pre, static_cast<TO*>(out), rows, hidden, write_h);   \
    } while (0)
    if (y_dtype == LLM_DT_F32 && out_dtype == LLM_DT_F32) LAUNCH(float, float);
    else if (y_dtype == LLM_DT_F32 && out_dtype == LLM_DT_BF16) LAUNCH(float, bf16);
    else if (y_dtype == LLM_DT_BF16 && out_dtype == LLM_DT_F32) LAUNCH(bf16, float);
    else if (y_dtype == LLM_DT_BF16 && out_dtype == LLM_DT_BF16) LAUNCH(bf16, bf16);
    else return LLM_REFUSED_DTYPE;
#undef LAUNCH
    return launch_status();
}
