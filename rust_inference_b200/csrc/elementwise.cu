// Row-wise kernels of the decoder step: embedding gather, RMSNorm, rotary position
// encoding fused with the cache write, and the standalone SiLU-gate.
//
// The residual stream is float32 in both precisions; `T` is the activation/storage
// type (float or bf16).  Statistics, rotation and SiLU are computed in float32.
#include "common.cuh"

using namespace ri;

// ----------------------------------------------------------------------------
// embedding: out[t, :] = table[ids[t], :] * scale        (transformer.rs:74-75; the factor is 1 there), `copies` times
// side by side (the parallel streams of a model that has several)
// ----------------------------------------------------------------------------
template <typename T>
__global__ void embed_gather_kernel(const T* __restrict__ table, const int* __restrict__ ids,
                                    float* __restrict__ out, int hidden, int copies, float scale) {
    const int t = blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();          // the ids may come from the previous step's sampler
    const int id = ids[t];
    float* o = out + (size_t)t * copies * hidden;
    if (!RI_BLOCK_IN_LIMIT(id, RI_LIMIT_VOCAB, RI_CHECK_TOKEN_ID)) {           // checked build: recorded, the row left zero
        for (int i = threadIdx.x; i < copies * hidden; i += blockDim.x) o[i] = 0.f;
        return;
    }
    const T* row = table + (size_t)id * hidden;
    if (sizeof(T) == 2 && (hidden & 7) == 0 && (reinterpret_cast<uintptr_t>(table) & 15) == 0 &&
        (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
        // 16 bytes (8 elements) per load, up to four loads of a thread on their way together: the row comes
        // from memory in one trip, not in one trip per element
        constexpr int AHEAD = 4;
        const uint4* src = reinterpret_cast<const uint4*>(row);
        const int n8 = hidden >> 3;
        for (int base = threadIdx.x; base < n8; base += AHEAD * blockDim.x) {
            uint4 v[AHEAD];
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int i = base + j * blockDim.x;
                if (i < n8) v[j] = src[i];
            }
#pragma unroll
            for (int j = 0; j < AHEAD; ++j) {
                const int i = base + j * blockDim.x;
                if (i < n8) {
                    const T* e = reinterpret_cast<const T*>(&v[j]);
                    const float4 lo = make_float4(to_f32<T>(e[0]) * scale, to_f32<T>(e[1]) * scale, to_f32<T>(e[2]) * scale, to_f32<T>(e[3]) * scale);
                    const float4 hi = make_float4(to_f32<T>(e[4]) * scale, to_f32<T>(e[5]) * scale, to_f32<T>(e[6]) * scale, to_f32<T>(e[7]) * scale);
                    for (int c = 0; c < copies; ++c) {
                        float4* dst = reinterpret_cast<float4*>(o + (size_t)c * hidden + 8 * (size_t)i);
                        dst[0] = lo;
                        dst[1] = hi;
                    }
                }
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = to_f32<T>(row[i]) * scale;
        for (int c = 0; c < copies; ++c) o[(size_t)c * hidden + i] = v;
    }
}

RI_API int ri_embed_gather(const void* table, int dtype, const int* ids, float* out, int n_tokens,
                           int hidden, int copies, float scale, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (copies < 1) return fail("embed_gather: %d copies", copies);
    cudaError_t e = cudaSuccess;
    if (dtype == RI_F32)
        e = launch_dependent(embed_gather_kernel<float>, n_tokens, 256, 0, stream, (const float*)table, ids, out, hidden, copies, scale);
    else if (dtype == RI_BF16)
        e = launch_dependent(embed_gather_kernel<__nv_bfloat16>, n_tokens, 256, 0, stream, (const __nv_bfloat16*)table, ids, out, hidden, copies, scale);
    else
        return fail("embed_gather: unknown dtype %d", dtype);
    return check_launch(e, "embed_gather");
}

// ----------------------------------------------------------------------------
// RMSNorm (math.rs:237-256): ss = sum x^2; rms = sqrt(ss/n + eps); y = x * (1/rms) * w.
// `rows` (may be null) picks the input row of each output row, so the final norm
// runs on the wanted positions only.
// ----------------------------------------------------------------------------
template <typename T>
__global__ void rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ w,
                               const int* __restrict__ rows, T* __restrict__ out, int n, float eps) {
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();          // x is the residual stream the previous kernel wrote
    const float* xr = x + (size_t)(rows ? rows[r] : r) * n;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        float v = xr[i];
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float rms = sqrtf(ss / (float)n + eps);
    const float scale = 1.0f / rms;
    T* o = out + (size_t)r * n;
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_f32<T>(xr[i] * scale * w[i]);
}

template <typename T> __device__ __forceinline__ void store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<uint32_t*>(&lo);
    v.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = v;
}

// The same in one pass for rows that are a multiple of 4 wide and at most 4 * PER * blockDim long:
// every thread keeps its float4s of the row in registers, so the row is read once, and the weights
// (which no kernel writes) are fetched before the wait for the previous kernel.
template <typename T, int PER>
__global__ void __launch_bounds__(1024)
rmsnorm_vec_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ rows,
                   T* __restrict__ out, int n, float eps) {
    __shared__ float scratch[33];
    const int r = blockIdx.x, n4 = n >> 2;
    float4 wv[PER], xv[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        wv[j] = i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int in_row = rows ? rows[r] : r;                // the wanted rows are fixed before the step's first kernel
    let_next_kernel_start();
    wait_for_previous_kernels();
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)in_row * n);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        xv[j] = i < n4 ? xr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += xv[j].x * xv[j].x + xv[j].y * xv[j].y + xv[j].z * xv[j].z + xv[j].w * xv[j].w;
    }
    ss = block_sum(ss, scratch);
    const float rms = sqrtf(ss / (float)n + eps);
    const float scale = 1.0f / rms;
    T* o = out + (size_t)r * n;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < n4)
            store4<T>(o + 4 * i, xv[j].x * scale * wv[j].x, xv[j].y * scale * wv[j].y, xv[j].z * scale * wv[j].z,
                      xv[j].w * scale * wv[j].w);
    }
    RI_PHASE_LATEST(5);
}

// Steps of many rows (prompts): one warp per row, the row in registers, no block-wide barrier; the
// weights are read again by every warp (they stay in L1/L2).  CH float4s per lane: rows of up to 512 * CH.
template <typename T, int CH>
__global__ void __launch_bounds__(256)
rmsnorm_warp_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ rows,
                    T* __restrict__ out, int n_rows, int n, float eps) {
    const int lane = threadIdx.x & 31, n4 = n >> 2;
    const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    let_next_kernel_start();
    wait_for_previous_kernels();
    if (r >= n_rows) return;
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * n);
    float4 xv[CH];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = lane + j * 32;
        xv[j] = i < n4 ? xr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += xv[j].x * xv[j].x + xv[j].y * xv[j].y + xv[j].z * xv[j].z + xv[j].w * xv[j].w;
    }
    ss = warp_sum(ss);
    const float scale = 1.0f / sqrtf(ss / (float)n + eps);
    T* o = out + (size_t)r * n;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = lane + j * 32;
        if (i < n4) {
            const float4 wv = reinterpret_cast<const float4*>(w)[i];
            store4<T>(o + 4 * i, xv[j].x * scale * wv.x, xv[j].y * scale * wv.y, xv[j].z * scale * wv.z,
                      xv[j].w * scale * wv.w);
        }
    }
}

template <typename T>
cudaError_t launch_rmsnorm(const float* x, const float* w, const int* rows, T* out, int n_rows, int n, float eps,
                           cudaStream_t stream) {
    const bool vec = n % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0;
    const int n4 = n / 4;
    if (vec && n_rows >= 256 && n4 <= 32 * 64) {
        // many rows: a warp per row (measured at 2,048 rows of 3584: 14-16 us with a block per row)
        const int ch = (n4 + 31) / 32;
        const int blocks = (n_rows + 7) / 8;
        if (ch <= 8) return launch_dependent(rmsnorm_warp_kernel<T, 8>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        if (ch <= 16) return launch_dependent(rmsnorm_warp_kernel<T, 16>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        if (ch <= 32) return launch_dependent(rmsnorm_warp_kernel<T, 32>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        return launch_dependent(rmsnorm_warp_kernel<T, 64>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
    }
    if (vec && n4 <= 4 * 1024) {
        // as many threads as float4s, rounded up to whole warps, at most 1024
        int threads = ((n4 + 31) / 32) * 32;
        if (threads > 1024) threads = 1024;
        const int per = (n4 + threads - 1) / threads;
        if (per <= 1) return launch_dependent(rmsnorm_vec_kernel<T, 1>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
        if (per <= 2) return launch_dependent(rmsnorm_vec_kernel<T, 2>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
        return launch_dependent(rmsnorm_vec_kernel<T, 4>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
    }
    const int threads = n >= 1024 ? 256 : 128;
    return launch_dependent(rmsnorm_kernel<T>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
}

RI_API int ri_rmsnorm(const float* x, const float* w, const int* rows, void* out, int out_dtype,
                      int n_rows, int n, float eps, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    cudaError_t e = cudaSuccess;
    if (out_dtype == RI_F32)
        e = launch_rmsnorm<float>(x, w, rows, (float*)out, n_rows, n, eps, stream);
    else if (out_dtype == RI_BF16)
        e = launch_rmsnorm<__nv_bfloat16>(x, w, rows, (__nv_bfloat16*)out, n_rows, n, eps, stream);
    else
        return fail("rmsnorm: unknown dtype %d", out_dtype);
    return check_launch(e, "rmsnorm");
}

// Two norms of the same rows with one pass over the statistics: out_a = x / rms * w_a, out_b = x / rms * w_b
// (a layer whose mixer and feed-forward read the same stream through norms of their own).  For steps of few
// rows, where a kernel's launch costs more than its work; a block per row.
namespace {
template <typename T>
__global__ void rmsnorm_pair_kernel(const float* x, const float* __restrict__ w_a, const float* __restrict__ w_b,
                                    T* __restrict__ out_a, T* __restrict__ out_b, int n, float eps, int vec) {
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();          // x is the residual stream the previous kernel wrote
    const float* xr = x + (size_t)r * n;
    float ss = 0.f;
    if (vec) {
        for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(xr)[i];
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) ss += xr[i] * xr[i];
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss / (float)n + eps);
    T* oa = out_a + (size_t)r * n;
    T* ob = out_b + (size_t)r * n;
    if (vec) {
        for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(xr)[i];
            const float4 a = reinterpret_cast<const float4*>(w_a)[i], b = reinterpret_cast<const float4*>(w_b)[i];
            store4<T>(oa + 4 * i, v.x * scale * a.x, v.y * scale * a.y, v.z * scale * a.z, v.w * scale * a.w);
            store4<T>(ob + 4 * i, v.x * scale * b.x, v.y * scale * b.y, v.z * scale * b.z, v.w * scale * b.w);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const float v = xr[i] * scale;
            oa[i] = from_f32<T>(v * w_a[i]);
            ob[i] = from_f32<T>(v * w_b[i]);
        }
    }
}
}  // namespace

RI_API int ri_rmsnorm_pair(const float* x, const float* w_a, const float* w_b, void* out_a, void* out_b, int out_dtype,
                           int n_rows, int n, float eps, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    const int vec = n % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w_a % 16 == 0 && (uintptr_t)w_b % 16 == 0 &&
                    (uintptr_t)out_a % 16 == 0 && (uintptr_t)out_b % 16 == 0;
    int threads = vec ? ((n / 4 + 31) / 32) * 32 : 256;
    threads = threads > 1024 ? 1024 : (threads < 32 ? 32 : threads);
    cudaError_t e;
    if (out_dtype == RI_F32)
        e = launch_dependent(rmsnorm_pair_kernel<float>, n_rows, threads, 0, stream, x, w_a, w_b, (float*)out_a, (float*)out_b, n, eps, vec);
    else if (out_dtype == RI_BF16)
        e = launch_dependent(rmsnorm_pair_kernel<__nv_bfloat16>, n_rows, threads, 0, stream, x, w_a, w_b, (__nv_bfloat16*)out_a,
                             (__nv_bfloat16*)out_b, n, eps, vec);
    else
        return fail("rmsnorm_pair: unknown dtype %d", out_dtype);
    return check_launch(e, "rmsnorm_pair");
}

// ----------------------------------------------------------------------------
// Layer norm with a weight and no bias: y = (x - mean) / sqrt(var + eps) * w, var the mean of the squared
// deviations from the mean (taken in a second pass over the row, which stays in registers: no
// E[x^2] - mean^2 cancellation).  Statistics in float32.  `rows` (may be null) picks the input rows.
// ----------------------------------------------------------------------------
namespace {
// few rows: a block per row, PER float4s of the row per thread
template <typename T, int PER>
__global__ void __launch_bounds__(1024)
layernorm_vec_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ rows,
                     T* __restrict__ out, int n, float eps) {
    __shared__ float scratch[33];
    const int r = blockIdx.x, n4 = n >> 2;
    float4 wv[PER], xv[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        wv[j] = i < n4 ? reinterpret_cast<const float4*>(w)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int in_row = rows ? rows[r] : r;
    let_next_kernel_start();
    wait_for_previous_kernels();
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)in_row * n);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        xv[j] = i < n4 ? xr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        sum += (xv[j].x + xv[j].y) + (xv[j].z + xv[j].w);
    }
    const float mean = block_sum(sum, scratch) / (float)n;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < n4) {
            xv[j].x -= mean; xv[j].y -= mean; xv[j].z -= mean; xv[j].w -= mean;
            ss += xv[j].x * xv[j].x + xv[j].y * xv[j].y + xv[j].z * xv[j].z + xv[j].w * xv[j].w;
        }
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    T* o = out + (size_t)r * n;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < n4)
            store4<T>(o + 4 * i, xv[j].x * scale * wv[j].x, xv[j].y * scale * wv[j].y, xv[j].z * scale * wv[j].z,
                      xv[j].w * scale * wv[j].w);
    }
}

// many rows: a warp per row, CH float4s per lane, no block-wide barrier
template <typename T, int CH>
__global__ void __launch_bounds__(256)
layernorm_warp_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ rows,
                      T* __restrict__ out, int n_rows, int n, float eps) {
    const int lane = threadIdx.x & 31, n4 = n >> 2;
    const int r = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    let_next_kernel_start();
    wait_for_previous_kernels();
    if (r >= n_rows) return;
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * n);
    float4 xv[CH];
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = lane + j * 32;
        xv[j] = i < n4 ? xr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        sum += (xv[j].x + xv[j].y) + (xv[j].z + xv[j].w);
    }
    const float mean = warp_sum(sum) / (float)n;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = lane + j * 32;
        if (i < n4) {
            xv[j].x -= mean; xv[j].y -= mean; xv[j].z -= mean; xv[j].w -= mean;
            ss += xv[j].x * xv[j].x + xv[j].y * xv[j].y + xv[j].z * xv[j].z + xv[j].w * xv[j].w;
        }
    }
    const float scale = 1.0f / sqrtf(warp_sum(ss) / (float)n + eps);
    T* o = out + (size_t)r * n;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = lane + j * 32;
        if (i < n4) {
            const float4 wv = reinterpret_cast<const float4*>(w)[i];
            store4<T>(o + 4 * i, xv[j].x * scale * wv.x, xv[j].y * scale * wv.y, xv[j].z * scale * wv.z,
                      xv[j].w * scale * wv.w);
        }
    }
}

// any width: a block per row, three passes over the row (it stays in L1)
template <typename T>
__global__ void layernorm_kernel(const float* __restrict__ x, const float* __restrict__ w, const int* __restrict__ rows,
                                 T* __restrict__ out, int n, float eps) {
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();
    const float* xr = x + (size_t)(rows ? rows[r] : r) * n;
    float sum = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) sum += xr[i];
    const float mean = block_sum(sum, scratch) / (float)n;
    float ss = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float d = xr[i] - mean;
        ss += d * d;
    }
    const float scale = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
    T* o = out + (size_t)r * n;
    for (int i = threadIdx.x; i < n; i += blockDim.x) o[i] = from_f32<T>((xr[i] - mean) * scale * w[i]);
}

template <typename T>
cudaError_t launch_layernorm(const float* x, const float* w, const int* rows, T* out, int n_rows, int n, float eps,
                             cudaStream_t stream) {
    const bool vec = n % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)out % 16 == 0;
    const int n4 = n / 4;
    if (vec && n_rows >= 256 && n4 <= 32 * 64) {
        const int ch = (n4 + 31) / 32;
        const int blocks = (n_rows + 7) / 8;
        if (ch <= 8) return launch_dependent(layernorm_warp_kernel<T, 8>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        if (ch <= 16) return launch_dependent(layernorm_warp_kernel<T, 16>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        if (ch <= 32) return launch_dependent(layernorm_warp_kernel<T, 32>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
        return launch_dependent(layernorm_warp_kernel<T, 64>, blocks, 256, 0, stream, x, w, rows, out, n_rows, n, eps);
    }
    if (vec && n4 <= 4 * 1024) {
        int threads = ((n4 + 31) / 32) * 32;
        if (threads > 1024) threads = 1024;
        const int per = (n4 + threads - 1) / threads;
        if (per <= 1) return launch_dependent(layernorm_vec_kernel<T, 1>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
        if (per <= 2) return launch_dependent(layernorm_vec_kernel<T, 2>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
        return launch_dependent(layernorm_vec_kernel<T, 4>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
    }
    const int threads = n >= 1024 ? 256 : 128;
    return launch_dependent(layernorm_kernel<T>, n_rows, threads, 0, stream, x, w, rows, out, n, eps);
}
}  // namespace

RI_API int ri_layernorm(const float* x, const float* w, const int* rows, void* out, int out_dtype,
                        int n_rows, int n, float eps, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    cudaError_t e = cudaSuccess;
    if (out_dtype == RI_F32)
        e = launch_layernorm<float>(x, w, rows, (float*)out, n_rows, n, eps, stream);
    else if (out_dtype == RI_BF16)
        e = launch_layernorm<__nv_bfloat16>(x, w, rows, (__nv_bfloat16*)out, n_rows, n, eps, stream);
    else
        return fail("layernorm: unknown dtype %d", out_dtype);
    return check_launch(e, "layernorm");
}

// ----------------------------------------------------------------------------
// Rotary position encoding + cache write.
//
// qkv is [n_tokens, ld] with q at column 0 (n_heads*hd), k at q_dim, v at q_dim + kv_dim.
// Every q head and every k head is rotated with the table row of the token's position
// (attention.rs:78-87, rope.rs:88-97); q is rotated in place, rotated k and plain v go
// to the token's cache position (attention.rs:89-90, kv_cache.rs:52-75).
//
// style 0: pairs (i, i + hd/2); style 1: pairs (2i, 2i+1), the reference's.  With `rot` < hd only the
// first `rot` channels of a head are rotated (pairs (i, i + rot/2) or (2i, 2i+1) within them, the table
// having rot/2 angles per position) and the rest pass unchanged; values may have a head size of their
// own (`v_hd`), their cache then being [page][kv head][page_size][v_hd].
// Cache layer layout: [page][kv head][page_size][hd]; page of position p of sequence b is
// page_table[slot(b) * max_pages + p / page_size].
// ----------------------------------------------------------------------------
template <typename T>
__global__ void rope_cache_write_kernel(T* __restrict__ qkv, int ld, const float* __restrict__ cos_t,
                                        const float* __restrict__ sin_t, const int* __restrict__ token_pos,
                                        const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                        const int* __restrict__ page_table, int max_pages,
                                        T* __restrict__ kcache, T* __restrict__ vcache,
                                        int n_heads, int n_kv_heads, int hd, int page_size, int style,
                                        int write_kv, int rot, int v_hd) {
    const int t = blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();          // the projections come from the previous kernel
    const int pos = token_pos[t];
    const int half = rot >> 1;
    T* row = qkv + (size_t)t * ld;
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    const int q_dim = n_heads * hd, kv_dim = n_kv_heads * hd;

    size_t cache_base = 0;
    if (write_kv) {
        const int slot = seq_slot[token_seq[t]];
        // checked build: a slot, a page index or a page outside its range is recorded and nothing is written
        if (!RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_BLOCK_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) {
            write_kv = 0;
        } else {
            const int page = page_table[(size_t)slot * max_pages + pos / page_size];
            if (!RI_BLOCK_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) write_kv = 0;
            cache_base = (size_t)page * n_kv_heads * page_size + (pos % page_size);      // in rows
        }
    }
    const size_t head_stride = (size_t)page_size * hd, v_head_stride = (size_t)page_size * v_hd;
    const size_t v_base = cache_base * v_hd;
    cache_base *= hd;

    // q heads: rotate in place
    for (int idx = threadIdx.x; idx < n_heads * half; idx += blockDim.x) {
        const int h = idx / half, i = idx % half;
        const int i0 = style == 0 ? i : 2 * i;
        const int i1 = style == 0 ? i + half : 2 * i + 1;
        T* v = row + h * hd;
        const float x0 = to_f32<T>(v[i0]), x1 = to_f32<T>(v[i1]);
        v[i0] = from_f32<T>(x0 * c[i] - x1 * s[i]);
        v[i1] = from_f32<T>(x0 * s[i] + x1 * c[i]);
    }
    if (!write_kv) return;
    // k heads: rotate into the cache
    for (int idx = threadIdx.x; idx < n_kv_heads * half; idx += blockDim.x) {
        const int h = idx / half, i = idx % half;
        const int i0 = style == 0 ? i : 2 * i;
        const int i1 = style == 0 ? i + half : 2 * i + 1;
        const T* v = row + q_dim + h * hd;
        const float x0 = to_f32<T>(v[i0]), x1 = to_f32<T>(v[i1]);
        T* dst = kcache + cache_base + h * head_stride;
        dst[i0] = from_f32<T>(x0 * c[i] - x1 * s[i]);
        dst[i1] = from_f32<T>(x0 * s[i] + x1 * c[i]);
    }
    // the channels of k beyond the rotated ones: copy
    for (int idx = threadIdx.x; idx < n_kv_heads * (hd - rot); idx += blockDim.x) {
        const int h = idx / (hd - rot), d = rot + idx % (hd - rot);
        kcache[cache_base + h * head_stride + d] = row[q_dim + h * hd + d];
    }
    // v heads: copy
    for (int idx = threadIdx.x; idx < n_kv_heads * v_hd; idx += blockDim.x) {
        const int h = idx / v_hd, d = idx % v_hd;
        vcache[v_base + h * v_head_stride + d] = row[q_dim + kv_dim + idx];
    }
}

// The same for bf16 rows whose head size is a multiple of 16, moved 16 bytes at a time: a thread takes
// 8 consecutive elements of a head (and, for the half-split pairing, their 8 partners half a head on),
// rotates them in float32 and writes them back the same way.
__device__ __forceinline__ void unpack8(const uint4& v, float* f) {
    const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 x = __bfloat1622float2(p[i]);
        f[2 * i] = x.x;
        f[2 * i + 1] = x.y;
    }
}
__device__ __forceinline__ uint4 pack8(const float* f) {
    uint4 v;
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int i = 0; i < 4; ++i) p[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    return v;
}

__global__ void rope_cache_write_vec_kernel(__nv_bfloat16* __restrict__ qkv, int ld, const float* __restrict__ cos_t,
                                            const float* __restrict__ sin_t, const int* __restrict__ token_pos,
                                            const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                            const int* __restrict__ page_table, int max_pages,
                                            __nv_bfloat16* __restrict__ kcache, __nv_bfloat16* __restrict__ vcache,
                                            int n_heads, int n_kv_heads, int hd, int page_size, int style,
                                            int write_kv) {
    const int t = blockIdx.x;
    let_next_kernel_start();
    const int pos = token_pos[t];                     // positions, slots, pages and angles: fixed before the step
    const int half = hd >> 1;
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    const int q_dim = n_heads * hd, kv_dim = n_kv_heads * hd;
    size_t cache_base = 0;
    if (write_kv) {
        const int slot = seq_slot[token_seq[t]];
        // checked build: a slot, a page index or a page outside its range is recorded and nothing is written
        if (!RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_BLOCK_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) {
            write_kv = 0;
        } else {
            const int page = page_table[(size_t)slot * max_pages + pos / page_size];
            if (!RI_BLOCK_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) write_kv = 0;
            cache_base = ((size_t)page * n_kv_heads * page_size + (pos % page_size)) * hd;
        }
    }
    const size_t head_stride = (size_t)page_size * hd;
    wait_for_previous_kernels();          // the projections come from the previous kernel
    __nv_bfloat16* row = qkv + (size_t)t * ld;

    const int heads = n_heads + (write_kv ? n_kv_heads : 0);
    if (style == 0) {
        const int per_head = half / 8;                // chunk pairs of a head
        for (int idx = threadIdx.x; idx < heads * per_head; idx += blockDim.x) {
            const int h = idx / per_head, j = idx % per_head;
            const __nv_bfloat16* src = row + (size_t)h * hd + 8 * j;      // q heads, then k heads: one run of columns
            float lo[8], hi[8], cs[8], sn[8], ylo[8], yhi[8];
            unpack8(*reinterpret_cast<const uint4*>(src), lo);
            unpack8(*reinterpret_cast<const uint4*>(src + half), hi);
            *reinterpret_cast<float4*>(cs) = *reinterpret_cast<const float4*>(c + 8 * j);
            *reinterpret_cast<float4*>(cs + 4) = *reinterpret_cast<const float4*>(c + 8 * j + 4);
            *reinterpret_cast<float4*>(sn) = *reinterpret_cast<const float4*>(s + 8 * j);
            *reinterpret_cast<float4*>(sn + 4) = *reinterpret_cast<const float4*>(s + 8 * j + 4);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                ylo[i] = lo[i] * cs[i] - hi[i] * sn[i];
                yhi[i] = lo[i] * sn[i] + hi[i] * cs[i];
            }
            __nv_bfloat16* dst = h < n_heads ? row + (size_t)h * hd + 8 * j
                                             : kcache + cache_base + (size_t)(h - n_heads) * head_stride + 8 * j;
            *reinterpret_cast<uint4*>(dst) = pack8(ylo);
            *reinterpret_cast<uint4*>(dst + half) = pack8(yhi);
        }
    } else {
        const int per_head = hd / 8;                  // chunks of a head, 4 adjacent pairs each
        for (int idx = threadIdx.x; idx < heads * per_head; idx += blockDim.x) {
            const int h = idx / per_head, j = idx % per_head;
            const __nv_bfloat16* src = row + (size_t)h * hd + 8 * j;
            float x[8], y[8], cs[4], sn[4];
            unpack8(*reinterpret_cast<const uint4*>(src), x);
            *reinterpret_cast<float4*>(cs) = *reinterpret_cast<const float4*>(c + 4 * j);
            *reinterpret_cast<float4*>(sn) = *reinterpret_cast<const float4*>(s + 4 * j);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                y[2 * i] = x[2 * i] * cs[i] - x[2 * i + 1] * sn[i];
                y[2 * i + 1] = x[2 * i] * sn[i] + x[2 * i + 1] * cs[i];
            }
            __nv_bfloat16* dst = h < n_heads ? row + (size_t)h * hd + 8 * j
                                             : kcache + cache_base + (size_t)(h - n_heads) * head_stride + 8 * j;
            *reinterpret_cast<uint4*>(dst) = pack8(y);
        }
    }
    if (!write_kv) return;
    const int v_chunks = hd / 8;
    for (int idx = threadIdx.x; idx < n_kv_heads * v_chunks; idx += blockDim.x) {
        const int h = idx / v_chunks, j = idx % v_chunks;
        *reinterpret_cast<uint4*>(vcache + cache_base + (size_t)h * head_stride + 8 * j) =
            *reinterpret_cast<const uint4*>(row + q_dim + kv_dim + (size_t)h * hd + 8 * j);
    }
}

RI_API int ri_rope_cache_write(void* qkv, int dtype, int ld, const float* cos_t, const float* sin_t,
                               const int* token_pos, const int* token_seq, const int* seq_slot,
                               const int* page_table, int max_pages, void* kcache, void* vcache,
                               int n_tokens, int n_heads, int n_kv_heads, int hd, int page_size,
                               int style, int write_kv, int rot, int v_hd, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rot < 0) rot = hd;                // 0: nothing is rotated, keys and values are only stored
    if (v_hd <= 0) v_hd = hd;
    if (rot % 2 || rot > hd) return fail("rope_cache_write: %d rotated channels of a head of %d", rot, hd);
    if (style != 0 && style != 1) return fail("rope_cache_write: unknown style %d", style);
    const int work = n_heads * hd / 2;
    const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
    cudaError_t e = cudaSuccess;
    const bool aligned = rot == hd && v_hd == hd && hd % 16 == 0 && ld % 8 == 0 && (uintptr_t)qkv % 16 == 0 && (uintptr_t)kcache % 16 == 0 &&
                         (uintptr_t)vcache % 16 == 0 && (uintptr_t)cos_t % 16 == 0 && (uintptr_t)sin_t % 16 == 0;
    if (dtype == RI_BF16 && aligned) {
        const int items = (n_heads + n_kv_heads) * hd / 16;
        const int vthreads = items >= 256 ? 256 : (items >= 128 ? 128 : 64);
        e = launch_dependent(rope_cache_write_vec_kernel, n_tokens, vthreads, 0, stream,
            (__nv_bfloat16*)qkv, ld, cos_t, sin_t, token_pos, token_seq, seq_slot, page_table, max_pages,
            (__nv_bfloat16*)kcache, (__nv_bfloat16*)vcache, n_heads, n_kv_heads, hd, page_size, style, write_kv);
        return check_launch(e, "rope_cache_write");
    }
    if (dtype == RI_F32)
        e = launch_dependent(rope_cache_write_kernel<float>, n_tokens, threads, 0, stream,
            (float*)qkv, ld, cos_t, sin_t, token_pos, token_seq, seq_slot, page_table, max_pages,
            (float*)kcache, (float*)vcache, n_heads, n_kv_heads, hd, page_size, style, write_kv, rot, v_hd);
    else if (dtype == RI_BF16)
        e = launch_dependent(rope_cache_write_kernel<__nv_bfloat16>, n_tokens, threads, 0, stream,
            (__nv_bfloat16*)qkv, ld, cos_t, sin_t, token_pos, token_seq, seq_slot, page_table, max_pages,
            (__nv_bfloat16*)kcache, (__nv_bfloat16*)vcache, n_heads, n_kv_heads, hd, page_size, style, write_kv, rot, v_hd);
    else
        return fail("rope_cache_write: unknown dtype %d", dtype);
    return check_launch(e, "rope_cache_write");
}

// ----------------------------------------------------------------------------
// Rotary position encoding + cache write for heads that are normalised first.
//
// qkv is [n_tokens, ld] with q at column 0 (n_heads * hd) and k after it (n_kv_heads * hd).  Every q and k
// head is divided by its root mean square, sqrt(mean(x^2) + eps), and multiplied by a weight of hd values
// that all heads share (q_w for queries, k_w for keys; null: the head is left as it is); then the first
// `rot` channels are rotated as above.  q is rewritten in place, k goes to the cache.  The values are
// either the columns after k (n_kv_heads * v_hd, copied; with `mix` v becomes (1 - mix[0]) v + mix[0] v_other, v_other a
// row of the same values at v_other + t * v_other_ld, in float32 with one rounding), or, with `v_from_k`, the key heads as they were
// projected, before norm and rotation (v_hd == hd; qkv then has no value columns).
// A warp per (token, head): the head is read once into shared memory as float32.
// ----------------------------------------------------------------------------
namespace {
constexpr int NORMED_ROPE_WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(NORMED_ROPE_WARPS * 32)
rope_normed_cache_write_kernel(T* __restrict__ qkv, int ld, const float* __restrict__ cos_t,
                               const float* __restrict__ sin_t, const float* __restrict__ q_w,
                               const float* __restrict__ k_w, float eps, const int* __restrict__ token_pos,
                               const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                               const int* __restrict__ page_table, int max_pages, T* __restrict__ kcache,
                               T* __restrict__ vcache, int n_tokens, int n_heads, int n_kv_heads, int hd, int page_size,
                               int style, int write_kv, int rot, int v_hd, int v_from_k, const float* __restrict__ mix,
                               const T* __restrict__ v_other, int v_other_ld) {
    extern __shared__ float head_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* x = head_smem + (size_t)warp * hd;
    const int heads = n_heads + n_kv_heads + (v_from_k ? 0 : n_kv_heads);     // copied value heads count as items too
    const long long item = (long long)blockIdx.x * NORMED_ROPE_WARPS + warp;
    let_next_kernel_start();
    wait_for_previous_kernels();          // the projections come from the previous kernel
    if (item >= (long long)n_tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item % heads);
    if (h >= n_heads && !write_kv) return;
    const int pos = token_pos[t];
    const int half = rot >> 1;
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    T* row = qkv + (size_t)t * ld;

    size_t cache_row = 0;                 // in rows of one kv head
    if (h >= n_heads) {
        const int slot = seq_slot[token_seq[t]];
        if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) return;
        const int page = page_table[(size_t)slot * max_pages + pos / page_size];
        if (!RI_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) return;
        cache_row = (size_t)page * n_kv_heads * page_size + (pos % page_size);
    }
    if (h >= n_heads + n_kv_heads) {      // a value head of its own: copy
        const int kh = h - n_heads - n_kv_heads;
        const T* src = row + (size_t)(n_heads + n_kv_heads) * hd + (size_t)kh * v_hd;
        T* dst = vcache + (cache_row + (size_t)kh * page_size) * v_hd;
        if (mix != nullptr) {
            const float m = mix[0];
            const T* other = v_other + (size_t)t * v_other_ld + (size_t)kh * v_hd;
            for (int d = lane; d < v_hd; d += 32) dst[d] = from_f32<T>((1.f - m) * to_f32<T>(src[d]) + m * to_f32<T>(other[d]));
            return;
        }
        for (int d = lane; d < v_hd; d += 32) dst[d] = src[d];
        return;
    }
    const bool is_q = h < n_heads;
    const int kh = h - n_heads;
    T* src = row + (size_t)h * hd;        // q heads, then k heads: one run of columns
    const float* w = is_q ? q_w : k_w;
    T* vdst = (!is_q && v_from_k) ? vcache + (cache_row + (size_t)kh * page_size) * hd : nullptr;
    float ss = 0.f;
    for (int d = lane; d < hd; d += 32) {
        const T raw = src[d];
        if (vdst != nullptr) vdst[d] = raw;                       // the value: the key as projected
        const float v = to_f32<T>(raw);
        x[d] = v;
        ss += v * v;
    }
    if (w != nullptr) {
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)hd + eps);
        for (int d = lane; d < hd; d += 32) x[d] = x[d] * scale * w[d];
    }
    __syncwarp();
    T* dst = is_q ? src : kcache + (cache_row + (size_t)kh * page_size) * hd;
    for (int i = lane; i < half; i += 32) {
        const int i0 = style == 0 ? i : 2 * i;
        const int i1 = style == 0 ? i + half : 2 * i + 1;
        const float x0 = x[i0], x1 = x[i1];
        dst[i0] = from_f32<T>(x0 * c[i] - x1 * s[i]);
        dst[i1] = from_f32<T>(x0 * s[i] + x1 * c[i]);
    }
    for (int d = rot + lane; d < hd; d += 32) dst[d] = from_f32<T>(x[d]);
}
// The same for bf16 heads of up to 256 channels (a multiple of 8), 16 bytes per lane: lane l of the warp holds the
// head's channels 8l .. 8l + 7 in registers, the sum of squares goes through shuffles, and the head is read and
// written once, 16 bytes at a time.  Adjacent pairs (style 1) lie inside a lane; for the halves pairing (style 0)
// a channel's partner lies in lane l ^ (rot / 16), which needs rot to be 16 times a power of two.  rot % 8 == 0.
__global__ void __launch_bounds__(NORMED_ROPE_WARPS * 32)
rope_normed_cache_write_vec_kernel(__nv_bfloat16* __restrict__ qkv, int ld, const float* __restrict__ cos_t,
                                   const float* __restrict__ sin_t, const float* __restrict__ q_w,
                                   const float* __restrict__ k_w, float eps, const int* __restrict__ token_pos,
                                   const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                   const int* __restrict__ page_table, int max_pages, __nv_bfloat16* __restrict__ kcache,
                                   __nv_bfloat16* __restrict__ vcache, int n_tokens, int n_heads, int n_kv_heads, int hd,
                                   int page_size, int style, int write_kv, int rot, int v_hd, int v_from_k,
                                   const float* __restrict__ mix, const __nv_bfloat16* __restrict__ v_other, int v_other_ld) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int heads = n_heads + n_kv_heads + (v_from_k ? 0 : n_kv_heads);
    const long long item = (long long)blockIdx.x * NORMED_ROPE_WARPS + warp;
    let_next_kernel_start();
    if (item >= (long long)n_tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item % heads);
    if (h >= n_heads && !write_kv) return;
    const int pos = token_pos[t];                     // positions, slots, pages and angles: fixed before the step
    const int half = rot >> 1;
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    size_t cache_row = 0;
    if (h >= n_heads) {
        const int slot = seq_slot[token_seq[t]];
        if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) return;
        const int page = page_table[(size_t)slot * max_pages + pos / page_size];
        if (!RI_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) return;
        cache_row = (size_t)page * n_kv_heads * page_size + (pos % page_size);
    }
    const int ch = 8 * lane;
    // this lane's angles (loaded before the wait: the tables are written once)
    float cs[8], sn[8];
    int n_ang = 0, a0 = 0;                            // style 1: 4 angles from ch / 2; style 0: 8 from ch % half
    if (ch < rot) {
        n_ang = style == 1 ? 4 : 8;
        a0 = style == 1 ? ch >> 1 : ch % half;
    }
#pragma unroll
    for (int i = 0; i < 8; i += 4) {
        if (i < n_ang) {
            *reinterpret_cast<float4*>(cs + i) = *reinterpret_cast<const float4*>(c + a0 + i);
            *reinterpret_cast<float4*>(sn + i) = *reinterpret_cast<const float4*>(s + a0 + i);
        } else {
            cs[i] = cs[i + 1] = cs[i + 2] = cs[i + 3] = 1.f;
            sn[i] = sn[i + 1] = sn[i + 2] = sn[i + 3] = 0.f;
        }
    }
    const bool is_q = h < n_heads;
    const float* w = is_q ? q_w : k_w;
    float wv[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) wv[i] = 1.f;
    if (w != nullptr && ch < hd && h < n_heads + n_kv_heads) {
        *reinterpret_cast<float4*>(wv) = *reinterpret_cast<const float4*>(w + ch);
        *reinterpret_cast<float4*>(wv + 4) = *reinterpret_cast<const float4*>(w + ch + 4);
    }
    wait_for_previous_kernels();          // the projections come from the previous kernel
    __nv_bfloat16* row = qkv + (size_t)t * ld;
    if (h >= n_heads + n_kv_heads) {      // a value head of its own: copy
        const int kh = h - n_heads - n_kv_heads;
        if (ch < v_hd) {
            uint4 v = *reinterpret_cast<const uint4*>(row + (size_t)(n_heads + n_kv_heads) * hd + (size_t)kh * v_hd + ch);
            if (mix != nullptr) {
                const float m = mix[0];
                float a[8], b[8];
                unpack8(v, a);
                unpack8(*reinterpret_cast<const uint4*>(v_other + (size_t)t * v_other_ld + (size_t)kh * v_hd + ch), b);
#pragma unroll
                for (int i = 0; i < 8; ++i) a[i] = (1.f - m) * a[i] + m * b[i];
                v = pack8(a);
            }
            *reinterpret_cast<uint4*>(vcache + (cache_row + (size_t)kh * page_size) * v_hd + ch) = v;
        }
        return;
    }
    const int kh = h - n_heads;
    __nv_bfloat16* src = row + (size_t)h * hd;
    float x[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = 0.f;
    if (ch < hd) {
        const uint4 raw = *reinterpret_cast<const uint4*>(src + ch);
        if (!is_q && v_from_k) *reinterpret_cast<uint4*>(vcache + (cache_row + (size_t)kh * page_size) * hd + ch) = raw;
        unpack8(raw, x);
    }
    if (w != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) ss += x[i] * x[i];
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)hd + eps);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] = x[i] * scale * wv[i];
    }
    float y[8];
    if (style == 1) {
#pragma unroll
        for (int p = 0; p < 4; ++p) {     // lanes beyond the rotated channels have cos 1, sin 0
            y[2 * p] = x[2 * p] * cs[p] - x[2 * p + 1] * sn[p];
            y[2 * p + 1] = x[2 * p] * sn[p] + x[2 * p + 1] * cs[p];
        }
    } else {
        const int partner = half >> 3;    // lanes between a channel and its partner
        const bool low = ch < half;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float other = __shfl_xor_sync(0xffffffffu, x[i], partner);
            y[i] = ch >= rot ? x[i] : (low ? x[i] * cs[i] - other * sn[i] : other * sn[i] + x[i] * cs[i]);
        }
    }
    if (ch < hd) {
        __nv_bfloat16* dst = is_q ? src : kcache + (cache_row + (size_t)kh * page_size) * hd;
        *reinterpret_cast<uint4*>(dst + ch) = pack8(y);
    }
}

// The same from float32 accumulators of a K-split projection [n_tokens, ld] (q, k and value columns; `bias`, one number per
// column or null, not yet added): the queries go to q_out [n_tokens, n_heads * hd], the values are rounded to T first, as a
// projection in T would leave them, and kept in v_keep [n_tokens, n_kv_heads * v_hd] as well where one is given, and the
// accumulators are left zeroed.  For steps of few tokens.
template <typename T>
__global__ void __launch_bounds__(NORMED_ROPE_WARPS * 32)
rope_normed_cache_write_acc_kernel(float* __restrict__ acc, int ld, const float* __restrict__ bias, T* __restrict__ q_out,
                                   T* __restrict__ v_keep, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                                   const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                   const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                                   const int* __restrict__ seq_slot, const int* __restrict__ page_table, int max_pages,
                                   T* __restrict__ kcache, T* __restrict__ vcache, int n_tokens, int n_heads, int n_kv_heads, int hd,
                                   int page_size, int style, int rot, int v_hd, const float* __restrict__ mix,
                                   const T* v_other, int v_other_ld) {
    extern __shared__ float head_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* x = head_smem + (size_t)warp * hd;
    const int heads = n_heads + 2 * n_kv_heads;
    const long long item = (long long)blockIdx.x * NORMED_ROPE_WARPS + warp;
    let_next_kernel_start();
    if (item >= (long long)n_tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item % heads);
    const int pos = token_pos[t];                     // positions, slots, pages and angles: fixed before the step
    const int half = rot >> 1;
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    size_t cache_row = 0;
    bool store = true;
    if (h >= n_heads) {
        const int slot = seq_slot[token_seq[t]];
        if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) {
            store = false;
        } else {
            const int page = page_table[(size_t)slot * max_pages + pos / page_size];
            if (!RI_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) store = false;
            cache_row = (size_t)page * n_kv_heads * page_size + (pos % page_size);
        }
    }
    wait_for_previous_kernels();          // the projections come from the previous kernel
    const int kh = h - n_heads, vh = kh - n_kv_heads;
    const bool is_v = vh >= 0;
    const int col = is_v ? (n_heads + n_kv_heads) * hd + vh * v_hd : h * hd;
    float* src = acc + (size_t)t * ld + col;
    if (is_v) {
        const float m = mix != nullptr ? mix[0] : 0.f;
        for (int d = lane; d < v_hd; d += 32) {
            const T own = from_f32<T>(src[d] + (bias != nullptr ? bias[col + d] : 0.f));
            src[d] = 0.f;
            float v = to_f32<T>(own);
            if (v_keep != nullptr) v_keep[((size_t)t * n_kv_heads + vh) * v_hd + d] = own;
            if (mix != nullptr) v = (1.f - m) * v + m * to_f32<T>(v_other[(size_t)t * v_other_ld + (size_t)vh * v_hd + d]);
            if (store) vcache[(cache_row + (size_t)vh * page_size) * v_hd + d] = from_f32<T>(v);
        }
        return;
    }
    float ss = 0.f;
    for (int d = lane; d < hd; d += 32) {
        const float v = src[d] + (bias != nullptr ? bias[col + d] : 0.f);
        src[d] = 0.f;
        x[d] = v;
        ss += v * v;
    }
    const float* w = kh < 0 ? q_w : k_w;
    if (w != nullptr) {
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)hd + eps);
        for (int d = lane; d < hd; d += 32) x[d] = x[d] * scale * w[d];
    }
    __syncwarp();
    if (!store) return;
    T* dst = kh < 0 ? q_out + ((size_t)t * n_heads + h) * hd : kcache + (cache_row + (size_t)kh * page_size) * hd;
    for (int i = lane; i < half; i += 32) {
        const int i0 = style == 0 ? i : 2 * i;
        const int i1 = style == 0 ? i + half : 2 * i + 1;
        const float x0 = x[i0], x1 = x[i1];
        dst[i0] = from_f32<T>(x0 * c[i] - x1 * s[i]);
        dst[i1] = from_f32<T>(x0 * s[i] + x1 * c[i]);
    }
    for (int d = rot + lane; d < hd; d += 32) dst[d] = from_f32<T>(x[d]);
}
}  // namespace

// Every layer writes its keys and values here (there is no reading form).
RI_API int ri_rope_normed_cache_write_acc(float* acc, int ld, const float* bias, void* q_out, void* v_keep, int dtype, const float* cos_t,
                                          const float* sin_t, const float* q_w, const float* k_w, float eps, const int* token_pos,
                                          const int* token_seq, const int* seq_slot, const int* page_table, int max_pages, void* kcache,
                                          void* vcache, int n_tokens, int n_heads, int n_kv_heads, int hd, int page_size, int style, int rot,
                                          int v_hd, const float* mix, const void* v_other, int v_other_ld, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rot < 0 || rot % 2 || rot > hd) return fail("rope_normed_cache_write_acc: %d rotated channels of a head of %d", rot, hd);
    if (rot > 0 && (cos_t == nullptr || sin_t == nullptr)) return fail("rope_normed_cache_write_acc: a rotation needs its tables");
    if (style != 0 && style != 1) return fail("rope_normed_cache_write_acc: unknown style %d", style);
    if (mix != nullptr && (v_other == nullptr || v_other_ld < n_kv_heads * v_hd))
        return fail("rope_normed_cache_write_acc: blended values need the rows they are blended with");
    const size_t smem = (size_t)NORMED_ROPE_WARPS * hd * sizeof(float);
    if (smem > 48 * 1024) return fail("rope_normed_cache_write_acc: heads of %d exceed %d", hd, 48 * 1024 / 4 / NORMED_ROPE_WARPS);
    const long long items = (long long)n_tokens * (n_heads + 2 * n_kv_heads);
    const unsigned blocks = (unsigned)((items + NORMED_ROPE_WARPS - 1) / NORMED_ROPE_WARPS);
    cudaError_t e;
#define RI_NORMED_ROPE_ACC(T) launch_dependent(rope_normed_cache_write_acc_kernel<T>, blocks, NORMED_ROPE_WARPS * 32, smem, stream, acc, ld, \
        bias, (T*)q_out, (T*)v_keep, cos_t, sin_t, q_w, k_w, eps, token_pos, token_seq, seq_slot, page_table, max_pages, (T*)kcache, \
        (T*)vcache, n_tokens, n_heads, n_kv_heads, hd, page_size, style, rot, v_hd, mix, (const T*)v_other, v_other_ld)
    if (dtype == RI_F32) e = RI_NORMED_ROPE_ACC(float);
    else if (dtype == RI_BF16) e = RI_NORMED_ROPE_ACC(__nv_bfloat16);
    else return fail("rope_normed_cache_write_acc: unknown dtype %d", dtype);
#undef RI_NORMED_ROPE_ACC
    return check_launch(e, "rope_normed_cache_write_acc");
}

RI_API int ri_rope_normed_cache_write(void* qkv, int dtype, int ld, const float* cos_t, const float* sin_t,
                                      const float* q_w, const float* k_w, float eps, const int* token_pos,
                                      const int* token_seq, const int* seq_slot, const int* page_table, int max_pages,
                                      void* kcache, void* vcache, int n_tokens, int n_heads, int n_kv_heads, int hd,
                                      int page_size, int style, int write_kv, int rot, int v_hd, int v_from_k,
                                      const float* mix, const void* v_other, int v_other_ld, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const bool unrotated = rot < 0;       // rot < 0: nothing is rotated (no tables); 0: the whole head
    if (unrotated) rot = 0;
    else if (rot == 0) rot = hd;
    if (v_hd <= 0) v_hd = hd;
    if (rot % 2 || rot > hd) return fail("rope_normed_cache_write: %d rotated channels of a head of %d", rot, hd);
    if (!unrotated && (cos_t == nullptr || sin_t == nullptr)) return fail("rope_normed_cache_write: a rotation needs its tables");
    if (style != 0 && style != 1) return fail("rope_normed_cache_write: unknown style %d", style);
    if (mix != nullptr && (v_from_k || v_other == nullptr || v_other_ld < n_kv_heads * v_hd))
        return fail("rope_normed_cache_write: blended values need the rows they are blended with");
    if (v_from_k && v_hd != hd) return fail("rope_normed_cache_write: values taken from keys of %d have the size %d", hd, v_hd);
    const size_t smem = (size_t)NORMED_ROPE_WARPS * hd * sizeof(float);
    if (smem > 48 * 1024) return fail("rope_normed_cache_write: heads of %d exceed %d", hd, 48 * 1024 / 4 / NORMED_ROPE_WARPS);
    const int heads = n_heads + n_kv_heads + (v_from_k ? 0 : n_kv_heads);
    const long long items = (long long)n_tokens * heads;
    const unsigned blocks = (unsigned)((items + NORMED_ROPE_WARPS - 1) / NORMED_ROPE_WARPS);
    cudaError_t e;
    const int lanes_apart = rot / 16;     // halves pairing: a channel's partner sits this many lanes away
    const bool pairing_ok = style == 1 || (rot % 16 == 0 && (lanes_apart & (lanes_apart - 1)) == 0);
    const bool aligned = hd % 8 == 0 && hd <= 256 && v_hd % 8 == 0 && v_hd <= 256 && rot % 8 == 0 && ld % 8 == 0 &&
                         (uintptr_t)qkv % 16 == 0 && (uintptr_t)kcache % 16 == 0 && (uintptr_t)vcache % 16 == 0 &&
                         (uintptr_t)cos_t % 16 == 0 && (uintptr_t)sin_t % 16 == 0 && (q_w == nullptr || (uintptr_t)q_w % 16 == 0) &&
                         (k_w == nullptr || (uintptr_t)k_w % 16 == 0) &&
                         (mix == nullptr || ((uintptr_t)v_other % 16 == 0 && v_other_ld % 8 == 0));
    if (dtype == RI_BF16 && aligned && pairing_ok && !unrotated) {
        e = launch_dependent(rope_normed_cache_write_vec_kernel, blocks, NORMED_ROPE_WARPS * 32, 0, stream, (__nv_bfloat16*)qkv, ld,
                             cos_t, sin_t, q_w, k_w, eps, token_pos, token_seq, seq_slot, page_table, max_pages,
                             (__nv_bfloat16*)kcache, (__nv_bfloat16*)vcache, n_tokens, n_heads, n_kv_heads, hd, page_size, style,
                             write_kv, rot, v_hd, v_from_k, mix, (const __nv_bfloat16*)v_other, v_other_ld);
        return check_launch(e, "rope_normed_cache_write");
    }
#define RI_NORMED_ROPE(T) launch_dependent(rope_normed_cache_write_kernel<T>, blocks, NORMED_ROPE_WARPS * 32, smem, stream, \
        (T*)qkv, ld, cos_t, sin_t, q_w, k_w, eps, token_pos, token_seq, seq_slot, page_table, max_pages, (T*)kcache, \
        (T*)vcache, n_tokens, n_heads, n_kv_heads, hd, page_size, style, write_kv, rot, v_hd, v_from_k, mix, (const T*)v_other, v_other_ld)
    if (dtype == RI_F32) e = RI_NORMED_ROPE(float);
    else if (dtype == RI_BF16) e = RI_NORMED_ROPE(__nv_bfloat16);
    else return fail("rope_normed_cache_write: unknown dtype %d", dtype);
#undef RI_NORMED_ROPE
    return check_launch(e, "rope_normed_cache_write");
}

// ----------------------------------------------------------------------------
// The same, fed from float32 accumulators.  When the q/k/v projection of a small step is split
// over K, its pieces are summed into a zeroed float32 buffer acc[n_tokens, ld]; this kernel adds
// the bias, rotates in float32 (q and k never pass through the storage type before rotation),
// writes q to q_out[n_tokens, q_dim] and k, v to the cache, and puts zeros back into `acc`, so
// that the buffer is clean for the next projection.
// ----------------------------------------------------------------------------
template <typename T>
__global__ void rope_cache_write_acc_kernel(float* __restrict__ acc, int ld, const float* __restrict__ bias,
                                            T* __restrict__ q_out, const float* __restrict__ cos_t,
                                            const float* __restrict__ sin_t, const int* __restrict__ token_pos,
                                            const int* __restrict__ token_seq, const int* __restrict__ seq_slot,
                                            const int* __restrict__ page_table, int max_pages,
                                            T* __restrict__ kcache, T* __restrict__ vcache, int n_heads,
                                            int n_kv_heads, int hd, int page_size, int style, int write_kv) {
    constexpr int PER = 4;                 // items a thread handles at once: their loads go out together
    const int t = blockIdx.x;
    const int half = hd >> 1;
    const int q_dim = n_heads * hd, kv_dim = n_kv_heads * hd;
    const int n_pairs = (n_heads + n_kv_heads) * half;
    float* row = acc + (size_t)t * ld;
    let_next_kernel_start();
    // Positions, slots, the page table, the angle tables and the bias are written by no kernel of the
    // step: they are read (for the first round of items) while the projection before this still runs.
    const int pos = token_pos[t];
    const float* c = cos_t + (size_t)pos * half;
    const float* s = sin_t + (size_t)pos * half;
    size_t cache_base = 0;
    if (write_kv) {
        const int slot = seq_slot[token_seq[t]];
        // checked build: a slot, a page index or a page outside its range is recorded and nothing is written
        if (!RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT) || !RI_BLOCK_IN_RANGE(pos / page_size, max_pages, RI_CHECK_PAGE_INDEX)) {
            write_kv = 0;
        } else {
            const int page = page_table[(size_t)slot * max_pages + pos / page_size];
            if (!RI_BLOCK_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) write_kv = 0;
            cache_base = ((size_t)page * n_kv_heads * page_size + (pos % page_size)) * hd;
        }
    }
    const size_t head_stride = (size_t)page_size * hd;

    float cs[PER], sn[PER], b0[PER], b1[PER];
    int c0[PER], c1[PER];
    auto constants = [&](int base) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = base + j * blockDim.x;
            if (idx < n_pairs) {
                const int h = idx / half, i = idx % half;
                c0[j] = h * hd + (style == 0 ? i : 2 * i);
                c1[j] = h * hd + (style == 0 ? i + half : 2 * i + 1);
                b0[j] = bias ? bias[c0[j]] : 0.f;
                b1[j] = bias ? bias[c1[j]] : 0.f;
                cs[j] = c[i];
                sn[j] = s[i];
            }
        }
    };
    constants(threadIdx.x);
    float v_first[PER], vb_first[PER];    // the first round of values and their bias
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int idx = threadIdx.x + j * blockDim.x;
        vb_first[j] = (bias != nullptr && idx < kv_dim) ? bias[q_dim + kv_dim + idx] : 0.f;
    }
    wait_for_previous_kernels();          // the projections come from the previous kernel

    // the first round of values goes out with the first round of pairs: one trip to memory, not two
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int idx = threadIdx.x + j * blockDim.x;
        if (idx < kv_dim) v_first[j] = row[q_dim + kv_dim + idx];
    }
    // rotary pairs of the q heads and then the k heads (same column order in the accumulator)
    for (int base = threadIdx.x; base < n_pairs; base += PER * blockDim.x) {
        if (base != (int)threadIdx.x) constants(base);
        float x0[PER], x1[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = base + j * blockDim.x;
            if (idx < n_pairs) {
                x0[j] = row[c0[j]] + b0[j];
                x1[j] = row[c1[j]] + b1[j];
            }
        }
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = base + j * blockDim.x;
            if (idx < n_pairs) {
                row[c0[j]] = 0.f;
                row[c1[j]] = 0.f;
                const float y0 = x0[j] * cs[j] - x1[j] * sn[j], y1 = x0[j] * sn[j] + x1[j] * cs[j];
                if (c0[j] < q_dim) {
                    q_out[(size_t)t * q_dim + c0[j]] = from_f32<T>(y0);
                    q_out[(size_t)t * q_dim + c1[j]] = from_f32<T>(y1);
                } else if (write_kv) {
                    const int h = (c0[j] - q_dim) / hd;
                    T* dst = kcache + cache_base + h * head_stride;
                    dst[c0[j] - q_dim - h * hd] = from_f32<T>(y0);
                    dst[c1[j] - q_dim - h * hd] = from_f32<T>(y1);
                }
            }
        }
    }
    // values: bias added, stored as they are
    for (int base = threadIdx.x; base < kv_dim; base += PER * blockDim.x) {
        float v[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = base + j * blockDim.x;
            if (idx < kv_dim) {
                if (base == (int)threadIdx.x) {
                    v[j] = v_first[j] + vb_first[j];
                } else {
                    v[j] = row[q_dim + kv_dim + idx];
                    if (bias) v[j] += bias[q_dim + kv_dim + idx];
                }
            }
        }
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = base + j * blockDim.x;
            if (idx < kv_dim) {
                row[q_dim + kv_dim + idx] = 0.f;
                if (write_kv) vcache[cache_base + (idx / hd) * head_stride + (idx % hd)] = from_f32<T>(v[j]);
            }
        }
    }
    RI_PHASE_LATEST(5);
}

RI_API int ri_rope_cache_write_acc(float* acc, int ld, const float* bias, void* q_out, int dtype, const float* cos_t,
                                   const float* sin_t, const int* token_pos, const int* token_seq,
                                   const int* seq_slot, const int* page_table, int max_pages, void* kcache,
                                   void* vcache, int n_tokens, int n_heads, int n_kv_heads, int hd, int page_size,
                                   int style, int write_kv, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (hd % 2) return fail("rope_cache_write: head_dim %d is odd", hd);
    if (style != 0 && style != 1) return fail("rope_cache_write: unknown style %d", style);
    if (ld != (n_heads + 2 * n_kv_heads) * hd) return fail("rope_cache_write: accumulator rows of %d, expected %d", ld, (n_heads + 2 * n_kv_heads) * hd);
    const int work = (n_heads + n_kv_heads) * hd / 2;
    const int threads = work >= 512 ? 512 : (work >= 256 ? 256 : 128);
    cudaError_t e = cudaSuccess;
    if (dtype == RI_F32)
        e = launch_dependent(rope_cache_write_acc_kernel<float>, n_tokens, threads, 0, stream,
            acc, ld, bias, (float*)q_out, cos_t, sin_t, token_pos, token_seq, seq_slot, page_table, max_pages,
            (float*)kcache, (float*)vcache, n_heads, n_kv_heads, hd, page_size, style, write_kv);
    else if (dtype == RI_BF16)
        e = launch_dependent(rope_cache_write_acc_kernel<__nv_bfloat16>, n_tokens, threads, 0, stream,
            acc, ld, bias, (__nv_bfloat16*)q_out, cos_t, sin_t, token_pos, token_seq, seq_slot, page_table, max_pages,
            (__nv_bfloat16*)kcache, (__nv_bfloat16*)vcache, n_heads, n_kv_heads, hd, page_size, style, write_kv);
    else
        return fail("rope_cache_write: unknown dtype %d", dtype);
    return check_launch(e, "rope_cache_write_acc");
}

// ----------------------------------------------------------------------------
// SiLU-gate: out[t, i] = silu(gu[t, i]) * gu[t, inter + i]      (mlp.rs:35-43)
// ----------------------------------------------------------------------------
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gu, T* __restrict__ out, int inter, size_t total) {
    size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const size_t t = idx / inter;
    const int i = (int)(idx % inter);
    const T* row = gu + t * 2 * (size_t)inter;
    out[idx] = from_f32<T>(silu_f32(to_f32<T>(row[i])) * to_f32<T>(row[inter + i]));
}

// ---------------------------------------------------------------------------------------
// Load-time helpers: a change of precision, and seeded normal numbers for the random-weights mode.
// ---------------------------------------------------------------------------------------
template <typename TI, typename TO>
__global__ void cast_kernel(const TI* __restrict__ in, TO* __restrict__ out, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_f32<TO>(to_f32<TI>(in[i]));      // bf16 -> float32 is exact; float32 -> bf16 rounds to nearest even
}

RI_API int ri_cast(const void* in, int in_dtype, void* out, int out_dtype, long long n, cudaStream_t stream) {
    if (n <= 0) return 0;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (in_dtype == RI_F32 && out_dtype == RI_BF16)
        cast_kernel<float, __nv_bfloat16><<<blocks, 256, 0, stream>>>((const float*)in, (__nv_bfloat16*)out, (size_t)n);
    else if (in_dtype == RI_BF16 && out_dtype == RI_F32)
        cast_kernel<__nv_bfloat16, float><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)in, (float*)out, (size_t)n);
    else
        return fail("cast: from dtype %d to dtype %d is not a change between float32 and bfloat16", in_dtype, out_dtype);
    return check_launch("cast");
}

__device__ __forceinline__ unsigned long long fill_mix64(unsigned long long z) {
    z += 0x9E3779B97F4A7C15ull;
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    return z ^ (z >> 31);
}

// Element i of a tensor keyed `key` is mean + std * sqrt(-2 ln u1) * cos(2 pi u2), with u1 in (0, 1] and
// u2 in [0, 1) the upper and the next 24 bits of mix64(key ^ mix64(i)): the same number whatever the
// launch shape, the device or the order tensors are made in.
template <typename T>
__global__ void fill_normal_kernel(T* __restrict__ out, size_t n, unsigned long long key, float mean, float std) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const unsigned long long z = fill_mix64(key ^ fill_mix64((unsigned long long)i));
    const float u1 = (float)((z >> 40) + 1ull) * (1.0f / 16777216.0f);
    const float u2 = (float)((z >> 16) & 0xFFFFFFull) * (1.0f / 16777216.0f);
    out[i] = from_f32<T>(mean + std * sqrtf(-2.0f * logf(u1)) * cospif(2.0f * u2));
}

RI_API int ri_fill_normal(void* out, int dtype, long long n, unsigned long long key, float mean, float std,
                          cudaStream_t stream) {
    if (n <= 0) return 0;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (dtype == RI_F32) fill_normal_kernel<float><<<blocks, 256, 0, stream>>>((float*)out, (size_t)n, key, mean, std);
    else if (dtype == RI_BF16) fill_normal_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((__nv_bfloat16*)out, (size_t)n, key, mean, std);
    else return fail("fill_normal: unknown dtype %d", dtype);
    return check_launch("fill_normal");
}

// ---------------------------------------------------------------------------------------
// The end of a decode step of n sequences (one token each): every sequence is one position
// longer, so the step's int32 arrays move on by one and the next step of the same sequences
// needs nothing from the host.  token_pos, seq_start and seq_len each grow by 1; token_ids
// already hold what the sampler drew.  Optionally (null pointers switch a part off): the
// sampler's per-row draw counters grow by 1; the drawn tokens are copied into slot
// (*turn % host_slots) of a ring in pinned host memory and into slot (*turn % log_slots) of a
// ring on the device; then *turn grows by 1.  One thread block; it runs last in the step.
// ---------------------------------------------------------------------------------------
__global__ void advance_decode_kernel(int* __restrict__ token_pos, int* __restrict__ seq_start,
                                      int* __restrict__ seq_len, int n, const int* __restrict__ token_ids,
                                      int* __restrict__ draw_counter, int* __restrict__ turn,
                                      int* __restrict__ host_ring, int host_slots, int* __restrict__ log_ring,
                                      int log_slots) {
    let_next_kernel_start();
    wait_for_previous_kernels();          // every kernel of the step has read the arrays; the sampler has written the tokens
    const int t = turn ? *turn : 0;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        token_pos[i] += 1;
        seq_start[i] += 1;
        seq_len[i] += 1;
        if (draw_counter) draw_counter[i] += 1;
        if (host_ring || log_ring) {
            const int tok = token_ids[i];
            if (host_ring) host_ring[(size_t)(t % host_slots) * n + i] = tok;
            if (log_ring) log_ring[(size_t)(t % log_slots) * n + i] = tok;
        }
    }
    if (host_ring) __threadfence_system();
    __syncthreads();                      // everyone has read *turn
    if (threadIdx.x == 0 && turn) *turn = t + 1;
}

RI_API int ri_advance_decode(int* token_pos, int* seq_start, int* seq_len, int n, const int* token_ids,
                             int* draw_counter, int* turn, int* host_ring, int host_slots, int* log_ring,
                             int log_slots, cudaStream_t stream) {
    if (n <= 0) return 0;
    if ((host_ring && host_slots < 1) || (log_ring && log_slots < 1)) return fail("advance_decode: a ring needs at least one slot");
    if ((host_ring || log_ring) && (!turn || !token_ids)) return fail("advance_decode: rings need the turn counter and the tokens");
    cudaError_t e = launch_dependent(advance_decode_kernel, dim3(1), dim3(256), (size_t)0, stream, token_pos, seq_start,
                                     seq_len, n, token_ids, draw_counter, turn, host_ring, host_slots, log_ring, log_slots);
    return check_launch(e, "advance_decode");
}

namespace {
template <typename T>
__global__ void scale_kernel(T* __restrict__ x, size_t n, float factor) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        x[i] = from_f32<T>(to_f32<T>(x[i]) * factor);
}
}  // namespace

// x *= factor, in place.
RI_API int ri_scale(void* x, int dtype, long long n, float factor, cudaStream_t stream) {
    if (n <= 0) return 0;
    const int blocks = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
    cudaError_t e;
    if (dtype == RI_F32) e = launch_dependent(scale_kernel<float>, blocks, 256, 0, stream, (float*)x, (size_t)n, factor);
    else if (dtype == RI_BF16)
        e = launch_dependent(scale_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)x, (size_t)n, factor);
    else return fail("scale: unknown dtype %d", dtype);
    return check_launch(e, "scale");
}

namespace {
// x[t, d] += other[t, d] + row[d]; either may be absent.
__global__ void stream_add_kernel(float* x, const float* other, const float* __restrict__ row, size_t total, int width) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        float v = x[i];
        if (other != nullptr) v += other[i];
        if (row != nullptr) v += row[i % width];
        x[i] = v;
    }
}

// x[t, c] *= sigmoid(gate[t, gate_col + c]) * factor, the product formed in float32 and rounded once.
template <typename T>
__global__ void sigmoid_gate_kernel(T* x, const T* gate, int gate_ld, int gate_col, size_t total, int width, float factor) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / width;
        const int c = (int)(i % width);
        const float g = to_f32<T>(gate[t * gate_ld + gate_col + c]);
        const float sig = g >= 0.f ? 1.f / (1.f + expf(-g)) : expf(g) / (1.f + expf(g));
        x[i] = from_f32<T>(to_f32<T>(x[i]) * sig * factor);
    }
}

// The same for bf16 rows of a multiple of 8 values whose gates start on a 16-byte boundary: 16 bytes per thread.
__global__ void sigmoid_gate_vec_kernel(uint4* x, const __nv_bfloat16* gate, int gate_ld, int gate_col, size_t total_vecs,
                                        int vecs, float factor) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total_vecs; i += (size_t)gridDim.x * blockDim.x) {
        const size_t t = i / vecs;
        const int c = (int)(i % vecs) * 8;
        uint4 xv = x[i];
        const uint4 gv = *reinterpret_cast<const uint4*>(gate + t * gate_ld + gate_col + c);
        __nv_bfloat162* xp = reinterpret_cast<__nv_bfloat162*>(&xv);
        const __nv_bfloat162* gp = reinterpret_cast<const __nv_bfloat162*>(&gv);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float2 a = __bfloat1622float2(xp[k]), g = __bfloat1622float2(gp[k]);
            const float s0 = g.x >= 0.f ? 1.f / (1.f + expf(-g.x)) : expf(g.x) / (1.f + expf(g.x));
            const float s1 = g.y >= 0.f ? 1.f / (1.f + expf(-g.y)) : expf(g.y) / (1.f + expf(g.y));
            xp[k] = __floats2bfloat162_rn(a.x * s0 * factor, a.y * s1 * factor);
        }
        x[i] = xv;
    }
}

// x = cap * tanh(x / cap)
__global__ void softcap_kernel(float* x, size_t total, float cap) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const float inv = 1.f / cap;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv);
}
}  // namespace

// x (float32 [n_rows, width]) += other (the same shape, or null) + row (float32 [width], or null), in place.
RI_API int ri_stream_add(float* x, const float* other, const float* row, int n_rows, int width, cudaStream_t stream) {
    const size_t total = (size_t)n_rows * width;
    if (total == 0 || (other == nullptr && row == nullptr)) return 0;
    const int blocks = (int)((total + 255) / 256 < 4096 ? (total + 255) / 256 : 4096);
    cudaError_t e = launch_dependent(stream_add_kernel, blocks, 256, 0, stream, x, other, row, total, width);
    return check_launch(e, "stream_add");
}

// x ([n_rows, width], contiguous) *= sigmoid(gate[:, gate_col .. gate_col + width]) * factor; gate has rows of gate_ld values.
RI_API int ri_sigmoid_gate(void* x, const void* gate, int dtype, int gate_ld, int gate_col, int n_rows, int width, float factor,
                           cudaStream_t stream) {
    const size_t total = (size_t)n_rows * width;
    if (total == 0) return 0;
    if (gate_col < 0 || gate_ld < gate_col + width) return fail("sigmoid_gate: rows of %d values hold no %d gates from column %d", gate_ld, width, gate_col);
    const int blocks = (int)((total + 255) / 256 < 4096 ? (total + 255) / 256 : 4096);
    cudaError_t e;
    if (dtype == RI_F32)
        e = launch_dependent(sigmoid_gate_kernel<float>, blocks, 256, 0, stream, (float*)x, (const float*)gate, gate_ld, gate_col,
                             total, width, factor);
    else if (dtype == RI_BF16 && width % 8 == 0 && gate_ld % 8 == 0 && gate_col % 8 == 0 && (uintptr_t)x % 16 == 0 &&
             (uintptr_t)gate % 16 == 0) {
        const size_t total_vecs = total / 8;
        const int vblocks = (int)((total_vecs + 255) / 256 < 4096 ? (total_vecs + 255) / 256 : 4096);
        e = launch_dependent(sigmoid_gate_vec_kernel, vblocks, 256, 0, stream, (uint4*)x, (const __nv_bfloat16*)gate, gate_ld,
                             gate_col, total_vecs, width / 8, factor);
    } else if (dtype == RI_BF16)
        e = launch_dependent(sigmoid_gate_kernel<__nv_bfloat16>, blocks, 256, 0, stream, (__nv_bfloat16*)x,
                             (const __nv_bfloat16*)gate, gate_ld, gate_col, total, width, factor);
    else return fail("sigmoid_gate: unknown dtype %d", dtype);
    return check_launch(e, "sigmoid_gate");
}

// x (float32, n values) = cap * tanh(x / cap), in place.
RI_API int ri_softcap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) return fail("softcap: a cap of %f is not positive", (double)cap);
    const int blocks = (int)((n + 255) / 256 < 4096 ? (n + 255) / 256 : 4096);
    cudaError_t e = launch_dependent(softcap_kernel, blocks, 256, 0, stream, x, (size_t)n, cap);
    return check_launch(e, "softcap");
}

RI_API int ri_silu_mul(const void* gu, void* out, int dtype, int n_tokens, int inter, cudaStream_t stream) {
    const size_t total = (size_t)n_tokens * inter;
    if (total == 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == RI_F32)
        silu_mul_kernel<float><<<blocks, 256, 0, stream>>>((const float*)gu, (float*)out, inter, total);
    else if (dtype == RI_BF16)
        silu_mul_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)gu, (__nv_bfloat16*)out, inter, total);
    else
        return fail("silu_mul: unknown dtype %d", dtype);
    return check_launch("silu_mul");
}

RI_DEFINE_LAST_ERROR()
