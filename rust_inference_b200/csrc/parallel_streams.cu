// One pass over the parallel hidden streams of a model that has several (float32 [tokens, S * n], a token's streams side by
// side), at the border between two sublayers:
//
//   write   y = branch * scale;   x_t <- sum_s mix[s, t] x_s + w[t] y          all streams at once from the old ones
//   read    u = sum_s r[s] x_s;   out = u / sqrt(mean(u^2) + eps) * norm       into the run dtype
//
// `branch` (float32 [tokens, n]) is the accumulator that the sublayer before added into; it is left zeroed for its next
// user.  Instead of an accumulator the result may be what routed experts left: branch = factor (sum_c weight[t, c]
// y[place[t top + c]] + shared[t]), y float32 rows in the order of the experts' lists (place null: pair t top + c is row
// t top + c), so that their sum needs no pass of its own.  Either half may be left out: no result (the streams are only
// read), no out (they are only written).  scale null: the branch as it is.  r null: the plain sum.  norm null: out
// receives u itself.  `rows` (reading only) picks the tokens.
//
// A block per token.  A thread owns four neighbouring columns, PER times blockDim * 4 apart.  It fetches all of them before it
// writes any (a store to the streams would hold back the loads behind it) and keeps its u until the sum of squares is
// known.  All arithmetic is float32.
#include "common.cuh"

using namespace ri;

namespace {

constexpr int MAX_STREAMS = 16;

struct Cols { float v[4]; };       // four neighbouring columns
__device__ __forceinline__ Cols load_cols(const float* p) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    return {{t.x, t.y, t.z, t.w}};
}
__device__ __forceinline__ void store_cols(float* p, const Cols& r) { *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]); }
__device__ __forceinline__ void store_cols(__nv_bfloat16* p, const Cols& r) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&lo);
    u.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
}

struct StreamsStep {
    float* x;                      // [tokens, streams * n]
    float* branch;                 // null: no accumulator
    const float* y;                // null: no experts' rows (neither: nothing is written)
    const float* weights;          // [tokens, top]
    const int* place;
    const float* shared;           // [tokens, n], or null
    float factor;
    int top;
    const float* scale;
    const float* mix;              // [from, to]
    const float* write;
    const float* read;
    const float* norm;
    const int* rows;
    void* out;                     // null: nothing is read
    float eps;
    int streams, n;
};

constexpr int MAX_TOP = 32;        // experts of a token whose rows are summed here

template <typename T, int S, int PER>
__global__ void __launch_bounds__(PER == 1 ? 1024 : 512) streams_step_kernel(StreamsStep p) {
    __shared__ float scratch[33];
    __shared__ float coef[S * S + 2 * S];             // mix, write, read
    __shared__ float pair_weight[MAX_TOP];
    __shared__ int pair_row[MAX_TOP];
    constexpr int V = 4, streams = S;
    const bool writes = p.branch != nullptr || p.y != nullptr;
    let_next_kernel_start();
    for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {        // weights of the model: written once
        float v = 0.f;
        if (i < S * S) {
            const int s = i / S, t = i % S;
            if (writes) v = p.mix[s * S + t];
        } else if (i < S * S + S) {
            const int t = i - S * S;
            if (writes) v = p.write[t];
        } else {
            const int s = i - S * S - S;
            v = p.read != nullptr ? p.read[s] : 1.f;
        }
        coef[i] = v;
    }
    const int row = p.rows != nullptr ? p.rows[blockIdx.x] : (int)blockIdx.x;
    wait_for_previous_kernels();
    if (p.y != nullptr && (int)threadIdx.x < p.top) {
        const int pair = row * p.top + (int)threadIdx.x;
        pair_weight[threadIdx.x] = p.weights[pair] * p.factor;
        pair_row[threadIdx.x] = p.place != nullptr ? p.place[pair] : pair;
    }
    __syncthreads();
    float* x = p.x + (size_t)row * streams * p.n;
    float* branch = p.branch != nullptr ? p.branch + (size_t)row * p.n : nullptr;
    Cols old[PER][S], y[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
        const bool mine = c < p.n;
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if (mine) {
                old[j][s] = load_cols(x + (size_t)s * p.n + c);
            } else {
#pragma unroll
                for (int k = 0; k < V; ++k) old[j][s].v[k] = 0.f;
            }
        }
        if (mine && branch != nullptr) {
            y[j] = load_cols(branch + c);
        } else {
#pragma unroll
            for (int k = 0; k < V; ++k) y[j].v[k] = 0.f;
        }
    }
    if (p.y != nullptr) {
        if (p.shared != nullptr) {
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int c = (threadIdx.x + j * blockDim.x) * V;
                if (c >= p.n) continue;
                const Cols sh = load_cols(p.shared + (size_t)row * p.n + c);
#pragma unroll
                for (int k = 0; k < V; ++k) y[j].v[k] = p.factor * sh.v[k];
            }
        }
#pragma unroll 4
        for (int e = 0; e < p.top; ++e) {
            const float w = pair_weight[e];
            const float* src = p.y + (size_t)pair_row[e] * p.n;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int c = (threadIdx.x + j * blockDim.x) * V;
                if (c >= p.n) continue;
                const Cols v = load_cols(src + c);
#pragma unroll
                for (int k = 0; k < V; ++k) y[j].v[k] = fmaf(w, v.v[k], y[j].v[k]);
            }
        }
    }
    Cols u[PER];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
#pragma unroll
        for (int k = 0; k < V; ++k) u[j].v[k] = 0.f;
        if (c >= p.n) continue;
        if (writes) {
            if (branch != nullptr) {
                Cols zero;
#pragma unroll
                for (int k = 0; k < V; ++k) zero.v[k] = 0.f;
                store_cols(branch + c, zero);
            }
            if (p.scale != nullptr) {
                const Cols ls = load_cols(p.scale + c);
#pragma unroll
                for (int k = 0; k < V; ++k) y[j].v[k] *= ls.v[k];
            }
#pragma unroll
            for (int t = 0; t < S; ++t) {
                Cols now;
                const float w = coef[S * S + t], r = coef[S * S + S + t];
#pragma unroll
                for (int k = 0; k < V; ++k) {
                    float a = w * y[j].v[k];
#pragma unroll
                    for (int s = 0; s < S; ++s) a = fmaf(coef[s * S + t], old[j][s].v[k], a);
                    now.v[k] = a;
                    u[j].v[k] = fmaf(r, a, u[j].v[k]);
                }
                store_cols(x + (size_t)t * p.n + c, now);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) {
                const float r = coef[S * S + S + s];
#pragma unroll
                for (int k = 0; k < V; ++k) u[j].v[k] = fmaf(r, old[j][s].v[k], u[j].v[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(u[j].v[k], u[j].v[k], ss);
    }
    if (p.out == nullptr) return;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)blockIdx.x * p.n;
    float inv = 1.f;
    if (p.norm != nullptr) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.n + p.eps);
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
        if (c >= p.n) continue;
        if (p.norm != nullptr) {
            const Cols w = load_cols(p.norm + c);
#pragma unroll
            for (int k = 0; k < V; ++k) u[j].v[k] = u[j].v[k] * inv * w.v[k];
        }
        store_cols(out + c, u[j]);
    }
}

// Any number of streams and any width and alignment: a column at a time, the streams read again for the normed result.
template <typename T>
__global__ void __launch_bounds__(256) streams_step_any_kernel(StreamsStep p) {
    __shared__ float scratch[33];
    const bool writes = p.branch != nullptr || p.y != nullptr;
    const int S = p.streams, n = p.n;
    const int row = p.rows != nullptr ? p.rows[blockIdx.x] : (int)blockIdx.x;
    let_next_kernel_start();
    wait_for_previous_kernels();
    float* x = p.x + (size_t)row * S * n;
    float ss = 0.f;
    auto read = [&](int c) {
        float u = 0.f;
        for (int s = 0; s < S; ++s) u = fmaf(p.read != nullptr ? p.read[s] : 1.f, x[(size_t)s * n + c], u);
        return u;
    };
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        if (writes) {
            float y = 0.f;
            if (p.branch != nullptr) {
                y = p.branch[(size_t)row * n + c];
                p.branch[(size_t)row * n + c] = 0.f;
            } else {
                if (p.shared != nullptr) y = p.factor * p.shared[(size_t)row * n + c];
                for (int e = 0; e < p.top; ++e) {
                    const int pair = row * p.top + e;
                    y = fmaf(p.weights[pair] * p.factor, p.y[(size_t)(p.place != nullptr ? p.place[pair] : pair) * n + c], y);
                }
            }
            if (p.scale != nullptr) y *= p.scale[c];
            float old[MAX_STREAMS];
            for (int s = 0; s < S; ++s) old[s] = x[(size_t)s * n + c];
            for (int t = 0; t < S; ++t) {
                float a = p.write[t] * y;
                for (int s = 0; s < S; ++s) a = fmaf(p.mix[s * S + t], old[s], a);
                x[(size_t)t * n + c] = a;
            }
        }
        if (p.out != nullptr) {
            const float u = read(c);
            ss = fmaf(u, u, ss);
        }
    }
    if (p.out == nullptr) return;
    float inv = 1.f;
    if (p.norm != nullptr) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)n + p.eps);
    T* out = reinterpret_cast<T*>(p.out) + (size_t)blockIdx.x * n;
    for (int c = threadIdx.x; c < n; c += blockDim.x) out[c] = from_f32<T>(p.norm != nullptr ? read(c) * inv * p.norm[c] : read(c));
}

constexpr int FEW_ROWS = 296;      // up to so many tokens a block is spread as wide as the row allows

template <typename T, int S>
cudaError_t launch_streams(const StreamsStep& p, int n_rows, cudaStream_t stream) {
    auto whole_warps = [](int threads) { return ((threads + 31) / 32) * 32; };
    const int cols = p.n / 4;
    if (cols <= 1024 && (n_rows <= FEW_ROWS || cols <= 128))
        return launch_dependent(streams_step_kernel<T, S, 1>, n_rows, whole_warps(cols), 0, stream, p);
    if (cols <= 2 * 512) return launch_dependent(streams_step_kernel<T, S, 2>, n_rows, whole_warps((cols + 1) / 2), 0, stream, p);
    return launch_dependent(streams_step_kernel<T, S, 4>, n_rows, whole_warps((cols + 3) / 4), 0, stream, p);
}

template <typename T>
cudaError_t launch_streams_n(const StreamsStep& p, int n_rows, bool vec, cudaStream_t stream) {
    if (vec && p.n <= 4 * 4 * 512) {
        if (p.streams == 1) return launch_streams<T, 1>(p, n_rows, stream);
        if (p.streams == 2) return launch_streams<T, 2>(p, n_rows, stream);
        if (p.streams == 3) return launch_streams<T, 3>(p, n_rows, stream);
        if (p.streams == 4) return launch_streams<T, 4>(p, n_rows, stream);
    }
    return launch_dependent(streams_step_any_kernel<T>, n_rows, 256, 0, stream, p);
}

}  // namespace

// n_rows: the tokens of x, or the number of `rows` (which go with reading only).  write holds whatever factor the
// sublayer's result joins the streams with.  Its result is `branch` or the experts' rows y (one of them, or neither).
RI_API int ri_streams_step(float* x, float* branch, const float* y, const float* weights, const int* place, const float* shared, float factor,
                           int top, const float* scale, const float* mix, const float* write, const float* read,
                           const float* norm, float eps, const int* rows, void* out, int out_dtype, int n_rows, int streams, int n,
                           cudaStream_t stream) {
    if (n_rows <= 0 || n <= 0) return 0;
    if (streams < 1 || streams > MAX_STREAMS) return fail("streams_step: %d streams, at most %d", streams, MAX_STREAMS);
    const bool writes = branch != nullptr || y != nullptr;
    if (!writes && out == nullptr) return fail("streams_step: nothing to write and nothing to read");
    if (branch != nullptr && y != nullptr) return fail("streams_step: a sublayer's result is an accumulator or experts' rows, not both");
    if (y != nullptr && (weights == nullptr || top < 1 || top > MAX_TOP)) return fail("streams_step: the rows of %d experts, at most %d", top, MAX_TOP);
    if (writes && (mix == nullptr || write == nullptr)) return fail("streams_step: writing needs its mixing and its weights");
    if (rows != nullptr && writes) return fail("streams_step: chosen rows are only read");
    StreamsStep p{x, branch, y, weights, place, shared, factor, top, scale, mix, write, read, norm, rows, out, eps, streams, n};
    bool vec = n % 4 == 0;
    for (const void* q : {(const void*)x, (const void*)branch, (const void*)y, (const void*)shared, (const void*)scale, (const void*)norm, (const void*)out})
        vec = vec && (uintptr_t)q % 16 == 0;
    cudaError_t e;
    if (out == nullptr || out_dtype == RI_F32) e = launch_streams_n<float>(p, n_rows, vec, stream);
    else if (out_dtype == RI_BF16) e = launch_streams_n<__nv_bfloat16>(p, n_rows, vec, stream);
    else return fail("streams_step: unknown dtype %d", out_dtype);
    return check_launch(e, "streams_step");
}

RI_DEFINE_LAST_ERROR()
