// One pass over the parallel hidden streams of a model that has several (float32 [tokens, S * n], a token's streams side by
// side), at the border between two sublayers:
//
//   write   y = branch * scale;   x_t <- sum_s mix[s, t] x_s + w[t] y          all streams at once from the old ones
//   read    u = sum_s r[s] x_s;   out = u / sqrt(mean(u^2) + eps) * norm       into the run dtype
//
// `branch` (float32 [tokens, n]) is the accumulator that the sublayer before added into; it is left zeroed for its next
// user.  Either half may be left out: no branch (the streams are only read), no out (they are only written).  scale null:
// the branch as it is.  r null: the plain sum.  norm null: out receives u itself.  `rows` (reading only) picks the tokens.
//
// A block per token.  A thread owns V neighbouring columns, PER times blockDim * V apart; it holds its columns of all S
// streams only while it mixes them, and its u until the sum of squares is known.  All arithmetic is float32.
#include "common.cuh"

using namespace ri;

namespace {

constexpr int MAX_STREAMS = 16;

template <int V> struct Cols { float v[V]; };
template <int V> __device__ __forceinline__ Cols<V> load_cols(const float* p) {
    Cols<V> r;
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_cols(float* p, const Cols<V>& r) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void store_cols(__nv_bfloat16* p, const Cols<V>& r) {
    if constexpr (V == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&lo);
        u.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else {
        *p = __float2bfloat16_rn(r.v[0]);
    }
}

struct StreamsStep {
    float* x;                      // [tokens, streams * n]
    float* branch;                 // null: nothing is written
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

// S: the number of streams, or the most that a block with a number of its own holds (S > 4)
template <typename T, int S, int V, int PER>
__global__ void __launch_bounds__(1024) streams_step_kernel(StreamsStep p) {
    __shared__ float scratch[33];
    __shared__ float coef[S * S + 2 * S];             // mix, write, read
    constexpr bool EXACT = S <= 4;
    const int streams = EXACT ? S : p.streams;
    let_next_kernel_start();
    for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {        // weights: written once
        float v = 0.f;
        if (i < S * S) {
            const int s = i / S, t = i % S;
            if (p.branch != nullptr && s < streams && t < streams) v = p.mix[s * streams + t];
        } else if (i < S * S + S) {
            const int t = i - S * S;
            if (p.branch != nullptr && t < streams) v = p.write[t];
        } else {
            const int s = i - S * S - S;
            if (s < streams) v = p.read != nullptr ? p.read[s] : 1.f;
        }
        coef[i] = v;
    }
    const int row = p.rows != nullptr ? p.rows[blockIdx.x] : (int)blockIdx.x;
    __syncthreads();
    wait_for_previous_kernels();
    float* x = p.x + (size_t)row * streams * p.n;
    float* branch = p.branch != nullptr ? p.branch + (size_t)row * p.n : nullptr;
    Cols<V> u[PER];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * V;
#pragma unroll
        for (int k = 0; k < V; ++k) u[j].v[k] = 0.f;
        if (c >= p.n) continue;
        Cols<V> old[S];
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if (EXACT || s < streams) {
                old[s] = load_cols<V>(x + (size_t)s * p.n + c);
            } else {
#pragma unroll
                for (int k = 0; k < V; ++k) old[s].v[k] = 0.f;
            }
        }
        if (branch != nullptr) {
            Cols<V> y = load_cols<V>(branch + c), zero;
#pragma unroll
            for (int k = 0; k < V; ++k) zero.v[k] = 0.f;
            store_cols<V>(branch + c, zero);
            if (p.scale != nullptr) {
                const Cols<V> ls = load_cols<V>(p.scale + c);
#pragma unroll
                for (int k = 0; k < V; ++k) y.v[k] *= ls.v[k];
            }
#pragma unroll
            for (int t = 0; t < S; ++t) {
                if (!EXACT && t >= streams) break;
                Cols<V> now;
                const float w = coef[S * S + t], r = coef[S * S + S + t];
#pragma unroll
                for (int k = 0; k < V; ++k) {
                    float a = w * y.v[k];
#pragma unroll
                    for (int s = 0; s < S; ++s) a = fmaf(coef[s * S + t], old[s].v[k], a);
                    now.v[k] = a;
                    u[j].v[k] = fmaf(r, a, u[j].v[k]);
                }
                store_cols<V>(x + (size_t)t * p.n + c, now);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) {
                const float r = coef[S * S + S + s];
#pragma unroll
                for (int k = 0; k < V; ++k) u[j].v[k] = fmaf(r, old[s].v[k], u[j].v[k]);
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
            const Cols<V> w = load_cols<V>(p.norm + c);
#pragma unroll
            for (int k = 0; k < V; ++k) u[j].v[k] = u[j].v[k] * inv * w.v[k];
        }
        store_cols<V>(out + c, u[j]);
    }
}

constexpr int FEW_ROWS = 296;      // up to so many tokens a block is spread as wide as the row allows
constexpr int SCALAR_PER = 16;     // rows of up to 16,384 columns of any width and alignment

template <typename T, int S>
cudaError_t launch_streams(const StreamsStep& p, int n_rows, bool vec, cudaStream_t stream) {
    auto whole_warps = [](int threads) { return ((threads + 31) / 32) * 32; };
    if constexpr (S > 4) vec = false;                 // a thread would not hold four columns of so many streams
    if (vec && p.n <= 4 * 1024 && (n_rows <= FEW_ROWS || p.n <= 512))
        return launch_dependent(streams_step_kernel<T, S, 4, 1>, n_rows, whole_warps(p.n / 4), 0, stream, p);
    if (vec) return launch_dependent(streams_step_kernel<T, S, 4, 4>, n_rows, whole_warps((p.n / 4 + 3) / 4), 0, stream, p);
    const int threads = whole_warps((p.n + SCALAR_PER - 1) / SCALAR_PER);
    return launch_dependent(streams_step_kernel<T, S, 1, SCALAR_PER>, n_rows, threads < 128 ? 128 : threads, 0, stream, p);
}

template <typename T>
cudaError_t launch_streams_n(const StreamsStep& p, int n_rows, bool vec, cudaStream_t stream) {
    switch (p.streams) {
        case 1: return launch_streams<T, 1>(p, n_rows, vec, stream);
        case 2: return launch_streams<T, 2>(p, n_rows, vec, stream);
        case 3: return launch_streams<T, 3>(p, n_rows, vec, stream);
        case 4: return launch_streams<T, 4>(p, n_rows, vec, stream);
        default: return launch_streams<T, MAX_STREAMS>(p, n_rows, vec, stream);
    }
}

}  // namespace

// n_rows: the tokens of x, or the number of `rows` (which go with reading only).  write holds whatever factor the
// sublayer's result joins the streams with.
RI_API int ri_streams_step(float* x, float* branch, const float* scale, const float* mix, const float* write, const float* read,
                           const float* norm, float eps, const int* rows, void* out, int out_dtype, int n_rows, int streams, int n,
                           cudaStream_t stream) {
    if (n_rows <= 0 || n <= 0) return 0;
    if (streams < 1 || streams > MAX_STREAMS) return fail("streams_step: %d streams, at most %d", streams, MAX_STREAMS);
    if (n > 16 * 1024) return fail("streams_step: rows of %d columns exceed %d", n, 16 * 1024);
    if (branch == nullptr && out == nullptr) return fail("streams_step: nothing to write and nothing to read");
    if (branch != nullptr && (mix == nullptr || write == nullptr)) return fail("streams_step: writing needs its mixing and its weights");
    if (rows != nullptr && branch != nullptr) return fail("streams_step: chosen rows are only read");
    StreamsStep p{x, branch, scale, mix, write, read, norm, rows, out, eps, streams, n};
    bool vec = n % 4 == 0;
    for (const void* q : {(const void*)x, (const void*)branch, (const void*)scale, (const void*)norm, (const void*)out})
        vec = vec && (uintptr_t)q % 16 == 0;
    cudaError_t e;
    if (out == nullptr || out_dtype == RI_F32) e = launch_streams_n<float>(p, n_rows, vec, stream);
    else if (out_dtype == RI_BF16) e = launch_streams_n<__nv_bfloat16>(p, n_rows, vec, stream);
    else return fail("streams_step: unknown dtype %d", out_dtype);
    return check_launch(e, "streams_step");
}

RI_DEFINE_LAST_ERROR()
