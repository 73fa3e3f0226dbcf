// Short causal convolutions over time, one filter per channel: y_t = sum_j w[j] x_(t - K + 1 + j), nothing before the
// sequence's start.  A sequence's last K - 1 inputs live in a per-slot area of the cache (float32, zeroed when a slot is
// handed out, oldest first) and are carried from step to step, so a prompt may be cut anywhere; a decode step is the same
// kernels with one token per sequence.  Two uses:
//
//   input_conv   what a layer's sublayers read: h = x / sqrt(mean(x^2) + eps) * w of the float32 stream (or x itself),
//                then h + conv(h), for one or two filters (the mixer's and the feed-forward's) that share h and with it the
//                carried inputs.  One kernel for norm, both convolutions and the rounding to the run dtype
//   conv_store   the projected queries, keys and values of an attention layer: bias, convolution, then the queries into
//                the run dtype and keys and values into the token's place of the paged cache
//
// Filters come tap by tap, [K, channels], the last row the current token's, so that neighbouring threads read neighbouring
// numbers.  All arithmetic is float32.  The carried inputs of a sequence whose new tokens are spread over several blocks
// move on in a second kernel (the first block may still read them); in a step of one token per sequence the first
// kernel does it.  What an earlier kernel of the step wrote is read after `wait_for_previous_kernels()` through plain
// pointers.
#include "common.cuh"
#include <initializer_list>

using namespace ri;

namespace {

template <int V> struct Pack { float v[V]; };
template <int V> __device__ __forceinline__ Pack<V> load_pack(const float* p) {
    Pack<V> r;
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) r.v[k] = p[k];
    }
    return r;
}
template <int V> __device__ __forceinline__ void store_pack(float* p, const Pack<V>& r) {
    if constexpr (V == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) p[k] = r.v[k];
    }
}
template <int V> __device__ __forceinline__ void store_pack(__nv_bfloat16* p, const Pack<V>& r) {
    if constexpr (V == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1]), hi = __floats2bfloat162_rn(r.v[2], r.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&lo);
        u.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else {
#pragma unroll
        for (int k = 0; k < V; ++k) p[k] = __float2bfloat16_rn(r.v[k]);
    }
}

struct InputConv {
    const float* x;            // [tokens, n] the stream
    const float* w;            // [n] the norm's factor, or null: h = x
    float eps;
    const float* taps_a;       // [K, n]
    const float* taps_b;       // [K, n] or null: one output
    int k_taps;
    float* carried;            // [slots, K - 1, n]
    void* out_a;
    void* out_b;
    const int* cu_seqlens;
    const int* token_seq;
    const int* seq_slot;
    int n_tokens, n, single;
};

constexpr int MAX_TOKENS = 8;           // tokens of a block
constexpr int MAX_BACK = 64;            // most taps - 1 a block can look back

// The reciprocal root mean square of one row, by the whole block (`scratch`: 33 floats).
template <int V>
__device__ __forceinline__ float block_inv_rms(const float* row, int n, float eps, float* scratch) {
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
        const Pack<V> x = load_pack<V>(row + c);
#pragma unroll
        for (int k = 0; k < V; ++k) ss = fmaf(x.v[k], x.v[k], ss);
    }
    ss = block_sum(ss, scratch);
    return 1.f / sqrtf(ss / (float)n + eps);
}

// A block takes TOKENS consecutive tokens of the packed step.  First the rows' statistics (a warp per row, or the whole
// block where there is one row), of the block's rows and of the K - 1 rows before them; then every thread owns V columns
// and walks down the tokens.
template <typename T, int V, int TOKENS, int KT>
__global__ void __launch_bounds__(1024) input_conv_kernel(InputConv p) {
    __shared__ float scratch[33];
    __shared__ float inv[MAX_TOKENS + MAX_BACK];
    let_next_kernel_start();
    const int K = KT > 0 ? KT : p.k_taps;
    const int t0 = blockIdx.x * TOKENS, t1 = min(p.n_tokens, t0 + TOKENS);
    const int b0 = p.token_seq[t0];
    const int back = min(K - 1, t0 - p.cu_seqlens[b0]);         // rows before the block's that its first sequence has in this step
    const int r0 = t0 - back;
    wait_for_previous_kernels();
    if (p.w != nullptr) {
        if (t1 - r0 == 1) {
            const float f = block_inv_rms<V>(p.x + (size_t)r0 * p.n, p.n, p.eps, scratch);
            if (threadIdx.x == 0) inv[0] = f;
        } else {
            const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
            for (int r = r0 + warp; r < t1; r += warps) {
                const float* row = p.x + (size_t)r * p.n;
                float ss = 0.f;
                for (int c = lane * V; c < p.n; c += 32 * V) {
                    const Pack<V> x = load_pack<V>(row + c);
#pragma unroll
                    for (int k = 0; k < V; ++k) ss = fmaf(x.v[k], x.v[k], ss);
                }
                ss = warp_sum(ss);
                if (lane == 0) inv[r - r0] = 1.f / sqrtf(ss / (float)p.n + p.eps);
            }
        }
        __syncthreads();
    }
    for (int c = threadIdx.x * V; c < p.n; c += blockDim.x * V) {
        Pack<V> wv;
#pragma unroll
        for (int k = 0; k < V; ++k) wv.v[k] = 1.f;
        if (p.w != nullptr) wv = load_pack<V>(p.w + c);
        Pack<V> ta[KT > 0 ? KT : 1], tb[KT > 0 ? KT : 1];
        if constexpr (KT > 0) {
#pragma unroll
            for (int j = 0; j < KT; ++j) {
                ta[j] = load_pack<V>(p.taps_a + (size_t)j * p.n + c);
                if (p.taps_b != nullptr) tb[j] = load_pack<V>(p.taps_b + (size_t)j * p.n + c);
            }
        }
        auto h_of = [&](int row) {
            Pack<V> h = load_pack<V>(p.x + (size_t)row * p.n + c);
            if (p.w != nullptr) {
                const float f = inv[row - r0];
#pragma unroll
                for (int k = 0; k < V; ++k) h.v[k] = h.v[k] * f * wv.v[k];
            }
            return h;
        };
        for (int t = t0; t < t1; ++t) {
            const int b = p.token_seq[t];
            const int i = t - p.cu_seqlens[b];                  // place among the sequence's new tokens
            int slot = p.seq_slot[b];
            if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) slot = 0;
            float* carried = p.carried + (size_t)slot * (K - 1) * p.n + c;
            const Pack<V> now = h_of(t);
            Pack<V> ya = now, yb = now;
#pragma unroll
            for (int j = 0; j < K; ++j) {                       // the input j tokens back
                const Pack<V> h = j == 0 ? now : (i >= j ? h_of(t - j) : load_pack<V>(carried + (size_t)(K - 1 + i - j) * p.n));
                Pack<V> fa, fb;
                if constexpr (KT > 0) {
                    fa = ta[K - 1 - j];
                    fb = tb[K - 1 - j];
                } else {
                    fa = load_pack<V>(p.taps_a + (size_t)(K - 1 - j) * p.n + c);
                    if (p.taps_b != nullptr) fb = load_pack<V>(p.taps_b + (size_t)(K - 1 - j) * p.n + c);
                }
#pragma unroll
                for (int k = 0; k < V; ++k) ya.v[k] = fmaf(fa.v[k], h.v[k], ya.v[k]);
                if (p.taps_b != nullptr) {
#pragma unroll
                    for (int k = 0; k < V; ++k) yb.v[k] = fmaf(fb.v[k], h.v[k], yb.v[k]);
                }
            }
            store_pack<V>(reinterpret_cast<T*>(p.out_a) + (size_t)t * p.n + c, ya);
            if (p.taps_b != nullptr) store_pack<V>(reinterpret_cast<T*>(p.out_b) + (size_t)t * p.n + c, yb);
            if (p.single && K > 1) {                            // one token per sequence: nobody else reads these carried inputs
                for (int s = 0; s < K - 2; ++s) store_pack<V>(carried + (size_t)s * p.n, load_pack<V>(carried + (size_t)(s + 1) * p.n));
                store_pack<V>(carried + (size_t)(K - 2) * p.n, now);
            }
        }
    }
}

// The carried inputs after a step of several tokens per sequence: a block per sequence.
template <int V>
__global__ void __launch_bounds__(256) input_conv_state_kernel(InputConv p) {
    __shared__ float scratch[33];
    __shared__ float inv[MAX_BACK];
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int K = p.k_taps, b = blockIdx.x;
    const int s0 = p.cu_seqlens[b], n_new = p.cu_seqlens[b + 1] - s0;
    const int slot = p.seq_slot[b];
    if (n_new <= 0 || !RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) return;
    for (int s = 0; s < K - 1; ++s) {
        const int src = n_new - (K - 1) + s;
        if (p.w != nullptr && src >= 0) {                       // uniform over the block
            const float f = block_inv_rms<V>(p.x + (size_t)(s0 + src) * p.n, p.n, p.eps, scratch);
            if (threadIdx.x == 0) inv[s] = f;
            __syncthreads();
        }
    }
    for (int c = threadIdx.x * V; c < p.n; c += blockDim.x * V) {
        float* carried = p.carried + (size_t)slot * (K - 1) * p.n + c;
        for (int s = 0; s < K - 1; ++s) {                       // ascending: an entry is read before a later round overwrites it
            const int src = n_new - (K - 1) + s;
            if (src < 0) {
                store_pack<V>(carried + (size_t)s * p.n, load_pack<V>(carried + (size_t)(s + n_new) * p.n));
                continue;
            }
            Pack<V> h = load_pack<V>(p.x + (size_t)(s0 + src) * p.n + c);
            if (p.w != nullptr) {
                const Pack<V> wv = load_pack<V>(p.w + c);
#pragma unroll
                for (int k = 0; k < V; ++k) h.v[k] = h.v[k] * inv[s] * wv.v[k];
            }
            store_pack<V>(carried + (size_t)s * p.n, h);
        }
    }
}

struct ConvStore {
    const float* z;            // [tokens, ld]: queries | keys | values, as projected
    int ld;
    const float* bias;         // [channels] or null
    const float* taps;         // [K, channels]
    int k_taps;
    float* carried;            // [slots, K - 1, channels], biases included
    void* q_out;               // [tokens, q_dim]
    void* kcache;
    void* vcache;
    const int* cu_seqlens;
    const int* token_pos;
    const int* token_seq;
    const int* seq_slot;
    const int* page_table;
    int max_pages, n_tokens, q_dim, n_kv_heads, hd, v_hd, page_size, single;
};

constexpr int STORE_TOKENS = 4;

// A thread owns V neighbouring channels (of one head) and walks down the block's tokens.
template <typename T, int V, int KT>
__global__ void __launch_bounds__(128) conv_store_kernel(ConvStore p) {
    const int K = KT > 0 ? KT : p.k_taps;
    const int kv_dim = p.n_kv_heads * p.hd, channels = p.q_dim + kv_dim + p.n_kv_heads * p.v_hd;
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const bool mine = c < channels;
    let_next_kernel_start();
    Pack<V> f[KT > 0 ? KT : 1], bias;
#pragma unroll
    for (int k = 0; k < V; ++k) bias.v[k] = 0.f;
    if (mine) {
        if (p.bias != nullptr) bias = load_pack<V>(p.bias + c);
        if constexpr (KT > 0) {
#pragma unroll
            for (int j = 0; j < KT; ++j) f[j] = load_pack<V>(p.taps + (size_t)j * channels + c);
        }
    }
    wait_for_previous_kernels();
    if (!mine) return;
    const int t0 = blockIdx.y * STORE_TOKENS, t1 = min(p.n_tokens, t0 + STORE_TOKENS);
    auto projected = [&](int t) {
        Pack<V> x = load_pack<V>(p.z + (size_t)t * p.ld + c);
#pragma unroll
        for (int k = 0; k < V; ++k) x.v[k] += bias.v[k];
        return x;
    };
    for (int t = t0; t < t1; ++t) {
        const int b = p.token_seq[t];
        const int i = t - p.cu_seqlens[b];
        int slot = p.seq_slot[b];
        if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) slot = 0;
        float* carried = p.carried + (size_t)slot * (K - 1) * channels + c;
        const Pack<V> now = projected(t);
        Pack<V> y;
#pragma unroll
        for (int k = 0; k < V; ++k) y.v[k] = 0.f;
#pragma unroll
        for (int j = 0; j < K; ++j) {
            const Pack<V> x = j == 0 ? now : (i >= j ? projected(t - j) : load_pack<V>(carried + (size_t)(K - 1 + i - j) * channels));
            Pack<V> w;
            if constexpr (KT > 0) w = f[K - 1 - j];
            else w = load_pack<V>(p.taps + (size_t)(K - 1 - j) * channels + c);
#pragma unroll
            for (int k = 0; k < V; ++k) y.v[k] = fmaf(w.v[k], x.v[k], y.v[k]);
        }
        if (p.single && K > 1) {
            for (int s = 0; s < K - 2; ++s) store_pack<V>(carried + (size_t)s * channels, load_pack<V>(carried + (size_t)(s + 1) * channels));
            store_pack<V>(carried + (size_t)(K - 2) * channels, now);
        }
        if (c < p.q_dim) {
            store_pack<V>(reinterpret_cast<T*>(p.q_out) + (size_t)t * p.q_dim + c, y);
            continue;
        }
        const int pos = p.token_pos[t];
        if (!RI_IN_RANGE(pos / p.page_size, p.max_pages, RI_CHECK_PAGE_INDEX)) continue;
        const int page = p.page_table[(size_t)slot * p.max_pages + pos / p.page_size];
        if (!RI_IN_LIMIT(page, RI_LIMIT_PAGES, RI_CHECK_PAGE)) continue;
        const size_t row0 = (size_t)page * p.n_kv_heads * p.page_size + pos % p.page_size;      // in rows; a head further is page_size rows on
        if (c < p.q_dim + kv_dim) {
            const int g = (c - p.q_dim) / p.hd, d = (c - p.q_dim) % p.hd;
            store_pack<V>(reinterpret_cast<T*>(p.kcache) + (row0 + (size_t)g * p.page_size) * p.hd + d, y);
        } else {
            const int g = (c - p.q_dim - kv_dim) / p.v_hd, d = (c - p.q_dim - kv_dim) % p.v_hd;
            store_pack<V>(reinterpret_cast<T*>(p.vcache) + (row0 + (size_t)g * p.page_size) * p.v_hd + d, y);
        }
    }
}

__global__ void __launch_bounds__(128) conv_store_state_kernel(const float* z, int ld, const float* __restrict__ bias, int channels,
                                                              int k_taps, float* carried_, const int* cu_seqlens, const int* seq_slot) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int s0 = cu_seqlens[b], n_new = cu_seqlens[b + 1] - s0;
    const int slot = seq_slot[b];
    if (n_new <= 0 || !RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) return;
    float* carried = carried_ + (size_t)slot * (k_taps - 1) * channels + c;
    const float add = bias != nullptr ? bias[c] : 0.f;
    for (int s = 0; s < k_taps - 1; ++s) {
        const int src = n_new - (k_taps - 1) + s;
        carried[(size_t)s * channels] = src >= 0 ? z[(size_t)(s0 + src) * ld + c] + add : carried[(size_t)(s + n_new) * channels];
    }
}

inline bool aligned16(std::initializer_list<const void*> ptrs) {
    for (const void* q : ptrs)
        if (reinterpret_cast<uintptr_t>(q) & 15) return false;
    return true;
}

template <typename T, int V, int TOKENS>
cudaError_t launch_input(const InputConv& p, cudaStream_t stream) {
    int threads = ((p.n / V + 31) / 32) * 32;
    const int most = TOKENS == 1 ? 1024 : 256;
    threads = threads > most ? most : threads;
    const int blocks = (p.n_tokens + TOKENS - 1) / TOKENS;
    switch (p.k_taps) {
        case 1: return launch_dependent(input_conv_kernel<T, V, TOKENS, 1>, blocks, threads, 0, stream, p);
        case 2: return launch_dependent(input_conv_kernel<T, V, TOKENS, 2>, blocks, threads, 0, stream, p);
        case 3: return launch_dependent(input_conv_kernel<T, V, TOKENS, 3>, blocks, threads, 0, stream, p);
        case 4: return launch_dependent(input_conv_kernel<T, V, TOKENS, 4>, blocks, threads, 0, stream, p);
        default: return launch_dependent(input_conv_kernel<T, V, TOKENS, 0>, blocks, threads, 0, stream, p);
    }
}

template <typename T>
cudaError_t dispatch_input(const InputConv& p, bool vec, cudaStream_t stream) {
    if (p.n_tokens < 512) return vec ? launch_input<T, 4, 1>(p, stream) : launch_input<T, 1, 1>(p, stream);
    if (p.n_tokens < 4096) return vec ? launch_input<T, 4, 4>(p, stream) : launch_input<T, 1, 4>(p, stream);
    return vec ? launch_input<T, 4, MAX_TOKENS>(p, stream) : launch_input<T, 1, MAX_TOKENS>(p, stream);
}

template <typename T, int V>
cudaError_t launch_store(const ConvStore& p, int channels, cudaStream_t stream) {
    const dim3 grid((channels / V + 127) / 128, (p.n_tokens + STORE_TOKENS - 1) / STORE_TOKENS);
    switch (p.k_taps) {
        case 2: return launch_dependent(conv_store_kernel<T, V, 2>, grid, 128, 0, stream, p);
        case 3: return launch_dependent(conv_store_kernel<T, V, 3>, grid, 128, 0, stream, p);
        case 4: return launch_dependent(conv_store_kernel<T, V, 4>, grid, 128, 0, stream, p);
        default: return launch_dependent(conv_store_kernel<T, V, 0>, grid, 128, 0, stream, p);
    }
}

}  // namespace

// x: float32 [n_tokens, n].  w (null: no norm), taps_a, taps_b (null: one output), carried: see `InputConv`.  out_a, out_b:
// [n_tokens, n] in `dtype`.  longest_run: the most new tokens any sequence brings.
RI_API int ri_input_conv(const float* x, const float* w, float eps, const float* taps_a, const float* taps_b, int k_taps,
                         float* carried, void* out_a, void* out_b, int dtype, const int* cu_seqlens, const int* token_seq,
                         const int* seq_slot, int n_tokens, int n_seqs, int n, int longest_run, cudaStream_t stream) {
    if (n_tokens <= 0 || n <= 0) return 0;
    if (k_taps < 1 || k_taps - 1 > MAX_BACK) return fail("input_conv: %d taps (1 to %d)", k_taps, MAX_BACK + 1);
    if (dtype != RI_F32 && dtype != RI_BF16) return fail("input_conv: unknown dtype %d", dtype);
    InputConv p{x, w, eps, taps_a, taps_b, k_taps, carried, out_a, out_b, cu_seqlens, token_seq, seq_slot, n_tokens, n,
                longest_run == 1 ? 1 : 0};
    const bool vec = n % 4 == 0 && aligned16({x, w, taps_a, taps_b, carried, out_a, out_b});
    cudaError_t e = dtype == RI_F32 ? dispatch_input<float>(p, vec, stream) : dispatch_input<__nv_bfloat16>(p, vec, stream);
    if (check_launch(e, "input_conv")) return 1;
    if (k_taps > 1 && !p.single) {
        e = vec ? launch_dependent(input_conv_state_kernel<4>, n_seqs, 256, 0, stream, p)
                : launch_dependent(input_conv_state_kernel<1>, n_seqs, 256, 0, stream, p);
        if (check_launch(e, "input_conv (carried inputs)")) return 1;
    }
    return 0;
}

// z: float32 rows, ld apart, with q_dim query channels, then n_kv_heads * hd key and n_kv_heads * v_hd value channels.  bias
// (float32, all channels, or null) is added before the convolution and is part of the carried inputs.  q_out [n_tokens,
// q_dim] and the caches ([pages, n_kv_heads, page_size, hd] / [.., v_hd]) in `dtype`.
RI_API int ri_conv_store(const float* z, int ld, const float* bias, const float* taps, int k_taps, float* carried, void* q_out,
                         void* kcache, void* vcache, int dtype, const int* cu_seqlens, const int* token_pos,
                         const int* token_seq, const int* seq_slot, const int* page_table, int max_pages, int n_tokens,
                         int n_seqs, int q_dim, int n_kv_heads, int hd, int v_hd, int page_size, int longest_run,
                         cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int channels = q_dim + n_kv_heads * (hd + v_hd);
    if (k_taps < 1 || q_dim < 1 || n_kv_heads < 1 || hd < 1 || v_hd < 1 || page_size < 1 || ld < channels)
        return fail("conv_store: %d taps, %d channels in rows of %d", k_taps, channels, ld);
    if ((n_tokens + STORE_TOKENS - 1) / STORE_TOKENS > 65535) return fail("conv_store: %d tokens exceed the grid limit", n_tokens);
    if (dtype != RI_F32 && dtype != RI_BF16) return fail("conv_store: unknown dtype %d", dtype);
    ConvStore p{z, ld, bias, taps, k_taps, carried, q_out, kcache, vcache, cu_seqlens, token_pos, token_seq, seq_slot, page_table,
                max_pages, n_tokens, q_dim, n_kv_heads, hd, v_hd, page_size, longest_run == 1 ? 1 : 0};
    const bool vec = (ld | q_dim | hd | v_hd) % 4 == 0 && aligned16({z, bias, taps, carried, q_out, kcache, vcache});
    cudaError_t e;
    if (dtype == RI_F32) e = vec ? launch_store<float, 4>(p, channels, stream) : launch_store<float, 1>(p, channels, stream);
    else e = vec ? launch_store<__nv_bfloat16, 4>(p, channels, stream) : launch_store<__nv_bfloat16, 1>(p, channels, stream);
    if (check_launch(e, "conv_store")) return 1;
    if (k_taps > 1 && !p.single) {
        e = launch_dependent(conv_store_state_kernel, dim3((channels + 127) / 128, n_seqs), 128, 0, stream, z, ld, bias, channels, k_taps,
                             carried, cu_seqlens, seq_slot);
        if (check_launch(e, "conv_store (carried inputs)")) return 1;
    }
    return 0;
}

RI_DEFINE_LAST_ERROR()
