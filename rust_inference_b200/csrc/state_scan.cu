// Recurrent mixers with a matrix state per head and ONE decay per head and token: the selective state space
// (scalar decay, the form its authors call state-space duality) and the gated delta rule.  Per head, with the state
// S [dim, vdim] in float32, the decay a_t, a key k_t [dim], a query q_t [dim], a value v_t [vdim] and a step s_t:
//
//     state space    S <- a S + k (s v)^T                      o = S^T q + skip * v
//     delta rule     S <- a S;  u = s (v - S^T k);  S <- S + k u^T      o = S^T q
//
// The delta rule also comes with a decay per key channel, S <- diag(a) S with a in [0, 1]^dim, which a low-rank map of the
// layer's input gives; the state space's form also with a decay per head that never changes and s = 1 (linear attention
// with a fixed decay).
//
// (state space: k = B, q = C, v = x, s = dt, a = exp(-exp(A_log) dt);  delta rule: s = beta, a = exp(-exp(A_log)
// softplus(.)); the read-out sees the token's own write.)  Heads share keys and queries in groups.  The state lives in
// a per-slot area of the cache, starts at zero when a slot is handed out and is carried from step to step; so do the
// last taps - 1 inputs of the short causal convolutions that come before the recurrence.  A prompt may therefore be
// cut anywhere, and a decode step is the same kernels with one token per sequence.
//
// Four kernels, all reading the step's arrays on the device (graph-safe), everything float32:
//   prepare     per token: the short convolution (+ bias) and silu over a range of the projection's columns; unit
//               vectors x / sqrt(sum x^2 + 1e-6) for the first heads of that range (the first of them times a factor);
//               the decay and the step of every head; decays per key channel from their low-rank input (steps of few
//               tokens, which also get a low-rank gate here) or from products formed before.  In a step of one token
//               per sequence it moves the carried inputs on as well
//   conv_state  per (sequence, channel): the convolution's carried inputs move on by the step's tokens
//   scan        per (sequence, head, tile of value columns): the recurrence over the sequence's new tokens in
//               order; the state is read first and written last
//   finish      per (token, group of channels): RMS norm over the group and a silu or sigmoid gate, before or after the norm
//
// What an earlier kernel of the step wrote is read after `wait_for_previous_kernels()` through plain pointers.
#include "common.cuh"

using namespace ri;

namespace {

__device__ __forceinline__ float softplus_f32(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f32(float x) {
    if (x >= 0.f) return 1.f / (1.f + expf(-x));
    const float e = expf(x);
    return e / (1.f + e);
}

// V consecutive floats as one access (V = 4: 16 bytes; the address must allow it).
template <int V> struct Floats { float v[V]; };
template <int V> __device__ __forceinline__ Floats<V> load_floats(const float* p) {
    Floats<V> r;
    if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}

struct Prepare {
    const float* z;            // [tokens, ld] the projection's results
    int ld;
    int conv_col, conv_ch;     // the convolved columns of z
    const float* taps;         // [conv_ch, k_taps], the last column is the current token's
    const float* conv_bias;    // null: none
    int k_taps;
    float* conv_state;         // [slots, k_taps - 1, conv_ch]: the inputs before the step, oldest first
    int unit_heads, unit_dim;  // the first unit_heads * unit_dim convolved channels are made unit vectors per head
    int scaled_heads;          // the first of those heads are also multiplied by unit_scale
    float unit_scale;
    int heads;                 // heads with a decay
    int decay_col;             // column of z with the decay's raw step, per head
    int step_col;              // >= 0: column of z whose sigmoid is the step (delta rule); < 0: the step is softplus(raw + bias)
    const float* a_log;        // [heads]
    const float* dt_bias;      // [heads]
    float* out;                // [tokens, out_ld] = [convolved channels | decay per head | step per head]
    int out_ld;
    const int* cu_seqlens;
    const int* token_seq;
    const int* seq_slot;
    int tile_ch;               // convolved channels per block: a multiple of unit_dim where there are unit vectors
    int conv_tiles;            // tiles of convolved channels (blockIdx.y); further tiles hold CHANNEL_TILE low-rank channels each
    int single;                // 1: every sequence brings one token, and the carried inputs move on here
    // decays per key channel, exp(-exp(a_log[head]) softplus(raw + dt_bias[channel])): channels 0: one decay per head
    int channels, head_dim;
    const float* raw;          // [tokens, channels] the low-rank map's result (may be `decay`), or null: formed here
    float* decay;              // [tokens, channels]
    const void* w2;            // [channels, rank], in the run dtype
    int rank, low_col;         // the low-rank input's columns of z
    // the low-rank gate, formed here as well (gate_channels 0: not): gate_out = gate_w2 . z[gate_low_col ..]
    int gate_channels, gate_rank, gate_low_col;
    const void* gate_w2;
    float* gate_out;           // [tokens, gate_channels]
    int w2_bf16;
    int n_tokens;
};

constexpr int CHANNEL_TILE = 256;

// A row of a low-rank map (rank values in the run dtype) times the input in shared memory.
template <typename T>
__device__ __forceinline__ float low_rank_dot(const T* __restrict__ w, const float* a, int rank) {
    float acc0 = 0.f, acc1 = 0.f;
    constexpr int V = 16 / sizeof(T);
    if (rank % V == 0) {
        for (int r = 0; r < rank; r += V) {
            const uint4 pk = *reinterpret_cast<const uint4*>(w + r);
            const T* e = reinterpret_cast<const T*>(&pk);
#pragma unroll
            for (int k = 0; k < V; k += 2) {
                acc0 = fmaf(to_f32<T>(e[k]), a[r + k], acc0);
                acc1 = fmaf(to_f32<T>(e[k + 1]), a[r + k + 1], acc1);
            }
        }
    } else {
        for (int r = 0; r < rank; ++r) acc0 = fmaf(to_f32<T>(w[r]), a[r], acc0);
    }
    return acc0 + acc1;
}

// A block per (token, tile of p.tile_ch convolved channels); tiles hold whole heads of the unit vectors.  The first
// tile's block also writes the heads' decays and steps.
__global__ void __launch_bounds__(256) scan_prepare_kernel(Prepare p) {
    extern __shared__ float ch[];                 // [tile_ch]
    const int t = blockIdx.x;
    const int c0 = blockIdx.y * p.tile_ch, c1 = min(p.conv_ch, c0 + p.tile_ch);
    let_next_kernel_start();
    wait_for_previous_kernels();
    if ((int)blockIdx.y >= p.conv_tiles) {
        // low-rank channels: the decays', then the gate's; a tile holds channels of one of the two
        const int tiles = (p.channels + CHANNEL_TILE - 1) / CHANNEL_TILE;
        const int tile = (int)blockIdx.y - p.conv_tiles;
        const bool gate = tile >= tiles;
        const int c = (gate ? tile - tiles : tile) * CHANNEL_TILE + (int)threadIdx.x;
        const bool formed = gate || p.raw == nullptr;
        const int rank = gate ? p.gate_rank : p.rank;
        if (formed) {
            const float* low = p.z + (size_t)t * p.ld + (gate ? p.gate_low_col : p.low_col);
            for (int r = threadIdx.x; r < rank; r += blockDim.x) ch[r] = low[r];
            __syncthreads();
        }
        if (c >= (gate ? p.gate_channels : p.channels)) return;
        float v;
        if (formed) {
            const void* w = gate ? p.gate_w2 : p.w2;
            v = p.w2_bf16 ? low_rank_dot(reinterpret_cast<const __nv_bfloat16*>(w) + (size_t)c * rank, ch, rank)
                          : low_rank_dot(reinterpret_cast<const float*>(w) + (size_t)c * rank, ch, rank);
        } else {
            v = p.raw[(size_t)t * p.channels + c];
        }
        if (gate) p.gate_out[(size_t)t * p.gate_channels + c] = v;
        else p.decay[(size_t)t * p.channels + c] = expf(-expf(p.a_log[c / p.head_dim]) * softplus_f32(v + p.dt_bias[c]));
        return;
    }
    const int b = p.token_seq[t];
    const int i = t - p.cu_seqlens[b];            // place among the sequence's new tokens
    int slot = p.seq_slot[b];
    if (!RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) slot = 0;
    const int K = p.k_taps;
    float* carried = p.conv_state + (size_t)slot * (K - 1) * p.conv_ch;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) {
        float acc = p.conv_bias != nullptr ? p.conv_bias[c] : 0.f;
        for (int k = 0; k < K; ++k) {             // the input k tokens back
            const int src = i - k;
            const float x = src >= 0 ? p.z[(size_t)(t - k) * p.ld + p.conv_col + c]
                                     : carried[(size_t)(K - 1 + src) * p.conv_ch + c];
            acc = fmaf(p.taps[(size_t)c * K + (K - 1 - k)], x, acc);
        }
        ch[c - c0] = silu_f32(acc);
        if (p.single && K > 1) {                  // the channel's inputs move on by this one token; only this thread has read them
            for (int s = 0; s < K - 2; ++s) carried[(size_t)s * p.conv_ch + c] = carried[(size_t)(s + 1) * p.conv_ch + c];
            carried[(size_t)(K - 2) * p.conv_ch + c] = p.z[(size_t)t * p.ld + p.conv_col + c];
        }
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    if (p.unit_heads > 0 && c0 < p.unit_heads * p.unit_dim) {
        const int h0 = c0 / p.unit_dim, h1 = min(p.unit_heads, c1 / p.unit_dim);     // tiles are multiples of unit_dim there
        for (int h = h0 + warp; h < h1; h += warps) {
            float* v = ch + (h - h0) * p.unit_dim;
            float ss = 0.f;
            for (int d = lane; d < p.unit_dim; d += 32) ss = fmaf(v[d], v[d], ss);
            ss = warp_sum(ss);
            const float f = (h < p.scaled_heads ? p.unit_scale : 1.f) / sqrtf(ss + 1e-6f);
            for (int d = lane; d < p.unit_dim; d += 32) v[d] *= f;
        }
        __syncthreads();
    }
    float* out = p.out + (size_t)t * p.out_ld;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) out[c] = ch[c - c0];
    if (blockIdx.y == 0)
        for (int h = threadIdx.x; h < p.heads; h += blockDim.x) {
            float dt = 0.f;
            if (p.channels == 0) {
                dt = softplus_f32(p.z[(size_t)t * p.ld + p.decay_col + h] + p.dt_bias[h]);
                out[p.conv_ch + h] = expf(-expf(p.a_log[h]) * dt);
            }
            out[p.conv_ch + p.heads + h] = p.step_col >= 0 ? sigmoid_f32(p.z[(size_t)t * p.ld + p.step_col + h]) : dt;
        }
}

// The same for steps of many tokens: a block takes PREP_TOKENS consecutive tokens and p.tile_ch convolved channels.  A thread
// owns V neighbouring channels, keeps their filters in registers and walks down the tokens (a row it looks back at is one
// it has just read); channels that are made unit vectors go through shared memory, the rest straight out.  Further tiles
// turn the low-rank products in `raw` into decays.
constexpr int PREP_TOKENS = 8;
template <int V, int KT>
__global__ void __launch_bounds__(256) scan_prepare_rows_kernel(Prepare p) {
    extern __shared__ float ch[];                 // [PREP_TOKENS][tile_ch]
    const int t0 = blockIdx.x * PREP_TOKENS, t1 = min(p.n_tokens, t0 + PREP_TOKENS);
    let_next_kernel_start();
    if ((int)blockIdx.y >= p.conv_tiles) {
        const int c = ((int)blockIdx.y - p.conv_tiles) * CHANNEL_TILE + (int)threadIdx.x;
        const bool mine = c < p.channels;
        const float rate = mine ? -expf(p.a_log[c / p.head_dim]) : 0.f, bias = mine ? p.dt_bias[c] : 0.f;
        wait_for_previous_kernels();
        if (!mine) return;
        for (int t = t0; t < t1; ++t) p.decay[(size_t)t * p.channels + c] = expf(rate * softplus_f32(p.raw[(size_t)t * p.channels + c] + bias));
        return;
    }
    const int c0 = blockIdx.y * p.tile_ch, c1 = min(p.conv_ch, c0 + p.tile_ch);
    const int K = KT > 0 ? KT : p.k_taps, unit_end = p.unit_heads * p.unit_dim;
    wait_for_previous_kernels();
    for (int c = c0 + (int)threadIdx.x * V; c < c1; c += blockDim.x * V) {
        float f[KT > 0 ? KT * V : 1];
        if constexpr (KT > 0) {
#pragma unroll
            for (int i = 0; i < KT * V; ++i) f[i] = p.taps[(size_t)c * KT + i];
        }
        float bias[V];
#pragma unroll
        for (int k = 0; k < V; ++k) bias[k] = p.conv_bias != nullptr ? p.conv_bias[c + k] : 0.f;
        for (int t = t0; t < t1; ++t) {
            const int b = p.token_seq[t];
            const int i = t - p.cu_seqlens[b];
            int slot = p.seq_slot[b];
            if (!RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) slot = 0;
            const float* carried = p.conv_state + (size_t)slot * (K - 1) * p.conv_ch + c;
            float acc[V];
#pragma unroll
            for (int k = 0; k < V; ++k) acc[k] = bias[k];
#pragma unroll
            for (int j = 0; j < K; ++j) {         // the input j tokens back
                const float* src = i >= j ? p.z + (size_t)(t - j) * p.ld + p.conv_col + c : carried + (size_t)(K - 1 + i - j) * p.conv_ch;
                const Floats<V> x = load_floats<V>(src);
#pragma unroll
                for (int k = 0; k < V; ++k)
                    acc[k] = fmaf(KT > 0 ? f[KT > 0 ? k * KT + (KT - 1 - j) : 0] : p.taps[(size_t)(c + k) * K + (K - 1 - j)], x.v[k], acc[k]);
            }
            float* dst = c < unit_end ? ch + (t - t0) * p.tile_ch + (c - c0) : p.out + (size_t)t * p.out_ld + c;
#pragma unroll
            for (int k = 0; k < V; ++k) acc[k] = silu_f32(acc[k]);
            if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(acc[0], acc[1], acc[2], acc[3]);
            else *dst = acc[0];
        }
    }
    if (c0 < unit_end) {
        __syncthreads();
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
        const int h0 = c0 / p.unit_dim, heads = min(p.unit_heads, c1 / p.unit_dim) - h0;         // tiles are multiples of unit_dim there
        for (int it = warp; it < heads * (t1 - t0); it += warps) {
            const int tk = it / heads, h = h0 + it % heads;
            const float* v = ch + tk * p.tile_ch + (h - h0) * p.unit_dim;
            float ss = 0.f;
            for (int d = lane; d < p.unit_dim; d += 32) ss = fmaf(v[d], v[d], ss);
            ss = warp_sum(ss);
            const float f = (h < p.scaled_heads ? p.unit_scale : 1.f) / sqrtf(ss + 1e-6f);
            float* dst = p.out + (size_t)(t0 + tk) * p.out_ld + h * p.unit_dim;
            for (int d = lane; d < p.unit_dim; d += 32) dst[d] = v[d] * f;
        }
    }
    if (blockIdx.y == 0)
        for (int it = threadIdx.x; it < (t1 - t0) * p.heads; it += blockDim.x) {
            const int t = t0 + it / p.heads, h = it % p.heads;
            float* out = p.out + (size_t)t * p.out_ld + p.conv_ch;
            float dt = 0.f;
            if (p.channels == 0) {
                dt = softplus_f32(p.z[(size_t)t * p.ld + p.decay_col + h] + p.dt_bias[h]);
                out[h] = expf(-expf(p.a_log[h]) * dt);
            }
            out[p.heads + h] = p.step_col >= 0 ? sigmoid_f32(p.z[(size_t)t * p.ld + p.step_col + h]) : dt;
        }
}

__global__ void conv_state_kernel(const float* z, int ld, int conv_col, int conv_ch, int k_taps, float* conv_state,
                                  const int* cu_seqlens, const int* seq_slot) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int b = blockIdx.y;
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= conv_ch) return;
    const int t0 = cu_seqlens[b], n = cu_seqlens[b + 1] - t0;
    const int slot = seq_slot[b];
    if (n <= 0 || !RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) return;
    float* carried = conv_state + (size_t)slot * (k_taps - 1) * conv_ch;
    for (int s = 0; s < k_taps - 1; ++s) {        // ascending: an entry is read before a later round overwrites it
        const int src = n - (k_taps - 1) + s;
        carried[(size_t)s * conv_ch + c] = src >= 0 ? z[(size_t)(t0 + src) * ld + conv_col + c]
                                                    : carried[(size_t)(s + n) * conv_ch + c];
    }
}

// Threads of a warp: lane = column_in_warp * R + r.  Thread (r, j) keeps ROWS consecutive rows (r * ROWS ...) of
// column j of the state in registers; sums over the rows are finished by log2(R) shuffles inside the warp.  The
// tokens' keys, queries, values, decays and steps come through shared memory in tiles, a key's and a query's row
// slices padded so that the eight slices' 16-byte reads fall into different banks.  There are two tiles: while the
// recurrence runs over one, asynchronous copies (16 bytes each where every column offset and the row length are
// multiples of four floats, 4 bytes each otherwise) fill the other, so the global loads' latency stays off the
// sequential path.
constexpr int R = 8;
constexpr int SCAN_WARPS = 4;
constexpr int COLS = SCAN_WARPS * 32 / R;        // value columns per block
constexpr int SCAN_THREADS = SCAN_WARPS * 32;

__device__ __forceinline__ void copy_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct Scan {
    const float* u;            // [tokens, ld]: the prepared rows
    int ld;
    int q_col, k_col, v_col, decay_col, step_col;
    const float* decay;        // CHANNELS: [tokens, heads * dim], a decay per key channel; FIXED: [heads], decays that never change
    const float* skip;         // [heads] or null: o += skip * v
    float* state;              // [slots, heads, dim, vdim]
    float* o;                  // [tokens, heads * vdim]
    const int* cu_seqlens;
    const int* seq_slot;
    int heads, groups, dim, vdim, tile_t;
    int vec;                   // 1: rows, columns and sizes allow 16-byte copies
    int piece, max_pieces;     // passes over pieces: tokens per piece, most pieces of a sequence
    float* piece_state;        // [seqs, max_pieces, heads, dim, vdim]: a piece's end state from zero, then its start state
    float* piece_decay;        // [seqs, max_pieces, heads]: the product of a piece's decays
};

// How a launch of the scan treats its tokens.  WHOLE: a block runs over all new tokens of its sequence from the slot's
// state and writes the state back.  For long runs of the state space, whose update is linear in the state with a scalar
// factor, three launches work on pieces of a sequence side by side: LOCAL scans every piece from zero (no read-out) and
// keeps its end state and the product of its decays; a carry kernel walks the pieces of a sequence per state element,
// start(p + 1) = decays(p) * start(p) + end(p), leaving every piece's start state and the sequence's final state in the
// slot; FINAL scans every piece again from its start state and writes the read-outs.
enum { WHOLE = 0, LOCAL = 1, FINAL = 2 };

// Where the decays come from: PER_TOKEN a column per head beside the steps; CHANNELS (the delta rule) a row per token and
// head with a value per key channel; FIXED (not the delta rule) one number per head for all tokens, with step 1.
enum { PER_TOKEN = 0, CHANNELS = 1, FIXED = 2 };

template <int ROWS, bool DELTA, int MODE, int DECAY>
__global__ void __launch_bounds__(SCAN_THREADS) state_scan_kernel(Scan p) {
    constexpr int SLICE = ROWS + 4;
    constexpr int V_AT = (DECAY == CHANNELS ? 3 : 2) * R * SLICE;     // k, q (, decays), then the block's values, decay and step
    constexpr int TOKEN = V_AT + COLS + 4;
    extern __shared__ __align__(16) float tile[];          // two tiles of tile_t tokens
    const int b = MODE == WHOLE ? blockIdx.x : blockIdx.x / p.max_pieces, h = blockIdx.y, j0 = blockIdx.z * COLS;
    const int pc = MODE == WHOLE ? 0 : blockIdx.x % p.max_pieces;
    const int r = threadIdx.x % R, jj = threadIdx.x / R;
    const int j = j0 + jj, i0 = r * ROWS;
    const bool live = j < p.vdim;
    for (int i = threadIdx.x; i < 2 * p.tile_t * TOKEN; i += SCAN_THREADS) tile[i] = 0.f;
    const float skip = p.skip != nullptr ? p.skip[h] : 0.f;
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int t0 = p.cu_seqlens[b] + (MODE == WHOLE ? 0 : pc * p.piece);
    const int t1 = MODE == WHOLE ? p.cu_seqlens[b + 1] : min(p.cu_seqlens[b + 1], t0 + p.piece);
    const int slot = p.seq_slot[b];
    if (t0 >= t1 || !RI_BLOCK_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) return;
    float* S = MODE == WHOLE ? p.state + (((size_t)slot * p.heads + h) * p.dim) * p.vdim
                             : p.piece_state + ((((size_t)b * p.max_pieces + pc) * p.heads + h) * p.dim) * p.vdim;
    constexpr int PAIRS = ROWS / 2;                        // two neighbouring rows at a time through the packed float32 pipe
    float2 s[PAIRS];
#pragma unroll
    for (int k = 0; k < ROWS; ++k) (k & 1 ? s[k / 2].y : s[k / 2].x) = (MODE != LOCAL && live && i0 + k < p.dim) ? S[(size_t)(i0 + k) * p.vdim + j] : 0.f;
    float decays = 1.f, v_before = 0.f;
    float2 q_before[PAIRS];
#pragma unroll
    for (int k = 0; k < PAIRS; ++k) q_before[k] = make_float2(0.f, 0.f);
    const float fixed = DECAY == FIXED ? p.decay[h] : 1.f;
    const int g = h / (p.heads / p.groups);
    const int q_off = p.q_col + g * p.dim, k_off = p.k_col + g * p.dim, v_off = p.v_col + h * p.vdim + j0;
    const int cols = min(COLS, p.vdim - j0);
    const int o_ld = p.heads * p.vdim;
    __syncthreads();                                      // the zeros are in place

    // A token's 16-byte pieces are shared out among the threads once, and a thread copies its piece of every token: where it
    // starts, how far the next token's lies, and its place in a token's part of the tile (-1: no piece).
    constexpr int ITEMS = ROWS <= 16 ? 1 : 2;
    const float* item_src[ITEMS];
    int item_step[ITEMS], item_at[ITEMS];
#pragma unroll
    for (int m = 0; m < ITEMS; ++m) {
        const int it = threadIdx.x + m * SCAN_THREADS;
        const int dq = p.dim >> 2, parts = DECAY == CHANNELS ? 3 : 2;
        const int part = dq > 0 ? it / dq : parts, c = 4 * (it - part * dq);
        item_src[m] = p.u;
        item_step[m] = p.ld;
        item_at[m] = -1;
        if (part < parts) {
            item_at[m] = part * R * SLICE + c / ROWS * SLICE + c % ROWS;
            item_src[m] = part == 0 ? p.u + k_off + c : part == 1 ? p.u + q_off + c : p.decay + (size_t)h * p.dim + c;
            if (part == 2) item_step[m] = p.heads * p.dim;
        } else if (it < parts * dq + (cols >> 2)) {
            const int cc = 4 * (it - parts * dq);
            item_at[m] = V_AT + cc;
            item_src[m] = p.u + v_off + cc;
        }
    }
    // the copies of the tokens tb .. tb + n_tok - 1 into one of the two tiles; every thread commits one group
    auto fetch = [&](float* dst, int tb, int n_tok) {
        if (p.vec) {
#pragma unroll
            for (int m = 0; m < ITEMS; ++m)
                if (item_at[m] >= 0)
                    for (int tok = 0; tok < n_tok; ++tok)
                        copy_async16(dst + tok * TOKEN + item_at[m], item_src[m] + (size_t)(tb + tok) * item_step[m]);
        } else {
            const int parts = DECAY == CHANNELS ? 3 : 2, per = parts * p.dim + cols;
            for (int tok = 0; tok < n_tok; ++tok) {
                const float* row = p.u + (size_t)(tb + tok) * p.ld;
                float* base = dst + tok * TOKEN;
                for (int it = threadIdx.x; it < per; it += SCAN_THREADS) {
                    if (it < p.dim) copy_async4(base + (it / ROWS) * SLICE + it % ROWS, row + k_off + it);
                    else if (it < 2 * p.dim) copy_async4(base + R * SLICE + ((it - p.dim) / ROWS) * SLICE + (it - p.dim) % ROWS, row + q_off + it - p.dim);
                    else if (DECAY == CHANNELS && it < 3 * p.dim) copy_async4(base + 2 * R * SLICE + ((it - 2 * p.dim) / ROWS) * SLICE + (it - 2 * p.dim) % ROWS, p.decay + ((size_t)(tb + tok) * p.heads + h) * p.dim + it - 2 * p.dim);
                    else copy_async4(base + V_AT + it - parts * p.dim, row + v_off + it - parts * p.dim);
                }
            }
        }
        if (DECAY == PER_TOKEN)
            for (int tok = threadIdx.x; tok < 2 * n_tok; tok += SCAN_THREADS) {      // decay and step of every token
                const int tk = tok >> 1, which = tok & 1;
                copy_async4(dst + tk * TOKEN + V_AT + COLS + which,
                            p.u + (size_t)(tb + tk) * p.ld + (which ? p.step_col : p.decay_col) + h);
            }
        if (DECAY == CHANNELS)
            for (int tk = threadIdx.x; tk < n_tok; tk += SCAN_THREADS)
                copy_async4(dst + tk * TOKEN + V_AT + COLS + 1, p.u + (size_t)(tb + tk) * p.ld + p.step_col + h);
        copy_async_commit();
    };

    const int tile_floats = p.tile_t * TOKEN;
    fetch(tile, t0, min(p.tile_t, t1 - t0));
    int buf = 0;
    for (int tb = t0; tb < t1; tb += p.tile_t, buf ^= 1) {
        const int n_tok = min(p.tile_t, t1 - tb);
        const int nb = tb + p.tile_t;
        if (nb < t1) {                                    // the next tile is on its way while this one is used
            fetch(tile + (buf ^ 1) * tile_floats, nb, min(p.tile_t, t1 - nb));
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        const float* cur = tile + buf * tile_floats;
        // Only the state chains the tokens.  What a token reads of the state before its own update (the delta rule's
        // S^T k) and the read-out of the token before (which wants the state after that one's update) are sums over the same
        // values, so they are formed together and their shuffles overlap; S^T k of the decayed state is taken as S^T (a k).
        // Unrolled, a token's loads overlap the token before.
#pragma unroll(DELTA ? 2 : 4)
        for (int tok = 0; tok < n_tok; ++tok) {
            const float* base = cur + tok * TOKEN;
            const float4* k4 = reinterpret_cast<const float4*>(base + r * SLICE);
            const float4* q4 = reinterpret_cast<const float4*>(base + R * SLICE + r * SLICE);
            const float4* a4 = reinterpret_cast<const float4*>(base + 2 * R * SLICE + r * SLICE);      // CHANNELS only
            const float v = base[V_AT + jj];
            const float a = DECAY == FIXED ? fixed : DECAY == CHANNELS ? 1.f : base[V_AT + COLS];
            const float step = DECAY == FIXED ? 1.f : base[V_AT + COLS + 1];
            float2 kk[PAIRS], qq[PAIRS], aa[PAIRS];
#pragma unroll
            for (int k = 0; k < ROWS / 4; ++k) {
                const float4 kv = k4[k];
                kk[2 * k] = make_float2(kv.x, kv.y); kk[2 * k + 1] = make_float2(kv.z, kv.w);
                if (MODE != LOCAL) {
                    const float4 qv = q4[k];
                    qq[2 * k] = make_float2(qv.x, qv.y); qq[2 * k + 1] = make_float2(qv.z, qv.w);
                }
                if (DECAY == CHANNELS) {
                    const float4 av = a4[k];
                    aa[2 * k] = make_float2(av.x, av.y); aa[2 * k + 1] = make_float2(av.z, av.w);
                }
            }
            if (MODE == LOCAL) decays *= a;
            float2 d2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)}, e2[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
            for (int k = 0; k < PAIRS; ++k) {
                if (DELTA) d2[k & 1] = __ffma2_rn(s[k], DECAY == CHANNELS ? __fmul2_rn(aa[k], kk[k]) : kk[k], d2[k & 1]);
                if (MODE != LOCAL) e2[k & 1] = __ffma2_rn(s[k], q_before[k], e2[k & 1]);
            }
            d2[0] = __fadd2_rn(d2[0], d2[1]);
            e2[0] = __fadd2_rn(e2[0], e2[1]);
            float dot = d2[0].x + d2[0].y, acc = e2[0].x + e2[0].y;
#pragma unroll
            for (int o = R / 2; o > 0; o >>= 1) {
                if (DELTA) dot += __shfl_xor_sync(0xffffffffu, dot, o);
                if (MODE != LOCAL) acc += __shfl_xor_sync(0xffffffffu, acc, o);
            }
            if (MODE != LOCAL) {
                if (live && r == 0 && tb + tok > t0) p.o[(size_t)(tb + tok - 1) * o_ld + h * p.vdim + j] = fmaf(skip, v_before, acc);
                v_before = v;
            }
            const float write = DELTA ? step * (v - (DECAY == CHANNELS ? dot : a * dot)) : step * v;
            const float2 write2 = make_float2(write, write), keep2 = make_float2(a, a);
#pragma unroll
            for (int k = 0; k < PAIRS; ++k) {
                s[k] = __ffma2_rn(DECAY == CHANNELS ? aa[k] : keep2, s[k], __fmul2_rn(kk[k], write2));
                if (MODE != LOCAL) q_before[k] = qq[k];
            }
        }
        __syncthreads();                                  // this tile may be overwritten by the fetch after next
    }
    if (MODE != LOCAL) {                                  // the last token's read-out
        float2 e2 = make_float2(0.f, 0.f);
#pragma unroll
        for (int k = 0; k < PAIRS; ++k) e2 = __ffma2_rn(s[k], q_before[k], e2);
        float acc = e2.x + e2.y;
#pragma unroll
        for (int o = R / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (live && r == 0) p.o[(size_t)(t1 - 1) * o_ld + h * p.vdim + j] = fmaf(skip, v_before, acc);
    }
    if constexpr (MODE != FINAL) {                        // there the carry kernel left the final state in the slot
#pragma unroll
        for (int k = 0; k < ROWS; ++k)
            if (live && i0 + k < p.dim) S[(size_t)(i0 + k) * p.vdim + j] = k & 1 ? s[k / 2].y : s[k / 2].x;
    }
    if (MODE == LOCAL && blockIdx.z == 0 && threadIdx.x == 0) p.piece_decay[((size_t)b * p.max_pieces + pc) * p.heads + h] = decays;
}

// Per (sequence, head, state element): the pieces' start states from their end states and decay products; the
// sequence's final state goes to the slot.
__global__ void __launch_bounds__(256) scan_carry_kernel(float* state, float* piece_state, const float* piece_decay,
                                                         const int* cu_seqlens, const int* seq_slot, int heads, int per_head,
                                                         int piece, int max_pieces) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int b = blockIdx.z, h = blockIdx.y;
    const int e = blockIdx.x * blockDim.x + threadIdx.x;
    const int n = cu_seqlens[b + 1] - cu_seqlens[b];
    const int slot = seq_slot[b];
    if (e >= per_head || n <= 0 || !RI_IN_LIMIT(slot, RI_LIMIT_SLOTS, RI_CHECK_SLOT)) return;
    const int pieces = (n + piece - 1) / piece;
    float* dst = state + ((size_t)slot * heads + h) * per_head + e;
    float s = *dst;
    // several pieces' loads are in flight before the first of their stores
    constexpr int AHEAD = 8;
    const size_t piece_step = (size_t)heads * per_head;
    float* ps = piece_state + ((size_t)b * max_pieces * heads + h) * per_head + e;
    const float* pd = piece_decay + (size_t)b * max_pieces * heads + h;
    for (int pc = 0; pc < pieces; pc += AHEAD) {
        float local[AHEAD], keep[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            local[i] = pc + i < pieces ? ps[(size_t)(pc + i) * piece_step] : 0.f;
            keep[i] = pc + i < pieces ? pd[(size_t)(pc + i) * heads] : 1.f;
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (pc + i < pieces) {
                ps[(size_t)(pc + i) * piece_step] = s;
                s = fmaf(keep[i], s, local[i]);
            }
    }
    *dst = s;
}

__device__ __forceinline__ float gate_f32(float x, int sigmoid) { return sigmoid ? sigmoid_f32(x) : silu_f32(x); }

// One warp per (token, group of `gs` channels): with gate_first the channels are multiplied by silu(gate) and then
// normalised, otherwise normalised and then multiplied (sigmoid != 0: by sigmoid(gate)); the weight of channel c of a token's row is w[c % w_len].
template <typename T>
__global__ void gated_group_norm_kernel(const float* x, int x_ld, const float* gate, int gate_ld, int gate_col,
                                        const float* __restrict__ w, int w_len, T* __restrict__ out, int n_tokens, int groups,
                                        int gs, int gate_first, int sigmoid, float eps, float out_scale) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (warp >= n_tokens * groups) return;
    const int t = warp / groups, g = warp % groups;
    const float* src = x + (size_t)t * x_ld + g * gs;
    const float* gt = gate + (size_t)t * gate_ld + gate_col + g * gs;
    float ss = 0.f;
    for (int d = lane; d < gs; d += 32) {
        const float v = gate_first ? src[d] * gate_f32(gt[d], sigmoid) : src[d];
        ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    const float inv = out_scale / sqrtf(ss / (float)gs + eps);
    T* dst = out + ((size_t)t * groups + g) * gs;
    for (int d = lane; d < gs; d += 32) {
        const float sg = gate_f32(gt[d], sigmoid);
        const float v = gate_first ? src[d] * sg : src[d];
        const float y = v * inv * w[(g * gs + d) % w_len];
        dst[d] = from_f32<T>(gate_first ? y : y * sg);
    }
}

// The same with a block per (token, group), for groups of many channels; V = 4: 16 bytes at a time, where rows, columns
// and the weight's length allow.
template <typename T, int V>
__global__ void __launch_bounds__(1024) gated_group_norm_block_kernel(const float* x, int x_ld, const float* gate, int gate_ld, int gate_col,
                                        const float* __restrict__ w, int w_len, T* __restrict__ out, int groups,
                                        int gs, int gate_first, int sigmoid, float eps, float out_scale) {
    __shared__ float scratch[33];
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int t = blockIdx.x / groups, g = blockIdx.x % groups;
    const float* src = x + (size_t)t * x_ld + g * gs;
    const float* gt = gate + (size_t)t * gate_ld + gate_col + g * gs;
    // the thread's first run of channels stays in registers; wider groups read the rest again
    Floats<V> x0, g0;
    float ss = 0.f;
    for (int d = threadIdx.x * V; d < gs; d += blockDim.x * V) {
        Floats<V> xv = load_floats<V>(src + d), gv = load_floats<V>(gt + d);
#pragma unroll
        for (int k = 0; k < V; ++k) {
            gv.v[k] = gate_f32(gv.v[k], sigmoid);
            const float v = gate_first ? xv.v[k] * gv.v[k] : xv.v[k];
            ss = fmaf(v, v, ss);
        }
        if (d == (int)threadIdx.x * V) { x0 = xv; g0 = gv; }
    }
    ss = block_sum(ss, scratch);
    const float inv = out_scale / sqrtf(ss / (float)gs + eps);
    T* dst = out + ((size_t)t * groups + g) * gs;
    for (int d = threadIdx.x * V; d < gs; d += blockDim.x * V) {
        Floats<V> xv = x0, gv = g0;
        if (d != (int)threadIdx.x * V) {
            xv = load_floats<V>(src + d);
            gv = load_floats<V>(gt + d);
#pragma unroll
            for (int k = 0; k < V; ++k) gv.v[k] = gate_f32(gv.v[k], sigmoid);
        }
        const Floats<V> wv = load_floats<V>(w + (g * gs + d) % w_len);
        float y[V];
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] = xv.v[k] * gv.v[k] * inv * wv.v[k];
        if constexpr (V == 4 && sizeof(T) == 2) {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(y[0], y[1]), hi = __floats2bfloat162_rn(y[2], y[3]);
            uint2 pk;
            pk.x = *reinterpret_cast<const uint32_t*>(&lo);
            pk.y = *reinterpret_cast<const uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(dst + d) = pk;
        } else if constexpr (V == 4) {
            *reinterpret_cast<float4*>(dst + d) = make_float4(y[0], y[1], y[2], y[3]);
        } else {
            dst[d] = from_f32<T>(y[0]);
        }
    }
}

constexpr int SCAN_SMEM_LIMIT = 44 * 1024;
constexpr int SCAN_SMEM_MOST = 216 * 1024;        // of an SM's 228 KB, with a kilobyte of the system's per block
constexpr int SMS = 148;

template <int ROWS, bool DELTA, int DECAY>
int launch_scan(dim3 grid, cudaStream_t stream, Scan p, int longest, int n_seqs) {
    const int token_bytes = ((DECAY == CHANNELS ? 3 : 2) * R * (ROWS + 4) + COLS + 4) * (int)sizeof(float);
    // A long one-pass scan is as slow as its most crowded SM.  Its blocks come onto the SMs while the kernel before still holds
    // some of them, so blocks are kept apart by their shared memory: no more fit an SM than it gets when all are spread evenly
    // (and the tiles are larger for it).
    const long long blocks = (long long)grid.x * grid.y * grid.z;
    const bool apart = p.piece <= 0 && longest >= 64 && blocks <= 4 * SMS;
    const int per_sm = (int)((blocks + SMS - 1) / SMS);
    const int budget = apart ? SCAN_SMEM_MOST / per_sm : SCAN_SMEM_LIMIT;
    int tile_t = budget / (2 * token_bytes);              // two tiles
    if (tile_t > (apart ? 32 : 16)) tile_t = apart ? 32 : 16;
    if (longest > 0 && tile_t > longest) tile_t = longest;
    if (tile_t < 1) tile_t = 1;
    p.tile_t = tile_t;
    size_t smem = (size_t)2 * tile_t * token_bytes;
    cudaError_t e;
    if (apart) {
        const size_t least = (size_t)(SCAN_SMEM_MOST / (per_sm + 1) + 8 * 1024);       // one block more would not fit
        if (smem < least) smem = least;
        static PerDeviceOnce once;
        if (int rc = raise_dynamic_smem(state_scan_kernel<ROWS, DELTA, WHOLE, DECAY>, SCAN_SMEM_MOST, once, "state_scan")) return rc;
    }
    if constexpr (!DELTA) {
        if (p.piece > 0) {
            const dim3 pieces(grid.x * p.max_pieces, grid.y, grid.z);
            e = launch_dependent(state_scan_kernel<ROWS, false, LOCAL, DECAY>, pieces, SCAN_THREADS, smem, stream, p);
            if (check_launch(e, "state_scan (pieces from zero)")) return 1;
            const int per_head = p.dim * p.vdim;
            e = launch_dependent(scan_carry_kernel, dim3((per_head + 255) / 256, p.heads, n_seqs), 256, 0, stream, p.state, p.piece_state,
                                 (const float*)p.piece_decay, p.cu_seqlens, p.seq_slot, p.heads, per_head, p.piece, p.max_pieces);
            if (check_launch(e, "state_scan (carry)")) return 1;
            e = launch_dependent(state_scan_kernel<ROWS, false, FINAL, DECAY>, pieces, SCAN_THREADS, smem, stream, p);
            return check_launch(e, "state_scan");
        }
    }
    e = launch_dependent(state_scan_kernel<ROWS, DELTA, WHOLE, DECAY>, grid, SCAN_THREADS, smem, stream, p);
    return check_launch(e, "state_scan");
}

template <int ROWS>
int pick_scan(bool delta, int decay, dim3 grid, cudaStream_t stream, Scan p, int longest, int n_seqs) {
    if (delta) return decay == CHANNELS ? launch_scan<ROWS, true, CHANNELS>(grid, stream, p, longest, n_seqs)
                                        : launch_scan<ROWS, true, PER_TOKEN>(grid, stream, p, longest, n_seqs);
    return decay == FIXED ? launch_scan<ROWS, false, FIXED>(grid, stream, p, longest, n_seqs)
                          : launch_scan<ROWS, false, PER_TOKEN>(grid, stream, p, longest, n_seqs);
}

}  // namespace

// A step's decays per key channel and its low-rank gate: see `Prepare`.  channels 0: none of it.
struct LowRank {
    int channels, head_dim;
    const float* raw;
    float* decay;
    const void* w2;
    int rank, low_col, gate_channels, gate_rank, gate_low_col;
    const void* gate_w2;
    float* gate_out;
    int w2_bf16;
};

static int scan_prepare(const float* z, int ld, int conv_col, int conv_ch, const float* taps, const float* conv_bias, int k_taps,
                        float* conv_state, int unit_heads, int unit_dim, int scaled_heads, float unit_scale, int heads,
                        int decay_col, int step_col, const float* a_log, const float* dt_bias, float* out, int out_ld,
                        const int* cu_seqlens, const int* token_seq, const int* seq_slot, int n_tokens, int n_seqs,
                        int longest_run, const LowRank& low, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (k_taps < 1 || conv_ch < 1) return fail("scan_prepare: a convolution of %d taps over %d channels", k_taps, conv_ch);
    if (conv_col < 0 || conv_col + conv_ch > ld || decay_col + (low.channels ? 0 : heads) > ld || step_col + heads > ld)
        return fail("scan_prepare: columns beyond the projection's %d", ld);
    if (unit_heads * unit_dim > conv_ch || scaled_heads > unit_heads) return fail("scan_prepare: unit vectors beyond the convolved channels");
    if (out_ld < conv_ch + 2 * heads) return fail("scan_prepare: output rows of %d values are too short", out_ld);
    // tiles of about 512 channels; where heads are made unit vectors a tile holds whole heads (a head wider than that
    // is a tile of its own)
    int tile_ch = 512;
    if (unit_heads > 0 && unit_dim > 0) tile_ch = unit_dim * ((512 + unit_dim - 1) / unit_dim);
    if (tile_ch > conv_ch) tile_ch = conv_ch;
    int shared_floats = tile_ch;
    const bool formed = low.channels > 0 && low.raw == nullptr;
    if (formed && low.rank > shared_floats) shared_floats = low.rank;
    if (low.gate_channels > 0 && low.gate_rank > shared_floats) shared_floats = low.gate_rank;
    const size_t smem = (size_t)shared_floats * sizeof(float);
    if (smem > 200 * 1024) return fail("scan_prepare: heads of %d channels do not fit shared memory", unit_dim);
    static PerDeviceOnce once;
    if (smem > 48 * 1024)
        if (int rc = raise_dynamic_smem(scan_prepare_kernel, 200 * 1024, once, "scan_prepare")) return rc;
    const int conv_tiles = (conv_ch + tile_ch - 1) / tile_ch;
    const int tiles = conv_tiles + (low.channels + CHANNEL_TILE - 1) / CHANNEL_TILE + (low.gate_channels + CHANNEL_TILE - 1) / CHANNEL_TILE;
    if (tiles > 65535) return fail("scan_prepare: %d tiles of channels exceed the grid limit", tiles);
    const int single = longest_run == 1 ? 1 : 0;
    Prepare p{z, ld, conv_col, conv_ch, taps, conv_bias, k_taps, conv_state, unit_heads, unit_dim, scaled_heads, unit_scale,
              heads, decay_col, step_col, a_log, dt_bias, out, out_ld, cu_seqlens, token_seq, seq_slot, tile_ch, conv_tiles, single,
              low.channels, low.head_dim, low.raw, low.decay, low.w2, low.rank, low.low_col, low.gate_channels, low.gate_rank,
              low.gate_low_col, low.gate_w2, low.gate_out, low.w2_bf16, n_tokens};
    cudaError_t e;
    // many tokens, the low-rank maps (if any) as products: several tokens per block
    int rows_ch = unit_heads > 0 && unit_dim > 0 ? unit_dim * ((1024 + unit_dim - 1) / unit_dim) : 1024;
    if (rows_ch > conv_ch) rows_ch = (conv_ch + 3) / 4 * 4;
    const size_t rows_smem = unit_heads > 0 ? (size_t)PREP_TOKENS * rows_ch * sizeof(float) : 0;
    if (n_tokens >= 64 * PREP_TOKENS && !formed && low.gate_channels == 0 && rows_smem <= 48 * 1024) {
        p.tile_ch = rows_ch;
        p.conv_tiles = (conv_ch + rows_ch - 1) / rows_ch;
        const dim3 grid((n_tokens + PREP_TOKENS - 1) / PREP_TOKENS, p.conv_tiles + (low.channels + CHANNEL_TILE - 1) / CHANNEL_TILE);
        const bool vec = (ld | conv_col | conv_ch | out_ld | rows_ch | (unit_heads * unit_dim)) % 4 == 0 &&
                         ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(conv_state)) & 15) == 0;
#define RI_PREP(V) (k_taps == 2 ? launch_dependent(scan_prepare_rows_kernel<V, 2>, grid, 256, rows_smem, stream, p)   \
                    : k_taps == 3 ? launch_dependent(scan_prepare_rows_kernel<V, 3>, grid, 256, rows_smem, stream, p) \
                    : k_taps == 4 ? launch_dependent(scan_prepare_rows_kernel<V, 4>, grid, 256, rows_smem, stream, p) \
                                  : launch_dependent(scan_prepare_rows_kernel<V, 0>, grid, 256, rows_smem, stream, p))
        e = vec ? RI_PREP(4) : RI_PREP(1);
#undef RI_PREP
    } else {
        e = launch_dependent(scan_prepare_kernel, dim3(n_tokens, tiles), 256, smem, stream, p);
    }
    if (check_launch(e, "scan_prepare")) return 1;
    if (k_taps > 1 && !single) {
        dim3 grid((conv_ch + 127) / 128, n_seqs);
        e = launch_dependent(conv_state_kernel, grid, 128, 0, stream, z, ld, conv_col, conv_ch, k_taps, conv_state, cu_seqlens, seq_slot);
        if (check_launch(e, "scan_prepare (carried inputs)")) return 1;
    }
    return 0;
}

// longest_run: the most new tokens any sequence brings (0: unknown); in a step of one token per sequence the carried inputs
// move on in the same kernel.
RI_API int ri_scan_prepare(const float* z, int ld, int conv_col, int conv_ch, const float* taps, const float* conv_bias,
                           int k_taps, float* conv_state, int unit_heads, int unit_dim, int scaled_heads, float unit_scale,
                           int heads, int decay_col, int step_col, const float* a_log, const float* dt_bias, float* out,
                           int out_ld, const int* cu_seqlens, const int* token_seq, const int* seq_slot, int n_tokens,
                           int n_seqs, int longest_run, cudaStream_t stream) {
    return scan_prepare(z, ld, conv_col, conv_ch, taps, conv_bias, k_taps, conv_state, unit_heads, unit_dim, scaled_heads, unit_scale,
                        heads, decay_col, step_col, a_log, dt_bias, out, out_ld, cu_seqlens, token_seq, seq_slot, n_tokens, n_seqs,
                        longest_run, LowRank{}, stream);
}

// The same with a decay per key channel, decay[t, c] = exp(-exp(a_log[c / head_dim]) softplus(x[t, c] + dt_bias[c])) for
// heads * head_dim channels.  x: `raw` (float32 [n_tokens, channels], may be `decay`), or with raw null w2 . z[t, low_col ..]
// formed here (w2 [channels, rank] in `w2_dtype`, rows on 16-byte boundaries where rank allows).  gate_channels > 0:
// gate_out[t, c] = gate_w2 . z[t, gate_low_col ..] as well.
RI_API int ri_scan_prepare_channels(const float* z, int ld, int conv_col, int conv_ch, const float* taps, const float* conv_bias,
                                    int k_taps, float* conv_state, int unit_heads, int unit_dim, int scaled_heads,
                                    float unit_scale, int heads, int step_col, const float* a_log, const float* dt_bias,
                                    float* out, int out_ld, const int* cu_seqlens, const int* token_seq, const int* seq_slot,
                                    int n_tokens, int n_seqs, int longest_run, int head_dim, const float* raw, float* decay,
                                    const void* w2, int rank, int low_col, int gate_channels, int gate_rank, int gate_low_col,
                                    const void* gate_w2, float* gate_out, int w2_dtype, cudaStream_t stream) {
    if (heads < 1 || head_dim < 1 || decay == nullptr) return fail("scan_prepare: decays of %d heads of %d channels", heads, head_dim);
    if (raw == nullptr && (w2 == nullptr || rank < 1 || low_col < 0 || low_col + rank > ld || (uintptr_t)w2 % 16))
        return fail("scan_prepare: a low-rank map of rank %d at column %d of %d", rank, low_col, ld);
    if (gate_channels > 0 && (gate_w2 == nullptr || gate_out == nullptr || gate_rank < 1 || gate_low_col < 0 ||
                              gate_low_col + gate_rank > ld || (uintptr_t)gate_w2 % 16))
        return fail("scan_prepare: a low-rank gate of rank %d at column %d of %d", gate_rank, gate_low_col, ld);
    if (w2_dtype != RI_F32 && w2_dtype != RI_BF16) return fail("scan_prepare: unknown dtype %d", w2_dtype);
    const LowRank low{heads * head_dim, head_dim, raw, decay, w2, rank, low_col, gate_channels, gate_rank, gate_low_col, gate_w2,
                      gate_out, w2_dtype == RI_BF16 ? 1 : 0};
    return scan_prepare(z, ld, conv_col, conv_ch, taps, conv_bias, k_taps, conv_state, unit_heads, unit_dim, scaled_heads, unit_scale,
                        heads, 0, step_col, a_log, dt_bias, out, out_ld, cu_seqlens, token_seq, seq_slot, n_tokens, n_seqs,
                        longest_run, low, stream);
}

// `rank` columns of z at low_col as a matrix of their own for a product with the low-rank map.  bfloat16: out [n_tokens, 2 *
// padded]: the value rounded and, in the second half, the rounding of the remainder (the map's matrix stands there twice
// side by side, so the product keeps 16 significant bits of the input); float32: out [n_tokens, padded].  Columns from rank
// to padded are zero.
namespace {
template <typename T>
__global__ void low_rank_rows_kernel(const float* z, int ld, int low_col, int rank, int padded, T* __restrict__ out, int n_tokens) {
    let_next_kernel_start();
    wait_for_previous_kernels();
    const int total = n_tokens * padded;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x) {
        const int t = i / padded, r = i % padded;
        const float v = r < rank ? z[(size_t)t * ld + low_col + r] : 0.f;
        if constexpr (sizeof(T) == 4) {
            out[i] = v;
        } else {
            const T hi = from_f32<T>(v);
            out[(size_t)t * 2 * padded + r] = hi;
            out[(size_t)t * 2 * padded + padded + r] = from_f32<T>(v - to_f32<T>(hi));
        }
    }
}
}  // namespace

RI_API int ri_low_rank_rows(const float* z, int ld, int low_col, int rank, int padded, void* out, int dtype, int n_tokens,
                            cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank < 1 || padded < rank || low_col < 0 || low_col + rank > ld || (long long)n_tokens * padded > 0x7fffffffLL)
        return fail("low_rank_rows: %d (%d) columns at %d of %d", rank, padded, low_col, ld);
    const int blocks = (int)(((long long)n_tokens * padded + 255) / 256 < 1184 ? ((long long)n_tokens * padded + 255) / 256 : 1184);
    cudaError_t e;
    if (dtype == RI_F32)
        e = launch_dependent(low_rank_rows_kernel<float>, blocks, 256, 0, stream, z, ld, low_col, rank, padded, (float*)out, n_tokens);
    else if (dtype == RI_BF16)
        e = launch_dependent(low_rank_rows_kernel<__nv_bfloat16>, blocks, 256, 0, stream, z, ld, low_col, rank, padded, (__nv_bfloat16*)out, n_tokens);
    else
        return fail("low_rank_rows: unknown dtype %d", dtype);
    return check_launch(e, "low_rank_rows");
}

// u: float32 [n_tokens, ld] with the columns of queries and keys ([groups, dim] each), values ([heads, vdim]), decays and
// steps ([heads] each).  state: float32 [slots, heads, dim, vdim].  o: float32 [n_tokens, heads * vdim].
// delta != 0: the gated delta rule; else the state space (with skip [heads] or null).  longest_run: the most new tokens
// any sequence brings (0: unknown), which sizes the scan's shared memory.  piece > 0 (state space only): the three passes
// over pieces of that many tokens, with scratch piece_state [n_seqs, max_pieces, heads, dim, vdim] and piece_decay
// [n_seqs, max_pieces, heads]; max_pieces * piece covers the longest run.  `decay` null: decays at decay_col; else, for the
// delta rule, a decay per key channel (float32 [n_tokens, heads * dim]; decay_col is not read), for the state space a decay
// per head that never changes (float32 [heads]; the step is 1, and neither decay_col nor step_col is read).
RI_API int ri_state_scan(const float* u, int ld, int q_col, int k_col, int v_col, int decay_col, int step_col, const float* decay,
                         const float* skip, float* state, float* o, const int* cu_seqlens, const int* seq_slot, int n_seqs,
                         int heads, int groups, int dim, int vdim, int delta, int longest_run, int piece, int max_pieces,
                         float* piece_state, float* piece_decay, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (groups <= 0 || heads % groups) return fail("state_scan: %d heads are not a multiple of %d groups", heads, groups);
    if (heads > 65535) return fail("state_scan: %d heads exceed the grid limit", heads);
    if (dim > 32 * R) return fail("state_scan: a state of %d rows exceeds %d", dim, 32 * R);
    int rows = (dim + R - 1) / R;
    rows = rows <= 4 ? 4 : rows <= 8 ? 8 : rows <= 16 ? 16 : 32;
    const int source = decay == nullptr ? PER_TOKEN : (delta ? CHANNELS : FIXED);
    const int vec = ((ld | q_col | k_col | v_col | dim | vdim) % 4 == 0 && (reinterpret_cast<uintptr_t>(u) & 15) == 0 &&
                     (source != CHANNELS || (reinterpret_cast<uintptr_t>(decay) & 15) == 0)) ? 1 : 0;
    if (piece > 0) {
        if (delta) return fail("state_scan: the delta rule's update is not a scalar times the state: no pieces");
        if (max_pieces < 1 || piece_state == nullptr || piece_decay == nullptr) return fail("state_scan: pieces need their scratch");
        if ((long long)n_seqs * max_pieces > 0x7fffffffLL || n_seqs > 65535) return fail("state_scan: %d sequences of %d pieces exceed the grid limit", n_seqs, max_pieces);
        if (longest_run <= 0 || longest_run > piece) longest_run = piece;
    }
    Scan p{u, ld, q_col, k_col, v_col, decay_col, step_col, decay, skip, state, o, cu_seqlens, seq_slot, heads, groups, dim, vdim, 1, vec,
           piece > 0 ? piece : 0, piece > 0 ? max_pieces : 1, piece_state, piece_decay};
    dim3 grid(n_seqs, heads, (vdim + COLS - 1) / COLS);
    if (rows == 4) return pick_scan<4>(delta != 0, source, grid, stream, p, longest_run, n_seqs);
    if (rows == 8) return pick_scan<8>(delta != 0, source, grid, stream, p, longest_run, n_seqs);
    if (rows == 16) return pick_scan<16>(delta != 0, source, grid, stream, p, longest_run, n_seqs);
    return pick_scan<32>(delta != 0, source, grid, stream, p, longest_run, n_seqs);
}

RI_API int ri_gated_group_norm(const float* x, int x_ld, const float* gate, int gate_ld, int gate_col, const float* w, int w_len,
                               void* out, int dtype, int n_tokens, int groups, int gs, int gate_first, int sigmoid, float eps,
                               float out_scale, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (groups <= 0 || gs <= 0 || w_len <= 0) return fail("gated_group_norm: %d groups of %d channels, %d weights", groups, gs, w_len);
    const long long warps = (long long)n_tokens * groups;
    const int blocks = (int)((warps * 32 + 255) / 256);
    const bool wide = gs >= 512 && warps <= 0x7fffffffLL;          // a block per group instead of a warp
    const bool vec = (gs | x_ld | gate_ld | gate_col | w_len) % 4 == 0 &&
                     ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) |
                       reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const int per = vec ? 4 : 1;
    int threads = ((gs + per - 1) / per + 31) / 32 * 32;
    threads = threads > 1024 ? 1024 : threads;
    cudaError_t e;
#define RI_NORM_WIDE(T, V) launch_dependent(gated_group_norm_block_kernel<T, V>, (int)warps, threads, 0, stream, x, x_ld, gate, gate_ld, \
                                            gate_col, w, w_len, (T*)out, groups, gs, gate_first, sigmoid, eps, out_scale)
#define RI_NORM(T) (!wide ? launch_dependent(gated_group_norm_kernel<T>, blocks, 256, 0, stream, x, x_ld, gate, gate_ld, gate_col, w,   \
                                             w_len, (T*)out, n_tokens, groups, gs, gate_first, sigmoid, eps, out_scale)                  \
                    : vec ? RI_NORM_WIDE(T, 4) : RI_NORM_WIDE(T, 1))
    if (dtype == RI_F32) e = RI_NORM(float);
    else if (dtype == RI_BF16) e = RI_NORM(__nv_bfloat16);
    else return fail("gated_group_norm: unknown dtype %d", dtype);
#undef RI_NORM
#undef RI_NORM_WIDE
    return check_launch(e, "gated_group_norm");
}

RI_DEFINE_LAST_ERROR()
