// The gated delta rule with a decay per head and key channel, over the flat batch of a step, from and into each
// request's state slot.  Per head, with the matrix state S [dim][vdim] in float32:
//
//   S <- diag(g_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t.
//
// `split_halves` hands the low-rank sums of the layer's input projection to the product with the second factors.
// `delta_prepare` forms everything that enters the recurrence for all tokens at once: the short causal convolution of q,
// k and v with silu, unit q and k, beta and the decays.  `delta_scan` walks the tokens of every entry.
//
// A request's slot is one row of floats: the states as [heads][vdim][dim] (the key channels of a value column side by
// side), then the convolution's last K - 1 inputs, oldest first ([K - 1][channels], channels = q | k | v).
#include "common.cuh"

#include <algorithm>

// ------------------------------------------------------------------------- low-rank sums, halved

// out[t] = (sums rounded to bfloat16 | what the rounding left, rounded to bfloat16); in float32 the sums themselves.
template <typename T>
__global__ void __launch_bounds__(256) split_halves_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int width,
                                                           int column, int count, T* __restrict__ out, int tokens) {
    pdl_trigger();
    pdl_wait();
    const size_t total = static_cast<size_t>(tokens) * count;
    for (size_t idx = blockIdx.x * static_cast<size_t>(256) + threadIdx.x; idx < total; idx += static_cast<size_t>(gridDim.x) * 256) {
        const size_t t = idx / count;
        const int i = static_cast<int>(idx % count);
        const float* src = proj + t * width + column + i;
        float sum = 0.0f;
        for (int s = 0; s < splits; ++s) sum += src[s * split_stride];
        if constexpr (sizeof(T) == 2) {
            const T high = from_float<T>(sum);
            out[t * 2 * count + i] = high;
            out[t * 2 * count + count + i] = from_float<T>(sum - to_float(high));
        } else {
            out[t * count + i] = sum;
        }
    }
}

ME_EXPORT int me_split_halves(const float* proj, int splits, long long split_stride, int width, int column, int count, void* out,
                              int out_type, int tokens, cudaStream_t stream) {
    if (tokens <= 0 || count <= 0) return 0;
    const size_t total = static_cast<size_t>(tokens) * count;
    const int blocks = static_cast<int>(std::min<size_t>((total + 255) / 256, 148 * 8));
    if (out_type == ME_BF16)
        return launch_kernel(split_halves_kernel<__nv_bfloat16>, blocks, 256, 0, stream, proj, splits, (size_t)split_stride, width,
                             column, count, static_cast<__nv_bfloat16*>(out), tokens);
    return launch_kernel(split_halves_kernel<float>, blocks, 256, 0, stream, proj, splits, (size_t)split_stride, width, column,
                         count, static_cast<float*>(out), tokens);
}

// -------------------------------------------------------------------------------------- prepare

constexpr int PREP_WARPS = 8;
constexpr int MAX_TAPS = 16;
constexpr int MAX_DIM = 512;

struct DeltaPrepArgs {
    const float* proj;  // [splits][tokens][width]
    int splits;
    size_t split_stride;
    int width;
    int q_col, k_col, v_col, beta_col;
    const float* second;  // [second_splits][tokens][second_width]: decay logits in the columns [0, heads * dim)
    int second_splits;
    size_t second_stride;
    int second_width;
    const float* conv;     // [K][channels]
    const float* a_log;    // [heads]
    const float* dt_bias;  // [heads * dim]
    const int* entry_of_token;
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    float* state;      // [slots + 1][slot_floats]
    size_t slot_floats, matrix;  // floats of a slot; of its matrix states
    float* qk;       // [tokens][qk_heads][2][dim]: unit q times q_scale, unit k
    float* gv;       // [tokens][heads][dim + vdim]: decays, then values
    float* scalars;  // [tokens][heads][2]: beta, q . k
    float q_scale, unit_eps;
    int tokens, heads, qk_heads, dim, vdim, K, channels, run;
};

struct ConvWindow {
    const DeltaPrepArgs& a;
    int first;             // the entry's first token
    const float* history;  // the request's past inputs, or null
    __device__ __forceinline__ float input(int token, int channel) const {
        const float* src = a.proj + static_cast<size_t>(token) * a.width + channel;
        float x = 0.0f;
        for (int s = 0; s < a.splits; ++s) x += src[s * a.split_stride];
        return x;
    }
    // silu of the convolution at the entry's token number n (columns q | k | v of the projection are the channels)
    __device__ __forceinline__ float operator()(int n, int channel) const {
        float sum = 0.0f;
        for (int j = 0; j < a.K; ++j) {
            const int from = n - (a.K - 1) + j;
            float x;
            if (from >= 0) x = input(first + from, channel);
            else if (history) x = history[static_cast<size_t>(from + a.K - 1) * a.channels + channel];
            else continue;
            sum = fmaf(a.conv[static_cast<size_t>(j) * a.channels + channel], x, sum);
        }
        return sum / (1.0f + expf(-sum));
    }
};

// The entry's last K - 1 inputs of one channel into the slot; row i is replaced by row i + count, read before it is replaced.
__device__ __forceinline__ void keep_history(const DeltaPrepArgs& a, const ConvWindow& window, float* slot, bool past, int count, int channel) {
    for (int i = 0; i < a.K - 1; ++i) {
        const int from = count - (a.K - 1) + i;
        float x = 0.0f;
        if (from >= 0) x = window.input(window.first + from, channel);
        else if (past) x = slot[static_cast<size_t>(i + count) * a.channels + channel];
        slot[static_cast<size_t>(i) * a.channels + channel] = x;
    }
}

// A q/k head of one token: unit q (times its scale), unit k and their dot product.  Lane l holds channels l + 32 i.
template <int PER>
__device__ __forceinline__ void store_unit_pair(const DeltaPrepArgs& a, size_t token, int item, int lane, float (&q)[PER], float (&k)[PER]) {
    float q_sq = 0.0f, k_sq = 0.0f;
#pragma unroll
    for (int i = 0; i < PER; ++i) q_sq = fmaf(q[i], q[i], q_sq), k_sq = fmaf(k[i], k[i], k_sq);
    const float q_inv = rsqrtf(warp_sum(q_sq) + a.unit_eps), k_inv = rsqrtf(warp_sum(k_sq) + a.unit_eps);
    float dot = 0.0f;
    float* dst = a.qk + (token * a.qk_heads + item) * 2 * a.dim;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + 32 * i;
        q[i] = q[i] * q_inv * a.q_scale, k[i] = k[i] * k_inv;
        dot = fmaf(q[i], k[i], dot);
        if (d < a.dim) dst[d] = q[i], dst[a.dim + d] = k[i];
    }
    dot = warp_sum(dot);
    const int per = a.heads / a.qk_heads;
    for (int h = lane; h < per; h += 32) a.scalars[(token * a.heads + item * per + h) * 2 + 1] = dot;
}

// The decays and beta of one head and token.
__device__ __forceinline__ void store_decays(const DeltaPrepArgs& a, const ConvWindow& window, size_t token, int head, float rate, int lane) {
    float* dst = a.gv + (token * a.heads + head) * (a.dim + a.vdim);
    const float* logits = a.second + token * a.second_width + head * a.dim;
    for (int d = lane; d < a.dim; d += 32) {
        float z = a.dt_bias[head * a.dim + d];
        for (int s = 0; s < a.second_splits; ++s) z += logits[s * a.second_stride + d];
        const float softplus = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
        dst[d] = 1.0f + expm1f(rate * softplus);  // the float nearest to the decay where it is near 1
    }
    if (lane == 0) a.scalars[(token * a.heads + head) * 2] = 1.0f / (1.0f + expf(-window.input(static_cast<int>(token), a.beta_col + head)));
}

// One warp per (a.run tokens, item): items [0, qk_heads) form q, k and q . k of a q/k head, items behind them v, the
// decays and beta of a head; a lane holds channels lane, lane + 32, ... (PER of them at most).  Tokens that have K - 1
// tokens of their entry in front of them slide a window of inputs in registers (KC = K; KC = 0: more taps than that, read
// again for every token).  The first K - 1 tokens of an entry reach into the request's past; the warp that holds the
// entry's first token computes all of them and then leaves the entry's last inputs of its channels in the slot, so that
// nothing is read after it was replaced.  Both forms add a channel's products in the same order.
constexpr int PREP_RUN = 8;           // tokens of a warp in a long step
constexpr int PREP_RUN_TOKENS = 512;  // from this many tokens on; a shorter step gives every token warps of its own

template <int PER, int KC>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prepare_kernel(DeltaPrepArgs a) {
    constexpr int WINDOW = KC > 1 ? KC - 1 : 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, item = blockIdx.y;
    const int run_begin = (blockIdx.x * PREP_WARPS + warp) * a.run, run_end = min(run_begin + a.run, a.tokens);
    pdl_trigger();
    pdl_wait();
    const bool is_qk = item < a.qk_heads;
    const int head = item - a.qk_heads;
    const float rate = is_qk ? 0.0f : -expf(a.a_log[head]);
    const int q_column = a.q_col + item * a.dim, k_column = a.k_col + item * a.dim;
    // channels of this lane: of q and k, or of v in the place of q
    const int column = is_qk ? q_column : a.v_col + head * a.vdim, extent = is_qk ? a.dim : a.vdim;
    const int blocks_of_v = is_qk ? 1 : (a.vdim + 32 * PER - 1) / (32 * PER);
    for (int block = 0; block < blocks_of_v; ++block) {  // a value head wider than 32 PER channels takes several rounds
        const int offset = block * 32 * PER;
        float held[2][WINDOW][PER], taps[2][KC > 0 ? KC : 1][PER];
        if constexpr (KC > 0) {
#pragma unroll
            for (int j = 0; j < KC; ++j)
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    const int d = offset + lane + 32 * i;
                    taps[0][j][i] = d < extent ? a.conv[static_cast<size_t>(j) * a.channels + column + d] : 0.0f;
                    taps[1][j][i] = is_qk && d < extent ? a.conv[static_cast<size_t>(j) * a.channels + k_column + d] : 0.0f;
                }
        }
        int filled = -1;  // the token in front of which the window stands
        for (int t = run_begin; t < run_end; ++t) {
            const int entry = a.entry_of_token[t], first = a.cu_tokens[entry], n0 = t - first;
            if (n0 > 0 && n0 < a.K - 1) continue;  // done by the warp of the entry's first token
            float* slot = a.state + static_cast<size_t>(a.state_slots[entry]) * a.slot_floats + a.matrix;
            const bool past = a.K > 1 && a.fresh[entry] == 0;
            const ConvWindow window{a, first, past ? slot : nullptr};
            float x[2][PER];
            if (KC > 0 && n0 >= a.K - 1) {
                if (filled != t) {
#pragma unroll
                    for (int w = 0; w < KC - 1; ++w)
#pragma unroll
                        for (int i = 0; i < PER; ++i) {
                            const int d = offset + lane + 32 * i;
                            held[0][w][i] = d < extent ? window.input(t - (KC - 1) + w, column + d) : 0.0f;
                            held[1][w][i] = is_qk && d < extent ? window.input(t - (KC - 1) + w, k_column + d) : 0.0f;
                        }
                }
#pragma unroll
                for (int which = 0; which < 2; ++which)
#pragma unroll
                    for (int i = 0; i < PER; ++i) {
                        const int d = offset + lane + 32 * i;
                        x[which][i] = 0.0f;
                        if (which == 1 && !is_qk) continue;
                        const float now = d < extent ? window.input(t, (which ? k_column : column) + d) : 0.0f;
                        float sum = 0.0f;
#pragma unroll
                        for (int w = 0; w < KC - 1; ++w) sum = fmaf(taps[which][w][i], held[which][w][i], sum);
                        sum = fmaf(taps[which][KC > 0 ? KC - 1 : 0][i], now, sum);
                        x[which][i] = sum / (1.0f + expf(-sum));
#pragma unroll
                        for (int w = 0; w + 1 < KC - 1; ++w) held[which][w][i] = held[which][w + 1][i];
                        if (KC > 1) held[which][WINDOW - 1][i] = now;
                    }
                filled = t + 1;
                if (is_qk) {
                    store_unit_pair<PER>(a, t, item, lane, x[0], x[1]);
                } else {
                    float* dst = a.gv + (static_cast<size_t>(t) * a.heads + head) * (a.dim + a.vdim) + a.dim;
#pragma unroll
                    for (int i = 0; i < PER; ++i)
                        if (offset + lane + 32 * i < extent) dst[offset + lane + 32 * i] = x[0][i];
                    if (block == 0) store_decays(a, window, t, head, rate, lane);
                }
                continue;
            }
            // the entry's first tokens, or more taps than the window holds
            const int count = a.cu_tokens[entry + 1] - first;
            const int run = n0 == 0 ? min(count, max(a.K - 1, 1)) : 1;
            for (int n = n0; n < n0 + run; ++n) {
                const size_t token = static_cast<size_t>(first + n);
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    const int d = offset + lane + 32 * i;
                    x[0][i] = d < extent ? window(n, column + d) : 0.0f;
                    x[1][i] = is_qk && d < extent ? window(n, k_column + d) : 0.0f;
                }
                if (is_qk) {
                    store_unit_pair<PER>(a, token, item, lane, x[0], x[1]);
                    continue;
                }
                float* dst = a.gv + (token * a.heads + head) * (a.dim + a.vdim) + a.dim;
#pragma unroll
                for (int i = 0; i < PER; ++i)
                    if (offset + lane + 32 * i < extent) dst[offset + lane + 32 * i] = x[0][i];
                if (block == 0) store_decays(a, window, token, head, rate, lane);
            }
            if (n0 != 0) continue;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int d = offset + lane + 32 * i;
                if (d >= extent) continue;
                keep_history(a, window, slot, past, count, column + d);
                if (is_qk) keep_history(a, window, slot, past, count, k_column + d);
            }
        }
    }
}

template <int PER>
static int launch_delta_prepare(const DeltaPrepArgs& a, cudaStream_t stream) {
    const dim3 grid((a.tokens + PREP_WARPS * a.run - 1) / (PREP_WARPS * a.run), a.qk_heads + a.heads);
    constexpr int THREADS = PREP_WARPS * 32;
    if (PER <= 4) {  // the window of a wider head does not fit the registers
        if (a.K == 1) return launch_kernel(delta_prepare_kernel<PER, PER <= 4 ? 1 : 0>, grid, THREADS, 0, stream, a);
        if (a.K == 2) return launch_kernel(delta_prepare_kernel<PER, PER <= 4 ? 2 : 0>, grid, THREADS, 0, stream, a);
        if (a.K == 3) return launch_kernel(delta_prepare_kernel<PER, PER <= 4 ? 3 : 0>, grid, THREADS, 0, stream, a);
        if (a.K == 4) return launch_kernel(delta_prepare_kernel<PER, PER <= 4 ? 4 : 0>, grid, THREADS, 0, stream, a);
    }
    return launch_kernel(delta_prepare_kernel<PER, 0>, grid, THREADS, 0, stream, a);
}

ME_EXPORT int me_delta_prepare(const float* proj, int splits, long long split_stride, int width, int q_col, int k_col, int v_col,
                               int beta_col, const float* second, int second_splits, long long second_stride, int second_width,
                               const float* conv, const float* a_log, const float* dt_bias, const int* entry_of_token,
                               const int* cu_tokens, const int* state_slots, const int* fresh, float* state, long long slot_floats,
                               long long matrix, float* qk, float* gv, float* scalars, float q_scale, float unit_eps, int tokens,
                               int heads, int qk_heads, int dim, int vdim, int taps_count, int channels, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (dim < 1 || vdim < 1 || heads < 1 || qk_heads < 1 || heads % qk_heads || taps_count < 1) return ME_ERR_ARGUMENT;
    // the channels of the convolution are the projection's first columns, q | k | v
    if (q_col != 0 || k_col != qk_heads * dim || v_col != 2 * qk_heads * dim || channels != v_col + heads * vdim) return ME_ERR_ARGUMENT;
    if (slot_floats < matrix + static_cast<long long>(taps_count - 1) * channels) return ME_ERR_ARGUMENT;
    if (dim > MAX_DIM || taps_count > MAX_TAPS) return ME_ERR_UNSUPPORTED;
    DeltaPrepArgs a{proj, splits, (size_t)split_stride, width, q_col, k_col, v_col, beta_col, second, second_splits,
                    (size_t)second_stride, second_width, conv, a_log, dt_bias, entry_of_token, cu_tokens, state_slots, fresh,
                    state, (size_t)slot_floats, (size_t)matrix, qk, gv, scalars, q_scale, unit_eps, tokens, heads, qk_heads,
                    dim, vdim, taps_count, channels, tokens >= PREP_RUN_TOKENS ? PREP_RUN : 1};
    if (dim <= 32) return launch_delta_prepare<1>(a, stream);
    if (dim <= 64) return launch_delta_prepare<2>(a, stream);
    if (dim <= 128) return launch_delta_prepare<4>(a, stream);
    if (dim <= 256) return launch_delta_prepare<8>(a, stream);
    return launch_delta_prepare<16>(a, stream);
}

// ----------------------------------------------------------------------------------------- scan

// A value column's state [dim] is held by L neighbouring lanes, R channels each (float4 number i of lane l holds channels
// 4 (i L + l) ..), and a lane holds C columns, which share what it reads of a token from shared memory: a warp walks 32 / L
// * C columns, so that a head needs several warps.  The walk's time is the latency of one token's step; the next token's q,
// k and decays are read while it runs.  Per token the two dots S^T k and S^T q of the decayed state run together and meet
// in one butterfly over the L lanes; o = S^T q + (q . k) u needs no second one after the correction.
// A block of WARPS warps shares the tokens' q, k, decays, values and scalars, fetched SC tokens ahead by asynchronous
// copies.  Columns are independent and a token's output depends on the tokens before it through the state alone: the
// bits are the same for a whole prompt, its portions and single decoded tokens.
constexpr int SCAN_WARPS = 4;  // most warps of a block

struct DeltaScanArgs {
    const float* qk;       // [tokens][qk_heads][2][dim]
    const float* gv;       // [tokens][heads][dim + vdim]
    const float* scalars;  // [tokens][heads][2]
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    float* state;  // [slots + 1][slot_floats], a slot starts with [heads][vdim][dim]
    size_t slot_floats;
    float* out;  // [tokens][heads][vdim]
    int heads, qk_heads, dim, vdim, vector;  // vector: 16-byte loads are aligned
};

__device__ __forceinline__ void copy_async_16(float* shared_dst, const float* global_src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(shared_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(global_src) : "memory");
}
__device__ __forceinline__ void copy_async_4(float* shared_dst, const float* global_src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(shared_dst));
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(global_src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

// What a lane reads of one token: its R channels of k, q and the decays.
template <int R>
struct TokenRow {
    float2 k[R / 2], q[R / 2], g[R / 2];
    template <int L>
    __device__ __forceinline__ void load(const float* q_s, const float* k_s, const float* g_s, int at) {
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const float4 k4 = *reinterpret_cast<const float4*>(k_s + at + 4 * i * L);
            const float4 q4 = *reinterpret_cast<const float4*>(q_s + at + 4 * i * L);
            const float4 g4 = *reinterpret_cast<const float4*>(g_s + at + 4 * i * L);
            k[2 * i] = make_float2(k4.x, k4.y), k[2 * i + 1] = make_float2(k4.z, k4.w);
            q[2 * i] = make_float2(q4.x, q4.y), q[2 * i + 1] = make_float2(q4.z, q4.w);
            g[2 * i] = make_float2(g4.x, g4.y), g[2 * i + 1] = make_float2(g4.z, g4.w);
        }
    }
};

template <int L, int R, int C, int SC>
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_kernel(DeltaScanArgs a) {
    constexpr int DP = L * R;  // the key channels a column has room for
    constexpr int GROUPS = 32 / L, COLUMNS = GROUPS * C;  // of a warp
    constexpr bool PREFETCH = R <= 16;  // registers for a second token's row
    extern __shared__ __align__(16) float staged[];
    const int threads = blockDim.x, columns = (threads >> 5) * COLUMNS;
    const int stage_floats = SC * (3 * DP + columns + 2);
    // one stage: q [SC][DP], k [SC][DP], g [SC][DP], v [SC][columns], scalars [SC][2]
    const int entry = blockIdx.x, head = blockIdx.y, qk_head = head / (a.heads / a.qk_heads);
    const int first_column = blockIdx.z * columns;
    const int lane = threadIdx.x & 31, part = lane % L;
    const int local_column = (threadIdx.x >> 5) * COLUMNS + lane / L;  // and GROUPS, 2 GROUPS, ... behind it
    const int dim = a.dim;
    for (int i = threadIdx.x; i < 2 * SC * 3 * (DP - dim); i += threads) {  // channels dim .. DP are zero for good
        const int stage = i / (SC * 3 * (DP - dim)), j = i % (SC * 3 * (DP - dim));
        staged[stage * stage_floats + (j / (DP - dim)) * DP + dim + j % (DP - dim)] = 0.0f;
    }
    const int begin = a.cu_tokens[entry], end = a.cu_tokens[entry + 1];
    float* state = a.state + static_cast<size_t>(a.state_slots[entry]) * a.slot_floats +
                   (static_cast<size_t>(head) * a.vdim + first_column + local_column) * dim;

    float2 s[C][R / 2];
    bool live[C];
#pragma unroll
    for (int c = 0; c < C; ++c) {
        live[c] = first_column + local_column + c * GROUPS < a.vdim;
        const bool load = live[c] && a.fresh[entry] == 0;
        const float* src = state + static_cast<size_t>(c) * GROUPS * dim;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int d = 4 * (i * L + part);
            float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (load && a.vector) {
                if (d < dim) q = *reinterpret_cast<const float4*>(src + d);
            } else if (load) {
                if (d < dim) q.x = src[d];
                if (d + 1 < dim) q.y = src[d + 1];
                if (d + 2 < dim) q.z = src[d + 2];
                if (d + 3 < dim) q.w = src[d + 3];
            }
            s[c][2 * i] = make_float2(q.x, q.y), s[c][2 * i + 1] = make_float2(q.z, q.w);
        }
    }

    auto stage_tokens = [&](int chunk, float* stage) {
        const int count = min(SC, end - chunk);
        float* q_s = stage;
        float* v_s = stage + SC * 3 * DP;
        float* scalars_s = v_s + SC * columns;
        if (a.vector) {
            const int quads = dim / 4;
            for (int i = threadIdx.x; i < count * 3 * quads; i += threads) {
                const int t = i / (3 * quads), j = i % (3 * quads), which = j / quads, d = (j % quads) * 4;
                const size_t token = static_cast<size_t>(chunk + t);
                const float* src = which < 2 ? a.qk + ((token * a.qk_heads + qk_head) * 2 + which) * dim + d
                                             : a.gv + (token * a.heads + head) * (dim + a.vdim) + d;
                copy_async_16(q_s + (which * SC + t) * DP + d, src);
            }
        } else {
            for (int i = threadIdx.x; i < count * 3 * dim; i += threads) {
                const int t = i / (3 * dim), j = i % (3 * dim), which = j / dim, d = j % dim;
                const size_t token = static_cast<size_t>(chunk + t);
                const float* src = which < 2 ? a.qk + ((token * a.qk_heads + qk_head) * 2 + which) * dim + d
                                             : a.gv + (token * a.heads + head) * (dim + a.vdim) + d;
                copy_async_4(q_s + (which * SC + t) * DP + d, src);
            }
        }
        for (int i = threadIdx.x; i < count * columns; i += threads) {
            const int t = i / columns, c = i % columns;
            if (first_column + c < a.vdim)
                copy_async_4(v_s + t * columns + c, a.gv + (static_cast<size_t>(chunk + t) * a.heads + head) * (dim + a.vdim) + dim + first_column + c);
        }
        for (int i = threadIdx.x; i < count * 2; i += threads)
            copy_async_4(scalars_s + i, a.scalars + (static_cast<size_t>(chunk + i / 2) * a.heads + head) * 2 + i % 2);
        copy_async_commit();
    };

    if (begin < end) stage_tokens(begin, staged);
    int buffer = 0;
    for (int chunk = begin; chunk < end; chunk += SC, buffer ^= 1) {
        const int count = min(SC, end - chunk);
        if (chunk + SC < end) {
            stage_tokens(chunk + SC, staged + (buffer ^ 1) * stage_floats);
            copy_async_wait<1>();
        } else {
            copy_async_wait<0>();
        }
        __syncthreads();
        const float* q_s = staged + buffer * stage_floats;
        const float* k_s = q_s + SC * DP;
        const float* g_s = k_s + SC * DP;
        const float* v_s = g_s + SC * DP;
        const float* scalars_s = v_s + SC * columns;
        TokenRow<R> row;
        row.template load<L>(q_s, k_s, g_s, 4 * part);
#pragma unroll 1
        for (int t = 0; t < count; ++t) {
            TokenRow<R> next;
            if constexpr (PREFETCH) next.template load<L>(q_s, k_s, g_s, min(t + 1, count - 1) * DP + 4 * part);
            const float beta = scalars_s[2 * t], dot = scalars_s[2 * t + 1];
            float dot_k[C], dot_q[C], v[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                v[c] = live[c] ? v_s[t * columns + local_column + c * GROUPS] : 0.0f;
                float2 on_k[2] = {make_float2(0.0f, 0.0f), make_float2(0.0f, 0.0f)};
                float2 on_q[2] = {make_float2(0.0f, 0.0f), make_float2(0.0f, 0.0f)};
#pragma unroll
                for (int i = 0; i < R / 2; ++i) {
                    s[c][i] = __fmul2_rn(row.g[i], s[c][i]);
                    on_k[i & 1] = __ffma2_rn(row.k[i], s[c][i], on_k[i & 1]);
                    on_q[i & 1] = __ffma2_rn(row.q[i], s[c][i], on_q[i & 1]);
                }
                dot_k[c] = (on_k[0].x + on_k[0].y) + (on_k[1].x + on_k[1].y);
                dot_q[c] = (on_q[0].x + on_q[0].y) + (on_q[1].x + on_q[1].y);
            }
#pragma unroll
            for (int offset = L / 2; offset > 0; offset >>= 1) {
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    dot_k[c] += __shfl_xor_sync(0xffffffffu, dot_k[c], offset);
                    dot_q[c] += __shfl_xor_sync(0xffffffffu, dot_q[c], offset);
                }
            }
            float* out = a.out + (static_cast<size_t>(chunk + t) * a.heads + head) * a.vdim + first_column + local_column;
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float u = beta * (v[c] - dot_k[c]);
                const float2 uu = make_float2(u, u);
#pragma unroll
                for (int i = 0; i < R / 2; ++i) s[c][i] = __ffma2_rn(row.k[i], uu, s[c][i]);
                if (live[c] && part == 0) out[c * GROUPS] = fmaf(dot, u, dot_q[c]);
            }
            if constexpr (PREFETCH) row = next;
            else row.template load<L>(q_s, k_s, g_s, min(t + 1, count - 1) * DP + 4 * part);
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
        if (!live[c]) continue;
        float* dst = state + static_cast<size_t>(c) * GROUPS * dim;
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const int d = 4 * (i * L + part);
            if (a.vector) {
                if (d < dim) *reinterpret_cast<float4*>(dst + d) = make_float4(s[c][2 * i].x, s[c][2 * i].y, s[c][2 * i + 1].x, s[c][2 * i + 1].y);
            } else {
                if (d < dim) dst[d] = s[c][2 * i].x;
                if (d + 1 < dim) dst[d + 1] = s[c][2 * i].y;
                if (d + 2 < dim) dst[d + 2] = s[c][2 * i + 1].x;
                if (d + 3 < dim) dst[d + 3] = s[c][2 * i + 1].y;
            }
        }
    }
}

template <int L, int R, int C, int SC>
static int launch_delta_scan(const DeltaScanArgs& a, int entries, cudaStream_t stream) {
    static SharedMemoryOptIn opt_in;
    constexpr int COLUMNS = 32 / L * C;
    // As many warps to a block as there are columns to share its tokens' fetches, fewer where the grid would not fill
    // the GPU.  The split changes nothing in a column's arithmetic.
    int warps = SCAN_WARPS;
    while (warps > 1 && (static_cast<long long>(entries) * a.heads * ((a.vdim + warps * COLUMNS - 1) / (warps * COLUMNS)) < 120 ||
                         (warps / 2) * COLUMNS >= a.vdim))
        warps /= 2;
    const int columns = warps * COLUMNS;
    const size_t smem = static_cast<size_t>(2) * SC * (3 * L * R + columns + 2) * sizeof(float);
    if (smem > 48 * 1024)
        if (const int e = opt_in(delta_scan_kernel<L, R, C, SC>, 200 * 1024)) return e;
    const dim3 grid(entries, a.heads, (a.vdim + columns - 1) / columns);
    return launch_kernel_in_order(delta_scan_kernel<L, R, C, SC>, grid, warps * 32, smem, stream, a);
}

ME_EXPORT int me_delta_scan(const float* qk, const float* gv, const float* scalars, const int* cu_tokens, const int* state_slots,
                            const int* fresh, float* state, long long slot_floats, float* out, int entries, int heads,
                            int qk_heads, int dim, int vdim, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (dim < 1 || vdim < 1 || heads < 1 || qk_heads < 1 || heads % qk_heads) return ME_ERR_ARGUMENT;
    if (slot_floats < static_cast<long long>(heads) * dim * vdim) return ME_ERR_ARGUMENT;
    const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const int vector = dim % 4 == 0 && vdim % 4 == 0 && slot_floats % 4 == 0 && aligned(qk) && aligned(gv) && aligned(state);
    DeltaScanArgs a{qk, gv, scalars, cu_tokens, state_slots, fresh, state, (size_t)slot_floats, out, heads, qk_heads, dim, vdim, vector};
    if (dim <= 32) return launch_delta_scan<8, 4, 2, 16>(a, entries, stream);
    if (dim <= 64) return launch_delta_scan<8, 8, 2, 16>(a, entries, stream);
    if (dim <= 128) return launch_delta_scan<8, 16, 2, 16>(a, entries, stream);
    if (dim <= 256) return launch_delta_scan<16, 16, 2, 8>(a, entries, stream);
    if (dim <= MAX_DIM) return launch_delta_scan<16, 32, 1, 8>(a, entries, stream);
    return ME_ERR_UNSUPPORTED;
}
