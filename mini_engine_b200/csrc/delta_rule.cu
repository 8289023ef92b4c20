// The gated delta rule with a decay per head and key channel, over the flat batch of a step, from and into each
// request's state slot.  Per head, with the matrix state S [dim][vdim] in float32:
//
//   S <- diag(g_t) S,   u_t = beta_t (v_t - S^T k_t),   S <- S + k_t u_t^T,   o_t = S^T q_t.
//
// Two relatives walk through the same kernel.  The generalized delta rule removes with a rate a per key channel what the unit
// key u = k / sqrt(k . k + eps) reads, both terms from the old state, and adds the key as it is:
//
//   S <- diag(g_t) S - (a_t * u_t) (u_t^T S) + k_t v_t^T,   o_t = S^T q_t.
//
// The recurrence with a bonus reads before it writes, the current token through a weight per key channel of its own:
//
//   o_t = (S + diag(b) k_t v_t^T)^T q_t,   S <- diag(g_t) S + k_t v_t^T.
//
// `state_prepare` makes what these two take.
//
// `split_halves` hands the low-rank sums of the layer's input projection (or their tanh) to the product with the second factors.
// `delta_prepare` forms everything that enters the recurrence for all tokens at once: the short causal convolution of q,
// k and v with silu, unit q and k, beta and the decays.  `delta_scan` walks the tokens of every entry.
//
// A request's slot is one row of floats: the states as [heads][vdim][dim] (the key channels of a value column side by
// side), then the convolution's last K - 1 inputs, oldest first ([K - 1][channels], channels = q | k | v).
#include "common.cuh"

#include <algorithm>

// ------------------------------------------------------------------------- low-rank sums, halved

// out[t] = (sums rounded to bfloat16 | what the rounding left, rounded to bfloat16); in float32 the sums themselves.  With
// `activate` the tanh of the sums in their place.
template <typename T>
__global__ void __launch_bounds__(256) split_halves_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int width,
                                                           int column, int count, T* __restrict__ out, int tokens, int activate) {
    pdl_trigger();
    pdl_wait();
    const size_t total = static_cast<size_t>(tokens) * count;
    for (size_t idx = blockIdx.x * static_cast<size_t>(256) + threadIdx.x; idx < total; idx += static_cast<size_t>(gridDim.x) * 256) {
        const size_t t = idx / count;
        const int i = static_cast<int>(idx % count);
        const float* src = proj + t * width + column + i;
        float sum = 0.0f;
        for (int s = 0; s < splits; ++s) sum += src[s * split_stride];
        if (activate) sum = tanhf(sum);
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
                              int out_type, int tokens, int activate, cudaStream_t stream) {
    if (tokens <= 0 || count <= 0) return 0;
    const size_t total = static_cast<size_t>(tokens) * count;
    const int blocks = static_cast<int>(std::min<size_t>((total + 255) / 256, 148 * 8));
    if (out_type == ME_BF16)
        return launch_kernel(split_halves_kernel<__nv_bfloat16>, blocks, 256, 0, stream, proj, splits, (size_t)split_stride, width,
                             column, count, static_cast<__nv_bfloat16*>(out), tokens, activate);
    return launch_kernel(split_halves_kernel<float>, blocks, 256, 0, stream, proj, splits, (size_t)split_stride, width, column,
                         count, static_cast<float*>(out), tokens, activate);
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
    int whole_runs_elsewhere;  // 1: whole runs of tokens are another launch's
};

__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + expf(-z)); }  // the division is within two ulp

struct ConvWindow {
    const DeltaPrepArgs& a;
    int first;             // the entry's first token
    const float* history;  // the request's past inputs, or null
    __device__ __forceinline__ float input(int token, int channel) const {
        const float* src = a.proj + static_cast<size_t>(token) * a.width + channel;
        float x = 0.0f;
#pragma unroll 4
        for (int s = 0; s < a.splits; ++s) x += src[s * a.split_stride];
        return x;
    }
    // silu of the convolution at the entry's token number n for COUNT channels of a lane (columns q | k | v of the
    // projection are the channels; the ones behind `extent` are zero): channel i is first_channel + channel(i).
    template <int COUNT, typename Channel>
    __device__ __forceinline__ void convolve(int n, int first_channel, int extent, Channel channel, float (&y)[COUNT]) const {
#pragma unroll
        for (int i = 0; i < COUNT; ++i) y[i] = 0.0f;
#pragma unroll 1
        for (int j = 0; j < a.K; ++j) {
            const int from = n - (a.K - 1) + j;
            if (from < 0 && !history) continue;
            // a past input is one row of the history, an input of this step the sum of its partial sums
            const float* src = from >= 0 ? a.proj + static_cast<size_t>(first + from) * a.width : history + static_cast<size_t>(from + a.K - 1) * a.channels;
            const int splits = from >= 0 ? a.splits : 1;
            float x[COUNT];
#pragma unroll
            for (int i = 0; i < COUNT; ++i) x[i] = 0.0f;
#pragma unroll 2
            for (int s = 0; s < splits; ++s)
#pragma unroll
                for (int i = 0; i < COUNT; ++i)
                    if (channel(i) < extent) x[i] += src[s * a.split_stride + first_channel + channel(i)];
#pragma unroll
            for (int i = 0; i < COUNT; ++i)
                if (channel(i) < extent) y[i] = fmaf(a.conv[static_cast<size_t>(j) * a.channels + first_channel + channel(i)], x[i], y[i]);
        }
#pragma unroll
        for (int i = 0; i < COUNT; ++i) y[i] = channel(i) < extent ? silu(y[i]) : 0.0f;
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

template <int PER>
__device__ __forceinline__ void load_neighbours(const float* src, float (&x)[PER]) {
    if constexpr (PER == 4) {
        const float4 q = *reinterpret_cast<const float4*>(src);
        x[0] = q.x, x[1] = q.y, x[2] = q.z, x[3] = q.w;
    } else if constexpr (PER == 2) {
        const float2 q = *reinterpret_cast<const float2*>(src);
        x[0] = q.x, x[1] = q.y;
    } else {
#pragma unroll
        for (int i = 0; i < PER; ++i) x[i] = src[i];
    }
}
template <int PER>
__device__ __forceinline__ void store_neighbours(float* dst, const float (&x)[PER]) {
    if constexpr (PER == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
    } else if constexpr (PER == 2) {
        *reinterpret_cast<float2*>(dst) = make_float2(x[0], x[1]);
    } else {
#pragma unroll
        for (int i = 0; i < PER; ++i) dst[i] = x[i];
    }
}

// The i-th channel of a lane: neighbours where a warp's lanes hold a head exactly, so that they may be fetched together.
template <int PER>
__device__ __forceinline__ int channel_of(int lane, int i, int extent) { return extent == 32 * PER ? lane * PER + i : lane + 32 * i; }

// A q/k head of one token: unit q (times its scale), unit k and their dot product.
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
        q[i] = q[i] * q_inv * a.q_scale, k[i] = k[i] * k_inv;
        dot = fmaf(q[i], k[i], dot);
    }
    if ((PER == 2 || PER == 4) && a.dim == 32 * PER && reinterpret_cast<uintptr_t>(a.qk) % 16 == 0) {
        store_neighbours<PER>(dst + lane * PER, q);
        store_neighbours<PER>(dst + a.dim + lane * PER, k);
    } else {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = channel_of<PER>(lane, i, a.dim);
            if (d < a.dim) dst[d] = q[i], dst[a.dim + d] = k[i];
        }
    }
    dot = warp_sum(dot);
    const int per = a.heads / a.qk_heads;
    for (int h = lane; h < per; h += 32) a.scalars[(token * a.heads + item * per + h) * 2 + 1] = dot;
}

__device__ __forceinline__ float decay_of(float z, float rate) {
    const float softplus = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
    return 1.0f + expm1f(rate * softplus);  // the float nearest to the decay where it is near 1
}

// The decays and beta of one head and token.
__device__ __forceinline__ void store_decays(const DeltaPrepArgs& a, const ConvWindow& window, size_t token, int head, float rate, int lane) {
    float* dst = a.gv + (token * a.heads + head) * (a.dim + a.vdim);
    const float* logits = a.second + token * a.second_width + head * a.dim;
    for (int d = lane; d < a.dim; d += 32) {
        float z = a.dt_bias[head * a.dim + d];
#pragma unroll 4
        for (int s = 0; s < a.second_splits; ++s) z += logits[s * a.second_stride + d];
        dst[d] = decay_of(z, rate);
    }
    if (lane == 0) a.scalars[(token * a.heads + head) * 2] = 1.0f / (1.0f + expf(-window.input(static_cast<int>(token), a.beta_col + head)));
}

// One warp per (a.run tokens, item): items [0, qk_heads) form q, k and q . k of a q/k head, items behind them v, the
// decays and beta of a head; a lane holds at most PER channels at a time.  The first K - 1 tokens of an entry reach into the
// request's past; the warp that holds the entry's first token computes all of them and then leaves the entry's last
// inputs of its channels in the slot, so that nothing is read after it was replaced.
constexpr int PREP_RUN = 8;           // tokens of a warp in a long step
constexpr int PREP_RUN_TOKENS = 512;  // from this many tokens on; a shorter step gives every token warps of its own

// Whether the PREP_RUN tokens from `run_begin` on lie in one entry with K - 1 of its tokens in front of them.
__device__ __forceinline__ bool whole_run(const DeltaPrepArgs& a, int run_begin) {
    if (run_begin + PREP_RUN > a.tokens) return false;
    const int entry = a.entry_of_token[run_begin];
    return a.entry_of_token[run_begin + PREP_RUN - 1] == entry && run_begin - a.cu_tokens[entry] >= a.K - 1;
}

// The whole runs of a long step, whose projections are not split: every input of the run is fetched before any is used.
// dim is 32 PER, vdim a multiple of it, every row and segment starts on 16 bytes.  The same bits as the kernel below.
template <int PER, int KC>
__global__ void __launch_bounds__(PREP_WARPS * 32, 2) delta_prepare_runs_kernel(DeltaPrepArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, item = blockIdx.y;
    const int run_begin = (blockIdx.x * PREP_WARPS + warp) * PREP_RUN;
    pdl_trigger();
    pdl_wait();
    if (run_begin >= a.tokens || !whole_run(a, run_begin)) return;
    constexpr int ROWS = PREP_RUN + KC - 1;
    auto fetch = [&](int column, float (&x)[ROWS][PER]) {
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
            load_neighbours<PER>(a.proj + static_cast<size_t>(run_begin - (KC - 1) + r) * a.width + column + lane * PER, x[r]);
    };
    auto convolve = [&](int column, const float (&x)[ROWS][PER], float (&y)[PREP_RUN][PER]) {
        float taps[KC][PER];
#pragma unroll
        for (int j = 0; j < KC; ++j) load_neighbours<PER>(a.conv + static_cast<size_t>(j) * a.channels + column + lane * PER, taps[j]);
#pragma unroll
        for (int t = 0; t < PREP_RUN; ++t)
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                float sum = 0.0f;
#pragma unroll
                for (int j = 0; j < KC; ++j) sum = fmaf(taps[j][i], x[t + j][i], sum);
                y[t][i] = silu(sum);
            }
    };
    if (item < a.qk_heads) {
        const int q_column = a.q_col + item * a.dim, k_column = a.k_col + item * a.dim;
        float x[ROWS][PER], q[PREP_RUN][PER], k[PREP_RUN][PER];
        fetch(q_column, x);
        convolve(q_column, x, q);
        fetch(k_column, x);
        convolve(k_column, x, k);
#pragma unroll
        for (int t = 0; t < PREP_RUN; ++t) store_unit_pair<PER>(a, run_begin + t, item, lane, q[t], k[t]);
        return;
    }
    const int head = item - a.qk_heads;
    const float rate = -expf(a.a_log[head]);
    const size_t step = static_cast<size_t>(a.heads) * (a.dim + a.vdim);
    float* dst = a.gv + (static_cast<size_t>(run_begin) * a.heads + head) * (a.dim + a.vdim) + lane * PER;
    float logits[PREP_RUN][PER], bias[PER];
#pragma unroll
    for (int t = 0; t < PREP_RUN; ++t)
        load_neighbours<PER>(a.second + static_cast<size_t>(run_begin + t) * a.second_width + head * a.dim + lane * PER, logits[t]);
    load_neighbours<PER>(a.dt_bias + head * a.dim + lane * PER, bias);
    if (lane < PREP_RUN) {
        const float z = a.proj[static_cast<size_t>(run_begin + lane) * a.width + a.beta_col + head];
        a.scalars[(static_cast<size_t>(run_begin + lane) * a.heads + head) * 2] = 1.0f / (1.0f + expf(-z));
    }
    for (int offset = 0; offset < a.vdim; offset += 32 * PER) {
        const int column = a.v_col + head * a.vdim + offset;
        float x[ROWS][PER], v[PREP_RUN][PER];
        fetch(column, x);
        convolve(column, x, v);
#pragma unroll
        for (int t = 0; t < PREP_RUN; ++t) store_neighbours<PER>(dst + t * step + a.dim + offset, v[t]);
    }
#pragma unroll
    for (int t = 0; t < PREP_RUN; ++t) {
#pragma unroll
        for (int i = 0; i < PER; ++i) logits[t][i] = decay_of(bias[i] + logits[t][i], rate);
        store_neighbours<PER>(dst + t * step, logits[t]);
    }
}

template <int PER>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prepare_kernel(DeltaPrepArgs a) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, item = blockIdx.y;
    const int run_begin = (blockIdx.x * PREP_WARPS + warp) * a.run, run_end = min(run_begin + a.run, a.tokens);  // (with whole runs elsewhere: one token)
    pdl_trigger();
    pdl_wait();
    if (run_begin >= a.tokens || (a.whole_runs_elsewhere && whole_run(a, run_begin / PREP_RUN * PREP_RUN))) return;
    const bool is_qk = item < a.qk_heads;
    const int head = item - a.qk_heads;
    const float rate = is_qk ? 0.0f : -expf(a.a_log[head]);
    const int q_column = a.q_col + item * a.dim, k_column = a.k_col + item * a.dim, v_column = a.v_col + head * a.vdim;
    for (int t = run_begin; t < run_end; ++t) {
        const int entry = a.entry_of_token[t], first = a.cu_tokens[entry], n0 = t - first;
        if (n0 > 0 && n0 < a.K - 1) continue;  // done by the warp of the entry's first token
        float* slot = a.state + static_cast<size_t>(a.state_slots[entry]) * a.slot_floats + a.matrix;
        const bool past = a.K > 1 && a.fresh[entry] == 0;
        const ConvWindow window{a, first, past ? slot : nullptr};
        const int count = a.cu_tokens[entry + 1] - first;
        const int run = n0 == 0 ? min(count, max(a.K - 1, 1)) : 1;
        for (int n = n0; n < n0 + run; ++n) {
            const size_t token = static_cast<size_t>(first + n);
            if (is_qk) {
                float q[PER], k[PER];
                const auto channel = [&](int i) { return channel_of<PER>(lane, i, a.dim); };
                window.template convolve<PER>(n, q_column, a.dim, channel, q);
                window.template convolve<PER>(n, k_column, a.dim, channel, k);
                store_unit_pair<PER>(a, token, item, lane, q, k);
            } else {
                float* dst = a.gv + (token * a.heads + head) * (a.dim + a.vdim) + a.dim;
                for (int e = 0; e < a.vdim; e += 128) {
                    float v[4];
                    const auto channel = [&](int i) { return e + lane + 32 * i; };
                    window.template convolve<4>(n, v_column, a.vdim, channel, v);
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (channel(i) < a.vdim) dst[channel(i)] = v[i];
                }
                store_decays(a, window, token, head, rate, lane);
            }
        }
        if (n0 != 0) continue;
        const int extent = is_qk ? a.dim : a.vdim;
        for (int d = lane; d < extent; d += 32) {
            keep_history(a, window, slot, past, count, (is_qk ? q_column : v_column) + d);
            if (is_qk) keep_history(a, window, slot, past, count, k_column + d);
        }
    }
}

template <int PER>
static int launch_delta_prepare(DeltaPrepArgs a, cudaStream_t stream) {
    dim3 grid((a.tokens + PREP_WARPS * a.run - 1) / (PREP_WARPS * a.run), a.qk_heads + a.heads);
    if constexpr (PER <= 4) {
        const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
        if (a.run == PREP_RUN && a.K >= 2 && a.K <= 4 && a.splits == 1 && a.second_splits == 1 && a.dim == 32 * PER &&
            a.vdim % (32 * PER) == 0 && a.width % 4 == 0 && a.second_width % 4 == 0 && aligned(a.proj) && aligned(a.second) &&
            aligned(a.conv) && aligned(a.dt_bias) && aligned(a.qk) && aligned(a.gv)) {
            const int code = a.K == 2   ? launch_kernel(delta_prepare_runs_kernel<PER, 2>, grid, PREP_WARPS * 32, 0, stream, a)
                             : a.K == 3 ? launch_kernel(delta_prepare_runs_kernel<PER, 3>, grid, PREP_WARPS * 32, 0, stream, a)
                                        : launch_kernel(delta_prepare_runs_kernel<PER, 4>, grid, PREP_WARPS * 32, 0, stream, a);
            if (code) return code;
            a.whole_runs_elsewhere = 1;  // what is left are the entries' ends: every token has warps of its own again
            a.run = 1;
        }
    }
    grid.x = (a.tokens + PREP_WARPS * a.run - 1) / (PREP_WARPS * a.run);
    return launch_kernel(delta_prepare_kernel<PER>, grid, PREP_WARPS * 32, 0, stream, a);
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
                    dim, vdim, taps_count, channels, tokens >= PREP_RUN_TOKENS ? PREP_RUN : 1, 0};
    if (dim <= 32) return launch_delta_prepare<1>(a, stream);
    if (dim <= 64) return launch_delta_prepare<2>(a, stream);
    if (dim <= 128) return launch_delta_prepare<4>(a, stream);
    if (dim <= 256) return launch_delta_prepare<8>(a, stream);
    return launch_delta_prepare<16>(a, stream);
}

// --------------------------------------------------------- prepare: the generalized rule and the bonus

enum : int { RULE_DELTA = 0, RULE_REMOVAL = 1, RULE_BONUS = 2 };

template <int RULE>
struct Rule;
// VECTORS: what the walk reads per token and head beside the values ([VECTORS][dim]); SCALARS: numbers per token and head.
template <>
struct Rule<RULE_DELTA> { static constexpr int VECTORS = 3, SCALARS = 2; };    // q, k, g; beta, q . k
template <>
struct Rule<RULE_REMOVAL> { static constexpr int VECTORS = 4, SCALARS = 4; };  // q g, k, g, a k; 1 / (k . k + eps), that times sum q a k, q . k
template <>
struct Rule<RULE_BONUS> { static constexpr int VECTORS = 3, SCALARS = 2; };    // q, k, g; sum q b k

// Columns of a product's partial sums.
struct Columns {
    const float* sums;  // [splits][tokens][width], moved to the first column
    int splits;
    size_t stride;
    int width;
    __device__ __forceinline__ float at(size_t token, int column) const {
        const float* src = sums + token * width + column;
        float x = 0.0f;
#pragma unroll 4
        for (int s = 0; s < splits; ++s) x += src[s * stride];
        return x;
    }
};

struct StatePrepArgs {
    Columns q, k, v, logits, rate;  // [heads * dim] each (v: [heads * vdim]); rate for the removal only
    const float* decay_bias;  // [heads * dim]: added to the decay's logits
    const float* channel;     // [heads * dim]: the removal's rate bias, or the bonus
    float* rows;              // [tokens][heads][VECTORS * dim + vdim]
    float* scalars;           // [tokens][heads][SCALARS]
    float decay_scale, unit_eps;
    int tokens, heads, dim, vdim;
};

// One warp per (token, head), a lane's channels 32 apart.  The decay is exp(-decay_scale * sigmoid(z)) (removal) or
// exp(-exp(z)) (bonus), as 1 + expm1: the float nearest to it where it is near 1.
template <int RULE, int PER>
__global__ void __launch_bounds__(PREP_WARPS * 32) state_prepare_kernel(StatePrepArgs a) {
    const long long item = static_cast<long long>(blockIdx.x) * PREP_WARPS + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    if (item >= static_cast<long long>(a.tokens) * a.heads) return;
    const size_t token = static_cast<size_t>(item / a.heads);
    const int head = static_cast<int>(item % a.heads), first = head * a.dim;
    constexpr int VECTORS = Rule<RULE>::VECTORS;
    float q[PER], k[PER], z[PER], rate[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + 32 * i;
        const bool live = d < a.dim;
        q[i] = live ? a.q.at(token, first + d) : 0.0f;
        k[i] = live ? a.k.at(token, first + d) : 0.0f;
        z[i] = live ? a.logits.at(token, first + d) + a.decay_bias[first + d] : 0.0f;
        if (RULE == RULE_REMOVAL) rate[i] = live ? a.rate.at(token, first + d) + a.channel[first + d] : 0.0f;
        else rate[i] = live ? a.channel[first + d] : 0.0f;
    }
    float* row = a.rows + static_cast<size_t>(item) * (VECTORS * a.dim + a.vdim);
    float squares = 0.0f, dot = 0.0f, weighted = 0.0f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + 32 * i;
        if (d >= a.dim) continue;
        float decay;
        if constexpr (RULE == RULE_REMOVAL) {
            decay = 1.0f + expm1f(-a.decay_scale / (1.0f + expf(-z[i])));
            const float removed = k[i] / (1.0f + expf(-rate[i]));  // a k
            row[d] = q[i] * decay;
            row[3 * a.dim + d] = removed;
            squares = fmaf(k[i], k[i], squares);
            dot = fmaf(q[i], k[i], dot);
            weighted = fmaf(q[i], removed, weighted);
        } else {
            decay = 1.0f + expm1f(-expf(z[i]));
            row[d] = q[i];
            weighted = fmaf(q[i] * rate[i], k[i], weighted);
        }
        row[a.dim + d] = k[i];
        row[2 * a.dim + d] = decay;
    }
    for (int e = lane; e < a.vdim; e += 32) row[VECTORS * a.dim + e] = a.v.at(token, head * a.vdim + e);
    weighted = warp_sum(weighted);
    float* scalars = a.scalars + static_cast<size_t>(item) * Rule<RULE>::SCALARS;
    if constexpr (RULE == RULE_REMOVAL) {
        squares = warp_sum(squares), dot = warp_sum(dot);
        const float inverse = 1.0f / (squares + a.unit_eps);
        if (lane == 0) scalars[0] = inverse, scalars[1] = inverse * weighted, scalars[2] = dot, scalars[3] = 0.0f;
    } else if (lane == 0) {
        scalars[0] = weighted, scalars[1] = 0.0f;
    }
}

// The same for key heads of 4 LANES channels and value heads as wide, with every row and range on 16 bytes: a lane takes four
// neighbouring channels, a warp 32 / LANES heads of one token.  All loads of a lane are issued before any is used.
template <int RULE, int LANES>
__global__ void __launch_bounds__(PREP_WARPS * 32) state_prepare_vec_kernel(StatePrepArgs a) {
    constexpr int VECTORS = Rule<RULE>::VECTORS, HEADS = 32 / LANES, DIM = 4 * LANES;
    const int lane = threadIdx.x & 31, part = lane % LANES;
    const int head = (blockIdx.y * PREP_WARPS + (threadIdx.x >> 5)) * HEADS + lane / LANES;
    const size_t token = blockIdx.x;
    const int column = head * DIM + part * 4;
    const bool live = head < a.heads;
    pdl_trigger();
    pdl_wait();
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    auto fetch = [&](const Columns& range) {
        float4 sum = zero;
        const float* src = range.sums + token * range.width + column;
#pragma unroll 4
        for (int s = 0; s < range.splits; ++s) {
            const float4 x = *reinterpret_cast<const float4*>(src + s * range.stride);
            sum.x += x.x, sum.y += x.y, sum.z += x.z, sum.w += x.w;
        }
        return sum;
    };
    float4 q4 = zero, k4 = zero, v4 = zero, z4 = zero, r4 = zero, b4 = zero, c4 = zero;
    if (live) {
        q4 = fetch(a.q), k4 = fetch(a.k), v4 = fetch(a.v), z4 = fetch(a.logits);
        if constexpr (RULE == RULE_REMOVAL) r4 = fetch(a.rate);
        b4 = *reinterpret_cast<const float4*>(a.decay_bias + column), c4 = *reinterpret_cast<const float4*>(a.channel + column);
    }
    const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w};
    const float z[4] = {z4.x + b4.x, z4.y + b4.y, z4.z + b4.z, z4.w + b4.w};
    const float channel[4] = {r4.x + c4.x, r4.y + c4.y, r4.z + c4.z, r4.w + c4.w};
    float decay[4], first[4], removed[4];
    float squares = 0.0f, dot = 0.0f, weighted = 0.0f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        if constexpr (RULE == RULE_REMOVAL) {
            decay[i] = 1.0f + expm1f(-a.decay_scale / (1.0f + expf(-z[i])));
            removed[i] = k[i] / (1.0f + expf(-channel[i]));
            first[i] = q[i] * decay[i];
            squares = fmaf(k[i], k[i], squares);
            dot = fmaf(q[i], k[i], dot);
            weighted = fmaf(q[i], removed[i], weighted);
        } else {
            decay[i] = 1.0f + expm1f(-expf(z[i]));
            first[i] = q[i];
            weighted = fmaf(q[i] * channel[i], k[i], weighted);
        }
    }
#pragma unroll
    for (int offset = LANES / 2; offset > 0; offset >>= 1) {
        weighted += __shfl_xor_sync(0xffffffffu, weighted, offset);
        if constexpr (RULE == RULE_REMOVAL) {
            squares += __shfl_xor_sync(0xffffffffu, squares, offset);
            dot += __shfl_xor_sync(0xffffffffu, dot, offset);
        }
    }
    if (!live) return;
    float* row = a.rows + (token * a.heads + head) * ((VECTORS + 1) * DIM) + part * 4;
    *reinterpret_cast<float4*>(row) = make_float4(first[0], first[1], first[2], first[3]);
    *reinterpret_cast<float4*>(row + DIM) = k4;
    *reinterpret_cast<float4*>(row + 2 * DIM) = make_float4(decay[0], decay[1], decay[2], decay[3]);
    if constexpr (RULE == RULE_REMOVAL) *reinterpret_cast<float4*>(row + 3 * DIM) = make_float4(removed[0], removed[1], removed[2], removed[3]);
    *reinterpret_cast<float4*>(row + VECTORS * DIM) = v4;
    if (part) return;
    float* scalars = a.scalars + (token * a.heads + head) * Rule<RULE>::SCALARS;
    if constexpr (RULE == RULE_REMOVAL) {
        const float inverse = 1.0f / (squares + a.unit_eps);
        *reinterpret_cast<float4*>(scalars) = make_float4(inverse, inverse * weighted, dot, 0.0f);
    } else {
        *reinterpret_cast<float2*>(scalars) = make_float2(weighted, 0.0f);
    }
}

static bool takes_vectors(const Columns& c) { return c.width % 4 == 0 && c.stride % 4 == 0 && reinterpret_cast<uintptr_t>(c.sums) % 16 == 0; }

template <int RULE, int LANES>
static int launch_state_prepare_vec(const StatePrepArgs& a, cudaStream_t stream) {
    constexpr int HEADS = PREP_WARPS * 32 / LANES;
    return launch_kernel(state_prepare_vec_kernel<RULE, LANES>, dim3(a.tokens, (a.heads + HEADS - 1) / HEADS), PREP_WARPS * 32, 0, stream, a);
}

template <int RULE>
static int launch_state_prepare(const StatePrepArgs& a, cudaStream_t stream) {
    const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    // the choice follows from the sizes and the engine's buffers alone
    if (a.vdim == a.dim && takes_vectors(a.q) && takes_vectors(a.k) && takes_vectors(a.v) && takes_vectors(a.logits) &&
        (RULE != RULE_REMOVAL || takes_vectors(a.rate)) && aligned(a.decay_bias) && aligned(a.channel) && aligned(a.rows) && aligned(a.scalars)) {
        if (a.dim == 32) return launch_state_prepare_vec<RULE, 8>(a, stream);
        if (a.dim == 64) return launch_state_prepare_vec<RULE, 16>(a, stream);
        if (a.dim == 128) return launch_state_prepare_vec<RULE, 32>(a, stream);
    }
    const long long items = static_cast<long long>(a.tokens) * a.heads;
    const int blocks = static_cast<int>((items + PREP_WARPS - 1) / PREP_WARPS);
    if (a.dim <= 32) return launch_kernel(state_prepare_kernel<RULE, 1>, blocks, PREP_WARPS * 32, 0, stream, a);
    if (a.dim <= 64) return launch_kernel(state_prepare_kernel<RULE, 2>, blocks, PREP_WARPS * 32, 0, stream, a);
    if (a.dim <= 128) return launch_kernel(state_prepare_kernel<RULE, 4>, blocks, PREP_WARPS * 32, 0, stream, a);
    return launch_kernel(state_prepare_kernel<RULE, 16>, blocks, PREP_WARPS * 32, 0, stream, a);
}

// The five column ranges are given as pointer, splits, stride and width each: q, k, v, the decay's logits, the removal's rate.
ME_EXPORT int me_state_prepare(const float* const* sums, const int* splits, const long long* strides, const int* widths, int rule,
                               const float* decay_bias, const float* channel, float* rows, float* scalars, float decay_scale,
                               float unit_eps, int tokens, int heads, int dim, int vdim, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (dim < 1 || vdim < 1 || heads < 1 || (rule != RULE_REMOVAL && rule != RULE_BONUS)) return ME_ERR_ARGUMENT;
    if (dim > MAX_DIM) return ME_ERR_UNSUPPORTED;
    Columns ranges[5];
    for (int i = 0; i < 5; ++i) ranges[i] = Columns{sums[i], splits[i], (size_t)strides[i], widths[i]};
    StatePrepArgs a{ranges[0], ranges[1], ranges[2], ranges[3], ranges[4], decay_bias, channel, rows, scalars, decay_scale,
                    unit_eps, tokens, heads, dim, vdim};
    return rule == RULE_REMOVAL ? launch_state_prepare<RULE_REMOVAL>(a, stream) : launch_state_prepare<RULE_BONUS>(a, stream);
}

// ----------------------------------------------------------------------------------------- scan

// A value column's state [dim] is held by L neighbouring lanes, R channels each (float4 number i of lane l holds channels
// 4 (i L + l) ..), and a lane holds C columns, which share what it reads of a token from shared memory: a warp walks 32 / L
// * C columns, so that a head needs several warps.  The walk's time is the latency of one token's step; the next token's q,
// k and decays are read while it runs.  Per token the two dots S^T k and S^T q of the decayed state run together and meet
// in one butterfly over the L lanes; o = S^T q + (q . k) u needs no second one after the correction.
// The walking warps of a block share the tokens' q, k, decays, values and scalars; one more warp fetches them, SC tokens
// ahead, by asynchronous copies, and stores the outputs of the SC tokens before.  Columns are independent and a token's output depends on the tokens before it through the state alone: the
// bits are the same for a whole prompt, its portions and single decoded tokens.
// The generalized rule reads S^T k and S^T (q g) of the old state in the same butterfly: with c = 1 / (k . k + eps) the removal is
// (a k) c (S^T k) and o = S^T (q g) - c (sum q a k) (S^T k) + (q . k) v.  With the bonus o = S^T q + (sum q b k) v.
constexpr int SCAN_WARPS = 4;  // most walking warps of a block

struct DeltaScanArgs {
    const float* qk;       // [tokens][qk_heads][2][dim] (the delta rule; else unused)
    const float* gv;       // [tokens][heads][dim + vdim]; the other rules: all vectors, [tokens][heads][VECTORS * dim + vdim]
    const float* scalars;  // [tokens][heads][SCALARS]
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    float* state;  // [slots + 1][slot_floats], a slot starts with [heads][vdim][dim]
    size_t slot_floats;
    float* out;  // [tokens][heads][vdim]
    int heads, qk_heads, dim, vdim, vector;  // vector: 16-byte loads are aligned
    int max_count = 0;                       // > 0: entries with more tokens than this are left to the chunked kernels
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

// What a lane reads of one token: its R channels of k, q and the decays (and of what the generalized rule removes).
template <int R, int VECTORS>
struct TokenRow {
    float2 k[R / 2], q[R / 2], g[R / 2], removed[VECTORS > 3 ? R / 2 : 1];
    template <int L>
    __device__ __forceinline__ void load(const float* at) {
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const float4 q4 = *reinterpret_cast<const float4*>(at + 4 * i * L);
            const float4 k4 = *reinterpret_cast<const float4*>(at + L * R + 4 * i * L);
            const float4 g4 = *reinterpret_cast<const float4*>(at + 2 * L * R + 4 * i * L);
            k[2 * i] = make_float2(k4.x, k4.y), k[2 * i + 1] = make_float2(k4.z, k4.w);
            q[2 * i] = make_float2(q4.x, q4.y), q[2 * i + 1] = make_float2(q4.z, q4.w);
            g[2 * i] = make_float2(g4.x, g4.y), g[2 * i + 1] = make_float2(g4.z, g4.w);
            if constexpr (VECTORS > 3) {
                const float4 a4 = *reinterpret_cast<const float4*>(at + 3 * L * R + 4 * i * L);
                removed[2 * i] = make_float2(a4.x, a4.y), removed[2 * i + 1] = make_float2(a4.z, a4.w);
            }
        }
    }
};

template <int RULE, int L, int R, int C, int SC>
__global__ void __launch_bounds__((SCAN_WARPS + 1) * 32) delta_scan_kernel(DeltaScanArgs a) {
    constexpr int VECTORS = Rule<RULE>::VECTORS, SCALARS = Rule<RULE>::SCALARS;
    constexpr int DP = L * R;  // the key channels a column has room for
    constexpr int GROUPS = 32 / L, COLUMNS = GROUPS * C;  // of a warp
    extern __shared__ __align__(16) float staged[];
    const int threads = blockDim.x, warp = threadIdx.x >> 5, warps = (threads >> 5) - 1, columns = warps * COLUMNS;
    const int stage_floats = SC * (VECTORS * DP + columns + SCALARS);
    float* results = staged + 2 * stage_floats;  // [2][SC][columns]
    const bool fetches = warp == warps;  // the last warp
    // one stage: q, k, the decays (and the rest) of every token [SC][VECTORS][DP], v [SC][columns], scalars [SC][SCALARS]
    const int entry = blockIdx.x, head = blockIdx.y, qk_head = head / (a.heads / a.qk_heads);
    const int first_column = blockIdx.z * columns;
    const int lane = threadIdx.x & 31, part = lane % L;
    const int local_column = warp * COLUMNS + lane / L;  // and GROUPS, 2 GROUPS, ... behind it
    const int dim = a.dim;
    for (int i = threadIdx.x; i < 2 * SC * VECTORS * (DP - dim); i += threads) {  // channels dim .. DP are zero for good
        const int stage = i / (SC * VECTORS * (DP - dim)), j = i % (SC * VECTORS * (DP - dim));
        staged[stage * stage_floats + (j / (DP - dim)) * DP + dim + j % (DP - dim)] = 0.0f;
    }
    const int begin = a.cu_tokens[entry], end = a.cu_tokens[entry + 1];
    if (a.max_count > 0 && end - begin > a.max_count) return;
    float* state = a.state + static_cast<size_t>(a.state_slots[entry]) * a.slot_floats +
                   (static_cast<size_t>(head) * a.vdim + first_column + local_column) * dim;

    float2 s[C][R / 2];
    bool live[C];
#pragma unroll
    for (int c = 0; c < C; ++c) {
        live[c] = !fetches && first_column + local_column + c * GROUPS < a.vdim;
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

    const int live_columns = min(columns, a.vdim - first_column);
    // The fetching warp's lane holds 16-byte pieces lane, lane + 32, ... of a token's q, k and decays (piece j belongs at
    // float 4 j of the token's row); their sources move on by one token at a time.
    constexpr int PIECES = (VECTORS * DP / 4 + 31) / 32;
    constexpr bool ONE_ROW = RULE != RULE_DELTA;  // all vectors of a token and head lie side by side
    const float* source[PIECES];
    bool wanted[PIECES];
    const size_t qk_step = static_cast<size_t>(a.qk_heads) * 2 * dim, gv_step = static_cast<size_t>(a.heads) * ((ONE_ROW ? VECTORS : 1) * dim + a.vdim);
    const float* qk_begin = a.qk + (static_cast<size_t>(begin) * a.qk_heads + qk_head) * 2 * dim;
    const float* gv_begin = a.gv + (static_cast<size_t>(begin) * a.heads + head) * ((ONE_ROW ? VECTORS : 1) * dim + a.vdim);
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
        const int j = lane + 32 * i, which = j / (DP / 4), d = j % (DP / 4) * 4;
        wanted[i] = which < VECTORS && d < dim;
        source[i] = ONE_ROW ? gv_begin + which * dim + d : which < 2 ? qk_begin + which * dim + d : gv_begin + d;
    }
    const float* value_source = gv_begin + (ONE_ROW ? VECTORS : 1) * dim + first_column;
    const float* scalar_source = a.scalars + (static_cast<size_t>(begin) * a.heads + head) * SCALARS;
    auto stage_tokens = [&](int chunk, float* stage) {
        const int count = min(SC, end - chunk);
        float* v_s = stage + SC * VECTORS * DP;
        for (int t = 0; t < count; ++t) {
            if (a.vector) {
#pragma unroll
                for (int i = 0; i < PIECES; ++i) {
                    if (wanted[i]) copy_async_16(stage + t * VECTORS * DP + 4 * (lane + 32 * i), source[i]);
                    source[i] += !ONE_ROW && (lane + 32 * i) / (DP / 4) < 2 ? qk_step : gv_step;
                }
            } else if constexpr (ONE_ROW) {
                const float* row = gv_begin + (chunk - begin + t) * gv_step;
                for (int j = lane; j < VECTORS * dim; j += 32) copy_async_4(stage + (t * VECTORS + j / dim) * DP + j % dim, row + j);
            } else {
                const float* qk = qk_begin + (chunk - begin + t) * qk_step;
                const float* gv = gv_begin + (chunk - begin + t) * gv_step;
                for (int j = lane; j < 2 * dim; j += 32) copy_async_4(stage + t * 3 * DP + j + (j < dim ? 0 : DP - dim), qk + j);
                for (int j = lane; j < dim; j += 32) copy_async_4(stage + (t * 3 + 2) * DP + j, gv + j);
            }
            for (int j = lane; j < live_columns; j += 32) copy_async_4(v_s + t * columns + j, value_source + j);
            if (lane < SCALARS) copy_async_4(v_s + SC * columns + SCALARS * t + lane, scalar_source + lane);
            value_source += gv_step;
            scalar_source += a.heads * SCALARS;
        }
        copy_async_commit();
    };

    auto store_results = [&](int chunk, const float* tile) {
        const int count = min(SC, end - chunk);
        float* out = a.out + (static_cast<size_t>(chunk) * a.heads + head) * a.vdim + first_column;
        for (int t = 0; t < count; ++t)
            for (int j = lane; j < live_columns; j += 32) out[static_cast<size_t>(t) * a.heads * a.vdim + j] = tile[t * columns + j];
    };

    __syncthreads();  // the zeros of the unused channels
    if (fetches && begin < end) {
        stage_tokens(begin, staged);
        copy_async_wait<0>();
    }
    __syncthreads();
    int buffer = 0;
    for (int chunk = begin; chunk < end; chunk += SC, buffer ^= 1) {
        const int count = min(SC, end - chunk);
        if (fetches) {
            if (chunk + SC < end) stage_tokens(chunk + SC, staged + (buffer ^ 1) * stage_floats);
            if (chunk > begin) store_results(chunk - SC, results + (buffer ^ 1) * SC * columns);
            copy_async_wait<0>();
            __syncthreads();
            continue;
        }
        const float* rows_s = staged + buffer * stage_floats + 4 * part;
        const float* v_s = staged + buffer * stage_floats + SC * VECTORS * DP;
        const float* scalars_s = v_s + SC * columns;
        // One token: its row is in registers already.
        auto walk = [&](const TokenRow<R, VECTORS>& row, int t) {
            const float2 scalars = *reinterpret_cast<const float2*>(scalars_s + SCALARS * t);  // the delta rule: beta, q . k
            const float q_dot_k = SCALARS > 2 ? scalars_s[SCALARS * t + (SCALARS > 2 ? 2 : 0)] : 0.0f;
            float dot_k[C], dot_q[C], v[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                v[c] = v_s[t * columns + local_column + c * GROUPS];  // a column behind the last one reads what is there and is never stored
                float2 on_k[2] = {make_float2(0.0f, 0.0f), make_float2(0.0f, 0.0f)};
                float2 on_q[2] = {make_float2(0.0f, 0.0f), make_float2(0.0f, 0.0f)};
#pragma unroll
                for (int i = 0; i < R / 2; ++i) {
                    if (RULE == RULE_DELTA) s[c][i] = __fmul2_rn(row.g[i], s[c][i]);
                    if (RULE != RULE_BONUS) on_k[i & 1] = __ffma2_rn(row.k[i], s[c][i], on_k[i & 1]);
                    on_q[i & 1] = __ffma2_rn(row.q[i], s[c][i], on_q[i & 1]);
                }
                dot_k[c] = (on_k[0].x + on_k[0].y) + (on_k[1].x + on_k[1].y);
                dot_q[c] = (on_q[0].x + on_q[0].y) + (on_q[1].x + on_q[1].y);
            }
#pragma unroll
            for (int offset = L / 2; offset > 0; offset >>= 1) {
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    if (RULE != RULE_BONUS) dot_k[c] += __shfl_xor_sync(0xffffffffu, dot_k[c], offset);
                    dot_q[c] += __shfl_xor_sync(0xffffffffu, dot_q[c], offset);
                }
            }
            float mine = 0.0f;  // lane number c of a group stores column c
#pragma unroll
            for (int c = 0; c < C; ++c) {
                float o;
                if constexpr (RULE == RULE_DELTA) {
                    const float u = scalars.x * (v[c] - dot_k[c]);
                    const float2 uu = make_float2(u, u);
#pragma unroll
                    for (int i = 0; i < R / 2; ++i) s[c][i] = __ffma2_rn(row.k[i], uu, s[c][i]);
                    o = fmaf(scalars.y, u, dot_q[c]);
                } else if constexpr (RULE == RULE_REMOVAL) {
                    const float read = -scalars.x * dot_k[c];
                    const float2 vv = make_float2(v[c], v[c]), rr = make_float2(read, read);
#pragma unroll
                    for (int i = 0; i < R / 2; ++i)
                        s[c][i] = __ffma2_rn(row.removed[i], rr, __ffma2_rn(row.k[i], vv, __fmul2_rn(row.g[i], s[c][i])));
                    o = fmaf(q_dot_k, v[c], fmaf(-scalars.y, dot_k[c], dot_q[c]));
                } else {
                    const float2 vv = make_float2(v[c], v[c]);
#pragma unroll
                    for (int i = 0; i < R / 2; ++i) s[c][i] = __ffma2_rn(row.g[i], s[c][i], __fmul2_rn(row.k[i], vv));
                    o = fmaf(scalars.x, v[c], dot_q[c]);
                }
                if (c == 0 || part == c) mine = o;
            }
            if (part < C) results[(buffer * SC + t) * columns + local_column + part * GROUPS] = mine;
        };
        TokenRow<R, VECTORS> even, odd;
        even.template load<L>(rows_s);
#pragma unroll 1
        for (int t = 0; t < count; t += 2) {
            if (t + 1 < count) odd.template load<L>(rows_s + (t + 1) * VECTORS * DP);
            walk(even, t);
            if (t + 1 >= count) break;
            if (t + 2 < count) even.template load<L>(rows_s + (t + 2) * VECTORS * DP);
            walk(odd, t + 1);
        }
        __syncthreads();
    }
    if (fetches && begin < end) store_results(begin + (end - begin - 1) / SC * SC, results + (buffer ^ 1) * SC * columns);
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

template <int RULE, int L, int R, int C, int SC>
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
    const size_t smem = static_cast<size_t>(2) * SC * (Rule<RULE>::VECTORS * L * R + 2 * columns + Rule<RULE>::SCALARS) * sizeof(float);
    if (smem > 48 * 1024)
        if (const int e = opt_in(delta_scan_kernel<RULE, L, R, C, SC>, 200 * 1024)) return e;
    const dim3 grid(entries, a.heads, (a.vdim + columns - 1) / columns);
    return launch_kernel_in_order(delta_scan_kernel<RULE, L, R, C, SC>, grid, (warps + 1) * 32, smem, stream, a);
}

template <int RULE>
static int dispatch_delta_scan(const DeltaScanArgs& a, int entries, cudaStream_t stream) {
    if (a.dim <= 32) return launch_delta_scan<RULE, 8, 4, 1, 16>(a, entries, stream);
    if (a.dim <= 64) return launch_delta_scan<RULE, 8, 8, 1, 16>(a, entries, stream);
    if (a.dim <= 128) return launch_delta_scan<RULE, 8, 16, 2, 16>(a, entries, stream);
    if (a.dim <= 256) return launch_delta_scan<RULE, 16, 16, 2, 8>(a, entries, stream);
    if (a.dim > MAX_DIM) return ME_ERR_UNSUPPORTED;
    if constexpr (RULE == RULE_REMOVAL)  // four vectors per token: a lane has room for fewer channels
        return launch_delta_scan<RULE, 32, 16, 2, 8>(a, entries, stream);
    else
        return launch_delta_scan<RULE, 16, 32, 1, 8>(a, entries, stream);
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
    return dispatch_delta_scan<RULE_DELTA>(a, entries, stream);
}

// The other rules, on what me_state_prepare made.  `max_count` > 0: entries with more tokens are left to me_state_chunks.
ME_EXPORT int me_state_walk(const float* rows, const float* scalars, const int* cu_tokens, const int* state_slots, const int* fresh,
                            float* state, long long slot_floats, float* out, int rule, int entries, int heads, int dim, int vdim,
                            int max_count, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (dim < 1 || vdim < 1 || heads < 1 || (rule != RULE_REMOVAL && rule != RULE_BONUS)) return ME_ERR_ARGUMENT;
    if (slot_floats < static_cast<long long>(heads) * dim * vdim) return ME_ERR_ARGUMENT;
    const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const int vector = dim % 4 == 0 && vdim % 4 == 0 && slot_floats % 4 == 0 && aligned(rows) && aligned(state);
    DeltaScanArgs a{nullptr, rows, scalars, cu_tokens, state_slots, fresh, state, (size_t)slot_floats, out, heads, heads, dim, vdim, vector, max_count};
    return rule == RULE_REMOVAL ? dispatch_delta_scan<RULE_REMOVAL>(a, entries, stream) : dispatch_delta_scan<RULE_BONUS>(a, entries, stream);
}
