// What stands between the products of a layer whose norm is elementwise and whose tokens look one step back.
//
// `tanh_norms`: the residual sum (partial sums of one or two sublayers, a bias, with or without the old stream), one or two
// dynamic-tanh norms of it, tanh(alpha * x) * w + b with a scalar alpha, and a token shift of the first norm's output, h + (h' -
// h) * shift with h' the previous token's h.  `token_mix`: that shift for a given h, with any number of weight vectors at once.
// `sum_rows`: the residual sum alone, rounded, into a column range.  `branch_norm_sum`: a weighted sum of sublayers that are
// RMS-normed first.  All arithmetic is float32.
//
// The shifts are column by column, so a thread walks a run of tokens with its columns and keeps the previous token's h in
// registers.  An entry's first token looks into the request's state (its last h of the step before, float32, in the slot of
// the request).  The thread of an entry's first token reads that state and then replaces it by the entry's last h, which it
// computes itself: no other thread touches the slot's columns, so nothing is read after it was replaced.  The stream is never
// updated in place (a run's first token needs the stream of the token in front of it): the sum goes to another buffer.
#include "common.cuh"

#include <algorithm>

constexpr int MIX_THREADS = 128;
constexpr int MIX_RUN = 8;            // tokens of a thread in a long step
constexpr int TANH_RUN = 4;           // the same for the norms, which hold more of a token
constexpr int MIX_RUN_TOKENS = 512;   // from this many tokens on

template <int V>
__device__ __forceinline__ void load_columns(const float* src, float (&x)[V]) {
    if constexpr (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(src);
        x[0] = q.x, x[1] = q.y, x[2] = q.z, x[3] = q.w;
    } else {
        x[0] = src[0];
    }
}
template <int V>
__device__ __forceinline__ void load_columns(const __nv_bfloat16* src, float (&x)[V]) {
    if constexpr (V == 4) {
        const uint2 q = *reinterpret_cast<const uint2*>(src);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
        x[0] = a.x, x[1] = a.y, x[2] = b.x, x[3] = b.y;
    } else {
        x[0] = to_float(src[0]);
    }
}
template <int V>
__device__ __forceinline__ void store_columns(float* dst, const float (&x)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1], x[2], x[3]);
    else dst[0] = x[0];
}
template <int V>
__device__ __forceinline__ void store_columns(__nv_bfloat16* dst, const float (&x)[V]) {
    if constexpr (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1]), b = __floats2bfloat162_rn(x[2], x[3]);
        *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else {
        dst[0] = from_float<__nv_bfloat16>(x[0]);
    }
}

// ------------------------------------------------------------------------- residual sum

// x + (sum of first's partial sums + sum of second's) + bias; null terms are absent.
struct StreamSum {
    const float* x;  // [tokens][width]
    const float* first;
    int first_splits;
    size_t first_stride;
    const float* second;
    int second_splits;
    size_t second_stride;
    const float* bias;  // [width]
    int width;

    // WHOLE: there is a stream and each sublayer brings one sum (the steps of many tokens, whose products are not split).
    template <int V, bool WHOLE = false>
    __device__ __forceinline__ void load(size_t token, int column, float (&sum)[V]) const {
        const size_t at = token * width + column;
        float part[V];
        if constexpr (WHOLE) {
            float y[V];
            load_columns<V>(first + at, sum);
            load_columns<V>(second + at, y);
            load_columns<V>(x + at, part);
#pragma unroll
            for (int i = 0; i < V; ++i) sum[i] = (sum[i] + y[i]) + part[i];
            return;
        }
#pragma unroll
        for (int i = 0; i < V; ++i) sum[i] = 0.0f;
        if (first) {
#pragma unroll 4
            for (int s = 0; s < first_splits; ++s) {
                load_columns<V>(first + s * first_stride + at, part);
#pragma unroll
                for (int i = 0; i < V; ++i) sum[i] += part[i];
            }
        }
        if (second) {
#pragma unroll 4
            for (int s = 0; s < second_splits; ++s) {
                load_columns<V>(second + s * second_stride + at, part);
#pragma unroll
                for (int i = 0; i < V; ++i) sum[i] += part[i];
            }
        }
        if (bias) {
            load_columns<V>(bias + column, part);
#pragma unroll
            for (int i = 0; i < V; ++i) sum[i] += part[i];
        }
        if (x) {
            load_columns<V>(x + at, part);
#pragma unroll
            for (int i = 0; i < V; ++i) sum[i] += part[i];
        }
    }
};

// ------------------------------------------------------------------------------ tanh norms

struct TanhNorm {
    const float* weight;  // [width]
    const float* bias;    // [width]
    const float* alpha;   // one number
    void* out;            // [tokens][width] in the output type
};

struct TanhArgs {
    StreamSum sum;
    float* x_out;       // [tokens][width] the summed stream (another buffer than sum.x), or null
    TanhNorm norms[2];  // the second may be absent (a null weight)
    const float* shift;  // [width] token shift of the first norm's output, or null
    float* state;        // [slots + 1][width] (with shift)
    const int* entry_of_token;
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    const int* rows;  // the tokens to take, or null: all
    int tokens, width;
};

// tanh from the exponential, 1 - 2 / (e^(2|z|) + 1), and below a quarter, where that difference loses digits, from its power
// series up to z^9 (the next term is 2e-9 of the value there).
__device__ __forceinline__ float tanh_of(float z) {
    const float size = fabsf(z), square = z * z;
    float series = fmaf(square, 62.0f / 2835.0f, -17.0f / 315.0f);
    series = fmaf(series, square, 2.0f / 15.0f);
    series = fmaf(series, square, -1.0f / 3.0f);
    series = fmaf(series * square, z, z);
    const float far = copysignf(1.0f - __fdividef(2.0f, __expf(fminf(2.0f * size, 80.0f)) + 1.0f), z);
    return size < 0.25f ? series : far;
}

template <int V>
struct TanhColumns {
    float weight[V], bias[V], alpha;
    __device__ __forceinline__ void load(const TanhNorm& n, int column) {
        load_columns<V>(n.weight + column, weight);
        load_columns<V>(n.bias + column, bias);
        alpha = *n.alpha;
    }
    __device__ __forceinline__ void apply(const float (&x)[V], float (&y)[V]) const {
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = fmaf(tanh_of(alpha * x[i]), weight[i], bias[i]);
    }
};

template <typename OutT, int V, int RUN, bool WHOLE = false>
__global__ void __launch_bounds__(MIX_THREADS) tanh_norms_kernel(TanhArgs a) {
    const int column = (blockIdx.y * MIX_THREADS + threadIdx.x) * V, begin = blockIdx.x * RUN;
    if (column >= a.width) return;
    TanhColumns<V> first, second;
    float shift[V];
    first.load(a.norms[0], column);
    if (a.norms[1].weight) second.load(a.norms[1], column);
    if (a.shift) load_columns<V>(a.shift + column, shift);
    pdl_trigger();
    pdl_wait();
    float x[RUN][V];
#pragma unroll
    for (int t = 0; t < RUN; ++t)
        if (begin + t < a.tokens) a.sum.template load<V, WHOLE>(a.rows ? a.rows[begin + t] : begin + t, column, x[t]);
    float previous[V];
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
        const int token = begin + t;
        if (token >= a.tokens) break;
        const size_t at = static_cast<size_t>(token) * a.width + column;
        if (a.x_out) store_columns<V>(a.x_out + at, x[t]);
        float h[V], y[V];
        first.apply(x[t], h);
        if (a.shift) {
            const int entry = a.entry_of_token[token], entry_begin = a.cu_tokens[entry];
            if (token == entry_begin) {
                float* slot = a.state + static_cast<size_t>(a.state_slots[entry]) * a.width + column;
                if (a.fresh[entry]) {
#pragma unroll
                    for (int i = 0; i < V; ++i) previous[i] = 0.0f;
                } else {
                    load_columns<V>(slot, previous);
                }
                const int last = a.cu_tokens[entry + 1] - 1;
                float newest[V];
                if (last == token) {
                    store_columns<V>(slot, h);
                } else {
                    a.sum.template load<V, WHOLE>(last, column, newest);
                    first.apply(newest, newest);
                    store_columns<V>(slot, newest);
                }
            } else if (t == 0) {
                a.sum.template load<V, WHOLE>(token - 1, column, previous);
                first.apply(previous, previous);
            }
#pragma unroll
            for (int i = 0; i < V; ++i) {
                y[i] = fmaf(previous[i] - h[i], shift[i], h[i]);
                previous[i] = h[i];
            }
            store_columns<V>(static_cast<OutT*>(a.norms[0].out) + at, y);
        } else {
            store_columns<V>(static_cast<OutT*>(a.norms[0].out) + at, h);
        }
        if (a.norms[1].weight) {
            second.apply(x[t], y);
            store_columns<V>(static_cast<OutT*>(a.norms[1].out) + at, y);
        }
    }
}

static bool aligned(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }
static bool sum_takes_vectors(const StreamSum& s) {
    return s.width % 4 == 0 && s.first_stride % 4 == 0 && s.second_stride % 4 == 0 && aligned(s.x) && aligned(s.first) &&
           aligned(s.second) && aligned(s.bias);
}

template <typename OutT>
static int launch_tanh_norms(const TanhArgs& a, cudaStream_t stream) {
    // the choice of vectors follows from the sizes and the engine's buffers alone
    bool vector = sum_takes_vectors(a.sum) && aligned(a.x_out) && aligned(a.shift) && aligned(a.state);
    for (const TanhNorm& n : a.norms) vector = vector && aligned(n.weight) && aligned(n.bias) && aligned(n.out);
    const int columns = MIX_THREADS * (vector ? 4 : 1), run = a.tokens >= MIX_RUN_TOKENS && vector ? TANH_RUN : 1;
    const dim3 grid((a.tokens + run - 1) / run, (a.width + columns - 1) / columns);
    if (!vector) return launch_kernel(tanh_norms_kernel<OutT, 1, 1>, grid, MIX_THREADS, 0, stream, a);
    if (run == 1) return launch_kernel(tanh_norms_kernel<OutT, 4, 1>, grid, MIX_THREADS, 0, stream, a);
    if (a.sum.x && a.sum.first && a.sum.first_splits == 1 && a.sum.second && a.sum.second_splits == 1 && !a.sum.bias)
        return launch_kernel(tanh_norms_kernel<OutT, 4, TANH_RUN, true>, grid, MIX_THREADS, 0, stream, a);
    return launch_kernel(tanh_norms_kernel<OutT, 4, TANH_RUN>, grid, MIX_THREADS, 0, stream, a);
}

ME_EXPORT int me_tanh_norms(const float* x, const float* first, int first_splits, long long first_stride, const float* second,
                            int second_splits, long long second_stride, const float* bias, float* x_out, const float* weight_a,
                            const float* bias_a, const float* alpha_a, void* out_a, const float* weight_b, const float* bias_b,
                            const float* alpha_b, void* out_b, const float* shift, float* state, const int* entry_of_token,
                            const int* cu_tokens, const int* state_slots, const int* fresh, const int* rows, int out_type,
                            int tokens, int width, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (width < 1 || (shift && (!state || rows)) || (x_out && (x_out == x || rows))) return ME_ERR_ARGUMENT;
    TanhArgs a{{x, first, first_splits, (size_t)first_stride, second, second_splits, (size_t)second_stride, bias, width},
               x_out, {{weight_a, bias_a, alpha_a, out_a}, {weight_b, bias_b, alpha_b, out_b}}, shift, state, entry_of_token,
               cu_tokens, state_slots, fresh, rows, tokens, width};
    return out_type == ME_BF16 ? launch_tanh_norms<__nv_bfloat16>(a, stream) : launch_tanh_norms<float>(a, stream);
}

// ----------------------------------------------------------------------------- sum into columns

template <typename OutT, int V>
__global__ void __launch_bounds__(MIX_THREADS) sum_rows_kernel(StreamSum sum, OutT* __restrict__ out, int out_width, int first_column) {
    const int column = (blockIdx.y * MIX_THREADS + threadIdx.x) * V;
    if (column >= sum.width) return;
    pdl_trigger();
    pdl_wait();
    float x[V];
    sum.load<V>(blockIdx.x, column, x);
    store_columns<V>(out + static_cast<size_t>(blockIdx.x) * out_width + first_column + column, x);
}

template <typename OutT>
static int launch_sum_rows(const StreamSum& sum, OutT* out, int out_width, int first_column, int tokens, cudaStream_t stream) {
    const bool vector = sum_takes_vectors(sum) && aligned(out) && out_width % 4 == 0 && first_column % 4 == 0;
    const int columns = MIX_THREADS * (vector ? 4 : 1);
    const dim3 grid(tokens, (sum.width + columns - 1) / columns);
    return vector ? launch_kernel(sum_rows_kernel<OutT, 4>, grid, MIX_THREADS, 0, stream, sum, out, out_width, first_column)
                  : launch_kernel(sum_rows_kernel<OutT, 1>, grid, MIX_THREADS, 0, stream, sum, out, out_width, first_column);
}

ME_EXPORT int me_sum_rows(const float* x, const float* first, int first_splits, long long first_stride, const float* second,
                          int second_splits, long long second_stride, const float* bias, void* out, int out_type, int out_width,
                          int first_column, int tokens, int width, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (width < 1 || first_column < 0 || first_column + width > out_width) return ME_ERR_ARGUMENT;
    const StreamSum sum{x, first, first_splits, (size_t)first_stride, second, second_splits, (size_t)second_stride, bias, width};
    return out_type == ME_BF16 ? launch_sum_rows(sum, static_cast<__nv_bfloat16*>(out), out_width, first_column, tokens, stream)
                               : launch_sum_rows(sum, static_cast<float*>(out), out_width, first_column, tokens, stream);
}

// ------------------------------------------------------------------------------------ token mix

struct MixArgs {
    const void* h;    // [tokens][width]
    const float* mu;  // [count][width]
    void* out;        // [count][tokens][width]
    float* state;     // slot s starts at s * slot_floats: the request's last h
    size_t slot_floats;
    const int* entry_of_token;
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    int tokens, width, count;
};

template <typename T, int V, int RUN>
__global__ void __launch_bounds__(MIX_THREADS) token_mix_kernel(MixArgs a) {
    const int column = (blockIdx.y * MIX_THREADS + threadIdx.x) * V, begin = blockIdx.x * RUN;
    if (column >= a.width) return;
    pdl_trigger();
    pdl_wait();
    const T* h = static_cast<const T*>(a.h) + column;
    float x[RUN][V], previous[RUN][V];
#pragma unroll
    for (int t = 0; t < RUN; ++t)
        if (begin + t < a.tokens) load_columns<V>(h + static_cast<size_t>(begin + t) * a.width, x[t]);
#pragma unroll
    for (int t = 0; t < RUN; ++t) {
        const int token = begin + t;
        if (token >= a.tokens) break;
        const int entry = a.entry_of_token[token];
        if (token != a.cu_tokens[entry]) {
            if (t == 0) {
                load_columns<V>(h + static_cast<size_t>(token - 1) * a.width, previous[t]);
            } else {
#pragma unroll
                for (int i = 0; i < V; ++i) previous[t][i] = x[t > 0 ? t - 1 : 0][i];
            }
            continue;
        }
        float* slot = a.state + a.state_slots[entry] * a.slot_floats + column;
        if (a.fresh[entry]) {
#pragma unroll
            for (int i = 0; i < V; ++i) previous[t][i] = 0.0f;
        } else {
            load_columns<V>(slot, previous[t]);
        }
        float newest[V];
        load_columns<V>(h + static_cast<size_t>(a.cu_tokens[entry + 1] - 1) * a.width, newest);
        store_columns<V>(slot, newest);
    }
    for (int s = 0; s < a.count; ++s) {
        float mu[V], y[V];
        load_columns<V>(a.mu + static_cast<size_t>(s) * a.width + column, mu);
        T* out = static_cast<T*>(a.out) + static_cast<size_t>(s) * a.tokens * a.width + column;
#pragma unroll
        for (int t = 0; t < RUN; ++t) {
            if (begin + t >= a.tokens) break;
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] = fmaf(previous[t][i] - x[t][i], mu[i], x[t][i]);
            store_columns<V>(out + static_cast<size_t>(begin + t) * a.width, y);
        }
    }
}

template <typename T>
static int launch_token_mix(const MixArgs& a, cudaStream_t stream) {
    const bool vector = a.width % 4 == 0 && a.slot_floats % 4 == 0 && aligned(a.h) && aligned(a.mu) && aligned(a.out) && aligned(a.state);
    const int columns = MIX_THREADS * (vector ? 4 : 1), run = a.tokens >= MIX_RUN_TOKENS && vector ? MIX_RUN : 1;
    const dim3 grid((a.tokens + run - 1) / run, (a.width + columns - 1) / columns);
    if (!vector) return launch_kernel(token_mix_kernel<T, 1, 1>, grid, MIX_THREADS, 0, stream, a);
    if (run == 1) return launch_kernel(token_mix_kernel<T, 4, 1>, grid, MIX_THREADS, 0, stream, a);
    return launch_kernel(token_mix_kernel<T, 4, MIX_RUN>, grid, MIX_THREADS, 0, stream, a);
}

// `state` points at the first slot's last h; slots are slot_floats apart.
ME_EXPORT int me_token_mix(const void* h, int type, const float* mu, void* out, float* state, long long slot_floats,
                           const int* entry_of_token, const int* cu_tokens, const int* state_slots, const int* fresh, int tokens,
                           int width, int count, cudaStream_t stream) {
    if (tokens <= 0 || count <= 0) return 0;
    if (width < 1 || slot_floats < width || h == out) return ME_ERR_ARGUMENT;
    MixArgs a{h, mu, out, state, (size_t)slot_floats, entry_of_token, cu_tokens, state_slots, fresh, tokens, width, count};
    return type == ME_BF16 ? launch_token_mix<__nv_bfloat16>(a, stream) : launch_token_mix<float>(a, stream);
}

// ----------------------------------------------------------------------- normed branches joined

// out[t] = sum_b factor_b * weight_b * y_b / sqrt(mean(y_b^2) + eps_b) with y_b the sum of the branch's partial sums: one
// block per token, the sums in shared memory between the two passes.
constexpr int NORM_BRANCHES = 4;
constexpr int BRANCH_THREADS = 256;

struct BranchNormArgs {
    const float* partial[NORM_BRANCHES];
    const float* weight[NORM_BRANCHES];
    int splits[NORM_BRANCHES];
    size_t stride[NORM_BRANCHES];
    float factor[NORM_BRANCHES], eps[NORM_BRANCHES];
    float* out;
    int branches, width;
};

template <int V>
__global__ void __launch_bounds__(BRANCH_THREADS) branch_norm_sum_kernel(BranchNormArgs a) {
    extern __shared__ __align__(16) float sums[];  // [branches][width]
    __shared__ float warp_sums[NORM_BRANCHES][BRANCH_THREADS / 32];
    const size_t row = static_cast<size_t>(blockIdx.x) * a.width;
    pdl_trigger();
    pdl_wait();
    float squares[NORM_BRANCHES] = {};
    for (int c = threadIdx.x * V; c < a.width; c += BRANCH_THREADS * V) {
#pragma unroll
        for (int b = 0; b < NORM_BRANCHES; ++b) {
            if (b >= a.branches) break;
            float y[V] = {}, part[V];
#pragma unroll 4
            for (int s = 0; s < a.splits[b]; ++s) {
                load_columns<V>(a.partial[b] + s * a.stride[b] + row + c, part);
#pragma unroll
                for (int i = 0; i < V; ++i) y[i] += part[i];
            }
#pragma unroll
            for (int i = 0; i < V; ++i) squares[b] = fmaf(y[i], y[i], squares[b]);
            store_columns<V>(sums + b * a.width + c, y);
        }
    }
#pragma unroll
    for (int b = 0; b < NORM_BRANCHES; ++b) {
        const float sum = warp_sum(squares[b]);
        if ((threadIdx.x & 31) == 0) warp_sums[b][threadIdx.x >> 5] = sum;
    }
    __syncthreads();
    float scale[NORM_BRANCHES];
#pragma unroll
    for (int b = 0; b < NORM_BRANCHES; ++b) {
        float sum = 0.0f;
#pragma unroll
        for (int w = 0; w < BRANCH_THREADS / 32; ++w) sum += warp_sums[b][w];
        scale[b] = b < a.branches ? a.factor[b] * rsqrtf(sum / static_cast<float>(a.width) + a.eps[b]) : 0.0f;
    }
    for (int c = threadIdx.x * V; c < a.width; c += BRANCH_THREADS * V) {  // a thread reads what it wrote itself
        float total[V] = {};
#pragma unroll
        for (int b = 0; b < NORM_BRANCHES; ++b) {
            if (b >= a.branches) break;
            float y[V], w[V];
            load_columns<V>(sums + b * a.width + c, y);
            load_columns<V>(a.weight[b] + c, w);
#pragma unroll
            for (int i = 0; i < V; ++i) total[i] = fmaf(w[i] * scale[b], y[i], total[i]);
        }
        store_columns<V>(a.out + row + c, total);
    }
}

ME_EXPORT int me_branch_norm_sum(const float* const* partials, const int* splits, const long long* strides, const float* const* weights,
                                 const float* factors, const float* eps, int branches, float* out, int tokens, int width,
                                 cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (branches < 1 || branches > NORM_BRANCHES) return ME_ERR_UNSUPPORTED;
    BranchNormArgs a{};
    bool vector = width % 4 == 0 && aligned(out);
    for (int b = 0; b < branches; ++b) {
        a.partial[b] = partials[b], a.weight[b] = weights[b], a.splits[b] = splits[b], a.stride[b] = (size_t)strides[b];
        a.factor[b] = factors[b], a.eps[b] = eps[b];
        vector = vector && aligned(partials[b]) && aligned(weights[b]) && strides[b] % 4 == 0;
    }
    a.out = out, a.branches = branches, a.width = width;
    const size_t smem = static_cast<size_t>(branches) * width * sizeof(float);
    if (smem > 200 * 1024) return ME_ERR_UNSUPPORTED;
    static SharedMemoryOptIn vector_opt_in, plain_opt_in;
    if (smem > 40 * 1024) {
        const int code = vector ? vector_opt_in(branch_norm_sum_kernel<4>, 200 * 1024) : plain_opt_in(branch_norm_sum_kernel<1>, 200 * 1024);
        if (code) return code;
    }
    return vector ? launch_kernel(branch_norm_sum_kernel<4>, tokens, BRANCH_THREADS, smem, stream, a)
                  : launch_kernel(branch_norm_sum_kernel<1>, tokens, BRANCH_THREADS, smem, stream, a);
}
