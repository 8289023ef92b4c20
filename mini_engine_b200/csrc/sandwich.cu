// Kernels of layers whose sublayers stand between two norms and behind a gate, with a short convolution over time in
// front of the mixer.
//
// `sandwich_norm`: everything between a sublayer's last product and the next sublayer's input, one block per row:
//
//   y    = (sum_s pending[s] + bias) * sigmoid(sum_s gate[s] + gate_bias)      (gate and biases may be absent)
//   x   += out_weight * y / rms(y)                                             (the residual sum)
//   out  = weight * x / rms(x)                                                 (the next sublayer's input)
//
// all in float32 with one rounding at the end.  `input_convolution`: h + conv(h) over the flat batch of a step, from and
// into each request's slot of past inputs.
#include "common.cuh"

#include <algorithm>

constexpr int MAX_SPLITS = 8;  // partial sums whose loads are issued together

__device__ __forceinline__ void add4(float4& a, const float4& b) { a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w; }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ void store4(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* dst, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 packed;
    packed.x = *reinterpret_cast<uint32_t*>(&lo);
    packed.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = packed;
}

struct SandwichArgs {
    float* x;              // [tokens][hidden], advanced unless `rows` is given
    const float* pending;  // [splits][tokens][hidden]
    int splits;
    size_t split_stride;
    const float* bias;  // [hidden] or null
    const float* gate;  // [gate_splits][tokens][hidden] or null
    int gate_splits;
    size_t gate_stride;
    const float* gate_bias;   // [hidden] or null
    const float* out_weight;  // [hidden]
    float out_eps;
    const float* weight;  // [hidden]
    float eps;
    void* out;
    const int* rows;  // null, or the source row of every output row
    int hidden;
};

// The sum of a value per thread over the block: butterfly in a warp, warps in ascending order.
template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.0f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += scratch[w];
    return total;
}

// VEC: four columns per thread and step (16-byte loads; every pointer aligned, at most SPLITS partial sums: 1 for the long
// steps, whose products are not split, so that more blocks fit an SM).  Which columns a thread adds follows from the width
// alone, so a row's statistics are the same bits in every step.
template <typename OutT, bool VEC, int THREADS, int SPLITS>
__global__ void __launch_bounds__(THREADS) sandwich_norm_kernel(SandwichArgs a) {
    extern __shared__ __align__(16) float row[];  // [hidden]: the gated output, then the new stream
    __shared__ float scratch[2][THREADS / 32];
    pdl_trigger();
    const int src = a.rows ? a.rows[blockIdx.x] : static_cast<int>(blockIdx.x);
    pdl_wait();
    const size_t offset = static_cast<size_t>(src) * a.hidden;
    float* x_row = a.x + offset;
    OutT* out = static_cast<OutT*>(a.out) + static_cast<size_t>(blockIdx.x) * a.hidden;
    const float width = static_cast<float>(a.hidden);
    float squares = 0.0f;
    if constexpr (VEC) {
        for (int i = threadIdx.x * 4; i < a.hidden; i += THREADS * 4) {
            float4 part[SPLITS], gates[SPLITS];
#pragma unroll
            for (int s = 0; s < SPLITS; ++s) {
                if (s < a.splits) part[s] = *reinterpret_cast<const float4*>(a.pending + s * a.split_stride + offset + i);
                if (a.gate && s < a.gate_splits) gates[s] = *reinterpret_cast<const float4*>(a.gate + s * a.gate_stride + offset + i);
            }
            float4 y = part[0];
#pragma unroll
            for (int s = 1; s < SPLITS; ++s)
                if (s < a.splits) add4(y, part[s]);
            if (a.bias) add4(y, *reinterpret_cast<const float4*>(a.bias + i));
            if (a.gate) {
                float4 g = gates[0];
#pragma unroll
                for (int s = 1; s < SPLITS; ++s)
                    if (s < a.gate_splits) add4(g, gates[s]);
                if (a.gate_bias) add4(g, *reinterpret_cast<const float4*>(a.gate_bias + i));
                y.x *= sigmoid(g.x), y.y *= sigmoid(g.y), y.z *= sigmoid(g.z), y.w *= sigmoid(g.w);
            }
            *reinterpret_cast<float4*>(row + i) = y;
            squares = fmaf(y.x, y.x, squares), squares = fmaf(y.y, y.y, squares);
            squares = fmaf(y.z, y.z, squares), squares = fmaf(y.w, y.w, squares);
        }
    } else {
        for (int i = threadIdx.x; i < a.hidden; i += THREADS) {
            float y = a.pending[offset + i];
            for (int s = 1; s < a.splits; ++s) y += a.pending[s * a.split_stride + offset + i];
            if (a.bias) y += a.bias[i];
            if (a.gate) {
                float g = a.gate[offset + i];
                for (int s = 1; s < a.gate_splits; ++s) g += a.gate[s * a.gate_stride + offset + i];
                if (a.gate_bias) g += a.gate_bias[i];
                y *= sigmoid(g);
            }
            row[i] = y;
            squares = fmaf(y, y, squares);
        }
    }
    // a thread reads back only what it wrote to `row` itself: no barrier is needed for that
    const float inv_out = rsqrtf(block_sum<THREADS>(squares, scratch[0]) / width + a.out_eps);
    squares = 0.0f;
    if constexpr (VEC) {
        for (int i = threadIdx.x * 4; i < a.hidden; i += THREADS * 4) {
            const float4 y = *reinterpret_cast<const float4*>(row + i), w = *reinterpret_cast<const float4*>(a.out_weight + i);
            float4 v = *reinterpret_cast<const float4*>(x_row + i);
            v.x += w.x * (y.x * inv_out), v.y += w.y * (y.y * inv_out), v.z += w.z * (y.z * inv_out), v.w += w.w * (y.w * inv_out);
            if (!a.rows) *reinterpret_cast<float4*>(x_row + i) = v;
            *reinterpret_cast<float4*>(row + i) = v;
            squares = fmaf(v.x, v.x, squares), squares = fmaf(v.y, v.y, squares);
            squares = fmaf(v.z, v.z, squares), squares = fmaf(v.w, v.w, squares);
        }
    } else {
        for (int i = threadIdx.x; i < a.hidden; i += THREADS) {
            const float v = x_row[i] + a.out_weight[i] * (row[i] * inv_out);
            if (!a.rows) x_row[i] = v;
            row[i] = v;
            squares = fmaf(v, v, squares);
        }
    }
    const float inv = rsqrtf(block_sum<THREADS>(squares, scratch[1]) / width + a.eps);
    if constexpr (VEC) {
        for (int i = threadIdx.x * 4; i < a.hidden; i += THREADS * 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + i), w = *reinterpret_cast<const float4*>(a.weight + i);
            store4(out + i, make_float4(w.x * (v.x * inv), w.y * (v.y * inv), w.z * (v.z * inv), w.w * (v.w * inv)));
        }
    } else {
        for (int i = threadIdx.x; i < a.hidden; i += THREADS) out[i] = from_float<OutT>(a.weight[i] * (row[i] * inv));
    }
}

template <typename OutT, bool VEC, int THREADS, int SPLITS>
static int launch_sandwich(const SandwichArgs& a, int count, cudaStream_t stream) {
    static SharedMemoryOptIn opt_in;
    const size_t smem = static_cast<size_t>(a.hidden) * sizeof(float);
    auto kernel = sandwich_norm_kernel<OutT, VEC, THREADS, SPLITS>;
    if (smem > 48 * 1024)
        if (const int e = opt_in(kernel, 200 * 1024)) return e;
    return launch_kernel(kernel, count, THREADS, smem, stream, a);
}

template <typename OutT, int THREADS>
static int launch_sandwich_threads(const SandwichArgs& a, int count, bool vec, cudaStream_t stream) {
    if (!vec) return launch_sandwich<OutT, false, THREADS, 1>(a, count, stream);
    if (a.splits == 1 && a.gate_splits <= 1) return launch_sandwich<OutT, true, THREADS, 1>(a, count, stream);
    return launch_sandwich<OutT, true, THREADS, MAX_SPLITS>(a, count, stream);
}

template <typename OutT>
static int launch_sandwich_width(const SandwichArgs& a, int count, bool vec, cudaStream_t stream) {
    return a.hidden > 2048 ? launch_sandwich_threads<OutT, 512>(a, count, vec, stream) : launch_sandwich_threads<OutT, 256>(a, count, vec, stream);
}

static bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

ME_EXPORT int me_sandwich_norm(float* x, const float* pending, int splits, long long split_stride, const float* bias,
                               const float* gate, int gate_splits, long long gate_stride, const float* gate_bias,
                               const float* out_weight, float out_eps, const float* weight, float eps, void* out, int out_type,
                               const int* rows, int count, int hidden, cudaStream_t stream) {
    if (count <= 0) return 0;
    if (pending == nullptr || splits < 1 || (gate != nullptr && gate_splits < 1)) return ME_ERR_ARGUMENT;
    if (static_cast<size_t>(hidden) * sizeof(float) > 200 * 1024) return ME_ERR_UNSUPPORTED;
    SandwichArgs a{x, pending, splits, (size_t)split_stride, bias, gate, gate_splits, (size_t)gate_stride, gate_bias,
                   out_weight, out_eps, weight, eps, out, rows, hidden};
    // The choice follows from the width and the engine's buffers, never from the rows of the step.
    const bool vec = hidden % 4 == 0 && splits <= MAX_SPLITS && gate_splits <= MAX_SPLITS && split_stride % 4 == 0 && gate_stride % 4 == 0 &&
                     aligned16(x) && aligned16(pending) && aligned16(bias) && aligned16(gate) && aligned16(gate_bias) &&
                     aligned16(out_weight) && aligned16(weight) && aligned16(out);
    return out_type == ME_BF16 ? launch_sandwich_width<__nv_bfloat16>(a, count, vec, stream)
                               : launch_sandwich_width<float>(a, count, vec, stream);
}

// ------------------------------------------------------------------ input convolution over time

// out_t = h_t + sum_j taps[j][c] * h_(t - K + 1 + j) per channel c, zeros in front of the sequence.  `state` holds the last
// K - 1 inputs of every request, oldest first ([slots + 1][K - 1][width] float32).  A thread takes V channels of
// `run` tokens; those with K - 1 tokens of their entry in front of them slide a window of inputs in registers (KC = K; KC =
// 0: more taps than that, read again for every token).  The first K - 1 tokens of an entry read the request's past; the
// thread that holds the entry's first token computes all of them and then leaves the entry's last inputs in the slot, so
// that nothing is read after it was replaced.  Both forms add the products in the same order.
constexpr int MAX_TAPS = 16;
constexpr int CONV_RUN = 8;            // tokens of a thread in a long step
constexpr int CONV_RUN_TOKENS = 512;   // from this many tokens on

struct ConvArgs {
    const void* h;      // [tokens][width]
    const float* taps;  // [K][width]
    const int* entry_of_token;
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    float* state;
    void* out;  // [tokens][width]
    int tokens, width, K, run;
};

template <int V>
__device__ __forceinline__ void load_row(const float* src, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 q = *reinterpret_cast<const float4*>(src);
        v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
        v[0] = src[0];
    }
}
template <int V>
__device__ __forceinline__ void load_row(const __nv_bfloat16* src, float (&v)[V]) {
    if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(src);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = lo.x, v[1] = lo.y, v[2] = hi.x, v[3] = hi.y;
    } else {
        v[0] = to_float(src[0]);
    }
}

template <int V>
__device__ __forceinline__ void store_row(float* dst, const float (&v)[V]) {
    if constexpr (V == 4) store4(dst, make_float4(v[0], v[1], v[2], v[3]));
    else dst[0] = v[0];
}
template <int V>
__device__ __forceinline__ void store_row(__nv_bfloat16* dst, const float (&v)[V]) {
    if constexpr (V == 4) store4(dst, make_float4(v[0], v[1], v[2], v[3]));
    else dst[0] = from_float<__nv_bfloat16>(v[0]);
}

template <typename T, int V, int KC>
__global__ void __launch_bounds__(256) input_convolution_kernel(ConvArgs a) {
    constexpr int WINDOW = KC > 1 ? KC - 1 : 1;
    const int c = (blockIdx.y * 256 + threadIdx.x) * V;
    const int run_begin = blockIdx.x * a.run, run_end = min(run_begin + a.run, a.tokens), K = a.K;
    pdl_trigger();
    pdl_wait();
    if (c >= a.width) return;
    const T* h = static_cast<const T*>(a.h);
    T* out = static_cast<T*>(a.out);
    float taps[KC > 0 ? KC : 1][V], held[WINDOW][V];
    if constexpr (KC > 0) {
#pragma unroll
        for (int j = 0; j < KC; ++j) load_row<V>(a.taps + static_cast<size_t>(j) * a.width + c, taps[j]);
    }
    int filled = -1;  // the token in front of which the window stands
    for (int t = run_begin; t < run_end; ++t) {
        const int entry = a.entry_of_token[t], first = a.cu_tokens[entry], n0 = t - first;
        if (n0 > 0 && n0 < K - 1) continue;  // done by the thread of the entry's first token
        if (KC > 0 && n0 >= K - 1) {
            if (filled != t) {
#pragma unroll
                for (int w = 0; w < KC - 1; ++w) load_row<V>(h + static_cast<size_t>(t - (KC - 1) + w) * a.width + c, held[w]);
            }
            float now[V], sum[V];
            load_row<V>(h + static_cast<size_t>(t) * a.width + c, now);
#pragma unroll
            for (int v = 0; v < V; ++v) {
                sum[v] = 0.0f;
#pragma unroll
                for (int w = 0; w < KC - 1; ++w) sum[v] = fmaf(taps[w][v], held[w][v], sum[v]);
                sum[v] = now[v] + fmaf(taps[KC > 0 ? KC - 1 : 0][v], now[v], sum[v]);
#pragma unroll
                for (int w = 0; w + 1 < KC - 1; ++w) held[w][v] = held[w + 1][v];
                if (KC > 1) held[WINDOW - 1][v] = now[v];
            }
            filled = t + 1;
            store_row<V>(out + static_cast<size_t>(t) * a.width + c, sum);
            continue;
        }
        // the entry's first tokens, or more taps than the window holds
        const int count = a.cu_tokens[entry + 1] - first;
        const int run = n0 == 0 ? min(count, max(K - 1, 1)) : 1;
        float* slot = a.state ? a.state + static_cast<size_t>(a.state_slots[entry]) * (K - 1) * a.width + c : nullptr;
        const bool past = slot != nullptr && a.fresh[entry] == 0;
        for (int n = n0; n < n0 + run; ++n) {
            const size_t at = static_cast<size_t>(first + n) * a.width + c;
            float sum[V], x[V], w[V];
#pragma unroll
            for (int v = 0; v < V; ++v) sum[v] = 0.0f;
            for (int j = 0; j < K; ++j) {
                const int from = n - (K - 1) + j;  // among the entry's tokens; negative: an earlier step's
                if (from >= 0) load_row<V>(h + static_cast<size_t>(first + from) * a.width + c, x);
                else if (past) load_row<V>(slot + static_cast<size_t>(from + K - 1) * a.width, x);
                else continue;
                load_row<V>(a.taps + static_cast<size_t>(j) * a.width + c, w);
#pragma unroll
                for (int v = 0; v < V; ++v) sum[v] = fmaf(w[v], x[v], sum[v]);
            }
            load_row<V>(h + at, x);
#pragma unroll
            for (int v = 0; v < V; ++v) sum[v] = x[v] + sum[v];
            store_row<V>(out + at, sum);
        }
        if (n0 != 0 || slot == nullptr) continue;
        for (int i = 0; i < K - 1; ++i) {  // ascending: row i is replaced by row i + count, which is read before it is replaced
            const int from = count - (K - 1) + i;
            float x[V];
#pragma unroll
            for (int v = 0; v < V; ++v) x[v] = 0.0f;
            if (from >= 0) load_row<V>(h + static_cast<size_t>(first + from) * a.width + c, x);
            else if (past) load_row<V>(slot + static_cast<size_t>(i + count) * a.width, x);
            store_row<V>(slot + static_cast<size_t>(i) * a.width, x);
        }
    }
}

template <typename T, int V>
static int launch_input_convolution(const ConvArgs& a, cudaStream_t stream) {
    const dim3 grid((a.tokens + a.run - 1) / a.run, (a.width + 256 * V - 1) / (256 * V));
    if (a.K == 1) return launch_kernel(input_convolution_kernel<T, V, 1>, grid, 256, 0, stream, a);
    if (a.K == 2) return launch_kernel(input_convolution_kernel<T, V, 2>, grid, 256, 0, stream, a);
    if (a.K == 3) return launch_kernel(input_convolution_kernel<T, V, 3>, grid, 256, 0, stream, a);
    if (a.K == 4) return launch_kernel(input_convolution_kernel<T, V, 4>, grid, 256, 0, stream, a);
    return launch_kernel(input_convolution_kernel<T, V, 0>, grid, 256, 0, stream, a);
}

ME_EXPORT int me_input_convolution(const void* h, int type, const float* taps, const int* entry_of_token, const int* cu_tokens,
                                   const int* state_slots, const int* fresh, float* state, void* out, int tokens, int width,
                                   int taps_count, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (taps_count < 1 || width < 1 || (taps_count > 1 && state == nullptr)) return ME_ERR_ARGUMENT;
    if (taps_count > MAX_TAPS) return ME_ERR_UNSUPPORTED;
    ConvArgs a{h, taps, entry_of_token, cu_tokens, state_slots, fresh, state, out, tokens, width, taps_count,
               tokens >= CONV_RUN_TOKENS ? CONV_RUN : 1};
    const bool vec = width % 4 == 0 && aligned16(h) && aligned16(taps) && aligned16(state) && aligned16(out);
    if (type == ME_BF16) return vec ? launch_input_convolution<__nv_bfloat16, 4>(a, stream) : launch_input_convolution<__nv_bfloat16, 1>(a, stream);
    return vec ? launch_input_convolution<float, 4>(a, stream) : launch_input_convolution<float, 1>(a, stream);
}
