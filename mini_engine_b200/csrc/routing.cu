// The router of a feed-forward made of many small units ("experts") of which a token uses a few.
//
// Per token: z = W_r h (+ a bias per unit) in float32 (h in the compute dtype, W_r float32).  Mode 0: s = sigmoid(z).  Mode
// 1: s = z itself and the chosen units' weights are the softmax over the chosen logits only.  Mode 2: s is the softmax of z
// over all units, the choice is made by s + correction (a learned number per unit), and the weights are the chosen s.
// The units form `group_count` equal groups of neighbours; a group's value is the sum of its two largest choice scores
// (of its only one when a group is a single unit), in mode 2 its largest, and only units of the `group_keep` best groups
// are eligible.  Among those the `top` largest choice scores are chosen; their weights are s / (sum of the chosen s +
// 1e-20) * weight_scale in mode 0, s * weight_scale in mode 2.  Ties go to the lower index.  The last units (`tensorless` of
// them) return their input: they count in everything above, their weights meet in identity_weight [T].  The kernel leaves a
// dense map `weights [T][units with tensors]` (zero for units that were not chosen), and the chosen units and their weights
// as lists `[T][top]`.  One more row of W_r (`shared_gate`) gives sigmoid(z) in shared_gate [T] and takes no part in the choice.
//
// A block takes TOKENS tokens (one, or four in a long step, which share what is read of the router): warp w forms the
// scores of units w, w + 8, ... for all of them; then warp i chooses for token i.  The sums run over the columns in a
// fixed order, so a token's choice never depends on the rest of the batch.
#include "common.cuh"

constexpr int ROUTE_WARPS = 8;
constexpr int MAX_UNITS = 1024;

struct RouteArgs {
    const void* h;        // [tokens][hidden]
    const float* router;  // [units (+ 1)][hidden]
    const float* bias;    // [units] added to the logits, or null
    int mode;             // 0: sigmoid scores over their sum; 1: the largest logits, softmax over the chosen ones; 2: softmax over all
    float* weights;       // [tokens][units - tensorless]
    int* chosen;          // [tokens][top]
    float* chosen_weight; // [tokens][top]
    int tokens, hidden, units, top, group_count, group_keep;
    float weight_scale;
    const float* correction;  // [units] or null
    int tensorless;
    float* identity_weight;  // [tokens] or null
    float* shared_gate;      // [tokens] or null
};

// The largest value of the warp and its index (the lowest among equals); index INT_MAX: there is none.
__device__ __forceinline__ void warp_argmax(float& value, int& index) {
#pragma unroll
    for (int offset = 16; offset > 0; offset >>= 1) {
        const float other = __shfl_xor_sync(0xffffffffu, value, offset);
        const int other_index = __shfl_xor_sync(0xffffffffu, index, offset);
        if (other > value || (other == value && other_index < index)) value = other, index = other_index;
    }
}

constexpr int MANY_TOKENS = 4, MANY_MAX_UNITS = 256;  // four tokens to a block, up to that many units
constexpr int MANY_FROM = 1024;                       // from this many tokens on

template <typename T, int TOKENS, int LIMIT>
__global__ void __launch_bounds__(ROUTE_WARPS * 32) route_kernel(RouteArgs a) {
    constexpr int NONE = 0x7fffffff;
    __shared__ float scores[TOKENS][LIMIT];   // what the weights are made of
    __shared__ float choices[TOKENS][LIMIT];  // what the choice is made by
    __shared__ float worths[TOKENS][LIMIT];   // of a group
    __shared__ unsigned char eligibles[TOKENS][LIMIT];
    const int first_token = blockIdx.x * TOKENS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    const T* rows_of_h[TOKENS];  // a block's last tokens may lie behind the step's: they repeat its last one and choose nothing
#pragma unroll
    for (int k = 0; k < TOKENS; ++k)
        rows_of_h[k] = static_cast<const T*>(a.h) + static_cast<size_t>(min(first_token + k, a.tokens - 1)) * a.hidden;
    const int rows = a.units + (a.shared_gate != nullptr ? 1 : 0), held = a.units - a.tensorless;
    // Lane l adds the products of columns 4 l .. 4 l + 3 (+ 128 j) in ascending order into four sums of its own, which
    // are then added in a fixed order: many loads in flight, and a token's scores are the same bits in every step.
    const bool quads = a.hidden % 4 == 0 && reinterpret_cast<uintptr_t>(a.router) % 16 == 0 && reinterpret_cast<uintptr_t>(a.h) % 8 == 0;
    for (int unit = warp; unit < rows; unit += ROUTE_WARPS) {
        const float* w = a.router + static_cast<size_t>(unit) * a.hidden;
        float sums[TOKENS];
        if (quads) {
            float part[TOKENS][4] = {};
#pragma unroll 4
            for (int i = lane * 4; i < a.hidden; i += 128) {
                const float4 weight = *reinterpret_cast<const float4*>(w + i);
#pragma unroll
                for (int k = 0; k < TOKENS; ++k) {
                    const T* h = rows_of_h[k] + i;
                    part[k][0] = fmaf(to_float(h[0]), weight.x, part[k][0]);
                    part[k][1] = fmaf(to_float(h[1]), weight.y, part[k][1]);
                    part[k][2] = fmaf(to_float(h[2]), weight.z, part[k][2]);
                    part[k][3] = fmaf(to_float(h[3]), weight.w, part[k][3]);
                }
            }
#pragma unroll
            for (int k = 0; k < TOKENS; ++k) sums[k] = (part[k][0] + part[k][1]) + (part[k][2] + part[k][3]);
        } else {
#pragma unroll
            for (int k = 0; k < TOKENS; ++k) {
                sums[k] = 0.0f;
                for (int i = lane; i < a.hidden; i += 32) sums[k] = fmaf(to_float(rows_of_h[k][i]), w[i], sums[k]);
            }
        }
#pragma unroll
        for (int k = 0; k < TOKENS; ++k) {
            float sum = warp_sum(sums[k]);
            if (unit == a.units) {  // the shared unit's gate
                if (lane == 0 && first_token + k < a.tokens) a.shared_gate[first_token + k] = 1.0f / (1.0f + expf(-sum));
                continue;
            }
            if (a.bias) sum += a.bias[unit];
            if (lane == 0) choices[k][unit] = scores[k][unit] = a.mode == 0 ? 1.0f / (1.0f + expf(-sum)) : sum;
        }
    }
    __syncthreads();
    const int token = first_token + warp;
    if (warp >= TOKENS || token >= a.tokens) return;
    float* score = scores[warp];
    float* choice = choices[warp];
    float* worth = worths[warp];
    unsigned char* eligible = eligibles[warp];
    for (int unit = lane; unit < a.units; unit += 32) {
        eligible[unit] = 0;
        if (unit < held) a.weights[static_cast<size_t>(token) * held + unit] = 0.0f;
    }
    __syncwarp();
    if (a.mode == 2) {
        float largest = -INFINITY, total = 0.0f;
        for (int u = lane; u < a.units; u += 32) largest = fmaxf(largest, score[u]);
        largest = warp_max(largest);
        for (int u = lane; u < a.units; u += 32) total += expf(score[u] - largest);
        total = warp_sum(total);
        for (int u = lane; u < a.units; u += 32) {
            score[u] = expf(score[u] - largest) / total;
            choice[u] = score[u] + (a.correction ? a.correction[u] : 0.0f);
        }
        __syncwarp();
    }
    const int per = a.units / a.group_count;
    for (int g = lane; g < a.group_count; g += 32) {
        float first = -INFINITY, second = -INFINITY;
        for (int u = g * per; u < (g + 1) * per; ++u) {
            const float s = choice[u];
            if (s > first) second = first, first = s;
            else if (s > second) second = s;
        }
        worth[g] = per > 1 && a.mode != 2 ? first + second : first;
    }
    __syncwarp();
    // The best groups, one at a time (group counts are small).
    for (int turn = 0; turn < a.group_keep; ++turn) {
        float value = -INFINITY;
        int best = NONE;
        for (int g = lane; g < a.group_count; g += 32)
            if (!eligible[g * per] && worth[g] > value) value = worth[g], best = g;
        warp_argmax(value, best);
        if (best == NONE) break;
        __syncwarp();
        for (int u = best * per + lane; u < (best + 1) * per; u += 32) eligible[u] = 1;
        __syncwarp();
    }
    int* chosen = a.chosen + static_cast<size_t>(token) * a.top;
    float* chosen_weight = a.chosen_weight + static_cast<size_t>(token) * a.top;
    float total = 0.0f, top_logit = 0.0f, denom = 0.0f;
    for (int turn = 0; turn < a.top; ++turn) {
        float value = -INFINITY;
        int best = NONE;
        for (int u = lane; u < a.units; u += 32)
            if (eligible[u] == 1 && choice[u] > value) value = choice[u], best = u;
        warp_argmax(value, best);
        if (lane == 0) chosen[turn] = best == NONE ? -1 : best;
        if (best == NONE) continue;
        if (turn == 0) top_logit = score[best];  // mode 1: the first choice holds the largest logit
        total += score[best];
        if (a.mode == 1) denom += expf(score[best] - top_logit);
        __syncwarp();
        if (lane == 0) eligible[best] = 2;
        __syncwarp();
    }
    if (lane != 0) return;
    const float inv = a.mode == 2 ? a.weight_scale : a.mode == 1 ? a.weight_scale / denom : a.weight_scale / (total + 1e-20f);
    float passed = 0.0f;
    for (int turn = 0; turn < a.top; ++turn) {
        const int u = chosen[turn];
        const float weight = u < 0 ? 0.0f : a.mode == 1 ? expf(score[u] - top_logit) * inv : score[u] * inv;
        chosen_weight[turn] = weight;
        if (u >= held) passed += weight;
        else if (u >= 0) a.weights[static_cast<size_t>(token) * held + u] = weight;
    }
    if (a.identity_weight != nullptr) a.identity_weight[token] = passed;
}

// `units` counts the tensorless units too; `shared_gate` says that the router has one more row.
ME_EXPORT int me_route(const void* h, int h_type, const float* router, const float* bias, int mode, float* weights,
                       int* chosen, float* chosen_weight, int tokens, int hidden, int units, int top, int group_count,
                       int group_keep, float weight_scale, const float* correction, int tensorless, float* identity_weight,
                       float* shared_gate, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (units < 1 || units > MAX_UNITS) return ME_ERR_UNSUPPORTED;
    if (group_count < 1 || units % group_count || group_keep < 1 || group_keep > group_count || top < 1 ||
        top > group_keep * (units / group_count))
        return ME_ERR_ARGUMENT;
    if (mode < 0 || mode > 2 || tensorless < 0 || tensorless >= units || (tensorless > 0 && identity_weight == nullptr)) return ME_ERR_ARGUMENT;
    if (correction != nullptr && mode != 2) return ME_ERR_ARGUMENT;
    RouteArgs a{h, router, bias, mode, weights, chosen, chosen_weight, tokens, hidden, units, top, group_count, group_keep, weight_scale,
                correction, tensorless, identity_weight, shared_gate};
    if (tokens >= MANY_FROM && units <= MANY_MAX_UNITS) {
        const int blocks = (tokens + MANY_TOKENS - 1) / MANY_TOKENS;
        if (h_type == ME_BF16) return launch_kernel(route_kernel<__nv_bfloat16, MANY_TOKENS, MANY_MAX_UNITS>, blocks, ROUTE_WARPS * 32, 0, stream, a);
        return launch_kernel(route_kernel<float, MANY_TOKENS, MANY_MAX_UNITS>, blocks, ROUTE_WARPS * 32, 0, stream, a);
    }
    if (h_type == ME_BF16) return launch_kernel(route_kernel<__nv_bfloat16, 1, MAX_UNITS>, tokens, ROUTE_WARPS * 32, 0, stream, a);
    return launch_kernel(route_kernel<float, 1, MAX_UNITS>, tokens, ROUTE_WARPS * 32, 0, stream, a);
}

// ------------------------------------------------------------- rows sorted by unit, for grouped products

// From the lists `chosen [T][top]` (choices outside [0, units) have no row): every (token, choice) gets a row in an array that is sorted by unit, each unit's
// run padded to a multiple of `pad` rows.  Leaves `row_of [T * top]` (the row of each choice), `token_of [capacity]`
// (the token of each row, -1 for padding and for the unused tail) and `unit_of_block [capacity / pad]` (the unit of
// every run of `pad` rows, -1 where no rows are).  One CTA; the order of a unit's rows among themselves is not
// fixed, and nothing depends on it: a row's products do not depend on its place.
constexpr int SORT_THREADS = 1024;

__global__ void __launch_bounds__(SORT_THREADS) sort_by_unit_kernel(const int* __restrict__ chosen, int items, int units, int pad,
                                                                    int capacity, int* __restrict__ row_of,
                                                                    int* __restrict__ token_of, int* __restrict__ unit_of_block,
                                                                    int top) {
    __shared__ int count[MAX_UNITS], first[MAX_UNITS];
    pdl_trigger();
    pdl_wait();
    for (int u = threadIdx.x; u < units; u += SORT_THREADS) count[u] = 0;
    for (int r = threadIdx.x; r < capacity; r += SORT_THREADS) token_of[r] = -1;
    for (int b = threadIdx.x; b < capacity / pad; b += SORT_THREADS) unit_of_block[b] = -1;
    __syncthreads();
    for (int i = threadIdx.x; i < items; i += SORT_THREADS) {
        const int u = chosen[i];
        if (u >= 0 && u < units) atomicAdd(&count[u], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int row = 0;
        for (int u = 0; u < units; ++u) {
            first[u] = row;
            const int blocks = (count[u] + pad - 1) / pad;
            for (int b = 0; b < blocks; ++b) unit_of_block[row / pad + b] = u;
            row += blocks * pad;
            count[u] = 0;  // becomes the cursor of the unit's run
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < items; i += SORT_THREADS) {
        const int u = chosen[i];
        if (u < 0 || u >= units) { row_of[i] = -1; continue; }
        const int row = first[u] + atomicAdd(&count[u], 1);
        row_of[i] = row;
        token_of[row] = i / top;
    }
}

// sorted[row] = h[token_of[row]] (zeros for rows without a token), 16 bytes per thread and step.
__global__ void gather_rows_kernel(const uint4* __restrict__ h, const int* __restrict__ token_of, uint4* __restrict__ sorted,
                                   int rows, int chunks) {
    pdl_trigger();
    pdl_wait();
    const size_t total = static_cast<size_t>(rows) * chunks;
    for (size_t idx = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; idx < total;
         idx += static_cast<size_t>(gridDim.x) * blockDim.x) {
        const int row = static_cast<int>(idx / chunks), chunk = static_cast<int>(idx % chunks);
        const int token = token_of[row];
        sorted[idx] = token >= 0 ? h[static_cast<size_t>(token) * chunks + chunk] : make_uint4(0u, 0u, 0u, 0u);
    }
}

// out[t] = sum over the token's choices, in their order, of weight[t][k] * sorted_out[row_of[t][k]], float32.
__global__ void combine_rows_kernel(const float* __restrict__ sorted_out, const int* __restrict__ row_of,
                                    const float* __restrict__ weight, float* __restrict__ out, int tokens, int top, int width) {
    pdl_trigger();
    pdl_wait();
    const size_t total = static_cast<size_t>(tokens) * width;
    for (size_t idx = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; idx < total;
         idx += static_cast<size_t>(gridDim.x) * blockDim.x) {
        const int t = static_cast<int>(idx / width), c = static_cast<int>(idx % width);
        float sum = 0.0f;
        for (int k = 0; k < top; ++k) {
            const int row = row_of[t * top + k];
            if (row >= 0) sum = fmaf(weight[t * top + k], sorted_out[static_cast<size_t>(row) * width + c], sum);
        }
        out[idx] = sum;
    }
}

ME_EXPORT int me_sort_by_unit(const int* chosen, int tokens, int top, int units, int pad, int capacity, int* row_of,
                              int* token_of, int* unit_of_block, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (units < 1 || units > MAX_UNITS || pad < 1 || capacity % pad) return ME_ERR_ARGUMENT;
    // every unit's run may end in a partly filled block
    if (static_cast<long long>(capacity) < static_cast<long long>(tokens) * top + static_cast<long long>(units) * (pad - 1))
        return ME_ERR_ARGUMENT;
    return launch_kernel(sort_by_unit_kernel, 1, SORT_THREADS, 0, stream, chosen, tokens * top, units, pad, capacity, row_of,
                         token_of, unit_of_block, top);
}

ME_EXPORT int me_gather_rows(const void* h, const int* token_of, void* sorted, int rows, int row_bytes, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (row_bytes % 16 || reinterpret_cast<uintptr_t>(h) % 16 || reinterpret_cast<uintptr_t>(sorted) % 16) return ME_ERR_ARGUMENT;
    const int chunks = row_bytes / 16;
    const size_t total = static_cast<size_t>(rows) * chunks;
    const int blocks = static_cast<int>((total + 255) / 256 < 148 * 32 ? (total + 255) / 256 : 148 * 32);
    return launch_kernel(gather_rows_kernel, blocks, 256, 0, stream, static_cast<const uint4*>(h), token_of,
                         static_cast<uint4*>(sorted), rows, chunks);
}

ME_EXPORT int me_combine_rows(const float* sorted_out, const int* row_of, const float* weight, float* out, int tokens, int top,
                              int width, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    const size_t total = static_cast<size_t>(tokens) * width;
    const int blocks = static_cast<int>((total + 255) / 256 < 148 * 32 ? (total + 255) / 256 : 148 * 32);
    return launch_kernel(combine_rows_kernel, blocks, 256, 0, stream, sorted_out, row_of, weight, out, tokens, top, width);
}

// ---------------------------------------------------------- the outputs of a token's units, joined

// out[t] = routed + identity_weight[t] * h[t] + shared_gate[t] * sum_s shared[s][t], float32.  `routed` is the sum of the
// partial sums routed[s][t], or (with row_of) sum_k weight[t][k] * sorted[row_of[t][k]] in the order of the choices.  The
// second and third term may be absent; a shared output without a gate has weight one.  V columns per thread.
struct FinishArgs {
    const float* routed;  // [routed_splits][tokens][width], or the sorted rows
    int routed_splits;
    size_t routed_stride;
    const int* row_of;    // [tokens][top] or null
    const float* weight;  // [tokens][top]
    int top;
    const void* h;  // [tokens][width]
    const float* identity_weight;
    const float* shared;  // [shared_splits][tokens][width] or null
    int shared_splits;
    size_t shared_stride;
    const float* shared_gate;
    float* out;
    int tokens, width;
};

template <int V>
struct Columns {
    float v[V];
    __device__ __forceinline__ void load(const float* src) {
        if constexpr (V == 4) {
            const float4 q = *reinterpret_cast<const float4*>(src);
            v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
        } else {
            v[0] = src[0];
        }
    }
    __device__ __forceinline__ void add(const Columns& other, float factor = 1.0f) {
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = fmaf(factor, other.v[i], v[i]);
    }
};

template <typename T, int V>
__global__ void __launch_bounds__(256) moe_finish_kernel(FinishArgs a) {
    pdl_trigger();
    pdl_wait();
    const size_t per = a.width / V, total = static_cast<size_t>(a.tokens) * per;
    for (size_t idx = blockIdx.x * static_cast<size_t>(256) + threadIdx.x; idx < total; idx += static_cast<size_t>(gridDim.x) * 256) {
        const size_t t = idx / per, at = idx * V, c = at - t * a.width;
        Columns<V> sum = {}, part;
        if (a.row_of) {
            for (int k = 0; k < a.top; ++k) {
                const int row = a.row_of[t * a.top + k];
                if (row < 0) continue;
                part.load(a.routed + static_cast<size_t>(row) * a.width + c);
                sum.add(part, a.weight[t * a.top + k]);
            }
        } else {
            for (int s = 0; s < a.routed_splits; ++s) {
                part.load(a.routed + s * a.routed_stride + at);
                sum.add(part);
            }
        }
        if (a.identity_weight) {
            const float weight = a.identity_weight[t];
            if (weight != 0.0f) {
#pragma unroll
                for (int i = 0; i < V; ++i) sum.v[i] = fmaf(weight, to_float(static_cast<const T*>(a.h)[at + i]), sum.v[i]);
            }
        }
        if (a.shared) {
            Columns<V> whole = {};
            for (int s = 0; s < a.shared_splits; ++s) {
                part.load(a.shared + s * a.shared_stride + at);
                whole.add(part);
            }
            sum.add(whole, a.shared_gate ? a.shared_gate[t] : 1.0f);
        }
        if constexpr (V == 4) *reinterpret_cast<float4*>(a.out + at) = make_float4(sum.v[0], sum.v[1], sum.v[2], sum.v[3]);
        else a.out[at] = sum.v[0];
    }
}

ME_EXPORT int me_moe_finish(const float* routed, int routed_splits, long long routed_stride, const int* row_of, const float* weight,
                            int top, const void* h, int h_type, const float* identity_weight, const float* shared, int shared_splits,
                            long long shared_stride, const float* shared_gate, float* out, int tokens, int width, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (routed == nullptr || out == nullptr || (row_of != nullptr && (weight == nullptr || top < 1))) return ME_ERR_ARGUMENT;
    FinishArgs a{routed, routed_splits, (size_t)routed_stride, row_of, weight, top, h, identity_weight, shared, shared_splits,
                 (size_t)shared_stride, shared_gate, out, tokens, width};
    const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool vec = width % 4 == 0 && routed_stride % 4 == 0 && shared_stride % 4 == 0 && aligned(routed) && aligned(shared) && aligned(out);
    const size_t total = static_cast<size_t>(tokens) * width / (vec ? 4 : 1);
    const int blocks = static_cast<int>((total + 255) / 256 < 148 * 32 ? (total + 255) / 256 : 148 * 32);
    if (h_type == ME_BF16)
        return vec ? launch_kernel(moe_finish_kernel<__nv_bfloat16, 4>, blocks, 256, 0, stream, a)
                   : launch_kernel(moe_finish_kernel<__nv_bfloat16, 1>, blocks, 256, 0, stream, a);
    return vec ? launch_kernel(moe_finish_kernel<float, 4>, blocks, 256, 0, stream, a)
               : launch_kernel(moe_finish_kernel<float, 1>, blocks, 256, 0, stream, a);
}
