// Matrix-state recurrences over long portions in chunks of 16 tokens: the generalized delta rule and the recurrence with a bonus
// of delta_rule.cu, on the same prepared rows.  With S the state in front of a chunk, and per token the key k, the decay g, the
// removal vector b (a times k; it removes b c (k^T S) with the number c = 1 / (k . k + eps)) and the query q,
//
//   y_t = c_t k_t^T S_(t-1),   S_t = diag(g_t) S_(t-1) - b_t y_t^T + k_t v_t^T,   o_t = q_t^T S_t
//
// (with a bonus there is no y, and o_t = q_t^T S_(t-1) + (sum q u k) v_t).  Inside a chunk everything but the products with S and
// v is known before S is.  With the decays multiplied up between two tokens, D(j, t) = g_(j+1) ... g_t, channel by channel, and
// r_t = q_t g_t (the bonus: q_t):
//
//   A_t = c_t k_t D(0, t-1)          R_t = r_t D(0, t-1)          what a token reads of the chunk's first state
//   AB[t][j] = c_t k_t . (D(j, t-1) b_j),   AK likewise with k_j,   RB[t][j] = r_t . (D(j, t-1) b_j),   RK likewise   (j < t)
//
// the reads are the solution of a triangular system, Y = A S + AK V - AB Y, and the outputs O = R S + RK V - RB Y (the diagonals of
// RB and RK are q . b and q . k, or the bonus).  Solved for S and V, Y = A' S + M1 V and O = R' S + M2 V, where A', R', M1, M2 come
// from a forward substitution per column.  The state behind the chunk is
//
//   diag(D(0, 16)) S + sum_t (D(t, 16) k_t) v_t^T - (D(t, 16) b_t) y_t^T.
//
// Decays are only ever multiplied up (never divided by one another), so that none over- or underflows into a wrong value.
//
// `chunk_record_kernel` makes A', R', M1, M2 and the decayed k and b of every chunk of every long entry, all side by side;
// `chunk_walk_kernel` walks an entry's chunks with the state in shared memory, two small products per chunk.  All of it is float32 on
// the CUDA cores.  A token's sums are ordered by its place in its portion's chunks: its bits depend on how its request was
// cut into steps, by rounding only.
#include "common.cuh"

#include <algorithm>

enum : int { RULE_REMOVAL = 1, RULE_BONUS = 2 };

constexpr int CHUNK = 16;
constexpr int COLUMNS = 32;  // value columns of a walking block
constexpr int THREADS = 128;       // of a recording block
constexpr int WALK_THREADS = 256;  // of a walking block
constexpr int WALK_WARPS = WALK_THREADS / 32;
constexpr int STAGES = 3;  // records that a walking block holds: two are on their way

template <int RULE>
struct Rule;
// VECTORS and SCALARS: what a prepared row holds (see delta_rule.cu); ROWS: rows of the two products of a chunk.
template <>
struct Rule<RULE_REMOVAL> { static constexpr int VECTORS = 4, SCALARS = 4, ROWS = 2 * CHUNK; };
template <>
struct Rule<RULE_BONUS> { static constexpr int VECTORS = 3, SCALARS = 2, ROWS = CHUNK; };

// A chunk's record: the reading matrix transposed, [DIM + CHUNK][ROWS] (the key channels of (A' | R'), then the tokens of (M1 |
// M2)), the writing matrix [ROWS][DIM] (decayed k, then decayed b) and the decay over the chunk [DIM].
template <int RULE, int DIM>
struct Record { static constexpr int FLOATS = (DIM + CHUNK) * Rule<RULE>::ROWS + Rule<RULE>::ROWS * DIM + DIM; };

struct ChunkArgs {
    const float* rows;     // [tokens][heads][VECTORS * dim + vdim]
    const float* scalars;  // [tokens][heads][SCALARS]
    const int* cu_tokens;
    const int* state_slots;
    const int* fresh;
    float* state;  // [slots + 1][slot_floats], a slot starts with [heads][vdim][dim]
    size_t slot_floats;
    float* out;      // [tokens][heads][vdim]
    float* records;  // [heads][max_chunks][record floats]: a walking block reads its records one after the other
    int entries, heads, dim, vdim, min_count, max_chunks;
};

// The entry that chunk number `chunk` belongs to (entries of at least min_count tokens, cut in order).
__device__ __forceinline__ bool locate_chunk(const ChunkArgs& a, int chunk, int& first_token, int& count) {
    int seen = 0;
    for (int b = 0; b < a.entries; ++b) {
        const int begin = a.cu_tokens[b], n = a.cu_tokens[b + 1] - begin;
        if (n < a.min_count) continue;
        const int chunks = (n + CHUNK - 1) / CHUNK;
        if (chunk < seen + chunks) {
            first_token = begin + (chunk - seen) * CHUNK;
            count = min(CHUNK, n - (chunk - seen) * CHUNK);
            return true;
        }
        seen += chunks;
    }
    return false;
}

template <int RULE, int DIM>
__global__ void __launch_bounds__(THREADS) chunk_record_kernel(ChunkArgs a) {
    constexpr int VECTORS = Rule<RULE>::VECTORS, SCALARS = Rule<RULE>::SCALARS, ROWS = Rule<RULE>::ROWS;
    constexpr bool REMOVES = RULE == RULE_REMOVAL;
    extern __shared__ __align__(16) float chunk_smem[];
    float* vectors = chunk_smem;                        // [VECTORS][CHUNK][DIM]: r, k, g (and b)
    float* pairs = vectors + VECTORS * CHUNK * DIM;     // [AK, RK (, AB, RB)][t][j]
    __shared__ float unit[CHUNK];                       // c
    const int head = blockIdx.y;
    pdl_trigger();
    pdl_wait();
    int first, count;
    if (!locate_chunk(a, blockIdx.x, first, count)) return;
    const int row_floats = VECTORS * a.dim + a.vdim;
    const float* rows = a.rows + (static_cast<size_t>(first) * a.heads + head) * row_floats;
    const float* scalars = a.scalars + (static_cast<size_t>(first) * a.heads + head) * SCALARS;
    const size_t row_step = static_cast<size_t>(a.heads) * row_floats;
    // Tokens behind the portion's end: no key, nothing removed, no decay.
    for (int i = threadIdx.x; i < CHUNK * VECTORS * (DIM / 4); i += THREADS) {
        const int t = i / (VECTORS * (DIM / 4)), which = i / (DIM / 4) % VECTORS, d = i % (DIM / 4) * 4;
        const float blank = which == 2 ? 1.0f : 0.0f;
        float4 x = make_float4(blank, blank, blank, blank);
        if (t < count && d < a.dim) x = *reinterpret_cast<const float4*>(rows + t * row_step + which * a.dim + d);
        *reinterpret_cast<float4*>(vectors + (which * CHUNK + t) * DIM + d) = x;
    }
    for (int i = threadIdx.x; i < (REMOVES ? 4 : 2) * CHUNK * CHUNK; i += THREADS) pairs[i] = 0.0f;
    __syncthreads();
    const float *r = vectors, *k = vectors + CHUNK * DIM, *g = vectors + 2 * CHUNK * DIM, *b = vectors + 3 * CHUNK * DIM;
    float *ak = pairs, *rk = pairs + CHUNK * CHUNK, *ab = pairs + 2 * CHUNK * CHUNK, *rb = pairs + 3 * CHUNK * CHUNK;
    if (threadIdx.x < CHUNK) {
        const int t = threadIdx.x;
        const float* mine = scalars + t * static_cast<size_t>(a.heads) * SCALARS;
        const bool live = t < count;
        if (REMOVES) {
            const float c = live ? mine[0] : 0.0f;
            unit[t] = c;
            rk[t * CHUNK + t] = live ? mine[2] : 0.0f;           // q . k
            rb[t * CHUNK + t] = live ? mine[1] / c : 0.0f;       // q . b
        } else {
            rk[t * CHUNK + t] = live ? mine[0] : 0.0f;
        }
    }
    __syncthreads();
    // Pairs of tokens: four lanes walk token j's key (the upper half of the block: its removal vector) through the later tokens.
    {
        constexpr int QUADS = DIM / 16;  // float4 pieces of a lane
        const int j = (threadIdx.x % 64) / 4, part = threadIdx.x % 4;
        const bool removal = threadIdx.x >= 64;
        if (REMOVES || !removal) {
            float4 p[QUADS];
#pragma unroll
            for (int i = 0; i < QUADS; ++i) p[i] = *reinterpret_cast<const float4*>((removal ? b : k) + j * DIM + i * 16 + part * 4);
#pragma unroll 1
            for (int t = 1; t < CHUNK; ++t) {
                float on_k = 0.0f, on_r = 0.0f;
#pragma unroll
                for (int i = 0; i < QUADS; ++i) {
                    const int at = t * DIM + i * 16 + part * 4;
                    const float4 r4 = *reinterpret_cast<const float4*>(r + at), g4 = *reinterpret_cast<const float4*>(g + at);
                    if (REMOVES) {
                        const float4 k4 = *reinterpret_cast<const float4*>(k + at);
                        on_k = fmaf(p[i].x, k4.x, fmaf(p[i].y, k4.y, fmaf(p[i].z, k4.z, fmaf(p[i].w, k4.w, on_k))));
                    }
                    on_r = fmaf(p[i].x, r4.x, fmaf(p[i].y, r4.y, fmaf(p[i].z, r4.z, fmaf(p[i].w, r4.w, on_r))));
                    if (t > j) p[i].x *= g4.x, p[i].y *= g4.y, p[i].z *= g4.z, p[i].w *= g4.w;
                }
#pragma unroll
                for (int offset = 1; offset < 4; offset <<= 1) {
                    if (REMOVES) on_k += __shfl_xor_sync(0xffffffffu, on_k, offset);
                    on_r += __shfl_xor_sync(0xffffffffu, on_r, offset);
                }
                if (t > j && part == 0) {
                    (removal ? rb : rk)[t * CHUNK + j] = on_r;
                    if (REMOVES) (removal ? ab : ak)[t * CHUNK + j] = unit[t] * on_k;
                }
            }
        }
    }
    __syncthreads();
    float* record = a.records + (static_cast<size_t>(head) * a.max_chunks + blockIdx.x) * Record<RULE, DIM>::FLOATS;
    float* writing = record + (DIM + CHUNK) * ROWS;
    // One column per thread: a key channel of A and R, or a token of AK and RK.
    for (int column = threadIdx.x; column < DIM + CHUNK; column += THREADS) {
        const bool channel = column < DIM;
        const int token = column - DIM;
        float x[CHUNK], y[CHUNK];
        float decay = 1.0f;
#pragma unroll
        for (int t = 0; t < CHUNK; ++t) {
            if (channel) {
                if (REMOVES) x[t] = unit[t] * k[t * DIM + column] * decay;
                y[t] = r[t * DIM + column] * decay;
                decay *= g[t * DIM + column];
            } else {
                if (REMOVES) x[t] = ak[t * CHUNK + token];
                y[t] = rk[t * CHUNK + token];
            }
        }
        if constexpr (REMOVES) {
#pragma unroll
            for (int t = 0; t < CHUNK; ++t) {
#pragma unroll
                for (int j = 0; j < CHUNK; j += 4) {
                    if (j > t) break;
                    const float4 ab4 = *reinterpret_cast<const float4*>(ab + t * CHUNK + j), rb4 = *reinterpret_cast<const float4*>(rb + t * CHUNK + j);
                    const float from_ab[4] = {ab4.x, ab4.y, ab4.z, ab4.w}, from_rb[4] = {rb4.x, rb4.y, rb4.z, rb4.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        if (j + i < t) x[t] = fmaf(-from_ab[i], x[j + i], x[t]), y[t] = fmaf(-from_rb[i], x[j + i], y[t]);
                }
                y[t] = fmaf(-rb[t * CHUNK + t], x[t], y[t]);
            }
        }
        float* dst = record + column * ROWS;
#pragma unroll
        for (int t = 0; t < CHUNK; t += 4) {
            if constexpr (REMOVES) *reinterpret_cast<float4*>(dst + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
            *reinterpret_cast<float4*>(dst + ROWS - CHUNK + t) = make_float4(y[t], y[t + 1], y[t + 2], y[t + 3]);
        }
        if (!channel) continue;
        decay = 1.0f;
#pragma unroll
        for (int t = CHUNK - 1; t >= 0; --t) {
            writing[t * DIM + column] = k[t * DIM + column] * decay;
            if constexpr (REMOVES) writing[(CHUNK + t) * DIM + column] = b[t * DIM + column] * decay;
            decay *= g[t * DIM + column];
        }
        writing[ROWS * DIM + column] = decay;
    }
}

__device__ __forceinline__ void copy_async_16(float* shared_dst, const float* global_src) {
    const uint32_t dst = static_cast<uint32_t>(__cvta_generic_to_shared(shared_dst));
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(global_src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory"); }

// One block of eight warps per (entry, head, 32 value columns).  A thread of the first four warps owns a tile of 4 channels x 4
// columns of the state (two of them at 128 channels) in registers, and shares it with the block through shared memory.  What
// the two products of a chunk read from shared memory is what they cost, so that a thread takes tiles as large as its registers
// hold and the warps share the terms and not the outputs: in the reading product every warp adds up an eighth of the terms for all
// outputs, ROWS / 4 rows x 4 columns to a lane; of what is written the other four warps add up half.
template <int RULE, int DIM>
__global__ void __launch_bounds__(WALK_THREADS) chunk_walk_kernel(ChunkArgs a) {
    constexpr int VECTORS = Rule<RULE>::VECTORS, ROWS = Rule<RULE>::ROWS, RECORD = Record<RULE, DIM>::FLOATS;
    constexpr bool REMOVES = RULE == RULE_REMOVAL;
    constexpr int STAGE = RECORD + CHUNK * COLUMNS;
    constexpr int TILES = DIM > 64 ? DIM / 64 : 1;
    constexpr int TALL = ROWS / 4;  // rows of a lane's part of the reading product
    extern __shared__ __align__(16) float chunk_smem[];
    float* stages = chunk_smem;                  // [STAGES]: record, values [CHUNK][COLUMNS]
    float* held = chunk_smem + STAGES * STAGE;   // the state [DIM][COLUMNS]
    float* minus_y = held + DIM * COLUMNS;       // [CHUNK][COLUMNS]
    float* partial = minus_y + CHUNK * COLUMNS;  // [warps][ROWS][COLUMNS]
    float* added = partial + WALK_WARPS * ROWS * COLUMNS;  // [DIM][COLUMNS]: the other warps' half of what is written
    const int entry = blockIdx.x, head = blockIdx.y, first_column = blockIdx.z * COLUMNS;
    pdl_trigger();
    pdl_wait();
    const int begin = a.cu_tokens[entry], count = a.cu_tokens[entry + 1] - begin;
    if (count < a.min_count) return;
    int first_chunk = 0;
    for (int e = 0; e < entry; ++e) {
        const int n = a.cu_tokens[e + 1] - a.cu_tokens[e];
        if (n >= a.min_count) first_chunk += (n + CHUNK - 1) / CHUNK;
    }
    const int chunks = (count + CHUNK - 1) / CHUNK;
    const int row_floats = VECTORS * a.dim + a.vdim;
    const float* values = a.rows + (static_cast<size_t>(begin) * a.heads + head) * row_floats + VECTORS * a.dim + first_column;
    const size_t row_step = static_cast<size_t>(a.heads) * row_floats;
    const float* records = a.records + (static_cast<size_t>(head) * a.max_chunks + first_chunk) * RECORD;
    auto fetch = [&](int chunk, float* stage) {
        const float* record = records + static_cast<size_t>(chunk) * RECORD;
        for (int i = threadIdx.x; i < RECORD / 4; i += WALK_THREADS) copy_async_16(stage + 4 * i, record + 4 * i);
        for (int i = threadIdx.x; i < CHUNK * COLUMNS / 4; i += WALK_THREADS) {
            const int t = chunk * CHUNK + i / (COLUMNS / 4), column = i % (COLUMNS / 4) * 4;
            float* dst = stage + RECORD + 4 * i;
            if (t < count && first_column + column < a.vdim) copy_async_16(dst, values + t * row_step + column);
            else *reinterpret_cast<float4*>(dst) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    };
#pragma unroll
    for (int i = 0; i < STAGES - 1; ++i) {  // a group per chunk, empty behind the last one
        if (i < chunks) fetch(i, stages + i * STAGE);
        copy_async_commit();
    }

    // The state's tile: channels [4 quad, +4), columns [4 strip, +4).
    const int strip = threadIdx.x % 8, quad = threadIdx.x % 128 / 8;
    const bool owner = threadIdx.x < 128;
    float4 s[TILES][4];  // [channel] of four columns
    float* state = a.state + static_cast<size_t>(a.state_slots[entry]) * a.slot_floats + (static_cast<size_t>(head) * a.vdim + first_column + 4 * strip) * a.dim;
    auto columns_of = [](float4& row, int c) -> float& { return c == 0 ? row.x : c == 1 ? row.y : c == 2 ? row.z : row.w; };
#pragma unroll
    for (int tile = 0; tile < TILES; ++tile) {
        const int d = 4 * (quad + 16 * tile);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (d < a.dim && first_column + 4 * strip + c < a.vdim && a.fresh[entry] == 0) x = *reinterpret_cast<const float4*>(state + static_cast<size_t>(c) * a.dim + d);
            columns_of(s[tile][0], c) = x.x, columns_of(s[tile][1], c) = x.y, columns_of(s[tile][2], c) = x.z, columns_of(s[tile][3], c) = x.w;
        }
        if (owner && d < DIM) {
#pragma unroll
            for (int i = 0; i < 4; ++i) *reinterpret_cast<float4*>(held + (d + i) * COLUMNS + 4 * strip) = s[tile][i];
        }
    }

    const int warp = threadIdx.x / 32, group = threadIdx.x % 32 / 8;  // rows [TALL group, +TALL) of the reading product, columns as above
    for (int chunk = 0; chunk < chunks; ++chunk) {
        float* stage = stages + chunk % STAGES * STAGE;
        copy_async_wait();
        __syncthreads();  // the record has landed, the state is in shared memory and nobody reads the oldest stage any more
        if (chunk + STAGES - 1 < chunks) fetch(chunk + STAGES - 1, stages + (chunk + STAGES - 1) % STAGES * STAGE);
        copy_async_commit();
        const float* v = stage + RECORD;
        float2 low[TALL], high[TALL];
#pragma unroll
        for (int i = 0; i < TALL; ++i) low[i] = high[i] = make_float2(0.0f, 0.0f);
        // A warp's share of the terms: channels of the state, then tokens' values.
        constexpr int TERMS = (DIM + CHUNK) / WALK_WARPS;
#pragma unroll (TERMS % 5 == 0 ? 5 : 6)
        for (int n = 0; n < TERMS; ++n) {
            const int term = warp * TERMS + n;
            const float* reading = stage + term * ROWS + TALL * group;
            const float4 x = *reinterpret_cast<const float4*>((term < DIM ? held + term * COLUMNS : v + (term - DIM) * COLUMNS) + 4 * strip);
            const float2 left = make_float2(x.x, x.y), right = make_float2(x.z, x.w);
#pragma unroll
            for (int q = 0; q < TALL; q += 4) {
                const float4 w = *reinterpret_cast<const float4*>(reading + q);
                low[q] = __ffma2_rn(make_float2(w.x, w.x), left, low[q]), high[q] = __ffma2_rn(make_float2(w.x, w.x), right, high[q]);
                low[q + 1] = __ffma2_rn(make_float2(w.y, w.y), left, low[q + 1]), high[q + 1] = __ffma2_rn(make_float2(w.y, w.y), right, high[q + 1]);
                low[q + 2] = __ffma2_rn(make_float2(w.z, w.z), left, low[q + 2]), high[q + 2] = __ffma2_rn(make_float2(w.z, w.z), right, high[q + 2]);
                low[q + 3] = __ffma2_rn(make_float2(w.w, w.w), left, low[q + 3]), high[q + 3] = __ffma2_rn(make_float2(w.w, w.w), right, high[q + 3]);
            }
        }
#pragma unroll
        for (int i = 0; i < TALL; ++i)
            *reinterpret_cast<float4*>(partial + (warp * ROWS + TALL * group + i) * COLUMNS + 4 * strip) = make_float4(low[i].x, low[i].y, high[i].x, high[i].y);
        __syncthreads();  // every warp's sums are there, and nobody reads the state any more
        if (threadIdx.x / 8 < ROWS) {
            const int row = threadIdx.x / 8, t = row - (ROWS - CHUNK);
            float4 z = *reinterpret_cast<const float4*>(partial + row * COLUMNS + 4 * strip);
#pragma unroll
            for (int part = 1; part < WALK_WARPS; ++part) {
                const float4 x = *reinterpret_cast<const float4*>(partial + (part * ROWS + row) * COLUMNS + 4 * strip);
                z.x += x.x, z.y += x.y, z.z += x.z, z.w += x.w;
            }
            if (REMOVES && row < CHUNK) {
                *reinterpret_cast<float4*>(minus_y + row * COLUMNS + 4 * strip) = make_float4(-z.x, -z.y, -z.z, -z.w);
            } else if (chunk * CHUNK + t < count && first_column + 4 * strip < a.vdim) {
                float* out = a.out + (static_cast<size_t>(begin + chunk * CHUNK + t) * a.heads + head) * a.vdim + first_column + 4 * strip;
                *reinterpret_cast<float4*>(out) = z;
            }
        }
        if (REMOVES) __syncthreads();  // the reads y are there
        const float* writing = stage + (DIM + CHUNK) * ROWS;
        // The owners add the first half of the written terms to their decayed tiles, the others add up the second half: the removals,
        // or the last tokens' keys and values.
        float2 first[TILES][4], second[TILES][4];
#pragma unroll
        for (int tile = 0; tile < TILES; ++tile) {
            const int d = min(4 * (quad + 16 * tile), DIM - 4);
            const float4 g = *reinterpret_cast<const float4*>(writing + ROWS * DIM + d);
            const float decay[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                first[tile][i] = owner ? make_float2(s[tile][i].x * decay[i], s[tile][i].y * decay[i]) : make_float2(0.0f, 0.0f);
                second[tile][i] = owner ? make_float2(s[tile][i].z * decay[i], s[tile][i].w * decay[i]) : make_float2(0.0f, 0.0f);
            }
            const float* written = writing + (owner ? 0 : ROWS / 2 * DIM) + d;
            const float* operand = (owner ? v : REMOVES ? minus_y : v + ROWS / 2 * COLUMNS) + 4 * strip;
#pragma unroll 8
            for (int n = 0; n < ROWS / 2; ++n) {
                const float4 w = *reinterpret_cast<const float4*>(written + n * DIM), x = *reinterpret_cast<const float4*>(operand + n * COLUMNS);
                const float weights[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    first[tile][i] = __ffma2_rn(make_float2(weights[i], weights[i]), make_float2(x.x, x.y), first[tile][i]);
                    second[tile][i] = __ffma2_rn(make_float2(weights[i], weights[i]), make_float2(x.z, x.w), second[tile][i]);
                }
            }
            if (!owner && 4 * (quad + 16 * tile) < DIM) {
#pragma unroll
                for (int i = 0; i < 4; ++i)
                    *reinterpret_cast<float4*>(added + (d + i) * COLUMNS + 4 * strip) = make_float4(first[tile][i].x, first[tile][i].y, second[tile][i].x, second[tile][i].y);
            }
        }
        __syncthreads();  // the second half is there
#pragma unroll
        for (int tile = 0; tile < TILES && owner; ++tile) {
            const int d = 4 * (quad + 16 * tile);
            if (d >= DIM) continue;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float4 x = *reinterpret_cast<const float4*>(added + (d + i) * COLUMNS + 4 * strip);
                s[tile][i] = make_float4(first[tile][i].x + x.x, first[tile][i].y + x.y, second[tile][i].x + x.z, second[tile][i].y + x.w);
                *reinterpret_cast<float4*>(held + (d + i) * COLUMNS + 4 * strip) = s[tile][i];
            }
        }
    }
#pragma unroll
    for (int tile = 0; tile < TILES; ++tile) {
        const int d = 4 * (quad + 16 * tile);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            if (owner && d < a.dim && first_column + 4 * strip + c < a.vdim)
                *reinterpret_cast<float4*>(state + static_cast<size_t>(c) * a.dim + d) =
                    make_float4(columns_of(s[tile][0], c), columns_of(s[tile][1], c), columns_of(s[tile][2], c), columns_of(s[tile][3], c));
        }
    }
}

// -------------------------------------------------------------------------------------- host

static int padded_dim(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : 128; }

// Key heads of up to 128 channels; both widths multiples of four.
ME_EXPORT int me_state_chunks_supports(int dim, int vdim) { return dim >= 4 && dim <= 128 && dim % 4 == 0 && vdim >= 4 && vdim % 4 == 0; }

ME_EXPORT int me_state_chunks_record_floats(int rule, int dim) {
    const int d = padded_dim(dim), rows = rule == RULE_REMOVAL ? 2 * CHUNK : CHUNK;
    return (d + CHUNK) * rows + rows * d + d;
}

template <int RULE, int DIM>
static int launch_chunks(const ChunkArgs& a, int max_chunks, cudaStream_t stream) {
    static SharedMemoryOptIn record_opt_in, walk_opt_in;
    constexpr int RECORD_SMEM = (Rule<RULE>::VECTORS * CHUNK * DIM + 4 * CHUNK * CHUNK) * sizeof(float);
    constexpr int WALK_SMEM = (STAGES * (Record<RULE, DIM>::FLOATS + CHUNK * COLUMNS) + 2 * DIM * COLUMNS + (CHUNK + WALK_WARPS * Rule<RULE>::ROWS) * COLUMNS) * sizeof(float);
    if (RECORD_SMEM > 48 * 1024)
        if (const int e = record_opt_in(chunk_record_kernel<RULE, DIM>, RECORD_SMEM)) return e;
    if (WALK_SMEM > 48 * 1024)
        if (const int e = walk_opt_in(chunk_walk_kernel<RULE, DIM>, WALK_SMEM)) return e;
    const int code = launch_kernel_in_order(chunk_record_kernel<RULE, DIM>, dim3(max_chunks, a.heads), THREADS, RECORD_SMEM, stream, a);
    if (code) return code;
    return launch_kernel_in_order(chunk_walk_kernel<RULE, DIM>, dim3(a.entries, a.heads, (a.vdim + COLUMNS - 1) / COLUMNS), WALK_THREADS, WALK_SMEM, stream, a);
}

template <int RULE>
static int dispatch_chunks(const ChunkArgs& a, int max_chunks, cudaStream_t stream) {
    const int d = padded_dim(a.dim);
    return d == 32 ? launch_chunks<RULE, 32>(a, max_chunks, stream) : d == 64 ? launch_chunks<RULE, 64>(a, max_chunks, stream) : launch_chunks<RULE, 128>(a, max_chunks, stream);
}

// The entries of at least `min_count` tokens, which have `max_chunks` chunks of 16 tokens or fewer between them.  `records` is
// scratch of max_chunks * heads * me_state_chunks_record_floats floats.
ME_EXPORT int me_state_chunks(const float* rows, const float* scalars, const int* cu_tokens, const int* state_slots, const int* fresh,
                              float* state, long long slot_floats, float* out, float* records, int rule, int entries, int heads, int dim,
                              int vdim, int min_count, int max_chunks, cudaStream_t stream) {
    if (entries <= 0 || max_chunks <= 0) return 0;
    if (heads < 1 || min_count < 1 || (rule != RULE_REMOVAL && rule != RULE_BONUS)) return ME_ERR_ARGUMENT;
    const auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    if (!me_state_chunks_supports(dim, vdim) || slot_floats % 4 || !aligned(rows) || !aligned(state) || !aligned(out) || !aligned(records))
        return ME_ERR_UNSUPPORTED;
    if (slot_floats < static_cast<long long>(heads) * dim * vdim) return ME_ERR_ARGUMENT;
    ChunkArgs a{rows, scalars, cu_tokens, state_slots, fresh, state, (size_t)slot_floats, out, records, entries, heads, dim, vdim, min_count, max_chunks};
    return rule == RULE_REMOVAL ? dispatch_chunks<RULE_REMOVAL>(a, max_chunks, stream) : dispatch_chunks<RULE_BONUS>(a, max_chunks, stream);
}
