// Linear attention with a matrix state and a decay per key channel, over packed steps of several sequences: gated linear
// attention (GLA) and the gated delta rule, and a one-token kernel that also serves memories with exponential gates.
//
// A float row holds queries and keys of `groups` heads (dim numbers each) and values of `heads` heads (vdim numbers each);
// value head h uses query and key head h / (heads / groups) and has decays exp(l) of its own, l [tokens][heads * dim].  Per
// head and position p of a sequence, with S (dim x vdim, float) zero before the first token and D_p = diag(exp(l_p)):
//
//   plain:  S_p = D_p S_(p-1) + k_p v_p^T
//   delta:  S_p = D_p S_(p-1) + k_p u_p^T,   u_p = beta_p (v_p - (D_p S_(p-1))^T k_p)
//   o_p = S_p^T q_p
//
// Everything here is float.  Per sequence the cache keeps S twice, one row per slot [2][heads][dim][vdim]: a step reads the
// half of the position before its first (by that position's parity) and writes the half of its last, so a one-token step
// that runs twice (a graph's capture after its warm-up) computes the same thing both times.
//
// Longer steps: a sequence's tokens are cut into chunks.  Within one, E(j, i) = exp(l_(j+1) + .. + l_i) per channel and S the
// state before it,
//   o_i    = (q_i * E(-1, i)) S + sum_(j<=i) P_ij u_j,            P_ij = sum_n q_in k_jn E(j, i)_n   (u = v without the delta)
//   S_next = E(-1, L-1) S + sum_j (k_j * E(j, L-1)) u_j^T
// and with A_ij = beta_i sum_n k_in k_jn E(j, i)_n for j < i the delta rule's u solve (I + A) U = beta (V - (K * E(-1, .)) S),
// so U = U0 - W S where U0 and W solve the same triangle for beta V and beta (K * E(-1, .)).  A first kernel makes what is
// local to a chunk (the decayed keys; for the delta rule W and U0), a second walks the chunks of a sequence (U, and the
// state before every chunk), and a third makes the outputs of all chunks side by side.
//
// No exponent is a difference of two running sums, so a channel that forgets nearly everything costs the tokens behind it
// no precision: P and A are made level by level.  On the level with halves of h tokens, for the pairs whose query lies in
// the right half and whose key lies in the left half of one block of 2h tokens, E(j, i) = exp(sum from the middle to i)
// exp(sum behind j to the middle), two factors of at most one; every pair i > j meets on exactly one level.
#include "common.cuh"

namespace skv {

constexpr int CS_PREPARE_THREADS = 128, CS_OUT_THREADS = 256;
constexpr float CS_LOG2E = 1.4426950408889634f;        // (inside a chunk decays are kept as powers of two)

struct ChannelShape {
    int heads, groups, dim, vdim;
    int row_stride, q_at, k_at, v_at;      // floats per row, and the columns where queries, keys and values start
    float q_scale;                         // a factor on the queries
    float unit_eps;                        // >= 0: queries and keys are divided by sqrt(sum of squares + unit_eps)
};

struct ChannelBatch {
    const int* positions;                  // [tokens]
    const int* cu_q;                       // [seqs + 1]
    const int* slot_ids;                   // [seqs]
    float* state;                          // [slots][state_stride], S from state_offset on
    long long state_stride, state_offset;
};

__device__ __forceinline__ float cs_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float cs_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float cs_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float cs_log_sigmoid(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// ---- a second, low-rank projection with what follows it -----------------------------------------------------------
// out[t][c] = f(bias[c] + sum_j wt[j][c] x[t][j]); wt is the weight transposed, [rank][channels].
enum { LOW_RANK_PLAIN = 0, LOW_RANK_LOG_SIGMOID = 1, LOW_RANK_SOFTPLUS = 2 };

struct LowRankEnd {
    int mode;
    const float* bias;                     // [channels] or null
    float factor;                          // LOG_SIGMOID: log(sigmoid(z)) * factor
    const float* rate;                     // SOFTPLUS: -rate[c / per_rate] * softplus(z)
    int per_rate;
};

__device__ __forceinline__ float low_rank_end(const LowRankEnd& end, float z, int c) {
    if (end.mode == LOW_RANK_LOG_SIGMOID) return cs_log_sigmoid(z) * end.factor;
    if (end.mode == LOW_RANK_SOFTPLUS) return -end.rate[c / end.per_rate] * cs_softplus(z);
    return z;
}

// A block takes TOK tokens and 256 EACH channels, a thread EACH neighbouring channels: a weight that is read serves all of the
// block's tokens, and a token's number all of the thread's channels.
template <int EACH>
__device__ __forceinline__ void low_rank_weights(const float* p, float (&w)[EACH]) {
#pragma unroll
    for (int e = 0; e < EACH; ++e) w[e] = p[e];
}
template <int EACH>
__device__ __forceinline__ void low_rank_weights(const __nv_bfloat16* p, float (&w)[EACH]) {
    if (EACH == 2) {
        const float2 pair = __bfloat1622float2(*(const __nv_bfloat162*)p);
        w[0] = pair.x; w[EACH - 1] = pair.y;
    } else {
        w[0] = __bfloat162float(p[0]);
    }
}

template <typename T, int TOK, int EACH>
__global__ void __launch_bounds__(256)
low_rank_kernel(const float* __restrict__ x, int x_stride, int rank, const T* __restrict__ wt, const LowRankEnd end,
                float* __restrict__ out, int n_tokens, int channels) {
    extern __shared__ __align__(16) float cs_smem[];          // [rank][TOK]
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * TOK, count = min(TOK, n_tokens - t0);
    for (int idx = threadIdx.x; idx < TOK * rank; idx += 256) {
        const int tok = idx / rank, j = idx - tok * rank;
        cs_smem[j * TOK + tok] = tok < count ? x[(size_t)(t0 + tok) * x_stride + j] : 0.0f;
    }
    __syncthreads();
    const int c = (blockIdx.y * 256 + threadIdx.x) * EACH;
    if (c >= channels) return;
    float z[TOK][EACH];
#pragma unroll
    for (int e = 0; e < EACH; ++e) {
        const float bias = end.bias ? end.bias[c + e] : 0.0f;
#pragma unroll
        for (int tok = 0; tok < TOK; ++tok) z[tok][e] = bias;
    }
#pragma unroll 4
    for (int j = 0; j < rank; ++j) {
        float w[EACH];
        low_rank_weights<EACH>(wt + (size_t)j * channels + c, w);
#pragma unroll
        for (int tok = 0; tok < TOK; tok += 4) {
            const float4 v = *(const float4*)(cs_smem + j * TOK + tok);
#pragma unroll
            for (int e = 0; e < EACH; ++e) {
                z[tok][e] = fmaf(w[e], v.x, z[tok][e]); z[tok + 1][e] = fmaf(w[e], v.y, z[tok + 1][e]);
                z[tok + 2][e] = fmaf(w[e], v.z, z[tok + 2][e]); z[tok + 3][e] = fmaf(w[e], v.w, z[tok + 3][e]);
            }
        }
    }
#pragma unroll
    for (int tok = 0; tok < TOK; ++tok) {
        if (tok >= count) continue;
        float* to = out + (size_t)(t0 + tok) * channels + c;
        if (EACH == 2) *(float2*)to = make_float2(low_rank_end(end, z[tok][0], c), low_rank_end(end, z[tok][EACH - 1], c + EACH - 1));
        else to[0] = low_rank_end(end, z[tok][0], c);
    }
}

// ---- chunks: what the three kernels share ------------------------------------------------------------------------
__device__ __forceinline__ int cs_pad(int n) { return (n + 3) & ~3; }

// Where a thread stands over rows of `width` items: its item of a row, its first row, and the rows between its turns (threads
// past the last whole row have none).  Made once: divisions inside the loops would cost more than what the loops do.
struct RowPlace { int row, item, rows, lanes; };
template <int THREADS>
__device__ __forceinline__ RowPlace row_place(int width) {
    const int lanes = min(width, THREADS), rows = THREADS / lanes, row = threadIdx.x / lanes;
    return {row < rows ? row : 1 << 20, (int)threadIdx.x - row * lanes, rows, lanes};
}

// to[t][n] (rows ld apart) = scale * from[t * stride + n], zero beyond L tokens and N numbers.
template <int CH>
__device__ __forceinline__ void load_chunk(float* to, int ld, const float* __restrict__ from, size_t stride, int L, int N, int n_pad,
                                           const RowPlace& one, const RowPlace& four, float scale = 1.0f) {
    if (((stride | (size_t)N) & 3) == 0 && ((uintptr_t)from & 15) == 0) {
        for (int n = four.item * 4; n < n_pad; n += 4 * four.lanes)
#pragma unroll 4
            for (int t = four.row; t < CH; t += four.rows) {
                const float4 x = t < L ? *(const float4*)(from + t * stride + n) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                *(float4*)(to + t * ld + n) = make_float4(x.x * scale, x.y * scale, x.z * scale, x.w * scale);
            }
    } else {
        for (int n = one.item; n < n_pad; n += one.lanes)
            for (int t = one.row; t < CH; t += one.rows) to[t * ld + n] = t < L && n < N ? from[t * stride + n] * scale : 0.0f;
    }
}

// Rows become unit vectors (eps >= 0) and are multiplied by `scale`; a warp per row.
template <int CH, int THREADS>
__device__ __forceinline__ void unit_rows(float* rows, int ld, int n_pad, float eps, float scale) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < CH; t += THREADS / 32) {
        float factor = scale;
        if (eps >= 0.0f) {
            float squares = 0.0f;
            for (int n = lane; n < n_pad; n += 32) squares = fmaf(rows[t * ld + n], rows[t * ld + n], squares);
            factor = scale / sqrtf(warp_sum(squares) + eps);
        }
        if (factor != 1.0f)
            for (int n = lane; n < n_pad; n += 32) rows[t * ld + n] *= factor;
    }
}

// One level: scaled[t] of a right half is right[t] * 2^(sum from the middle to t), of a left half left[t] * 2^(sum behind t); l
// holds the logarithms of the decays to base two.
template <int CH, int HALF>
__device__ __forceinline__ void scale_level(float* scaled, const float* right, const float* left, const float* l, int ld, int n_pad,
                                            const RowPlace& one) {
    constexpr int SEGMENTS = CH / HALF;
    for (int n = one.item; n < n_pad; n += one.lanes)
        for (int segment = one.row; segment < SEGMENTS; segment += one.rows) {
            const int from = segment * HALF * ld + n;
            float sum = 0.0f;
            if (segment & 1) {
#pragma unroll 8
                for (int t = 0; t < HALF; ++t) {
                    const int at = from + t * ld;
                    sum += l[at];
                    scaled[at] = right[at] * exp2f(sum);
                }
            } else {
#pragma unroll 8
                for (int t = HALF - 1; t >= 0; --t) {
                    const int at = from + t * ld;
                    scaled[at] = left[at] * exp2f(sum);
                    sum += l[at];
                }
            }
        }
}

__device__ __forceinline__ float cs_dot4(const float4 a, const float4 b, float acc) {
    acc = fmaf(a.x, b.x, acc); acc = fmaf(a.y, b.y, acc); acc = fmaf(a.z, b.z, acc);
    return fmaf(a.w, b.w, acc);
}

// The level's pairs: w[i][j] = scaled[i] . scaled[j].
template <int CH, int THREADS, int HALF>
__device__ __forceinline__ void level_products(float* w, const float* scaled, int ld, int n_pad) {
    constexpr int PAIRS = CH * HALF / 2, LDW = CH + 4;
    if constexpr (PAIRS >= THREADS) {
        constexpr int EACH = PAIRS / THREADS, ROWS = THREADS / HALF;       // a thread's pairs share the key
        static_assert(EACH * ROWS == HALF || EACH == 1, "one block of 2 HALF tokens");
        const int r = threadIdx.x % (HALF * HALF), block = threadIdx.x / (HALF * HALF) * 2 * HALF;
        const int i = block + HALF + r / HALF, j = block + r % HALF;
        float acc[EACH];
#pragma unroll
        for (int e = 0; e < EACH; ++e) acc[e] = 0.0f;
        for (int n = 0; n < n_pad; n += 4) {
            const float4 key = *(const float4*)(scaled + j * ld + n);
#pragma unroll
            for (int e = 0; e < EACH; ++e) acc[e] = cs_dot4(*(const float4*)(scaled + (i + e * ROWS) * ld + n), key, acc[e]);
        }
#pragma unroll
        for (int e = 0; e < EACH; ++e) w[(i + e * ROWS) * LDW + j] = acc[e];
    } else {
        constexpr int PARTS = THREADS / PAIRS;                             // threads of a pair
        const int pair = threadIdx.x / PARTS, part = threadIdx.x % PARTS;
        const int r = pair % (HALF * HALF), block = pair / (HALF * HALF) * 2 * HALF;
        const int i = block + HALF + r / HALF, j = block + r % HALF;
        float acc = 0.0f;
        for (int n = 4 * part; n < n_pad; n += 4 * PARTS)
            acc = cs_dot4(*(const float4*)(scaled + i * ld + n), *(const float4*)(scaled + j * ld + n), acc);
#pragma unroll
        for (int offset = PARTS >> 1; offset > 0; offset >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, offset);
        if (part == 0) w[i * LDW + j] = acc;
    }
}

template <int CH, int THREADS, int HALF>
__device__ __forceinline__ void one_level(float* w, float* scaled, const float* right, const float* left, const float* l, int ld, int n_pad,
                                          const RowPlace& one) {
    scale_level<CH, HALF>(scaled, right, left, l, ld, n_pad, one);
    __syncthreads();
    level_products<CH, THREADS, HALF>(w, scaled, ld, n_pad);
    __syncthreads();
}

// w[i][j] (rows CH + 4 apart) = sum_n right[i][n] left[j][n] E(j, i)[n] for j < i.  Tokens past the chunk's last hold zeros.
template <int CH, int THREADS>
__device__ __forceinline__ void decayed_products(float* w, float* scaled, const float* right, const float* left, const float* l, int ld,
                                                 int n_pad, const RowPlace& one) {
    if constexpr (CH >= 32) one_level<CH, THREADS, 16>(w, scaled, right, left, l, ld, n_pad, one);
    one_level<CH, THREADS, 8>(w, scaled, right, left, l, ld, n_pad, one);
    one_level<CH, THREADS, 4>(w, scaled, right, left, l, ld, n_pad, one);
    one_level<CH, THREADS, 2>(w, scaled, right, left, l, ld, n_pad, one);
    one_level<CH, THREADS, 1>(w, scaled, right, left, l, ld, n_pad, one);
}

// scaled[t] = x[t] * 2^(l_0 + .. + l_t)
template <int CH>
__device__ __forceinline__ void scale_from_start(float* scaled, const float* x, const float* l, int ld, int n_pad, const RowPlace& one) {
    constexpr int SEGMENT = CH / 4;
    for (int n = one.item; n < n_pad; n += one.lanes)
        for (int segment = one.row; segment < 4; segment += one.rows) {
            float sum = 0.0f;
            for (int t = 0; t < segment * SEGMENT; ++t) sum += l[t * ld + n];
#pragma unroll
            for (int t = 0; t < SEGMENT; ++t) {
                const int at = (segment * SEGMENT + t) * ld + n;
                sum += l[at];
                scaled[at] = x[at] * exp2f(sum);
            }
        }
}

// ---- first kernel, plain ------------------------------------------------------------------------------------------
// keys[t][h * dim + n] = k * E(t, last of the chunk), factors[(s * max_chunks + chunk)][h * dim + n] = E over the chunk.
template <int CH>
__global__ void __launch_bounds__(256)
channel_keys_kernel(const float* __restrict__ rows, const float* __restrict__ log_decay, float* __restrict__ keys,
                    float* __restrict__ factors, int max_chunks, const ChannelShape shape, const int* __restrict__ cu_q) {
    pdl_launch_dependents();
    pdl_wait();
    const int channels = shape.heads * shape.dim, c = blockIdx.x * 256 + threadIdx.x, chunk = blockIdx.y, s = blockIdx.z;
    const int first = cu_q[s] + chunk * CH, L = min(CH, cu_q[s + 1] - first);
    if (L <= 0 || c >= channels) return;
    const int head = c / shape.dim, n = c - head * shape.dim, g = head / (shape.heads / shape.groups);
    const float* k = rows + (size_t)first * shape.row_stride + shape.k_at + g * shape.dim + n;
    float kr[CH], lr[CH];
#pragma unroll
    for (int t = 0; t < CH; ++t) {
        kr[t] = t < L ? k[(size_t)t * shape.row_stride] : 0.0f;
        lr[t] = t < L ? log_decay[(size_t)(first + t) * channels + c] : 0.0f;
    }
    float sum = 0.0f;
#pragma unroll
    for (int t = CH - 1; t >= 0; --t) {
        if (t < L) keys[(size_t)(first + t) * channels + c] = kr[t] * expf(sum);
        sum += lr[t];
    }
    factors[((size_t)s * max_chunks + chunk) * channels + c] = expf(sum);
}

// ---- first kernel, delta rule ----------------------------------------------------------------------------------------
// Also w_rows[t][h * dim + n] = W and u[t][h * vdim + e] = U0.  A block per (chunk, head, sequence).
template <int CH, int BLOCKS>
__global__ void __launch_bounds__(CS_PREPARE_THREADS, BLOCKS)
delta_prepare_kernel(const float* __restrict__ rows, const float* __restrict__ log_decay, const float* __restrict__ beta_rows,
                     int beta_stride, float* __restrict__ keys, float* __restrict__ factors, float* __restrict__ w_rows,
                     float* __restrict__ u, int max_chunks, const ChannelShape shape, const int* __restrict__ cu_q) {
    extern __shared__ __align__(16) float cs_smem[];
    constexpr int LDW = CH + 4;
    pdl_launch_dependents();
    pdl_wait();
    const int H = shape.heads, N = shape.dim, P = shape.vdim, n_pad = cs_pad(N), ld = n_pad + 4;
    float* k = cs_smem;                    // [CH][ld]
    float* l = k + CH * ld;                // [CH][ld]
    float* scaled = l + CH * ld;           // [CH][ld]
    float* A = scaled + CH * ld;           // [CH][LDW]
    float* AT = A + CH * LDW;              // [CH][LDW]: transposed, times beta of the row
    float* beta = AT + CH * LDW;           // [CH]
    const int chunk = blockIdx.x, head = blockIdx.y, s = blockIdx.z, g = head / (H / shape.groups);
    const int first = cu_q[s] + chunk * CH, L = min(CH, cu_q[s + 1] - first);
    if (L <= 0) return;
    const int channels = H * N;
    const RowPlace one = row_place<CS_PREPARE_THREADS>(n_pad), four = row_place<CS_PREPARE_THREADS>(n_pad >> 2);
    load_chunk<CH>(k, ld, rows + (size_t)first * shape.row_stride + shape.k_at + g * N, shape.row_stride, L, N, n_pad, one, four);
    load_chunk<CH>(l, ld, log_decay + (size_t)first * channels + head * N, channels, L, N, n_pad, one, four, CS_LOG2E);
    if (threadIdx.x < CH) beta[threadIdx.x] = threadIdx.x < L ? cs_sigmoid(beta_rows[(size_t)(first + threadIdx.x) * beta_stride + head]) : 0.0f;
    __syncthreads();
    unit_rows<CH, CS_PREPARE_THREADS>(k, ld, n_pad, shape.unit_eps, 1.0f);
    __syncthreads();
    // the decayed keys and the chunk's factor
    for (int n = threadIdx.x; n < N; n += CS_PREPARE_THREADS) {
        float sum = 0.0f;
        for (int t = CH - 1; t >= 0; --t) {
            if (t < L) keys[(size_t)(first + t) * channels + head * N + n] = k[t * ld + n] * exp2f(sum);
            sum += l[t * ld + n];
        }
        factors[((size_t)s * max_chunks + chunk) * channels + head * N + n] = exp2f(sum);
    }
    decayed_products<CH, CS_PREPARE_THREADS>(A, scaled, k, k, l, ld, n_pad, one);
    scale_from_start<CH>(scaled, k, l, ld, n_pad, one);
    for (int idx = threadIdx.x; idx < CH * CH; idx += CS_PREPARE_THREADS) {
        const int j = idx / CH, i = idx - j * CH;
        AT[j * LDW + i] = j < i ? A[i * LDW + j] * beta[i] : 0.0f;
    }
    __syncthreads();
    // (I + A) X = beta [K * E | V]: a thread takes a column, and a row that is done is taken off all rows below it
    for (int column = threadIdx.x; column < N + P; column += CS_PREPARE_THREADS) {
        const bool is_key = column < N;
        const int c = is_key ? column : column - N;
        const float* v = rows + (size_t)first * shape.row_stride + shape.v_at + head * P + c;
        float x[CH];
#pragma unroll
        for (int i = 0; i < CH; ++i) x[i] = i < L ? beta[i] * (is_key ? scaled[i * ld + c] : v[(size_t)i * shape.row_stride]) : 0.0f;
#pragma unroll
        for (int j = 0; j < CH - 1; ++j) {
#pragma unroll
            for (int i = (j + 1) & ~3; i < CH; i += 4) {
                const float4 a = *(const float4*)(AT + j * LDW + i);       // (zero up to the diagonal)
                if (i > j) x[i] = fmaf(-a.x, x[j], x[i]);
                if (i + 1 > j) x[i + 1] = fmaf(-a.y, x[j], x[i + 1]);
                if (i + 2 > j) x[i + 2] = fmaf(-a.z, x[j], x[i + 2]);
                if (i + 3 > j) x[i + 3] = fmaf(-a.w, x[j], x[i + 3]);
            }
        }
        float* to = is_key ? w_rows + (size_t)first * channels + head * N + c : u + (size_t)first * H * P + (size_t)head * P + c;
        const size_t stride = is_key ? channels : H * P;
#pragma unroll
        for (int i = 0; i < CH; ++i)
            if (i < L) to[i * stride] = x[i];
    }
}

// ---- second kernel: the walk over a sequence's chunks ---------------------------------------------------------------
// A block per (slice of C value columns, head, sequence); a thread owns two key channels by two columns of S per 64
// channels.  states [seqs][max_chunks][heads][dim][vdim] gets the state before every chunk; with the delta rule
// u [tokens][heads * vdim] turns from U0 into U.  The next chunks' rows are on their way while one is worked on (a ring of two
// or four).
__device__ __forceinline__ void cs_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cs_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// What a thread copies of an array's rows for every chunk: made once, so that a chunk costs it little but the copies.  Rows of
// `items` pieces of 16 bytes (vec) or of 4.
struct StagePlan {
    const float* src;                      // this thread's piece of its first row of chunk 0
    int dst;                               // where it goes within the array's place of a stage
    int row, rows;                         // its first row and the rows between its turns
    size_t src_step;
    int dst_step;
    int item, items, lanes;                // its first piece of a row, the pieces, and those between its turns within a row
};

template <int THREADS>
__device__ __forceinline__ StagePlan stage_plan(const float* from, size_t stride, int ld, int items, bool vec) {
    const RowPlace place = row_place<THREADS>(items);
    const int each = vec ? 4 : 1, row = min(place.row, 1 << 14);
    return {from + (size_t)row * stride + place.item * each, row * ld + place.item * each, row, place.rows, place.rows * stride, place.rows * ld,
            place.item, items, place.lanes};
}

// Rows [0, rows) of a chunk that starts `skip` floats into the array; those past `there` become zero.
__device__ __forceinline__ void stage_rows(float* to, const StagePlan& plan, size_t skip, int there, int rows, bool vec) {
    for (int more = 0; plan.item + more < plan.items; more += plan.lanes) {        // (once, unless a row has more pieces than threads)
        float* at = to + plan.dst + more * (vec ? 4 : 1);
        const float* src = plan.src + skip + more * (vec ? 4 : 1);
        for (int t = plan.row; t < rows; t += plan.rows) {
            if (vec) {
                if (t < there) cs_copy16(at, src);
                else *(float4*)at = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            } else {
                if (t < there) cs_copy4(at, src);
                else *at = 0.0f;
            }
            at += plan.dst_step;
            src += plan.src_step;
        }
    }
}

template <int CH, int C, bool DELTA>
__global__ void __launch_bounds__(C * 16)
channel_walk_kernel(const float* __restrict__ keys, const float* __restrict__ factors, const float* __restrict__ w_rows, float* u,
                    const float* __restrict__ values, int value_stride, float* __restrict__ states, int max_chunks, int stages,
                    const ChannelShape shape, const ChannelBatch batch) {
    extern __shared__ __align__(16) float cs_smem[];
    constexpr int THREADS = C * 16;
    pdl_launch_dependents();
    pdl_wait();
    const int H = shape.heads, N = shape.dim, P = shape.vdim, n_pad = cs_pad(N), ld = n_pad + 4, channels = H * N;
    const int e0 = blockIdx.x * C, head = blockIdx.y, s = blockIdx.z, width = min(C, P - e0);
    const int first = batch.cu_q[s], count = batch.cu_q[s + 1] - first;
    if (count <= 0) return;
    const int set = CH * ld * (DELTA ? 2 : 1) + CH * C + n_pad;
    float* S = cs_smem;                    // [n_pad][C]
    float* sets = S + n_pad * C;
    const int p_first = batch.positions[first], p_last = p_first + count - 1;
    float* slot = batch.state + (size_t)batch.slot_ids[s] * batch.state_stride + batch.state_offset;
    const size_t half = (size_t)H * N * P, mine = (size_t)head * N * P + e0;
    const float* before = slot + (size_t)((p_first - 1) & 1) * half + mine;
    for (int idx = threadIdx.x; idx < n_pad * C; idx += THREADS) {
        const int n = idx / C, c = idx - n * C;
        S[idx] = p_first > 0 && n < N && c < width ? before[(size_t)n * P + c] : 0.0f;
    }
    for (int idx = threadIdx.x; idx < stages * set; idx += THREADS) sets[idx] = 0.0f;        // (what pads stays zero)
    __syncthreads();
    const bool vec_n = (N & 3) == 0;
    const int u_stride = DELTA ? H * P : value_stride;
    const float* u_from = DELTA ? u + (size_t)head * P + e0 : values + (size_t)head * P + e0;
    const bool vec_u = ((u_stride | P | e0) & 3) == 0 && ((uintptr_t)u_from & 15) == 0 && (width & 3) == 0;
    const int n_items = vec_n ? N >> 2 : N, u_items = vec_u ? width >> 2 : width;
    const size_t chunk_keys = (size_t)CH * channels, chunk_values = (size_t)CH * u_stride;
    const StagePlan key_plan = stage_plan<THREADS>(keys + (size_t)first * channels + head * N, channels, ld, n_items, vec_n);
    const StagePlan value_plan = stage_plan<THREADS>(u_from + (size_t)first * u_stride, u_stride, C, u_items, vec_u);
    const StagePlan factor_plan = stage_plan<THREADS>(factors + (size_t)s * max_chunks * channels + head * N, 0, n_pad, n_items, vec_n);
    const float* w_first = DELTA ? w_rows + (key_plan.src - keys) : nullptr;
    auto stage = [&](int which, int chunk) {
        float* kh = sets + which * set;
        const int L = min(CH, count - chunk * CH);
        stage_rows(kh, key_plan, chunk * chunk_keys, L, CH, vec_n);
        if (DELTA) {
            StagePlan w_plan = key_plan;
            w_plan.src = w_first;
            stage_rows(kh + CH * ld, w_plan, chunk * chunk_keys, L, CH, vec_n);
        }
        float* ut = kh + CH * ld * (DELTA ? 2 : 1);
        stage_rows(ut, value_plan, chunk * chunk_values, L, CH, vec_u);
        stage_rows(ut + CH * C, factor_plan, (size_t)chunk * channels, 1, 1, vec_n);
    };
    const int rg = threadIdx.x / (C / 2), c0 = (threadIdx.x % (C / 2)) * 2;
    const int chunks = (count + CH - 1) / CH;
    const bool pairs = (P & 1) == 0;
    for (int ahead = 0; ahead < stages - 1; ++ahead) {
        if (ahead < chunks) stage(ahead, ahead);
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    for (int chunk = 0; chunk < chunks; ++chunk) {
        if (stages == 4) asm volatile("cp.async.wait_group 2;" ::: "memory");
        else asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                   // this chunk's rows are there, and everybody is done with the one before
        if (chunk + stages - 1 < chunks) stage((chunk + stages - 1) & (stages - 1), chunk + stages - 1);
        asm volatile("cp.async.commit_group;" ::: "memory");
        float* kh = sets + (chunk & (stages - 1)) * set;
        float* w = kh + CH * ld;
        float* ut = kh + CH * ld * (DELTA ? 2 : 1);
        const float* f = ut + CH * C;
        const int t0 = first + chunk * CH, L = min(CH, count - chunk * CH);
        if (DELTA) {
            if (rg < CH) {                 // a token by two columns a thread
                float2 acc = *(const float2*)(ut + rg * C + c0);
                const float* w_row = w + rg * ld;
#pragma unroll 4
                for (int n = 0; n < n_pad; n += 4) {
                    const float4 wv = *(const float4*)(w_row + n);
                    const float2 s0 = *(const float2*)(S + n * C + c0), s1 = *(const float2*)(S + (n + 1) * C + c0);
                    const float2 s2 = *(const float2*)(S + (n + 2) * C + c0), s3 = *(const float2*)(S + (n + 3) * C + c0);
                    acc.x = fmaf(-wv.x, s0.x, acc.x); acc.y = fmaf(-wv.x, s0.y, acc.y);
                    acc.x = fmaf(-wv.y, s1.x, acc.x); acc.y = fmaf(-wv.y, s1.y, acc.y);
                    acc.x = fmaf(-wv.z, s2.x, acc.x); acc.y = fmaf(-wv.z, s2.y, acc.y);
                    acc.x = fmaf(-wv.w, s3.x, acc.x); acc.y = fmaf(-wv.w, s3.y, acc.y);
                }
                *(float2*)(ut + rg * C + c0) = acc;                        // (nobody else reads or writes these yet)
                if (rg < L) {
                    float* to = u + (size_t)(t0 + rg) * H * P + (size_t)head * P + e0 + c0;
                    if (pairs && c0 + 1 < width) *(float2*)to = acc;
                    else {
                        if (c0 < width) to[0] = acc.x;
                        if (c0 + 1 < width) to[1] = acc.y;
                    }
                }
            }
            __syncthreads();               // U is there, and everybody is done with S as it was
        }
        float* kept = states + (((size_t)s * max_chunks + chunk) * H + head) * (size_t)N * P + e0 + c0;
        for (int n0 = rg * 2; n0 < n_pad; n0 += 64) {
            float2 sv[2];
            const float2 fv = *(const float2*)(f + n0);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                sv[x] = *(const float2*)(S + (n0 + x) * C + c0);
                if (n0 + x < N) {
                    if (pairs && c0 + 1 < width) *(float2*)(kept + (size_t)(n0 + x) * P) = sv[x];
                    else {
                        if (c0 < width) kept[(size_t)(n0 + x) * P] = sv[x].x;
                        if (c0 + 1 < width) kept[(size_t)(n0 + x) * P + 1] = sv[x].y;
                    }
                }
                sv[x].x *= x == 0 ? fv.x : fv.y;
                sv[x].y *= x == 0 ? fv.x : fv.y;
            }
#pragma unroll
            for (int j = 0; j < CH; ++j) {
                const float2 kv = *(const float2*)(kh + j * ld + n0);
                const float2 uv = *(const float2*)(ut + j * C + c0);
                sv[0].x = fmaf(kv.x, uv.x, sv[0].x); sv[0].y = fmaf(kv.x, uv.y, sv[0].y);
                sv[1].x = fmaf(kv.y, uv.x, sv[1].x); sv[1].y = fmaf(kv.y, uv.y, sv[1].y);
            }
#pragma unroll
            for (int x = 0; x < 2; ++x) *(float2*)(S + (n0 + x) * C + c0) = sv[x];
        }
    }
    // (a thread writes what it owns)
    float* after = slot + (size_t)(p_last & 1) * half + mine + c0;
    for (int n0 = rg * 2; n0 < N; n0 += 64)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            if (n0 + x >= N) continue;
            const float2 sv = *(const float2*)(S + (n0 + x) * C + c0);
            if (c0 < width) after[(size_t)(n0 + x) * P] = sv.x;
            if (c0 + 1 < width) after[(size_t)(n0 + x) * P + 1] = sv.y;
        }
}

// ---- third kernel: outputs ---------------------------------------------------------------------------------------------
// A block per (chunk, head, sequence): threads in 16 x 16, each with CH / 16 tokens and four columns of a tile of 64.
// values: the row of (token, head) at values + token * value_stride + head * vdim (v, or the delta rule's U).
template <int CH>
__global__ void __launch_bounds__(CS_OUT_THREADS, 4)
channel_output_kernel(const float* __restrict__ rows, const float* __restrict__ log_decay, const float* __restrict__ values,
                      int value_stride, const float* __restrict__ states, float* __restrict__ out, int max_chunks,
                      const ChannelShape shape, const int* __restrict__ cu_q) {
    extern __shared__ __align__(16) float cs_smem[];
    constexpr int LDW = CH + 4, RI = CH / 16;
    pdl_launch_dependents();
    pdl_wait();
    const int H = shape.heads, N = shape.dim, P = shape.vdim, n_pad = cs_pad(N), ld = n_pad + 4;
    float* q = cs_smem;                    // [CH][ld]
    float* scaled = q + CH * ld;           // [CH][ld]
    float* w = scaled + CH * ld;           // [CH][LDW]
    float* vs = w + CH * LDW;              // [CH][64]
    float* k = vs + CH * 64;               // [CH][ld]
    float* l = k + CH * ld;                // [CH][ld]
    float* st = k;                         // [n_pad][64], once keys and decays have been used
    const int chunk = blockIdx.x, head = blockIdx.y, s = blockIdx.z, g = head / (H / shape.groups);
    const int first = cu_q[s] + chunk * CH, L = min(CH, cu_q[s + 1] - first);
    if (L <= 0) return;
    const float* base = rows + (size_t)first * shape.row_stride;
    const RowPlace one = row_place<CS_OUT_THREADS>(n_pad), four = row_place<CS_OUT_THREADS>(n_pad >> 2);
    load_chunk<CH>(q, ld, base + shape.q_at + g * N, shape.row_stride, L, N, n_pad, one, four);
    load_chunk<CH>(k, ld, base + shape.k_at + g * N, shape.row_stride, L, N, n_pad, one, four);
    load_chunk<CH>(l, ld, log_decay + (size_t)first * H * N + head * N, (size_t)H * N, L, N, n_pad, one, four, CS_LOG2E);
    for (int idx = threadIdx.x; idx < CH * LDW; idx += CS_OUT_THREADS) w[idx] = 0.0f;
    __syncthreads();
    unit_rows<CH, CS_OUT_THREADS>(q, ld, n_pad, shape.unit_eps, shape.q_scale);
    if (shape.unit_eps >= 0.0f) unit_rows<CH, CS_OUT_THREADS>(k, ld, n_pad, shape.unit_eps, 1.0f);
    __syncthreads();
    {   // a token's own key
        constexpr int PARTS = CS_OUT_THREADS / CH;
        const int i = threadIdx.x / PARTS, part = threadIdx.x % PARTS;
        float acc = 0.0f;
        for (int n = 4 * part; n < n_pad; n += 4 * PARTS) acc = cs_dot4(*(const float4*)(q + i * ld + n), *(const float4*)(k + i * ld + n), acc);
#pragma unroll
        for (int offset = PARTS >> 1; offset > 0; offset >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, offset);
        if (part == 0) w[i * LDW + i] = acc;
    }
    decayed_products<CH, CS_OUT_THREADS>(w, scaled, q, k, l, ld, n_pad, one);
    scale_from_start<CH>(scaled, q, l, ld, n_pad, one);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, i0 = ty * RI;
    const float* before = states + (((size_t)s * max_chunks + chunk) * H + head) * (size_t)N * P;
    const float* vbase = values + (size_t)first * value_stride + (size_t)head * P;
    const bool vec_s = (P & 3) == 0, vec_v = ((value_stride | P) & 3) == 0 && ((uintptr_t)vbase & 15) == 0;
    const int j_end = min(L, (i0 + RI + 3) & ~3);
    for (int e0 = 0; e0 < P; e0 += 64) {
        __syncthreads();                   // keys and decays, or the tile before, have been used
        if (vec_v) {
            for (int idx = threadIdx.x; idx < CH * 16; idx += CS_OUT_THREADS) {
                const int j = idx >> 4, e = (idx & 15) * 4;
                *(float4*)(vs + j * 64 + e) = j < L && e0 + e < P ? *(const float4*)(vbase + (size_t)j * value_stride + e0 + e) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        } else {
            for (int idx = threadIdx.x; idx < CH * 64; idx += CS_OUT_THREADS) {
                const int j = idx >> 6, e = idx & 63;
                vs[idx] = j < L && e0 + e < P ? vbase[(size_t)j * value_stride + e0 + e] : 0.0f;
            }
        }
        if (vec_s) {
#pragma unroll 4
            for (int idx = threadIdx.x; idx < n_pad * 16; idx += CS_OUT_THREADS) {
                const int n = idx >> 4, e = (idx & 15) * 4;
                *(float4*)(st + n * 64 + e) = n < N && e0 + e < P ? *(const float4*)(before + (size_t)n * P + e0 + e) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        } else {
            for (int idx = threadIdx.x; idx < n_pad * 64; idx += CS_OUT_THREADS) {
                const int n = idx >> 6, e = idx & 63;
                st[idx] = n < N && e0 + e < P ? before[(size_t)n * P + e0 + e] : 0.0f;
            }
        }
        __syncthreads();
        float acc[RI][4];
#pragma unroll
        for (int a = 0; a < RI; ++a)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[a][e] = 0.0f;
        auto add = [&](const float* left, int left_ld, const float* right, int row) {      // four rows of `right` at a time
            float4 r[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) r[x] = *(const float4*)(right + (row + x) * 64 + tx * 4);
#pragma unroll
            for (int a = 0; a < RI; ++a) {
                const float4 f = *(const float4*)(left + (i0 + a) * left_ld + row);
                acc[a][0] = fmaf(f.x, r[0].x, acc[a][0]); acc[a][1] = fmaf(f.x, r[0].y, acc[a][1]);
                acc[a][2] = fmaf(f.x, r[0].z, acc[a][2]); acc[a][3] = fmaf(f.x, r[0].w, acc[a][3]);
                acc[a][0] = fmaf(f.y, r[1].x, acc[a][0]); acc[a][1] = fmaf(f.y, r[1].y, acc[a][1]);
                acc[a][2] = fmaf(f.y, r[1].z, acc[a][2]); acc[a][3] = fmaf(f.y, r[1].w, acc[a][3]);
                acc[a][0] = fmaf(f.z, r[2].x, acc[a][0]); acc[a][1] = fmaf(f.z, r[2].y, acc[a][1]);
                acc[a][2] = fmaf(f.z, r[2].z, acc[a][2]); acc[a][3] = fmaf(f.z, r[2].w, acc[a][3]);
                acc[a][0] = fmaf(f.w, r[3].x, acc[a][0]); acc[a][1] = fmaf(f.w, r[3].y, acc[a][1]);
                acc[a][2] = fmaf(f.w, r[3].z, acc[a][2]); acc[a][3] = fmaf(f.w, r[3].w, acc[a][3]);
            }
        };
#pragma unroll 2
        for (int n = 0; n < n_pad; n += 4) add(scaled, ld, st, n);          // what the state before the chunk gives
        for (int j = 0; j < j_end; j += 4) add(w, LDW, vs, j);              // what the chunk's own tokens give
        const int e = e0 + tx * 4;
#pragma unroll
        for (int a = 0; a < RI; ++a) {
            if (i0 + a >= L || e >= P) continue;
            float* to = out + ((size_t)(first + i0 + a) * H + head) * P + e;
            if (vec_s) {
                *(float4*)to = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (e + x < P) to[x] = acc[a][x];
            }
        }
    }
}

// ---- one token a sequence, from the projection to the output projection's input --------------------------------------
// A block per (head, sequence).  Three kinds of memory:
//   STEP_CHANNEL  decays per key channel from a low-rank projection
//   STEP_DELTA    the same with the delta rule, a short convolution with silu in front (its last inputs in a ring, row
//                 position mod taps) and unit vectors
//   STEP_EXP      one decay per head from exponential gates with a running maximum m and a normaliser n per key channel:
//                 m' = max(f + m, i), S' = exp(f + m - m') S + exp(i - m') k v^T, n' likewise with k alone,
//                 o = S'^T q / (max(|n' . q|, exp(-m')) + denominator_eps);  i = cap tanh((row + b) / cap),
//                 f = log sigmoid(cap tanh((row + b) / cap)).  A half of the state is S of all heads, then n; the two m of
//                 every head lie behind the halves.
// Then o over its root mean square per head, times a weight, times a gate (sigmoid or silu of a column of the row, or of a
// low-rank projection), in the compute dtype.
enum { STEP_CHANNEL = 0, STEP_DELTA = 1, STEP_EXP = 2 };
constexpr int MS_THREADS = 256, MS_HELD = 16;

struct MatrixStep {
    ChannelShape shape;
    int kind;
    const float* conv_w;                   // [channels][taps] over the row's first columns, or null
    int taps, channels;
    long long ring_offset;
    const skv_t* decay_wt;                 // [decay_rank][heads * dim]
    int decay_at, decay_rank;              // the column where the low-rank part starts
    LowRankEnd decay_end;
    int beta_at;
    int input_at, forget_at;               // STEP_EXP: columns of the gates' logits
    const float* input_bias;
    const float* forget_bias;
    float cap, denominator_eps;
    int gate_at, gate_rank, gate_silu;     // gate_rank 0: the logits are the row's columns from gate_at on
    const skv_t* gate_wt;                  // [gate_rank][heads * vdim]
    const float* norm;                     // [heads * vdim]
    float eps;
};

// z[c] = sum_j wt[j][c0 + c] x[j] for c < count; x in shared memory; partial [max(count, MS_THREADS)].  Ends with a barrier.
template <typename T>
__device__ __forceinline__ void low_rank_columns(float* z, float* partial, const float* x, int rank, const T* __restrict__ wt,
                                                 int total, int c0, int count) {
    if (count >= MS_THREADS) {
        for (int c = threadIdx.x; c < count; c += MS_THREADS) {
            float sum = 0.0f;
#pragma unroll 8
            for (int j = 0; j < rank; ++j) sum = fmaf(to_float(wt[(size_t)j * total + c0 + c]), x[j], sum);
            z[c] = sum;
        }
        __syncthreads();
        return;
    }
    const int parts = MS_THREADS / count, part = threadIdx.x / count, c = threadIdx.x - part * count;
    if (part < parts) {
        float sum = 0.0f;
#pragma unroll 8
        for (int j = part; j < rank; j += parts) sum = fmaf(to_float(wt[(size_t)j * total + c0 + c]), x[j], sum);
        partial[part * count + c] = sum;
    }
    __syncthreads();
    if (threadIdx.x < count) {
        float sum = 0.0f;
        for (int r = 0; r < parts; ++r) sum += partial[r * count + threadIdx.x];
        z[threadIdx.x] = sum;
    }
    __syncthreads();
}

__host__ __device__ __forceinline__ int ms_smem_floats(int N, int P, int rank, int vec) {
    const int wide = N > P ? N : P, columns = 2 * MS_THREADS * vec;
    return 3 * ((N + 3) & ~3) + 3 * ((P + 3) & ~3) + ((rank + 3) & ~3) + (columns > wide ? columns : wide) + 40;
}

// Sums of three numbers over the block; every thread gets them.  `scratch` holds 24 floats and may be reused after a barrier.
__device__ __forceinline__ float3 block_sum3(float a, float b, float c, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a); b = warp_sum(b); c = warp_sum(c);
    __syncthreads();
    if (lane == 0) { scratch[3 * warp] = a; scratch[3 * warp + 1] = b; scratch[3 * warp + 2] = c; }
    __syncthreads();
    float3 sums = make_float3(0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int w = 0; w < MS_THREADS / 32; ++w) { sums.x += scratch[3 * w]; sums.y += scratch[3 * w + 1]; sums.z += scratch[3 * w + 2]; }
    return sums;
}

template <typename T, int VEC, int KIND>
__global__ void __launch_bounds__(MS_THREADS)
matrix_step_kernel(const float* __restrict__ rows, T* __restrict__ out, int out_stride, const MatrixStep a, const ChannelBatch batch) {
    extern __shared__ __align__(16) float cs_smem[];
    const int H = a.shape.heads, N = a.shape.dim, P = a.shape.vdim, n4 = (N + 3) & ~3, p4 = (P + 3) & ~3;
    float* q = cs_smem;                    // [N]
    float* k = q + n4;                     // [N]
    float* d = k + n4;                     // [N]: the decays
    float* v = d + n4;                     // [P]
    float* o = v + p4;                     // [P]
    float* u = o + p4;                     // [P]: what is written beside the key
    float* scratch = u + p4;               // [40]
    float* lora = scratch + 40;            // [rank]
    float* partial = lora + (((KIND == STEP_EXP ? 0 : max(a.decay_rank, a.gate_rank)) + 3) & ~3);   // [2 * MS_THREADS * VEC]
    pdl_launch_dependents();
    const int head = blockIdx.x, s = blockIdx.y, g = head / (H / a.shape.groups);
    const int t = batch.cu_q[s], p = batch.positions[t];
    const float* row = rows + (size_t)t * a.shape.row_stride;
    float* slot = batch.state + (size_t)batch.slot_ids[s] * batch.state_stride;
    const size_t half = (size_t)H * N * P + (KIND == STEP_EXP ? (size_t)H * N : 0);
    const float* half_before = slot + batch.state_offset + (size_t)((p - 1) & 1) * half;
    float* half_after = slot + batch.state_offset + (size_t)(p & 1) * half;
    const float* __restrict__ before = half_before + (size_t)head * N * P;
    float* __restrict__ after = half_after + (size_t)head * N * P;
    const int columns = P / VEC, lanes = min(columns, MS_THREADS), per_pass = MS_THREADS / lanes;
    const int r0 = threadIdx.x / lanes, c_lane = threadIdx.x - r0 * lanes;
    float old[MS_HELD][VEC];
    auto fetch = [&](int n0, int c) {      // this thread's next numbers of the state before the token
#pragma unroll
        for (int x = 0; x < MS_HELD; ++x) {
            const int n = n0 + x * per_pass;
            const bool there = p > 0 && n < N && c < columns && r0 < per_pass;
            if (VEC == 4) {
                const float4 z = there ? *(const float4*)(before + (size_t)n * P + c * 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                old[x][0] = z.x; old[x][1 % VEC] = z.y; old[x][2 % VEC] = z.z; old[x][3 % VEC] = z.w;
            } else {
                old[x][0] = there ? before[(size_t)n * P + c] : 0.0f;
            }
        }
    };
    // The step's metadata came with a copy in front of all its kernels, which also put everything that earlier steps
    // launched behind it; the state before this token was written in an earlier step.  So the first part of it is fetched
    // while the projection in front of this kernel still runs.
    fetch(r0, c_lane);
    pdl_wait();
    // queries, keys and values of the token
    if (KIND == STEP_DELTA) {
        float* ring = slot + a.ring_offset;
        const bool first_of_group = head % (H / a.shape.groups) == 0;
        for (int i = threadIdx.x; i < P + 2 * N; i += MS_THREADS) {
            const int c = i < P ? a.shape.v_at + head * P + i : (i < P + N ? a.shape.k_at + g * N + i - P : a.shape.q_at + g * N + i - P - N);
            float sum = 0.0f;
            for (int j = 0; j < a.taps; ++j) {
                const int back = a.taps - 1 - j;
                if (p - back < 0) continue;
                sum = fmaf(a.conv_w[(size_t)c * a.taps + j], back == 0 ? row[c] : ring[(size_t)((p - back) % a.taps) * a.channels + c], sum);
            }
            const float value = cs_silu(sum);
            if (i < P) v[i] = value;
            else if (i < P + N) k[i - P] = value;
            else q[i - P - N] = value;
            // (the one row of the ring that no tap of this token reads)
            if (a.taps > 1 && (i < P || first_of_group)) ring[(size_t)(p % a.taps) * a.channels + c] = row[c];
        }
    } else {
        for (int i = threadIdx.x; i < N; i += MS_THREADS) {
            q[i] = row[a.shape.q_at + g * N + i] * a.shape.q_scale;
            k[i] = row[a.shape.k_at + g * N + i];
        }
        for (int i = threadIdx.x; i < P; i += MS_THREADS) v[i] = row[a.shape.v_at + head * P + i];
    }
    if (KIND != STEP_EXP)
        for (int j = threadIdx.x; j < a.decay_rank; j += MS_THREADS) lora[j] = row[a.decay_at + j];
    __syncthreads();
    float floor_of_weight = 0.0f, weight = 0.0f;
    if (KIND == STEP_EXP) {
        const float* m_before = slot + batch.state_offset + 2 * half + (size_t)((p - 1) & 1) * H + head;
        const float i = a.cap * tanhf((row[a.input_at + head] + a.input_bias[head]) / a.cap);
        const float f = cs_log_sigmoid(a.cap * tanhf((row[a.forget_at + head] + a.forget_bias[head]) / a.cap));
        const float m = p > 0 ? *m_before : 0.0f, top = fmaxf(f + m, i);
        const float keep = expf(f + m - top), take = expf(i - top);
        floor_of_weight = expf(-top);
        const float* n_before = half_before + (size_t)H * N * P + (size_t)head * N;
        float* n_after = half_after + (size_t)H * N * P + (size_t)head * N;
        float dot = 0.0f;
        for (int n = threadIdx.x; n < N; n += MS_THREADS) {
            const float taken = k[n] * take;
            const float fresh = fmaf(keep, p > 0 ? n_before[n] : 0.0f, taken);
            n_after[n] = fresh;
            dot = fmaf(fresh, q[n], dot);
            k[n] = taken;
            d[n] = keep;
        }
        if (threadIdx.x == 0) slot[batch.state_offset + 2 * half + (size_t)(p & 1) * H + head] = top;
        weight = block_sum(dot, scratch);
    } else {
        low_rank_columns(d, partial, lora, a.decay_rank, a.decay_wt, H * N, head * N, N);
        for (int n = threadIdx.x; n < N; n += MS_THREADS)
            d[n] = expf(low_rank_end(a.decay_end, d[n] + (a.decay_end.bias ? a.decay_end.bias[head * N + n] : 0.0f), head * N + n));
    }
    float key_dot_query = 0.0f, beta = 0.0f;
    if (KIND == STEP_DELTA) {
        float sq = 0.0f, sk = 0.0f, qk = 0.0f;
        for (int n = threadIdx.x; n < N; n += MS_THREADS) {
            sq = fmaf(q[n], q[n], sq); sk = fmaf(k[n], k[n], sk); qk = fmaf(q[n], k[n], qk);
        }
        const float3 sums = block_sum3(sq, sk, qk, scratch);
        sq = sums.x; sk = sums.y; qk = sums.z;
        const bool unit = a.shape.unit_eps >= 0.0f;
        const float fq = unit ? a.shape.q_scale / sqrtf(sq + a.shape.unit_eps) : a.shape.q_scale;
        const float fk = unit ? 1.0f / sqrtf(sk + a.shape.unit_eps) : 1.0f;
        for (int n = threadIdx.x; n < N; n += MS_THREADS) { q[n] *= fq; k[n] *= fk; }
        key_dot_query = qk * fq * fk;
        beta = cs_sigmoid(row[a.beta_at + head]);
    }
    __syncthreads();
    for (int cb = 0; cb < columns; cb += lanes) {      // (more than one pass only where a row has more columns than threads)
        const int c = cb + c_lane;
        const bool working = r0 < per_pass && c < columns;
        float acc[VEC], seen[VEC], ve[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) { acc[e] = 0.0f; seen[e] = 0.0f; ve[e] = working ? v[c * VEC + e] : 0.0f; }
        auto store = [&](int n, const float (&fresh)[VEC]) {
            if (VEC == 4) *(float4*)(after + (size_t)n * P + c * 4) = make_float4(fresh[0], fresh[1 % VEC], fresh[2 % VEC], fresh[3 % VEC]);
            else after[(size_t)n * P + c] = fresh[0];
        };
        const int block = per_pass * MS_HELD;
        if (working)
            for (int n0 = r0; n0 < N; n0 += block) {
                if (cb > 0 || n0 > r0) fetch(n0, c);
#pragma unroll
                for (int x = 0; x < MS_HELD; ++x) {
                    const int n = n0 + x * per_pass;
                    if (n >= N) break;
                    const float dn = d[n], kn = k[n], qn = q[n];
                    float fresh[VEC];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        if (KIND == STEP_DELTA) {
                            fresh[e] = dn * old[x][e];
                            seen[e] = fmaf(fresh[e], kn, seen[e]);
                        } else {
                            fresh[e] = fmaf(dn, old[x][e], kn * ve[e]);
                        }
                        acc[e] = fmaf(fresh[e], qn, acc[e]);
                    }
                    if (KIND != STEP_DELTA) store(n, fresh);
                }
            }
        if (r0 < per_pass) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                partial[(r0 * lanes + c_lane) * VEC + e] = acc[e];
                if (KIND == STEP_DELTA) partial[MS_THREADS * VEC + (r0 * lanes + c_lane) * VEC + e] = seen[e];
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < lanes * VEC; i += MS_THREADS) {
            const int e = cb * VEC + i;
            if (e >= P) continue;
            float sum = 0.0f, old_value = 0.0f;
            for (int r = 0; r < per_pass; ++r) {
                sum += partial[r * lanes * VEC + i];
                if (KIND == STEP_DELTA) old_value += partial[MS_THREADS * VEC + r * lanes * VEC + i];
            }
            if (KIND == STEP_DELTA) {
                u[e] = beta * (v[e] - old_value);
                sum = fmaf(key_dot_query, u[e], sum);
            }
            if (KIND == STEP_EXP) sum = sum / (fmaxf(fabsf(weight), floor_of_weight) + a.denominator_eps);
            o[e] = sum;
        }
        __syncthreads();
        if (KIND == STEP_DELTA && working) {           // the state again, now with what is written
            const bool held = N <= block && cb == 0;
            float ue[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) ue[e] = u[c * VEC + e];
            for (int n0 = r0; n0 < N; n0 += block) {
                if (!held) fetch(n0, c);
#pragma unroll
                for (int x = 0; x < MS_HELD; ++x) {
                    const int n = n0 + x * per_pass;
                    if (n >= N) break;
                    float fresh[VEC];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) fresh[e] = fmaf(k[n], ue[e], d[n] * old[x][e]);
                    store(n, fresh);
                }
            }
        }
    }
    // the norm over the head and the gate
    if (a.gate_rank > 0) {
        for (int j = threadIdx.x; j < a.gate_rank; j += MS_THREADS) lora[j] = row[a.gate_at + j];
        __syncthreads();
        low_rank_columns(u, partial, lora, a.gate_rank, a.gate_wt, H * P, head * P, P);
    }
    float squares = 0.0f;
    for (int e = threadIdx.x; e < P; e += MS_THREADS) squares = fmaf(o[e], o[e], squares);
    const float factor = 1.0f / sqrtf(block_sum(squares, scratch) / (float)P + a.eps);
    T* to = out + (size_t)t * out_stride + (size_t)head * P;
    for (int e = threadIdx.x; e < P; e += MS_THREADS) {
        const float z = a.gate_rank > 0 ? u[e] : row[a.gate_at + head * P + e];
        to[e] = from_float<T>(o[e] * factor * a.norm[head * P + e] * (a.gate_silu ? cs_silu(z) : cs_sigmoid(z)));
    }
    if (head == H - 1)                                 // columns that pad the row to whole 16 bytes
        for (int i = H * P + threadIdx.x; i < out_stride; i += MS_THREADS) out[(size_t)t * out_stride + i] = from_float<T>(0.0f);
}

static int cs_reserve(const void* kernel, size_t bytes, const char* name) {
    if (bytes <= 48 * 1024) return 0;
    if (bytes > 220 * 1024) return fail(name, "the sizes are too large for this kernel's shared memory");
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
        return fail(name, "cannot reserve shared memory");
    return 0;
}

static size_t cs_output_smem(int ch, int dim) {
    const int n_pad = (dim + 3) & ~3, ld = n_pad + 4, tail = 2 * ch * ld > 64 * n_pad ? 2 * ch * ld : 64 * n_pad;
    return (size_t)(2 * ch * ld + ch * (ch + 4) + ch * 64 + tail) * sizeof(float);
}

static size_t cs_prepare_smem(int ch, int dim) {
    return (size_t)(3 * ch * (((dim + 3) & ~3) + 4) + 2 * ch * (ch + 4) + ch) * sizeof(float);
}

static size_t cs_walk_smem(int ch, int cols, int dim, bool delta, int stages) {
    const int n_pad = (dim + 3) & ~3, ld = n_pad + 4;
    return (size_t)(n_pad * cols + stages * (ch * ld * (delta ? 2 : 1) + ch * cols + n_pad)) * sizeof(float);
}

// The longest chunk whose tiles fit: 32 tokens or 16.
static int cs_chunk(int dim) {
    return cs_output_smem(32, dim) <= 200 * 1024 && cs_walk_smem(32, 16, dim, true, 2) <= 200 * 1024 ? 32 : 16;
}

static int cs_check(const char* name, const ChannelShape& shape, const ChannelBatch& batch, long long state_floats) {
    if (shape.heads <= 0 || shape.groups <= 0 || shape.heads % shape.groups || shape.dim <= 0 || shape.vdim <= 0)
        return fail(name, "heads must be a positive multiple of the query and key heads, and sizes positive");
    if (shape.heads > 65535) return fail(name, "too many heads");
    const int qk = shape.groups * shape.dim, v = shape.heads * shape.vdim;
    if (shape.q_at < 0 || shape.k_at < 0 || shape.v_at < 0 || shape.q_at + qk > shape.row_stride ||
        shape.k_at + qk > shape.row_stride || shape.v_at + v > shape.row_stride)
        return fail(name, "queries, keys and values must lie inside a row");
    if (!batch.positions || !batch.cu_q || !batch.slot_ids || !batch.state)
        return fail(name, "the step's metadata and the state are needed");
    if (batch.state_offset < 0 || batch.state_offset + state_floats > batch.state_stride)
        return fail(name, "a slot's state is too small");
    return 0;
}

}  // namespace skv

using namespace skv;

// x: float [n, x_stride] (the first `rank` columns count); wt [rank, channels] in the compute dtype; out float [n, channels].
SKV_EXPORT int skv_low_rank(const float* x, int x_stride, int rank, const void* wt, const float* bias, int mode, float factor,
                            const float* rate, int per_rate, float* out, int n, int channels, cudaStream_t stream) {
    const char* name = "skv_low_rank";
    if (n <= 0) return 0;
    if (!x || !wt || !out || rank <= 0 || channels <= 0 || x_stride < rank || mode < 0 || mode > LOW_RANK_SOFTPLUS ||
        (mode == LOW_RANK_SOFTPLUS && (!rate || per_rate <= 0)))
        return fail(name, "sizes do not agree or a pointer is missing");
    const LowRankEnd end = {mode, bias, factor, rate, per_rate};
    const bool many = n >= 256 && (size_t)rank * 16 * sizeof(float) <= 48 * 1024;
    const int tok = many ? 16 : 4;
    const size_t smem = (size_t)rank * tok * sizeof(float);
    if (smem > 48 * 1024) return fail(name, "the rank is too large");
    const int each = many && channels % 2 == 0 && (((uintptr_t)wt | (uintptr_t)out) & 7) == 0 ? 2 : 1;
    auto kernel = each == 2 ? low_rank_kernel<skv_t, 16, 2> : (many ? low_rank_kernel<skv_t, 16, 1> : low_rank_kernel<skv_t, 4, 1>);
    return launch_pdl(name, kernel, dim3((n + tok - 1) / tok, (channels + 256 * each - 1) / (256 * each)), dim3(256), smem, stream, x, x_stride,
                      rank, (const skv_t*)wt, end, out, n, channels);
}

// Floats of scratch for a step: decayed keys [tokens][heads * dim], factors and states per chunk, and for the delta rule W
// [tokens][heads * dim] and U [tokens][heads * vdim].
SKV_EXPORT long long skv_channel_state_scratch(int n_tokens, int n_seqs, int max_q_len, int heads, int dim, int vdim, int delta) {
    const int ch = cs_chunk(dim);
    const long long chunks = (long long)n_seqs * ((max_q_len + ch - 1) / ch), hn = (long long)heads * dim;
    const auto whole = [](long long floats) { return (floats + 3) & ~3LL; };
    return whole(n_tokens * hn) * (delta ? 2 : 1) + whole(chunks * hn) + whole(chunks * hn * vdim) + (delta ? whole((long long)n_tokens * heads * vdim) : 0);
}

// rows: float [n_tokens, row_stride]; log_decay: float [n_tokens, heads * dim]; out: float [n_tokens, heads * vdim].
// beta_rows (null: no delta rule): the logit of (token, head) at beta_rows[token * beta_stride + head].
SKV_EXPORT int skv_channel_state(const float* rows, int row_stride, int q_at, int k_at, int v_at, float q_scale, float unit_eps,
                                 const float* log_decay, const float* beta_rows, int beta_stride, float* out, float* scratch,
                                 int n_tokens, int n_seqs, int heads, int groups, int dim, int vdim, int max_q_len,
                                 const int* positions, const int* token_seq, const int* cu_q, const int* slot_ids,
                                 float* state, long long state_stride, long long state_offset, cudaStream_t stream) {
    const char* name = "skv_channel_state";
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (!rows || !log_decay || !out || !scratch) return fail(name, "rows, decays, scratch and a place for the result are needed");
    if (n_seqs > 65535 || max_q_len <= 0) return fail(name, "too many sequences in one step, or no tokens");
    const bool delta = beta_rows != nullptr;
    if (!delta && unit_eps >= 0.0f) return fail(name, "unit vectors go with the delta rule");
    const ChannelShape shape = {heads, groups, dim, vdim, row_stride, q_at, k_at, v_at, q_scale, unit_eps};
    const ChannelBatch batch = {positions, cu_q, slot_ids, state, state_stride, state_offset};
    if (int code = cs_check(name, shape, batch, 2LL * heads * dim * vdim)) return code;
    if (((uintptr_t)rows | (uintptr_t)out | (uintptr_t)scratch | (uintptr_t)log_decay) & 15) return fail(name, "operands must be 16-byte aligned");
    const int ch = cs_chunk(dim), max_chunks = (max_q_len + ch - 1) / ch;
    const auto whole = [](size_t floats) { return (floats + 3) & ~(size_t)3; };
    const size_t hn = (size_t)heads * dim, chunks = (size_t)n_seqs * max_chunks;
    float* keys = scratch;
    float* factors = keys + whole(n_tokens * hn);
    float* states = factors + whole(chunks * hn);
    float* w_rows = delta ? states + whole(chunks * hn * vdim) : nullptr;
    float* u = delta ? w_rows + whole(n_tokens * hn) : nullptr;
    if (max_chunks > 65535) return fail(name, "too many tokens in one sequence's step");
    const dim3 grid(max_chunks, heads, n_seqs);
    if (delta) {
        const size_t smem = cs_prepare_smem(ch, dim);
        // (one turn of columns: more blocks an SM, with fewer registers; several: fewer)
        auto kernel = ch == 32 ? (dim + vdim <= CS_PREPARE_THREADS ? delta_prepare_kernel<32, 5> : delta_prepare_kernel<32, 3>)
                               : delta_prepare_kernel<16, 3>;
        if (int code = cs_reserve((const void*)kernel, smem, name)) return code;
        if (int code = launch_pdl(name, kernel, grid, dim3(CS_PREPARE_THREADS), smem, stream, rows, log_decay, beta_rows, beta_stride,
                                  keys, factors, w_rows, u, max_chunks, shape, cu_q))
            return code;
    } else {
        auto kernel = ch == 32 ? channel_keys_kernel<32> : channel_keys_kernel<16>;
        if (int code = launch_pdl(name, kernel, dim3((unsigned)((hn + 255) / 256), max_chunks, n_seqs), dim3(256), 0, stream, rows,
                                  log_decay, keys, factors, max_chunks, shape, cu_q))
            return code;
    }
    const float* values = delta ? u : rows + v_at;
    const int value_stride = delta ? heads * vdim : row_stride;
    {
        // slices of 32 value columns where that gives blocks enough, else 16
        const bool wide = 4LL * ((vdim + 31) / 32) * heads * n_seqs >= 3 * sm_count() && cs_walk_smem(ch, 32, dim, delta, 2) <= 200 * 1024;
        const int cols = wide ? 32 : 16;
        // a ring of four where no block has to wait for another's shared memory
        const size_t four = cs_walk_smem(ch, cols, dim, delta, 4);
        const bool alone = (long long)((vdim + cols - 1) / cols) * heads * n_seqs <= sm_count();
        const int stages = max_chunks > 2 && four <= (alone ? 200 : 100) * 1024 ? 4 : 2;
        const size_t smem = cs_walk_smem(ch, cols, dim, delta, stages);
        auto kernel = ch == 32 ? (wide ? (delta ? channel_walk_kernel<32, 32, true> : channel_walk_kernel<32, 32, false>)
                                       : (delta ? channel_walk_kernel<32, 16, true> : channel_walk_kernel<32, 16, false>))
                               : (wide ? (delta ? channel_walk_kernel<16, 32, true> : channel_walk_kernel<16, 32, false>)
                                       : (delta ? channel_walk_kernel<16, 16, true> : channel_walk_kernel<16, 16, false>));
        if (int code = cs_reserve((const void*)kernel, smem, name)) return code;
        if (int code = launch_pdl(name, kernel, dim3((vdim + cols - 1) / cols, heads, n_seqs), dim3(cols * 16), smem, stream,
                                  (const float*)keys, (const float*)factors, (const float*)w_rows, u, values, value_stride, states,
                                  max_chunks, stages, shape, batch))
            return code;
    }
    const size_t smem = cs_output_smem(ch, dim);
    auto kernel = ch == 32 ? channel_output_kernel<32> : channel_output_kernel<16>;
    if (int code = cs_reserve((const void*)kernel, smem, name)) return code;
    return launch_pdl(name, kernel, grid, dim3(CS_OUT_THREADS), smem, stream, rows, log_decay, values, value_stride,
                      (const float*)states, out, max_chunks, shape, cu_q);
}

// One token a sequence (see matrix_step_kernel): rows float [n_seqs, row_stride] of the input projection, out
// [n_seqs, out_stride] in the compute dtype.
SKV_EXPORT int skv_matrix_step(int kind, const float* rows, int row_stride, int q_at, int k_at, int v_at, float q_scale,
                               float unit_eps, const float* conv_w, int taps, long long ring_offset, const void* decay_wt,
                               int decay_at, int decay_rank, const float* decay_bias, int decay_mode, float decay_factor,
                               const float* decay_rate, int beta_at, int input_at, int forget_at, const float* input_bias,
                               const float* forget_bias, float cap, float denominator_eps, int gate_at, int gate_rank,
                               int gate_silu, const void* gate_wt, const float* norm, float eps, void* out, int out_stride,
                               int n_seqs, int heads, int groups, int dim, int vdim, const int* positions, const int* token_seq,
                               const int* cu_q, const int* slot_ids, float* state, long long state_stride,
                               long long state_offset, cudaStream_t stream) {
    const char* name = "skv_matrix_step";
    if (n_seqs <= 0) return 0;
    if (kind < STEP_CHANNEL || kind > STEP_EXP) return fail(name, "unknown kind of memory");
    if (!rows || !norm || !out || n_seqs > 65535 || out_stride < heads * vdim) return fail(name, "a pointer is missing or sizes do not agree");
    const ChannelShape shape = {heads, groups, dim, vdim, row_stride, q_at, k_at, v_at, q_scale, unit_eps};
    const ChannelBatch batch = {positions, cu_q, slot_ids, state, state_stride, state_offset};
    const long long hn = (long long)heads * dim;
    if (int code = cs_check(name, shape, batch, 2 * hn * vdim + (kind == STEP_EXP ? 2 * hn + 2 * heads : 0))) return code;
    MatrixStep a = {};
    a.shape = shape; a.kind = kind;
    a.gate_at = gate_at; a.gate_rank = gate_rank; a.gate_silu = gate_silu; a.gate_wt = (const skv_t*)gate_wt; a.norm = norm; a.eps = eps;
    if (gate_at < 0 || gate_rank < 0 || gate_at + (gate_rank > 0 ? gate_rank : heads * vdim) > row_stride || (gate_rank > 0 && !gate_wt))
        return fail(name, "the gate must lie inside a row");
    if (kind == STEP_EXP) {
        if (!input_bias || !forget_bias || !(cap > 0.0f) || input_at < 0 || forget_at < 0 || input_at + heads > row_stride ||
            forget_at + heads > row_stride || gate_rank > 0)
            return fail(name, "the exponential gates must lie inside a row");
        a.input_at = input_at; a.forget_at = forget_at; a.input_bias = input_bias; a.forget_bias = forget_bias;
        a.cap = cap; a.denominator_eps = denominator_eps;
    } else {
        if (!decay_wt || decay_rank <= 0 || decay_at < 0 || decay_at + decay_rank > row_stride || decay_mode < LOW_RANK_LOG_SIGMOID ||
            decay_mode > LOW_RANK_SOFTPLUS || (decay_mode == LOW_RANK_SOFTPLUS && !decay_rate))
            return fail(name, "the decays' low-rank part must lie inside a row");
        a.decay_wt = (const skv_t*)decay_wt; a.decay_at = decay_at; a.decay_rank = decay_rank;
        a.decay_end = {decay_mode, decay_bias, decay_factor, decay_rate, dim};
    }
    if (kind == STEP_DELTA) {
        const int channels = 2 * groups * dim + heads * vdim;
        if (!conv_w || taps <= 0 || beta_at < 0 || beta_at + heads > row_stride || channels > row_stride || ring_offset < 0 ||
            (taps > 1 && ring_offset + (long long)taps * channels > state_stride))
            return fail(name, "the convolution's channels must lie inside a row and its ring inside a slot's state");
        a.conv_w = conv_w; a.taps = taps; a.channels = channels; a.ring_offset = ring_offset; a.beta_at = beta_at;
    }
    const bool vec = vdim % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0 && ((uintptr_t)state & 15) == 0 &&
                     (kind != STEP_EXP || hn % 4 == 0);
    const int rank = kind == STEP_EXP ? 0 : (decay_rank > gate_rank ? decay_rank : gate_rank);
    const size_t smem = (size_t)ms_smem_floats(dim, vdim, rank, vec ? 4 : 1) * sizeof(float);
    auto kernel = kind == STEP_CHANNEL ? (vec ? matrix_step_kernel<skv_t, 4, STEP_CHANNEL> : matrix_step_kernel<skv_t, 1, STEP_CHANNEL>)
                : kind == STEP_DELTA   ? (vec ? matrix_step_kernel<skv_t, 4, STEP_DELTA> : matrix_step_kernel<skv_t, 1, STEP_DELTA>)
                                       : (vec ? matrix_step_kernel<skv_t, 4, STEP_EXP> : matrix_step_kernel<skv_t, 1, STEP_EXP>);
    if (int code = cs_reserve((const void*)kernel, smem, name)) return code;
    return launch_pdl(name, kernel, dim3(heads, n_seqs), dim3(MS_THREADS), smem, stream, rows, (skv_t*)out, out_stride, a, batch);
}
