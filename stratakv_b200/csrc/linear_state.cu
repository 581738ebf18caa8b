// Linear attention with a matrix state and a decay per head, over packed steps of several sequences: what the mixers of
// the Mamba-2 and Lightning families have in common, with the steps around it that are theirs alone.
//
// A float row holds queries and keys of `groups` heads (dim numbers each) and values of `heads` heads (vdim numbers each);
// value head h uses query and key head h / (heads / groups).  Per head and position p of a sequence
//
//   S_p = exp(l_p) S_(p-1) + c_p k_p v_p^T      (dim x vdim, zero before the first token)
//   o_p = out_scale S_p^T q_p + skip v_p
//
// with l_p <= 0 the logarithm of the decay (one number per head, or one per token and head), c_p a factor on the key
// (or 1) and skip a number per head (or 0).  Queries, keys and values may pass silu as they are read.
//
// With a floor on the denominator (memories with exponential gates) n_p = exp(l_p) n_(p-1) + c_p k_p is kept beside S and
// o_p = out_scale S_p^T q_p / (max(|out_scale n_p . q_p|, floor_p) + floor_eps).
//
// Everything here is float.  Per sequence the cache keeps S twice, one row per slot [2][heads][dim][vdim] (with a floor a
// half is [heads][dim][vdim] and then n, [heads][dim]): a step reads
// the half of the position before its first (by that position's parity) and writes the half of its last, so a one-token
// step that runs twice (a graph's capture after its warm-up) computes the same thing both times.
//
// One token a sequence: one kernel, a block per (head, sequence).  Longer steps: a sequence's tokens are cut into chunks.
// With S the state before a chunk of L tokens, counted 0 .. L-1 within it,
//   o_i    = exp(l_0 + .. + l_i) S^T q_i + sum_(j<=i) exp(l_(j+1) + .. + l_i) c_j (q_i . k_j) v_j
//   S_next = exp(l_0 + .. + l_(L-1)) S + sum_j exp(l_(j+1) + .. + l_(L-1)) c_j k_j v_j^T
// so a first kernel leaves every chunk's own sum (the second term of S_next) and its decay, a second walks the chunks of
// a sequence and replaces each sum by the state before its chunk, and a third makes the outputs of all chunks side by
// side.  The exponents are sums of numbers of one sign, made from the tokens between and never as a difference of two
// running sums: a token that forgets nearly everything does not cost the tokens after it their precision.
#include "common.cuh"

namespace skv {

constexpr int LS_THREADS = 256;

struct LinearStateShape {
    int heads, groups, dim, vdim;
    int row_stride, q_at, k_at, v_at;      // floats per row, and the columns where queries, keys and values start
    int silu;                              // queries, keys and values pass silu as they are read
};

struct LinearStateDecay {
    const float* decay;                    // [heads]: one decay per head, or null
    const float* log_decay;                // [tokens][heads]: one logarithm per token and head (decay null)
    const float* key_scale;                // [tokens][heads] or null
    const float* skip;                     // [heads] or null
    float out_scale;
    const float* floor;                    // [tokens][heads] or null: the outputs are divided (see above)
    float floor_eps;
};

// Floats of one half of the state, and of one chunk's sums: S of all heads, and with a floor n of all heads.
__device__ __forceinline__ size_t ls_half(const LinearStateShape& shape, const LinearStateDecay& decay) {
    return (size_t)shape.heads * shape.dim * (shape.vdim + (decay.floor ? 1 : 0));
}

struct LinearStateBatch {
    const int* positions;                  // [tokens]
    const int* cu_q;                       // [seqs + 1]
    const int* slot_ids;                   // [seqs]
    float* state;                          // [slots][state_stride], S from state_offset on
    long long state_stride, state_offset;
};

__device__ __forceinline__ float ls_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float ls_softplus(float z) { return z > 20.0f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float ls_read(const float* x, int silu) { return silu ? ls_silu(*x) : *x; }
__device__ __forceinline__ float ls_log(float decay) { return decay > 0.0f ? logf(decay) : -INFINITY; }

// ---- one token a sequence ----------------------------------------------------------------------------------------
// What the Mamba-2 mixer does between its input projection and the recurrence, for the new token: a causal convolution
// with bias and silu on the channels [values | keys | queries] (the row's first columns; what lies before the token
// comes from a ring of the last inputs, row position mod taps), and the step size.
struct ConvStep {
    const float* conv_w;                   // [channels][taps], the last column weighs the current token; null: no such step
    const float* conv_b;                   // [channels]
    const float* dt_bias;                  // [heads]
    const float* a_log;                    // [heads]
    int taps, channels, dt_at;             // dt_at: the column of the row where the step sizes start
    long long ring_offset;                 // floats from the start of a slot's row: [taps][channels]
};

__device__ __forceinline__ float conv_one(const float* __restrict__ row, const float* ring, const ConvStep& conv, int p, int c) {
    float sum = conv.conv_b[c];
    for (int j = 0; j < conv.taps; ++j) {
        const int back = conv.taps - 1 - j;
        if (p - back < 0) continue;
        const float u = back == 0 ? row[c] : ring[(size_t)((p - back) % conv.taps) * conv.channels + c];
        sum = fmaf(conv.conv_w[(size_t)c * conv.taps + j], u, sum);
    }
    return ls_silu(sum);
}

// VEC: vdim is a multiple of 4 and a thread takes four neighbouring columns of S; else one column.
template <int VEC>
__global__ void __launch_bounds__(LS_THREADS)
linear_state_step_kernel(const float* __restrict__ rows, float* __restrict__ out, const LinearStateShape shape,
                         const LinearStateDecay decay, const ConvStep conv, const LinearStateBatch batch) {
    extern __shared__ __align__(16) float ls_smem[];
    const int H = shape.heads, N = shape.dim, P = shape.vdim;
    const int n_pad = (N + 3) & ~3;
    float* q = ls_smem;                        // [N]
    float* k = q + n_pad;                      // [N]
    float* v = k + n_pad;                      // [P rounded up]
    float* partial = v + ((P + 3) & ~3);       // [LS_THREADS * VEC]
    __shared__ float head_numbers[2];          // the decay, the skip
    pdl_launch_dependents();
    const int head = blockIdx.x, s = blockIdx.y, g = head / (H / shape.groups);
    const int t = batch.cu_q[s], p = batch.positions[t];
    const float* row = rows + (size_t)t * shape.row_stride;
    float* slot = batch.state + (size_t)batch.slot_ids[s] * batch.state_stride;
    const size_t half_size = (size_t)H * N * P;
    const float* __restrict__ before = slot + batch.state_offset + (size_t)((p - 1) & 1) * half_size + (size_t)head * N * P;
    float* __restrict__ after = slot + batch.state_offset + (size_t)(p & 1) * half_size + (size_t)head * N * P;
    const int columns = P / VEC;                       // threads of a row of S
    const int lanes = min(columns, LS_THREADS), per_pass = LS_THREADS / lanes;
    const int r0 = threadIdx.x / lanes, c0 = threadIdx.x - r0 * lanes;
    constexpr int AHEAD = 8;
    float old[AHEAD][VEC];
    auto fetch = [&](int n0, int c) {                  // this thread's next numbers of the state before the token
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int n = n0 + u * per_pass;
            const bool there = p > 0 && n < N && c < columns && r0 < per_pass;
            if (VEC == 4) {
                const float4 x = there ? *(const float4*)(before + (size_t)n * P + c * 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                old[u][0] = x.x; old[u][1 % VEC] = x.y; old[u][2 % VEC] = x.z; old[u][3 % VEC] = x.w;
            } else {
                old[u][0] = there ? before[(size_t)n * P + c] : 0.0f;
            }
        }
    };
    // The step's metadata came with a copy in front of all its kernels, which also put everything that earlier steps
    // launched behind it; the state before this token was written in an earlier step.  So the first part of it is fetched
    // while the projection in front of this kernel still runs.
    fetch(r0, c0);
    pdl_wait();
    float scale = 1.0f;
    if (conv.conv_w) {
        float* ring = slot + conv.ring_offset;
        const bool first_of_group = head % (H / shape.groups) == 0;
        const float dt = ls_softplus(row[conv.dt_at + head] + conv.dt_bias[head]);
        scale = dt;
        for (int i = threadIdx.x; i < P + 2 * N; i += LS_THREADS) {
            const int c = i < P ? shape.v_at + head * P + i
                                : (i < P + N ? shape.k_at + g * N + i - P : shape.q_at + g * N + i - P - N);
            const float value = conv_one(row, ring, conv, p, c);
            if (i < P) v[i] = value;
            else if (i < P + N) k[i - P] = value * scale;
            else q[i - P - N] = value;
            // (the one row of the ring that no tap of this token reads)
            if (conv.taps > 1 && (i < P || first_of_group)) ring[(size_t)(p % conv.taps) * conv.channels + c] = row[c];
        }
        if (threadIdx.x == 0) head_numbers[0] = expf(-expf(conv.a_log[head]) * dt);
    } else {
        if (decay.key_scale) scale = decay.key_scale[(size_t)t * H + head];
        for (int i = threadIdx.x; i < N; i += LS_THREADS) {
            q[i] = ls_read(row + shape.q_at + g * N + i, shape.silu);
            k[i] = ls_read(row + shape.k_at + g * N + i, shape.silu) * scale;
        }
        for (int i = threadIdx.x; i < P; i += LS_THREADS) v[i] = ls_read(row + shape.v_at + head * P + i, shape.silu);
        if (threadIdx.x == 0) head_numbers[0] = decay.decay ? decay.decay[head] : expf(decay.log_decay[(size_t)t * H + head]);
    }
    if (threadIdx.x == 1) head_numbers[1] = decay.skip ? decay.skip[head] : 0.0f;
    __syncthreads();
    const float a = head_numbers[0];
    for (int cb = 0; cb < columns; cb += lanes) {      // (more than one pass only where a row has more columns than threads)
        const int c = cb + c0;
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = 0.0f;
        if (r0 < per_pass && c < columns) {
            float ve[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) ve[e] = v[c * VEC + e];
            for (int n0 = r0; n0 < N; n0 += per_pass * AHEAD) {
                if (cb > 0 || n0 > r0) fetch(n0, c);
#pragma unroll
                for (int u = 0; u < AHEAD; ++u) {
                    const int n = n0 + u * per_pass;
                    if (n >= N) break;
                    float fresh[VEC];
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        fresh[e] = fmaf(a, old[u][e], k[n] * ve[e]);
                        acc[e] = fmaf(fresh[e], q[n], acc[e]);
                    }
                    if (VEC == 4) *(float4*)(after + (size_t)n * P + c * 4) = make_float4(fresh[0], fresh[1 % VEC], fresh[2 % VEC], fresh[3 % VEC]);
                    else after[(size_t)n * P + c] = fresh[0];
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < VEC; ++e)
            if (r0 < per_pass) partial[(r0 * lanes + c0) * VEC + e] = acc[e];
        __syncthreads();
        for (int i = threadIdx.x; i < lanes * VEC; i += LS_THREADS) {
            const int e = cb * VEC + i;
            if (e >= P) continue;
            float o = 0.0f;
            for (int r = 0; r < per_pass; ++r) o += partial[r * lanes * VEC + i];
            out[((size_t)t * H + head) * P + e] = fmaf(head_numbers[1], v[e], o * decay.out_scale);
        }
    }
}

// Where a thread stands in the 16 x 16 arrangement over a tile: a warp is four rows by eight columns of threads, so that a
// 16-byte load a thread of either operand is one pass over shared memory (64 and 128 different bytes).
__device__ __forceinline__ int tile_x() { return (threadIdx.x & 7) | ((threadIdx.x >> 5 & 1) << 3); }
__device__ __forceinline__ int tile_y() { return (threadIdx.x >> 3 & 3) | ((threadIdx.x >> 6) << 2); }

// ---- longer steps ----------------------------------------------------------------------------------------------
// The exponents of a chunk, in shared memory: l[j] and c[j] of every token, up_to[j] = exp(l_0 + .. + l_j) and
// behind[j] = exp(l_(j+1) + .. + l_(L-1)).  Called by the first warp; a lane holds CH / 32 neighbouring tokens (one token, of
// which half the lanes have none, where a chunk is 16).
template <int CH>
__device__ __forceinline__ void chunk_exponents(float* l, float* c, float* up_to, float* behind, const LinearStateDecay& decay,
                                                int H, int head, int first, int L) {
    constexpr int EACH = CH >= 32 ? CH / 32 : 1;
    const int lane = threadIdx.x & 31;
    const float constant = decay.decay ? ls_log(decay.decay[head]) : 0.0f;
    float mine[EACH], key[EACH], total = 0.0f;
#pragma unroll
    for (int e = 0; e < EACH; ++e) {
        const int j = lane * EACH + e;
        mine[e] = j < L ? (decay.decay ? constant : decay.log_decay[(size_t)(first + j) * H + head]) : 0.0f;
        key[e] = j < L ? (decay.key_scale ? decay.key_scale[(size_t)(first + j) * H + head] : 1.0f) : 0.0f;
        total += mine[e];
    }
    float below = total, above = total;                       // sums over this lane and the lanes on either side of it
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
        const float from_below = __shfl_up_sync(0xffffffffu, below, offset);
        const float from_above = __shfl_down_sync(0xffffffffu, above, offset);
        if (lane >= offset) below += from_below;
        if (lane + offset < 32) above += from_above;
    }
    // (the neighbours' sums alone: never a difference of two sums)
    float before = __shfl_up_sync(0xffffffffu, below, 1), after = __shfl_down_sync(0xffffffffu, above, 1);
    if (lane == 0) before = 0.0f;
    if (lane == 31) after = 0.0f;
    if (lane * EACH >= CH) return;
    float sum = before;
#pragma unroll
    for (int e = 0; e < EACH; ++e) {
        const int j = lane * EACH + e;
        l[j] = mine[e];
        c[j] = key[e];
        sum += mine[e];
        up_to[j] = expf(decay.decay ? (float)(j + 1) * constant : sum);
    }
    sum = after;
#pragma unroll
    for (int e = EACH - 1; e >= 0; --e) {
        const int j = lane * EACH + e;
        behind[j] = j < L - 1 ? expf(decay.decay ? (float)(L - 1 - j) * constant : sum) : 1.0f;
        sum += mine[e];
    }
}

// sums [seqs][max_chunks][heads][dim][vdim], factors [seqs][max_chunks][heads].  Threads in 16 x 16, each with RN rows and
// four columns of S; a tile of 16 RN x 64 at a time.
template <int CH, int RN>
__global__ void __launch_bounds__(LS_THREADS)
linear_state_sum_kernel(const float* __restrict__ rows, float* __restrict__ sums, float* __restrict__ factors, int max_chunks,
                        const LinearStateShape shape, const LinearStateDecay decay, const int* __restrict__ cu_q) {
    extern __shared__ __align__(16) float ls_smem[];
    constexpr int TN = 16 * RN;
    const int H = shape.heads, N = shape.dim, P = shape.vdim;
    float* ks = ls_smem;                                  // [CH][TN], weighed
    float* vs = ks + CH * TN;                             // [CH][64]
    float* l = vs + CH * 64;                              // [CH]
    float* c = l + CH;                                    // [CH]
    float* up_to = c + CH;                                // [CH]
    float* behind = up_to + CH;                           // [CH]
    pdl_launch_dependents();
    pdl_wait();
    const int chunk = blockIdx.x, head = blockIdx.y, s = blockIdx.z, g = head / (H / shape.groups);
    const int first = cu_q[s] + chunk * CH, L = min(CH, cu_q[s + 1] - first);
    if (L <= 0) return;
    if (threadIdx.x < 32) chunk_exponents<CH>(l, c, up_to, behind, decay, H, head, first, L);
    __syncthreads();
    const size_t place = ((size_t)s * max_chunks + chunk) * H + head;
    if (threadIdx.x == 0) factors[place] = up_to[L - 1];
    float* chunk_sums = sums + ((size_t)s * max_chunks + chunk) * ls_half(shape, decay);
    float* mine = chunk_sums + (size_t)head * N * P;
    const int tx = tile_x(), ty = tile_y();
    const bool vec = ((shape.row_stride | shape.k_at | shape.v_at | N | P) & 3) == 0;
    for (int n0 = 0; n0 < N; n0 += TN) {
        if (vec) {
#pragma unroll 4
            for (int idx = threadIdx.x; idx < L * (TN / 4); idx += LS_THREADS) {
                const int j = idx / (TN / 4), n = (idx - j * (TN / 4)) * 4;
                float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (n0 + n < N) {
                    x = *(const float4*)(rows + (size_t)(first + j) * shape.row_stride + shape.k_at + g * N + n0 + n);
                    if (shape.silu) x = make_float4(ls_silu(x.x), ls_silu(x.y), ls_silu(x.z), ls_silu(x.w));
                }
                const float wj = c[j] * behind[j];
                *(float4*)(ks + j * TN + n) = make_float4(x.x * wj, x.y * wj, x.z * wj, x.w * wj);
            }
        } else {
            for (int idx = threadIdx.x; idx < L * TN; idx += LS_THREADS) {
                const int j = idx / TN, n = idx - j * TN;
                ks[idx] = n0 + n < N ? ls_read(rows + (size_t)(first + j) * shape.row_stride + shape.k_at + g * N + n0 + n, shape.silu) * (c[j] * behind[j]) : 0.0f;
            }
        }
        for (int e0 = 0; e0 < P; e0 += 64) {
            if (n0 == 0 || P > 64) {                      // (one tile of values stays for all tiles of keys)
                if (vec) {
                    for (int idx = threadIdx.x; idx < L * 16; idx += LS_THREADS) {
                        const int j = idx >> 4, e = (idx & 15) * 4;
                        float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                        if (e0 + e < P) {
                            x = *(const float4*)(rows + (size_t)(first + j) * shape.row_stride + shape.v_at + head * P + e0 + e);
                            if (shape.silu) x = make_float4(ls_silu(x.x), ls_silu(x.y), ls_silu(x.z), ls_silu(x.w));
                        }
                        *(float4*)(vs + j * 64 + e) = x;
                    }
                } else {
                    for (int idx = threadIdx.x; idx < L * 64; idx += LS_THREADS) {
                        const int j = idx >> 6, e = idx & 63;
                        vs[idx] = e0 + e < P ? ls_read(rows + (size_t)(first + j) * shape.row_stride + shape.v_at + head * P + e0 + e, shape.silu) : 0.0f;
                    }
                }
            }
            __syncthreads();
            if (decay.floor && e0 == 0) {                 // the keys' own sum
                float* key_sums = chunk_sums + (size_t)H * N * P + (size_t)head * N;
                for (int n = threadIdx.x; n < TN && n0 + n < N; n += LS_THREADS) {
                    float sum = 0.0f;
                    for (int j = 0; j < L; ++j) sum += ks[j * TN + n];
                    key_sums[n0 + n] = sum;
                }
            }
            float acc[RN][4];
#pragma unroll
            for (int i = 0; i < RN; ++i)
#pragma unroll
                for (int jj = 0; jj < 4; ++jj) acc[i][jj] = 0.0f;
#pragma unroll 4
            for (int j = 0; j < L; ++j) {
                float kr[RN];
#pragma unroll
                for (int i = 0; i < RN; i += 4) {
                    const float4 x = *(const float4*)(ks + j * TN + (i / 4) * 64 + ty * 4);
                    kr[i] = x.x; kr[i + 1] = x.y; kr[i + 2] = x.z; kr[i + 3] = x.w;
                }
                const float4 ve = *(const float4*)(vs + j * 64 + tx * 4);
#pragma unroll
                for (int i = 0; i < RN; ++i) {
                    acc[i][0] = fmaf(kr[i], ve.x, acc[i][0]); acc[i][1] = fmaf(kr[i], ve.y, acc[i][1]);
                    acc[i][2] = fmaf(kr[i], ve.z, acc[i][2]); acc[i][3] = fmaf(kr[i], ve.w, acc[i][3]);
                }
            }
#pragma unroll
            for (int i = 0; i < RN; ++i) {
                const int n = n0 + (i / 4) * 64 + ty * 4 + (i & 3), e = e0 + tx * 4;
                if (n >= N || e >= P) continue;
                float* to = mine + (size_t)n * P + e;
                if (vec) {
                    *(float4*)to = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
                } else {
#pragma unroll
                    for (int jj = 0; jj < 4; ++jj)
                        if (e + jj < P) to[jj] = acc[i][jj];
                }
            }
            __syncthreads();
        }
    }
}

// Walks a sequence's chunks: every chunk's sum is replaced by the state before the chunk; the state after the last chunk
// goes to the cache.  Several chunks' sums are fetched before any state is stored over them (a store between two loads of
// the same array would make each load wait for the one before).
__global__ void __launch_bounds__(LS_THREADS)
linear_state_carry_kernel(float* __restrict__ sums, const float* __restrict__ factors, int max_chunks, int chunk_len,
                          const LinearStateShape shape, const LinearStateDecay decay, const LinearStateBatch batch) {
    pdl_launch_dependents();
    pdl_wait();
    const int H = shape.heads, cells = shape.dim * shape.vdim;
    const int head = blockIdx.y, s = blockIdx.z;
    const int at = blockIdx.x * LS_THREADS + threadIdx.x;
    if (at >= cells + (decay.floor ? shape.dim : 0)) return;
    const int first = batch.cu_q[s], count = batch.cu_q[s + 1] - first;
    if (count <= 0) return;
    const int p_first = batch.positions[first], p_last = p_first + count - 1;
    const size_t half_size = ls_half(shape, decay);
    const size_t mine = at < cells ? (size_t)head * cells + at : (size_t)H * cells + (size_t)head * shape.dim + (at - cells);
    float* slot = batch.state + (size_t)batch.slot_ids[s] * batch.state_stride + batch.state_offset;
    float S = p_first > 0 ? slot[(size_t)((p_first - 1) & 1) * half_size + mine] : 0.0f;
    const int chunks = (count + chunk_len - 1) / chunk_len;
    float* cell = sums + (size_t)s * max_chunks * half_size + mine;
    const float* factor = factors + (size_t)s * max_chunks * H + head;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float own[AHEAD], f[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            own[i] = c0 + i < chunks ? __ldcg(cell + (size_t)(c0 + i) * half_size) : 0.0f;
            f[i] = c0 + i < chunks ? __ldcg(factor + (size_t)(c0 + i) * H) : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (c0 + i < chunks) {
                cell[(size_t)(c0 + i) * half_size] = S;
                S = fmaf(f[i], S, own[i]);
            }
    }
    slot[(size_t)(p_last & 1) * half_size + mine] = S;
}

// Rows of a chunk, transposed into shared memory: to[n][i] (rows LD apart) = x of token i, number n; zero beyond N and L.
template <int CH, int LD>
__device__ __forceinline__ void load_transposed(float* to, const float* __restrict__ from, int row_stride, int N, int n_pad,
                                                int L, int silu, bool vec) {
    if (vec) {
        // eight tokens by four 16-byte pieces a warp: whole sectors of every row, and two-way bank conflicts at most
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        const int pieces = n_pad >> 2;
        constexpr int ROWS = CH / 8, AHEAD = 4, WARPS = LS_THREADS / 32;
        const int rounds = ROWS * ((pieces + 3) >> 2);
        for (int r0 = warp; r0 < rounds; r0 += AHEAD * WARPS) {        // (several loads on their way before the first store)
            float4 x[AHEAD];
#pragma unroll
            for (int u = 0; u < AHEAD; ++u) {
                const int r = r0 + u * WARPS;
                const int i = (r % ROWS) * 8 + (lane & 7), piece = (r / ROWS) * 4 + (lane >> 3);
                x[u] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (r < rounds && i < L && piece * 4 < N) x[u] = *(const float4*)(from + (size_t)i * row_stride + piece * 4);
            }
#pragma unroll
            for (int u = 0; u < AHEAD; ++u) {
                const int r = r0 + u * WARPS;
                const int i = (r % ROWS) * 8 + (lane & 7), piece = (r / ROWS) * 4 + (lane >> 3);
                if (r >= rounds || piece >= pieces) continue;
                if (silu) x[u] = make_float4(ls_silu(x[u].x), ls_silu(x[u].y), ls_silu(x[u].z), ls_silu(x[u].w));
                float* at = to + piece * 4 * LD + i;
                at[0] = x[u].x; at[LD] = x[u].y; at[2 * LD] = x[u].z; at[3 * LD] = x[u].w;
            }
        }
        return;
    }
    for (int idx = threadIdx.x; idx < CH * n_pad; idx += LS_THREADS) {
        const int i = idx / n_pad, n = idx - i * n_pad;
        to[n * LD + i] = i < L && n < N ? ls_read(from + (size_t)i * row_stride + n, silu) : 0.0f;
    }
}

// The outputs of one chunk of one head; sums holds the state before every chunk (what linear_state_carry_kernel left).
// Threads in 16 x 16, each with CH / 16 tokens and four columns.  n_pad: dim rounded up to a multiple of 4.
template <int CH>
__global__ void __launch_bounds__(LS_THREADS)
linear_state_output_kernel(const float* __restrict__ rows, const float* __restrict__ sums, float* __restrict__ out,
                           int max_chunks, int n_pad, const LinearStateShape shape, const LinearStateDecay decay,
                           const int* __restrict__ cu_q) {
    extern __shared__ __align__(16) float ls_smem[];
    constexpr int LD = CH + 4, RI = CH / 16;              // a thread's tokens, and its keys in the scores
    const int H = shape.heads, N = shape.dim, P = shape.vdim;
    float* qT = ls_smem;                                  // [n_pad][LD]
    float* kT = qT + n_pad * LD;                          // [n_pad][LD]; then the state's tile [n_pad][64]
    float* wT = kT + n_pad * (LD > 64 ? LD : 64);         // [CH][LD]: the scores, indexed [key][query]
    float* vs = wT + CH * LD;                             // [CH][64]
    float* l = vs + CH * 64;                              // [CH]
    float* c = l + CH;                                    // [CH]
    float* up_to = c + CH;                                // [CH]
    float* behind = up_to + CH;                           // [CH]
    float* spans = behind + CH;                           // [16]: the sum of l over a thread's tokens, for every row of threads
    float* factor = spans + 16;                           // [CH]: what a token's output is multiplied by
    pdl_launch_dependents();
    pdl_wait();
    const int chunk = blockIdx.x, head = blockIdx.y, s = blockIdx.z, g = head / (H / shape.groups);
    const int first = cu_q[s] + chunk * CH, L = min(CH, cu_q[s + 1] - first);
    if (L <= 0) return;
    const bool vec_qk = ((shape.row_stride | shape.q_at | shape.k_at | N) & 3) == 0;
    const bool vec_v = ((shape.row_stride | shape.v_at | P) & 3) == 0 && (!decay.floor || ((H * N) & 3) == 0);
    const float* base = rows + (size_t)first * shape.row_stride;
    if (threadIdx.x < 32) {
        chunk_exponents<CH>(l, c, up_to, behind, decay, H, head, first, L);
        __syncwarp();
        if (threadIdx.x < 16) {
            float sum = 0.0f;
#pragma unroll
            for (int x = 0; x < RI; ++x) sum += l[threadIdx.x * RI + x];
            spans[threadIdx.x] = sum;
        }
    }
    load_transposed<CH, LD>(qT, base + shape.q_at + g * N, shape.row_stride, N, n_pad, L, shape.silu, vec_qk);
    load_transposed<CH, LD>(kT, base + shape.k_at + g * N, shape.row_stride, N, n_pad, L, shape.silu, vec_qk);
    __syncthreads();
    const bool constant = decay.decay != nullptr;
    const int tx = tile_x(), ty = tile_y();
    const int i0 = ty * RI, j0 = tx * RI;
    {
        float acc[RI][RI];
#pragma unroll
        for (int a = 0; a < RI; ++a)
#pragma unroll
            for (int b = 0; b < RI; ++b) acc[a][b] = 0.0f;
        if (j0 <= i0) {
#pragma unroll 4
            for (int n = 0; n < n_pad; ++n) {
                float qi[RI], kj[RI];
                if (RI == 4) {
                    const float4 a = *(const float4*)(qT + n * LD + i0), b = *(const float4*)(kT + n * LD + j0);
                    qi[0] = a.x; qi[1 % RI] = a.y; qi[2 % RI] = a.z; qi[3 % RI] = a.w;
                    kj[0] = b.x; kj[1 % RI] = b.y; kj[2 % RI] = b.z; kj[3 % RI] = b.w;
                } else {
#pragma unroll
                    for (int a = 0; a < RI; ++a) { qi[a] = qT[n * LD + i0 + a]; kj[a] = kT[n * LD + j0 + a]; }
                }
#pragma unroll
                for (int a = 0; a < RI; ++a)
#pragma unroll
                    for (int b = 0; b < RI; ++b) acc[a][b] = fmaf(qi[a], kj[b], acc[a][b]);
            }
        }
        // the exponents between: what lies between the two tiles, then the tokens inside either
        float between = 0.0f;
        if (!constant && j0 < i0) {
            for (int x = tx + 1; x < ty; ++x) between += spans[x];
            between += l[i0];
        }
#pragma unroll
        for (int b = 0; b < RI; ++b) {
            const int j = j0 + b;
            float sum = between;
            if (j0 < i0) {
#pragma unroll
                for (int x = RI - 1; x > 0; --x)
                    if (x > b) sum += l[j0 + x];
            }
#pragma unroll
            for (int a = 0; a < RI; ++a) {
                const int i = i0 + a;
                float weight = 0.0f;
                if (j <= i && i < L) {
                    float exponent;
                    if (constant) {
                        exponent = i == j ? 0.0f : (float)(i - j) * l[0];
                    } else if (j0 < i0) {
                        if (a > 0) sum += l[i];
                        exponent = sum;
                    } else {
                        exponent = 0.0f;
                        for (int x = j + 1; x <= i; ++x) exponent += l[x];
                    }
                    weight = acc[a][b] * expf(exponent) * c[j];
                }
                wT[j * LD + i] = weight;
            }
        }
    }
    float carry[RI];
#pragma unroll
    for (int a = 0; a < RI; ++a) carry[a] = i0 + a < L ? up_to[i0 + a] : 0.0f;
    const float skip = decay.skip ? decay.skip[head] : 0.0f;
    const float* chunk_before = sums + ((size_t)s * max_chunks + chunk) * ls_half(shape, decay);
    const float* before = chunk_before + (size_t)head * N * P;
    if (decay.floor) {
        __syncthreads();                                  // (the scores are in place)
        if (threadIdx.x < 4 * CH) {
            const float* n_before = chunk_before + (size_t)H * N * P + (size_t)head * N;
            const int i = threadIdx.x >> 2, part = threadIdx.x & 3;
            float dot = 0.0f, own = 0.0f;
            for (int n = part; n < N; n += 4) dot = fmaf(qT[n * LD + i], n_before[n], dot);
            for (int j = part; j <= i; j += 4) own += wT[j * LD + i];
            dot = i < L ? fmaf(dot, up_to[i], own) : 0.0f;
            dot += __shfl_xor_sync(0xffffffffu, dot, 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 2);
            if (part == 0)
                factor[i] = i < L ? decay.out_scale / (fmaxf(fabsf(dot * decay.out_scale), decay.floor[(size_t)(first + i) * H + head]) + decay.floor_eps) : 0.0f;
        }
    } else if (threadIdx.x < CH) {
        factor[threadIdx.x] = decay.out_scale;
    }
    float* st = kT;
    const int j_end = min(L, ((ty | 3) + 1) * RI);        // (the four rows of threads of a warp walk the same keys)
    for (int e0 = 0; e0 < P; e0 += 64) {
        __syncthreads();                                  // the scores are in place; the tiles before have been read
        if (vec_v) {
#pragma unroll
            for (int idx = threadIdx.x; idx < CH * 16; idx += LS_THREADS) {
                const int j = idx >> 4, e = (idx & 15) * 4;
                float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (j < L && e0 + e < P) {
                    x = *(const float4*)(base + (size_t)j * shape.row_stride + shape.v_at + head * P + e0 + e);
                    if (shape.silu) x = make_float4(ls_silu(x.x), ls_silu(x.y), ls_silu(x.z), ls_silu(x.w));
                }
                *(float4*)(vs + j * 64 + e) = x;
            }
#pragma unroll 8
            for (int idx = threadIdx.x; idx < N * 16; idx += LS_THREADS) {
                const int n = idx >> 4, e = (idx & 15) * 4;
                *(float4*)(st + n * 64 + e) = e0 + e < P ? *(const float4*)(before + (size_t)n * P + e0 + e) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        } else {
            for (int idx = threadIdx.x; idx < CH * 64; idx += LS_THREADS) {
                const int j = idx >> 6, e = idx & 63;
                vs[idx] = j < L && e0 + e < P ? ls_read(base + (size_t)j * shape.row_stride + shape.v_at + head * P + e0 + e, shape.silu) : 0.0f;
            }
            for (int idx = threadIdx.x; idx < N * 64; idx += LS_THREADS) {
                const int n = idx >> 6, e = idx & 63;
                st[idx] = e0 + e < P ? before[(size_t)n * P + e0 + e] : 0.0f;
            }
        }
        __syncthreads();
        float acc[RI][4];
#pragma unroll
        for (int a = 0; a < RI; ++a)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[a][e] = 0.0f;
#pragma unroll 4
        for (int n = 0; n < N; ++n) {                     // what the state before the chunk gives
            const float4 sv = *(const float4*)(st + n * 64 + tx * 4);
            float qi[RI];
            if (RI == 4) {
                const float4 a = *(const float4*)(qT + n * LD + i0);
                qi[0] = a.x; qi[1 % RI] = a.y; qi[2 % RI] = a.z; qi[3 % RI] = a.w;
            } else {
#pragma unroll
                for (int a = 0; a < RI; ++a) qi[a] = qT[n * LD + i0 + a];
            }
#pragma unroll
            for (int a = 0; a < RI; ++a) {
                acc[a][0] = fmaf(qi[a], sv.x, acc[a][0]); acc[a][1] = fmaf(qi[a], sv.y, acc[a][1]);
                acc[a][2] = fmaf(qi[a], sv.z, acc[a][2]); acc[a][3] = fmaf(qi[a], sv.w, acc[a][3]);
            }
        }
#pragma unroll
        for (int a = 0; a < RI; ++a)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[a][e] *= carry[a];
#pragma unroll 4
        for (int j = 0; j < j_end; ++j) {                 // what the chunk's own tokens give
            const float4 ve = *(const float4*)(vs + j * 64 + tx * 4);
            float wi[RI];
            if (RI == 4) {
                const float4 a = *(const float4*)(wT + j * LD + i0);
                wi[0] = a.x; wi[1 % RI] = a.y; wi[2 % RI] = a.z; wi[3 % RI] = a.w;
            } else {
#pragma unroll
                for (int a = 0; a < RI; ++a) wi[a] = wT[j * LD + i0 + a];
            }
#pragma unroll
            for (int a = 0; a < RI; ++a) {
                acc[a][0] = fmaf(wi[a], ve.x, acc[a][0]); acc[a][1] = fmaf(wi[a], ve.y, acc[a][1]);
                acc[a][2] = fmaf(wi[a], ve.z, acc[a][2]); acc[a][3] = fmaf(wi[a], ve.w, acc[a][3]);
            }
        }
        const int e = e0 + tx * 4;
#pragma unroll
        for (int a = 0; a < RI; ++a) {
            const int i = i0 + a;
            if (i >= L || e >= P) continue;
            const float4 own = *(const float4*)(vs + i * 64 + tx * 4);
            const float f = factor[i];
            const float o[4] = {fmaf(skip, own.x, acc[a][0] * f), fmaf(skip, own.y, acc[a][1] * f), fmaf(skip, own.z, acc[a][2] * f),
                                fmaf(skip, own.w, acc[a][3] * f)};
            float* to = out + ((size_t)(first + i) * H + head) * P + e;
            if ((P & 3) == 0) {
                *(float4*)to = make_float4(o[0], o[1], o[2], o[3]);
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (e + x < P) to[x] = o[x];
            }
        }
    }
}

// ---- Mamba-2's steps between its input projection and the recurrence, for steps of more than one token a sequence --------
// A thread takes one channel of CONV_TOKENS neighbouring tokens and keeps the last inputs in registers (up to 8 taps).
constexpr int CONV_TOKENS = 16, CONV_HELD = 8;

__global__ void __launch_bounds__(256)
conv_silu_kernel(const float* __restrict__ rows, int row_stride, const float* __restrict__ conv_w,
                 const float* __restrict__ conv_b, int channels, int taps, float* __restrict__ out, int n_tokens,
                 const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                 const int* __restrict__ slot_ids, const float* __restrict__ state, long long state_stride,
                 long long ring_offset) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int t0 = blockIdx.y * CONV_TOKENS, t1 = min(n_tokens, t0 + CONV_TOKENS);
    const float bias = conv_b ? conv_b[c] : 0.0f;
    const float* weights = conv_w + (size_t)c * taps;
    const bool held = taps <= CONV_HELD;
    float w[CONV_HELD], u[CONV_HELD];                     // w[b], u[b]: the weight and the input of the token b back
#pragma unroll
    for (int b = 0; b < CONV_HELD; ++b) { w[b] = held && b < taps ? weights[taps - 1 - b] : 0.0f; u[b] = 0.0f; }
    if (held && token_seq[t0] == token_seq[t1 - 1]) {
        // all tokens of one sequence: every input is fetched before the first is used
        const int s = token_seq[t0], p = positions[t0], first = cu_q[s];
        const float* ring = state + (size_t)slot_ids[s] * state_stride + ring_offset;
        float x[CONV_TOKENS];
#pragma unroll
        for (int i = 0; i < CONV_TOKENS; ++i) x[i] = t0 + i < t1 ? rows[(size_t)(t0 + i) * row_stride + c] : 0.0f;
#pragma unroll
        for (int b = 1; b < CONV_HELD; ++b)               // u[b]: the input b tokens before this block's first
            if (b < taps && p - b >= 0)
                u[b] = t0 - b >= first ? rows[(size_t)(t0 - b) * row_stride + c] : ring[(size_t)((p - b) % taps) * channels + c];
#pragma unroll
        for (int i = 0; i < CONV_TOKENS; ++i) {
            float sum = bias;
#pragma unroll
            for (int b = CONV_HELD - 1; b >= 0; --b) sum = fmaf(w[b], i >= b ? x[i >= b ? i - b : 0] : u[i < b ? b - i : 0], sum);
            if (t0 + i < t1) out[(size_t)(t0 + i) * channels + c] = ls_silu(sum);
        }
        return;
    }
    int seq = -1;
    for (int t = t0; t < t1; ++t) {
        const int s = token_seq[t], p = positions[t];
        float sum = bias;
        if (held) {
            if (s != seq) {                               // this block's first token of a sequence: fetch what lies before it
                seq = s;
                const int first = cu_q[s];
                const float* ring = state + (size_t)slot_ids[s] * state_stride + ring_offset;
#pragma unroll
                for (int b = 1; b < CONV_HELD; ++b) {
                    float x = 0.0f;
                    if (b < taps && p - b >= 0)
                        x = t - b >= first ? rows[(size_t)(t - b) * row_stride + c] : ring[(size_t)((p - b) % taps) * channels + c];
                    u[b] = x;
                }
            }
            u[0] = rows[(size_t)t * row_stride + c];
#pragma unroll
            for (int b = CONV_HELD - 1; b >= 0; --b) sum = fmaf(w[b], u[b], sum);
#pragma unroll
            for (int b = CONV_HELD - 1; b > 0; --b) u[b] = u[b - 1];
        } else {
            const int first = cu_q[s];
            const float* ring = state + (size_t)slot_ids[s] * state_stride + ring_offset;
            for (int j = 0; j < taps; ++j) {
                const int back = taps - 1 - j;
                if (p - back < 0) continue;
                const float x = t - back >= first ? rows[(size_t)(t - back) * row_stride + c] : ring[(size_t)((p - back) % taps) * channels + c];
                sum = fmaf(weights[j], x, sum);
            }
        }
        out[(size_t)t * channels + c] = ls_silu(sum);
    }
}

// dt[t][h] = softplus(row's step size + dt_bias[h]), log_decay[t][h] = -exp(a_log[h]) dt[t][h].
__global__ void __launch_bounds__(256)
step_sizes_kernel(const float* __restrict__ rows, int row_stride, int dt_at, const float* __restrict__ dt_bias,
                  const float* __restrict__ a_log, int heads, int n_tokens, float* __restrict__ dt, float* __restrict__ log_decay) {
    pdl_launch_dependents();
    pdl_wait();
    const long long item = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (item >= (long long)n_tokens * heads) return;
    const int t = (int)(item / heads), h = (int)(item - (long long)t * heads);
    const float step = ls_softplus(rows[(size_t)t * row_stride + dt_at + h] + dt_bias[h]);
    dt[item] = step;
    log_decay[item] = -expf(a_log[h]) * step;
}

// ---- exponential gates with a running maximum ---------------------------------------------------------------------------
// i = cap tanh((row + b) / cap), f = log sigmoid(cap tanh((row + b) / cap)), m_t = max(f_t + m_(t-1), i_t) with m = 0 before
// the first token; then log_decay = f_t + m_(t-1) - m_t, key_scale = exp(i_t - m_t) and floor = exp(-m_t), each
// [tokens][heads]: what linear_state reads.  The state of a slot holds m twice, [2][heads] from m_offset on, by the parity of
// the last position.  A block per (head, sequence); a thread takes EG_EACH neighbouring tokens.  A run of tokens turns m into
// max(F + m, M) with F the sum of its f, and two runs behind one another make another such pair, which the block scans.
constexpr int EG_EACH = 4, EG_THREADS = 512;

struct GateRun { float F, M; };
__device__ __forceinline__ GateRun behind_run(GateRun a, GateRun b) { return {a.F + b.F, fmaxf(b.F + a.M, b.M)}; }

__global__ void __launch_bounds__(EG_THREADS)
exp_gates_kernel(const float* __restrict__ rows, int row_stride, int input_at, int forget_at, const float* __restrict__ input_bias,
                 const float* __restrict__ forget_bias, float cap, float* __restrict__ log_decay, float* __restrict__ key_scale,
                 float* __restrict__ floor, int heads, const LinearStateBatch batch) {
    __shared__ GateRun warp_runs[EG_THREADS / 32];
    __shared__ float carried;
    pdl_launch_dependents();
    pdl_wait();
    const int head = blockIdx.x, s = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int first = batch.cu_q[s], count = batch.cu_q[s + 1] - first;
    if (count <= 0) return;
    const int p_first = batch.positions[first], p_last = p_first + count - 1;
    float* maxima = batch.state + (size_t)batch.slot_ids[s] * batch.state_stride + batch.state_offset + head;      // (m_offset)
    if (threadIdx.x == 0) carried = p_first > 0 ? maxima[(size_t)((p_first - 1) & 1) * heads] : 0.0f;
    const float bi = input_bias[head], bf = forget_bias[head];
    for (int t0 = 0; t0 < count; t0 += EG_THREADS * EG_EACH) {
        float i[EG_EACH], f[EG_EACH];
        const int mine = t0 + threadIdx.x * EG_EACH;
        GateRun run = {0.0f, -INFINITY};
#pragma unroll
        for (int e = 0; e < EG_EACH; ++e) {
            i[e] = -INFINITY;
            f[e] = 0.0f;
            if (mine + e < count) {
                const float* row = rows + (size_t)(first + mine + e) * row_stride;
                i[e] = cap * tanhf((row[input_at + head] + bi) / cap);
                const float z = cap * tanhf((row[forget_at + head] + bf) / cap);
                f[e] = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
            }
        }
#pragma unroll
        for (int e = 0; e < EG_EACH; ++e) run = behind_run(run, {f[e], i[e]});
        // the runs of the lanes below, then of the warps below
        GateRun upto = run;
#pragma unroll
        for (int offset = 1; offset < 32; offset <<= 1) {
            const GateRun below = {__shfl_up_sync(0xffffffffu, upto.F, offset), __shfl_up_sync(0xffffffffu, upto.M, offset)};
            if (lane >= offset) upto = behind_run(below, upto);
        }
        if (lane == 31) warp_runs[warp] = upto;
        GateRun before = {__shfl_up_sync(0xffffffffu, upto.F, 1), __shfl_up_sync(0xffffffffu, upto.M, 1)};
        if (lane == 0) before = {0.0f, -INFINITY};
        __syncthreads();
        GateRun lower = {0.0f, -INFINITY};
        for (int x = 0; x < warp; ++x) lower = behind_run(lower, warp_runs[x]);
        before = behind_run(lower, before);
        float m = fmaxf(before.F + carried, before.M);
        __syncthreads();                                  // (everybody has read what was carried)
#pragma unroll
        for (int e = 0; e < EG_EACH; ++e) {
            if (mine + e >= count) break;
            const float top = fmaxf(f[e] + m, i[e]);
            const size_t at = (size_t)(first + mine + e) * heads + head;
            log_decay[at] = f[e] + m - top;
            key_scale[at] = expf(i[e] - top);
            floor[at] = expf(-top);
            m = top;
            if (mine + e == min(count, t0 + EG_THREADS * EG_EACH) - 1) {       // the last token of this round
                carried = m;
                if (mine + e == count - 1) maxima[(size_t)(p_last & 1) * heads] = m;
            }
        }
        __syncthreads();
    }
}

// ---- a norm with a gate ------------------------------------------------------------------------------------------------
enum { GATE_SIGMOID = 0, GATE_SILU_FIRST = 1, GATE_SILU = 2 };
__device__ __forceinline__ float gate_after(float z, int mode) { return (mode == GATE_SILU ? z : 1.0f) / (1.0f + expf(-z)); }

// out = gated norm of float rows y [tokens, width]: the row in `groups` equal parts, each divided by its own root mean
// square, times a weight, and a gate on every number: sigmoid(gate) or silu(gate) after the norm, or silu(gate) before it.
// A block per (token, part); the part stays in shared memory between the two passes.
template <typename T>
__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ y, const float* __restrict__ gate, int gate_stride, const float* __restrict__ weight,
                  int width, int groups, float eps, int mode, T* __restrict__ out, int out_stride) {
    extern __shared__ __align__(16) float gn_part[];
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, part = blockIdx.y, size = width / groups, at = part * size;
    const float* row = y + (size_t)t * width + at;
    const float* g = gate + (size_t)t * gate_stride + at;
    T* to = out + (size_t)t * out_stride + at;
    const float* w = weight + at;
    float squares = 0.0f;
    const bool vec = ((size | width | gate_stride | out_stride) & 3) == 0 &&
                     (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)weight | (uintptr_t)out) & 15) == 0;
    if (vec) {
        for (int i = 4 * threadIdx.x; i < size; i += 1024) {
            float4 v = *(const float4*)(row + i);
            if (mode == GATE_SILU_FIRST) {
                const float4 z = *(const float4*)(g + i);
                v.x *= ls_silu(z.x); v.y *= ls_silu(z.y); v.z *= ls_silu(z.z); v.w *= ls_silu(z.w);
            }
            squares = fmaf(v.x, v.x, squares); squares = fmaf(v.y, v.y, squares);
            squares = fmaf(v.z, v.z, squares); squares = fmaf(v.w, v.w, squares);
            *(float4*)(gn_part + i) = v;
        }
    } else {
        for (int i = threadIdx.x; i < size; i += 256) {
            float v = row[i];
            if (mode == GATE_SILU_FIRST) v *= ls_silu(g[i]);
            squares = fmaf(v, v, squares);
            gn_part[i] = v;
        }
    }
    const float factor = 1.0f / sqrtf(block_sum(squares, scratch) / (float)size + eps);
    if (vec) {
        for (int i = 4 * threadIdx.x; i < size; i += 1024) {
            float4 v = *(const float4*)(gn_part + i);
            const float4 x = *(const float4*)(w + i);
            v.x *= factor * x.x; v.y *= factor * x.y; v.z *= factor * x.z; v.w *= factor * x.w;
            if (mode != GATE_SILU_FIRST) {
                const float4 z = *(const float4*)(g + i);
                v.x *= gate_after(z.x, mode); v.y *= gate_after(z.y, mode); v.z *= gate_after(z.z, mode); v.w *= gate_after(z.w, mode);
            }
            if (sizeof(T) == 4) {
                *(float4*)(to + i) = v;
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
                *(uint2*)(to + i) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += 256) {
            float v = gn_part[i] * factor * w[i];
            if (mode != GATE_SILU_FIRST) v *= gate_after(g[i], mode);
            to[i] = from_float<T>(v);
        }
    }
    if (part == groups - 1)
        for (int i = width + threadIdx.x; i < out_stride; i += 256) out[(size_t)t * out_stride + i] = from_float<T>(0.0f);
}

// The same with a warp per (token, part) for parts of at most 128 HELD numbers (a multiple of 4) in steps of many tokens.
template <typename T, int HELD>
__global__ void __launch_bounds__(256)
gated_norm_parts_kernel(const float* __restrict__ y, const float* __restrict__ gate, int gate_stride,
                        const float* __restrict__ weight, int width, int groups, float eps, int mode,
                        T* __restrict__ out, int out_stride, int items) {
    pdl_launch_dependents();
    pdl_wait();
    const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= items) return;
    const int t = item / groups, part = item - t * groups, size = width / groups, at = part * size;
    const float* row = y + (size_t)t * width + at;
    const float* g = gate + (size_t)t * gate_stride + at;
    const float* w = weight + at;
    T* to = out + (size_t)t * out_stride + at;
    float4 v[HELD], z[HELD];
#pragma unroll
    for (int j = 0; j < HELD; ++j) {
        const int i = 4 * (lane + 32 * j);
        v[j] = z[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i < size) { v[j] = *(const float4*)(row + i); z[j] = *(const float4*)(g + i); }
    }
    float squares = 0.0f;
#pragma unroll
    for (int j = 0; j < HELD; ++j) {
        if (mode == GATE_SILU_FIRST) { v[j].x *= ls_silu(z[j].x); v[j].y *= ls_silu(z[j].y); v[j].z *= ls_silu(z[j].z); v[j].w *= ls_silu(z[j].w); }
        squares += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float factor = 1.0f / sqrtf(warp_sum(squares) / (float)size + eps);
#pragma unroll
    for (int j = 0; j < HELD; ++j) {
        const int i = 4 * (lane + 32 * j);
        if (i >= size) continue;
        const float4 x = *(const float4*)(w + i);
        float4 r = make_float4(v[j].x * factor * x.x, v[j].y * factor * x.y, v[j].z * factor * x.z, v[j].w * factor * x.w);
        if (mode != GATE_SILU_FIRST) {
            r.x *= gate_after(z[j].x, mode); r.y *= gate_after(z[j].y, mode); r.z *= gate_after(z[j].z, mode); r.w *= gate_after(z[j].w, mode);
        }
        if (sizeof(T) == 4) {
            *(float4*)(to + i) = r;
        } else {
            const __nv_bfloat162 lo = __floats2bfloat162_rn(r.x, r.y), hi = __floats2bfloat162_rn(r.z, r.w);
            *(uint2*)(to + i) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
        }
    }
    if (part == groups - 1)
        for (int i = width + lane; i < out_stride; i += 32) out[(size_t)t * out_stride + i] = from_float<T>(0.0f);
}

static int ls_reserve(const void* kernel, size_t bytes, const char* name) {
    if (bytes <= 48 * 1024) return 0;
    if (bytes > 220 * 1024) return fail(name, "the sizes are too large for this kernel's shared memory");
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess)
        return fail(name, "cannot reserve shared memory");
    return 0;
}

static size_t ls_output_smem(int ch, int dim) {
    const int n_pad = (dim + 3) & ~3, ld = ch + 4;
    return (size_t)(n_pad * ld + n_pad * (ld > 64 ? ld : 64) + ch * ld + ch * 64 + 5 * ch + 16) * sizeof(float);
}

// The longest chunk whose tiles fit: 64 tokens, 32, or 16.
static int ls_chunk(int dim) {
    return ls_output_smem(64, dim) <= 200 * 1024 ? 64 : (ls_output_smem(32, dim) <= 200 * 1024 ? 32 : 16);
}

static int ls_check(const char* name, const LinearStateShape& shape, const LinearStateBatch& batch, bool with_floor) {
    if (shape.heads <= 0 || shape.groups <= 0 || shape.heads % shape.groups || shape.dim <= 0 || shape.vdim <= 0)
        return fail(name, "heads must be a positive multiple of the query and key heads, and sizes positive");
    if (shape.heads > 65535) return fail(name, "too many heads");
    const int qk = shape.groups * shape.dim, v = shape.heads * shape.vdim;
    if (shape.q_at < 0 || shape.k_at < 0 || shape.v_at < 0 || shape.q_at + qk > shape.row_stride ||
        shape.k_at + qk > shape.row_stride || shape.v_at + v > shape.row_stride)
        return fail(name, "queries, keys and values must lie inside a row");
    if (!batch.positions || !batch.cu_q || !batch.slot_ids || !batch.state)
        return fail(name, "the step's metadata and the state are needed");
    if (batch.state_offset < 0 || batch.state_offset + 2LL * shape.heads * shape.dim * (shape.vdim + (with_floor ? 1 : 0)) > batch.state_stride)
        return fail(name, "a slot's state is too small: two halves of heads * dim * vdim floats (and heads * dim with a floor) are needed");
    return 0;
}

}  // namespace skv

using namespace skv;

// Floats of scratch for a step whose longest sequence brings max_q_len tokens (0 for one token a sequence).
SKV_EXPORT long long skv_linear_state_scratch(int n_seqs, int max_q_len, int heads, int dim, int vdim, int with_floor) {
    if (max_q_len <= 1 && !with_floor) return 0;
    const int ch = ls_chunk(dim);
    return (long long)n_seqs * ((max_q_len + ch - 1) / ch) * heads * ((long long)dim * (vdim + (with_floor ? 1 : 0)) + 1);
}

// rows: float [n_tokens, row_stride]; out: float [n_tokens, heads * vdim].  decay [heads], or log_decay [n_tokens, heads];
// key_scale [n_tokens, heads] and skip [heads] may be null.  state: float [slots][state_stride].
SKV_EXPORT int skv_linear_state(const float* rows, int row_stride, int q_at, int k_at, int v_at, int silu, const float* decay,
                                const float* log_decay, const float* key_scale, const float* skip, float out_scale,
                                const float* floor, float floor_eps, float* out, float* scratch, int n_tokens, int n_seqs, int heads, int groups, int dim, int vdim,
                                int max_q_len, const int* positions, const int* token_seq, const int* cu_q,
                                const int* slot_ids, float* state, long long state_stride, long long state_offset,
                                cudaStream_t stream) {
    const char* name = "skv_linear_state";
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (!rows || !out || (!decay && !log_decay)) return fail(name, "rows, a decay and a place for the result are needed");
    if (n_seqs > 65535 || max_q_len <= 0) return fail(name, "too many sequences in one step, or no tokens");
    const LinearStateShape shape = {heads, groups, dim, vdim, row_stride, q_at, k_at, v_at, silu};
    const LinearStateDecay decays = {decay, log_decay, key_scale, skip, out_scale, floor, floor_eps};
    const LinearStateBatch batch = {positions, cu_q, slot_ids, state, state_stride, state_offset};
    if (int code = ls_check(name, shape, batch, floor != nullptr)) return code;
    if (((uintptr_t)rows | (uintptr_t)out | (uintptr_t)state | (uintptr_t)scratch) & 15) return fail(name, "operands must be 16-byte aligned");
    if (max_q_len == 1 && !floor) {
        if (n_tokens != n_seqs) return fail(name, "one token a sequence means as many tokens as sequences");
        ConvStep none = {};
        const bool vec = vdim % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0;
        const size_t smem = (size_t)(2 * ((dim + 3) & ~3) + ((vdim + 3) & ~3) + LS_THREADS * (vec ? 4 : 1)) * sizeof(float);
        auto kernel = vec ? linear_state_step_kernel<4> : linear_state_step_kernel<1>;
        if (int code = ls_reserve((const void*)kernel, smem, name)) return code;
        return launch_pdl(name, kernel, dim3(heads, n_seqs), dim3(LS_THREADS), smem, stream, rows, out, shape, decays, none, batch);
    }
    if (!scratch) return fail(name, "a step of more than one token a sequence needs scratch for its chunks");
    const int ch = ls_chunk(dim), max_chunks = (max_q_len + ch - 1) / ch;
    if (ls_output_smem(ch, dim) > 220 * 1024) return fail(name, "the head size is too large for this kernel's shared memory");
    float* sums = scratch;
    const int per_key = vdim + (floor ? 1 : 0);           // numbers a key channel keeps
    float* factors = scratch + (size_t)n_seqs * max_chunks * heads * dim * per_key;
    const bool wide = dim > 64;
    const dim3 grid(max_chunks, heads, n_seqs);
    {
        const size_t smem = (size_t)(ch * (wide ? 128 : 64) + ch * 64 + 4 * ch) * sizeof(float);
        auto kernel = ch == 64 ? (wide ? linear_state_sum_kernel<64, 8> : linear_state_sum_kernel<64, 4>)
                     : ch == 32 ? (wide ? linear_state_sum_kernel<32, 8> : linear_state_sum_kernel<32, 4>)
                                : (wide ? linear_state_sum_kernel<16, 8> : linear_state_sum_kernel<16, 4>);
        if (int code = ls_reserve((const void*)kernel, smem, name)) return code;
        if (int code = launch_pdl(name, kernel, grid, dim3(LS_THREADS), smem, stream, rows, sums, factors, max_chunks, shape, decays, cu_q))
            return code;
    }
    if (int code = launch_pdl(name, linear_state_carry_kernel, dim3((dim * per_key + LS_THREADS - 1) / LS_THREADS, heads, n_seqs),
                              dim3(LS_THREADS), 0, stream, sums, (const float*)factors, max_chunks, ch, shape, decays, batch))
        return code;
    const size_t smem = ls_output_smem(ch, dim);
    auto kernel = ch == 64 ? linear_state_output_kernel<64> : (ch == 32 ? linear_state_output_kernel<32> : linear_state_output_kernel<16>);
    if (int code = ls_reserve((const void*)kernel, smem, name)) return code;
    return launch_pdl(name, kernel, grid, dim3(LS_THREADS), smem, stream, rows, (const float*)sums, out, max_chunks,
                      (dim + 3) & ~3, shape, decays, cu_q);
}

// One token a sequence of a Mamba-2 mixer, in one kernel: rows float [n_seqs, row_stride] hold the input projection with
// the convolved channels first, [values: heads * vdim | keys: groups * dim | queries: groups * dim], and the step sizes at
// dt_at.  The state of a slot holds S twice from state_offset on and the ring of the last inputs [taps][channels] from
// ring_offset on.
SKV_EXPORT int skv_mamba2_step(const float* rows, int row_stride, const float* conv_w, const float* conv_b, int taps, int dt_at,
                               const float* dt_bias, const float* a_log, const float* skip, float* out, int n_seqs, int heads,
                               int groups, int dim, int vdim, const int* positions, const int* token_seq, const int* cu_q,
                               const int* slot_ids, float* state, long long state_stride, long long state_offset,
                               long long ring_offset, cudaStream_t stream) {
    const char* name = "skv_mamba2_step";
    if (n_seqs <= 0) return 0;
    if (!rows || !conv_w || !conv_b || !dt_bias || !a_log || !out || taps <= 0) return fail(name, "a weight or a place for the result is missing");
    if (n_seqs > 65535) return fail(name, "too many sequences in one step");
    const int inner = heads * vdim, channels = inner + 2 * groups * dim;
    const LinearStateShape shape = {heads, groups, dim, vdim, row_stride, inner + groups * dim, inner, 0, 0};
    const LinearStateDecay decays = {nullptr, nullptr, nullptr, skip, 1.0f, nullptr, 0.0f};
    const LinearStateBatch batch = {positions, cu_q, slot_ids, state, state_stride, state_offset};
    const ConvStep conv = {conv_w, conv_b, dt_bias, a_log, taps, channels, dt_at, ring_offset};
    if (int code = ls_check(name, shape, batch, false)) return code;
    if (dt_at < 0 || dt_at + heads > row_stride || ring_offset < 0 ||
        (taps > 1 && ring_offset + (long long)taps * channels > state_stride))
        return fail(name, "the step sizes must lie inside a row and the ring inside a slot's state");
    if (((uintptr_t)rows | (uintptr_t)out | (uintptr_t)state) & 15) return fail(name, "operands must be 16-byte aligned");
    const bool vec = vdim % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0;
    const size_t smem = (size_t)(2 * ((dim + 3) & ~3) + ((vdim + 3) & ~3) + LS_THREADS * (vec ? 4 : 1)) * sizeof(float);
    auto kernel = vec ? linear_state_step_kernel<4> : linear_state_step_kernel<1>;
    if (int code = ls_reserve((const void*)kernel, smem, name)) return code;
    return launch_pdl(name, kernel, dim3(heads, n_seqs), dim3(LS_THREADS), smem, stream, rows, out, shape, decays, conv, batch);
}

// out [n_tokens, channels] float = silu(conv_b + causal convolution over time of the rows' first `channels` columns); what
// lies before the step comes from the ring [taps][channels] at ring_offset of a slot's state.
SKV_EXPORT int skv_conv_silu(const float* rows, int row_stride, const float* conv_w, const float* conv_b, int channels, int taps,
                             float* out, int n_tokens, const int* positions, const int* token_seq, const int* cu_q,
                             const int* slot_ids, const float* state, long long state_stride, long long ring_offset,
                             cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!rows || !conv_w || !out || !positions || !token_seq || !cu_q || !slot_ids || (taps > 1 && !state))
        return fail("skv_conv_silu", "a pointer is missing");
    if (channels <= 0 || taps <= 0 || row_stride < channels || (taps > 1 && (ring_offset < 0 || ring_offset + (long long)taps * channels > state_stride)))
        return fail("skv_conv_silu", "sizes do not agree");
    const int rows_of_blocks = (n_tokens + CONV_TOKENS - 1) / CONV_TOKENS;
    if (rows_of_blocks > 65535) return fail("skv_conv_silu", "too many tokens in one step");
    return launch_pdl("skv_conv_silu", conv_silu_kernel, dim3((channels + 255) / 256, rows_of_blocks), dim3(256), 0, stream, rows,
                      row_stride, conv_w, conv_b, channels, taps, out, n_tokens, positions, token_seq, cu_q, slot_ids, state,
                      state_stride, ring_offset);
}

SKV_EXPORT int skv_step_sizes(const float* rows, int row_stride, int dt_at, const float* dt_bias, const float* a_log, int heads,
                              int n_tokens, float* dt, float* log_decay, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (!rows || !dt_bias || !a_log || !dt || !log_decay || heads <= 0 || dt_at < 0 || dt_at + heads > row_stride)
        return fail("skv_step_sizes", "the step sizes must lie inside a row");
    const long long items = (long long)n_tokens * heads;
    return launch_pdl("skv_step_sizes", step_sizes_kernel, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, stream, rows,
                      row_stride, dt_at, dt_bias, a_log, heads, n_tokens, dt, log_decay);
}

// y float [n, width], gate float rows gate_stride apart, weight float [width], out [n, out_stride] in the compute dtype.
SKV_EXPORT int skv_gated_norm(const float* y, const float* gate, int gate_stride, const float* weight, int width, int groups,
                              float eps, int mode, void* out, int out_stride, int n, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!y || !gate || !weight || !out || width <= 0 || groups <= 0 || width % groups || gate_stride < width || out_stride < width || groups > 65535 ||
        mode < GATE_SIGMOID || mode > GATE_SILU)
        return fail("skv_gated_norm", "sizes do not agree");
    const int size = width / groups;
    if ((long long)n * groups >= 2048 && (long long)n * groups <= 0x7fffffff && size <= 512 &&
        ((size | width | gate_stride | out_stride) & 3) == 0 && (((uintptr_t)y | (uintptr_t)gate | (uintptr_t)weight | (uintptr_t)out) & 15) == 0)
        return launch_pdl("skv_gated_norm", size <= 256 ? gated_norm_parts_kernel<skv_t, 2> : gated_norm_parts_kernel<skv_t, 4>, dim3((n * groups + 7) / 8), dim3(256), 0, stream, y, gate,
                          gate_stride, weight, width, groups, eps, mode, (skv_t*)out, out_stride, n * groups);
    const size_t smem = (size_t)size * sizeof(float);
    auto kernel = gated_norm_kernel<skv_t>;
    if (int code = ls_reserve((const void*)kernel, smem, "skv_gated_norm")) return code;
    return launch_pdl("skv_gated_norm", kernel, dim3(n, groups), dim3(256), smem, stream, y, gate, gate_stride, weight, width,
                      groups, eps, mode, (skv_t*)out, out_stride);
}

// rows float [n_tokens, row_stride] with the gates' logits at columns input_at and forget_at; log_decay, key_scale and floor
// float [n_tokens, heads]; a slot's state holds [2][heads] floats from m_offset on.
SKV_EXPORT int skv_exp_gates(const float* rows, int row_stride, int input_at, int forget_at, const float* input_bias,
                             const float* forget_bias, float cap, float* log_decay, float* key_scale, float* floor, int heads,
                             int n_seqs, const int* positions, const int* token_seq, const int* cu_q, const int* slot_ids,
                             float* state, long long state_stride, long long m_offset, cudaStream_t stream) {
    const char* name = "skv_exp_gates";
    if (n_seqs <= 0) return 0;
    if (!rows || !input_bias || !forget_bias || !log_decay || !key_scale || !floor || !positions || !cu_q || !slot_ids || !state)
        return fail(name, "a pointer is missing");
    if (heads <= 0 || n_seqs > 65535 || !(cap > 0.0f) || input_at < 0 || forget_at < 0 || input_at + heads > row_stride ||
        forget_at + heads > row_stride || m_offset < 0 || m_offset + 2LL * heads > state_stride)
        return fail(name, "the gates must lie inside a row and the maxima inside a slot's state");
    const LinearStateBatch batch = {positions, cu_q, slot_ids, state, state_stride, m_offset};
    return launch_pdl(name, exp_gates_kernel, dim3(heads, n_seqs), dim3(EG_THREADS), 0, stream, rows, row_stride, input_at,
                      forget_at, input_bias, forget_bias, cap, log_decay, key_scale, floor, heads, batch);
}
