// From the float rows [q | k | v] of a fused projection to attention's inputs, in one kernel with a block per token:
//
//   bias   added to the whole row first, if there is one;
//   q, k   an RMS norm with a weight over all query heads together and one over all key heads together (either may be
//          left out), then rotary positions on the first `rotated` numbers of every head (pairs (2i, 2i+1) or
//          (i, i + rotated/2));
//   v      taken as it is, or mixed with another layer's values of the same token: v <- (1 - m) v + m first;
//   out    queries in the compute dtype, keys and values into their places of the paged cache, and, for a layer whose
//          values others mix in, the float values of the step's tokens.
//
// A head may be stored wider than it is (query, key and value heads padded with zeros to a common width, so that the
// attention kernels built for that width serve other sizes): q_out is [tokens, heads * width], the caches
// [block][kv_head][block_size][width], or keys `dim` and values `vdim` wide with width 0.
#include "common.cuh"

namespace skv {

constexpr int NR_THREADS = 256;

struct NormedRotary {
    int heads, kv_heads, dim, vdim, q_width, v_width, row_stride;
    const float* q_weight;         // [heads * dim] or null
    const float* k_weight;         // [kv_heads * dim] or null
    float eps;
    const float* bias;             // [heads * dim + kv_heads * (dim + vdim)] or null
    const float2* cos_sin;         // [positions][rotated / 2] or null
    int rotated, interleaved;
    const float* mix;              // one number, or null
    const float* first;            // [tokens][kv_heads * vdim] (with mix)
    float* keep;                   // [tokens][kv_heads * vdim] or null
    int write_kv;
};

// Sums of two numbers over the block; every thread gets both.  `scratch` holds 18 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) { scratch[2 * warp] = a; scratch[2 * warp + 1] = b; }
    __syncthreads();
    float ta = 0.0f, tb = 0.0f;
#pragma unroll
    for (int w = 0; w < NR_THREADS / 32; ++w) { ta += scratch[2 * w]; tb += scratch[2 * w + 1]; }
    return make_float2(ta, tb);
}

// VEC: head sizes, widths and the row stride are multiples of 4, the rotation is interleaved (or absent, or its halves are
// multiples of 4) and every pointer is 16-byte aligned: four neighbouring numbers (two pairs, or one side of four) a thread
// and round.
template <typename T, bool VEC>
__global__ void __launch_bounds__(NR_THREADS)
normed_rotary_kernel(const float* __restrict__ rows, const int* __restrict__ positions, const int* __restrict__ token_seq,
                     const int* __restrict__ block_table, int table_width, T* __restrict__ q_out, T* __restrict__ k_cache,
                     T* __restrict__ v_cache, int block_size, const NormedRotary a) {
    __shared__ float scratch[2 * NR_THREADS / 32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const float* q = rows + (size_t)t * a.row_stride;
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    const float* k = q + nq;
    const float* v = k + nk;
    const float* bq = a.bias;                           // (null: no bias anywhere)
    const float* bk = bq ? bq + nq : nullptr;
    const float* bv = bq ? bk + nk : nullptr;
    auto load4 = [](const float* x, const float* b, int c) {
        float4 z = *(const float4*)(x + c);
        if (b) {
            const float4 w = *(const float4*)(b + c);
            z.x += w.x; z.y += w.y; z.z += w.z; z.w += w.w;
        }
        return z;
    };
    auto load1 = [](const float* x, const float* b, int c) { return b ? x[c] + b[c] : x[c]; };
    const int pos = positions[t];
    size_t base = 0;                                    // the token's row of key head 0, in rows of one head's vector
    if (a.write_kv) base = (size_t)block_table[(size_t)token_seq[t] * table_width + pos / block_size] * a.kv_heads * block_size + pos % block_size;
    const float2* angles = a.cos_sin ? a.cos_sin + (size_t)pos * (a.rotated >> 1) : nullptr;
    float q_factor = 1.0f, k_factor = 1.0f;
    if (a.q_weight || a.k_weight) {
        float sq = 0.0f, sk = 0.0f;
        if (VEC) {
            if (a.q_weight)
                for (int i = 4 * threadIdx.x; i < nq; i += 4 * NR_THREADS) {
                    const float4 x = load4(q, bq, i);
                    sq = fmaf(x.x, x.x, sq); sq = fmaf(x.y, x.y, sq); sq = fmaf(x.z, x.z, sq); sq = fmaf(x.w, x.w, sq);
                }
            if (a.k_weight)
                for (int i = 4 * threadIdx.x; i < nk; i += 4 * NR_THREADS) {
                    const float4 x = load4(k, bk, i);
                    sk = fmaf(x.x, x.x, sk); sk = fmaf(x.y, x.y, sk); sk = fmaf(x.z, x.z, sk); sk = fmaf(x.w, x.w, sk);
                }
        } else {
            if (a.q_weight) for (int i = threadIdx.x; i < nq; i += NR_THREADS) { const float x = load1(q, bq, i); sq = fmaf(x, x, sq); }
            if (a.k_weight) for (int i = threadIdx.x; i < nk; i += NR_THREADS) { const float x = load1(k, bk, i); sk = fmaf(x, x, sk); }
        }
        const float2 sums = block_sum2(sq, sk, scratch);
        if (a.q_weight) q_factor = 1.0f / sqrtf(sums.x / (float)nq + a.eps);
        if (a.k_weight) k_factor = 1.0f / sqrtf(sums.y / (float)nk + a.eps);
    }
    const float mix = a.mix ? *a.mix : 0.0f;
    if (VEC) {
        auto store4 = [](T* to, float4 x) {
            if (sizeof(T) == 4) {
                *(float4*)to = x;
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(x.x, x.y), hi = __floats2bfloat162_rn(x.z, x.w);
                *(uint2*)to = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
            }
        };
        const int quads = a.q_width >> 2, q_items = a.heads * quads, k_items = a.write_kv ? a.kv_heads * quads : 0;
        for (int item = threadIdx.x; item < q_items + k_items; item += NR_THREADS) {
            const bool is_query = item < q_items;
            const int index = is_query ? item : item - q_items;
            const int head = index / quads, d = (index - head * quads) * 4;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (d < a.dim) {
                const float* weight = is_query ? a.q_weight : a.k_weight;
                const float f = is_query ? q_factor : k_factor;
                auto normed4 = [&](int c) {
                    float4 z = load4(is_query ? q : k, is_query ? bq : bk, c);
                    if (weight) {
                        const float4 w = *(const float4*)(weight + c);
                        z.x *= f * w.x; z.y *= f * w.y; z.z *= f * w.z; z.w *= f * w.w;
                    }
                    return z;
                };
                const int c = head * a.dim + d;
                x = normed4(c);
                if (a.interleaved) {
                    if (d < a.rotated) {
                        const float2 cs = angles[d >> 1];
                        const float u = x.x * cs.x - x.y * cs.y;
                        x.y = x.y * cs.x + x.x * cs.y;
                        x.x = u;
                    }
                    if (d + 2 < a.rotated) {
                        const float2 cs = angles[(d >> 1) + 1];
                        const float u = x.z * cs.x - x.w * cs.y;
                        x.w = x.w * cs.x + x.z * cs.y;
                        x.z = u;
                    }
                } else if (d < a.rotated) {
                    const int half = a.rotated >> 1;
                    const bool low = d < half;
                    const float4 m = normed4(low ? c + half : c - half);
                    const float sign = low ? -1.0f : 1.0f;
                    const float2* turn = angles + (low ? d : d - half);
                    const float2 t0 = turn[0], t1 = turn[1], t2 = turn[2], t3 = turn[3];
                    x = make_float4(x.x * t0.x + sign * m.x * t0.y, x.y * t1.x + sign * m.y * t1.y,
                                    x.z * t2.x + sign * m.z * t2.y, x.w * t3.x + sign * m.w * t3.y);
                }
            }
            store4(is_query ? q_out + ((size_t)t * a.heads + head) * a.q_width + d
                            : k_cache + (base + (size_t)head * block_size) * a.q_width + d, x);
        }
        const int v_quads = a.v_width >> 2;
        for (int item = threadIdx.x; item < a.kv_heads * v_quads; item += NR_THREADS) {
            const int head = item / v_quads, d = (item - head * v_quads) * 4;
            float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (d < a.vdim) {
                const size_t c = (size_t)head * a.vdim + d;
                x = load4(v, bv, (int)c);
                if (a.keep) *(float4*)(a.keep + (size_t)t * nv + c) = x;
                if (a.mix) {
                    const float4 f = *(const float4*)(a.first + (size_t)t * nv + c);
                    x = make_float4(fmaf(mix, f.x, (1.0f - mix) * x.x), fmaf(mix, f.y, (1.0f - mix) * x.y),
                                    fmaf(mix, f.z, (1.0f - mix) * x.z), fmaf(mix, f.w, (1.0f - mix) * x.w));
                }
            }
            if (a.write_kv) store4(v_cache + (base + (size_t)head * block_size) * a.v_width + d, x);
        }
        return;
    }
    const int half = a.rotated >> 1;
    auto value_at = [&](bool is_query, int head, int d) {
        const int c = head * a.dim + d;
        const float* weight = is_query ? a.q_weight : a.k_weight;
        const float x = load1(is_query ? q : k, is_query ? bq : bk, c);
        return weight ? x * ((is_query ? q_factor : k_factor) * weight[c]) : x;
    };
    const int q_items = a.heads * a.q_width, k_items = a.write_kv ? a.kv_heads * a.q_width : 0;
    for (int item = threadIdx.x; item < q_items + k_items; item += NR_THREADS) {
        const bool is_query = item < q_items;
        const int index = is_query ? item : item - q_items;
        const int head = index / a.q_width, d = index - head * a.q_width;
        float x = 0.0f;
        if (d < a.dim) {
            x = value_at(is_query, head, d);
            if (d < a.rotated) {
                const bool low = a.interleaved ? !(d & 1) : d < half;
                const int mate = a.interleaved ? (d ^ 1) : (low ? d + half : d - half);
                const float2 cs = angles[a.interleaved ? (d >> 1) : (low ? d : d - half)];
                const float other = value_at(is_query, head, mate);
                x = low ? x * cs.x - other * cs.y : x * cs.x + other * cs.y;
            }
        }
        T* to = is_query ? q_out + ((size_t)t * a.heads + head) * a.q_width : k_cache + (base + (size_t)head * block_size) * a.q_width;
        to[d] = from_float<T>(x);
    }
    for (int item = threadIdx.x; item < a.kv_heads * a.v_width; item += NR_THREADS) {
        const int head = item / a.v_width, d = item - head * a.v_width;
        float x = 0.0f;
        if (d < a.vdim) {
            const size_t c = (size_t)head * a.vdim + d;
            x = load1(v, bv, (int)c);
            if (a.keep) a.keep[(size_t)t * nv + c] = x;
            if (a.mix) x = fmaf(mix, a.first[(size_t)t * nv + c], (1.0f - mix) * x);
        }
        if (a.write_kv) v_cache[(base + (size_t)head * block_size) * a.v_width + d] = from_float<T>(x);
    }
}

}  // namespace skv

using namespace skv;

// rows float [n, row_stride]: [heads * dim queries | kv_heads * dim keys | kv_heads * vdim values | ...]; q_out
// [n, heads * q_width], k_cache [blocks, kv_heads, block_size, q_width], v_cache [.., v_width] in the compute dtype.
SKV_EXPORT int skv_normed_rotary(const float* rows, int row_stride, const float* bias, const float* q_weight, const float* k_weight, float eps,
                                 const float* cos_sin, int rotated, int interleaved, const float* mix, const float* first,
                                 float* keep, const int* positions, const int* token_seq, const int* block_table,
                                 int table_width, void* q_out, void* k_cache, void* v_cache, int n, int heads, int kv_heads,
                                 int dim, int vdim, int q_width, int v_width, int block_size, int write_kv,
                                 cudaStream_t stream) {
    const char* name = "skv_normed_rotary";
    if (n <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || block_size <= 0 || q_width < dim || v_width < vdim ||
        row_stride < heads * dim + kv_heads * (dim + vdim) || rotated < 0 || rotated > dim || (rotated & 1))
        return fail(name, "sizes do not agree");
    if (!rows || !positions || !token_seq || !block_table || !q_out || !k_cache || !v_cache || (rotated > 0 && !cos_sin) || (mix && !first))
        return fail(name, "a pointer is missing");
    const NormedRotary a = {heads, kv_heads, dim, vdim, q_width, v_width, row_stride, q_weight, k_weight, eps, bias,
                            (const float2*)(rotated > 0 ? cos_sin : nullptr), rotated, interleaved, mix, first, keep, write_kv};
    const bool vec = ((dim | vdim | q_width | v_width | row_stride) & 3) == 0 && (interleaved || rotated % 8 == 0) &&
                     (((uintptr_t)rows | (uintptr_t)bias | (uintptr_t)q_weight | (uintptr_t)k_weight | (uintptr_t)first | (uintptr_t)keep |
                       (uintptr_t)q_out | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) == 0;
    auto kernel = vec ? normed_rotary_kernel<skv_t, true> : normed_rotary_kernel<skv_t, false>;
    return launch_pdl(name, kernel, dim3(n), dim3(NR_THREADS), 0, stream, rows, positions, token_seq, block_table, table_width,
                      (skv_t*)q_out, (skv_t*)k_cache, (skv_t*)v_cache, block_size, a);
}
