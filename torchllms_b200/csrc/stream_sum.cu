// Blocks whose sublayers all read one norm's rows and whose results enter the stream in one sum.
//
// stream_add: h += coef * sum_i t_i / sqrt(mean(t_i^2) + eps) * w_i + sum_j p_j   (h float32, in place),
//             up to two normed terms (a pair of mixers side by side) and up to three plain ones; the new
//             stream also leaves in bfloat16 where the next product wants it so.
// polynorm:   a N(z) + b N(z^2) + c N(z^3) + e over a row, N(y) = y / sqrt(mean(y^2) + eps), powers element
//             by element; one pass gathers the three sums of squares, one writes.
// side_gate:  gelu_tanh(u) * table[token]: the gate of a per-token input.
//
// stream_inject: h[t] += e[t] + r: a second stream and one row for all tokens (either may be absent), float32.
//
// stream_join:   out[t] = [h[t] + c * d | e[t]], the input of a product that makes the next stream from this one (its pending sum
//                included) and another; the next stream starts as a row shared by all tokens.
//
// group_norm:    x = h[t] + c * d;  every one of `groups` equal runs of neighbouring columns is divided by its own
//                sqrt(mean(x^2) + eps), the row is multiplied by w, and x replaces h[t] (c: a vector, or ones).
//
// sum_partials: the planes of a split-K product added up and rounded once (for readers that take no partial sums).
//
// Sums, norms and the stream are float32 whatever the terms' dtype.  Every term may arrive as float32 partial sums
// [splits][T][width] of a split-K product (planes `plane` elements apart); the kernels add the planes up as they read.
#include "common.cuh"

namespace {

constexpr int MAX_NORMED = 2, MAX_PLAIN = 3;

__device__ __forceinline__ float block_sum(float v, float* part) {
    // part: 33 floats of shared memory
    v = warp_sum(v);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) part[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < n_warps ? part[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) part[32] = t;
    }
    __syncthreads();
    return part[32];
}

__device__ __forceinline__ float load_as(const void* p, int dtype, size_t at) {
    return dtype == TL_BF16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[at]) : reinterpret_cast<const float*>(p)[at];
}

// the sum over the planes of a split-K product (or the one plane there is)
__device__ __forceinline__ float load_sum(const void* p, int dtype, int splits, long long plane, size_t at) {
    float v = load_as(p, dtype, at);
    for (int s = 1; s < splits; ++s) v += reinterpret_cast<const float*>(p)[(size_t)s * plane + at];
    return v;
}

struct SumParams {
    float* h;                         // [T][dim]
    const void* normed[MAX_NORMED];   // [T][dim] each
    const float* weight[MAX_NORMED];  // [dim] each
    int normed_dtype[MAX_NORMED], normed_splits[MAX_NORMED];
    long long normed_plane[MAX_NORMED];
    const void* plain[MAX_PLAIN];     // [T][dim] each
    int plain_dtype[MAX_PLAIN], plain_splits[MAX_PLAIN];
    long long plain_plane[MAX_PLAIN];
    int n_normed, n_plain, dim;
    float coef, eps;
    __nv_bfloat16* rows;              // [T][dim] or null
};

// a CTA per token
__global__ void stream_add_kernel(const SumParams p) {
    __shared__ float part[33];
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t base = (size_t)blockIdx.x * p.dim;
    float r[MAX_NORMED];
#pragma unroll
    for (int i = 0; i < MAX_NORMED; ++i) {
        r[i] = 0.f;
        if (i < p.n_normed) {
            float ssq = 0.f;
            for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
                const float v = load_sum(p.normed[i], p.normed_dtype[i], p.normed_splits[i], p.normed_plane[i], base + d);
                ssq = fmaf(v, v, ssq);
            }
            r[i] = rsqrtf(block_sum(ssq, part) / (float)p.dim + p.eps);
        }
    }
    for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
        float m = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_NORMED; ++i)
            if (i < p.n_normed)
                m += load_sum(p.normed[i], p.normed_dtype[i], p.normed_splits[i], p.normed_plane[i], base + d) * r[i] * p.weight[i][d];
        float v = p.h[base + d] + p.coef * m;
#pragma unroll
        for (int i = 0; i < MAX_PLAIN; ++i)
            if (i < p.n_plain) v += load_sum(p.plain[i], p.plain_dtype[i], p.plain_splits[i], p.plain_plane[i], base + d);
        p.h[base + d] = v;
        if (p.rows != nullptr) p.rows[base + d] = __float2bfloat16_rn(v);
    }
}

template <typename TI, typename TO>
__global__ void polynorm_kernel(const TI* __restrict__ z, int splits, long long plane, const float* __restrict__ coef,
                                TO* __restrict__ out, int width, float eps) {
    __shared__ float part[33];
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t base = (size_t)blockIdx.x * width;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int d = threadIdx.x; d < width; d += blockDim.x) {
        float v = to_float(z[base + d]);
        for (int sp = 1; sp < splits; ++sp) v += to_float(z[(size_t)sp * plane + base + d]);
        const float v2 = v * v, v3 = v2 * v;
        s2 += v2;
        s4 = fmaf(v2, v2, s4);
        s6 = fmaf(v3, v3, s6);
    }
    const float inv = 1.f / (float)width;
    const float r1 = rsqrtf(block_sum(s2, part) * inv + eps);
    const float r2 = rsqrtf(block_sum(s4, part) * inv + eps);
    const float r3 = rsqrtf(block_sum(s6, part) * inv + eps);
    const float a = coef[0] * r1, b = coef[1] * r2, c = coef[2] * r3, e = coef[3];
    for (int d = threadIdx.x; d < width; d += blockDim.x) {
        float v = to_float(z[base + d]);
        for (int sp = 1; sp < splits; ++sp) v += to_float(z[(size_t)sp * plane + base + d]);
        const float v2 = v * v;
        out[base + d] = from_float<TO>(a * v + b * v2 + c * (v2 * v) + e);
    }
}

template <typename TI, typename TT, typename TO>
__global__ void side_gate_kernel(const TI* __restrict__ u, int splits, long long plane, const int* __restrict__ token_ids,
                                 const TT* __restrict__ table, TO* __restrict__ out, long long total, int width, int vocab) {
    grid_launch_dependents();
    grid_dependency_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / width;
        const int c = (int)(i - t * width);
        int tok = token_ids[t];
        if (!TL_CHECK(tok >= 0 && tok < vocab, TL_DBG_TOKEN_ID)) tok = 0;
        float x = to_float(u[i]);
        for (int sp = 1; sp < splits; ++sp) x += to_float(u[(size_t)sp * plane + i]);
        const float g = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
        out[i] = from_float<TO>(g * to_float(table[(size_t)tok * width + c]));
    }
}

__global__ void stream_inject_kernel(float* __restrict__ h, const float* __restrict__ rows, const float* __restrict__ row,
                                     long long total, int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        float v = h[i];
        if (rows != nullptr) v += rows[i];
        if (row != nullptr) v += row[i % width];
        h[i] = v;
    }
}

// VEC: four columns per thread and turn (columns and planes are multiples of 4)
template <int VEC>
struct Cols { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Cols<VEC> load_cols(const float* p) {
    Cols<VEC> c;
    if (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        c.v[0] = x.x; c.v[VEC > 1 ? 1 : 0] = x.y; c.v[VEC > 2 ? 2 : 0] = x.z; c.v[VEC > 3 ? 3 : 0] = x.w;
    } else c.v[0] = *p;
    return c;
}
template <int VEC> __device__ __forceinline__ Cols<VEC> load_cols(const __nv_bfloat16* p) {
    Cols<VEC> c;
    if (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        c.v[0] = a.x; c.v[VEC > 1 ? 1 : 0] = a.y; c.v[VEC > 2 ? 2 : 0] = b.x; c.v[VEC > 3 ? 3 : 0] = b.y;
    } else c.v[0] = __bfloat162float(*p);
    return c;
}
template <int VEC> __device__ __forceinline__ void store_cols(float* p, const Cols<VEC>& c) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[VEC > 1 ? 1 : 0], c.v[VEC > 2 ? 2 : 0], c.v[VEC > 3 ? 3 : 0]);
    else *p = c.v[0];
}
template <int VEC> __device__ __forceinline__ void store_cols(__nv_bfloat16* p, const Cols<VEC>& c) {
    if (VEC == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(c.v[0], c.v[VEC > 1 ? 1 : 0]), b = __floats2bfloat162_rn(c.v[VEC > 2 ? 2 : 0], c.v[VEC > 3 ? 3 : 0]);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned*>(&a);
        raw.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    } else *p = __float2bfloat16_rn(c.v[0]);
}

// the stream with its pending sum: h + scale * (sum of delta's planes); delta and scale may be null
template <int VEC, typename TD>
__device__ __forceinline__ Cols<VEC> summed(const float* h, const TD* delta, int splits, long long plane, const float* scale, size_t at, int d) {
    Cols<VEC> x = load_cols<VEC>(h + at);
    if (delta != nullptr) {
        Cols<VEC> y = load_cols<VEC>(delta + at);
#pragma unroll 4
        for (int s = 1; s < splits; ++s) {
            const Cols<VEC> z = load_cols<VEC>(delta + (size_t)s * plane + at);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y.v[i] += z.v[i];
        }
        if (scale != nullptr) {
            const Cols<VEC> c = load_cols<VEC>(scale + d);
#pragma unroll
            for (int i = 0; i < VEC; ++i) y.v[i] *= c.v[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; ++i) x.v[i] += y.v[i];
    }
    return x;
}

template <int VEC, typename TD, typename TO>
__global__ void stream_join_kernel(const float* __restrict__ h, const TD* __restrict__ delta, int splits, long long plane,
                                   const float* __restrict__ scale, const float* __restrict__ rows, const float* __restrict__ row,
                                   TO* __restrict__ out, float* __restrict__ h_next, long long n_chunks, int width) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int per_row = width / VEC;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n_chunks; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / per_row;
        const int d = (int)(i - t * per_row) * VEC;
        const size_t at = (size_t)t * width + d;
        store_cols<VEC>(out + (size_t)t * 2 * width + d, summed<VEC>(h, delta, splits, plane, scale, at, d));
        store_cols<VEC>(out + (size_t)t * 2 * width + width + d, load_cols<VEC>(rows + at));
        Cols<VEC> r;
#pragma unroll
        for (int e = 0; e < VEC; ++e) r.v[e] = 0.f;
        if (row != nullptr) r = load_cols<VEC>(row + d);
        store_cols<VEC>(h_next + at, r);
    }
}

// A CTA per row.  The warps form teams, one per group where there are warps enough, and a team walks its groups
// (all teams the same number of times); a thread reads back only what it kept in shared memory itself.
template <int VEC, typename TD, typename TO>
__global__ void group_norm_kernel(float* __restrict__ h, const TD* __restrict__ delta, int splits, long long plane,
                                  const float* __restrict__ scale, const float* __restrict__ weight, TO* __restrict__ out,
                                  const int* __restrict__ pick, int dim, int groups, int teams, float eps, int write_back) {
    extern __shared__ __align__(16) float row_buf[];
    __shared__ float part[32];
    grid_launch_dependents();
    int r = pick != nullptr ? pick[blockIdx.x] : (int)blockIdx.x;
    if (!tl_check_row(r)) r = 0;
    grid_dependency_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    const int per_team = n_warps / teams, team = warp / per_team;
    const int in_team = (warp - team * per_team) * 32 + lane, size = dim / groups;
    const size_t base = (size_t)r * dim;
    TO* o = out + (size_t)blockIdx.x * dim;
    const int rounds = (groups + teams - 1) / teams;
    for (int k = 0; k < rounds; ++k) {
        const int g = k * teams + team;
        const bool mine = team < teams && g < groups;
        float ssq = 0.f;
        if (mine) {
            for (int c = in_team * VEC; c < size; c += per_team * 32 * VEC) {
                const int d = g * size + c;
                const Cols<VEC> x = summed<VEC>(h, delta, splits, plane, scale, base + d, d);
                store_cols<VEC>(row_buf + d, x);
                if (write_back) store_cols<VEC>(h + base + d, x);
#pragma unroll
                for (int i = 0; i < VEC; ++i) ssq = fmaf(x.v[i], x.v[i], ssq);
            }
        }
        ssq = warp_sum(ssq);
        if (k > 0) __syncthreads();            // part[] of the round before is read
        if (lane == 0) part[warp] = ssq;
        __syncthreads();
        if (!mine) continue;
        float total = 0.f;
        for (int w = 0; w < per_team; ++w) total += part[team * per_team + w];
        const float rs = rsqrtf(total / (float)size + eps);
        for (int c = in_team * VEC; c < size; c += per_team * 32 * VEC) {
            const int d = g * size + c;
            Cols<VEC> x = load_cols<VEC>(row_buf + d);
            const Cols<VEC> w = load_cols<VEC>(weight + d);
#pragma unroll
            for (int i = 0; i < VEC; ++i) x.v[i] *= rs * w.v[i];
            store_cols<VEC>(o + d, x);
        }
    }
}

template <typename TO>
__global__ void sum_partials_kernel(const float* __restrict__ parts, int splits, long long plane, TO* __restrict__ out, long long total) {
    grid_launch_dependents();
    grid_dependency_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        float v = parts[i];
        for (int sp = 1; sp < splits; ++sp) v += parts[(size_t)sp * plane + i];
        out[i] = from_float<TO>(v);
    }
}

// threads of a CTA that owns a row: few rows (a decode step, whose terms are often many planes of partial sums) are
// all the parallelism there is, so a row gets as many threads as it has pairs of columns
int row_threads(int width, int n_rows) {
    if (n_rows <= 64) {
        const int t = ((width / 2 + 31) / 32) * 32;
        return t > 1024 ? 1024 : t < 128 ? 128 : t;
    }
    return width >= 2048 ? 512 : width >= 512 ? 256 : 128;
}

}  // namespace

// h: float32 [n_tokens][dim], updated in place; normed / plain: arrays of n_normed (<= 2) / n_plain (<= 3) pointers to
// [splits][n_tokens][dim] tensors with their dtype codes, plane counts (1: no partial sums; more only in float32) and
// the planes' distance in elements; weights: n_normed pointers to float32 [dim]; rows: bfloat16 [n_tokens][dim] or null.
extern "C" int tl_stream_add(float* h, const void* const* normed, const int* normed_dtype, const int* normed_splits,
                             const long long* normed_plane, const float* const* weights, int n_normed, const void* const* plain,
                             const int* plain_dtype, const int* plain_splits, const long long* plain_plane, int n_plain, float coef,
                             float eps, void* rows, int n_tokens, int dim, void* stream) {
    if (n_tokens <= 0) return TL_OK;
    if (dim <= 0 || n_normed < 0 || n_normed > MAX_NORMED || n_plain < 0 || n_plain > MAX_PLAIN) return TL_BAD_SIZE;
    SumParams p = {};
    p.h = h; p.n_normed = n_normed; p.n_plain = n_plain; p.dim = dim; p.coef = coef; p.eps = eps;
    p.rows = reinterpret_cast<__nv_bfloat16*>(rows);
    for (int i = 0; i < n_normed; ++i) {
        if (normed_dtype[i] != TL_F32 && normed_dtype[i] != TL_BF16) return TL_BAD_DTYPE;
        if (normed_splits[i] < 1 || (normed_splits[i] > 1 && normed_dtype[i] != TL_F32)) return TL_BAD_SIZE;
        p.normed[i] = normed[i]; p.normed_dtype[i] = normed_dtype[i]; p.weight[i] = weights[i];
        p.normed_splits[i] = normed_splits[i]; p.normed_plane[i] = normed_plane[i];
    }
    for (int i = 0; i < n_plain; ++i) {
        if (plain_dtype[i] != TL_F32 && plain_dtype[i] != TL_BF16) return TL_BAD_DTYPE;
        if (plain_splits[i] < 1 || (plain_splits[i] > 1 && plain_dtype[i] != TL_F32)) return TL_BAD_SIZE;
        p.plain[i] = plain[i]; p.plain_dtype[i] = plain_dtype[i]; p.plain_splits[i] = plain_splits[i]; p.plain_plane[i] = plain_plane[i];
    }
    return (int)tl_launch(stream_add_kernel, dim3(n_tokens), dim3(row_threads(dim, n_tokens)), 0, (cudaStream_t)stream, p);
}

// z: [splits][n_tokens][width]; coef: float32 [4] = (a, b, c, e); out: [n_tokens][width].
extern "C" int tl_polynorm(const void* z, int in_dtype, int splits, long long plane, const float* coef, void* out, int out_dtype,
                           int n_tokens, int width, float eps, void* stream) {
    if (n_tokens <= 0) return TL_OK;
    if (width <= 0 || splits < 1 || (splits > 1 && in_dtype != TL_F32)) return TL_BAD_SIZE;
    const dim3 grid(n_tokens), block(row_threads(width, n_tokens));
    cudaStream_t s = (cudaStream_t)stream;
    if (in_dtype == TL_F32 && out_dtype == TL_F32)
        return (int)tl_launch(polynorm_kernel<float, float>, grid, block, 0, s, (const float*)z, splits, plane, coef, (float*)out, width, eps);
    if (in_dtype == TL_F32 && out_dtype == TL_BF16)
        return (int)tl_launch(polynorm_kernel<float, __nv_bfloat16>, grid, block, 0, s, (const float*)z, splits, plane, coef, (__nv_bfloat16*)out, width, eps);
    if (in_dtype == TL_BF16 && out_dtype == TL_BF16)
        return (int)tl_launch(polynorm_kernel<__nv_bfloat16, __nv_bfloat16>, grid, block, 0, s, (const __nv_bfloat16*)z, splits, plane, coef,
                              (__nv_bfloat16*)out, width, eps);
    return TL_BAD_DTYPE;
}

// u: [splits][n_tokens][width] of u_dtype (float32 where splits > 1); table: [vocab][width] and out: [n_tokens][width] of dtype.
extern "C" int tl_side_gate(const void* u, int u_dtype, int splits, long long plane, const int* token_ids, const void* table, void* out,
                            int dtype, int n_tokens, int width, int vocab, void* stream) {
    if (n_tokens <= 0) return TL_OK;
    if (width <= 0 || vocab <= 0 || splits < 1 || (splits > 1 && u_dtype != TL_F32)) return TL_BAD_SIZE;
    const long long total = (long long)n_tokens * width;
    const dim3 grid((unsigned)((total + 255) / 256 > 148 * 8 ? 148 * 8 : (total + 255) / 256)), block(256);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == TL_F32 && u_dtype == TL_F32)
        return (int)tl_launch(side_gate_kernel<float, float, float>, grid, block, 0, s, (const float*)u, splits, plane, token_ids,
                              (const float*)table, (float*)out, total, width, vocab);
    if (dtype == TL_BF16 && u_dtype == TL_F32)
        return (int)tl_launch(side_gate_kernel<float, __nv_bfloat16, __nv_bfloat16>, grid, block, 0, s, (const float*)u, splits, plane,
                              token_ids, (const __nv_bfloat16*)table, (__nv_bfloat16*)out, total, width, vocab);
    if (dtype == TL_BF16 && u_dtype == TL_BF16)
        return (int)tl_launch(side_gate_kernel<__nv_bfloat16, __nv_bfloat16, __nv_bfloat16>, grid, block, 0, s, (const __nv_bfloat16*)u,
                              splits, plane, token_ids, (const __nv_bfloat16*)table, (__nv_bfloat16*)out, total, width, vocab);
    return TL_BAD_DTYPE;
}

// parts: float32 [splits][total], planes `plane` elements apart; out: [total] of out_dtype.
extern "C" int tl_sum_partials(const float* parts, int splits, long long plane, void* out, int out_dtype, long long total, void* stream) {
    if (total <= 0) return TL_OK;
    if (splits < 1) return TL_BAD_SIZE;
    long long blocks = (total + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    const dim3 grid((unsigned)blocks), block(256);
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == TL_F32) return (int)tl_launch(sum_partials_kernel<float>, grid, block, 0, s, parts, splits, plane, (float*)out, total);
    if (out_dtype == TL_BF16)
        return (int)tl_launch(sum_partials_kernel<__nv_bfloat16>, grid, block, 0, s, parts, splits, plane, (__nv_bfloat16*)out, total);
    return TL_BAD_DTYPE;
}

// h: float32 [n_tokens][width], updated in place; rows: float32 [n_tokens][width] or null; row: float32 [width] or null
extern "C" int tl_stream_inject(float* h, const float* rows, const float* row, int n_tokens, int width, void* stream) {
    if (n_tokens <= 0 || width <= 0) return TL_OK;
    const long long total = (long long)n_tokens * width;
    long long blocks = (total + 255) / 256;
    if (blocks > 148 * 8) blocks = 148 * 8;
    return (int)tl_launch(stream_inject_kernel, dim3((unsigned)blocks), dim3(256), 0, (cudaStream_t)stream, h, rows, row, total, width);
}

// h: float32 [n_tokens][width] (left as it is); delta: [splits][n_tokens][width] of delta_dtype (float32 where splits > 1) or
// null, planes `plane` elements apart; scale: float32 [width] or null; rows: float32 [n_tokens][width]; row: float32
// [width] or null; out: [n_tokens][2 * width] of out_dtype; h_next: float32 [n_tokens][width], row (or zeros) in every token.
extern "C" int tl_stream_join(const float* h, const void* delta, int delta_dtype, int splits, long long plane, const float* scale,
                              const float* rows, const float* row, void* out, int out_dtype, float* h_next, int n_tokens, int width,
                              void* stream) {
    if (n_tokens <= 0) return TL_OK;
    if (width <= 0 || splits < 1 || rows == nullptr || h_next == h || (splits > 1 && delta_dtype != TL_F32)) return TL_BAD_SIZE;
    const bool vec = width % 4 == 0 && plane % 4 == 0 && aligned16(h) && aligned16(delta) && aligned16(scale) && aligned16(rows) &&
                     aligned16(row) && aligned16(out) && aligned16(h_next);
    const long long n_chunks = (long long)n_tokens * (vec ? width / 4 : width);
    long long blocks = (n_chunks + 255) / 256;
    if (blocks > 148 * 16) blocks = 148 * 16;
    const dim3 grid((unsigned)blocks), block(256);
    cudaStream_t s = (cudaStream_t)stream;
#define TL_JOIN(TD, TO)                                                                                                            \
    return (int)(vec ? tl_launch(stream_join_kernel<4, TD, TO>, grid, block, 0, s, h, (const TD*)delta, splits, plane, scale, rows, row, \
                                 (TO*)out, h_next, n_chunks, width)                                                                \
                     : tl_launch(stream_join_kernel<1, TD, TO>, grid, block, 0, s, h, (const TD*)delta, splits, plane, scale, rows, row, \
                                 (TO*)out, h_next, n_chunks, width))
    if (delta_dtype == TL_F32 && out_dtype == TL_F32) TL_JOIN(float, float);
    if (delta_dtype == TL_F32 && out_dtype == TL_BF16) TL_JOIN(float, __nv_bfloat16);
    if (delta_dtype == TL_BF16 && out_dtype == TL_BF16) TL_JOIN(__nv_bfloat16, __nv_bfloat16);
    if (delta_dtype == TL_BF16 && out_dtype == TL_F32) TL_JOIN(__nv_bfloat16, float);
#undef TL_JOIN
    return TL_BAD_DTYPE;
}

// h: float32 [rows of the stream][dim], replaced by the sum where write_back; delta, scale as above (delta rows are h's); weight:
// float32 [dim]; pick: int32 [n_out] rows of h, or null (row o is row o of h); out: [n_out][dim] of out_dtype.
extern "C" int tl_group_norm(float* h, const void* delta, int delta_dtype, int splits, long long plane, const float* scale,
                             const float* weight, void* out, int out_dtype, const int* pick, int n_out, int dim, int groups, float eps,
                             int write_back, void* stream) {
    if (n_out <= 0) return TL_OK;
    if (dim <= 0 || groups <= 0 || dim % groups != 0 || splits < 1 || (splits > 1 && delta_dtype != TL_F32)) return TL_BAD_SIZE;
    const size_t smem = (size_t)dim * sizeof(float);
    if (smem > 200 * 1024) return TL_TOO_LARGE;
    const bool vec = (dim / groups) % 4 == 0 && plane % 4 == 0 && aligned16(h) && aligned16(delta) && aligned16(scale) &&
                     aligned16(weight) && aligned16(out);
    int warps = (dim / (vec ? 4 : 1) + 31) / 32;
    const int most = n_out >= 512 ? 8 : 32;              // many rows: smaller CTAs, more of them resident
    warps = warps < 2 ? 2 : (warps > most ? most : warps);
    const int teams = groups < warps ? groups : warps;
    warps = warps / teams * teams;
    const dim3 grid(n_out), block(warps * 32);
    cudaStream_t s = (cudaStream_t)stream;
#define TL_GN(V, TD, TO)                                                                                                          \
    do {                                                                                                                          \
        static int raised = 0;                                                                                                    \
        if (smem > 48 * 1024 && (int)smem > raised) {                                                                             \
            cudaError_t e = cudaFuncSetAttribute(group_norm_kernel<V, TD, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                                  \
            raised = (int)smem;                                                                                                   \
        }                                                                                                                         \
        return (int)tl_launch(group_norm_kernel<V, TD, TO>, grid, block, smem, s, h, (const TD*)delta, splits, plane, scale, weight, \
                              (TO*)out, pick, dim, groups, teams, eps, write_back);                                               \
    } while (0)
#define TL_GN_PICK(TD, TO) do { if (vec) TL_GN(4, TD, TO); else TL_GN(1, TD, TO); } while (0)
    if (delta_dtype == TL_F32 && out_dtype == TL_F32) TL_GN_PICK(float, float);
    if (delta_dtype == TL_F32 && out_dtype == TL_BF16) TL_GN_PICK(float, __nv_bfloat16);
    if (delta_dtype == TL_BF16 && out_dtype == TL_BF16) TL_GN_PICK(__nv_bfloat16, __nv_bfloat16);
    if (delta_dtype == TL_BF16 && out_dtype == TL_F32) TL_GN_PICK(__nv_bfloat16, float);
#undef TL_GN_PICK
#undef TL_GN
    return TL_BAD_DTYPE;
}
