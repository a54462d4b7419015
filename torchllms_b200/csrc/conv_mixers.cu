// What stands between a mixer's stacked input projection and its attention or recurrence where every channel of
// q, k and v passes a short causal convolution over time first:  y_t = sum_j w[j][c] u_(t - taps + 1 + j), the last
// taps - 1 inputs of every request being its state (zeros for a fresh one).
//
// conv_rope_store: row [q heads | k heads | v heads | extra]: convolution of the q, k and v columns, rotation of the
//                  first rot coordinates of every q and k head (coordinate i with i + rot / 2), k and v into their pages,
//                  q and scale * sigmoid(extra) as tensors.
// delta_prep:      row [q heads | k heads | v | small | low | ...]: convolution and silu of the q, k and v columns; every
//                  head of q and k as a unit vector in float32 (q times a scale); v, the small columns and the low ones
//                  (padded with zeros to a row that a product can take) as tensors of their own.
// channel_decay:   g = exp(-rate_h softplus(z + bias)) per head and key coordinate, float32.
//
// Rows are column ranges of wider rows (a row pitch) and may be float32 partial sums of a split-K product (planes),
// added up on the way in.  A thread (conv_rope_store) or a warp (delta_prep) owns columns of TOK tokens of a
// portion, with a window of the inputs before them in registers.  In a step of short portions it also leaves the new
// state; with longer portions a kernel of its own does that afterwards, since several owners read the old one.
// All arithmetic is float32.
#include "common.cuh"

namespace {

constexpr int MAX_TAPS = 8;
constexpr int TOK = 4;             // tokens of a portion that one owner of columns takes: all its loads are in flight at once
constexpr int NT = 128;

struct ConvInput {
    const void* proj;        // [splits][T] rows of pitch ld
    int splits;
    long long plane, ld;
    const float* w;          // [taps][C], the last row the current token's
    float* state;            // [slots] rows of pitch state_pitch, each [taps - 1][C]; null with one tap
    long long state_pitch;
    const int* q_start;      // [B + 1]
    const int* state_slot;   // [B]
    const int* fresh;        // [B]
    int C, taps, n_chunks;
};

template <int VEC> struct Cols { float v[VEC]; };

template <int VEC> __device__ __forceinline__ Cols<VEC> load_cols(const float* p) {
    Cols<VEC> c;
    if constexpr (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        c.v[0] = x.x; c.v[1] = x.y; c.v[2] = x.z; c.v[3] = x.w;
    } else if constexpr (VEC == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        c.v[0] = x.x; c.v[1] = x.y;
    } else c.v[0] = *p;
    return c;
}
template <int VEC> __device__ __forceinline__ Cols<VEC> load_cols(const __nv_bfloat16* p) {
    Cols<VEC> c;
    if constexpr (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        c.v[0] = a.x; c.v[1] = a.y; c.v[2] = b.x; c.v[3] = b.y;
    } else if constexpr (VEC == 2) {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
        c.v[0] = a.x; c.v[1] = a.y;
    } else c.v[0] = __bfloat162float(*p);
    return c;
}
template <int VEC> __device__ __forceinline__ void store_cols(float* p, const Cols<VEC>& c) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
    else if constexpr (VEC == 2) *reinterpret_cast<float2*>(p) = make_float2(c.v[0], c.v[1]);
    else *p = c.v[0];
}
template <int VEC> __device__ __forceinline__ void store_cols(__nv_bfloat16* p, const Cols<VEC>& c) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(c.v[0], c.v[1]), b = __floats2bfloat162_rn(c.v[2], c.v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<const unsigned*>(&a);
        raw.y = *reinterpret_cast<const unsigned*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    } else if constexpr (VEC == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(c.v[0], c.v[1]);
    else *p = __float2bfloat16_rn(c.v[0]);
}
template <int VEC> __device__ __forceinline__ Cols<VEC> zero_cols() {
    Cols<VEC> c;
#pragma unroll
    for (int e = 0; e < VEC; ++e) c.v[e] = 0.f;
    return c;
}

// VEC columns of row t, planes added up (bfloat16 rows have one plane: without a loop behind every load, a thread's loads
// go out together)
template <int VEC, typename TI>
__device__ __forceinline__ Cols<VEC> row_cols(const ConvInput& p, long long t, int c) {
    const TI* src = reinterpret_cast<const TI*>(p.proj) + t * p.ld + c;
    Cols<VEC> x = load_cols<VEC>(src);
    if constexpr (sizeof(TI) == sizeof(float)) {
        for (int s = 1; s < p.splits; ++s) {
            const Cols<VEC> y = load_cols<VEC>(src + s * p.plane);
#pragma unroll
            for (int e = 0; e < VEC; ++e) x.v[e] += y.v[e];
        }
    }
    return x;
}

// the input `rel` places from the portion's start (negative: from the state, zero for a fresh request)
template <int VEC, typename TI>
__device__ __forceinline__ Cols<VEC> conv_cols(const ConvInput& p, int start, int rel, int c, const float* st, bool fresh) {
    if (rel >= 0) return row_cols<VEC, TI>(p, (long long)start + rel, c);
    if (fresh || st == nullptr) return zero_cols<VEC>();
    return load_cols<VEC>(st + (size_t)(p.taps - 1 + rel) * p.C + c);
}

// VEC columns of the TOK rows from row t on, of which n are there (zeros behind them)
template <int VEC, typename TI>
__device__ __forceinline__ void rows_cols(const ConvInput& p, long long t, int n, int c, Cols<VEC> (&x)[TOK]) {
    if (n == TOK) {
#pragma unroll
        for (int i = 0; i < TOK; ++i) x[i] = row_cols<VEC, TI>(p, t + i, c);
    } else {
#pragma unroll
        for (int i = 0; i < TOK; ++i) x[i] = i < n ? row_cols<VEC, TI>(p, t + i, c) : zero_cols<VEC>();
    }
}

// The last TM inputs of VEC channels and their taps (taps < TM: the oldest places weigh nothing and hold zeros).
template <int VEC, int TM>
struct Window {
    Cols<VEC> in[TM];
    Cols<VEC> w[TM];
    template <typename TI>
    __device__ __forceinline__ void open(const ConvInput& p, int start, int r0, int c, const float* st, bool fresh) {
        const int off = TM - p.taps;
#pragma unroll
        for (int j = 0; j < TM; ++j) w[j] = j >= off ? load_cols<VEC>(p.w + (size_t)(j - off) * p.C + c) : zero_cols<VEC>();
        // before the first push: the inputs r0 - (TM - 1) .. r0 - 1 lie in places 1 .. TM - 1
        in[0] = zero_cols<VEC>();
        if (r0 >= TM - 1) {                             // (all of them inside the portion: loads without conditions)
#pragma unroll
            for (int j = 1; j < TM; ++j) in[j] = row_cols<VEC, TI>(p, (long long)start + r0 - TM + j, c);
            return;
        }
#pragma unroll
        for (int j = 1; j < TM; ++j)
            in[j] = j > off ? conv_cols<VEC, TI>(p, start, r0 - TM + j, c, st, fresh) : zero_cols<VEC>();
    }
    __device__ __forceinline__ Cols<VEC> push(const Cols<VEC>& x) {
#pragma unroll
        for (int j = 0; j + 1 < TM; ++j) in[j] = in[j + 1];
        in[TM - 1] = x;
        Cols<VEC> y;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < TM; ++j) acc = fmaf(w[j].v[e], in[j].v[e], acc);
            y.v[e] = acc;
        }
        return y;
    }
    // the last taps - 1 inputs as the request's state
    __device__ __forceinline__ void leave(const ConvInput& p, float* st, int c) const {
        const int off = TM - p.taps;
#pragma unroll
        for (int j = 1; j < TM; ++j)
            if (j > off) store_cols<VEC>(st + (size_t)(j - off - 1) * p.C + c, in[j]);
    }
};

struct StoreParams {
    ConvInput x;
    const int* positions;
    const float* table;        // [table_rows][rot / 2][2]
    const int* slot_mapping;
    void* q_out;               // [T][n_q][hd]
    void* extra_out;           // [T][n_extra]
    void* k_pages;             // [pages][n_k][page_size][hd]
    void* v_pages;             // [pages][n_k][page_size][dv]
    int n_q, n_k, hd, dv, rot, n_extra, page_size, table_rows, n_items;
    float extra_scale;
};

// A thread per item: a rotated pair of VEC-column runs of a head, VEC columns that pass unrotated (the rest of a q or k
// head, a v head), or VEC columns of the gate.
template <typename TI, typename T, int VEC, int TM>
__global__ void __launch_bounds__(NT) conv_rope_store_kernel(const StoreParams p) {
    grid_launch_dependents();
    const int item = blockIdx.x * NT + threadIdx.x;
    const int b = blockIdx.z;
    const int half = p.rot >> 1, qk = p.n_q + p.n_k;
    const int pair_items = half / VEC, head_items = pair_items + (p.hd - p.rot) / VEC;
    const int n_qk = qk * head_items, n_v = p.n_k * p.dv / VEC;
    grid_dependency_wait();
    const int start = p.x.q_start[b], len = p.x.q_start[b + 1] - start;
    const int r0 = blockIdx.y * TOK, n = min(len - r0, TOK);
    if (n <= 0 || item >= p.n_items) return;
    if (item >= n_qk + n_v) {                                   // the gate's columns take no part in the convolution
        const int c = (item - n_qk - n_v) * VEC;
        T* out = reinterpret_cast<T*>(p.extra_out);
        Cols<VEC> x[TOK];
        rows_cols<VEC, TI>(p.x, (long long)start + r0, n, p.x.C + c, x);
#pragma unroll
        for (int i = 0; i < TOK; ++i) {
            if (i >= n) break;
#pragma unroll
            for (int e = 0; e < VEC; ++e) x[i].v[e] = p.extra_scale / (1.f + expf(-x[i].v[e]));
            store_cols<VEC>(out + ((size_t)start + r0 + i) * p.n_extra + c, x[i]);
        }
        return;
    }
    // where this item's columns lie in the row and in their head
    int head, d0, c0, c1 = -1, kind;                            // kind: 0 q, 1 k, 2 v
    if (item < n_qk) {
        head = item / head_items;
        const int i = item - head * head_items;
        if (i < pair_items) { d0 = i * VEC; c1 = head * p.hd + d0 + half; }
        else d0 = p.rot + (i - pair_items) * VEC;
        c0 = head * p.hd + d0;
        kind = head < p.n_q ? 0 : 1;
        if (kind == 1) head -= p.n_q;
    } else {
        const int c = (item - n_qk) * VEC;
        head = c / p.dv;
        d0 = c - head * p.dv;
        c0 = qk * p.hd + c;
        kind = 2;
    }
    // where every token's angles and its place in the pages are: asked for ahead of the rows
    int pos[TOK], slots[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        pos[i] = c1 >= 0 && i < n ? p.positions[start + r0 + i] : 0;
        slots[i] = kind != 0 && i < n ? p.slot_mapping[start + r0 + i] : 0;
    }
    const bool fresh = p.x.fresh[b] != 0;
    float* st = p.x.state != nullptr ? p.x.state + (size_t)p.x.state_slot[b] * p.x.state_pitch : nullptr;
    Window<VEC, TM> wa, wb;
    wa.template open<TI>(p.x, start, r0, c0, st, fresh);
    if (c1 >= 0) wb.template open<TI>(p.x, start, r0, c1, st, fresh);
    Cols<VEC> xa[TOK], xb[TOK];
    rows_cols<VEC, TI>(p.x, (long long)start + r0, n, c0, xa);
    if (c1 >= 0) rows_cols<VEC, TI>(p.x, (long long)start + r0, n, c1, xb);
    float2 cs[TOK][VEC];
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        (void)TL_CHECK(pos[i] >= 0 && pos[i] < p.table_rows, TL_DBG_POSITION);
        const int row = pos[i] < 0 ? 0 : (pos[i] >= p.table_rows ? p.table_rows - 1 : pos[i]);
#pragma unroll
        for (int e = 0; e < VEC; ++e)
            cs[i][e] = c1 >= 0 ? *reinterpret_cast<const float2*>(p.table + (size_t)row * p.rot + 2 * (d0 + e)) : make_float2(0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        if (i >= n) break;
        const int t = start + r0 + i;
        Cols<VEC> ya = wa.push(xa[i]), yb;
        if (c1 >= 0) {
            yb = wb.push(xb[i]);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                const float u = ya.v[e], v = yb.v[e];
                ya.v[e] = u * cs[i][e].x - v * cs[i][e].y;
                yb.v[e] = v * cs[i][e].x + u * cs[i][e].y;
            }
        }
        T* dst;
        if (kind == 0) dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * p.n_q + head) * p.hd + d0;
        else {
            const int sm = slots[i];
            const int page = sm / p.page_size, slot = sm - page * p.page_size;
            if (!(TL_CHECK(sm >= 0, TL_DBG_SLOT) && tl_check_page(page))) continue;
            const size_t at = ((size_t)page * p.n_k + head) * p.page_size + slot;
            dst = kind == 1 ? reinterpret_cast<T*>(p.k_pages) + at * p.hd + d0 : reinterpret_cast<T*>(p.v_pages) + at * p.dv + d0;
        }
        store_cols<VEC>(dst, ya);
        if (c1 >= 0) store_cols<VEC>(dst + half, yb);
    }
    if (p.x.n_chunks == 1 && st != nullptr) {                   // nobody else reads or writes these channels' state
        wa.leave(p.x, st, c0);
        if (c1 >= 0) wb.leave(p.x, st, c1);
    }
}

// the state after a step with longer portions: every (request, channel) by one thread, reads before writes
template <typename TI>
__global__ void __launch_bounds__(NT) conv_state_kernel(const ConvInput p) {
    grid_launch_dependents();
    grid_dependency_wait();
    const int c = blockIdx.x * NT + threadIdx.x, b = blockIdx.y;
    if (c >= p.C) return;
    const int start = p.q_start[b], len = p.q_start[b + 1] - start;
    if (len <= 0) return;
    const bool fresh = p.fresh[b] != 0;
    float* st = p.state + (size_t)p.state_slot[b] * p.state_pitch;
    float keep[MAX_TAPS - 1];
#pragma unroll
    for (int r = 0; r < MAX_TAPS - 1; ++r)
        keep[r] = r < p.taps - 1 ? conv_cols<1, TI>(p, start, len - (p.taps - 1) + r, c, st, fresh).v[0] : 0.f;
#pragma unroll
    for (int r = 0; r < MAX_TAPS - 1; ++r)
        if (r < p.taps - 1) st[(size_t)r * p.C + c] = keep[r];
}

struct DeltaParams {
    ConvInput x;
    float* q;                // [T][n_qk]
    float* k;                // [T][n_qk]
    void* v;                 // [T][n_v]
    void* small;             // [T][n_small]
    void* low;               // [T][low_pad]
    int heads, hd, n_qk, n_v, n_small, n_low, low_pad, v_units, n_units;
    float q_scale, unit_eps;
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }

constexpr int UNIT = 128;          // columns of a unit that is no head

// A warp per unit: a head of q or of k, UNIT columns of v, or UNIT columns of what follows.  A lane owns IT runs of VEC
// columns, 32 VEC apart.
template <typename TI, typename T, int VEC, int IT, int TM>
__global__ void __launch_bounds__(NT) delta_prep_kernel(const DeltaParams p) {
    grid_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int unit = blockIdx.x * (NT / 32) + (threadIdx.x >> 5), b = blockIdx.z;
    grid_dependency_wait();
    const int start = p.x.q_start[b], len = p.x.q_start[b + 1] - start;
    const int r0 = blockIdx.y * TOK, n = min(len - r0, TOK);
    if (n <= 0 || unit >= p.n_units) return;
    if (unit >= 2 * p.heads + p.v_units) {                       // the columns behind the convolution: [small | low, padded]
        const int base = (unit - 2 * p.heads - p.v_units) * UNIT;
        for (int e = lane; e < UNIT; e += 32) {
            const int c = base + e;
            if (c >= p.n_small + p.low_pad) break;
            Cols<1> x[TOK];
            rows_cols<1, TI>(p.x, (long long)start + r0, c < p.n_small + p.n_low ? n : 0, p.x.C + c, x);
#pragma unroll
            for (int i = 0; i < TOK; ++i) {
                if (i >= n) break;
                const size_t t = (size_t)start + r0 + i;
                if (c < p.n_small) reinterpret_cast<T*>(p.small)[t * p.n_small + c] = from_float<T>(x[i].v[0]);
                else reinterpret_cast<T*>(p.low)[t * p.low_pad + (c - p.n_small)] = from_float<T>(x[i].v[0]);
            }
        }
        return;
    }
    const bool is_v = unit >= 2 * p.heads;
    const int c_lo = is_v ? 2 * p.n_qk + (unit - 2 * p.heads) * UNIT : unit * p.hd;
    const int width = is_v ? min(UNIT, p.n_v - (unit - 2 * p.heads) * UNIT) : p.hd;
    const bool fresh = p.x.fresh[b] != 0;
    float* st = p.x.state != nullptr ? p.x.state + (size_t)p.x.state_slot[b] * p.x.state_pitch : nullptr;
    Window<VEC, TM> win[IT];
    bool mine[IT];
#pragma unroll
    for (int it = 0; it < IT; ++it) {
        const int d = (it * 32 + lane) * VEC;
        mine[it] = d < width;
        if (mine[it]) win[it].template open<TI>(p.x, start, r0, c_lo + d, st, fresh);
    }
    const bool is_q = unit < p.heads;
    const float scale = is_q ? p.q_scale : 1.f;
    float* qk_out = is_q ? p.q + (size_t)unit * p.hd : p.k + (size_t)(unit - p.heads) * p.hd;
    Cols<VEC> y[IT][TOK];
#pragma unroll
    for (int it = 0; it < IT; ++it)
        rows_cols<VEC, TI>(p.x, (long long)start + r0, mine[it] ? n : 0, c_lo + (it * 32 + lane) * VEC, y[it]);
    float ssq[TOK];
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        ssq[i] = 0.f;
        if (i < n) {
#pragma unroll
            for (int it = 0; it < IT; ++it) {
                if (!mine[it]) continue;
                y[it][i] = win[it].push(y[it][i]);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    const float a = silu_f(y[it][i].v[e]);
                    y[it][i].v[e] = a;
                    ssq[i] = fmaf(a, a, ssq[i]);
                }
            }
        }
    }
    if (!is_v) {
#pragma unroll
        for (int i = 0; i < TOK; ++i) ssq[i] = rsqrtf(warp_sum(ssq[i]) + p.unit_eps) * scale;
    }
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
        if (i >= n) break;
        const size_t t = (size_t)start + r0 + i;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            if (!mine[it]) continue;
            const int d = (it * 32 + lane) * VEC;
            if (is_v) store_cols<VEC>(reinterpret_cast<T*>(p.v) + t * p.n_v + (c_lo - 2 * p.n_qk) + d, y[it][i]);
            else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[it][i].v[e] *= ssq[i];
                store_cols<VEC>(qk_out + t * p.n_qk + d, y[it][i]);
            }
        }
    }
    if (p.x.n_chunks == 1 && st != nullptr) {
#pragma unroll
        for (int it = 0; it < IT; ++it)
            if (mine[it]) win[it].leave(p.x, st, c_lo + (it * 32 + lane) * VEC);
    }
}

template <typename TI>
__global__ void __launch_bounds__(256) channel_decay_kernel(const TI* __restrict__ z, long long ldz, const float* __restrict__ rate,
                                                            const float* __restrict__ bias, float* __restrict__ out, int width, int dk) {
    grid_launch_dependents();
    grid_dependency_wait();
    const size_t t = blockIdx.x;
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= width) return;
    const float a = to_float(z[t * ldz + c]) + bias[c];
    out[t * width + c] = expf(-rate[c / dk] * (a > 20.f ? a : log1pf(expf(a))));
}

int launch_state(const ConvInput& x, int in_dtype, int n_seqs, cudaStream_t s) {
    const dim3 grid((x.C + NT - 1) / NT, n_seqs);
    return in_dtype == TL_F32 ? (int)tl_launch(conv_state_kernel<float>, grid, dim3(NT), 0, s, x)
                              : (int)tl_launch(conv_state_kernel<__nv_bfloat16>, grid, dim3(NT), 0, s, x);
}

bool good_input(const ConvInput& x, int in_dtype, int n_seqs, int max_q_len) {
    return (x.splits == 1 || in_dtype == TL_F32) && x.taps >= 1 && x.taps <= MAX_TAPS && x.splits >= 1 && n_seqs <= 65535 && max_q_len > 0 && x.n_chunks <= 65535 &&
           (x.taps == 1 || x.state != nullptr);
}

// whether rows, taps and state may be read so many columns at a time (column offsets are the caller's to check)
bool vector_input(const ConvInput& x, int in_dtype, int vec) {
    const uintptr_t a = reinterpret_cast<uintptr_t>(x.proj), w = reinterpret_cast<uintptr_t>(x.w), st = reinterpret_cast<uintptr_t>(x.state);
    return x.C % vec == 0 && x.ld % vec == 0 && x.plane % vec == 0 && a % ((in_dtype == TL_F32 ? 4 : 2) * vec) == 0 && w % (4 * vec) == 0 &&
           x.state_pitch % vec == 0 && st % (4 * vec) == 0;
}

}  // namespace

// proj: [splits][n_tokens] rows of pitch ld (elements of in_dtype), planes `plane` apart, columns [q heads | k heads | v heads |
// extra]; w: float32 [taps][q, k and v columns]; state: float32 rows of pitch state_pitch per slot, [taps - 1][columns] each (null
// with one tap); table: float32 [table_rows, rot / 2, 2]; q_out [n_tokens, n_q, hd], extra_out [n_tokens, n_extra] and pages
// ([pages, n_k, page_size, hd] and [.., dv]) of dtype.
extern "C" int tl_conv_rope_store(const void* proj, int in_dtype, int splits, long long plane, long long ld, const float* w, int taps,
                                  float* state, long long state_pitch, const int* q_start, const int* state_slot, const int* fresh,
                                  const int* positions, const float* table, const int* slot_mapping, void* q_out, void* extra_out,
                                  void* k_pages, void* v_pages, int dtype, int n_tokens, int n_seqs, int max_q_len, int n_q, int n_k,
                                  int hd, int dv, int rot, int n_extra, float extra_scale, int page_size, int table_rows, void* stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return TL_OK;
    if (n_q <= 0 || n_k <= 0 || hd <= 0 || dv <= 0 || rot < 0 || (rot & 1) || rot > hd || n_extra < 0 || page_size <= 0 || table_rows <= 0)
        return TL_BAD_SIZE;
    if (k_pages == nullptr || v_pages == nullptr || slot_mapping == nullptr || (n_extra > 0 && extra_out == nullptr)) return TL_BAD_SIZE;
    StoreParams p;
    p.x.proj = proj; p.x.splits = splits; p.x.plane = plane; p.x.ld = ld; p.x.w = w; p.x.state = taps > 1 ? state : nullptr;
    p.x.state_pitch = taps > 1 ? state_pitch : 0; p.x.q_start = q_start; p.x.state_slot = state_slot; p.x.fresh = fresh;
    p.x.C = (n_q + n_k) * hd + n_k * dv; p.x.taps = taps; p.x.n_chunks = (max_q_len + TOK - 1) / TOK;
    if (!good_input(p.x, in_dtype, n_seqs, max_q_len)) return TL_BAD_SIZE;
    p.positions = positions; p.table = table; p.slot_mapping = slot_mapping; p.q_out = q_out; p.extra_out = extra_out;
    p.k_pages = k_pages; p.v_pages = v_pages; p.n_q = n_q; p.n_k = n_k; p.hd = hd; p.dv = dv; p.rot = rot; p.n_extra = n_extra;
    p.page_size = page_size; p.table_rows = table_rows; p.extra_scale = extra_scale;
    // (two columns a thread: with more, a rotated pair's windows cost the registers of a third warp; more than four taps
    // go one column at a time)
    const bool vec = taps <= 4 && vector_input(p.x, in_dtype, 2) && (rot / 2) % 2 == 0 && hd % 2 == 0 && dv % 2 == 0 && n_extra % 2 == 0 &&
                     aligned16(q_out) && aligned16(extra_out) && aligned16(k_pages) && aligned16(v_pages) && aligned16(table);
    const int V = vec ? 2 : 1;
    const long long items = (long long)(n_q + n_k) * (rot / 2 / V + (hd - rot) / V) + (long long)n_k * dv / V + n_extra / V;
    if (items > (1ll << 30)) return TL_BAD_SIZE;
    p.n_items = (int)items;
    const dim3 grid((p.n_items + NT - 1) / NT, p.x.n_chunks, n_seqs), block(NT);
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
#define TL_STORE(TI, T, VEC, TM) tl_launch(conv_rope_store_kernel<TI, T, VEC, TM>, grid, block, 0, s, p)
#define TL_STORE_PICK(TI, T)                                                                                   \
    e = vec ? TL_STORE(TI, T, 2, 4)                                                                            \
            : (taps <= 4 ? TL_STORE(TI, T, 1, 4) : TL_STORE(TI, T, 1, MAX_TAPS))
    if (in_dtype == TL_F32 && dtype == TL_F32) TL_STORE_PICK(float, float);
    else if (in_dtype == TL_F32 && dtype == TL_BF16) TL_STORE_PICK(float, __nv_bfloat16);
    else if (in_dtype == TL_BF16 && dtype == TL_BF16) TL_STORE_PICK(__nv_bfloat16, __nv_bfloat16);
    else return TL_BAD_DTYPE;
#undef TL_STORE_PICK
#undef TL_STORE
    if (e != cudaSuccess) return (int)e;
    return p.x.n_chunks > 1 && p.x.state != nullptr ? launch_state(p.x, in_dtype, n_seqs, s) : TL_OK;
}

// proj as above with columns [q heads | k heads | v | small | low | ...]; w: float32 [taps][2 * heads * hd + n_v]; q, k: float32
// [n_tokens][heads * hd]; v [n_tokens][n_v], small [n_tokens][n_small], low [n_tokens][low_pad] of dtype (low null with n_low 0).
extern "C" int tl_delta_prep(const void* proj, int in_dtype, int splits, long long plane, long long ld, const float* w, int taps,
                             float* state, long long state_pitch, const int* q_start, const int* state_slot, const int* fresh, float* q,
                             float* k, void* v, void* small, void* low, int dtype, int n_tokens, int n_seqs, int max_q_len, int heads,
                             int hd, int n_v, int n_small, int n_low, int low_pad, float q_scale, float unit_eps, void* stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return TL_OK;
    if (heads <= 0 || hd <= 0 || hd > 256 || n_v <= 0 || n_small < 0 || n_low < 0 || low_pad < n_low) return TL_BAD_SIZE;
    if ((n_small > 0 && small == nullptr) || (n_low > 0 && low == nullptr)) return TL_BAD_SIZE;
    DeltaParams p;
    p.x.proj = proj; p.x.splits = splits; p.x.plane = plane; p.x.ld = ld; p.x.w = w; p.x.state = taps > 1 ? state : nullptr;
    p.x.state_pitch = taps > 1 ? state_pitch : 0; p.x.q_start = q_start; p.x.state_slot = state_slot; p.x.fresh = fresh;
    p.x.C = 2 * heads * hd + n_v; p.x.taps = taps; p.x.n_chunks = (max_q_len + TOK - 1) / TOK;
    if (!good_input(p.x, in_dtype, n_seqs, max_q_len)) return TL_BAD_SIZE;
    p.q = q; p.k = k; p.v = v; p.small = small; p.low = low; p.heads = heads; p.hd = hd; p.n_qk = heads * hd; p.n_v = n_v;
    p.n_small = n_small; p.n_low = n_low; p.low_pad = n_low > 0 ? low_pad : 0; p.q_scale = q_scale; p.unit_eps = unit_eps;
    p.v_units = (n_v + UNIT - 1) / UNIT;
    p.n_units = 2 * heads + p.v_units + (n_small + p.low_pad + UNIT - 1) / UNIT;
    const bool vec = taps <= 4 && vector_input(p.x, in_dtype, 4) && hd % 4 == 0 && n_v % 4 == 0 && aligned16(q) && aligned16(k) && aligned16(v);
    const dim3 grid((p.n_units + NT / 32 - 1) / (NT / 32), p.x.n_chunks, n_seqs), block(NT);
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
#define TL_PREP(TI, T, VEC, IT, TM) tl_launch(delta_prep_kernel<TI, T, VEC, IT, TM>, grid, block, 0, s, p)
#define TL_PREP_PICK(TI, T)                                                                                    \
    e = vec ? (hd <= 128 ? TL_PREP(TI, T, 4, 1, 4) : TL_PREP(TI, T, 4, 2, 4))                                  \
            : (taps <= 4 ? TL_PREP(TI, T, 1, 8, 4) : TL_PREP(TI, T, 1, 8, MAX_TAPS))
    if (in_dtype == TL_F32 && dtype == TL_F32) TL_PREP_PICK(float, float);
    else if (in_dtype == TL_F32 && dtype == TL_BF16) TL_PREP_PICK(float, __nv_bfloat16);
    else if (in_dtype == TL_BF16 && dtype == TL_BF16) TL_PREP_PICK(__nv_bfloat16, __nv_bfloat16);
    else return TL_BAD_DTYPE;
#undef TL_PREP_PICK
#undef TL_PREP
    if (e != cudaSuccess) return (int)e;
    return p.x.n_chunks > 1 && p.x.state != nullptr ? launch_state(p.x, in_dtype, n_seqs, s) : TL_OK;
}

// z: [n_tokens] rows of pitch ldz (elements of in_dtype), `width` columns used; rate: float32 [width / dk]; bias: float32 [width];
// out: float32 [n_tokens][width] = exp(-rate softplus(z + bias)).
extern "C" int tl_channel_decay(const void* z, int in_dtype, long long ldz, const float* rate, const float* bias, float* out, int n_tokens,
                                int width, int dk, void* stream) {
    if (n_tokens <= 0) return TL_OK;
    if (width <= 0 || dk <= 0 || width % dk != 0 || width > 65535 * 256) return TL_BAD_SIZE;
    const dim3 grid(n_tokens, (width + 255) / 256), block(256);
    cudaStream_t s = (cudaStream_t)stream;
    if (in_dtype == TL_F32) return (int)tl_launch(channel_decay_kernel<float>, grid, block, 0, s, (const float*)z, ldz, rate, bias, out, width, dk);
    if (in_dtype == TL_BF16)
        return (int)tl_launch(channel_decay_kernel<__nv_bfloat16>, grid, block, 0, s, (const __nv_bfloat16*)z, ldz, rate, bias, out, width, dk);
    return TL_BAD_DTYPE;
}
