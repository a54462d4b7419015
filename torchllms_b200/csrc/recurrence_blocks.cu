// The matrix recurrences of matrix_state.cu for long portions: four tokens at a time.
//
// With S the state before a block of four tokens, g_t a token's decay (a number, or one per key coordinate acting on
// its own row of S), P_j = g_0 .. g_j, and D_ij = g_(i+1) .. g_j (so that P_j = g_0 D_0j):
//     d_j = (P_j k_j)^T S,   A_ij = (D_ij k_j) . k_i  (i < j),   u_j = beta_j (v_j - d_j - sum_(i<j) A_ij u_i)
//     o_j = (P_j q_j)^T S + sum_(i<=j) B_ij u_i,                 B_ij = (D_ij q_j) . k_i
//     S  <- P_3 S + sum_i (D_i3 k_i) u_i^T
// which is the token-by-token rule written out (no division, no approximation: only the order of additions differs);
// for the fixed decay u_j = v_j.  The sums over the key size that a block needs are all taken from one and the same S:
// one round of shuffles for four tokens instead of four rounds one after the other.
//
// A CTA of 4 warps per (4 * 32 / KS * NC columns, head, request).  A warp's lanes are 32 / KS groups of NC columns x KS
// slices of the key size: lane (group, s) keeps S[s R + r][its NC columns], r < R, in registers, in pairs of neighbouring
// r (fma.rn.f32x2).  16 tokens are fetched at a time; a warp turns the four of its own block into P_j k_j, P_j q_j, D_i3 k_i and
// P_3 (rows in shared memory, slices padded so that they start in different banks) and the scalars A, B, beta; then
// all warps walk the four blocks while the next 16 tokens are on their way.  All arithmetic is float32.
#include "common.cuh"

namespace {

constexpr int NT = 128, BLOCK = 4, CHUNK = 16, NC = 2;

enum Decay : int { FIXED = 0, HEAD = 1, CHANNEL_DECAYS = 3 };

struct BlocksParams {
    const float* q;          // [T][G * dk]
    const float* k;          // [T][G * dk]
    const void* v;           // [T] rows of pitch ldv, H * dv columns
    long long ldv;
    const void* beta;        // [T] rows of pitch ldg, H columns (delta rule)
    const void* gate;        // [T] rows of pitch ldz, H columns (a decay per head)
    long long ldg, ldz;
    const float* g;          // [T][H * dk]: decays per channel
    const float* decay;      // [H]: the fixed decay, or exp(A_log)
    const float* decay_bias; // [H]
    float* state;            // [slots] rows of pitch state_pitch, each [H][dv][dk]
    long long state_pitch;
    const int* q_start;
    const int* state_slot;
    const int* fresh;
    float* out;              // [T][H * dv]
    int H, G, dk, dv;
};

typedef unsigned long long pair_t;         // two floats

__device__ __forceinline__ pair_t pack2(float lo, float hi) {
    pair_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpack2(pair_t p) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p));
    return r;
}
__device__ __forceinline__ pair_t fma2(pair_t a, pair_t b, pair_t c) {
    pair_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ pair_t mul2(pair_t a, pair_t b) {
    pair_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ ulonglong2 row4(const float* p) { return *reinterpret_cast<const ulonglong2*>(p); }

// 16 values over the W lanes of a group: lane s of the group ends with the sums of values s * (16 / W) ... in v[0] ... (of a
// whole warp: with sum s / 2)
template <int W>
__device__ __forceinline__ void reduce_scatter(float (&v)[16], int lane) {
#pragma unroll
    for (int mask = W / 2, m = 8; mask >= 1; mask >>= 1, m >>= 1) {
        const bool up = (lane & mask) != 0;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (i >= m) break;
            const float send = up ? v[i] : v[i + m], keep = up ? v[i + m] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
        }
    }
    if (W == 32) v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
}

template <int R, int KS, int MODE, typename TV>
__global__ void __launch_bounds__(NT) recurrence_blocks_kernel(const BlocksParams p) {
    extern __shared__ __align__(16) float smem[];
    grid_launch_dependents();
    constexpr bool DELTA = MODE != FIXED;
    constexpr int SLOT = R + 4;                          // a slice in shared memory
    constexpr int PITCH = KS * SLOT;
    constexpr int COLS = 4 * (32 / KS) * NC;             // columns of a CTA
    constexpr int XN = (KS * R + 31) / 32;               // coordinates of a row that a lane brings
    constexpr int V_EACH = (CHUNK * COLS + NT - 1) / NT;
    constexpr int M = 16 / KS;                           // sums that a lane is left with
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int s = lane & (KS - 1);
    const int h = blockIdx.y, b = blockIdx.z;
    const int jl = (warp * (32 / KS) + lane / KS) * NC, j0 = blockIdx.x * COLS + jl;
    const int hq = h / (p.H / p.G);
    float* skp = smem;                                  // [CHUNK][PITCH]: P_j k_j (delta rule)
    float* sqp = skp + (DELTA ? CHUNK * PITCH : 0);     // [CHUNK][PITCH]: P_j q_j
    float* skn = sqp + CHUNK * PITCH;                   // [CHUNK][PITCH]: D_i3 k_i
    float* sp = skn + CHUNK * PITCH;                    // [CHUNK / BLOCK][PITCH]: P_3
    float* sv = sp + CHUNK / BLOCK * PITCH;             // [CHUNK][COLS]
    float* sab = sv + CHUNK * COLS;                     // [CHUNK][8]: A_0j A_1j A_2j beta_j B_0j B_1j B_2j B_3j (B_ij = 0 for i > j)
    for (int i = threadIdx.x; i < CHUNK * 8; i += NT) sab[i] = 0.f;
    grid_dependency_wait();
    const int start = p.q_start[b], len = p.q_start[b + 1] - start;
    if (len <= 0) return;
    float* st = p.state + (size_t)p.state_slot[b] * p.state_pitch + ((size_t)h * p.dv + j0) * p.dk;
    const bool fresh = p.fresh[b] != 0;
    pair_t S[NC][R / 2];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int r = 0; r < R; r += 2) {
            const int i = s * R + r;
            const bool in = !fresh && j0 + c < p.dv;
            S[c][r / 2] = pack2(in && i < p.dk ? st[(size_t)c * p.dk + i] : 0.f, in && i + 1 < p.dk ? st[(size_t)c * p.dk + i + 1] : 0.f);
        }
    const float fixed = MODE == FIXED ? p.decay[h] : 0.f, rate = MODE == HEAD ? p.decay[h] : 0.f, dbias = MODE == HEAD ? p.decay_bias[h] : 0.f;
    const TV* v = reinterpret_cast<const TV*>(p.v);
    const int qk_row = p.G * p.dk;
    float fq[BLOCK][XN], fk[BLOCK][XN], fd[MODE == CHANNEL_DECAYS ? BLOCK : 1][XN], fv[V_EACH], fa = 0.f, fb = 0.f;
    // the rows of the 16 tokens from t0 on, into registers: a warp brings the four tokens of its block (past the portion's
    // end: zeros, and decays of one)
    auto fetch = [&](int t0) {
        const int n = min(len - t0, CHUNK);
#pragma unroll
        for (int w = 0; w < BLOCK; ++w) {
            const int tt = warp * BLOCK + w;
            const size_t t = (size_t)(start + t0 + tt);
#pragma unroll
            for (int it = 0; it < XN; ++it) {
                const int d = lane + 32 * it;
                const bool in = tt < n && d < p.dk;
                fq[w][it] = in ? p.q[t * qk_row + (size_t)hq * p.dk + d] : 0.f;
                fk[w][it] = in ? p.k[t * qk_row + (size_t)hq * p.dk + d] : 0.f;
                if (MODE == CHANNEL_DECAYS) fd[w][it] = in ? p.g[(t * p.H + h) * p.dk + d] : 1.f;
            }
        }
#pragma unroll
        for (int i = 0; i < V_EACH; ++i) {
            const int e = threadIdx.x + i * NT, tt = e / COLS, c = e - tt * COLS, col = blockIdx.x * COLS + c;
            fv[i] = (tt < n && col < p.dv) ? to_float(v[(size_t)(start + t0 + tt) * p.ldv + (size_t)h * p.dv + col]) : 0.f;
        }
        if (DELTA && lane < BLOCK && warp * BLOCK + lane < n) {
            const size_t t = (size_t)(start + t0 + warp * BLOCK + lane);
            if (MODE == HEAD) fa = to_float(reinterpret_cast<const TV*>(p.gate)[t * p.ldz + h]);
            fb = to_float(reinterpret_cast<const TV*>(p.beta)[t * p.ldg + h]);
        }
    };
    fetch(0);
    for (int t0 = 0; t0 < len; t0 += CHUNK) {
        const int n = min(len - t0, CHUNK);
        __syncthreads();                                // the tokens before have been used
        // ---- this warp's block from registers into shared memory
        float gs[BLOCK];                                // decays that are numbers
        if (MODE == HEAD) {
            const float a = fa + dbias;
            const float mine = warp * BLOCK + lane < n ? expf(-rate * (a > 20.f ? a : log1pf(expf(a)))) : 1.f;
#pragma unroll
            for (int w = 0; w < BLOCK; ++w) gs[w] = __shfl_sync(0xffffffffu, mine, w);
        } else if (MODE == FIXED) {
#pragma unroll
            for (int w = 0; w < BLOCK; ++w) gs[w] = warp * BLOCK + w < n ? fixed : 1.f;
        }
        float ab[16];                                   // A01 A02 A12 A03 A13 A23 | B00 B01 B11 B02 B12 B22 B03 B13 B23 B33
#pragma unroll
        for (int i = 0; i < 16; ++i) ab[i] = 0.f;
#pragma unroll
        for (int it = 0; it < XN; ++it) {
            const int d = lane + 32 * it;
            const int at = (d / R) * SLOT + (d & (R - 1));
            const float g0 = MODE == CHANNEL_DECAYS ? fd[0][it] : gs[0], g1 = MODE == CHANNEL_DECAYS ? fd[MODE == CHANNEL_DECAYS ? 1 : 0][it] : gs[1];
            const float g2 = MODE == CHANNEL_DECAYS ? fd[MODE == CHANNEL_DECAYS ? 2 : 0][it] : gs[2], g3 = MODE == CHANNEL_DECAYS ? fd[MODE == CHANNEL_DECAYS ? 3 : 0][it] : gs[3];
            const float k0 = fk[0][it], k1 = fk[1][it], k2 = fk[2][it], k3 = fk[3][it];
            const float q0 = fq[0][it], q1 = fq[1][it], q2 = fq[2][it], q3 = fq[3][it];
            const float p1 = g0 * g1, p2 = p1 * g2, p3 = p2 * g3;
            const float e01 = g1 * k0, e02 = g2 * e01, e03 = g3 * e02, e12 = g2 * k1, e13 = g3 * e12, e23 = g3 * k2;
            if (DELTA) {
                ab[0] = fmaf(k1, e01, ab[0]);
                ab[1] = fmaf(k2, e02, ab[1]);
                ab[2] = fmaf(k2, e12, ab[2]);
                ab[3] = fmaf(k3, e03, ab[3]);
                ab[4] = fmaf(k3, e13, ab[4]);
                ab[5] = fmaf(k3, e23, ab[5]);
            }
            ab[6] = fmaf(q0, k0, ab[6]);
            ab[7] = fmaf(q1, e01, ab[7]);
            ab[8] = fmaf(q1, k1, ab[8]);
            ab[9] = fmaf(q2, e02, ab[9]);
            ab[10] = fmaf(q2, e12, ab[10]);
            ab[11] = fmaf(q2, k2, ab[11]);
            ab[12] = fmaf(q3, e03, ab[12]);
            ab[13] = fmaf(q3, e13, ab[13]);
            ab[14] = fmaf(q3, e23, ab[14]);
            ab[15] = fmaf(q3, k3, ab[15]);
            if (d < KS * R) {
                const int row = warp * BLOCK * PITCH + at;
                if (DELTA) {
                    skp[row] = g0 * k0;
                    skp[row + PITCH] = p1 * k1;
                    skp[row + 2 * PITCH] = p2 * k2;
                    skp[row + 3 * PITCH] = p3 * k3;
                }
                sqp[row] = g0 * q0;
                sqp[row + PITCH] = p1 * q1;
                sqp[row + 2 * PITCH] = p2 * q2;
                sqp[row + 3 * PITCH] = p3 * q3;
                skn[row] = e03;
                skn[row + PITCH] = e13;
                skn[row + 2 * PITCH] = e23;
                skn[row + 3 * PITCH] = k3;
                sp[warp * PITCH + at] = p3;
            }
        }
        // the warp's 32 lanes hold parts of 16 sums: lane l ends with sum l / 2
        reduce_scatter<32>(ab, lane);
        {
            const int i = lane >> 1;
            int at;                                     // where sum i belongs
            if (i < 6) {                                // A_ij in the order 01 02 12 03 13 23
                const int jj = i < 1 ? 1 : i < 3 ? 2 : 3, ii = i < 1 ? 0 : i < 3 ? i - 1 : i - 3;
                at = jj * 8 + ii;
            } else {                                    // B_ij in the order 00 01 11 02 12 22 03 13 23 33
                const int x = i - 6, jj = x < 1 ? 0 : x < 3 ? 1 : x < 6 ? 2 : 3, ii = x - jj * (jj + 1) / 2;
                at = jj * 8 + 4 + ii;
            }
            if ((lane & 1) == 0) sab[warp * BLOCK * 8 + at] = ab[0];
            if (DELTA && lane < BLOCK) sab[(warp * BLOCK + lane) * 8 + 3] = warp * BLOCK + lane < n ? 1.f / (1.f + expf(-fb)) : 0.f;
        }
#pragma unroll
        for (int i = 0; i < V_EACH; ++i)
            if (threadIdx.x + i * NT < CHUNK * COLS) sv[threadIdx.x + i * NT] = fv[i];
        __syncthreads();
        if (t0 + CHUNK < len) fetch(t0 + CHUNK);        // in flight while these tokens are walked
        // ---- the blocks
        for (int w = 0; w * BLOCK < n; ++w) {
            pair_t d2[BLOCK][NC], o2[BLOCK][NC];
#pragma unroll
            for (int j = 0; j < BLOCK; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) d2[j][c] = o2[j][c] = 0ull;
#pragma unroll
            for (int r = 0; r < R / 4; ++r)
#pragma unroll
                for (int j = 0; j < BLOCK; ++j) {
                    const int row = (w * BLOCK + j) * PITCH + s * SLOT + 4 * r;
                    const ulonglong2 qv = row4(sqp + row);
#pragma unroll
                    for (int c = 0; c < NC; ++c) o2[j][c] = fma2(S[c][2 * r + 1], qv.y, fma2(S[c][2 * r], qv.x, o2[j][c]));
                    if (DELTA) {
                        const ulonglong2 kv = row4(skp + row);
#pragma unroll
                        for (int c = 0; c < NC; ++c) d2[j][c] = fma2(S[c][2 * r + 1], kv.y, fma2(S[c][2 * r], kv.x, d2[j][c]));
                    }
                }
            float sums[16];                             // d_jc at 2 j + c, o_jc at 8 + 2 j + c
#pragma unroll
            for (int j = 0; j < BLOCK; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float2 x = unpack2(d2[j][c]), y = unpack2(o2[j][c]);
                    sums[2 * j + c] = x.x + x.y;
                    sums[8 + 2 * j + c] = y.x + y.y;
                }
            reduce_scatter<KS>(sums, lane);             // lane s of a group holds sums s * M ... s * M + M - 1
            float u[BLOCK][NC];
#pragma unroll
            for (int j = 0; j < BLOCK; ++j) {
                const float2 vj = *reinterpret_cast<const float2*>(sv + (w * BLOCK + j) * COLS + jl);
                u[j][0] = vj.x;
                u[j][1] = vj.y;
            }
            if (DELTA) {
#pragma unroll
                for (int j = 0; j < BLOCK; ++j) {
                    const float4 a = *reinterpret_cast<const float4*>(sab + (w * BLOCK + j) * 8);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        const int i = 2 * j + c;
                        float x = u[j][c] - __shfl_sync(0xffffffffu, sums[i % M], i / M, KS);
                        if (j > 0) x = fmaf(-a.x, u[0][c], x);
                        if (j > 1) x = fmaf(-a.y, u[1][c], x);
                        if (j > 2) x = fmaf(-a.z, u[2][c], x);
                        u[j][c] = a.w * x;
                    }
                }
            }
            if (s * M >= 8) {                           // the lanes that hold o
#pragma unroll
                for (int i = 0; i < M; ++i) {
                    const int x = s * M + i - 8, j = x >> 1, c = x & 1;
                    const float4 bj = *reinterpret_cast<const float4*>(sab + (w * BLOCK + j) * 8 + 4);
                    float o = sums[i];
                    o = fmaf(bj.x, c ? u[0][1] : u[0][0], o);
                    o = fmaf(bj.y, c ? u[1][1] : u[1][0], o);
                    o = fmaf(bj.z, c ? u[2][1] : u[2][0], o);
                    o = fmaf(bj.w, c ? u[3][1] : u[3][0], o);
                    if (w * BLOCK + j < n && j0 + c < p.dv)
                        p.out[((size_t)(start + t0 + w * BLOCK + j) * p.H + h) * p.dv + j0 + c] = o;
                }
            }
            pair_t uu[BLOCK][NC];
#pragma unroll
            for (int j = 0; j < BLOCK; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) uu[j][c] = pack2(u[j][c], u[j][c]);
#pragma unroll
            for (int r = 0; r < R / 4; ++r) {
                const ulonglong2 pv = row4(sp + w * PITCH + s * SLOT + 4 * r);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    S[c][2 * r] = mul2(S[c][2 * r], pv.x);
                    S[c][2 * r + 1] = mul2(S[c][2 * r + 1], pv.y);
                }
#pragma unroll
                for (int j = 0; j < BLOCK; ++j) {
                    const ulonglong2 kv = row4(skn + (w * BLOCK + j) * PITCH + s * SLOT + 4 * r);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        S[c][2 * r] = fma2(kv.x, uu[j][c], S[c][2 * r]);
                        S[c][2 * r + 1] = fma2(kv.y, uu[j][c], S[c][2 * r + 1]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int r = 0; r < R; r += 2) {
            const int i = s * R + r;
            const float2 x = unpack2(S[c][r / 2]);
            if (j0 + c < p.dv && i < p.dk) st[(size_t)c * p.dk + i] = x.x;
            if (j0 + c < p.dv && i + 1 < p.dk) st[(size_t)c * p.dk + i + 1] = x.y;
        }
}

template <int R, int KS, int MODE, typename TV>
cudaError_t launch_blocks(const BlocksParams& p, int n_seqs, cudaStream_t s) {
    constexpr int PITCH = KS * (R + 4), COLS = 4 * (32 / KS) * NC;
    constexpr size_t smem = ((size_t)((MODE != FIXED ? 3 : 2) * CHUNK + CHUNK / BLOCK) * PITCH + CHUNK * COLS + CHUNK * 8) * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(recurrence_blocks_kernel<R, KS, MODE, TV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return tl_launch(recurrence_blocks_kernel<R, KS, MODE, TV>, dim3((p.dv + COLS - 1) / COLS, p.H, n_seqs), dim3(NT), smem, s, p);
}

template <int MODE, typename TV>
cudaError_t launch_sizes(const BlocksParams& p, int n_seqs, cudaStream_t s) {
    if (p.dk <= 32) return launch_blocks<8, 4, MODE, TV>(p, n_seqs, s);
    if (p.dk <= 64) return launch_blocks<8, 8, MODE, TV>(p, n_seqs, s);
    if (p.dk <= 128) return launch_blocks<8, 16, MODE, TV>(p, n_seqs, s);
    return launch_blocks<16, 16, MODE, TV>(p, n_seqs, s);
}

}  // namespace

// As tl_linear_recurrence for modes 0 and 1; mode 3: gate is float32 [n_tokens][heads * dk], the decays per channel themselves.
extern "C" int tl_recurrence_blocks(const float* q, const float* k, const void* v, int v_dtype, long long ldv, const void* beta,
                                    long long ldg, const void* gate, long long ldz, const float* decay, const float* decay_bias, float* state,
                                    long long state_pitch, const int* q_start, const int* state_slot, const int* fresh,
                                    float* out, int n_tokens, int n_seqs, int heads, int qk_heads, int dk, int dv, int mode, void* stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return TL_OK;
    if (heads <= 0 || qk_heads <= 0 || heads % qk_heads != 0 || dk <= 0 || dk > 256 || dv <= 0 || n_seqs > 65535 || heads > 65535)
        return TL_BAD_SIZE;
    if ((mode != FIXED && mode != HEAD && mode != CHANNEL_DECAYS) || (mode != CHANNEL_DECAYS && decay == nullptr)) return TL_BAD_SIZE;
    if (mode != FIXED && (beta == nullptr || gate == nullptr || (mode == HEAD && decay_bias == nullptr))) return TL_BAD_SIZE;
    BlocksParams p;
    p.q = q; p.k = k; p.v = v; p.ldv = ldv; p.beta = beta; p.gate = gate; p.ldg = ldg; p.ldz = ldz;
    p.g = mode == CHANNEL_DECAYS ? (const float*)gate : nullptr; p.decay = decay; p.decay_bias = decay_bias;
    p.state = state; p.state_pitch = state_pitch; p.q_start = q_start; p.state_slot = state_slot; p.fresh = fresh; p.out = out;
    p.H = heads; p.G = qk_heads; p.dk = dk; p.dv = dv;
    cudaStream_t s = (cudaStream_t)stream;
#define TL_BLOCKS(TV)                                                                                                \
    (int)(mode == FIXED ? launch_sizes<FIXED, TV>(p, n_seqs, s) : mode == HEAD ? launch_sizes<HEAD, TV>(p, n_seqs, s) \
                                                                               : launch_sizes<CHANNEL_DECAYS, TV>(p, n_seqs, s))
    if (v_dtype == TL_F32) return TL_BLOCKS(float);
    if (v_dtype == TL_BF16) return TL_BLOCKS(__nv_bfloat16);
#undef TL_BLOCKS
    return TL_BAD_DTYPE;
}
