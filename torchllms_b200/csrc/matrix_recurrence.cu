// Recurrences whose per-request state is a matrix per head: a dk x dv matrix S in float32 that every token updates and
// reads, o = S^T q, with
//     fixed decay:  S <- d_h S + k v^T
//     delta rule:   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T     (g: a number per head, or one per head and key
//                   coordinate, each acting on its own row of S)
// A state row holds S^T: [heads][dv][dk], a column's keys side by side.  All arithmetic is float32.
//
// Steps of short portions (decoding): recurrence_steps_kernel.  A warp owns STEP_COLS columns of a head, a lane four
// neighbouring keys of each (or 2 x 4): the state is read and written once, 16 bytes a lane, and the sums over the keys
// that a token needs (two per column, taken from the decayed state before its update, and k . q:
// o = S^T q + u (k . q)) are one round of shuffles.
//
// Steps with long portions: recurrence_blocks_kernel, four tokens at a time.  With S the state before a block, g_t a
// token's decay, P_j = g_0 .. g_j, and D_ij = g_(i+1) .. g_j (so that P_j = g_0 D_0j):
//     d_j = (P_j k_j)^T S,   A_ij = (D_ij k_j) . k_i  (i < j),   u_j = beta_j (v_j - d_j - sum_(i<j) A_ij u_i)
//     o_j = (P_j q_j)^T S + sum_(i<=j) B_ij u_i,                 B_ij = (D_ij q_j) . k_i
//     S  <- P_3 S + sum_i (D_i3 k_i) u_i^T
// which is the token-by-token rule written out (no division, no approximation: only the order of additions differs);
// for the fixed decay u_j = v_j.  The sums over the key size that a block needs are all taken from one and the same S:
// one round of shuffles for four tokens instead of four rounds one after the other.
//
// A CTA per (4 * 32 / KS * NC columns, head, request).  Four of its warps walk blocks: their lanes are 32 / KS groups of NC
// columns x KS slices of the key size, and lane (group, s) keeps S[s R + r][its NC columns], r < R, in registers, in pairs
// of neighbouring r (fma.rn.f32x2).  Four other warps prepare the next 16 tokens meanwhile: each turns the four tokens of a
// block into P_j k_j, P_j q_j, D_i3 k_i and P_3 (rows in shared memory, slices padded so that they start in different
// banks) and the scalars A, B, beta, while the tokens after those are on their way from global memory.
#include "common.cuh"

namespace {

constexpr int WALKERS = 128, NT = 256, BLOCK = 4, CHUNK = 16, NC = 2;      // (threads that walk; of a CTA)
constexpr int STEP_NT = 128, STEP_COLS = 8;

enum Decay : int { FIXED = 0, HEAD = 1, CHANNEL = 2 };

struct RecurrenceParams {
    const float* q;          // [T][G * dk]
    const float* k;          // [T][G * dk]
    const void* v;           // [T] rows of pitch ldv, H * dv columns
    long long ldv;
    const void* beta;        // [T] rows of pitch ldg, H columns (delta rule)
    const void* gate;        // [T] rows of pitch ldz, H or (steps, a decay per channel) H * dk columns: logits
    long long ldg, ldz;
    const float* g;          // [T][H * dk]: decays per channel (blocks)
    const float* decay;      // [H]: the fixed decay, or exp(A_log)
    const float* decay_bias; // [H] or [H * dk]
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

template <int R, int KS, int MODE>
struct BlocksLayout {
    static constexpr bool DELTA = MODE != FIXED;
    static constexpr int SLOT = R + 4;                   // a slice in shared memory
    static constexpr int PITCH = KS * SLOT;
    static constexpr int COLS = (WALKERS / 32) * (32 / KS) * NC;      // columns of a CTA
    // one buffer of 16 tokens, in floats
    static constexpr int KP = 0;                                     // [CHUNK][PITCH]: P_j k_j (delta rule)
    static constexpr int QP = KP + (DELTA ? CHUNK * PITCH : 0);      // [CHUNK][PITCH]: P_j q_j
    static constexpr int KN = QP + CHUNK * PITCH;                    // [CHUNK][PITCH]: D_i3 k_i
    static constexpr int P3 = KN + CHUNK * PITCH;                    // [CHUNK / BLOCK][PITCH]
    static constexpr int V = P3 + CHUNK / BLOCK * PITCH;             // [CHUNK][COLS]
    static constexpr int AB = V + CHUNK * COLS;                      // [CHUNK][8]: A_0j A_1j A_2j beta_j B_0j B_1j B_2j B_3j (B_ij = 0 for i > j)
    static constexpr int SIZE = AB + CHUNK * 8;
};

// The warps that prepare: tokens from global memory into registers, a chunk ahead, and from there into a buffer.
template <int R, int KS, int MODE, typename TV>
struct Preparer {
    using L = BlocksLayout<R, KS, MODE>;
    static constexpr int XN = (KS * R + 31) / 32;        // coordinates of a row that a lane brings
    static constexpr int V_EACH = (CHUNK * L::COLS + WALKERS - 1) / WALKERS;
    float fq[BLOCK][XN], fk[BLOCK][XN], fd[MODE == CHANNEL ? BLOCK : 1][XN];
    TV fv[V_EACH], fa, fb;                               // (converted when they are used: a conversion would wait for the load)

    // the 16 tokens from t0 on: a warp brings the four of its block (past the portion's end: zeros, and decays of one)
    __device__ __forceinline__ void fetch(const RecurrenceParams& p, int start, int len, int t0, int tid, int h, int hq) {
        const int lane = tid & 31, warp = tid >> 5, n = min(len - t0, CHUNK), qk_row = p.G * p.dk;
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
                if (MODE == CHANNEL) fd[w][it] = in ? p.g[(t * p.H + h) * p.dk + d] : 1.f;
            }
        }
        const TV* v = reinterpret_cast<const TV*>(p.v);
#pragma unroll
        for (int i = 0; i < V_EACH; ++i) {
            const int e = tid + i * WALKERS, tt = e / L::COLS, c = e - tt * L::COLS, col = blockIdx.x * L::COLS + c;
            fv[i] = (tt < n && col < p.dv) ? v[(size_t)(start + t0 + tt) * p.ldv + (size_t)h * p.dv + col] : from_float<TV>(0.f);
        }
        if (L::DELTA && lane < BLOCK && warp * BLOCK + lane < n) {
            const size_t t = (size_t)(start + t0 + warp * BLOCK + lane);
            if (MODE == HEAD) fa = reinterpret_cast<const TV*>(p.gate)[t * p.ldz + h];
            fb = reinterpret_cast<const TV*>(p.beta)[t * p.ldg + h];
        }
    }

    __device__ __forceinline__ void put(const RecurrenceParams& p, float* buf, int n, int tid, int h) {
        const int lane = tid & 31, warp = tid >> 5;
        float gs[BLOCK];                                // decays that are numbers
        if (MODE == HEAD) {
            const float a = to_float(fa) + p.decay_bias[h];
            const float mine = lane < BLOCK && warp * BLOCK + lane < n ? expf(-p.decay[h] * (a > 20.f ? a : log1pf(expf(a)))) : 1.f;
#pragma unroll
            for (int w = 0; w < BLOCK; ++w) gs[w] = __shfl_sync(0xffffffffu, mine, w);
        } else if (MODE == FIXED) {
            const float d = p.decay[h];
#pragma unroll
            for (int w = 0; w < BLOCK; ++w) gs[w] = warp * BLOCK + w < n ? d : 1.f;
        }
        float ab[16];                                   // A01 A02 A12 A03 A13 A23 | B00 B01 B11 B02 B12 B22 B03 B13 B23 B33
#pragma unroll
        for (int i = 0; i < 16; ++i) ab[i] = 0.f;
#pragma unroll
        for (int it = 0; it < XN; ++it) {
            const int d = lane + 32 * it;
            constexpr int C = MODE == CHANNEL ? 1 : 0;
            const float g0 = C ? fd[0][it] : gs[0], g1 = C ? fd[C][it] : gs[1], g2 = C ? fd[2 * C][it] : gs[2], g3 = C ? fd[3 * C][it] : gs[3];
            const float k0 = fk[0][it], k1 = fk[1][it], k2 = fk[2][it], k3 = fk[3][it];
            const float q0 = fq[0][it], q1 = fq[1][it], q2 = fq[2][it], q3 = fq[3][it];
            const float p1 = g0 * g1, p2 = p1 * g2, p3 = p2 * g3;
            const float e01 = g1 * k0, e02 = g2 * e01, e03 = g3 * e02, e12 = g2 * k1, e13 = g3 * e12, e23 = g3 * k2;
            if (L::DELTA) {
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
                const int at = (d / R) * L::SLOT + (d & (R - 1)), row = warp * BLOCK * L::PITCH + at;
                if (L::DELTA) {
                    buf[L::KP + row] = g0 * k0;
                    buf[L::KP + row + L::PITCH] = p1 * k1;
                    buf[L::KP + row + 2 * L::PITCH] = p2 * k2;
                    buf[L::KP + row + 3 * L::PITCH] = p3 * k3;
                }
                buf[L::QP + row] = g0 * q0;
                buf[L::QP + row + L::PITCH] = p1 * q1;
                buf[L::QP + row + 2 * L::PITCH] = p2 * q2;
                buf[L::QP + row + 3 * L::PITCH] = p3 * q3;
                buf[L::KN + row] = e03;
                buf[L::KN + row + L::PITCH] = e13;
                buf[L::KN + row + 2 * L::PITCH] = e23;
                buf[L::KN + row + 3 * L::PITCH] = k3;
                buf[L::P3 + warp * L::PITCH + at] = p3;
            }
        }
        reduce_scatter<32>(ab, lane);                   // lane l ends with sum l / 2
        const int i = lane >> 1;
        int at;                                         // where sum i belongs
        if (i < 6) {                                    // A_ij in the order 01 02 12 03 13 23
            const int jj = i < 1 ? 1 : i < 3 ? 2 : 3, ii = i < 1 ? 0 : i < 3 ? i - 1 : i - 3;
            at = jj * 8 + ii;
        } else {                                        // B_ij in the order 00 01 11 02 12 22 03 13 23 33
            const int x = i - 6, jj = x < 1 ? 0 : x < 3 ? 1 : x < 6 ? 2 : 3, ii = x - jj * (jj + 1) / 2;
            at = jj * 8 + 4 + ii;
        }
        if ((lane & 1) == 0) buf[L::AB + warp * BLOCK * 8 + at] = ab[0];
        if (L::DELTA && lane < BLOCK) buf[L::AB + (warp * BLOCK + lane) * 8 + 3] = warp * BLOCK + lane < n ? 1.f / (1.f + expf(-to_float(fb))) : 0.f;
#pragma unroll
        for (int i2 = 0; i2 < V_EACH; ++i2)
            if (tid + i2 * WALKERS < CHUNK * L::COLS) buf[L::V + tid + i2 * WALKERS] = to_float(fv[i2]);
    }
};

template <int R, int KS, int MODE, typename TV>
__global__ void __launch_bounds__(NT) recurrence_blocks_kernel(const RecurrenceParams p) {
    extern __shared__ __align__(16) float smem[];
    using L = BlocksLayout<R, KS, MODE>;
    grid_launch_dependents();
    constexpr int M = 16 / KS;                           // sums that a lane is left with
    const int h = blockIdx.y, b = blockIdx.z, hq = h / (p.H / p.G);
    for (int i = threadIdx.x; i < 2 * CHUNK * 8; i += NT) smem[(i / (CHUNK * 8)) * L::SIZE + L::AB + i % (CHUNK * 8)] = 0.f;
    grid_dependency_wait();
    const int start = p.q_start[b], len = p.q_start[b + 1] - start;
    if (len <= 0) return;
    __syncthreads();                                     // the scalars' zeros are set
    const int n_chunks = (len + CHUNK - 1) / CHUNK;
    if (threadIdx.x >= WALKERS) {
        // ---- the warps that prepare stay one chunk ahead; both sides meet at one barrier per chunk
        const int tid = threadIdx.x - WALKERS;
        Preparer<R, KS, MODE, TV> prep;
        prep.fetch(p, start, len, 0, tid, h, hq);
        for (int c = 0; c < n_chunks; ++c) {
            prep.put(p, smem + (c & 1) * L::SIZE, min(len - c * CHUNK, CHUNK), tid, h);
            if (c + 1 < n_chunks) prep.fetch(p, start, len, (c + 1) * CHUNK, tid, h, hq);
            __syncthreads();
        }
        __syncthreads();
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int s = lane & (KS - 1);
    const int jl = (warp * (32 / KS) + lane / KS) * NC, j0 = blockIdx.x * L::COLS + jl;
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
    for (int chunk = 0; chunk < n_chunks; ++chunk) {
        __syncthreads();                                 // this chunk's buffer is filled, the other one may be filled again
        const float* buf = smem + (chunk & 1) * L::SIZE;
        const int t0 = chunk * CHUNK, n = min(len - t0, CHUNK);
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
                    const int row = (w * BLOCK + j) * L::PITCH + s * L::SLOT + 4 * r;
                    const ulonglong2 qv = row4(buf + L::QP + row);
#pragma unroll
                    for (int c = 0; c < NC; ++c) o2[j][c] = fma2(S[c][2 * r + 1], qv.y, fma2(S[c][2 * r], qv.x, o2[j][c]));
                    if (L::DELTA) {
                        const ulonglong2 kv = row4(buf + L::KP + row);
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
                const float2 vj = *reinterpret_cast<const float2*>(buf + L::V + (w * BLOCK + j) * L::COLS + jl);
                u[j][0] = vj.x;
                u[j][1] = vj.y;
            }
            if (L::DELTA) {
                float dj[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) dj[i] = __shfl_sync(0xffffffffu, sums[i % M], i / M, KS);
#pragma unroll
                for (int j = 0; j < BLOCK; ++j) {
                    const float4 a = *reinterpret_cast<const float4*>(buf + L::AB + (w * BLOCK + j) * 8);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        float x = u[j][c] - dj[2 * j + c];
                        if (j > 0) x = fmaf(-a.x, u[0][c], x);
                        if (j > 1) x = fmaf(-a.y, u[1][c], x);
                        if (j > 2) x = fmaf(-a.z, u[2][c], x);
                        u[j][c] = a.w * x;
                    }
                }
            }
            pair_t uu[BLOCK][NC];
#pragma unroll
            for (int j = 0; j < BLOCK; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) uu[j][c] = pack2(u[j][c], u[j][c]);
#pragma unroll
            for (int r = 0; r < R / 4; ++r) {
                const ulonglong2 pv = row4(buf + L::P3 + w * L::PITCH + s * L::SLOT + 4 * r);
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    S[c][2 * r] = mul2(S[c][2 * r], pv.x);
                    S[c][2 * r + 1] = mul2(S[c][2 * r + 1], pv.y);
                }
#pragma unroll
                for (int j = 0; j < BLOCK; ++j) {
                    const ulonglong2 kv = row4(buf + L::KN + (w * BLOCK + j) * L::PITCH + s * L::SLOT + 4 * r);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        S[c][2 * r] = fma2(kv.x, uu[j][c], S[c][2 * r]);
                        S[c][2 * r + 1] = fma2(kv.y, uu[j][c], S[c][2 * r + 1]);
                    }
                }
            }
            if (s * M >= 8) {                           // the lanes that hold o
#pragma unroll
                for (int i = 0; i < M; ++i) {
                    const int x = s * M + i - 8, j = x >> 1, c = x & 1;
                    const float4 bj = *reinterpret_cast<const float4*>(buf + L::AB + (w * BLOCK + j) * 8 + 4);
                    float o = sums[i];
                    o = fmaf(bj.x, c ? u[0][1] : u[0][0], o);
                    o = fmaf(bj.y, c ? u[1][1] : u[1][0], o);
                    o = fmaf(bj.z, c ? u[2][1] : u[2][0], o);
                    o = fmaf(bj.w, c ? u[3][1] : u[3][0], o);
                    if (w * BLOCK + j < n && j0 + c < p.dv)
                        p.out[((size_t)(start + t0 + w * BLOCK + j) * p.H + h) * p.dv + j0 + c] = o;
                }
            }
        }
    }
    __syncthreads();
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

// four keys of a column, or of a row of q, k or decays, from key i on (zeros past dk)
template <bool VEC>
__device__ __forceinline__ float4 keys4(const float* p, int i, int dk) {
    if (VEC) return i < dk ? *reinterpret_cast<const float4*>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(i < dk ? p[i] : 0.f, i + 1 < dk ? p[i + 1] : 0.f, i + 2 < dk ? p[i + 2] : 0.f, i + 3 < dk ? p[i + 3] : 0.f);
}
__device__ __forceinline__ float dot4(float4 a, float4 b, float c) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c)))); }

// VEC: keys come in fours (dk and the state's pitch are multiples of 4, rows aligned); IT: runs of 128 keys
template <int IT, bool VEC, int MODE, typename TV>
__global__ void __launch_bounds__(STEP_NT) recurrence_steps_kernel(const RecurrenceParams p) {
    grid_launch_dependents();
    constexpr bool DELTA = MODE != FIXED;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.y, b = blockIdx.z, hq = h / (p.H / p.G);
    const int j0 = (blockIdx.x * (STEP_NT / 32) + warp) * STEP_COLS;
    grid_dependency_wait();
    const int start = p.q_start[b], len = p.q_start[b + 1] - start;
    if (len <= 0 || j0 >= p.dv) return;
    float* st = p.state + (size_t)p.state_slot[b] * p.state_pitch + ((size_t)h * p.dv + j0) * p.dk;
    const bool fresh = p.fresh[b] != 0;
    const int n_cols = min(STEP_COLS, p.dv - j0);
    float4 S[STEP_COLS][IT];
#pragma unroll
    for (int c = 0; c < STEP_COLS; ++c)
#pragma unroll
        for (int it = 0; it < IT; ++it)
            S[c][it] = !fresh && c < n_cols ? keys4<VEC>(st + (size_t)c * p.dk, (it * 32 + lane) * 4, p.dk) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float rate = p.decay[h];                       // (the fixed decay itself in that mode)
    for (int i = 0; i < len; ++i) {
        const size_t t = (size_t)start + i;
        float4 q[IT], k[IT], g[IT];
        float vt = 0.f, beta = 1.f, gs = rate;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int d = (it * 32 + lane) * 4;
            q[it] = keys4<VEC>(p.q + (t * p.G + hq) * p.dk, d, p.dk);
            k[it] = keys4<VEC>(p.k + (t * p.G + hq) * p.dk, d, p.dk);
            if (MODE == CHANNEL) {
                float a[4];
                const TV* z = reinterpret_cast<const TV*>(p.gate) + t * p.ldz + (size_t)h * p.dk;
#pragma unroll
                for (int e = 0; e < 4; ++e) a[e] = d + e < p.dk ? to_float(z[d + e]) + p.decay_bias[(size_t)h * p.dk + d + e] : 0.f;
#pragma unroll
                for (int e = 0; e < 4; ++e) a[e] = expf(-rate * (a[e] > 20.f ? a[e] : log1pf(expf(a[e]))));
                g[it] = make_float4(a[0], a[1], a[2], a[3]);
            }
        }
        if (lane < n_cols) vt = to_float(reinterpret_cast<const TV*>(p.v)[t * p.ldv + (size_t)h * p.dv + j0 + lane]);
        if (DELTA) beta = 1.f / (1.f + expf(-to_float(reinterpret_cast<const TV*>(p.beta)[t * p.ldg + h])));
        if (MODE == HEAD) {
            const float a = to_float(reinterpret_cast<const TV*>(p.gate)[t * p.ldz + h]) + p.decay_bias[h];
            gs = expf(-rate * (a > 20.f ? a : log1pf(expf(a))));
        }
        float kq = 0.f;
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            kq = dot4(k[it], q[it], kq);
            if (MODE != CHANNEL) g[it] = make_float4(gs, gs, gs, gs);
        }
        kq = warp_sum(kq);
        float sums[16];                                  // S^T k of the columns, then S^T q
#pragma unroll
        for (int c = 0; c < STEP_COLS; ++c) {
            float dk_ = 0.f, dq_ = 0.f;
#pragma unroll
            for (int it = 0; it < IT; ++it) {
                S[c][it].x *= g[it].x;
                S[c][it].y *= g[it].y;
                S[c][it].z *= g[it].z;
                S[c][it].w *= g[it].w;
                if (DELTA) dk_ = dot4(S[c][it], k[it], dk_);
                dq_ = dot4(S[c][it], q[it], dq_);
            }
            sums[c] = dk_;
            sums[STEP_COLS + c] = dq_;
        }
        reduce_scatter<32>(sums, lane);                  // lane l holds sum l / 2
        const float dk_mine = __shfl_sync(0xffffffffu, sums[0], (2 * lane) & 31), dq_mine = __shfl_sync(0xffffffffu, sums[0], (2 * lane + 16) & 31);
        // lane c < STEP_COLS finishes column c
        const float u = DELTA ? beta * (vt - dk_mine) : vt;
        if (lane < n_cols) p.out[(t * p.H + h) * p.dv + j0 + lane] = fmaf(u, kq, dq_mine);
#pragma unroll
        for (int c = 0; c < STEP_COLS; ++c) {
            const float uc = __shfl_sync(0xffffffffu, u, c);
#pragma unroll
            for (int it = 0; it < IT; ++it) {
                S[c][it].x = fmaf(k[it].x, uc, S[c][it].x);
                S[c][it].y = fmaf(k[it].y, uc, S[c][it].y);
                S[c][it].z = fmaf(k[it].z, uc, S[c][it].z);
                S[c][it].w = fmaf(k[it].w, uc, S[c][it].w);
            }
        }
    }
#pragma unroll
    for (int c = 0; c < STEP_COLS; ++c)
#pragma unroll
        for (int it = 0; it < IT; ++it) {
            const int i = (it * 32 + lane) * 4;
            float* at = st + (size_t)c * p.dk + i;
            if (c >= n_cols || i >= p.dk) continue;
            if (VEC) *reinterpret_cast<float4*>(at) = S[c][it];
            else {
                at[0] = S[c][it].x;
                if (i + 1 < p.dk) at[1] = S[c][it].y;
                if (i + 2 < p.dk) at[2] = S[c][it].z;
                if (i + 3 < p.dk) at[3] = S[c][it].w;
            }
        }
}

template <int R, int KS, int MODE, typename TV>
cudaError_t launch_blocks(const RecurrenceParams& p, int n_seqs, cudaStream_t s) {
    using L = BlocksLayout<R, KS, MODE>;
    constexpr size_t smem = 2 * L::SIZE * sizeof(float);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(recurrence_blocks_kernel<R, KS, MODE, TV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return tl_launch(recurrence_blocks_kernel<R, KS, MODE, TV>, dim3((p.dv + L::COLS - 1) / L::COLS, p.H, n_seqs), dim3(NT), smem, s, p);
}

template <int MODE, typename TV>
cudaError_t launch_block_sizes(const RecurrenceParams& p, int n_seqs, cudaStream_t s) {
    if (p.dk <= 32) return launch_blocks<8, 4, MODE, TV>(p, n_seqs, s);
    if (p.dk <= 64) return launch_blocks<8, 8, MODE, TV>(p, n_seqs, s);
    if (p.dk <= 128) return launch_blocks<8, 16, MODE, TV>(p, n_seqs, s);
    return launch_blocks<16, 16, MODE, TV>(p, n_seqs, s);
}

template <int MODE, typename TV>
cudaError_t launch_steps(const RecurrenceParams& p, int n_seqs, cudaStream_t s) {
    constexpr int COLS = STEP_NT / 32 * STEP_COLS;
    const dim3 grid((p.dv + COLS - 1) / COLS, p.H, n_seqs), block(STEP_NT);
    const bool vec = p.dk % 4 == 0 && p.state_pitch % 4 == 0 && aligned16(p.state) && aligned16(p.q) && aligned16(p.k);
    if (p.dk <= 128)
        return vec ? tl_launch(recurrence_steps_kernel<1, true, MODE, TV>, grid, block, 0, s, p)
                   : tl_launch(recurrence_steps_kernel<1, false, MODE, TV>, grid, block, 0, s, p);
    return vec ? tl_launch(recurrence_steps_kernel<2, true, MODE, TV>, grid, block, 0, s, p)
               : tl_launch(recurrence_steps_kernel<2, false, MODE, TV>, grid, block, 0, s, p);
}

template <typename TV>
int launch_mode(const RecurrenceParams& p, int n_seqs, int mode, bool blocks, cudaStream_t s) {
    if (blocks)
        return (int)(mode == FIXED ? launch_block_sizes<FIXED, TV>(p, n_seqs, s) : mode == HEAD ? launch_block_sizes<HEAD, TV>(p, n_seqs, s)
                                                                                               : launch_block_sizes<CHANNEL, TV>(p, n_seqs, s));
    return (int)(mode == FIXED ? launch_steps<FIXED, TV>(p, n_seqs, s) : mode == HEAD ? launch_steps<HEAD, TV>(p, n_seqs, s)
                                                                                     : launch_steps<CHANNEL, TV>(p, n_seqs, s));
}

}  // namespace

// q, k: float32 [n_tokens][qk_heads * dk]; v: rows of pitch ldv, heads * dv columns; state: float32, per slot a row of
// pitch state_pitch holding [heads][dv][dk]; out: float32 [n_tokens][heads * dv].
// mode 0: decay is [heads], the fixed decay.  Otherwise the delta rule: beta are rows of pitch ldg with `heads` columns of
// logits (of v's dtype), decay is exp(A_log) per head.  mode 1: gate are rows of pitch ldz with `heads` columns and
// decay_bias [heads] the bias inside the softplus.  mode 2, a decay per channel: gate has heads * dk columns and decay_bias
// heads * dk numbers, or, with blocks != 0, gate is float32 [n_tokens][heads * dk], the decays themselves.
// blocks != 0: for steps with long portions, four tokens at a time.
extern "C" int tl_linear_recurrence(const float* q, const float* k, const void* v, int v_dtype, long long ldv, const void* beta,
                                    long long ldg, const void* gate, long long ldz, const float* decay, const float* decay_bias, float* state,
                                    long long state_pitch, const int* q_start, const int* state_slot, const int* fresh,
                                    float* out, int n_tokens, int n_seqs, int heads, int qk_heads, int dk, int dv, int mode, int blocks,
                                    void* stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return TL_OK;
    if (heads <= 0 || qk_heads <= 0 || heads % qk_heads != 0 || dk <= 0 || dk > 256 || dv <= 0 || n_seqs > 65535 || heads > 65535)
        return TL_BAD_SIZE;
    if (mode < FIXED || mode > CHANNEL || decay == nullptr) return TL_BAD_SIZE;
    if (mode != FIXED && (beta == nullptr || gate == nullptr || decay_bias == nullptr)) return TL_BAD_SIZE;
    RecurrenceParams p;
    p.q = q; p.k = k; p.v = v; p.ldv = ldv; p.beta = beta; p.gate = gate; p.ldg = ldg; p.ldz = ldz;
    p.g = mode == CHANNEL && blocks ? (const float*)gate : nullptr; p.decay = decay; p.decay_bias = decay_bias;
    p.state = state; p.state_pitch = state_pitch; p.q_start = q_start; p.state_slot = state_slot; p.fresh = fresh; p.out = out;
    p.H = heads; p.G = qk_heads; p.dk = dk; p.dv = dv;
    cudaStream_t s = (cudaStream_t)stream;
    if (v_dtype == TL_F32) return launch_mode<float>(p, n_seqs, mode, blocks != 0, s);
    if (v_dtype == TL_BF16) return launch_mode<__nv_bfloat16>(p, n_seqs, mode, blocks != 0, s);
    return TL_BAD_DTYPE;
}
