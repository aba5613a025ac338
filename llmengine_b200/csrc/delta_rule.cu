// The gated delta rule: a matrix state S (n x p) per request and head that decays, is corrected towards the value it should give
// for the present key, and is read by the present query,
//   S <- a_t S;  u = b_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t,
// with unit queries and keys (x / sqrt(sum(x^2) + eps) per group, the queries then times a constant), a write strength b_t =
// sigmoid(.) and a decay a_t = exp(-exp(A_log) softplus(. + dt_bias)) per token and head.  Everything is 32-bit.  The columns of
// S (one coordinate of v each, n values) are independent of one another.
//
// Single tokens (delta_step_kernel): the state is read and written once, whole columns by neighbouring lanes, 16 bytes a lane;
// norms and gates are formed in the kernel.  The kernel takes any number of tokens, one after the other: it is also the plain
// form of portions.
//
// Portions (delta_prepare_kernel, delta_tile_kernel): a request's tokens are taken FOUR at a time.  With G(i, j) = the product of
// the decays of tokens j + 1 .. i (G(i) from the block's start) and S0 the state before the block,
//   u_i = b_i (v_i - G(i) S0^T k_i - sum_(j < i) G(i, j) (k_j . k_i) u_j),
//   o_i = G(i) S0^T q_i + sum_(j <= i) G(i, j) (k_j . q_i) u_j,
//   S   = G(3) S0 + sum_j G(3, j) k_j u_j^T,
// which is the rule above written out: the eight products with S0 do not wait for one another, their sums over the lanes are
// formed together, and what is left in sequence is a triangular solve of four numbers per column.  The numbers that do not
// depend on a column (40 per block and head) and the unit vectors are made by delta_prepare_kernel for all blocks side by side.
// No quotient of decays is ever formed, so a decay of zero is harmless.  A block at a portion's end is filled up with tokens that
// change nothing (k = q = 0, b = 0, a = 1); how a prompt is cut into steps changes the order of the sums and nothing else.
#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

namespace {

constexpr int BLOCK = 4, QUADS = 10;             // tokens of a block; groups of four numbers that a block and head need

__device__ __forceinline__ float softplus32(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float write_strength(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float decay_of(float z, float a_log) { return expf(-expf(a_log) * softplus32(z)); }

// Two 32-bit values in one 64-bit register and the packed multiply-add on both (each half rounds as fmaf does).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ float sum2(f32x2 v) {
    float lo, hi;
    unpack2(v, lo, hi);
    return lo + hi;
}

__device__ __forceinline__ void copy_async_4(float* dst, const float* src, bool valid) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 4 : 0) : "memory");
}
__device__ __forceinline__ void copy_async_16(float* dst, const float* src, bool valid) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Sum over the L lanes that share a column.
template <int L> __device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// The rows of a column that lane `sub` of L holds are 4 (sub + L m) + e, m < M, e < 4: neighbouring lanes read 16-byte pieces
// that stand side by side.
template <int L, int M>
__device__ __forceinline__ void load_rows(const float* __restrict__ p, int n, int sub, bool vec, bool ok, float (&r)[4 * M]) {
#pragma unroll
    for (int m = 0; m < M; ++m) {
        const int row = 4 * (sub + L * m);
        if (vec) {
            const float4 f = ok && row < n ? *(const float4*)(p + row) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            r[4 * m] = f.x; r[4 * m + 1] = f.y; r[4 * m + 2] = f.z; r[4 * m + 3] = f.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) r[4 * m + e] = ok && row + e < n ? p[row + e] : 0.0f;
        }
    }
}
template <int L, int M>
__device__ __forceinline__ void store_rows(float* __restrict__ p, int n, int sub, bool vec, bool ok, const float (&r)[4 * M]) {
    if (!ok) return;
#pragma unroll
    for (int m = 0; m < M; ++m) {
        const int row = 4 * (sub + L * m);
        if (vec) {
            if (row < n) *(float4*)(p + row) = make_float4(r[4 * m], r[4 * m + 1], r[4 * m + 2], r[4 * m + 3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (row + e < n) p[row + e] = r[4 * m + e];
        }
    }
}

// ----------------------------------------------------------------------------- one token after the other
// A lane holds rows of C columns; a warp's 32 / L groups of lanes stand on neighbouring sets of C columns.
constexpr int STEP_WARPS = 4;

template <int L, int M, int C>
__global__ void __launch_bounds__(32 * STEP_WARPS) delta_step_kernel(LlmeDeltaArgs a, int vec_state, int vec_qk) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, sub = lane % L, grp = lane / L;
    const int col0 = ((blockIdx.x * STEP_WARPS + warp) * (32 / L) + grp) * C;
    const int h = blockIdx.y, r = a.rows ? a.rows[blockIdx.z] : (int)blockIdx.z, n = a.n, p = a.p;
    const int first = a.cu_q_lens[r], last = a.cu_q_lens[r + 1], g = h / (a.heads / a.qk_groups);
    if (((blockIdx.x * STEP_WARPS + warp) * (32 / L)) * C >= p) return;      // (the whole warp)
    float* st = a.state + (size_t)a.state_slots[r] * a.state_stride + ((size_t)h * p + col0) * n;
    float S[C][4 * M];
#pragma unroll
    for (int c = 0; c < C; ++c) load_rows<L, M>(st + (size_t)c * n, n, sub, vec_state, col0 + c < p, S[c]);
    const float a_log = a.a_log[h], dt_bias = a.dt_bias[h];
    for (int t = first; t < last; ++t) {
        float q[4 * M], k[4 * M], v[C];
        load_rows<L, M>(a.q + (size_t)t * a.ldq + (size_t)g * n, n, sub, vec_qk, true, q);
        load_rows<L, M>(a.k + (size_t)t * a.ldk + (size_t)g * n, n, sub, vec_qk, true, k);
#pragma unroll
        for (int c = 0; c < C; ++c) v[c] = col0 + c < p ? a.v[(size_t)t * a.ldv + (size_t)h * p + col0 + c] : 0.0f;
        const float beta = write_strength(a.write[(size_t)t * a.ld_gates + h]);
        const float keep = decay_of(a.forget[(size_t)t * a.ld_gates + h] + dt_bias, a_log);
        float sq = 0.0f, sk = 0.0f;
#pragma unroll
        for (int i = 0; i < 4 * M; ++i) {
            sq = fmaf(q[i], q[i], sq);
            sk = fmaf(k[i], k[i], sk);
        }
        const float iq = a.q_scale / sqrtf(lanes_sum<L>(sq) + a.unit_eps), ik = 1.0f / sqrtf(lanes_sum<L>(sk) + a.unit_eps);
#pragma unroll
        for (int i = 0; i < 4 * M; ++i) {
            q[i] *= iq;
            k[i] *= ik;
        }
        float known[C];                                         // what the decayed state gives for the key
#pragma unroll
        for (int c = 0; c < C; ++c) {
            known[c] = 0.0f;
#pragma unroll
            for (int i = 0; i < 4 * M; ++i) {
                S[c][i] *= keep;
                known[c] = fmaf(S[c][i], k[i], known[c]);
            }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) known[c] = lanes_sum<L>(known[c]);
        float o[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const float u = beta * (v[c] - known[c]);
            o[c] = 0.0f;
#pragma unroll
            for (int i = 0; i < 4 * M; ++i) {
                S[c][i] = fmaf(k[i], u, S[c][i]);
                o[c] = fmaf(S[c][i], q[i], o[c]);
            }
        }
#pragma unroll
        for (int c = 0; c < C; ++c) {
            o[c] = lanes_sum<L>(o[c]);
            if (sub == 0 && col0 + c < p) a.out[(size_t)t * a.ldo + (size_t)h * p + col0 + c] = o[c];
        }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) store_rows<L, M>(st + (size_t)c * n, n, sub, vec_state, col0 + c < p, S[c]);
}

template <int L, int M, int C>
void launch_step(const LlmeDeltaArgs& a, int vec_state, int vec_qk, cudaStream_t s) {
    constexpr int COLS = STEP_WARPS * (32 / L) * C;
    llme_launch(delta_step_kernel<L, M, C>, dim3((a.p + COLS - 1) / COLS, a.heads, a.n_rows), dim3(32 * STEP_WARPS), 0, s, a, vec_state, vec_qk);
}

// ----------------------------------------------------------------------------- portions: what no column has a say in
// Block number of request r's b-th block: floor(first token / 4) + r + b (distinct for all blocks of a step).
__device__ __forceinline__ int first_block(const int* __restrict__ cu, int r) { return (cu[r] >> 2) + r; }

// One warp per (block, query/key group): unit queries and keys, their products within the block, and per head of the group
//   0: b_i   1: b_i G(i)   2: A10 A20 A21 A30   3: A31 A32 0 G(3)   4: G(3, i)   5: G(i)   6 + i: B_i0 .. B_i3
// with A_ij = b_i G(i, j) k_j . k_i and B_ij = G(i, j) k_j . q_i (zero for j > i).
template <int R>
__global__ void __launch_bounds__(128) delta_prepare_kernel(LlmeDeltaArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, id = blockIdx.x, g = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (g >= a.qk_groups) return;
    int lo = 0, hi = a.requests;                                // the last request whose first block is not behind `id`
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (first_block(a.cu_q_lens, mid) <= id) lo = mid; else hi = mid;
    }
    const int len = a.cu_q_lens[lo + 1] - a.cu_q_lens[lo], at = BLOCK * (id - first_block(a.cu_q_lens, lo));
    if (at < 0 || at >= len || len < 2) return;                 // a number no block has, or a single token
    const int t0 = a.cu_q_lens[lo] + at, count = min(BLOCK, len - at), n = a.n, n4 = (n + 3) & ~3;
    float q[BLOCK][R], k[BLOCK][R];
#pragma unroll
    for (int j = 0; j < BLOCK; ++j)
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int e = lane + 32 * i;
            const bool ok = j < count && e < n;
            q[j][i] = ok ? a.q[(size_t)(t0 + j) * a.ldq + (size_t)g * n + e] : 0.0f;
            k[j][i] = ok ? a.k[(size_t)(t0 + j) * a.ldk + (size_t)g * n + e] : 0.0f;
        }
#pragma unroll
    for (int j = 0; j < BLOCK; ++j) {
        float sq = 0.0f, sk = 0.0f;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            sq = fmaf(q[j][i], q[j][i], sq);
            sk = fmaf(k[j][i], k[j][i], sk);
        }
        const float iq = a.q_scale / sqrtf(warp_sum(sq) + a.unit_eps), ik = 1.0f / sqrtf(warp_sum(sk) + a.unit_eps);
        float* uq = a.unit + ((size_t)(t0 + j) * 2 * a.qk_groups + g) * n4;
        float* uk = uq + (size_t)a.qk_groups * n4;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int e = lane + 32 * i;
            q[j][i] *= iq;
            k[j][i] *= ik;
            if (j < count && e < n4) {
                uq[e] = q[j][i];
                uk[e] = k[j][i];
            }
        }
    }
    float kk[BLOCK][BLOCK], qk[BLOCK][BLOCK];                   // [i][j], j < i and j <= i
#pragma unroll
    for (int i = 0; i < BLOCK; ++i)
#pragma unroll
        for (int j = 0; j <= i; ++j) {
            float x = 0.0f, y = 0.0f;
#pragma unroll
            for (int e = 0; e < R; ++e) {
                if (j < i) x = fmaf(k[j][e], k[i][e], x);
                y = fmaf(k[j][e], q[i][e], y);
            }
            if (j < i) kk[i][j] = warp_sum(x);
            qk[i][j] = warp_sum(y);
        }
    // four lanes per head: each forms its token's two gates, all four then hold the block's
    const int rep = a.heads / a.qk_groups, j = lane & 3;
    for (int x0 = 0; x0 < rep; x0 += 8) {
        const int x = x0 + (lane >> 2), h = g * rep + x;
        float beta = 0.0f, keep = 1.0f;
        if (x < rep && j < count) {
            beta = write_strength(a.write[(size_t)(t0 + j) * a.ld_gates + h]);
            keep = decay_of(a.forget[(size_t)(t0 + j) * a.ld_gates + h] + a.dt_bias[h], a.a_log[h]);
        }
        float b[BLOCK], w[BLOCK];
#pragma unroll
        for (int i = 0; i < BLOCK; ++i) {
            b[i] = __shfl_sync(0xffffffffu, beta, (lane & ~3) + i);
            w[i] = __shfl_sync(0xffffffffu, keep, (lane & ~3) + i);
        }
        if (x >= rep) continue;
        const float g1 = w[0] * w[1], g2 = g1 * w[2], g3 = g2 * w[3], w12 = w[1] * w[2], w23 = w[2] * w[3], w123 = w12 * w[3];
        float4* o = (float4*)(a.coef + ((size_t)id * a.heads + h) * (4 * QUADS));
        if (j == 0) {
            o[0] = make_float4(b[0], b[1], b[2], b[3]);
            o[4] = make_float4(w123, w23, w[3], 1.0f);
            o[8] = make_float4(w12 * qk[2][0], w[2] * qk[2][1], qk[2][2], 0.0f);
        } else if (j == 1) {
            o[1] = make_float4(b[0] * w[0], b[1] * g1, b[2] * g2, b[3] * g3);
            o[5] = make_float4(w[0], g1, g2, g3);
            o[9] = make_float4(w123 * qk[3][0], w23 * qk[3][1], w[3] * qk[3][2], qk[3][3]);
        } else if (j == 2) {
            o[2] = make_float4(b[1] * w[1] * kk[1][0], b[2] * w12 * kk[2][0], b[2] * w[2] * kk[2][1], b[3] * w123 * kk[3][0]);
            o[6] = make_float4(qk[0][0], 0.0f, 0.0f, 0.0f);
        } else {
            o[3] = make_float4(b[3] * w23 * kk[3][1], b[3] * w[3] * kk[3][2], 0.0f, g3);
            o[7] = make_float4(w[1] * qk[1][0], qk[1][1], 0.0f, 0.0f);
        }
    }
}

// ----------------------------------------------------------------------------- portions: four tokens at a time
// A block of W warps takes W * 32 / L * C neighbouring columns of one (request, head).  Unit queries and keys, values and the
// blocks' numbers come into shared memory TT tokens at a time by asynchronous copies, NS tiles deep.
constexpr int TT = 16;

template <int L, int M, int C, int W, int NS>
struct DeltaTile {
    static constexpr int ROW = 4 * L * M, COLS = W * (32 / L) * C;
    float q[NS][TT][ROW], k[NS][TT][ROW], v[NS][TT][COLS], coef[NS][TT / BLOCK][4 * QUADS];
};

template <int L, int M, int C, int W, int NS>
__global__ void __launch_bounds__(32 * W) delta_tile_kernel(LlmeDeltaArgs a, int vec_state) {
    using Tile = DeltaTile<L, M, C, W, NS>;
    constexpr int ROW = Tile::ROW, COLS = Tile::COLS, P2 = 2 * M;         // packed pairs of rows a lane holds per column
    extern __shared__ __align__(16) unsigned char smem_raw[];
    Tile& sm = *reinterpret_cast<Tile*>(smem_raw);
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane % L;
    const int jb = blockIdx.x * COLS, mine = (warp * (32 / L) + lane / L) * C, col0 = jb + mine;
    const int h = blockIdx.y, r = a.rows ? a.rows[blockIdx.z] : (int)blockIdx.z, n = a.n, p = a.p, n4 = (n + 3) & ~3;
    const int first = a.cu_q_lens[r], last = a.cu_q_lens[r + 1], g = h / (a.heads / a.qk_groups);
    const int block0 = first_block(a.cu_q_lens, r);
    const float* uq = a.unit + (size_t)g * n4;
    const size_t ldu = (size_t)2 * a.qk_groups * n4, to_k = (size_t)a.qk_groups * n4;

    auto fetch = [&](int tile) {
        const int s = tile % NS, t0 = first + tile * TT;
        if (t0 < last) {
            for (int i = tid; i < TT * (ROW / 4); i += 32 * W) {
                const int u = i / (ROW / 4), e = (i % (ROW / 4)) * 4;
                const bool ok = t0 + u < last && e < n4;
                const float* src = ok ? uq + (size_t)(t0 + u) * ldu + e : a.unit;
                copy_async_16(&sm.q[s][u][e], src, ok);
                copy_async_16(&sm.k[s][u][e], ok ? src + to_k : a.unit, ok);
            }
            for (int i = tid; i < TT * COLS; i += 32 * W) {
                const int u = i / COLS, c = i % COLS;
                const bool ok = t0 + u < last && jb + c < p;
                copy_async_4(&sm.v[s][u][c], ok ? a.v + (size_t)(t0 + u) * a.ldv + (size_t)h * p + jb + c : a.v, ok);
            }
            for (int i = tid; i < TT / BLOCK * QUADS; i += 32 * W) {
                const int b = i / QUADS, e = (i % QUADS) * 4;
                const bool ok = t0 + BLOCK * b < last;
                copy_async_16(&sm.coef[s][b][e], ok ? a.coef + ((size_t)(block0 + tile * (TT / BLOCK) + b) * a.heads + h) * (4 * QUADS) + e : a.coef, ok);
            }
        }
        copy_async_commit();                                    // one group a tile, also an empty one: the waits below count them
    };

    float* st = a.state + (size_t)a.state_slots[r] * a.state_stride + ((size_t)h * p + col0) * n;
    f32x2 S[C][P2];
#pragma unroll
    for (int s = 0; s < NS - 1; ++s) fetch(s);
#pragma unroll
    for (int c = 0; c < C; ++c) {
        float rows[4 * M];
        load_rows<L, M>(st + (size_t)c * n, n, sub, vec_state, col0 + c < p, rows);
#pragma unroll
        for (int i = 0; i < P2; ++i) S[c][i] = pack2(rows[2 * i], rows[2 * i + 1]);
    }
    const int tiles = (last - first + TT - 1) / TT;
    for (int tile = 0; tile < tiles; ++tile) {
        copy_async_wait<NS - 2>();                              // the tile has landed
        __syncthreads();                                        // ... for every thread, and the tile before has been read by all
        fetch(tile + NS - 1);
        const int s = tile % NS, t0 = first + tile * TT;
#pragma unroll
        for (int b = 0; b < TT / BLOCK; ++b) {
            if (t0 + BLOCK * b >= last) break;                  // (uniform over the block)
            f32x2 k[BLOCK][P2];
            float part[C][2 * BLOCK];                           // this lane's share of S0^T k_i, then of S0^T q_i
#pragma unroll
            for (int i = 0; i < BLOCK; ++i) {
                f32x2 acc[C];
#pragma unroll
                for (int c = 0; c < C; ++c) acc[c] = pack2(0.0f, 0.0f);
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const ulonglong2 f = *(const ulonglong2*)&sm.k[s][BLOCK * b + i][4 * (sub + L * m)];
                    k[i][2 * m] = f.x;
                    k[i][2 * m + 1] = f.y;
#pragma unroll
                    for (int c = 0; c < C; ++c) acc[c] = fma2(S[c][2 * m + 1], f.y, fma2(S[c][2 * m], f.x, acc[c]));
                }
#pragma unroll
                for (int c = 0; c < C; ++c) part[c][i] = sum2(acc[c]);
            }
#pragma unroll
            for (int i = 0; i < BLOCK; ++i) {
                f32x2 acc[C];
#pragma unroll
                for (int c = 0; c < C; ++c) acc[c] = pack2(0.0f, 0.0f);
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const ulonglong2 f = *(const ulonglong2*)&sm.q[s][BLOCK * b + i][4 * (sub + L * m)];
#pragma unroll
                    for (int c = 0; c < C; ++c) acc[c] = fma2(S[c][2 * m + 1], f.y, fma2(S[c][2 * m], f.x, acc[c]));
                }
#pragma unroll
                for (int c = 0; c < C; ++c) part[c][BLOCK + i] = sum2(acc[c]);
            }
            const float4* cf = (const float4*)sm.coef[s][b];
            const float4 cb = cf[0], cbg = cf[1], ca = cf[2], ca2 = cf[3], cu = cf[4];
            const int mi = sub & 3;
            const float gi = sm.coef[s][b][20 + mi];
            const float4 cB = cf[6 + mi];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                // lanes exchange halves of what they hold until lane `sub` has the whole sum number sub % 8: 0..3 with the
                // keys, 4..7 with the queries
                const bool up4 = sub & 4, up2 = sub & 2, up1 = sub & 1;
                float x[4], y[2], z;
#pragma unroll
                for (int i = 0; i < 4; ++i) x[i] = (up4 ? part[c][i + 4] : part[c][i]) + __shfl_xor_sync(0xffffffffu, up4 ? part[c][i] : part[c][i + 4], 4);
#pragma unroll
                for (int i = 0; i < 2; ++i) y[i] = (up2 ? x[i + 2] : x[i]) + __shfl_xor_sync(0xffffffffu, up2 ? x[i] : x[i + 2], 2);
                z = (up1 ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, up1 ? y[0] : y[1], 1);
#pragma unroll
                for (int o = 8; o < L; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
                const int base = lane & ~(L - 1);
                const float d0 = __shfl_sync(0xffffffffu, z, base), d1 = __shfl_sync(0xffffffffu, z, base + 1);
                const float d2 = __shfl_sync(0xffffffffu, z, base + 2), d3 = __shfl_sync(0xffffffffu, z, base + 3);
                const float v0 = sm.v[s][BLOCK * b][mine + c], v1 = sm.v[s][BLOCK * b + 1][mine + c];
                const float v2 = sm.v[s][BLOCK * b + 2][mine + c], v3 = sm.v[s][BLOCK * b + 3][mine + c];
                const float u0 = fmaf(-cbg.x, d0, cb.x * v0);
                const float u1 = fmaf(-ca.x, u0, fmaf(-cbg.y, d1, cb.y * v1));
                const float u2 = fmaf(-ca.z, u1, fmaf(-ca.y, u0, fmaf(-cbg.z, d2, cb.z * v2)));
                const float u3 = fmaf(-ca2.y, u2, fmaf(-ca2.x, u1, fmaf(-ca.w, u0, fmaf(-cbg.w, d3, cb.w * v3))));
                if (sub >= 4 && sub < 8) {
                    const int t = t0 + BLOCK * b + mi;
                    const float o = fmaf(cB.w, u3, fmaf(cB.z, u2, fmaf(cB.y, u1, fmaf(cB.x, u0, gi * z))));
                    if (t < last && col0 + c < p) a.out[(size_t)t * a.ldo + (size_t)h * p + col0 + c] = o;
                }
                const float w0 = cu.x * u0, w1 = cu.y * u1, w2 = cu.z * u2, w3 = cu.w * u3;
                const f32x2 p0 = pack2(w0, w0), p1 = pack2(w1, w1), p2 = pack2(w2, w2), p3 = pack2(w3, w3), gt = pack2(ca2.w, ca2.w);
#pragma unroll
                for (int i = 0; i < P2; ++i)
                    S[c][i] = fma2(k[3][i], p3, fma2(k[2][i], p2, fma2(k[1][i], p1, fma2(k[0][i], p0, mul2(gt, S[c][i])))));
            }
        }
    }
    copy_async_wait<0>();                                       // (empty groups only; nothing is in flight when the block leaves)
#pragma unroll
    for (int c = 0; c < C; ++c) {
        float rows[4 * M];
#pragma unroll
        for (int i = 0; i < P2; ++i) unpack2(S[c][i], rows[2 * i], rows[2 * i + 1]);
        store_rows<L, M>(st + (size_t)c * n, n, sub, vec_state, col0 + c < p, rows);
    }
}

template <int L, int M, int C, int W, int NS>
int launch_tile(const LlmeDeltaArgs& a, int vec_state, cudaStream_t s) {
    using Tile = DeltaTile<L, M, C, W, NS>;
    auto kernel = delta_tile_kernel<L, M, C, W, NS>;
    static bool configured = false;
    if (!configured) {
        if (sizeof(Tile) > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(Tile)) != cudaSuccess)
            LLME_REFUSE("delta_rule: %zu bytes of shared memory are not available", sizeof(Tile));
        configured = true;
    }
    llme_launch(kernel, dim3((a.p + Tile::COLS - 1) / Tile::COLS, a.heads, a.n_rows), dim3(32 * W), sizeof(Tile), s, a, vec_state);
    LLME_LAUNCH_STATUS();
}

bool rows_of_16(const void* p, long long stride, int n) { return (uintptr_t)p % 16 == 0 && stride % 4 == 0 && n % 4 == 0; }

int check(const LlmeDeltaArgs& a) {
    if (!a.q || !a.k || !a.v || !a.write || !a.forget || !a.dt_bias || !a.a_log || !a.state || !a.out || !a.cu_q_lens || !a.state_slots)
        LLME_REFUSE("delta_rule: null pointer");
    if (a.heads <= 0 || a.n <= 0 || a.p <= 0 || a.qk_groups <= 0 || a.heads % a.qk_groups) LLME_REFUSE("delta_rule: %d heads in %d groups", a.heads, a.qk_groups);
    if (a.n > 512) LLME_REFUSE("delta_rule: a state of %d rows per column, this build takes up to 512", a.n);
    if (a.heads > 65535 || a.n_rows > 65535) LLME_REFUSE("delta_rule: too many heads or requests for one launch");
    if (!(a.unit_eps > 0.0f)) LLME_REFUSE("delta_rule: the unit norm's eps must be positive");
    return 0;
}

}  // namespace

// The requests `rows` (all of the step's without it), token after token.
LLME_API int llme_delta_step(const LlmeDeltaArgs* args, cudaStream_t stream) {
    const LlmeDeltaArgs& a = *args;
    if (a.n_rows <= 0) return 0;
    if (int rc = check(a)) return rc;
    const int vs = rows_of_16(a.state, a.state_stride, a.n), vq = rows_of_16(a.q, a.ldq, a.n) && rows_of_16(a.k, a.ldk, a.n);
    if (a.n <= 32) launch_step<8, 1, 4>(a, vs, vq, stream);
    else if (a.n <= 64) launch_step<16, 1, 4>(a, vs, vq, stream);
    else if (a.n <= 128) launch_step<32, 1, 4>(a, vs, vq, stream);
    else if (a.n <= 256) launch_step<32, 2, 4>(a, vs, vq, stream);
    else launch_step<32, 4, 4>(a, vs, vq, stream);
    LLME_LAUNCH_STATUS();
}

// The requests `rows`, each with two tokens or more, four tokens at a time.
LLME_API int llme_delta_portions(const LlmeDeltaArgs* args, cudaStream_t stream) {
    const LlmeDeltaArgs& a = *args;
    if (a.n_rows <= 0) return 0;
    if (int rc = check(a)) return rc;
    if (!a.unit || !a.coef || ((uintptr_t)a.unit | (uintptr_t)a.coef) % 16) LLME_REFUSE("delta_rule: portions need their workspace");
    const dim3 blocks(a.tokens / BLOCK + a.requests + 1, (a.qk_groups + 3) / 4);
    if (a.n <= 32) llme_launch(delta_prepare_kernel<1>, blocks, dim3(128), 0, stream, a);
    else if (a.n <= 64) llme_launch(delta_prepare_kernel<2>, blocks, dim3(128), 0, stream, a);
    else if (a.n <= 128) llme_launch(delta_prepare_kernel<4>, blocks, dim3(128), 0, stream, a);
    else if (a.n <= 256) llme_launch(delta_prepare_kernel<8>, blocks, dim3(128), 0, stream, a);
    else llme_launch(delta_prepare_kernel<16>, blocks, dim3(128), 0, stream, a);
    const int vs = rows_of_16(a.state, a.state_stride, a.n);
    if (a.n <= 32) return launch_tile<8, 1, 1, 4, 3>(a, vs, stream);
    if (a.n <= 64) return launch_tile<8, 2, 1, 4, 3>(a, vs, stream);
    if (a.n <= 128) return launch_tile<8, 4, 1, 4, 3>(a, vs, stream);
    if (a.n <= 256) return launch_tile<16, 4, 1, 4, 3>(a, vs, stream);
    return launch_tile<32, 4, 1, 4, 2>(a, vs, stream);
}
