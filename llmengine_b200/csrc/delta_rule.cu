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
// Portions (delta_prepare_kernel, delta_tile_kernel): a request's tokens are taken EIGHT at a time.  With G(i, j) = the product of
// the decays of tokens j + 1 .. i (G(i) from the block's start) and S0 the state before the block,
//   u_i = r_i - sum_(j < i) A_ij u_j,   r_i = b_i (v_i - G(i) S0^T k_i),   A_ij = b_i G(i, j) k_j . k_i,
//   o_i = G(i) S0^T q_i + sum_(j <= i) B_ij u_j,   B_ij = G(i, j) k_j . q_i,
//   S   = G(7) S0 + sum_j G(7, j) k_j u_j^T,
// which is the rule above written out.  The sixteen products with S0 do not wait for one another, and their sums over the lanes are
// formed together.  What does not depend on a column is made by delta_prepare_kernel for all blocks side by side: the unit vectors,
// the inverse N of the unit lower triangular I + A, and B N, so that u = N r and o = G S0^T q + (B N) r: lane i of a column forms
// u_i and o_i from the eight r's, and nothing is left to be solved in sequence.  No quotient of decays is ever formed, so a decay of
// zero is harmless.  A block at a portion's end is filled up with tokens that change nothing (k = q = 0, b = 0, a = 1); how a
// prompt is cut into steps changes the order of the sums and nothing else.
#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

namespace {

constexpr int BLOCK = 8, ROW_NUMBERS = 20;       // tokens of a block; numbers that a token of a block and head needs: b, b G, G, G(7, .),
constexpr int NUMBERS = BLOCK * ROW_NUMBERS;      // a row of N, a row of B N

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
// Block number of request r's b-th block: floor(first token / 8) + r + b (distinct for all blocks of a step).
__device__ __forceinline__ int first_block(const int* __restrict__ cu, int r) { return cu[r] / BLOCK + r; }

// Sums over the warp of 32 values a lane: lane i ends with the sum of everybody's v[i].
__device__ __forceinline__ float sums_of_32(float (&v)[32], int lane) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) v[i] = (up ? v[i + o] : v[i]) + __shfl_xor_sync(0xffffffffu, up ? v[i] : v[i + o], o);
    }
    return v[0];
}

// One warp per (block, query/key group).
constexpr int PREPARE_WARPS = 4;

__global__ void __launch_bounds__(32 * PREPARE_WARPS) delta_prepare_kernel(LlmeDeltaArgs a) {
    // sums: [0, 36) k_j . q_i at i (i + 1) / 2 + j; [36, 64) k_j . k_i (j < i) at i (i - 1) / 2 + j; [64, 72) |q_i|^2; [72, 80) |k_i|^2
    __shared__ float sums_of[PREPARE_WARPS][96];
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, id = blockIdx.x, g = blockIdx.y * PREPARE_WARPS + warp;
    if (g >= a.qk_groups) return;
    int lo = 0, hi = a.requests;                                // the last request whose first block is not behind `id`
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (first_block(a.cu_q_lens, mid) <= id) lo = mid; else hi = mid;
    }
    const int len = a.cu_q_lens[lo + 1] - a.cu_q_lens[lo], at = BLOCK * (id - first_block(a.cu_q_lens, lo));
    if (at < 0 || at >= len || len < 2) return;                 // a number no block has, or a single token
    const int t0 = a.cu_q_lens[lo] + at, count = min(BLOCK, len - at), n = a.n, n4 = (n + 3) & ~3;
    float* sums = sums_of[warp];
    const float* qp = a.q + (size_t)t0 * a.ldq + (size_t)g * n;
    const float* kp = a.k + (size_t)t0 * a.ldk + (size_t)g * n;
    {
        float s0[32], s1[32], s2[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) s0[i] = s1[i] = s2[i] = 0.0f;
        auto slot = [&](int i) -> float& { return i < 32 ? s0[i] : i < 64 ? s1[i - 32] : s2[i - 64]; };
        for (int e = lane; e < n; e += 32) {
            float q[BLOCK], k[BLOCK];
#pragma unroll
            for (int j = 0; j < BLOCK; ++j) {
                q[j] = j < count ? qp[(size_t)j * a.ldq + e] : 0.0f;
                k[j] = j < count ? kp[(size_t)j * a.ldk + e] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < BLOCK; ++i) {
                slot(64 + i) = fmaf(q[i], q[i], slot(64 + i));
                slot(72 + i) = fmaf(k[i], k[i], slot(72 + i));
#pragma unroll
                for (int j = 0; j <= i; ++j) {
                    slot(i * (i + 1) / 2 + j) = fmaf(k[j], q[i], slot(i * (i + 1) / 2 + j));
                    if (j < i) slot(36 + i * (i - 1) / 2 + j) = fmaf(k[j], k[i], slot(36 + i * (i - 1) / 2 + j));
                }
            }
        }
        sums[lane] = sums_of_32(s0, lane);
        sums[32 + lane] = sums_of_32(s1, lane);
        sums[64 + lane] = sums_of_32(s2, lane);
    }
    __syncwarp();
    // 1 / |.| of the queries (times their constant) and of the keys, in the places of their squares
    if (lane < 2 * BLOCK) sums[64 + lane] = (lane < BLOCK ? a.q_scale : 1.0f) / sqrtf(sums[64 + lane] + a.unit_eps);
    __syncwarp();
    float iq[BLOCK], ik[BLOCK];
#pragma unroll
    for (int j = 0; j < BLOCK; ++j) {
        iq[j] = sums[64 + j];
        ik[j] = sums[72 + j];
    }
    for (int e = lane; e < n4; e += 32) {
        float* uq = a.unit + ((size_t)t0 * 2 * a.qk_groups + g) * n4 + e;
#pragma unroll
        for (int j = 0; j < BLOCK; ++j) {
            if (j >= count) break;
            uq[(size_t)j * 2 * a.qk_groups * n4] = e < n ? qp[(size_t)j * a.ldq + e] * iq[j] : 0.0f;
            uq[((size_t)j * 2 + 1) * a.qk_groups * n4] = e < n ? kp[(size_t)j * a.ldk + e] * ik[j] : 0.0f;
        }
    }
    // eight lanes per head: each forms its token's two gates, all eight then hold the block's, and lane j forms column j of N and B N
    const int rep = a.heads / a.qk_groups, j = lane & 7;
    for (int x0 = 0; x0 < rep; x0 += 4) {
        const int x = x0 + (lane >> 3), h = g * rep + x;
        float beta = 0.0f, keep = 1.0f;
        if (x < rep && j < count) {
            beta = write_strength(a.write[(size_t)(t0 + j) * a.ld_gates + h]);
            keep = decay_of(a.forget[(size_t)(t0 + j) * a.ld_gates + h] + a.dt_bias[h], a.a_log[h]);
        }
        float b[BLOCK], w[BLOCK];
#pragma unroll
        for (int i = 0; i < BLOCK; ++i) {
            b[i] = __shfl_sync(0xffffffffu, beta, (lane & ~7) + i);
            w[i] = __shfl_sync(0xffffffffu, keep, (lane & ~7) + i);
        }
        if (x >= rep) continue;
        float* o = a.coef + ((size_t)id * a.heads + h) * NUMBERS;
        float G[BLOCK], N[BLOCK], from_start = 1.0f, to_end = 1.0f;
#pragma unroll
        for (int i = 0; i < BLOCK; ++i) {
#pragma unroll
            for (int m = 0; m < i; ++m) G[m] *= w[i];            // G(i, m)
            G[i] = 1.0f;
            float below = 0.0f, read = 0.0f;
#pragma unroll
            for (int m = 0; m < i; ++m) below = fmaf(G[m] * (sums[36 + i * (i - 1) / 2 + m] * ik[m]), N[m], below);
            N[i] = i == j ? 1.0f : -(b[i] * ik[i]) * below;      // zero above the diagonal: `below` is zero there
#pragma unroll
            for (int m = 0; m <= i; ++m) read = fmaf(G[m] * (sums[i * (i + 1) / 2 + m] * ik[m]), N[m], read);
            o[i * ROW_NUMBERS + 4 + j] = N[i];
            o[i * ROW_NUMBERS + 12 + j] = read * iq[i];
            if (i <= j) from_start *= w[i];
            else to_end *= w[i];
        }
        const float mine = beta;
        *(float4*)(o + j * ROW_NUMBERS) = make_float4(mine, mine * from_start, from_start, to_end);
    }
}

// ----------------------------------------------------------------------------- portions: eight tokens at a time
// A block of W warps takes W * 32 / L * C neighbouring columns of one (request, head).  Unit queries and keys, values and the
// blocks' numbers come into shared memory TT tokens at a time by asynchronous copies, NS tiles deep.
constexpr int TT = 16;

template <int L, int M, int C, int W, int NS>
struct DeltaTile {
    static constexpr int ROW = 4 * L * M, COLS = W * (32 / L) * C;
    float q[NS][TT][ROW], k[NS][TT][ROW], v[NS][TT][COLS], coef[NS][TT / BLOCK][NUMBERS];
};

template <int L, int M, int C, int W, int NS>
__global__ void __launch_bounds__(32 * W) delta_tile_kernel(LlmeDeltaArgs a, int vec_state) {
    using Tile = DeltaTile<L, M, C, W, NS>;
    constexpr int ROW = Tile::ROW, COLS = Tile::COLS, P2 = 2 * M;         // packed pairs of rows a lane holds per column
    extern __shared__ __align__(16) unsigned char smem_raw[];
    Tile& sm = *reinterpret_cast<Tile*>(smem_raw);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane % L, row = sub & 7, base = lane & ~(L - 1);
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
            for (int i = tid; i < TT / BLOCK * (NUMBERS / 4); i += 32 * W) {
                const int b = i / (NUMBERS / 4), e = (i % (NUMBERS / 4)) * 4;
                const bool ok = t0 + BLOCK * b < last;
                copy_async_16(&sm.coef[s][b][e], ok ? a.coef + ((size_t)(block0 + tile * (TT / BLOCK) + b) * a.heads + h) * NUMBERS + e : a.coef, ok);
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
#pragma unroll 1
        for (int b = 0; b < TT / BLOCK; ++b) {
            if (t0 + BLOCK * b >= last) break;                  // (uniform over the block)
            f32x2 k[BLOCK][P2];
            float part[C][2 * BLOCK];                           // this lane's share of S0^T k_i, then of S0^T q_i
#pragma unroll
            for (int i = 0; i < BLOCK; ++i)
#pragma unroll
                for (int m = 0; m < M; ++m) {
                    const ulonglong2 f = *(const ulonglong2*)&sm.k[s][BLOCK * b + i][4 * (sub + L * m)];
                    k[i][2 * m] = f.x;
                    k[i][2 * m + 1] = f.y;
                }
            const float* cf = sm.coef[s][b] + row * ROW_NUMBERS;
            const float4 own = *(const float4*)cf;              // b, b G, G and G(7, .) of the token this lane stands for
            const float total = sm.coef[s][b][(BLOCK - 1) * ROW_NUMBERS + 2];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                f32x2 acc[BLOCK];
#pragma unroll
                for (int i = 0; i < BLOCK; ++i) acc[i] = mul2(S[c][0], k[i][0]);
#pragma unroll
                for (int e = 1; e < P2; ++e)
#pragma unroll
                    for (int i = 0; i < BLOCK; ++i) acc[i] = fma2(S[c][e], k[i][e], acc[i]);
#pragma unroll
                for (int i = 0; i < BLOCK; ++i) part[c][i] = sum2(acc[i]);
            }
            {
                f32x2 acc[C][BLOCK];
#pragma unroll
                for (int m = 0; m < M; ++m)
#pragma unroll
                    for (int i = 0; i < BLOCK; ++i) {
                        const ulonglong2 f = *(const ulonglong2*)&sm.q[s][BLOCK * b + i][4 * (sub + L * m)];
#pragma unroll
                        for (int c = 0; c < C; ++c)
                            acc[c][i] = fma2(S[c][2 * m + 1], f.y, m == 0 ? mul2(S[c][0], f.x) : fma2(S[c][2 * m], f.x, acc[c][i]));
                    }
#pragma unroll
                for (int c = 0; c < C; ++c)
#pragma unroll
                    for (int i = 0; i < BLOCK; ++i) part[c][BLOCK + i] = sum2(acc[c][i]);
            }
            const float4 n0 = *(const float4*)(cf + 4), n1 = *(const float4*)(cf + 8), r0 = *(const float4*)(cf + 12), r1 = *(const float4*)(cf + 16);
#pragma unroll
            for (int c = 0; c < C; ++c) {
                // lanes exchange halves of what they hold until every lane has two whole sums: those of token sub % 8 with its key
                // and with its query
                const bool up4 = sub & 4, up2 = sub & 2, up1 = sub & 1;
                float x[2][4], y[2][2], z[2];
#pragma unroll
                for (int f = 0; f < 2; ++f)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const float low = part[c][BLOCK * f + i], high = part[c][BLOCK * f + i + 4];
                        x[f][i] = (up4 ? high : low) + __shfl_xor_sync(0xffffffffu, up4 ? low : high, 4);
                    }
#pragma unroll
                for (int f = 0; f < 2; ++f)
#pragma unroll
                    for (int i = 0; i < 2; ++i) y[f][i] = (up2 ? x[f][i + 2] : x[f][i]) + __shfl_xor_sync(0xffffffffu, up2 ? x[f][i] : x[f][i + 2], 2);
#pragma unroll
                for (int f = 0; f < 2; ++f) {
                    z[f] = (up1 ? y[f][1] : y[f][0]) + __shfl_xor_sync(0xffffffffu, up1 ? y[f][0] : y[f][1], 1);
#pragma unroll
                    for (int o = 8; o < L; o <<= 1) z[f] += __shfl_xor_sync(0xffffffffu, z[f], o);
                }
                const f32x2 kept = pack2(total, total);
#pragma unroll
                for (int e = 0; e < P2; ++e) S[c][e] = mul2(kept, S[c][e]);
                // r of this lane's token, everybody's r, then u and o of this lane's token
                const float mine_r = fmaf(-own.y, z[0], own.x * sm.v[s][BLOCK * b + row][mine + c]);
                float rr[BLOCK];
#pragma unroll
                for (int i = 0; i < BLOCK; ++i) rr[i] = __shfl_sync(0xffffffffu, mine_r, base + i);
                const float u = fmaf(n1.w, rr[7], n1.z * rr[6]) + fmaf(n1.y, rr[5], n1.x * rr[4]) + (fmaf(n0.w, rr[3], n0.z * rr[2]) + fmaf(n0.y, rr[1], n0.x * rr[0]));
                const float write = own.w * u;
                float o = own.z * z[1];
                o = fmaf(r0.x, rr[0], o); o = fmaf(r0.y, rr[1], o); o = fmaf(r0.z, rr[2], o); o = fmaf(r0.w, rr[3], o);
                o = fmaf(r1.x, rr[4], o); o = fmaf(r1.y, rr[5], o); o = fmaf(r1.z, rr[6], o); o = fmaf(r1.w, rr[7], o);
                const int t = t0 + BLOCK * b + row;
                if (sub < BLOCK && t < last && col0 + c < p) a.out[(size_t)t * a.ldo + (size_t)h * p + col0 + c] = o;
#pragma unroll
                for (int i = 0; i < BLOCK; ++i) {
                    const float wi = __shfl_sync(0xffffffffu, write, base + i);
                    const f32x2 w2 = pack2(wi, wi);
#pragma unroll
                    for (int e = 0; e < P2; ++e) S[c][e] = fma2(k[i][e], w2, S[c][e]);
                }
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
    // An ordinary launch, which waits for the kernel before it: let in early, the blocks would crowd on the first SMs that have
    // room (there are about as many blocks as SMs), and the walk would take twice its time.
    kernel<<<dim3((a.p + Tile::COLS - 1) / Tile::COLS, a.heads, a.n_rows), 32 * W, sizeof(Tile), s>>>(a, vec_state);
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

// The requests `rows`, each with two tokens or more, eight tokens at a time.
LLME_API int llme_delta_portions(const LlmeDeltaArgs* args, cudaStream_t stream) {
    const LlmeDeltaArgs& a = *args;
    if (a.n_rows <= 0) return 0;
    if (int rc = check(a)) return rc;
    if (!a.unit || !a.coef || ((uintptr_t)a.unit | (uintptr_t)a.coef) % 16) LLME_REFUSE("delta_rule: portions need their workspace");
    const dim3 blocks(a.tokens / BLOCK + a.requests + 1, (a.qk_groups + PREPARE_WARPS - 1) / PREPARE_WARPS);
    llme_launch(delta_prepare_kernel, blocks, dim3(32 * PREPARE_WARPS), 0, stream, a);
    const int vs = rows_of_16(a.state, a.state_stride, a.n);
    // 16 columns a block either way: one a lane on four warps where there are few blocks (the walk's latency counts: 297 against
    // 350 us for 2,048 tokens of 16 heads of 128 x 128), two a lane on two warps where there are many (what is read from shared
    // memory counts: 410 against 465 us for 32 heads, 168 against 237 us for four requests of 512 tokens)
    const bool many = (long long)((a.p + 15) / 16) * a.heads * a.n_rows >= 200;
    if (a.n <= 32) return many ? launch_tile<8, 1, 2, 2, 3>(a, vs, stream) : launch_tile<8, 1, 1, 4, 3>(a, vs, stream);
    if (a.n <= 64) return many ? launch_tile<8, 2, 2, 2, 3>(a, vs, stream) : launch_tile<8, 2, 1, 4, 3>(a, vs, stream);
    if (a.n <= 128) return many ? launch_tile<8, 4, 2, 2, 3>(a, vs, stream) : launch_tile<8, 4, 1, 4, 3>(a, vs, stream);
    if (a.n <= 256) return launch_tile<16, 4, 1, 4, 3>(a, vs, stream);
    return launch_tile<32, 4, 1, 4, 2>(a, vs, stream);
}
