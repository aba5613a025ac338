// Differential attention of single decoded tokens on the tensor cores (bfloat16, mma.sync m16n8k16, 32-bit scores and sums), compiled
// per pair of sizes: -DDK=<query/key size of a map> -DDV=<value size>, multiples of 16 up to 128.
//
// A head has two maps, softmaxes with queries and keys of their own over the same values.  A block serves one request, one value
// head (with the two key heads that are its maps), up to eight of its query heads and one share of the request's keys: rows 0-7
// of its 16-row tile are the heads under map 1, rows 8-15 the same heads under map 2, so both maps' probabilities are one operand
// of the product with the values and no value is read twice.  The four warps work independently: warp w takes the 16-key
// sub-tiles w, w + 4, ... of the block's share through a cp.async pipeline of its own.  At the end the warps' parts meet in
// shared memory and the block's part (maximum, sum, unnormalised output per row) goes to scratch memory; a second kernel adds
// the shares of both maps and writes the finished head: u = a1 - weight a2, u / sqrt(mean(u^2) + eps) * scale.
//
// A cache page holds [key heads][page_size][DK] keys (key head 2 g + m is map m of value head g), then [value heads][page_size][DV]
// values.  A token's result depends only on its own query and the keys of its request, never on what else is in the launch.
#include "common.cuh"
#include "kernel_args.h"

#ifndef DK
#error "compile with -DDK=<query/key size> -DDV=<value size>"
#endif
static_assert(DK % 16 == 0 && DV % 16 == 0 && DK >= 16 && DV >= 16 && DK <= 128 && DV <= 128, "sizes: multiples of 16 up to 128");

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

namespace {

typedef __nv_bfloat16 bf16;
constexpr int THREADS = 128, WARPS = THREADS / 32, SUB = 16, HEADS = 8, STAGES = 3;
constexpr int LDK = DK + 8, LDV = DV + 8;                      // rows apart from one another's banks
constexpr int STAGE_ELEMS = SUB * (2 * LDK + LDV);
constexpr int PART = DV + 2;                                   // a row's part: maximum (base 2), sum, outputs
constexpr int SMEM_BYTES = WARPS * STAGES * STAGE_ELEMS * (int)sizeof(bf16);
static_assert(WARPS * 16 * PART * 4 <= SMEM_BYTES, "the warps' parts take the place of the stages");
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(gmem), "r"(valid ? 16 : 0));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* smem) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const void* smem) {
    const unsigned a = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float* d, const unsigned* a, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const unsigned*>(&v);
}

// Sixteen rows of N values, one behind the other in a page: every lane's addresses are a constant apart.
template <int N, int LD>
__device__ __forceinline__ void load_rows(bf16* dst, const bf16* src, int lane) {
    constexpr int C = N / 8, PASSES = (SUB * C + 31) / 32;
    if (32 % C == 0) {
        dst += (lane / C) * LD + (lane % C) * 8;
        src += (lane / C) * N + (lane % C) * 8;
#pragma unroll
        for (int i = 0; i < PASSES; ++i) cp_async16(dst + i * (32 / C) * LD, src + i * (32 / C) * N, true);
    } else {
#pragma unroll
        for (int i = 0; i < PASSES; ++i) {
            const int idx = lane + 32 * i;
            if (SUB * C % 32 == 0 || idx < SUB * C) cp_async16(dst + (idx / C) * LD + (idx % C) * 8, src + idx * 8, true);
        }
    }
}

// grid (splits, value heads * chunks of eight query heads, requests)
__global__ void __launch_bounds__(THREADS) maps_decode_kernel(LlmeMapsDecodeArgs a) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int req = a.rows[blockIdx.z], rep = a.heads / a.groups, chunks = (rep + HEADS - 1) / HEADS;
    const int g = blockIdx.y / chunks, h0 = (blockIdx.y - g * chunks) * HEADS;
    const int ctx = a.ctx_lens[req], ps = a.page_size;
    const int* bt = a.block_tables + (size_t)a.table_rows[req] * a.max_blocks;
    const size_t page_elems = (size_t)ps * a.groups * (2 * DK + DV);
    const bf16* cache = (const bf16*)a.cache;
    const int subs = (ctx + SUB - 1) / SUB, per = (subs + a.splits - 1) / a.splits;
    const int first = blockIdx.x * per + warp, last = min(subs, ((int)blockIdx.x + 1) * per);
    bf16* stages = (bf16*)smem_raw + (size_t)warp * STAGES * STAGE_ELEMS;
    const bool one_page = ps % SUB == 0;                       // a sub-tile then lies in one page
    const int ps_shift = (ps & (ps - 1)) == 0 ? __ffs(ps) - 1 : -1;

    auto block_of = [&](int j) { return ps_shift >= 0 ? j >> ps_shift : j / ps; };
    // The page of a warp's sub-tile, looked up one sub-tile before its keys are asked for: the look-up's latency is then not in
    // front of theirs.
    auto page_of = [&](int sub) -> int { return one_page && sub < last ? bt[block_of(sub * SUB)] : 0; };
    const size_t k1_at = (size_t)2 * g * ps * DK, k2_at = k1_at + (size_t)ps * DK, v_at = (size_t)2 * a.groups * ps * DK + (size_t)g * ps * DV;
    auto load = [&](int sub, int stage, int page) {
        bf16* dst = stages + (size_t)stage * STAGE_ELEMS;
        const int j0 = sub * SUB;
        if (one_page && j0 + SUB <= ctx) {                     // the usual case: sixteen rows of one page, addresses a constant apart
            const bf16* at = cache + (size_t)page * page_elems;
            const int off = j0 - block_of(j0) * ps;
            load_rows<DK, LDK>(dst, at + k1_at + (size_t)off * DK, lane);
            load_rows<DK, LDK>(dst + SUB * LDK, at + k2_at + (size_t)off * DK, lane);
            load_rows<DV, LDV>(dst + 2 * SUB * LDK, at + v_at + (size_t)off * DV, lane);
            return;
        }
#pragma unroll 1
        for (int r = 0; r < SUB; ++r) {                        // row by row; rows behind the last key become zeros
            const int j = j0 + r;
            const bool ok = j < ctx;
            const int blk = ok ? block_of(j) : 0;
            const bf16* at = cache + (ok ? (size_t)bt[blk] * page_elems : 0);
            const size_t off = ok ? j - blk * ps : 0;
            if (lane < DK / 8) cp_async16(dst + r * LDK + lane * 8, at + (ok ? k1_at + off * DK : 0) + lane * 8, ok);
            if (lane < DK / 8) cp_async16(dst + (SUB + r) * LDK + lane * 8, at + (ok ? k2_at + off * DK : 0) + lane * 8, ok);
            if (lane < DV / 8) cp_async16(dst + 2 * SUB * LDK + r * LDV + lane * 8, at + (ok ? v_at + off * DV : 0) + lane * 8, ok);
        }
    };

    unsigned qf[DK / 16][4];                                   // rows: map 1's heads, then map 2's
    const float sc = a.scale * LOG2E;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f}, o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.0f;

    // Two sub-tiles are on their way while one is worked on.  Keys that earlier steps stored are asked for before the kernel before
    // this one (it stores the newest key and finishes the queries) is done.
    int stage = 0, fill = 0, page = page_of(first);
    bool waited = false;
#pragma unroll 1
    for (int it = 0;; ++it) {
        const int ahead = first + it * WARPS, sub = ahead - 2 * WARPS;
        if (!waited && (it == 2 || (ahead + 1) * SUB >= ctx)) {
            pdl_wait();
            waited = true;
        }
        if (ahead < last) load(ahead, fill, page);
        cp_async_commit();
        fill = fill == STAGES - 1 ? 0 : fill + 1;
        page = page_of(ahead + WARPS);
        if (it < 2) continue;
        if (it == 2) {
            const bf16* q = (const bf16*)a.q + ((size_t)a.cu_q_lens[req] * a.heads * 2 + (size_t)2 * g * rep) * DK;
            const int h = h0 + (lane >> 2);
            const bool ok = h < rep;
#pragma unroll
            for (int k = 0; k < DK / 16; ++k)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    qf[k][e] = ok ? *reinterpret_cast<const unsigned*>(q + ((size_t)(e & 1) * rep + h) * DK + k * 16 + (e >> 1) * 8 + (lane & 3) * 2) : 0u;
        }
        if (sub >= last) break;
        cp_async_wait<2>();
        __syncwarp();
        const bf16* K = stages + (size_t)stage * STAGE_ELEMS;
        const bf16* V = K + 2 * SUB * LDK;
        float s[2][2][4] = {};                                 // [map][keys 0-7 | 8-15]
#pragma unroll
        for (int k = 0; k < DK / 16; ++k)
#pragma unroll
            for (int mp = 0; mp < 2; ++mp) {
                unsigned b0, b1, b2, b3;
                ldmatrix_x4(b0, b1, b2, b3, K + mp * SUB * LDK + ((lane & 7) + (lane >> 4) * 8) * LDK + k * 16 + ((lane >> 3) & 1) * 8);
                mma_bf16(s[mp][0], qf[k], b0, b1);
                mma_bf16(s[mp][1], qf[k], b2, b3);
            }
        float p[2][4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {                      // values 0, 1 belong to a row of map 1, values 2, 3 to the same head's of map 2
                const int j = sub * SUB + n * 8 + (lane & 3) * 2 + (e & 1);
                p[n][e] = j < ctx ? s[e >> 1][n][e] * sc : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], p[n][e]);
            }
        float corr[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            const float m_new = fmaxf(m[h], mx[h]);            // (a sub-tile holds at least one key of the request: finite)
            corr[h] = exp2f(m[h] - m_new);
            m[h] = m_new;
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                p[n][e] = exp2f(p[n][e] - m[e >> 1]);
                sum[e >> 1] += p[n][e];
            }
#pragma unroll
        for (int h = 0; h < 2; ++h) l[h] = l[h] * corr[h] + sum[h];      // (this lane's share; the lanes are added up at the end)
        if (__any_sync(0xffffffffu, corr[0] != 1.0f || corr[1] != 1.0f)) {      // (a maximum moves in the first few sub-tiles, hardly ever later)
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) {
                o[n][0] *= corr[0]; o[n][1] *= corr[0];
                o[n][2] *= corr[1]; o[n][3] *= corr[1];
            }
        }
        const unsigned pf[4] = {pack_bf16(p[0][0], p[0][1]), pack_bf16(p[0][2], p[0][3]), pack_bf16(p[1][0], p[1][1]), pack_bf16(p[1][2], p[1][3])};
#pragma unroll
        for (int n = 0; n < DV / 8; n += 2) {
            unsigned b0, b1, b2, b3;
            ldmatrix_x4_trans(b0, b1, b2, b3, V + ((lane & 7) + ((lane >> 3) & 1) * 8) * LDV + n * 8 + (lane >> 4) * 8);
            mma_bf16(o[n], pf, b0, b1);
            mma_bf16(o[n + 1], pf, b2, b3);
        }
        __syncwarp();                                          // every lane is done with the stage before it is filled again
        stage = stage == STAGES - 1 ? 0 : stage + 1;
    }
    cp_async_wait<0>();
    __syncthreads();
    pdl_launch_dependents();
    float* parts = (float*)smem_raw;                           // [warp][16][PART]
    {
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
            l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
            float* part = parts + ((size_t)warp * 16 + (lane >> 2) + h * 8) * PART;
            if ((lane & 3) == 0) {
                part[0] = m[h];
                part[1] = l[h];
            }
#pragma unroll
            for (int n = 0; n < DV / 8; ++n) {
                part[2 + n * 8 + (lane & 3) * 2] = o[n][h * 2];
                part[2 + n * 8 + (lane & 3) * 2 + 1] = o[n][h * 2 + 1];
            }
        }
    }
    __syncthreads();
    float* out = a.scratch + (((size_t)blockIdx.z * gridDim.y + blockIdx.y) * a.splits + blockIdx.x) * 16 * PART;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int row = warp * 4 + i;
        if (h0 + (row & 7) >= rep) continue;
        float mm = -INFINITY, w[WARPS], ll = 0.0f;
#pragma unroll
        for (int v = 0; v < WARPS; ++v) mm = fmaxf(mm, parts[((size_t)v * 16 + row) * PART]);
        const float base = mm == -INFINITY ? 0.0f : mm;        // a share without keys
#pragma unroll
        for (int v = 0; v < WARPS; ++v) {
            w[v] = exp2f(parts[((size_t)v * 16 + row) * PART] - base);
            ll += parts[((size_t)v * 16 + row) * PART + 1] * w[v];
        }
        for (int d = lane; d < DV; d += 32) {
            float acc = 0.0f;
#pragma unroll
            for (int v = 0; v < WARPS; ++v) acc += parts[((size_t)v * 16 + row) * PART + 2 + d] * w[v];
            out[row * PART + 2 + d] = acc;
        }
        if (lane == 0) {
            out[row * PART] = mm;
            out[row * PART + 1] = ll;
        }
    }
}

// One block per (request, head): its warps deal the shares of both maps among themselves; then the difference and its norm.
__global__ void __launch_bounds__(THREADS) maps_finish_kernel(LlmeMapsDecodeArgs a) {
    __shared__ float sums[WARPS][DV], red[32];
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.x;
    const int req = a.rows[blockIdx.y], rep = a.heads / a.groups, chunks = (rep + HEADS - 1) / HEADS;
    const int g = h / rep, hh = h - g * rep, unit = g * chunks + hh / HEADS;
    const float* parts = a.scratch + ((size_t)blockIdx.y * a.groups * chunks + unit) * a.splits * 16 * PART + (size_t)(hh % HEADS) * PART;
    constexpr int R = (DV + 31) / 32;
    float f[2], u[R];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {                           // lane s looks after share s
        const float* mine = parts + (size_t)lane * 16 * PART + (size_t)mp * 8 * PART;
        const bool in = lane < a.splits;
        const float ms = in ? mine[0] : -INFINITY, ls = in ? mine[1] : 0.0f;
        const float top = warp_max(ms), w = in ? exp2f(ms - top) : 0.0f;
        f[mp] = (mp == 0 ? 1.0f : -a.diff_weight) / warp_sum(ls * w) * w;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) u[i] = 0.0f;
#pragma unroll 4
    for (int s = warp; s < a.splits; s += WARPS) {
        const float f1 = __shfl_sync(0xffffffffu, f[0], s), f2 = __shfl_sync(0xffffffffu, f[1], s);
        const float* mine = parts + (size_t)s * 16 * PART + 2;
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int d = lane + 32 * i;
            if (d < DV) u[i] = fmaf(f2, mine[8 * PART + d], fmaf(f1, mine[d], u[i]));
        }
    }
#pragma unroll
    for (int i = 0; i < R; ++i)
        if (lane + 32 * i < DV) sums[warp][lane + 32 * i] = u[i];
    __syncthreads();
    const int d = threadIdx.x;                                 // (DV is at most the block's width)
    float v = 0.0f;
    if (d < DV) {
#pragma unroll
        for (int w = 0; w < WARPS; ++w) v += sums[w][d];
    }
    const float r = a.diff_scale / sqrtf(block_sum(v * v, red) / (float)DV + a.diff_eps);
    if (d < DV) ((bf16*)a.out)[((size_t)a.cu_q_lens[req] * a.heads + h) * DV + d] = __float2bfloat16_rn(v * r);
}

}  // namespace

// (request, value head, eight query heads) units of a launch, and the scratch floats of `splits` shares each.
LLME_API long long llme_maps_decode_scratch_floats(int n_rows, int heads, int groups, int splits) {
    const int rep = heads / groups;
    return (long long)n_rows * groups * ((rep + HEADS - 1) / HEADS) * splits * 16 * PART;
}

LLME_API int llme_maps_decode(const LlmeMapsDecodeArgs* args, cudaStream_t stream) {
    const LlmeMapsDecodeArgs& a = *args;
    if (a.n_rows <= 0) return 0;
    if (!a.q || !a.cache || !a.out || !a.scratch || !a.rows || !a.cu_q_lens || !a.ctx_lens || !a.table_rows || !a.block_tables) LLME_REFUSE("maps_decode: null pointer");
    if (a.heads <= 0 || a.groups <= 0 || a.heads % a.groups || a.page_size <= 0 || a.max_blocks <= 0) LLME_REFUSE("maps_decode: bad size");
    if (a.splits < 1 || a.splits > 32) LLME_REFUSE("maps_decode: %d shares, this build takes 1 to 32", a.splits);
    if (!(a.diff_eps > 0.0f)) LLME_REFUSE("maps_decode: eps must be positive");
    if (((uintptr_t)a.q | (uintptr_t)a.cache) & 15) LLME_REFUSE("maps_decode: operands must be 16-byte aligned");
    const int units = a.groups * ((a.heads / a.groups + HEADS - 1) / HEADS);
    if (units > 65535 || a.n_rows > 65535) LLME_REFUSE("maps_decode: too many heads or requests for one launch");
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(maps_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_BYTES) != cudaSuccess)
            LLME_REFUSE("maps_decode: %d bytes of shared memory are not available", SMEM_BYTES);
        configured = true;
    }
    llme_launch(maps_decode_kernel, dim3(a.splits, units, a.n_rows), dim3(THREADS), (size_t)SMEM_BYTES, stream, a);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) {
        snprintf(llme_error_buffer(), 512, "%s", cudaGetErrorString(e));
        return (int)e;
    }
    llme_launch(maps_finish_kernel, dim3(a.heads, a.n_rows), dim3(THREADS), 0, stream, a);
    LLME_LAUNCH_STATUS();
}
