// The grouped product of a mixture of experts for many tokens on the fifth-generation tensor cores: one product per expert over
// the (token, choice) pairs that were routed to it, which stand side by side in the list of pairs.
//
// Rows that have to be gathered by token are first written side by side (gather_rows_kernel); from then on a tile of 128 pairs of
// an expert is a plain box of a matrix, and the pipeline is that of the dense product (gemm_tcgen05.cu): TMA brings 128 x 64
// pieces of the rows and 256 x 64 pieces of the expert's matrix into shared memory (128-byte swizzle, four stages), one thread
// issues tcgen05.mma (128 x 256 x 16) into tensor memory, double-buffered, and four warps read the accumulator back, apply the
// activation and store whole 128-byte pieces of the rows, scattered by pair where asked.  A box at the end of an expert's rows
// runs on into the next expert's: those rows are computed and not stored.  The experts' matrices are one matrix [E n, k].
//
// Persistent: one block per SM walks over the tiles (expert, 128 rows, columns), which it counts from the routing's offsets.
// act 1: a tile's 256 accumulator columns are 128 gate rows and the 128 up rows of the same outputs, silu(gate) * up is stored;
// act 2: max(product, 0)^2.  Waits are bounded as in the dense product; llme_grouped_tcgen05_status() reports a give-up.
#include <cuda.h>

#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

namespace {

#include "umma.cuh"

constexpr int BN = 256, STAGES = 4, MAX_EXPERTS = 1024;
constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2, STAGING = 4 * 4096;
constexpr unsigned TMEM_COLS = 512;
constexpr size_t SMEM = 1024 + (size_t)STAGES * (A_BYTES + B_BYTES) + STAGING + (2 * STAGES + 4) * 8 + 16 + 2 * (MAX_EXPERTS + 1) * 4;
static_assert(SMEM <= 232448, "the block's shared memory must fit an SM");

struct Tile { int row0, end, col0, expert; };      // first row, end of the expert's rows, first output column

// Tile t: the column tiles of a row tile follow one another.
__device__ __forceinline__ Tile find_tile(const int* starts, const int* offsets, int E, int n_tiles, int out_cols, int t) {
    const int m = t / n_tiles;
    int lo = 0, hi = E;                             // the last expert whose first row tile is not behind m
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (starts[mid] <= m) lo = mid; else hi = mid;
    }
    Tile o;
    o.expert = lo;
    o.row0 = offsets[lo] + (m - starts[lo]) * BM;
    o.end = offsets[lo + 1];
    o.col0 = (t - m * n_tiles) * out_cols;
    return o;
}

template <int ACT, typename O>
__global__ void __launch_bounds__(THREADS, 1)
grouped_tcgen05_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, LlmeGroupedArgs a) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* a_tiles = smem;
    unsigned char* b_tiles = smem + STAGES * A_BYTES;
    unsigned char* staging = b_tiles + STAGES * B_BYTES;
    unsigned long long* full = reinterpret_cast<unsigned long long*>(staging + STAGING);
    unsigned long long* empty = full + STAGES;
    unsigned long long* acc_full = empty + STAGES;                 // [2]
    unsigned long long* acc_empty = acc_full + 2;                  // [2]
    unsigned* tmem_holder = reinterpret_cast<unsigned*>(acc_empty + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);
    int* offsets = reinterpret_cast<int*>(tmem_holder + 4);        // [E + 1]
    int* starts = offsets + MAX_EXPERTS + 1;                       // [E + 1]: the first row tile of every expert

    constexpr int OUT_COLS = ACT == 1 ? BN / 2 : BN;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = a.num_experts;
    const int n_out = ACT == 1 ? a.n / 2 : a.n, n_tiles = (n_out + OUT_COLS - 1) / OUT_COLS, k_blocks = (a.k + BK - 1) / BK;
    for (int e = threadIdx.x; e <= E; e += THREADS) offsets[e] = a.offsets[e];
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(full + s, 1);
            mbar_init(empty + s, 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(acc_full + b, 1);
            mbar_init(acc_empty + b, 4);                           // one arrival per epilogue warp
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    if (warp == 0) {                                               // running count of row tiles
        int base = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + lane, tiles = e < E ? (offsets[e + 1] - offsets[e] + BM - 1) / BM : 0;
            int sum = tiles;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += up;
            }
            if (e < E) starts[e] = base + sum - tiles;
            base += __shfl_sync(0xffffffffu, sum, 31);
        }
        if (lane == 0) starts[E] = base;
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_holder)), "r"(TMEM_COLS));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem_base = *tmem_holder;
    const int tiles = starts[E] * n_tiles;

    if (warp == 0) {
        // ------------------------------------------------------------------ producer
        if (lane == 0) {
            unsigned it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const Tile tl = find_tile(starts, offsets, E, n_tiles, OUT_COLS, t);
                const int w0 = tl.expert * a.n + tl.col0, w1 = ACT == 1 ? w0 + n_out : w0 + BN / 2;
                for (int kb = 0; kb < k_blocks; ++kb, ++it) {
                    const unsigned s = it % STAGES;
                    ok = mbar_wait(empty + s, ((it / STAGES) & 1) ^ 1, abort_flag, 1) && !*abort_flag;
                    if (!ok) break;
                    mbar_expect_tx(full + s, A_BYTES + B_BYTES);
                    tma_load_2d(a_tiles + s * A_BYTES, &map_x, kb * BK, tl.row0, full + s);
                    tma_load_2d(b_tiles + s * B_BYTES, &map_w, kb * BK, w0, full + s);
                    tma_load_2d(b_tiles + s * B_BYTES + B_BYTES / 2, &map_w, kb * BK, w1, full + s);
                }
            }
            if (!ok) {                              // gave up somewhere: let the copies that may still be in flight land
                const unsigned first = it > STAGES ? it - STAGES : 0;
                for (unsigned j = first; j < it; ++j)
                    for (unsigned i = 0; i < WAIT_LIMIT && !mbar_try_wait(full + j % STAGES, (j / STAGES) & 1); ++i) {}
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------------------------ MMA issuer
        if (lane == 0) {
            constexpr unsigned idesc = umma_idesc(BM, BN);
            unsigned it = 0;
            bool ok = true;
            int i = 0;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++i) {
                const int b = i & 1;
                ok = mbar_wait(acc_empty + b, ((i >> 1) & 1) ^ 1, abort_flag, 4);   // the epilogue has drained this buffer
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned tmem_d = tmem_base + (unsigned)(b * BN);
                for (int kb = 0; kb < k_blocks; ++kb, ++it) {
                    const unsigned s = it % STAGES;
                    ok = mbar_wait(full + s, (it / STAGES) & 1, abort_flag, 2);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const unsigned long long da = umma_desc(a_tiles + s * A_BYTES), db = umma_desc(b_tiles + s * B_BYTES);
#pragma unroll
                    for (int k = 0; k < BK / UMMA_K; ++k) umma_bf16(tmem_d, da + 2 * k, db + 2 * k, idesc, (kb > 0 || k > 0) ? 1u : 0u);
                    umma_commit(empty + s);
                }
                if (!ok) break;
                umma_commit(acc_full + b);
            }
        }
    } else {
        // ------------------------------------------------------------------ epilogue (warps 2..5)
        const int quarter = warp & 3;               // the TMEM lanes this warp may read: 32 * (warp % 4) ...
        constexpr int COLS = 128 / (int)sizeof(O);  // output columns per 128-byte piece of a row
        constexpr int EACH = 16 / (int)sizeof(O);   // and per 16 bytes
        unsigned char* buf = staging + quarter * 4096;
        O* out = (O*)a.out;
        int i = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x, ++i) {
            const Tile tl = find_tile(starts, offsets, E, n_tiles, OUT_COLS, t);
            const int row = tl.row0 + quarter * 32 + lane, b = i & 1;
            const int dst = row < tl.end ? (a.scatter ? a.order[row] : row) : -1;
            if (!__all_sync(0xffffffffu, mbar_wait(acc_full + b, (i >> 1) & 1, abort_flag, 3))) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            __syncwarp();
            const unsigned tmem_row = tmem_base + ((unsigned)(quarter * 32) << 16) + (unsigned)(b * BN);
#pragma unroll 1
            for (int c = 0; c < OUT_COLS; c += COLS) {
#pragma unroll
                for (int half = 0; half < COLS / 32; ++half) {
                    unsigned v[32];
                    tmem_ld_32x32(tmem_row + (unsigned)(c + half * 32), v);
                    if (ACT == 1) {
                        unsigned up[32];
                        tmem_ld_32x32(tmem_row + (unsigned)(BN / 2 + c + half * 32), up);
                        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                        for (int j = 0; j < 32; ++j) {
                            const float g = __bfloat162float(__float2bfloat16_rn(__uint_as_float(v[j])));
                            const float u = __bfloat162float(__float2bfloat16_rn(__uint_as_float(up[j])));
                            v[j] = __float_as_uint(silu_mul_bf16(g, u));
                        }
                    } else {
                        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                        if (ACT == 2) {
#pragma unroll
                            for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(relu2(__uint_as_float(v[j])));
                        }
                        if (ACT == 3) {
#pragma unroll
                            for (int j = 0; j < 32; ++j) v[j] = __float_as_uint(gelu_erf(__uint_as_float(v[j])));
                        }
                    }
                    if (c + COLS >= OUT_COLS && half == COLS / 32 - 1) {     // the tile has left tensor memory
                        asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
                        __syncwarp();
                        if (lane == 0) mbar_arrive(acc_empty + b);
                    }
                    // row `lane` of the piece; its 16-byte chunk q goes to place q ^ (lane % 8), so that neither side collides
                    if (sizeof(O) == 4) {
#pragma unroll
                        for (int q = 0; q < 8; ++q)
                            *reinterpret_cast<uint4*>(buf + lane * 128 + ((q ^ (lane & 7)) << 4)) = make_uint4(v[4 * q], v[4 * q + 1], v[4 * q + 2], v[4 * q + 3]);
                    } else {
#pragma unroll
                        for (int q = 0; q < 4; ++q) {
                            uint4 pk;
                            unsigned* pw = reinterpret_cast<unsigned*>(&pk);
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(v[8 * q + 2 * e]), __uint_as_float(v[8 * q + 2 * e + 1]));
                                pw[e] = *reinterpret_cast<unsigned*>(&h);
                            }
                            *reinterpret_cast<uint4*>(buf + lane * 128 + (((half * 4 + q) ^ (lane & 7)) << 4)) = pk;
                        }
                    }
                }
                __syncwarp();
                const int q = lane & 7, col = tl.col0 + c + q * EACH;
#pragma unroll
                for (int rr = lane >> 3; rr < 32; rr += 4) {                 // eight lanes store a row's 128 bytes
                    const int to = __shfl_sync(0xffffffffu, dst, rr);
                    const uint4 piece = *reinterpret_cast<const uint4*>(buf + rr * 128 + ((q ^ (rr & 7)) << 4));
                    if (to >= 0 && col < n_out) *reinterpret_cast<uint4*>(out + (size_t)to * a.ldo + col) = piece;
                }
                __syncwarp();
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS));
    }
}

// rows[r] = x[order[r] / top_k]: a pair's token, side by side with the other pairs of its expert
__global__ void gather_rows_kernel(const uint4* __restrict__ x, long long ldx, uint4* __restrict__ rows, const int* __restrict__ order, int top_k,
                                   int pieces) {
    pdl_launch_dependents();
    pdl_wait();
    const uint4* from = x + (size_t)(order[blockIdx.x] / top_k) * ldx;
    uint4* to = rows + (size_t)blockIdx.x * pieces;
    for (int i = threadIdx.x; i < pieces; i += blockDim.x) to[i] = from[i];
}

template <int ACT, typename O>
int launch(const LlmeGroupedArgs& a, const void* x, long long ldx, cudaStream_t s) {
    alignas(64) CUtensorMap mx, mw;
    if (int rc = make_map(&mx, x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.pairs, a.k, ldx, BM, BK)) return rc;
    if (int rc = make_map(&mw, a.w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, (long long)a.num_experts * a.n, a.k, a.ldw, BN / 2, BK)) return rc;
    auto kernel = grouped_tcgen05_kernel<ACT, O>;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
        if (e != cudaSuccess) LLME_REFUSE("grouped_tcgen05: cannot reserve %zu bytes of shared memory: %s", SMEM, cudaGetErrorString(e));
        configured = true;
    }
    kernel<<<sm_count(), THREADS, SMEM, s>>>(mx, mw, a);
    LLME_LAUNCH_STATUS();
}

}  // namespace

// 1 if llme_grouped_tcgen05 takes this product (whole 16-byte pieces everywhere, the experts' matrices one behind the other).
LLME_API int llme_grouped_tcgen05_supports(const LlmeGroupedArgs* args, int out_dtype) {
    const LlmeGroupedArgs& a = *args;
    const int n_out = a.act == 1 ? a.n / 2 : a.n, el = out_dtype == LLME_F32 ? 4 : 2;
    return a.num_experts >= 1 && a.num_experts <= MAX_EXPERTS && a.k >= 8 && a.k % 8 == 0 && a.ldx % 8 == 0 && a.ldw % 8 == 0 && a.n >= 8 &&
           n_out % 8 == 0 && a.w_expert == a.n * a.ldw && (long long)a.num_experts * a.n < (1LL << 31) && a.ldo * el % 16 == 0 &&
           (((uintptr_t)a.x | (uintptr_t)a.w | (uintptr_t)a.out) & 15) == 0;
}

// bfloat16 operands; `rows` [pairs, k]: where rows that are gathered by token come to stand side by side (not needed without).
LLME_API int llme_grouped_tcgen05(const LlmeGroupedArgs* args, void* rows, int out_dtype, cudaStream_t stream) {
    const LlmeGroupedArgs& a = *args;
    if (a.pairs <= 0 || a.n <= 0) return 0;
    if (!a.x || !a.w || !a.out || !a.offsets || !a.order || a.top_k <= 0) LLME_REFUSE("grouped_tcgen05: null pointer or no choices");
    if (a.act < 0 || a.act > 3 || (out_dtype != LLME_F32 && out_dtype != LLME_BF16) || !llme_grouped_tcgen05_supports(args, out_dtype))
        LLME_REFUSE("grouped_tcgen05: sizes or strides that are not whole 16-byte pieces");
    const void* x = a.x;
    long long ldx = a.ldx;
    if (a.gather) {
        if (!rows || (uintptr_t)rows % 16) LLME_REFUSE("grouped_tcgen05: gathered rows need a place");
        const int pieces = a.k / 8;
        llme_launch(gather_rows_kernel, dim3(a.pairs), dim3(pieces >= 256 ? 256 : (pieces + 31) / 32 * 32), 0, stream, (const uint4*)a.x, a.ldx / 8,
                    (uint4*)rows, a.order, a.top_k, pieces);
        x = rows;
        ldx = a.k;
    }
    if (out_dtype == LLME_F32)
        return a.act == 1 ? launch<1, float>(a, x, ldx, stream) : a.act == 2 ? launch<2, float>(a, x, ldx, stream) : a.act == 3 ? launch<3, float>(a, x, ldx, stream) : launch<0, float>(a, x, ldx, stream);
    return a.act == 1 ? launch<1, bf16>(a, x, ldx, stream) : a.act == 2 ? launch<2, bf16>(a, x, ldx, stream) : a.act == 3 ? launch<3, bf16>(a, x, ldx, stream) : launch<0, bf16>(a, x, ldx, stream);
}

// Reads and clears the error flag of the kernel (synchronises the device).  0 = no wait ever gave up.
LLME_API int llme_grouped_tcgen05_status() {
    int v = 0, zero = 0;
    if (cudaMemcpyFromSymbol(&v, g_status, sizeof(int)) != cudaSuccess) return -1;
    if (v != 0) cudaMemcpyToSymbol(g_status, &zero, sizeof(int));
    return v;
}
