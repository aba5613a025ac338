// A mixture of experts: routing (sigmoid scores, the largest few chosen, perhaps only inside the groups with the largest sums of
// their two best scores, weights normalised over the chosen; or the
// softmax over the chosen logits alone; or the softmax over all with a correction of the choice and a limit to the best
// groups), the list
// of (token, choice) pairs expert by expert, one product per expert over its pairs (plain form: any sizes, both types,
// 32-bit FMA in a fixed order of k, so that a row never depends on what shares its tile), and the weighted sum of a
// token's pairs in the order of its choices.  The tensor-core form of the grouped product is csrc/moe_tc.cu.
#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

// ----------------------------------------------------------------------------- routing
// One warp per token: `top_k` rounds of a warp-wide argmax over what is not chosen yet (ties: the lower index).  Modes 0 and 1 choose
// by the logits, mode 2 by the softmax over all of them plus a correction (`choice`, the warp's place in shared memory).
__device__ __forceinline__ void warp_argmax(float& best, int& bi) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (oi >= 0 && (bi < 0 || ob > best || (ob == best && oi < bi))) { best = ob; bi = oi; }
    }
}

// 32-bit values of shared memory that a warp's routing needs
__host__ __device__ __forceinline__ int route_place(const LlmeMoeRouteArgs& a) {
    return a.mode == 2 ? a.num_experts : (a.mode == 0 && a.keep > 0 && a.keep < a.groups) ? a.num_experts + a.groups : 0;
}

__device__ __forceinline__ void route_token(const LlmeMoeRouteArgs& a, int t, int lane, float* __restrict__ choice) {
    const float* z = a.logits + (size_t)t * a.ld;
    const int E = a.num_experts;
    unsigned taken = 0;                                   // bit i: this lane's i-th choice (lane + 32 i) is chosen, or not on offer
    float total = 0.0f, first = 0.0f, top = -INFINITY, rsum = 1.0f;
    if (a.mode == 2) {
        for (int i = lane; i < E; i += 32) top = fmaxf(top, z[i]);
        top = warp_max(top);
        float sum = 0.0f;
        for (int i = lane; i < E; i += 32) sum += expf(z[i] - top);
        rsum = 1.0f / warp_sum(sum);
        for (int i = lane; i < E; i += 32) choice[i] = expf(z[i] - top) * rsum + (a.correction ? a.correction[i] : 0.0f);
        __syncwarp();
        if (a.keep < a.groups) {
            // the best member of the groups not kept yet names the next group to keep
            const int size = E / a.groups;
            unsigned offered = 0;
            for (int k = 0; k < a.keep; ++k) {
                float best = -INFINITY;
                int bi = -1;
                for (int i = lane, n = 0; i < E; i += 32, ++n)
                    if (!((offered >> n) & 1u) && (bi < 0 || choice[i] > best)) { best = choice[i]; bi = i; }
                warp_argmax(best, bi);
                const int group = bi / size;
                for (int i = lane, n = 0; i < E; i += 32, ++n)
                    if (i / size == group) offered |= 1u << n;
            }
            taken = ~offered;
        }
    }
    if (a.mode == 0 && a.keep > 0 && a.keep < a.groups) {
        // a group is as good as the sum of its two largest scores: lane g adds them up for the groups g, g + 32, ...
        const int size = E / a.groups;
        float* total_of = choice + E;
        for (int i = lane; i < E; i += 32) choice[i] = 1.0f / (1.0f + expf(-z[i]));
        __syncwarp();
        for (int g = lane; g < a.groups; g += 32) {
            float one = -1.0f, two = -1.0f;
            for (int i = g * size; i < (g + 1) * size; ++i) {
                const float s = choice[i];
                two = fmaxf(two, fminf(one, s));
                one = fmaxf(one, s);
            }
            total_of[g] = size > 1 ? one + two : one;
        }
        __syncwarp();
        unsigned offered = 0;
        for (int k = 0; k < a.keep; ++k) {
            float best = -INFINITY;
            int bi = -1;
            for (int g = lane; g < a.groups; g += 32)
                if (total_of[g] >= 0.0f && (bi < 0 || total_of[g] > best)) { best = total_of[g]; bi = g; }
            warp_argmax(best, bi);
            for (int i = lane, n = 0; i < E; i += 32, ++n)
                if (i / size == bi) offered |= 1u << n;
            __syncwarp();
            if (lane == 0) total_of[bi] = -1.0f;               // kept: out of the next rounds
            __syncwarp();
        }
        taken = ~offered;
    }
    float score[8];
    int chosen[8];
    for (int k = 0; k < a.top_k; ++k) {
        float best = -INFINITY;
        int bi = -1;
        for (int i = lane, n = 0; i < E; i += 32, ++n) {
            if ((taken >> n) & 1u) continue;
            const float v = a.mode == 2 ? choice[i] : z[i];
            if (bi < 0 || v > best) { best = v; bi = i; }
        }
        warp_argmax(best, bi);
        if (bi >= 0 && (bi & 31) == lane) taken |= 1u << (bi >> 5);
        if (k == 0) first = best;
        // mode 1: the softmax over the chosen logits alone, relative to the largest of them (the first chosen)
        const float s = a.mode == 2 ? expf(z[bi] - top) * rsum : a.mode == 1 ? expf(best - first) : 1.0f / (1.0f + expf(-best));
        score[k & 7] = s;
        chosen[k & 7] = bi;
        total += s;
        if (a.top_k > 8 && lane == 0) {                   // more choices than the registers hold: store as they come
            a.experts[(size_t)t * a.top_k + k] = bi;
            a.weights[(size_t)t * a.top_k + k] = s;
        }
    }
    const float norm = a.mode == 2 ? a.scale : a.scale / (a.mode == 1 ? total : total + 1e-20f);
    if (lane == 0) {
        for (int k = 0; k < a.top_k; ++k) {
            const size_t at = (size_t)t * a.top_k + k;
            if (a.top_k <= 8) {
                a.experts[at] = chosen[k];
                a.weights[at] = score[k] * norm;
            } else {
                a.weights[at] *= norm;
            }
        }
    }
    __syncwarp();
}

__global__ void moe_route_kernel(LlmeMoeRouteArgs a) {
    extern __shared__ float choices[];                    // mode 2: [warps][E]; mode 0 with groups: [warps][E + groups]
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x * (blockDim.x >> 5) + warp;
    if (t >= a.tokens) return;
    route_token(a, t, lane, choices + (size_t)warp * route_place(a));
    for (int k = lane; k < a.top_k; k += 32) atomicAdd(a.counts + a.experts[(size_t)t * a.top_k + k], 1);
}

// Exclusive sums of counts[0 .. E) (shared memory) into cursor[0 .. E] and offsets[0 .. E], by the block's first warp.
__device__ __forceinline__ void expert_offsets(const int* counts, int E, int* cursor, int* __restrict__ offsets) {
    if (threadIdx.x >= 32) return;
    const int lane = threadIdx.x;
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane, c = e < E ? counts[e] : 0;
        int sum = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        if (e < E) {
            cursor[e] = base + sum - c;
            offsets[e] = base + sum - c;
        }
        base += __shfl_sync(0xffffffffu, sum, 31);
    }
    if (lane == 0) {
        cursor[E] = base;
        offsets[E] = base;
    }
}

// One block: offsets from the counts, the pairs placed expert by expert, the counts cleared for the next launch.  The
// order of the pairs inside an expert's range is whatever the atomics give: no result depends on it, since every row
// of a grouped product is computed by itself.
__global__ void moe_order_kernel(LlmeMoeRouteArgs a) {
    extern __shared__ int cursor[];                       // [E + 1], then the counts [E]
    pdl_launch_dependents();
    pdl_wait();
    const int E = a.num_experts, P = a.tokens * a.top_k;
    int* counts = cursor + E + 1;
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        counts[e] = a.counts[e];
        a.counts[e] = 0;
    }
    __syncthreads();
    expert_offsets(counts, E, cursor, a.offsets);
    __syncthreads();
    for (int i = threadIdx.x; i < P; i += blockDim.x) a.order[atomicAdd(cursor + a.experts[i], 1)] = i;
}

// A step of few tokens: routing and ordering by one block, in one launch.
constexpr int ROUTE_FEW = 64, ROUTE_WARPS = 16;

__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_few_kernel(LlmeMoeRouteArgs a) {
    extern __shared__ float choices[];                    // [warps][route_place], then the cursors [E + 1] and the counts [E]
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = a.num_experts, P = a.tokens * a.top_k;
    int* cursor = (int*)(choices + (size_t)ROUTE_WARPS * route_place(a));
    int* counts = cursor + E + 1;
    for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
    for (int t = warp; t < a.tokens; t += ROUTE_WARPS) route_token(a, t, lane, choices + (size_t)warp * route_place(a));
    __syncthreads();
    for (int i = threadIdx.x; i < P; i += blockDim.x) atomicAdd(counts + a.experts[i], 1);
    __syncthreads();
    expert_offsets(counts, E, cursor, a.offsets);
    __syncthreads();
    for (int i = threadIdx.x; i < P; i += blockDim.x) a.order[atomicAdd(cursor + a.experts[i], 1)] = i;
}

LLME_API int llme_moe_route(const LlmeMoeRouteArgs* args, cudaStream_t stream) {
    const LlmeMoeRouteArgs& a = *args;
    if (a.tokens <= 0) return 0;
    if (!a.logits || !a.experts || !a.weights || !a.offsets || !a.order || !a.counts) LLME_REFUSE("moe_route: null pointer");
    if (a.mode < 0 || a.mode > 2) LLME_REFUSE("moe_route: unknown mode %d", a.mode);
    if (a.num_experts <= 0 || a.num_experts > 1024 || a.top_k <= 0 || a.top_k > a.num_experts)
        LLME_REFUSE("moe_route: %d of %d experts (at most 1024)", a.top_k, a.num_experts);
    const bool grouped = a.mode == 2 || (a.mode == 0 && a.keep > 0 && a.keep < a.groups);
    if (grouped && (a.groups <= 0 || a.num_experts % a.groups || a.keep <= 0 || a.keep > a.groups || a.top_k > a.num_experts / a.groups * a.keep))
        LLME_REFUSE("moe_route: %d of %d groups of %d experts do not offer %d", a.keep, a.groups, a.num_experts, a.top_k);
    const size_t lists = (size_t)(2 * a.num_experts + 1) * sizeof(int), place = (size_t)route_place(a) * sizeof(float);
    if (a.tokens <= ROUTE_FEW && ROUTE_WARPS * place + lists <= 48 * 1024) {
        llme_launch(moe_route_few_kernel, dim3(1), dim3(32 * ROUTE_WARPS), ROUTE_WARPS * place + lists, stream, a);
        LLME_LAUNCH_STATUS();
    }
    const int wpb = 4;
    llme_launch(moe_route_kernel, dim3((a.tokens + wpb - 1) / wpb), dim3(wpb * 32), wpb * place, stream, a);
    cudaError_t e = cudaGetLastError();
    if (e != cudaSuccess) {
        snprintf(llme_error_buffer(), 512, "%s", cudaGetErrorString(e));
        return (int)e;
    }
    llme_launch(moe_order_kernel, dim3(1), dim3(1024), lists, stream, a);
    LLME_LAUNCH_STATUS();
}

// ----------------------------------------------------------------------------- one product per expert, plain form
// The row tiles of all experts are numbered one after the other; a block finds the expert of its tile from the offsets.
__device__ __forceinline__ bool find_tile(const int* __restrict__ offsets, int E, int BM, int tile, int* expert, int* first, int* rows) {
    int seen = 0;
    for (int e = 0; e < E; ++e) {
        const int lo = offsets[e], n = offsets[e + 1] - lo;
        const int tiles = (n + BM - 1) / BM;
        if (tile < seen + tiles) {
            const int at = (tile - seen) * BM;
            *expert = e;
            *first = lo + at;
            *rows = n - at < BM ? n - at : BM;
            return true;
        }
        seen += tiles;
    }
    return false;
}

constexpr int GM = 16, GN = 64, GK = 16;

template <typename T, typename W, typename O>
__global__ void __launch_bounds__(256) grouped_linear_kernel(LlmeGroupedArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ int s_tile[3];
    __shared__ int s_src[GM], s_dst[GM];
    __shared__ float xs[GM][GK + 1];
    __shared__ float ws[2][GN][GK + 1];
    if (threadIdx.x == 0) {
        int e = -1, first = 0, rows = 0;
        if (!find_tile(a.offsets, a.num_experts, GM, blockIdx.y, &e, &first, &rows)) e = -1;
        s_tile[0] = e; s_tile[1] = first; s_tile[2] = rows;
    }
    __syncthreads();
    const int e = s_tile[0], first = s_tile[1], rows = s_tile[2];
    if (e < 0) return;
    if (threadIdx.x < GM) {
        const int r = threadIdx.x;
        const int pair = r < rows ? a.order[first + r] : -1;
        s_src[r] = r < rows ? (a.gather ? pair / a.top_k : first + r) : -1;
        s_dst[r] = r < rows ? (a.scatter ? pair : first + r) : -1;
    }
    __syncthreads();
    const bool gated = a.act == 1;
    const int n_out = gated ? a.n / 2 : a.n;
    const int col0 = blockIdx.x * GN;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;        // row ty, columns tx + 16 c
    const W* w = (const W*)a.w + (size_t)e * a.w_expert;
    float acc[2][4] = {};
    for (int k0 = 0; k0 < a.k; k0 += GK) {
        {
            const int r = threadIdx.x >> 4, kk = threadIdx.x & 15;
            const int src = s_src[r];
            xs[r][kk] = (src >= 0 && k0 + kk < a.k) ? to_f32(((const T*)a.x)[(size_t)src * a.ldx + k0 + kk]) : 0.0f;
        }
        for (int i = threadIdx.x; i < (gated ? 2 : 1) * GN * GK; i += 256) {
            const int half = i / (GN * GK), c = (i / GK) % GN, kk = i % GK;
            const int row = half * n_out + col0 + c;
            ws[half][c][kk] = (col0 + c < n_out && k0 + kk < a.k) ? to_f32(w[(size_t)row * a.ldw + k0 + kk]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < GK; ++kk) {
            const float xv = xs[ty][kk];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                acc[0][c] = fmaf(xv, ws[0][tx + 16 * c][kk], acc[0][c]);
                if (gated) acc[1][c] = fmaf(xv, ws[1][tx + 16 * c][kk], acc[1][c]);
            }
        }
        __syncthreads();
    }
    const int dst = s_dst[ty];
    if (dst < 0) return;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const int col = col0 + tx + 16 * c;
        if (col >= n_out) continue;
        float v = acc[0][c];
        if (a.act == 2) v = relu2(v);
        if (a.act == 3) v = gelu_erf(v);
        if (gated) {
            // gate and up pass through the type of the activations first, as they do when the activation is a kernel of its own
            const float g = to_f32(from_f32<T>(acc[0][c])), u = to_f32(from_f32<T>(acc[1][c]));
            v = (g / (1.0f + expf(-g))) * u;
        }
        ((O*)a.out)[(size_t)dst * a.ldo + col] = from_f32<O>(v);
    }
}

LLME_API int llme_grouped_linear(const LlmeGroupedArgs* args, int x_dtype, int w_dtype, int out_dtype, cudaStream_t stream) {
    const LlmeGroupedArgs& a = *args;
    if (a.pairs <= 0 || a.n <= 0) return 0;
    if (!a.x || !a.w || !a.out || !a.offsets || !a.order) LLME_REFUSE("grouped_linear: null pointer");
    if (a.num_experts <= 0 || a.top_k <= 0 || a.k <= 0 || a.act < 0 || a.act > 3 || (a.act == 1 && a.n % 2)) LLME_REFUSE("grouped_linear: bad size");
    const int n_out = a.act == 1 ? a.n / 2 : a.n;
    const int most = a.num_experts < a.pairs ? a.num_experts : a.pairs;
    int tiles = (a.pairs + GM - 1) / GM + most;
    if (tiles > a.pairs) tiles = a.pairs;
    const dim3 grid((n_out + GN - 1) / GN, tiles);
#define LLME_GL(T, W, O) llme_launch(grouped_linear_kernel<T, W, O>, grid, dim3(256), 0, stream, a)
    if (x_dtype == LLME_F32 && w_dtype == LLME_F32 && out_dtype == LLME_F32) LLME_GL(float, float, float);
    else if (x_dtype == LLME_BF16 && w_dtype == LLME_BF16 && out_dtype == LLME_BF16) LLME_GL(__nv_bfloat16, __nv_bfloat16, __nv_bfloat16);
    else if (x_dtype == LLME_BF16 && w_dtype == LLME_BF16 && out_dtype == LLME_F32) LLME_GL(__nv_bfloat16, __nv_bfloat16, float);
    else LLME_REFUSE("grouped_linear: unsupported dtypes %d / %d / %d", x_dtype, w_dtype, out_dtype);
#undef LLME_GL
    LLME_LAUNCH_STATUS();
}

// ----------------------------------------------------------------------------- the weighted sum of a token's pairs
// A choice whose expert is `first_identity` or a later one stands for the token's row of `same` (type S) instead of a row of y.
template <typename S>
__global__ void moe_combine_kernel(const float* __restrict__ y, long long ldy, const float* __restrict__ weights, const float* __restrict__ base,
                                   float* __restrict__ out, int top_k, int cols, const float* __restrict__ base_gate, long long ld_gate,
                                   const int* __restrict__ experts, const S* __restrict__ same, long long ld_same, int first_identity) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const float share = base && base_gate ? 1.0f / (1.0f + expf(-base_gate[(size_t)t * ld_gate])) : 1.0f;   // the shared expert's gate
    for (int j = blockIdx.y * blockDim.x + threadIdx.x; j < cols; j += gridDim.y * blockDim.x) {
        float v = 0.0f;
        for (int k = 0; k < top_k; ++k) {
            const size_t pair = (size_t)t * top_k + k;
            const float row = same && experts[pair] >= first_identity ? to_f32(same[(size_t)t * ld_same + j]) : y[pair * ldy + j];
            v = fmaf(weights[pair], row, v);
        }
        out[(size_t)t * cols + j] = base ? base[(size_t)t * cols + j] * share + v : v;
    }
}

// Four columns a thread where the rows allow it: the same sums.
template <typename S> __device__ __forceinline__ float4 four_of(const S* p);
template <> __device__ __forceinline__ float4 four_of<float>(const float* p) { return *(const float4*)p; }
template <> __device__ __forceinline__ float4 four_of<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *(const uint2*)p;
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&raw.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&raw.y);
    return make_float4(a.x, a.y, b.x, b.y);
}

template <typename S>
__global__ void moe_combine_vec_kernel(const float* __restrict__ y, long long ldy, const float* __restrict__ weights, const float* __restrict__ base,
                                       float* __restrict__ out, int top_k, int cols, const float* __restrict__ base_gate, long long ld_gate,
                                       const int* __restrict__ experts, const S* __restrict__ same, long long ld_same, int first_identity) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const float share = base && base_gate ? 1.0f / (1.0f + expf(-base_gate[(size_t)t * ld_gate])) : 1.0f;
    for (int j = 4 * (blockIdx.y * blockDim.x + threadIdx.x); j < cols; j += 4 * gridDim.y * blockDim.x) {
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const float4 b = base ? *(const float4*)(base + (size_t)t * cols + j) : v;
#pragma unroll 4
        for (int k = 0; k < top_k; ++k) {
            const size_t pair = (size_t)t * top_k + k;
            const float4 row = same && experts[pair] >= first_identity ? four_of<S>(same + (size_t)t * ld_same + j) : *(const float4*)(y + pair * ldy + j);
            const float w = weights[pair];
            v = make_float4(fmaf(w, row.x, v.x), fmaf(w, row.y, v.y), fmaf(w, row.z, v.z), fmaf(w, row.w, v.w));
        }
        if (base) v = make_float4(b.x * share + v.x, b.y * share + v.y, b.z * share + v.z, b.w * share + v.w);
        *(float4*)(out + (size_t)t * cols + j) = v;
    }
}

// out[t] = base[t] (times sigmoid(base_gate[t * ld_gate]), where given) + sum over the choices of weight times the pair's row of y,
// or, with `same` (same_dtype) and `experts`, times the token's row of `same` for choices from `first_identity` on.
LLME_API int llme_moe_combine(const float* y, long long ldy, const float* weights, const float* base, float* out, int tokens, int top_k, int cols,
                              const float* base_gate, long long ld_gate, const int* experts, const void* same, long long ld_same, int same_dtype,
                              int first_identity, cudaStream_t stream) {
    if (tokens <= 0 || cols <= 0) return 0;
    if (!y || !weights || !out || top_k <= 0 || (same && !experts)) LLME_REFUSE("moe_combine: null pointer or no choices");
    if (same && same_dtype != LLME_F32 && same_dtype != LLME_BF16) LLME_REFUSE("moe_combine: unsupported dtype %d", same_dtype);
    const int threads = 128;
    const bool vec = cols % 4 == 0 && ldy % 4 == 0 && ld_same % 4 == 0 && (((uintptr_t)y | (uintptr_t)base | (uintptr_t)out) & 15) == 0 && ((uintptr_t)same & 15) == 0;
    const int each = vec ? 4 * threads : threads;
    int pieces = (cols + each - 1) / each;
    const int wanted = (592 + tokens - 1) / tokens;
    if (pieces > wanted) pieces = wanted;
    const dim3 grid(tokens, pieces < 1 ? 1 : pieces);
#define LLME_MC(K, S) llme_launch(K<S>, grid, dim3(threads), 0, stream, y, ldy, weights, base, out, top_k, cols, base_gate, ld_gate, experts, (const S*)same, ld_same, first_identity)
    if (same && same_dtype == LLME_BF16) { if (vec) LLME_MC(moe_combine_vec_kernel, __nv_bfloat16); else LLME_MC(moe_combine_kernel, __nv_bfloat16); }
    else { if (vec) LLME_MC(moe_combine_vec_kernel, float); else LLME_MC(moe_combine_kernel, float); }
#undef LLME_MC
    LLME_LAUNCH_STATUS();
}
