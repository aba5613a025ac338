// Grouped-query attention whose keys and values differ in width, with a window that keeps the first positions of a
// request and a learned sink per head in the softmax denominator: the step between the projections and the cache
// (norm over the whole projection, partial rotation, cache write) and the plain attention kernel (one warp per
// (token, query head), any sizes, both types: the 32-bit path, the fallback and the twin of the tensor-core kernel).
//
// A cache page holds the keys of its tokens, [nkv][page_size][dk], and behind them the values, [nkv][page_size][dv].
// A token's result depends only on its own query and the keys of its request, never on what else is in the launch.
#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

// Value heads of a layer, and the values of a page: with a `value_share` n of more than one, n neighbouring key heads share one value
// head (the maps of a differential attention).
__device__ __forceinline__ int value_heads(int nkv, int share) { return share > 1 ? nkv / share : nkv; }
__device__ __forceinline__ size_t page_values(int nkv, int nv, int ps, int dk, int dv) { return (size_t)ps * ((size_t)nkv * dk + (size_t)nv * dv); }

// ----------------------------------------------------------------------------- norm, rotation, cache write
// One value of a projection row after the norm (x * rinv * gain) and the rotation of its head's first `dims`
// coordinates in rotate-half pairs (i, i + dims/2) by position * inv_freq[i], cosine and sine times `amp`.
// `interleaved`: the pairs are (2i, 2i + 1) instead.
template <typename T>
__device__ __forceinline__ float finished_value(const T* __restrict__ row, const float* __restrict__ gain, float rinv, int head, int d, int dk,
                                                const float* __restrict__ inv_freq, int dims, float amp, int position, int interleaved) {
    const int base = head * dk;
    auto normed = [&](int j) -> float {
        const float v = to_f32(row[base + j]);
        return gain ? (v * rinv) * gain[base + j] : v;
    };
    if (!inv_freq || d >= dims) return normed(d);
    const int half = dims >> 1, i = interleaved ? d >> 1 : (d < half ? d : d - half);
    float s, c;
    sincosf((float)position * inv_freq[i], &s, &c);
    s *= amp;
    c *= amp;
    const float u = normed(interleaved ? 2 * i : i), w = normed(interleaved ? 2 * i + 1 : i + half);
    const bool first = interleaved ? !(d & 1) : d < half;
    return first ? u * c - w * s : w * c + u * s;
}

// I: the type of the projections (that of everything else, or 32-bit where they come from a convolution); T: the type of the
// finished queries and of the cache.
template <typename I, typename T>
__global__ void window_post_kernel(LlmeWindowPostArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int t = blockIdx.x, dk = a.dk, dv = a.dv, ps = a.page_size;
    const int pos = a.positions[t];
    const int nv = value_heads(a.nkv, a.value_share);
    const int qn = a.nh * dk, kn = a.nkv * dk, vn = nv * dv;
    const I* q = (const I*)a.q_in + (size_t)t * a.q_stride;
    float rq = 1.0f, rk = 1.0f;
    if (a.q_gain) {
        float ss = 0.0f;
        for (int j = threadIdx.x; j < qn; j += blockDim.x) {
            const float v = to_f32(q[j]);
            ss += v * v;
        }
        rq = 1.0f / sqrtf(block_sum(ss, scratch) / (float)qn + a.eps);
    }
    T* qo = (T*)a.q_out + (size_t)t * qn;
    for (int j = threadIdx.x; j < qn; j += blockDim.x)
        qo[j] = from_f32<T>(finished_value(q, a.q_gain, rq, j / dk, j % dk, dk, a.inv_freq, a.rot_dims, a.amplitude, pos, a.interleaved));
    const int slot = (a.cache && a.slot_mapping) ? a.slot_mapping[t] : -1;
    if (!a.k_in || slot < 0) return;                    // uniform over the block
    const I* k = (const I*)a.k_in + (size_t)t * a.k_stride;
    const I* v = (const I*)a.v_in + (size_t)t * a.v_stride;
    if (a.k_gain) {
        float ss = 0.0f;
        for (int j = threadIdx.x; j < kn; j += blockDim.x) {
            const float x = to_f32(k[j]);
            ss += x * x;
        }
        rk = 1.0f / sqrtf(block_sum(ss, scratch) / (float)kn + a.eps);
    }
    const int page = slot / ps, off = slot - page * ps;
    T* kpage = (T*)a.cache + (size_t)page * page_values(a.nkv, nv, ps, dk, dv);
    T* vpage = kpage + (size_t)a.nkv * ps * dk;
    for (int j = threadIdx.x; j < kn; j += blockDim.x) {
        const int g = j / dk, d = j - g * dk;
        kpage[((size_t)g * ps + off) * dk + d] = from_f32<T>(finished_value(k, a.k_gain, rk, g, d, dk, a.inv_freq, a.rot_dims, a.amplitude, pos, a.interleaved));
    }
    for (int j = threadIdx.x; j < vn; j += blockDim.x) {
        const int g = j / dv, d = j - g * dv;
        vpage[((size_t)g * ps + off) * dv + d] = from_f32<T>(to_f32(v[j]));
    }
}

// The same step for designs that norm every head by itself (gains of one head's size, shared by the heads) and whose
// projections have biases: one warp per (token, head); the biased head is read twice (sum of squares, then the values).
// The value may be the key's own projection (v_in = k_in): it is stored as projected, with its bias, before the norm.
template <typename T>
__device__ __forceinline__ void finish_head(const T* __restrict__ in, const float* __restrict__ bias, const float* __restrict__ gain, float eps, int dk,
                                            const float* __restrict__ inv_freq, int dims, float amp, int position, T* __restrict__ out, int lane,
                                            int interleaved) {
    auto raw = [&](int j) -> float {
        const float v = to_f32(in[j]);
        return bias ? to_f32(from_f32<T>(v + bias[j])) : v;      // a projection's output has the type of the products
    };
    float rinv = 1.0f;
    if (gain) {
        float ss = 0.0f;
        for (int j = lane; j < dk; j += 32) {
            const float v = raw(j);
            ss += v * v;
        }
        rinv = 1.0f / sqrtf(warp_sum(ss) / (float)dk + eps);
    }
    auto normed = [&](int j) -> float { return gain ? (raw(j) * rinv) * gain[j] : raw(j); };
    const int half = dims >> 1;
    for (int d = lane; d < dk; d += 32) {
        float v;
        if (!inv_freq || d >= dims) v = normed(d);
        else {
            const int i = interleaved ? d >> 1 : (d < half ? d : d - half);
            float s, c;
            sincosf((float)position * inv_freq[i], &s, &c);
            s *= amp;
            c *= amp;
            const float u = normed(interleaved ? 2 * i : i), w = normed(interleaved ? 2 * i + 1 : i + half);
            v = (interleaved ? !(d & 1) : d < half) ? u * c - w * s : w * c + u * s;
        }
        out[d] = from_f32<T>(v);
    }
}

template <typename T>
__global__ void window_post_heads_kernel(LlmeWindowPostArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int warps = blockDim.x >> 5, lane = threadIdx.x & 31;
    const int item = blockIdx.x * warps + (threadIdx.x >> 5);       // (token, head of q | head of k | head of v)
    const bool stores = a.k_in != nullptr;
    const int nv = value_heads(a.nkv, a.value_share), per_token = a.nh + (stores ? a.nkv + nv : 0);
    if (item >= a.tokens * per_token) return;
    const int t = item / per_token, hh = item - t * per_token;
    const int dk = a.dk, dv = a.dv, ps = a.page_size, pos = a.positions[t];
    if (hh < a.nh) {
        finish_head((const T*)a.q_in + (size_t)t * a.q_stride + hh * dk, a.q_bias ? a.q_bias + hh * dk : nullptr, a.q_gain, a.eps, dk,
                    a.inv_freq, a.rot_dims, a.amplitude, pos, (T*)a.q_out + ((size_t)t * a.nh + hh) * dk, lane, a.interleaved);
        return;
    }
    const int slot = a.slot_mapping[t];
    if (slot < 0) return;
    const int page = slot / ps, off = slot - page * ps;
    T* kpage = (T*)a.cache + (size_t)page * page_values(a.nkv, nv, ps, dk, dv);
    if (hh < a.nh + a.nkv) {
        const int g = hh - a.nh;
        finish_head((const T*)a.k_in + (size_t)t * a.k_stride + g * dk, a.k_bias ? a.k_bias + g * dk : nullptr, a.k_gain, a.eps, dk,
                    a.inv_freq, a.rot_dims, a.amplitude, pos, kpage + ((size_t)g * ps + off) * dk, lane, a.interleaved);
        return;
    }
    const int g = hh - a.nh - a.nkv;
    const T* v = (const T*)a.v_in + (size_t)t * a.v_stride + g * dv;
    T* vo = kpage + (size_t)a.nkv * ps * dk + ((size_t)g * ps + off) * dv;
    for (int d = lane; d < dv; d += 32) vo[d] = a.v_bias ? from_f32<T>(to_f32(v[d]) + a.v_bias[g * dv + d]) : v[d];
}

// The same step for designs that divide every query and key head by its root mean square BEHIND the rotation (no weight): a
// block takes a token (or a share of its heads), forms the token's cosines and sines once, and a warp finishes a head at a time
// with its values in registers.
template <typename T, int KR>
__global__ void __launch_bounds__(256) window_post_unit_kernel(LlmeWindowPostArgs a) {
    extern __shared__ float cs[];                                    // [rot_dims / 2] cosines, then sines
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, warps = blockDim.x >> 5, lane = threadIdx.x & 31;
    const int dk = a.dk, dv = a.dv, ps = a.page_size, half = a.inv_freq ? a.rot_dims >> 1 : 0;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)a.positions[t] * a.inv_freq[i], &s, &c);
        cs[i] = c * a.amplitude;
        cs[half + i] = s * a.amplitude;
    }
    __syncthreads();
    const int slot = a.k_in ? a.slot_mapping[t] : -1;
    const int page = slot >= 0 ? slot / ps : 0, off = slot - page * ps;
    const int nv = value_heads(a.nkv, a.value_share);
    T* kpage = (T*)a.cache + (size_t)page * page_values(a.nkv, nv, ps, dk, dv);
    const int heads = a.nh + (slot >= 0 ? a.nkv + nv : 0);
    for (int hh = blockIdx.y * warps + (threadIdx.x >> 5); hh < heads; hh += gridDim.y * warps) {
        if (hh >= a.nh + a.nkv) {
            const int g = hh - a.nh - a.nkv;
            const T* v = (const T*)a.v_in + (size_t)t * a.v_stride + g * dv;
            T* vo = kpage + (size_t)a.nkv * ps * dk + ((size_t)g * ps + off) * dv;
            for (int d = lane; d < dv; d += 32) vo[d] = v[d];
            continue;
        }
        const bool query = hh < a.nh;
        const int g = hh - a.nh;
        const T* in = query ? (const T*)a.q_in + (size_t)t * a.q_stride + hh * dk : (const T*)a.k_in + (size_t)t * a.k_stride + g * dk;
        T* out = query ? (T*)a.q_out + ((size_t)t * a.nh + hh) * dk : kpage + ((size_t)g * ps + off) * dk;
        float x[KR], ss = 0.0f;
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const int d = lane + 32 * i;
            x[i] = d < dk ? to_f32(in[d]) : 0.0f;
            if (d < 2 * half) {
                const int e = a.interleaved ? d >> 1 : (d < half ? d : d - half);
                const bool first = a.interleaved ? !(d & 1) : d < half;
                const float other = to_f32(in[a.interleaved ? d ^ 1 : (first ? d + half : d - half)]);
                x[i] = first ? x[i] * cs[e] - other * cs[half + e] : x[i] * cs[e] + other * cs[half + e];
            }
            ss = fmaf(x[i], x[i], ss);
        }
        const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)dk + a.eps);
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const int d = lane + 32 * i;
            if (d < dk) out[d] = from_f32<T>(x[i] * rinv);
        }
    }
}

// The same for heads of up to 128 coordinates in fours, rotated coordinates in eights (neighbouring pairs: in fours), rows that start on
// whole pieces: a lane holds four neighbouring coordinates and has their partners itself (neighbouring pairs) or gets them from the
// lane that holds them; a warp has two heads on their way at a time.  It also serves designs that norm every head by itself with
// gains BEFORE the rotation (`head_norm`, no biases).
template <typename T> struct Four;
template <> struct Four<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *(const float4*)p; }
    static __device__ __forceinline__ void store(float* p, float4 v) { *(float4*)p = v; }
};
template <> struct Four<__nv_bfloat16> {
    static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
        const uint2 raw = *(const uint2*)p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&raw.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&raw.y);
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
        uint2 raw;
        *(__nv_bfloat162*)&raw.x = __floats2bfloat162_rn(v.x, v.y);
        *(__nv_bfloat162*)&raw.y = __floats2bfloat162_rn(v.z, v.w);
        *(uint2*)p = raw;
    }
};

// LANES lanes hold a head (its size in fours, rounded up to 8, 16 or 32), so a warp finishes 32 / LANES heads at a time.
template <typename T, int LANES>
__global__ void __launch_bounds__(256) window_post_fours_kernel(LlmeWindowPostArgs a) {
    extern __shared__ __align__(16) float cs4[];                     // [rot_dims / 2] cosines, then sines
    pdl_launch_dependents();
    pdl_wait();
    constexpr int EACH = 32 / LANES;                                 // heads a warp has in hand
    const int t = blockIdx.x, warps = blockDim.x >> 5, lane = threadIdx.x & (LANES - 1), d = 4 * lane;
    const int dk = a.dk, dv = a.dv, ps = a.page_size, half = a.inv_freq ? a.rot_dims >> 1 : 0;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s, c;
        sincosf((float)a.positions[t] * a.inv_freq[i], &s, &c);
        cs4[i] = c * a.amplitude;
        cs4[half + i] = s * a.amplitude;
    }
    const int slot = a.k_in ? a.slot_mapping[t] : -1;
    const int page = slot >= 0 ? slot / ps : 0, off = slot - page * ps;
    const int nv = value_heads(a.nkv, a.value_share);
    T* kpage = (T*)a.cache + (size_t)page * page_values(a.nkv, nv, ps, dk, dv);
    const int heads = a.nh + (slot >= 0 ? a.nkv : 0), stride = gridDim.y * warps * EACH;
    const T* qrow = (const T*)a.q_in + (size_t)t * a.q_stride;
    const T* krow = (const T*)a.k_in + (size_t)t * a.k_stride;
    const bool turned = d < 2 * half, first = d < half, inside = d < dk;
    const int partner = !turned ? lane : first ? lane + half / 4 : lane - half / 4;
    auto source = [&](int hh) -> const T* { return hh < a.nh ? qrow + hh * dk : krow + (hh - a.nh) * dk; };
    auto head_sum = [&](float v) {                                   // over the lanes of a head
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        return v;
    };
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    int hh = (blockIdx.y * warps + (threadIdx.x >> 5)) * EACH + (threadIdx.x & 31) / LANES;
    float4 x = hh < heads && inside ? Four<T>::load(source(hh) + d) : zero, ahead = zero;
    if (slot >= 0) {                                                 // the values, as they are
        const T* vrow = (const T*)a.v_in + (size_t)t * a.v_stride;
        T* vpage = kpage + (size_t)a.nkv * ps * dk + (size_t)off * dv;
        const int pieces = dv / 4;
        for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < nv * pieces; i += gridDim.y * blockDim.x) {
            const int g = i / pieces, e = 4 * (i - g * pieces);
            Four<T>::store(vpage + (size_t)g * ps * dv + e, Four<T>::load(vrow + g * dv + e));
        }
    }
    __syncthreads();
    float4 c = make_float4(1.0f, 1.0f, 1.0f, 1.0f), s = zero, gq = c, gk = c;
    if (a.head_norm && inside && a.q_gain) {
        gq = *(const float4*)(a.q_gain + d);
        gk = a.k_gain ? *(const float4*)(a.k_gain + d) : gk;
    }
    if (turned && a.interleaved) {                                   // pairs (d, d + 1) and (d + 2, d + 3): frequencies d/2, d/2 + 1
        const float c0 = cs4[d >> 1], c1 = cs4[(d >> 1) + 1], s0 = cs4[half + (d >> 1)], s1 = cs4[half + (d >> 1) + 1];
        c = make_float4(c0, c0, c1, c1);
        s = make_float4(-s0, s0, -s1, s1);
    } else if (turned) {
        c = *(const float4*)&cs4[first ? d : d - half];
        s = *(const float4*)&cs4[half + (first ? d : d - half)];
        if (first) s = make_float4(-s.x, -s.y, -s.z, -s.w);          // u cos - v sin, v cos + u sin
    }
    // (every lane of a warp takes the same number of turns: exchanges are between all of them)
    for (int h0 = hh - (threadIdx.x & 31) / LANES; h0 < heads; h0 += stride, hh += stride, x = ahead) {
        const int nx = hh + stride;
        ahead = nx < heads && inside ? Four<T>::load(source(nx) + d) : zero;
        if (a.head_norm) {
            const float ss = head_sum(fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w))));
            const float rinv = 1.0f / sqrtf(ss / (float)dk + a.eps);
            const float4 g = hh < a.nh ? gq : gk;
            x = make_float4(x.x * rinv * g.x, x.y * rinv * g.y, x.z * rinv * g.z, x.w * rinv * g.w);
        }
        const float4 o = a.interleaved ? make_float4(x.y, x.x, x.w, x.z)
                                       : make_float4(__shfl_sync(0xffffffffu, x.x, partner, LANES), __shfl_sync(0xffffffffu, x.y, partner, LANES),
                                                     __shfl_sync(0xffffffffu, x.z, partner, LANES), __shfl_sync(0xffffffffu, x.w, partner, LANES));
        if (turned) x = make_float4(x.x * c.x + o.x * s.x, x.y * c.y + o.y * s.y, x.z * c.z + o.z * s.z, x.w * c.w + o.w * s.w);
        float rinv = 1.0f;
        if (a.unit_norm) {
            const float ss = head_sum(fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w))));
            rinv = 1.0f / sqrtf(ss / (float)dk + a.eps);
        }
        T* out = hh < a.nh ? (T*)a.q_out + ((size_t)t * a.nh + hh) * dk : kpage + ((size_t)(hh - a.nh) * ps + off) * dk;
        if (inside && hh < heads) Four<T>::store(out + d, make_float4(x.x * rinv, x.y * rinv, x.z * rinv, x.w * rinv));
    }
}

// A block per token, or several where the step has few; a block has eight warps of `each` heads.
static dim3 post_grid(const LlmeWindowPostArgs& a, int each = 1) {
    const int heads = a.nh + (a.k_in ? a.nkv + (a.value_share > 1 ? a.nkv / a.value_share : a.nkv) : 0), most = (heads + 8 * each - 1) / (8 * each);
    const int fill = (592 + a.tokens - 1) / a.tokens;
    return dim3(a.tokens, most < fill ? most : fill);
}

template <typename T>
static bool launch_post_fours(const LlmeWindowPostArgs& a, cudaStream_t s) {
    const size_t smem = (size_t)(a.inv_freq ? a.rot_dims : 0) * sizeof(float), piece = 4 * sizeof(T);
    const bool fours = a.dk % 4 == 0 && a.dv % 4 == 0 && a.dk <= 128 && (!a.inv_freq || a.rot_dims % (a.interleaved ? 4 : 8) == 0) &&
                       a.q_stride % 4 == 0 && a.k_stride % 4 == 0 && a.v_stride % 4 == 0 && ((uintptr_t)a.q_gain | (uintptr_t)a.k_gain) % 16 == 0 &&
                       ((uintptr_t)a.q_in | (uintptr_t)a.k_in | (uintptr_t)a.v_in | (uintptr_t)a.q_out | (uintptr_t)a.cache) % piece == 0;
    if (!fours) return false;
    if (a.dk <= 32) llme_launch(window_post_fours_kernel<T, 8>, post_grid(a, 4), dim3(256), smem, s, a);
    else if (a.dk <= 64) llme_launch(window_post_fours_kernel<T, 16>, post_grid(a, 2), dim3(256), smem, s, a);
    else llme_launch(window_post_fours_kernel<T, 32>, post_grid(a), dim3(256), smem, s, a);
    return true;
}

template <typename T>
static int launch_post_unit(const LlmeWindowPostArgs& a, cudaStream_t s) {
    const dim3 grid = post_grid(a), block(256);
    const size_t smem = (size_t)(a.inv_freq ? a.rot_dims : 0) * sizeof(float);
    if (launch_post_fours<T>(a, s)) LLME_LAUNCH_STATUS();
    if (a.dk <= 32) llme_launch(window_post_unit_kernel<T, 1>, grid, block, smem, s, a);
    else if (a.dk <= 64) llme_launch(window_post_unit_kernel<T, 2>, grid, block, smem, s, a);
    else if (a.dk <= 128) llme_launch(window_post_unit_kernel<T, 4>, grid, block, smem, s, a);
    else if (a.dk <= 256) llme_launch(window_post_unit_kernel<T, 8>, grid, block, smem, s, a);
    else if (a.dk <= 512) llme_launch(window_post_unit_kernel<T, 16>, grid, block, smem, s, a);
    else LLME_REFUSE("window_post: a query/key size of %d is larger than 512", a.dk);
    LLME_LAUNCH_STATUS();
}

LLME_API int llme_window_post(const LlmeWindowPostArgs* args, int dtype, cudaStream_t stream) {
    const LlmeWindowPostArgs& a = *args;
    if (a.tokens <= 0) return 0;
    if (!a.q_in || !a.q_out || !a.positions) LLME_REFUSE("window_post: null pointer");
    if ((a.k_in == nullptr) != (a.v_in == nullptr)) LLME_REFUSE("window_post: keys and values are stored together");
    if (a.k_in && (!a.cache || !a.slot_mapping || a.page_size <= 0)) LLME_REFUSE("window_post: keys without a cache to store them in");
    if (a.nh <= 0 || a.nkv <= 0 || a.dk <= 0 || a.dv <= 0) LLME_REFUSE("window_post: non-positive size");
    if (a.value_share > 1 && a.nkv % a.value_share) LLME_REFUSE("window_post: %d key heads do not share values %d at a time", a.nkv, a.value_share);
    if (a.inv_freq && (a.rot_dims <= 0 || a.rot_dims % 2 || a.rot_dims > a.dk))
        LLME_REFUSE("window_post: %d rotated coordinates of %d need an even count", a.rot_dims, a.dk);
    if ((a.q_gain || a.k_gain) && !(a.eps > 0.0f)) LLME_REFUSE("window_post: eps must be positive");
    const bool wide_in = a.in_f32 && dtype != LLME_F32;     // 32-bit projections, everything else in the type of the products
    if (a.unit_norm) {
        if (wide_in || a.q_gain || a.k_gain || a.q_bias || a.k_bias || a.v_bias) LLME_REFUSE("window_post: the norm behind the rotation stands alone");
        if (!(a.eps > 0.0f)) LLME_REFUSE("window_post: eps must be positive");
        if (dtype == LLME_F32) return launch_post_unit<float>(a, stream);
        if (dtype == LLME_BF16) return launch_post_unit<__nv_bfloat16>(a, stream);
        LLME_REFUSE("window_post: unsupported dtype %d", dtype);
    }
    if (a.head_norm || a.q_bias || a.k_bias || a.v_bias) {
        if (wide_in) LLME_REFUSE("window_post: 32-bit projections come without biases and without the norm per head");
        if (!a.head_norm && (a.q_gain || a.k_gain)) LLME_REFUSE("window_post: biases come with the norm per head or with no norm");
        if (a.head_norm && a.q_gain && (a.k_gain || !a.k_in) && !a.q_bias && !a.k_bias && !a.v_bias && !a.unit_norm) {
            if (dtype == LLME_F32 ? launch_post_fours<float>(a, stream) : dtype == LLME_BF16 ? launch_post_fours<__nv_bfloat16>(a, stream) : false)
                LLME_LAUNCH_STATUS();
        }
        const long long items = (long long)a.tokens * (a.nh + (a.k_in ? a.nkv + (a.value_share > 1 ? a.nkv / a.value_share : a.nkv) : 0));
        const int wpb = 4;
        if (dtype == LLME_F32) llme_launch(window_post_heads_kernel<float>, dim3((unsigned)((items + wpb - 1) / wpb)), dim3(wpb * 32), 0, stream, a);
        else if (dtype == LLME_BF16) llme_launch(window_post_heads_kernel<__nv_bfloat16>, dim3((unsigned)((items + wpb - 1) / wpb)), dim3(wpb * 32), 0, stream, a);
        else LLME_REFUSE("window_post: unsupported dtype %d", dtype);
        LLME_LAUNCH_STATUS();
    }
    const int qn = a.nh * a.dk;
    const int threads = qn >= 2048 ? 512 : (qn >= 512 ? 256 : 128);
    if (dtype == LLME_F32) llme_launch(window_post_kernel<float, float>, dim3(a.tokens), dim3(threads), 0, stream, a);
    else if (dtype == LLME_BF16 && wide_in) llme_launch(window_post_kernel<float, __nv_bfloat16>, dim3(a.tokens), dim3(threads), 0, stream, a);
    else if (dtype == LLME_BF16) llme_launch(window_post_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(a.tokens), dim3(threads), 0, stream, a);
    else LLME_REFUSE("window_post: unsupported dtype %d", dtype);
    LLME_LAUNCH_STATUS();
}

// ----------------------------------------------------------------------------- plain attention
template <typename T, int KR, int VR>
__global__ void window_attention_plain_kernel(LlmeWindowAttnArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int warps_per_block = blockDim.x >> 5;
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * warps_per_block + (threadIdx.x >> 5);
    const int h = blockIdx.y;
    if (t >= a.tokens) return;
    const int dk = a.dk, dv = a.dv, ps = a.page_size;
    const int kvh = h / (a.nh / a.nkv);
    const int p = a.positions[t];
    const int lo = (a.window > 0 && p - a.window + 1 > 0) ? p - a.window + 1 : 0;
    const int first = a.keep_first < lo ? a.keep_first : lo;       // keys 0 .. first-1 are seen beside the window
    const int* bt = a.block_tables + (size_t)a.token_request[t] * a.max_blocks;
    const int share = a.value_share > 1 ? a.value_share : 1;
    const size_t page_elems = page_values(a.nkv, a.nkv / share, ps, dk, dv);

    float q[KR], acc[VR];
    const T* qp = (const T*)a.q + ((size_t)t * a.nh + h) * dk;
#pragma unroll
    for (int i = 0; i < KR; ++i) {
        const int d = lane + 32 * i;
        q[i] = d < dk ? to_f32(qp[d]) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < VR; ++i) acc[i] = 0.0f;
    // the sink is one more term of the denominator: a score that is not scaled and has no value
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.0f : 0.0f;
    for (int jj = 0; jj < first + (p - lo + 1); ++jj) {
        const int j = jj < first ? jj : lo + (jj - first);
        const int page = bt[j / ps];
        const int off = j - (j / ps) * ps;
        const T* kp = (const T*)a.cache + (size_t)page * page_elems + ((size_t)kvh * ps + off) * dk;
        const T* vp = (const T*)a.cache + (size_t)page * page_elems + (size_t)a.nkv * ps * dk + ((size_t)(kvh / share) * ps + off) * dv;
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < KR; ++i) {
            const int d = lane + 32 * i;
            if (d < dk) s += q[i] * to_f32(kp[d]);
        }
        s = warp_sum(s) * a.scale;
        if (a.softcap > 0.0f) s = a.softcap * tanhf(s / a.softcap);
        const float m_new = fmaxf(m, s);
        const float corr = expf(m - m_new);       // exp(-inf) = 0 on the first key
        const float e = expf(s - m_new);
        l = l * corr + e;
#pragma unroll
        for (int i = 0; i < VR; ++i) {
            const int d = lane + 32 * i;
            if (d < dv) acc[i] = acc[i] * corr + e * to_f32(vp[d]);
        }
        m = m_new;
    }
    T* op = (T*)a.out + ((size_t)t * a.nh + h) * dv;
    const float inv = 1.0f / l;
#pragma unroll
    for (int i = 0; i < VR; ++i) {
        const int d = lane + 32 * i;
        if (d < dv) op[d] = from_f32<T>(acc[i] * inv);
    }
}

template <typename T, int KR>
static int launch_plain_v(const LlmeWindowAttnArgs& a, cudaStream_t s) {
    const int wpb = 4;
    dim3 grid((a.tokens + wpb - 1) / wpb, a.nh);
    const int regs = (a.dv + 31) / 32;
    if (regs <= 1) llme_launch(window_attention_plain_kernel<T, KR, 1>, dim3(grid), dim3(wpb * 32), 0, s, a);
    else if (regs <= 2) llme_launch(window_attention_plain_kernel<T, KR, 2>, dim3(grid), dim3(wpb * 32), 0, s, a);
    else if (regs <= 4) llme_launch(window_attention_plain_kernel<T, KR, 4>, dim3(grid), dim3(wpb * 32), 0, s, a);
    else if (regs <= 8) llme_launch(window_attention_plain_kernel<T, KR, 8>, dim3(grid), dim3(wpb * 32), 0, s, a);
    else if (regs <= 16) llme_launch(window_attention_plain_kernel<T, KR, 16>, dim3(grid), dim3(wpb * 32), 0, s, a);
    else LLME_REFUSE("window attention: a value size of %d is larger than 512", a.dv);
    LLME_LAUNCH_STATUS();
}

template <typename T>
static int launch_plain(const LlmeWindowAttnArgs& a, cudaStream_t s) {
    const int regs = (a.dk + 31) / 32;
    if (regs <= 1) return launch_plain_v<T, 1>(a, s);
    if (regs <= 2) return launch_plain_v<T, 2>(a, s);
    if (regs <= 4) return launch_plain_v<T, 4>(a, s);
    if (regs <= 8) return launch_plain_v<T, 8>(a, s);
    if (regs <= 16) return launch_plain_v<T, 16>(a, s);
    LLME_REFUSE("window attention: a query/key size of %d is larger than 512", a.dk);
}

LLME_API int llme_window_attention_plain(const LlmeWindowAttnArgs* args, int dtype, cudaStream_t stream) {
    const LlmeWindowAttnArgs& a = *args;
    if (a.tokens <= 0) return 0;
    if (!a.q || !a.cache || !a.out || !a.positions || !a.token_request || !a.block_tables) LLME_REFUSE("window attention: null pointer");
    if (a.nh <= 0 || a.nkv <= 0 || a.nh % a.nkv) LLME_REFUSE("window attention: %d query heads are not a multiple of %d key/value heads", a.nh, a.nkv);
    if (a.dk <= 0 || a.dv <= 0 || a.page_size <= 0 || a.max_blocks <= 0 || a.window < 0 || a.keep_first < 0) LLME_REFUSE("window attention: bad size");
    if (a.nh > 65535) LLME_REFUSE("window attention: more than 65535 query heads");
    if (a.value_share > 1 && a.nkv % a.value_share) LLME_REFUSE("window attention: %d key heads do not share values %d at a time", a.nkv, a.value_share);
    if (dtype == LLME_F32) return launch_plain<float>(a, stream);
    if (dtype == LLME_BF16) return launch_plain<__nv_bfloat16>(a, stream);
    LLME_REFUSE("window attention: unsupported dtype %d", dtype);
}
