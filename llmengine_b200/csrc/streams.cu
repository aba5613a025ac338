// Residual streams (hyper-connections): a token's residual is S streams of D values side by side, 32-bit.  One kernel stands
// between two sublayers: it takes the result of the one before into the streams, sums what the next one reads out of them
// and norms that sum, so the streams cross memory once in either direction per sublayer.
//
//   with y:    g = sigmoid(gate + bias);  x_t <- sum_s mix[s, t] x_s + put[t] y g   for all t, from the old x
//   with out:  u = sum_s read[s] x_s;     out = u / sqrt(mean(u^2) + eps) * gain
//
// A block owns a row; the sums over the streams and over the row are formed in a fixed order, so a row never depends on what
// else is in the launch.
#include "common.cuh"
#include "kernel_args.h"

LLME_API const char* llme_last_error() { return llme_error_buffer(); }

namespace {

typedef __nv_bfloat16 bf16;
constexpr int MOST_STREAMS = 16;

// sigmoid(z): in the 32-bit path, and where the products take bfloat16 (a few units in the last place of 32-bit)
__device__ __forceinline__ float gate_of(float z, float) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gate_of(float z, bf16) { return __frcp_rn(1.0f + __expf(-z)); }

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ float4 fma4(float a, float4 b, float4 c) { return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w)); }

// Any width and up to 16 streams, a column a thread at a time.
template <typename G, typename O>
__global__ void stream_norm_kernel(LlmeStreamNormArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[32];
    const int S = a.streams, D = a.size, i = blockIdx.x, r = a.rows ? a.rows[i] : i;
    float* x = a.x + (size_t)r * S * D;
    // the sum that is read of column j; `update`: from the streams as they stand, updated on the way (and stored, unless rows are picked)
    auto column = [&](int j, bool update) -> float {
        float old[MOST_STREAMS], u = 0.0f;
        for (int s = 0; s < S; ++s) old[s] = x[(size_t)s * D + j];
        float v = 0.0f;
        if (update) {
            v = a.y[(size_t)r * D + j];
            if (a.gate) v *= gate_of(to_f32(((const G*)a.gate)[(size_t)r * a.ldg + j]) + a.gate_bias[j], O());
        }
        for (int t = 0; t < S; ++t) {
            float n = old[t];
            if (update) {
                n = 0.0f;
                for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], old[s], n);
                n = fmaf(a.put[t], v, n);
                if (!a.rows) x[(size_t)t * D + j] = n;
            }
            if (a.read) u = fmaf(a.read[t], n, u);
        }
        return u;
    };
    float ss = 0.0f;
    for (int j = threadIdx.x; j < D; j += blockDim.x) {
        const float u = column(j, a.y != nullptr);
        ss += u * u;
    }
    if (!a.out) return;
    const float rinv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)D + a.eps);
    O* out = (O*)a.out + (size_t)i * D;
    // (a column's second reading is by the thread that stored it)
    for (int j = threadIdx.x; j < D; j += blockDim.x) out[j] = from_f32<O>(column(j, a.y != nullptr && a.rows) * rinv * a.gain[j]);
}

// Widths in fours, S streams known when compiling: a thread keeps V groups of four columns in registers from the first load to the
// last store; everything a row needs is on its way at once, what the weights give before the kernel before this one has finished.
template <int S, int V, typename G, typename O>
__global__ void __launch_bounds__(512) stream_norm_fours_kernel(LlmeStreamNormArgs a) {
    __shared__ float scratch[32];
    const int D = a.size, i = blockIdx.x, groups = D >> 2;
    float mix[S * S], put[S], read[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        read[s] = a.out ? a.read[s] : 0.0f;
        put[s] = a.y ? a.put[s] : 0.0f;
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s * S + t] = a.y ? a.mix[s * S + t] : (s == t ? 1.0f : 0.0f);
    }
    const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    float4 gain[V], bias[V];
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int j = threadIdx.x + k * blockDim.x;
        const bool in = j < groups;
        gain[k] = in && a.out ? load4<float>(a.gain + 4 * j) : zero;
        bias[k] = in && a.gate ? load4<float>(a.gate_bias + 4 * j) : zero;
    }
    pdl_launch_dependents();
    pdl_wait();
    const int r = a.rows ? a.rows[i] : i;
    float* x = a.x + (size_t)r * S * D;
    float4 old[V][S], y[V], g[V];
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int j = threadIdx.x + k * blockDim.x;
        const bool in = j < groups;
#pragma unroll
        for (int s = 0; s < S; ++s) old[k][s] = in ? load4<float>(x + (size_t)s * D + 4 * j) : zero;
        y[k] = in && a.y ? load4<float>(a.y + (size_t)r * D + 4 * j) : zero;
        g[k] = in && a.gate ? load4<G>((const G*)a.gate + (size_t)r * a.ldg + 4 * j) : zero;
    }
    float4 u[V];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int j = threadIdx.x + k * blockDim.x;
        u[k] = zero;
        if (j >= groups) continue;
        if (a.y) {
            if (a.gate)
                y[k] = make_float4(y[k].x * gate_of(g[k].x + bias[k].x, O()), y[k].y * gate_of(g[k].y + bias[k].y, O()),
                                   y[k].z * gate_of(g[k].z + bias[k].z, O()), y[k].w * gate_of(g[k].w + bias[k].w, O()));
#pragma unroll
            for (int t = 0; t < S; ++t) {
                float4 n = zero;
#pragma unroll
                for (int s = 0; s < S; ++s) n = fma4(mix[s * S + t], old[k][s], n);
                n = fma4(put[t], y[k], n);
                if (!a.rows) store4(x + (size_t)t * D + 4 * j, n);
                u[k] = fma4(read[t], n, u[k]);
            }
        } else {
#pragma unroll
            for (int t = 0; t < S; ++t) u[k] = fma4(read[t], old[k][t], u[k]);
        }
        ss += u[k].x * u[k].x + u[k].y * u[k].y + u[k].z * u[k].z + u[k].w * u[k].w;
    }
    if (!a.out) return;
    const float rinv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)D + a.eps);
    O* out = (O*)a.out + (size_t)i * D;
#pragma unroll
    for (int k = 0; k < V; ++k) {
        const int j = threadIdx.x + k * blockDim.x;
        if (j < groups)
            store4(out + 4 * j, make_float4(u[k].x * rinv * gain[k].x, u[k].y * rinv * gain[k].y, u[k].z * rinv * gain[k].z, u[k].w * rinv * gain[k].w));
    }
}

template <int S, typename G, typename O>
bool launch_fours(const LlmeStreamNormArgs& a, cudaStream_t st) {
    const int groups = a.size / 4;
    auto threads = [&](int per) { return dim3(((groups + per - 1) / per + 31) / 32 * 32); };
    // few rows: short chains matter, a row is spread over many threads; many rows: two groups a thread, so that an SM holds more rows
    // with their loads on their way (2,048 rows of 4 x 2,048: 29 us against 40 us)
    if (groups <= 512 && a.tokens <= 296) llme_launch(stream_norm_fours_kernel<S, 1, G, O>, dim3(a.tokens), threads(1), 0, st, a);
    else if (groups <= 1024) llme_launch(stream_norm_fours_kernel<S, 2, G, O>, dim3(a.tokens), threads(2), 0, st, a);
    else if (groups <= 2048) llme_launch(stream_norm_fours_kernel<S, 4, G, O>, dim3(a.tokens), threads(4), 0, st, a);
    else return false;
    return true;
}

template <typename G, typename O>
int launch(const LlmeStreamNormArgs& a, cudaStream_t st) {
    const bool fours = a.size % 4 == 0 && a.ldg % 4 == 0 && (((uintptr_t)a.x | (uintptr_t)a.y | (uintptr_t)a.gate_bias | (uintptr_t)a.gain) & 15) == 0 &&
                       (uintptr_t)a.gate % (4 * sizeof(G)) == 0 && (uintptr_t)a.out % (4 * sizeof(O)) == 0;
    bool done = false;
    if (fours) {
        if (a.streams == 1) done = launch_fours<1, G, O>(a, st);
        else if (a.streams == 2) done = launch_fours<2, G, O>(a, st);
        else if (a.streams == 3) done = launch_fours<3, G, O>(a, st);
        else if (a.streams == 4) done = launch_fours<4, G, O>(a, st);
    }
    if (!done) llme_launch(stream_norm_kernel<G, O>, dim3(a.tokens), dim3(a.size >= 1024 ? 512 : 128), 0, st, a);
    LLME_LAUNCH_STATUS();
}

}  // namespace

LLME_API int llme_stream_norm(const LlmeStreamNormArgs* args, cudaStream_t stream) {
    const LlmeStreamNormArgs& a = *args;
    if (a.tokens <= 0) return 0;
    if (!a.x || a.size <= 0 || (!a.y && !a.out)) LLME_REFUSE("stream_norm: null pointer, non-positive size or nothing to do");
    if (a.streams < 1 || a.streams > MOST_STREAMS) LLME_REFUSE("stream_norm: %d streams, this build takes 1 to %d", a.streams, MOST_STREAMS);
    if (a.y && (!a.mix || !a.put)) LLME_REFUSE("stream_norm: a result without its weights");
    if (a.gate && (!a.y || !a.gate_bias)) LLME_REFUSE("stream_norm: a gate without a result or a bias");
    if (a.out && (!a.read || !a.gain || !(a.eps > 0.0f))) LLME_REFUSE("stream_norm: a norm needs its read weights, gain and a positive eps");
    if (a.gate && a.gate_dtype != LLME_F32 && a.gate_dtype != LLME_BF16) LLME_REFUSE("stream_norm: unsupported gate dtype %d", a.gate_dtype);
    if (a.out && a.out_dtype != LLME_F32 && a.out_dtype != LLME_BF16) LLME_REFUSE("stream_norm: unsupported output dtype %d", a.out_dtype);
    const bool g32 = !a.gate || a.gate_dtype == LLME_F32, o32 = !a.out || a.out_dtype == LLME_F32;
    if (g32) return o32 ? launch<float, float>(a, stream) : launch<float, bf16>(a, stream);
    return o32 ? launch<bf16, float>(a, stream) : launch<bf16, bf16>(a, stream);
}
