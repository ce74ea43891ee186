// Parallel 32-bit residual streams (hyper-connections): writing a sublayer's output into all streams, reading the next
// sublayer's input from them, and its norm, in one launch and one pass over the row.  Per row of S streams of W values:
//     x_t <- sum_s mix[s, t] x_s + out[t] y        all streams at once from the old ones (skipped without a pending y)
//     u   =  sum_s read[s] x_s
//     h   =  rms(u) * w                            stored as bf16 or f32, zero-padded to `width` columns
// The streams of the input may lie at any stride (0: all are the embedding).  Counterpart of residual_norm.cu's one stream.
#include "ps_common.cuh"

namespace ps {

constexpr int kSnMaxStreams = 64;

struct StreamNormArgs {
    const float* x; long long row_stride, stream_stride;       // elements; stream t of row r at x + r * row_stride + t * stream_stride
    float* x_out;                                              // [rows, S, W] or null: the streams are not needed again
    int W, S;
    const float* mix; const float* out; const float* y; int ldy;         // y null: nothing is pending
    const float* read; const float* w; float eps;
    void* h; int width;                                        // h null: the streams are only written
};

template <typename T> __device__ __forceinline__ T sn_cast(float v);
template <> __device__ __forceinline__ float sn_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 sn_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

template <int VEC> __device__ __forceinline__ void sn_load(const float* p, float (&v)[VEC]) {
    if constexpr (VEC == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else v[0] = *p;
}
template <int VEC> __device__ __forceinline__ void sn_store(float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}

// Norm of the row's `u` in shared memory; ends the kernel's work on the row.
template <typename T, int VEC>
__device__ __forceinline__ void sn_norm(const StreamNormArgs& g, const float* u, float ss, float* red) {
    const int r = blockIdx.x;
    float sum[1] = {ss};
    block_sum_n<1>(sum, red);
    const float inv = rsqrtf(sum[0] / (float)g.W + g.eps);
    T* h = reinterpret_cast<T*>(g.h) + (size_t)r * g.width;
    for (int i = threadIdx.x * VEC; i < g.W; i += blockDim.x * VEC) {
        float v[VEC], w[VEC];
        sn_load<VEC>(u + i, v);
        sn_load<VEC>(g.w + i, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] *= inv * w[e];
        if constexpr (VEC == 4 && sizeof(T) == 2)
            *reinterpret_cast<uint2*>(h + i) = make_uint2(f32x2_to_bf16x2_bits(v[0], v[1]), f32x2_to_bf16x2_bits(v[2], v[3]));
        else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) h[i + e] = sn_cast<T>(v[e]);
        }
    }
    for (int i = g.W + threadIdx.x; i < g.width; i += blockDim.x) h[i] = sn_cast<T>(0.f);
}

// One CTA per row; S streams known at compile time.
template <typename T, int S, int VEC>
__global__ void __launch_bounds__(512) stream_norm_kernel(const StreamNormArgs g) {
    extern __shared__ __align__(16) float sn_row[];
    __shared__ float red[64];
    cudaTriggerProgrammaticLaunchCompletion();
    float mix[S][S], out[S], rd[S];                            // weights: not written by the predecessor
#pragma unroll
    for (int s = 0; s < S; ++s) {
        out[s] = g.y != nullptr ? __ldg(g.out + s) : 0.f;
        rd[s] = g.h != nullptr ? __ldg(g.read + s) : 0.f;
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = g.y != nullptr ? __ldg(g.mix + s * S + t) : 0.f;
    }
    cudaGridDependencySynchronize();
    const int r = blockIdx.x, W = g.W;
    const float* x = g.x + (size_t)r * g.row_stride;
    const float* y = g.y != nullptr ? g.y + (size_t)r * g.ldy : nullptr;
    float* xo = g.x_out != nullptr ? g.x_out + (size_t)r * S * W : nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < W; i += blockDim.x * VEC) {
        float v[S][VEC], u[VEC];
#pragma unroll
        for (int s = 0; s < S; ++s) sn_load<VEC>(x + s * g.stream_stride + i, v[s]);
        if (y != nullptr) {
            float vy[VEC], n[S][VEC];
            sn_load<VEC>(y + i, vy);
#pragma unroll
            for (int t = 0; t < S; ++t)
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    float a = out[t] * vy[e];
#pragma unroll
                    for (int s = 0; s < S; ++s) a = fmaf(mix[s][t], v[s][e], a);
                    n[t][e] = a;
                }
#pragma unroll
            for (int t = 0; t < S; ++t) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[t][e] = n[t][e];
                if (xo != nullptr) sn_store<VEC>(xo + (size_t)t * W + i, v[t]);
            }
        }
        if (g.h == nullptr) continue;
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float a = 0.f;
#pragma unroll
            for (int s = 0; s < S; ++s) a = fmaf(rd[s], v[s][e], a);
            u[e] = a;
            ss = fmaf(a, a, ss);
        }
        sn_store<VEC>(sn_row + i, u);
    }
    if (g.h != nullptr) sn_norm<T, VEC>(g, sn_row, ss, red);
}

// Any number of streams up to kSnMaxStreams: weights in shared memory, the streams of one column in local storage.
template <typename T>
__global__ void __launch_bounds__(256) stream_norm_any_kernel(const StreamNormArgs g) {
    extern __shared__ __align__(16) float sn_row[];
    __shared__ float red[64], s_mix[kSnMaxStreams * kSnMaxStreams], s_out[kSnMaxStreams], s_read[kSnMaxStreams];
    cudaTriggerProgrammaticLaunchCompletion();
    const int S = g.S, r = blockIdx.x, W = g.W;
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = g.y != nullptr ? g.mix[i] : 0.f;
    for (int i = threadIdx.x; i < S; i += blockDim.x) { s_out[i] = g.y != nullptr ? g.out[i] : 0.f; s_read[i] = g.h != nullptr ? g.read[i] : 0.f; }
    cudaGridDependencySynchronize();
    __syncthreads();
    float ss = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float v[kSnMaxStreams];
        for (int s = 0; s < S; ++s) v[s] = g.x[(size_t)r * g.row_stride + s * g.stream_stride + i];
        const float y = g.y != nullptr ? g.y[(size_t)r * g.ldy + i] : 0.f;
        float u = 0.f;
        for (int t = 0; t < S; ++t) {
            float a = v[t];
            if (g.y != nullptr) {
                a = s_out[t] * y;
                for (int s = 0; s < S; ++s) a = fmaf(s_mix[s * S + t], v[s], a);
                if (g.x_out != nullptr) g.x_out[((size_t)r * S + t) * W + i] = a;
            }
            u = fmaf(s_read[t], a, u);
        }
        ss = fmaf(u, u, ss);
        sn_row[i] = u;
    }
    if (g.h != nullptr) sn_norm<T, 1>(g, sn_row, ss, red);
}

template <typename T, int S>
static int launch_stream_norm(const StreamNormArgs& g, int rows, bool vec, cudaStream_t stream) {
    const size_t smem = (size_t)g.W * 4;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(stream_norm_kernel<T, S, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(stream_norm_kernel<T, S, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        attr_set = true;
    }
    const dim3 block(rows <= 148 && g.W >= 2048 ? 512 : 256);             // few rows: one wide CTA each
    return vec ? launch_pdl(stream_norm_kernel<T, S, 4>, dim3(rows), block, smem, stream, g)
               : launch_pdl(stream_norm_kernel<T, S, 1>, dim3(rows), block, smem, stream, g);
}

template <typename T>
static int launch_stream_norm_any(const StreamNormArgs& g, int rows, bool vec, cudaStream_t stream) {
    switch (g.S) {
        case 1: return launch_stream_norm<T, 1>(g, rows, vec, stream);
        case 2: return launch_stream_norm<T, 2>(g, rows, vec, stream);
        case 3: return launch_stream_norm<T, 3>(g, rows, vec, stream);
        case 4: return launch_stream_norm<T, 4>(g, rows, vec, stream);
        case 6: return launch_stream_norm<T, 6>(g, rows, vec, stream);
        case 8: return launch_stream_norm<T, 8>(g, rows, vec, stream);
        default: break;
    }
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(stream_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        attr_set = true;
    }
    return launch_pdl(stream_norm_any_kernel<T>, dim3(rows), dim3(256), (size_t)g.W * 4, stream, g);
}

}  // namespace ps

// `x_out` may be the buffer `x` points into (same layout) or null; `h` may be null.
PS_API int ps_stream_norm(const void* x, long long row_stride, long long stream_stride, void* x_out, int rows, int W, int S, const void* mix,
                          const void* out, const void* y, int ldy, const void* read, const void* w, float eps, void* h, int h_f32, int width,
                          cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || W <= 0 || W > 32768 || S < 1 || S > kSnMaxStreams || (y != nullptr && (mix == nullptr || out == nullptr || ldy < W)) ||
        (h != nullptr && (read == nullptr || w == nullptr || width < W)))
        return (int)cudaErrorInvalidValue;
    StreamNormArgs g;
    g.x = (const float*)x; g.row_stride = row_stride; g.stream_stride = stream_stride; g.x_out = (float*)x_out; g.W = W; g.S = S;
    g.mix = (const float*)mix; g.out = (const float*)out; g.y = (const float*)y; g.ldy = ldy; g.read = (const float*)read;
    g.w = (const float*)w; g.eps = eps; g.h = h; g.width = width;
    const uintptr_t al = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)w | (uintptr_t)h;
    const bool vec = W % 4 == 0 && ldy % 4 == 0 && width % 4 == 0 && row_stride % 4 == 0 && stream_stride % 4 == 0 && al % 16 == 0;
    return h_f32 ? launch_stream_norm_any<float>(g, rows, vec, stream) : launch_stream_norm_any<__nv_bfloat16>(g, rows, vec, stream);
}
