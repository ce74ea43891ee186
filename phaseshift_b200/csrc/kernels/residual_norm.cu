// 32-bit residual stream: embedding gather into fp32 rows, and the residual update fused with the norm that follows it.
//
// ps_residual_norm, per row of W values:
//     x += coef * (rms(a) * wa + rms(b) * wb)      two mixer branches, each normed over the width, or
//     x += coef * y                                one projection output
//     x += add ; x += step                         optional (embedding output and step vector at the start of a pass)
//     h  = rms(x) * w * scale                      optional; stored as bf16 or f32, zero-padded to `width` columns, with a
//                                                  constant 1 in column W when asked for (the projection's bias column)
// so a residual update, the loop bookkeeping and the next projection's input cost one launch and one pass over the rows.
// The hybrid decoder keeps a bf16 residual inside its projection epilogues instead (gemm_bs.cu, gemv_core.cuh).
#include "ps_common.cuh"

namespace ps {

template <typename T> __device__ __forceinline__ T rn_cast(float v);
template <> __device__ __forceinline__ float rn_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 rn_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

// out[r, :] = table[ids[r], :] widened to fp32; an id outside [0, vocab) writes zeros and flags the status word.
template <typename T>
__global__ void embed_f32_kernel(const int* ids, const T* table, int vocab, int W, float* out, uint32_t* status) {
    const int r = blockIdx.x, id = ids[r];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) set_status(status, PS_DEV_BAD_INDEX);
    const T* src = table + (size_t)(ok ? id : 0) * W;
    float* dst = out + (size_t)r * W;
    for (int i = threadIdx.x; i < W; i += blockDim.x) dst[i] = ok ? (float)src[i] : 0.f;
}

struct ResidualNormArgs {
    const float* x; float* x_out; int W;
    const float* a; int lda; const float* wa;
    const float* b; int ldb; const float* wb;
    const float* y; int ldy;
    float coef;
    const float* add; const float* step;
    const float* w; float eps; float scale;
    void* h; int width; int one;
};

template <int VEC> struct FVec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ FVec<VEC> fload(const float* p) {
    FVec<VEC> r;
    if constexpr (VEC == 4) { const float4 t = *reinterpret_cast<const float4*>(p); r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w; }
    else r.v[0] = *p;
    return r;
}
template <int VEC> __device__ __forceinline__ void fstore(float* p, const FVec<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}

// One CTA per row; the updated row waits in shared memory for its sum of squares.
template <typename T, int VEC>
__global__ void residual_norm_kernel(const ResidualNormArgs g) {
    extern __shared__ __align__(16) float rn_row[];
    __shared__ float red[64];
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int r = blockIdx.x, W = g.W, stride = blockDim.x * VEC;
    const float* x = g.x + (size_t)r * W;
    const float* a = g.a != nullptr ? g.a + (size_t)r * g.lda : nullptr;
    const float* b = g.a != nullptr ? g.b + (size_t)r * g.ldb : nullptr;
    const float* y = g.y != nullptr ? g.y + (size_t)r * g.ldy : nullptr;
    float ia = 0.f, ib = 0.f;
    if (a != nullptr) {
        float ss[2] = {0.f, 0.f};
        for (int i = threadIdx.x * VEC; i < W; i += stride) {
            const FVec<VEC> va = fload<VEC>(a + i), vb = fload<VEC>(b + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) { ss[0] = fmaf(va.v[e], va.v[e], ss[0]); ss[1] = fmaf(vb.v[e], vb.v[e], ss[1]); }
        }
        block_sum_n<2>(ss, red);
        ia = rsqrtf(ss[0] / (float)W + g.eps) * g.coef;
        ib = rsqrtf(ss[1] / (float)W + g.eps) * g.coef;
    }
    float ss[1] = {0.f};
    for (int i = threadIdx.x * VEC; i < W; i += stride) {
        FVec<VEC> v = fload<VEC>(x + i);
        if (a != nullptr) {
            const FVec<VEC> va = fload<VEC>(a + i), vb = fload<VEC>(b + i), wa = fload<VEC>(g.wa + i), wb = fload<VEC>(g.wb + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] += va.v[e] * ia * wa.v[e] + vb.v[e] * ib * wb.v[e];
        } else if (y != nullptr) {
            const FVec<VEC> vy = fload<VEC>(y + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] = fmaf(g.coef, vy.v[e], v.v[e]);
        }
        if (g.add != nullptr) {
            const FVec<VEC> t = fload<VEC>(g.add + (size_t)r * W + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] += t.v[e];
        }
        if (g.step != nullptr) {
            const FVec<VEC> t = fload<VEC>(g.step + i);
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] += t.v[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss[0] = fmaf(v.v[e], v.v[e], ss[0]);
        if (g.x_out != nullptr) fstore<VEC>(g.x_out + (size_t)r * W + i, v);
        fstore<VEC>(rn_row + i, v);
    }
    if (g.h == nullptr) return;
    block_sum_n<1>(ss, red);
    const float inv = rsqrtf(ss[0] / (float)W + g.eps);
    T* h = reinterpret_cast<T*>(g.h) + (size_t)r * g.width;
    for (int i = threadIdx.x * VEC; i < W; i += stride) {
        const FVec<VEC> v = fload<VEC>(rn_row + i), w = fload<VEC>(g.w + i);
        float o[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = v.v[e] * inv * w.v[e] * g.scale;
        if constexpr (VEC == 4 && sizeof(T) == 2)
            *reinterpret_cast<uint2*>(h + i) = make_uint2(f32x2_to_bf16x2_bits(o[0], o[1]), f32x2_to_bf16x2_bits(o[2], o[3]));
        else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) h[i + e] = rn_cast<T>(o[e]);
        }
    }
    for (int i = W + threadIdx.x; i < g.width; i += blockDim.x) h[i] = rn_cast<T>(i == W && g.one ? 1.f : 0.f);
}

}  // namespace ps

PS_API int ps_embed_f32(const void* ids, const void* table, int table_f32, int rows, int vocab, int W, void* out, void* status,
                        cudaStream_t stream) {
    if (rows <= 0 || W <= 0) return (int)cudaErrorInvalidValue;
    if (table_f32) ps::embed_f32_kernel<float><<<rows, 256, 0, stream>>>((const int*)ids, (const float*)table, vocab, W, (float*)out, (uint32_t*)status);
    else ps::embed_f32_kernel<__nv_bfloat16><<<rows, 256, 0, stream>>>((const int*)ids, (const __nv_bfloat16*)table, vocab, W, (float*)out, (uint32_t*)status);
    return PS_LAUNCH_CHECK();
}

// `x_out` may equal `x` or be null (nothing but the norm is wanted); `a`/`b` and `y` exclude each other; `h` may be null.
PS_API int ps_residual_norm(const void* x, void* x_out, int rows, int W, const void* a, int lda, const void* wa, const void* b, int ldb,
                            const void* wb, const void* y, int ldy, float coef, const void* add, const void* step, const void* w,
                            float eps, float scale, void* h, int h_f32, int width, int one, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || W <= 0 || W > 32768 || (a != nullptr && (b == nullptr || wa == nullptr || wb == nullptr || y != nullptr)) ||
        (h != nullptr && (w == nullptr || width < W + (one ? 1 : 0))))
        return (int)cudaErrorInvalidValue;
    ResidualNormArgs g;
    g.x = (const float*)x; g.x_out = (float*)x_out; g.W = W; g.a = (const float*)a; g.lda = lda; g.wa = (const float*)wa;
    g.b = (const float*)b; g.ldb = ldb; g.wb = (const float*)wb; g.y = (const float*)y; g.ldy = ldy; g.coef = coef;
    g.add = (const float*)add; g.step = (const float*)step; g.w = (const float*)w; g.eps = eps; g.scale = scale;
    g.h = h; g.width = width; g.one = one;
    const uintptr_t al = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)a | (uintptr_t)b | (uintptr_t)wa | (uintptr_t)wb | (uintptr_t)y |
                         (uintptr_t)add | (uintptr_t)step | (uintptr_t)w | (uintptr_t)h;
    const bool vec = W % 4 == 0 && lda % 4 == 0 && ldb % 4 == 0 && ldy % 4 == 0 && width % 4 == 0 && al % 16 == 0;
    const size_t smem = (size_t)W * 4;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(residual_norm_kernel<float, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<float, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<__nv_bfloat16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        attr_set = true;
    }
    // few rows: one wide CTA per row (latency); many rows: smaller CTAs, several per SM
    const dim3 block(rows <= 64 && W >= 2048 ? 1024 : 256);
    if (h_f32) return vec ? launch_pdl(residual_norm_kernel<float, 4>, dim3(rows), block, smem, stream, g)
                          : launch_pdl(residual_norm_kernel<float, 1>, dim3(rows), block, smem, stream, g);
    return vec ? launch_pdl(residual_norm_kernel<__nv_bfloat16, 4>, dim3(rows), block, smem, stream, g)
               : launch_pdl(residual_norm_kernel<__nv_bfloat16, 1>, dim3(rows), block, smem, stream, g);
}
