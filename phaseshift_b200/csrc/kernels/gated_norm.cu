// The end of a sublayer in models that norm what a sublayer returns (32-bit residual stream), in one launch per row of W values:
//     y  = ca * a + cb * b                         one or two projection outputs, or
//     y  = sum_k weight_k ye[index_k]              a mixture's experts
//     y *= sigmoid(gate + gate_bias)
//     x += groupnorm(y) * w                        every one of `groups` consecutive parts over its own root mean square
//     h  = x, or groupnorm(x) * final_w            the next projection's input: bf16 or f32, zero-padded to `width` columns
// With nothing pending only h is written.
// ps_soft_limit bounds logits: cap * tanh(z / cap).
#include "ps_common.cuh"

namespace ps {

struct GatedNormArgs {
    const float* x; float* x_out; int W, groups; float eps;
    const float* a; int lda; float ca;
    const float* b; int ldb; float cb;                     // may be null
    int top; const int* index; const float* weight; const float* ye; int ldye;
    const void* gate; int ldg; const float* gate_bias; const float* w;
    const float* final_w; void* h; int width;              // both may be null
};

enum GnSource : int { GN_NONE = 0, GN_PROJECTIONS = 1, GN_EXPERTS = 2 };
constexpr int kGnMaxTop = 32;

template <int VEC> struct GnVec { float v[VEC]; };
template <int VEC> __device__ __forceinline__ GnVec<VEC> gn_load(const float* p) {
    GnVec<VEC> r;
    if constexpr (VEC == 4) { const float4 t = *reinterpret_cast<const float4*>(p); r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w; }
    else r.v[0] = *p;
    return r;
}
template <int VEC> __device__ __forceinline__ GnVec<VEC> gn_load(const __nv_bfloat16* p) {
    GnVec<VEC> r;
    if constexpr (VEC == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const float2 lo = bf16x2_bits_to_f32x2(t.x), hi = bf16x2_bits_to_f32x2(t.y);
        r.v[0] = lo.x; r.v[1] = lo.y; r.v[2] = hi.x; r.v[3] = hi.y;
    } else r.v[0] = bf16_to_f32(*p);
    return r;
}
template <int VEC> __device__ __forceinline__ void gn_store(float* p, const GnVec<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VEC> __device__ __forceinline__ void gn_store(__nv_bfloat16* p, const GnVec<VEC>& r) {
    if constexpr (VEC == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f32x2_to_bf16x2_bits(r.v[0], r.v[1]), f32x2_to_bf16x2_bits(r.v[2], r.v[3]));
    else *p = f32_to_bf16(r.v[0]);
}

// 1 / root mean square of every group of the row in shared memory; `part`: max(groups, warps) floats.  Ends with a barrier.
__device__ __forceinline__ void group_scales(const float* row, int W, int groups, float eps, float* part, float* inv) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    const int size = W / groups, per = nw > groups ? nw / groups : 1;         // warps that share a group
    for (int it = warp; it < groups * per; it += nw) {
        const float* p = row + (it / per) * size;
        float s = 0.f;
        for (int i = (it % per) * 32 + lane; i < size; i += per * 32) s = fmaf(p[i], p[i], s);
        s = warp_sum(s);
        if (lane == 0) part[it] = s;
    }
    __syncthreads();
    for (int g = threadIdx.x; g < groups; g += blockDim.x) {
        float s = 0.f;
        for (int k = 0; k < per; ++k) s += part[g * per + k];
        inv[g] = rsqrtf(s / (float)size + eps);
    }
    __syncthreads();
}

// One CTA per row.  VEC: elements of a load (a group holds whole ones).
template <typename T, typename G, int VEC, int SRC>
__global__ void gated_norm_kernel(const GatedNormArgs g) {
    extern __shared__ __align__(16) float gn_smem[];
    float* row = gn_smem;                                    // [W]
    const int spare = (max(g.groups, 32) + 3) / 4 * 4;
    float* part = row + (g.W + 3) / 4 * 4;
    float* inv = part + spare;
    __shared__ int s_at[SRC == GN_EXPERTS ? kGnMaxTop : 1];
    __shared__ float s_w[SRC == GN_EXPERTS ? kGnMaxTop : 1];
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int r = blockIdx.x, W = g.W, stride = blockDim.x * VEC, first = threadIdx.x * VEC, size = W / g.groups;
    const float* x = g.x + (size_t)r * W;
    T* h = reinterpret_cast<T*>(g.h) + (size_t)r * g.width;
    if constexpr (SRC == GN_EXPERTS) {
        if ((int)threadIdx.x < g.top) { s_at[threadIdx.x] = g.index[(size_t)r * g.top + threadIdx.x]; s_w[threadIdx.x] = g.weight[(size_t)r * g.top + threadIdx.x]; }
        __syncthreads();
    }
    if constexpr (SRC != GN_NONE) {
        const G* gate = reinterpret_cast<const G*>(g.gate) + (size_t)r * g.ldg;
        for (int i = first; i < W; i += stride) {
            GnVec<VEC> y;
            const GnVec<VEC> gv = gn_load<VEC>(gate + i), gb = gn_load<VEC>(g.gate_bias + i);
            if constexpr (SRC == GN_PROJECTIONS) {
                y = gn_load<VEC>(g.a + (size_t)r * g.lda + i);
#pragma unroll
                for (int e = 0; e < VEC; ++e) y.v[e] *= g.ca;
                if (g.b != nullptr) {
                    const GnVec<VEC> t = gn_load<VEC>(g.b + (size_t)r * g.ldb + i);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(g.cb, t.v[e], y.v[e]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) y.v[e] = 0.f;
                for (int k0 = 0; k0 < g.top; k0 += 4) {                      // four rows' loads in flight together
                    GnVec<VEC> u[4];
                    float wk[4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const int at = k0 + j < g.top ? s_at[k0 + j] : -1;
                        wk[j] = at >= 0 ? s_w[k0 + j] : 0.f;
                        if (at >= 0) u[j] = gn_load<VEC>(g.ye + (size_t)at * g.ldye + i);
                        else {
#pragma unroll
                            for (int e = 0; e < VEC; ++e) u[j].v[e] = 0.f;
                        }
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int e = 0; e < VEC; ++e) y.v[e] = fmaf(wk[j], u[j].v[e], y.v[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) y.v[e] = y.v[e] / (1.f + expf(-(gv.v[e] + gb.v[e])));
            gn_store<VEC>(row + i, y);
        }
        __syncthreads();
        group_scales(row, W, g.groups, g.eps, part, inv);
    }
    for (int i = first; i < W; i += stride) {
        GnVec<VEC> v = gn_load<VEC>(x + i);
        if constexpr (SRC != GN_NONE) {
            const GnVec<VEC> y = gn_load<VEC>(row + i), w = gn_load<VEC>(g.w + i);
            const float s = inv[i / size];
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] += y.v[e] * s * w.v[e];
            gn_store<VEC>(g.x_out + (size_t)r * W + i, v);
        }
        if (g.final_w != nullptr) gn_store<VEC>(row + i, v);
        else if (g.h != nullptr) gn_store<VEC>(h + i, v);
    }
    if (g.h == nullptr) return;
    if (g.final_w != nullptr) {
        __syncthreads();
        group_scales(row, W, g.groups, g.eps, part, inv);
        for (int i = first; i < W; i += stride) {
            GnVec<VEC> v = gn_load<VEC>(row + i);
            const GnVec<VEC> w = gn_load<VEC>(g.final_w + i);
            const float s = inv[i / size];
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] *= s * w.v[e];
            gn_store<VEC>(h + i, v);
        }
    }
    GnVec<1> zero;
    zero.v[0] = 0.f;
    for (int i = W + threadIdx.x; i < g.width; i += blockDim.x) gn_store<1>(h + i, zero);
}

template <typename T, typename G, int VEC, int SRC>
static int launch_gn(const GatedNormArgs& g, int rows, cudaStream_t stream) {
    const size_t smem = ((size_t)(g.W + 3) / 4 * 4 + 2 * (((g.groups > 32 ? g.groups : 32) + 3) / 4 * 4)) * 4;
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(gated_norm_kernel<T, G, VEC, SRC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        set = true;
    }
    // few rows: one wide CTA per row (latency); many rows: smaller CTAs, several per SM
    const dim3 block(rows <= 64 && g.W >= 2048 ? 1024 : 256);
    return launch_pdl(gated_norm_kernel<T, G, VEC, SRC>, dim3(rows), block, smem, stream, g);
}

template <typename T, typename G, int VEC>
static int launch_gn_source(const GatedNormArgs& g, int rows, cudaStream_t stream) {
    if (g.gate == nullptr) return launch_gn<T, G, VEC, GN_NONE>(g, rows, stream);
    return g.top > 0 ? launch_gn<T, G, VEC, GN_EXPERTS>(g, rows, stream) : launch_gn<T, G, VEC, GN_PROJECTIONS>(g, rows, stream);
}

__global__ void __launch_bounds__(256) soft_limit_kernel(float* z, size_t n, float cap) {
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const size_t stride = (size_t)gridDim.x * 256 * 4;
    for (size_t i = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4; i < n; i += stride) {
        if (i + 3 < n) {
            float4 v = *reinterpret_cast<float4*>(z + i);
            v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap); v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap);
            *reinterpret_cast<float4*>(z + i) = v;
        } else
            for (size_t j = i; j < n; ++j) z[j] = cap * tanhf(z[j] / cap);
    }
}

}  // namespace ps

// `gate` null: nothing is pending, x_out is not written and everything up to `w` is unused.  `top` 0: y = ca * a + cb * b (`b` may be
// null); `top` > 0: the experts' sum, index -1: nothing.  `final_w` and `h` may be null; `x_out` may equal `x`.  The gate is bf16 or
// (`gate_f32`) fp32, h too (`h_f32`).
PS_API int ps_gated_norm(const void* x, void* x_out, int rows, int W, int groups, float eps, const void* a, int lda, float ca, const void* b,
                         int ldb, float cb, int top, const void* index, const void* weight, const void* ye, int ldye, const void* gate, int ldg,
                         int gate_f32, const void* gate_bias, const void* w, const void* final_w, void* h, int h_f32, int width,
                         cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || W <= 0 || groups < 1 || W % groups || top < 0 || top > kGnMaxTop || (h != nullptr && width < W) || (gate == nullptr && h == nullptr) ||
        (gate != nullptr && (x_out == nullptr || gate_bias == nullptr || w == nullptr || (top > 0 ? ye == nullptr : a == nullptr))))
        return (int)cudaErrorInvalidValue;
    GatedNormArgs g;
    g.x = (const float*)x; g.x_out = (float*)x_out; g.W = W; g.groups = groups; g.eps = eps; g.a = (const float*)a; g.lda = lda; g.ca = ca;
    g.b = (const float*)b; g.ldb = ldb; g.cb = cb; g.top = top; g.index = (const int*)index; g.weight = (const float*)weight; g.ye = (const float*)ye;
    g.ldye = ldye; g.gate = gate; g.ldg = ldg; g.gate_bias = (const float*)gate_bias; g.w = (const float*)w; g.final_w = (const float*)final_w;
    g.h = h; g.width = width;
    const uintptr_t al = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)a | (uintptr_t)b | (uintptr_t)ye | (uintptr_t)gate | (uintptr_t)gate_bias |
                         (uintptr_t)w | (uintptr_t)final_w | (uintptr_t)h;
    const bool vec = W / groups % 4 == 0 && lda % 4 == 0 && ldb % 4 == 0 && ldye % 4 == 0 && ldg % 4 == 0 && width % 4 == 0 && al % 16 == 0;
    if (h_f32) return vec ? launch_gn_source<float, float, 4>(g, rows, stream) : launch_gn_source<float, float, 1>(g, rows, stream);
    if (gate_f32) return vec ? launch_gn_source<__nv_bfloat16, float, 4>(g, rows, stream) : launch_gn_source<__nv_bfloat16, float, 1>(g, rows, stream);
    return vec ? launch_gn_source<__nv_bfloat16, __nv_bfloat16, 4>(g, rows, stream) : launch_gn_source<__nv_bfloat16, __nv_bfloat16, 1>(g, rows, stream);
}

// `n` contiguous fp32 values, 16-byte aligned.
PS_API int ps_soft_limit(void* z, long long n, float cap, cudaStream_t stream) {
    if (n <= 0 || !(cap > 0.f) || (uintptr_t)z % 16) return (int)cudaErrorInvalidValue;
    const long long ctas = (n + 1023) / 1024;
    return ps::launch_pdl(ps::soft_limit_kernel, dim3((unsigned)(ctas < 1184 ? ctas : 1184)), dim3(256), 0, stream, (float*)z, (size_t)n, cap);
}
