// 32-bit residual stream: embedding gather into fp32 rows, and the residual update fused with the norm that follows it.
//
// ps_residual_norm, per row of W values:
//     x += coef * (rms(a) * wa + rms(b) * wb)      two mixer branches, each normed over the width, or
//     x += coef * y                                one projection output
//     x += coef * (sum_k weight_k ye[index_k] + same * hin (+ y))    a mixture's experts, its input and a shared expert's output
//     x += add ; x += step                         optional (embedding output; step vector of a pass or a projection's bias)
//     h  = rms(x) * w * scale                      optional; stored as bf16 or f32, zero-padded to `width` columns, with a
//                                                  constant 1 in column W when asked for (the projection's bias column)
// so a residual update, the loop bookkeeping and the next projection's input cost one launch and one pass over the rows.
// ps_embed_pairs starts a model whose embedding adds a row per token and one per pair of neighbouring tokens: the sum, normed.
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

struct EmbedPairsArgs {
    const int* ids; const void* table; const void* pairs; int vocab, buckets; long long mul_prev, mul_cur;
    const float* w; float eps; int W;
    const int* row_slot; const int* seqs; int n_seqs;
    int* last_token;             // [slots]: the last token of every sequence
    float* out; uint32_t* status;
};

// grid = n_seqs CTAs for the first rows of the sequences' portions (the only ones that look into the state, which they then
// replace) + one CTA per row
template <typename T>
__global__ void __launch_bounds__(256) embed_pairs_kernel(const EmbedPairsArgs a) {
    extern __shared__ float ep_row[];
    __shared__ float red[32];
    int row, prev;
    if ((int)blockIdx.x < a.n_seqs) {
        const int* sd = a.seqs + 4 * blockIdx.x;
        if (sd[1] <= 0 || sd[2] < 0) return;
        row = sd[0];
        prev = sd[3] == 0 ? -1 : a.last_token[sd[2]];
        __syncthreads();
        if (threadIdx.x == 0) a.last_token[sd[2]] = a.ids[row + sd[1] - 1];
    } else {
        row = blockIdx.x - a.n_seqs;
        const int slot = a.row_slot[row];
        if (slot < 0) {                                              // padding row
            for (int i = threadIdx.x; i < a.W; i += blockDim.x) a.out[(size_t)row * a.W + i] = 0.f;
            return;
        }
        if (row == 0 || a.row_slot[row - 1] != slot) return;
        prev = a.ids[row - 1];
    }
    const int cur = a.ids[row];
    const bool ok = cur >= 0 && cur < a.vocab;
    if (!ok && threadIdx.x == 0) set_status(a.status, PS_DEV_BAD_INDEX);
    long long at = a.buckets;
    if (prev >= 0) {
        at = ((long long)prev * a.mul_prev + (long long)cur * a.mul_cur) % a.buckets;
        if (at < 0) at += a.buckets;
    }
    const T* e = reinterpret_cast<const T*>(a.table) + (size_t)(ok ? cur : 0) * a.W;
    const T* p = reinterpret_cast<const T*>(a.pairs) + (size_t)at * a.W;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.W; i += blockDim.x) {
        const float v = (float)e[i] + (float)p[i];
        ep_row[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.W + a.eps);
    for (int i = threadIdx.x; i < a.W; i += blockDim.x) a.out[(size_t)row * a.W + i] = ep_row[i] * inv * a.w[i];
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
    // a mixture's contribution (y: its shared expert, may be null)
    int top; const int* index; const float* weight; const float* same; const float* ye; int ldye; const void* hin; int ldh;
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

constexpr int kRnMaxTop = 32;
template <int VEC> __device__ __forceinline__ FVec<VEC> fload_as(const float* p) { return fload<VEC>(p); }
template <int VEC> __device__ __forceinline__ FVec<VEC> fload_as(const __nv_bfloat16* p) {
    FVec<VEC> r;
    if constexpr (VEC == 4) {
        const uint2 t = *reinterpret_cast<const uint2*>(p);
        const float2 lo = bf16x2_bits_to_f32x2(t.x), hi = bf16x2_bits_to_f32x2(t.y);
        r.v[0] = lo.x; r.v[1] = lo.y; r.v[2] = hi.x; r.v[3] = hi.y;
    } else r.v[0] = bf16_to_f32(*p);
    return r;
}

// One CTA per row; the updated row waits in shared memory for its sum of squares.  EXPERTS: what is pending is a mixture's.
template <typename T, int VEC, bool EXPERTS>
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
    __shared__ int s_at[EXPERTS ? kRnMaxTop : 1];
    __shared__ float s_w[EXPERTS ? kRnMaxTop : 1];
    [[maybe_unused]] float same = 0.f;
    if constexpr (EXPERTS) {
        if ((int)threadIdx.x < g.top) { s_at[threadIdx.x] = g.index[(size_t)r * g.top + threadIdx.x]; s_w[threadIdx.x] = g.weight[(size_t)r * g.top + threadIdx.x]; }
        same = g.same[r];
        __syncthreads();
    }
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
        if constexpr (EXPERTS) {
            FVec<VEC> s;
            if (y != nullptr) s = fload<VEC>(y + i);
            else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) s.v[e] = 0.f;
            }
            if (same != 0.f) {
                const FVec<VEC> u = fload_as<VEC>(reinterpret_cast<const T*>(g.hin) + (size_t)r * g.ldh + i);
#pragma unroll
                for (int e = 0; e < VEC; ++e) s.v[e] = fmaf(same, u.v[e], s.v[e]);
            }
            for (int k0 = 0; k0 < g.top; k0 += 4) {                      // four rows' loads in flight together
                FVec<VEC> u[4];
                float wk[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int at = k0 + j < g.top ? s_at[k0 + j] : -1;
                    wk[j] = at >= 0 ? s_w[k0 + j] : 0.f;
                    if (at >= 0) u[j] = fload<VEC>(g.ye + (size_t)at * g.ldye + i);
                    else {
#pragma unroll
                        for (int e = 0; e < VEC; ++e) u[j].v[e] = 0.f;
                    }
                }
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int e = 0; e < VEC; ++e) s.v[e] = fmaf(wk[j], u[j].v[e], s.v[e]);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) v.v[e] = fmaf(g.coef, s.v[e], v.v[e]);
        } else if (a != nullptr) {
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

template <bool EXPERTS>
static int launch_residual_norm(const ResidualNormArgs& g, int rows, int h_f32, bool vec, cudaStream_t stream) {
    const size_t smem = (size_t)g.W * 4;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(residual_norm_kernel<float, 1, EXPERTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<float, 4, EXPERTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<__nv_bfloat16, 1, EXPERTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(residual_norm_kernel<__nv_bfloat16, 4, EXPERTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        attr_set = true;
    }
    // few rows: one wide CTA per row (latency); many rows: smaller CTAs, several per SM
    const dim3 block(rows <= 64 && g.W >= 2048 ? 1024 : 256);
    if (h_f32) return vec ? launch_pdl(residual_norm_kernel<float, 4, EXPERTS>, dim3(rows), block, smem, stream, g)
                          : launch_pdl(residual_norm_kernel<float, 1, EXPERTS>, dim3(rows), block, smem, stream, g);
    return vec ? launch_pdl(residual_norm_kernel<__nv_bfloat16, 4, EXPERTS>, dim3(rows), block, smem, stream, g)
               : launch_pdl(residual_norm_kernel<__nv_bfloat16, 1, EXPERTS>, dim3(rows), block, smem, stream, g);
}

}  // namespace ps

// `pairs`: [buckets + 1, W], the last row for the first token of a sequence; tables bf16 or (`f32`) fp32.
PS_API int ps_embed_pairs(const void* ids, const void* table, const void* pairs, int f32, int rows, int vocab, int buckets, long long mul_prev,
                          long long mul_cur, const void* w, float eps, int W, const void* row_slot, const void* seqs, int n_seqs,
                          void* last_token, void* out, void* status, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || W <= 0 || W > 32768 || buckets < 1 || n_seqs < 1) return (int)cudaErrorInvalidValue;
    EmbedPairsArgs a;
    a.ids = (const int*)ids; a.table = table; a.pairs = pairs; a.vocab = vocab; a.buckets = buckets; a.mul_prev = mul_prev; a.mul_cur = mul_cur;
    a.w = (const float*)w; a.eps = eps; a.W = W; a.row_slot = (const int*)row_slot; a.seqs = (const int*)seqs; a.n_seqs = n_seqs;
    a.last_token = (int*)last_token; a.out = (float*)out; a.status = (uint32_t*)status;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(embed_pairs_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        cudaFuncSetAttribute(embed_pairs_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        set = true;
    }
    if (f32) embed_pairs_kernel<float><<<n_seqs + rows, 256, (size_t)W * 4, stream>>>(a);
    else embed_pairs_kernel<__nv_bfloat16><<<n_seqs + rows, 256, (size_t)W * 4, stream>>>(a);
    return PS_LAUNCH_CHECK();
}

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
    ResidualNormArgs g = {};
    g.x = (const float*)x; g.x_out = (float*)x_out; g.W = W; g.a = (const float*)a; g.lda = lda; g.wa = (const float*)wa;
    g.b = (const float*)b; g.ldb = ldb; g.wb = (const float*)wb; g.y = (const float*)y; g.ldy = ldy; g.coef = coef;
    g.add = (const float*)add; g.step = (const float*)step; g.w = (const float*)w; g.eps = eps; g.scale = scale;
    g.h = h; g.width = width; g.one = one;
    const uintptr_t al = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)a | (uintptr_t)b | (uintptr_t)wa | (uintptr_t)wb | (uintptr_t)y |
                         (uintptr_t)add | (uintptr_t)step | (uintptr_t)w | (uintptr_t)h;
    const bool vec = W % 4 == 0 && lda % 4 == 0 && ldb % 4 == 0 && ldy % 4 == 0 && width % 4 == 0 && al % 16 == 0;
    return launch_residual_norm<false>(g, rows, h_f32, vec, stream);
}

// As ps_residual_norm with a mixture pending: row r adds coef * (sum over its `top` places of weight * ye[index] (index -1: nothing)
// + same * hin[r] + shared[r]); `hin` has the type of `h`, `shared` may be null.
PS_API int ps_residual_norm_experts(const void* x, void* x_out, int rows, int W, const void* index, const void* weight, const void* same,
                                    int top, const void* ye, int ldye, const void* hin, int ldh, const void* shared, int lds, float coef,
                                    const void* step, const void* w, float eps, void* h, int h_f32, int width, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || W <= 0 || W > 32768 || top < 1 || top > kRnMaxTop || (h != nullptr && (w == nullptr || width < W))) return (int)cudaErrorInvalidValue;
    ResidualNormArgs g = {};
    g.x = (const float*)x; g.x_out = (float*)x_out; g.W = W; g.y = (const float*)shared; g.ldy = lds; g.coef = coef; g.step = (const float*)step;
    g.w = (const float*)w; g.eps = eps; g.scale = 1.f; g.h = h; g.width = width;
    g.top = top; g.index = (const int*)index; g.weight = (const float*)weight; g.same = (const float*)same; g.ye = (const float*)ye; g.ldye = ldye;
    g.hin = hin; g.ldh = ldh;
    const uintptr_t al = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)ye | (uintptr_t)hin | (uintptr_t)shared | (uintptr_t)step | (uintptr_t)w | (uintptr_t)h;
    const bool vec = W % 4 == 0 && ldye % 4 == 0 && ldh % 4 == 0 && lds % 4 == 0 && width % 4 == 0 && al % 16 == 0;
    return launch_residual_norm<true>(g, rows, h_f32, vec, stream);
}
