// From a projection row [q heads | k heads | v heads] to an attention's queries, keys and values, in one launch: a short causal
// convolution over time on every channel, a norm of the queries and of the keys over all heads at once, rotation of the first
// dimensions of every query and key head, division of a head by its root mean square, mixing with another layer's values, and the
// append to the pages.  Every part is optional (HeadsSpec in ops/specs.py); all of it is computed in 32-bit.
//
// The convolution's history is state: [slots, taps - 1, channels], the projected row of position p in row p % (taps - 1).  A row
// whose predecessors lie in the same step reads them from the projection; the first taps - 1 rows of a sequence's portion look
// into the history.  One CTA per sequence runs those rows and then stores the portion's last rows, so that nobody reads a row of
// the history that another CTA replaces; the other rows are spread over the other CTAs, a few consecutive ones for each (they
// share the convolution's weights and most of what it reads).
#include "ps_common.cuh"
#include "turn_angle.cuh"

namespace ps {

struct AttnHeadsArgs {
    const void* proj; int ld;
    int H, G, D, dim, vdim;                      // D: engine size of a head, dim / vdim: the model's sizes of keys and values
    int pairs, halves, unit, taps;
    float eps, turn_size;
    const double* freq;                          // [pairs]
    const float* q_norm; const float* k_norm;    // [H * D], [G * D] or null
    const void* conv_w; void* history;           // [taps, channels], [slots, taps - 1, channels]
    float mix; const void* saved_in; void* saved_out;      // [rows, G * vdim] or null
    void* q_out; void* k_pool; void* v_pool;
    const int* row_slot; const int* row_pos; const int* block_table; int max_blocks, page_tokens, num_pages;
    const int* seqs; int n_seqs, rows, group;
    uint32_t* status;
};

__device__ __forceinline__ float4 ah_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ah_load4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf16x2_bits_to_f32x2(v.x), b = bf16x2_bits_to_f32x2(v.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ah_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ah_store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(f32x2_to_bf16x2_bits(v.x, v.y), f32x2_to_bf16x2_bits(v.z, v.w));
}
__device__ __forceinline__ float4 ah_fma4(float4 a, float4 b, float4 c) {
    return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
template <typename T> __device__ __forceinline__ T ah_cast(float v);
template <> __device__ __forceinline__ float ah_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ah_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

// One row; `back`: rows of the same portion before it (taps or more: all that the convolution looks back to).
template <typename T, bool CONV>
__device__ __forceinline__ void heads_row(const AttnHeadsArgs& a, int row, int back, float* sx, float* s_sin, float* s_cos, float* s_inv,
                                          float* red) {
    const int t = threadIdx.x, n = blockDim.x, D = a.D, HD = a.H * D, KD = (a.H + a.G) * D, C = KD + a.G * D;
    const int slot = a.row_slot[row], pos = a.row_pos[row];
    T* q_out = reinterpret_cast<T*>(a.q_out) + (size_t)row * HD;
    if (slot < 0 || pos < 0) {                                       // padding row
        for (int c = 4 * t; c < HD; c += 4 * n) ah_store4(q_out + c, make_float4(0.f, 0.f, 0.f, 0.f));
        return;
    }
    const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld;
    const T* w = reinterpret_cast<const T*>(a.conv_w);
    const T* hist = reinterpret_cast<const T*>(a.history) + (size_t)slot * (a.taps - 1) * C;
    float ss[2] = {0.f, 0.f};
    for (int c = 4 * t; c < C; c += 4 * n) {
        float4 x = ah_load4(src + c);
        if constexpr (CONV) {
            const float4 wl = ah_load4(w + (size_t)(a.taps - 1) * C + c);
            x = make_float4(x.x * wl.x, x.y * wl.y, x.z * wl.z, x.w * wl.w);
            for (int j = 1; j < a.taps && j <= pos; ++j) {
                const T* u = j <= back ? src - (size_t)j * a.ld : hist + (size_t)((pos - j) % (a.taps - 1)) * C;
                x = ah_fma4(ah_load4(u + c), ah_load4(w + (size_t)(a.taps - 1 - j) * C + c), x);
            }
        }
        *reinterpret_cast<float4*>(sx + c) = x;
        const float sq = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
        if (c < HD) ss[0] += sq;
        else if (c < KD) ss[1] += sq;
    }
    for (int i = t; i < a.pairs; i += n) {
        float s, c;
        turn_angle(pos, a.freq[i], &s, &c);
        s_sin[i] = s * a.turn_size; s_cos[i] = c * a.turn_size;
    }
    float norm[2] = {1.f, 1.f};
    if (a.q_norm != nullptr) {
        block_sum_n<2>(ss, red);
        norm[0] = rsqrtf(ss[0] / (float)(a.H * a.dim) + a.eps);
        norm[1] = rsqrtf(ss[1] / (float)(a.G * a.dim) + a.eps);
    }
    __syncthreads();
    if (a.unit) {                                                    // a turn changes no length
        for (int h = t >> 5; h < a.H + a.G; h += n >> 5) {
            float s = 0.f;
            for (int d = 4 * (t & 31); d < D; d += 128) {
                const float4 x = *reinterpret_cast<const float4*>(sx + h * D + d);
                s += fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
            }
            s = warp_sum(s);
            if ((t & 31) == 0) s_inv[h] = rsqrtf(s / (float)a.dim + a.eps);
        }
        __syncthreads();
    }
    const int blk = pos / a.page_tokens, off = pos % a.page_tokens;
    const int page = blk < a.max_blocks ? a.block_table[(size_t)slot * a.max_blocks + blk] : -1;
    const bool mapped = page >= 0 && page < a.num_pages;
    if (!mapped && t == 0) set_status(a.status, PS_DEV_BAD_INDEX);
    for (int c = 4 * t; c < C; c += 4 * n) {
        const int head = c / D, d = c % D;
        float o[4];
        if (c < KD) {
            const bool isq = c < HD;
            const float* wn = a.q_norm == nullptr ? nullptr : isq ? a.q_norm : a.k_norm - HD;
            const float nm = isq ? norm[0] : norm[1];
            auto x = [&](int i) { return wn == nullptr ? sx[i] : sx[i] * nm * wn[i]; };
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int de = d + e;
                float v = x(c + e);
                if (a.halves) {
                    if (de < a.pairs) v = v * s_cos[de] - x(c + e + a.pairs) * s_sin[de];
                    else if (de < 2 * a.pairs) v = v * s_cos[de - a.pairs] + x(c + e - a.pairs) * s_sin[de - a.pairs];
                } else if (de < 2 * a.pairs) {
                    const int i = de >> 1;
                    v = (e & 1) ? v * s_cos[i] + x(c + e - 1) * s_sin[i] : v * s_cos[i] - x(c + e + 1) * s_sin[i];
                }
                o[e] = v;
            }
            if (a.unit) {
                const float inv = s_inv[head];
#pragma unroll
                for (int e = 0; e < 4; ++e) o[e] *= inv;
            }
        } else {
            const size_t at = (size_t)row * a.G * a.vdim + (size_t)(head - a.H - a.G) * a.vdim + d;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                o[e] = sx[c + e];
                if (d + e >= a.vdim) continue;
                if (a.saved_out != nullptr) reinterpret_cast<T*>(a.saved_out)[at + e] = ah_cast<T>(o[e]);
                if (a.saved_in != nullptr) o[e] = (1.f - a.mix) * o[e] + a.mix * (float)reinterpret_cast<const T*>(a.saved_in)[at + e];
            }
        }
        const float4 v = make_float4(o[0], o[1], o[2], o[3]);
        if (c < HD) ah_store4(q_out + c, v);
        else if (mapped) {
            const int kvh = c < KD ? head - a.H : head - a.H - a.G;
            T* pool = reinterpret_cast<T*>(c < KD ? a.k_pool : a.v_pool);
            ah_store4(pool + (((size_t)page * a.G + kvh) * a.page_tokens + off) * D + d, v);
        }
    }
}

// grid: (CONV: n_seqs CTAs for the first rows of the sequences' portions) + ceil(rows / group)
template <typename T, bool CONV>
__global__ void __launch_bounds__(512) attn_heads_kernel(const AttnHeadsArgs a) {
    extern __shared__ __align__(16) float sx[];
    __shared__ float red[64];
    const int C = (a.H + 2 * a.G) * a.D;
    float* s_sin = sx + C;
    float* s_cos = s_sin + a.pairs;
    float* s_inv = s_cos + a.pairs;
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int hist_rows = CONV ? a.taps - 1 : 0;
    int block = blockIdx.x;
    if (CONV) {
        if (block < a.n_seqs) {
            const int* sd = a.seqs + 4 * block;
            const int row0 = sd[0], n_rows = sd[1], slot = sd[2], pos0 = sd[3];
            if (n_rows <= 0 || slot < 0) return;
            for (int r = 0; r < min(n_rows, hist_rows); ++r) {
                heads_row<T, CONV>(a, row0 + r, r, sx, s_sin, s_cos, s_inv, red);
                __syncthreads();
            }
            T* hist = reinterpret_cast<T*>(a.history) + (size_t)slot * hist_rows * C;
            for (int r = max(0, n_rows - hist_rows); r < n_rows; ++r) {
                const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)(row0 + r) * a.ld;
                T* dst = hist + (size_t)((pos0 + r) % hist_rows) * C;
                for (int c = 4 * (int)threadIdx.x; c < C; c += 4 * blockDim.x) ah_store4(dst + c, ah_load4(src + c));
            }
            return;
        }
        block -= a.n_seqs;
    }
    for (int i = 0; i < a.group; ++i) {
        const int row = block * a.group + i;
        if (row >= a.rows) return;
        // (a step's rows of one sequence follow one another, and no two of its sequences share a slot)
        if (CONV && hist_rows > 0 && a.row_slot[row] >= 0 && (row < hist_rows || a.row_slot[row - hist_rows] != a.row_slot[row])) continue;
        heads_row<T, CONV>(a, row, a.taps, sx, s_sin, s_cos, s_inv, red);
        __syncthreads();
    }
}

template <typename T, bool CONV>
static int launch_heads(const AttnHeadsArgs& a, cudaStream_t stream) {
    const size_t smem = sizeof(float) * ((size_t)(a.H + 2 * a.G) * a.D + 2 * a.pairs + a.H + a.G);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(attn_heads_kernel<T, CONV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        set = true;
    }
    const int blocks = (CONV ? a.n_seqs : 0) + (a.rows + a.group - 1) / a.group;
    return launch_pdl(attn_heads_kernel<T, CONV>, dim3(blocks), dim3(a.rows <= 64 ? 512 : 256), smem, stream, a);
}

}  // namespace ps

// `f32`: projection, history, saved values, queries and pools are fp32 instead of bf16.  D a multiple of 4, `ld` of 4.
PS_API int ps_attn_heads(const void* proj, int ld, int f32, int rows, int H, int G, int D, int dim, int vdim, int pairs, int halves,
                         int unit, float eps, float turn_size, const void* freq, const void* q_norm, const void* k_norm, int taps,
                         const void* conv_w, void* history, float mix, const void* saved_in, void* saved_out, void* q_out, void* k_pool,
                         void* v_pool, const void* row_slot, const void* row_pos, const void* block_table, int max_blocks,
                         int page_tokens, int num_pages, const void* seqs, int n_seqs, void* status, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || H <= 0 || G <= 0 || D % 4 || ld % 4 || dim > D || vdim > D || 2 * pairs > dim || taps < 1 || (taps > 1 && (conv_w == nullptr || history == nullptr)) ||
        (conv_w != nullptr && n_seqs <= 0) || (q_norm == nullptr) != (k_norm == nullptr) ||
        ((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)history | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool) % 16)
        return (int)cudaErrorInvalidValue;
    AttnHeadsArgs a;
    a.proj = proj; a.ld = ld; a.H = H; a.G = G; a.D = D; a.dim = dim; a.vdim = vdim; a.pairs = pairs; a.halves = halves; a.unit = unit;
    a.taps = taps; a.eps = eps; a.turn_size = turn_size; a.freq = (const double*)freq; a.q_norm = (const float*)q_norm;
    a.k_norm = (const float*)k_norm; a.conv_w = conv_w; a.history = history; a.mix = mix; a.saved_in = saved_in; a.saved_out = saved_out;
    a.q_out = q_out; a.k_pool = k_pool; a.v_pool = v_pool; a.row_slot = (const int*)row_slot; a.row_pos = (const int*)row_pos;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.page_tokens = page_tokens; a.num_pages = num_pages;
    a.seqs = (const int*)seqs; a.n_seqs = n_seqs; a.rows = rows; a.group = rows >= 1024 ? 4 : 1; a.status = (uint32_t*)status;
    if (conv_w != nullptr) return f32 ? launch_heads<float, true>(a, stream) : launch_heads<__nv_bfloat16, true>(a, stream);
    return f32 ? launch_heads<float, false>(a, stream) : launch_heads<__nv_bfloat16, false>(a, stream);
}
