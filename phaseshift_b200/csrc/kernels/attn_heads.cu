// From a projection row [q heads | k heads | v heads] to an attention's queries, keys and values, in one launch: a short causal
// convolution over time on every channel, a norm of the queries and of the keys over all heads at once, rotation of the first
// dimensions of every query and key head, division of a head by its root mean square, mixing with another layer's values, and the
// append to the pages.  Every part is optional (HeadsSpec in ops/specs.py); all of it is computed in 32-bit.
//
// The convolution's history is state: [slots, taps - 1, channels], the projected row of position p in row p % (taps - 1).  A row
// whose predecessors lie in the same step reads them from the projection; the first taps - 1 rows of a sequence's portion look
// into the history.  Those have CTAs of their own, and the last of a sequence's to finish (a ticket, no waiting) stores the
// portion's last rows, so that nobody reads a row of the history that another CTA has replaced.
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
    const int* seqs; int n_seqs, rows;
    int* tickets;                                // [n_seqs], zero between launches
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
// Eight elements as they lie in memory, widened where they are used.
template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> {
    uint4 v;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ float4 half(int i) const {
        const float2 a = bf16x2_bits_to_f32x2(i ? v.z : v.x), b = bf16x2_bits_to_f32x2(i ? v.w : v.y);
        return make_float4(a.x, a.y, b.x, b.y);
    }
};
template <> struct Raw8<float> {
    float4 v[2];
    __device__ __forceinline__ void load(const float* p) { v[0] = reinterpret_cast<const float4*>(p)[0]; v[1] = reinterpret_cast<const float4*>(p)[1]; }
    __device__ __forceinline__ float4 half(int i) const { return v[i]; }
};
__device__ __forceinline__ float4 ah_fma4(float4 a, float4 b, float4 c) {
    return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
template <typename T> __device__ __forceinline__ T ah_cast(float v);
template <> __device__ __forceinline__ float ah_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ah_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

__device__ __forceinline__ void ah_prefetch(const void* p, size_t bytes) {
    for (size_t i = (size_t)threadIdx.x * 128; i < bytes; i += (size_t)blockDim.x * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(p) + i));
}

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
    const int blk = pos / a.page_tokens, off = pos % a.page_tokens;
    const int page = blk < a.max_blocks ? a.block_table[(size_t)slot * a.max_blocks + blk] : -1;
    const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld;
    const T* w = reinterpret_cast<const T*>(a.conv_w);
    const T* hist = reinterpret_cast<const T*>(a.history) + (size_t)slot * (a.taps - 1) * C;
    float ss[2] = {0.f, 0.f};
    auto put = [&](int c, float4 x) {                                // a finished channel group
        const float sq = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
        if (c < HD) ss[0] += sq;
        else if (c < KD) ss[1] += sq;
        if (a.q_norm != nullptr && c < KD) {                         // (the norms' factors follow in the second pass: a turn is linear)
            const float4 nw = ah_load4(c < HD ? a.q_norm + c : a.k_norm + c - HD);
            x = make_float4(x.x * nw.x, x.y * nw.y, x.z * nw.z, x.w * nw.w);
        }
        *reinterpret_cast<float4*>(sx + c) = x;
    };
    if constexpr (CONV) {
        for (int j0 = 0; j0 < a.taps; j0 += 4) {                     // four taps at a time, their loads in flight together
            const T* u[4];
            const T* wt = w + (size_t)(a.taps - 1 - j0) * C;
            const int m = min(4, min(a.taps, pos + 1) - j0);         // (zeros before the sequence's start)
            const bool last = j0 + 4 >= a.taps;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = j0 + e;
                u[e] = e >= m ? src : j <= back ? src - (size_t)j * a.ld : hist + (size_t)((pos - j) % (a.taps - 1)) * C;
            }
            for (int c = 8 * t; c < C; c += 8 * n) {
                Raw8<T> uu[4], ww[4];
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (e < m) { uu[e].load(u[e] + c); ww[e].load(wt - (size_t)e * C + c); }
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    float4 x = j0 > 0 ? *reinterpret_cast<const float4*>(sx + c + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (e < m) x = ah_fma4(uu[e].half(i), ww[e].half(i), x);
                    if (last) put(c + 4 * i, x);
                    else *reinterpret_cast<float4*>(sx + c + 4 * i) = x;
                }
            }
        }
    } else {
#pragma unroll 4
        for (int c = 8 * t; c < C; c += 8 * n) {
            Raw8<T> x;
            x.load(src + c);
            put(c, x.half(0));
            put(c + 4, x.half(1));
        }
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
    const bool mapped = page >= 0 && page < a.num_pages;
    if (!mapped && t == 0) set_status(a.status, PS_DEV_BAD_INDEX);
    const bool quads = a.pairs % 4 == 0 && a.halves;                 // a group of four lies in one half
    const int heads_on = 4 * n / D, dims_on = 4 * n % D;             // from one of a thread's groups to its next
    for (int c = 4 * t, head = c / D, d = c % D; c < C; c += 4 * n, head += heads_on, d += dims_on, head += d >= D, d -= d >= D ? D : 0) {
        float4 o = *reinterpret_cast<const float4*>(sx + c);
        if (c < KD) {
            if (d >= 2 * a.pairs) {
            } else if (quads) {
                const bool low = d < a.pairs;
                const float4 u = *reinterpret_cast<const float4*>(sx + (low ? c + a.pairs : c - a.pairs));
                const int i = low ? d : d - a.pairs;
                const float4 s = *reinterpret_cast<const float4*>(s_sin + i), k = *reinterpret_cast<const float4*>(s_cos + i);
                const float m = low ? -1.f : 1.f;
                o = make_float4(o.x * k.x + m * u.x * s.x, o.y * k.y + m * u.y * s.y, o.z * k.z + m * u.z * s.z, o.w * k.w + m * u.w * s.w);
            } else if (a.halves) {
                float v[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int de = d + e;
                    if (de < a.pairs) v[e] = v[e] * s_cos[de] - sx[c + e + a.pairs] * s_sin[de];
                    else if (de < 2 * a.pairs) v[e] = v[e] * s_cos[de - a.pairs] + sx[c + e - a.pairs] * s_sin[de - a.pairs];
                }
                o = make_float4(v[0], v[1], v[2], v[3]);
            } else {
                const int i = d >> 1;
                o = make_float4(o.x * s_cos[i] - o.y * s_sin[i], o.y * s_cos[i] + o.x * s_sin[i], o.z, o.w);
                if (i + 1 < a.pairs) {
                    const float z = o.z;
                    o.z = z * s_cos[i + 1] - o.w * s_sin[i + 1]; o.w = o.w * s_cos[i + 1] + z * s_sin[i + 1];
                }
            }
            const float f = (c < HD ? norm[0] : norm[1]) * (a.unit ? s_inv[head] : 1.f);
            o = make_float4(o.x * f, o.y * f, o.z * f, o.w * f);
        } else if (a.saved_out != nullptr || a.saved_in != nullptr) {
            const size_t at = (size_t)row * a.G * a.vdim + (size_t)(head - a.H - a.G) * a.vdim + d;
            if (a.vdim % 4 == 0) {
                if (d < a.vdim) {
                    if (a.saved_out != nullptr) ah_store4(reinterpret_cast<T*>(a.saved_out) + at, o);
                    if (a.saved_in != nullptr) {
                        const float4 u = ah_load4(reinterpret_cast<const T*>(a.saved_in) + at);
                        const float m = a.mix, r = 1.f - a.mix;
                        o = make_float4(r * o.x + m * u.x, r * o.y + m * u.y, r * o.z + m * u.z, r * o.w + m * u.w);
                    }
                }
            } else {
                float v[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    if (d + e >= a.vdim) continue;
                    if (a.saved_out != nullptr) reinterpret_cast<T*>(a.saved_out)[at + e] = ah_cast<T>(v[e]);
                    if (a.saved_in != nullptr) v[e] = (1.f - a.mix) * v[e] + a.mix * (float)reinterpret_cast<const T*>(a.saved_in)[at + e];
                }
                o = make_float4(v[0], v[1], v[2], v[3]);
            }
        }
        if (c < HD) ah_store4(q_out + c, o);
        else if (mapped) {
            const int kvh = c < KD ? head - a.H : head - a.H - a.G;
            T* pool = reinterpret_cast<T*>(c < KD ? a.k_pool : a.v_pool);
            ah_store4(pool + (((size_t)page * a.G + kvh) * a.page_tokens + off) * D + d, o);
        }
    }
}

// grid: (CONV: n_seqs * (taps - 1) CTAs for the first rows of the sequences' portions) + rows
template <typename T, bool CONV>
__global__ void __launch_bounds__(1024) attn_heads_kernel(const AttnHeadsArgs a) {
    extern __shared__ __align__(16) float sx[];
    __shared__ float red[64];
    const int C = (a.H + 2 * a.G) * a.D;
    const int pairs4 = (a.pairs + 3) / 4 * 4;
    float* s_sin = sx + C;
    float* s_cos = s_sin + pairs4;
    float* s_inv = s_cos + pairs4;
    // the layer's constants towards L2 while the projection drains
    if (a.rows <= 64) {
        ah_prefetch(a.freq, (size_t)a.pairs * 8);
        if (CONV) ah_prefetch(a.conv_w, (size_t)a.taps * C * sizeof(T));
        if (a.q_norm != nullptr) { ah_prefetch(a.q_norm, (size_t)a.H * a.D * 4); ah_prefetch(a.k_norm, (size_t)a.G * a.D * 4); }
    }
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int hist_rows = CONV ? a.taps - 1 : 0;
    int block = blockIdx.x;
    if (CONV) {
        if (block < a.n_seqs * hist_rows) {
            const int seq = block / hist_rows, r = block % hist_rows;
            const int* sd = a.seqs + 4 * seq;
            const int row0 = sd[0], n_rows = sd[1], slot = sd[2], pos0 = sd[3], mine = min(n_rows, hist_rows);
            if (r >= mine || slot < 0) return;
            heads_row<T, CONV>(a, row0 + r, r, sx, s_sin, s_cos, s_inv, red);
            if (mine > 1) {
                __shared__ int s_last;
                __syncthreads();
                if (threadIdx.x == 0) {
                    __threadfence();
                    s_last = atomicAdd(&a.tickets[seq], 1) == mine - 1;
                    if (s_last) { a.tickets[seq] = 0; __threadfence(); }
                }
                __syncthreads();
                if (!s_last) return;
            }
            T* hist = reinterpret_cast<T*>(a.history) + (size_t)slot * hist_rows * C;
            for (int r0 = max(0, n_rows - hist_rows); r0 < n_rows; r0 += 4)
                for (int c = 4 * (int)threadIdx.x; c < C; c += 4 * blockDim.x) {
                    float4 x[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (r0 + e < n_rows) x[e] = ah_load4(reinterpret_cast<const T*>(a.proj) + (size_t)(row0 + r0 + e) * a.ld + c);
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (r0 + e < n_rows) ah_store4(hist + (size_t)((pos0 + r0 + e) % hist_rows) * C + c, x[e]);
                }
            return;
        }
        block -= a.n_seqs * hist_rows;
    }
    const int row = block;
    // (a step's rows of one sequence follow one another, and no two of its sequences share a slot)
    if (CONV && hist_rows > 0 && a.row_slot[row] >= 0 && (row < hist_rows || a.row_slot[row - hist_rows] != a.row_slot[row])) return;
    heads_row<T, CONV>(a, row, a.taps, sx, s_sin, s_cos, s_inv, red);
}

template <typename T, bool CONV>
static int launch_heads(const AttnHeadsArgs& a, cudaStream_t stream) {
    const size_t smem = sizeof(float) * ((size_t)(a.H + 2 * a.G) * a.D + 2 * (a.pairs + 3) + a.H + a.G);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(attn_heads_kernel<T, CONV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        set = true;
    }
    const int blocks = (CONV ? a.n_seqs * (a.taps - 1) : 0) + a.rows;
    return launch_pdl(attn_heads_kernel<T, CONV>, dim3(blocks), dim3(a.rows <= 64 ? 1024 : 256), smem, stream, a);
}

}  // namespace ps

// `tickets` ([n_seqs] ints, zero, left zero): for convolutions of more than two taps.  `f32`: projection, history, saved values, queries and pools are fp32 instead of bf16.  D and `ld` multiples of 8.
PS_API int ps_attn_heads(const void* proj, int ld, int f32, int rows, int H, int G, int D, int dim, int vdim, int pairs, int halves,
                         int unit, float eps, float turn_size, const void* freq, const void* q_norm, const void* k_norm, int taps,
                         const void* conv_w, void* history, float mix, const void* saved_in, void* saved_out, void* q_out, void* k_pool,
                         void* v_pool, const void* row_slot, const void* row_pos, const void* block_table, int max_blocks,
                         int page_tokens, int num_pages, const void* seqs, int n_seqs, void* tickets, void* status, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || H <= 0 || G <= 0 || D % 8 || ld % 8 || dim > D || vdim > D || 2 * pairs > dim || taps < 1 || (taps > 1 && (conv_w == nullptr || history == nullptr)) ||
        (conv_w != nullptr && n_seqs <= 0) || (taps > 2 && tickets == nullptr) || (q_norm == nullptr) != (k_norm == nullptr) ||
        ((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)history | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)q_norm |
         (uintptr_t)k_norm | (uintptr_t)saved_in | (uintptr_t)saved_out) % 16)
        return (int)cudaErrorInvalidValue;
    AttnHeadsArgs a;
    a.proj = proj; a.ld = ld; a.H = H; a.G = G; a.D = D; a.dim = dim; a.vdim = vdim; a.pairs = pairs; a.halves = halves; a.unit = unit;
    a.taps = taps; a.eps = eps; a.turn_size = turn_size; a.freq = (const double*)freq; a.q_norm = (const float*)q_norm;
    a.k_norm = (const float*)k_norm; a.conv_w = conv_w; a.history = history; a.mix = mix; a.saved_in = saved_in; a.saved_out = saved_out;
    a.q_out = q_out; a.k_pool = k_pool; a.v_pool = v_pool; a.row_slot = (const int*)row_slot; a.row_pos = (const int*)row_pos;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.page_tokens = page_tokens; a.num_pages = num_pages;
    a.seqs = (const int*)seqs; a.n_seqs = n_seqs; a.rows = rows; a.tickets = (int*)tickets; a.status = (uint32_t*)status;
    if (conv_w != nullptr) return f32 ? launch_heads<float, true>(a, stream) : launch_heads<__nv_bfloat16, true>(a, stream);
    return f32 ? launch_heads<float, false>(a, stream) : launch_heads<__nv_bfloat16, false>(a, stream);
}
