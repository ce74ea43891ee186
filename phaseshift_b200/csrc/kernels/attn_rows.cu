// Key (and value) append without rotation, and per-row attention for any head size in bf16 or 32-bit.
//
// ps_attn_append copies the query columns of a projection row to the dense query buffer and its key and value columns to their
// page.  ps_attn_rows is the plain form of the attention (with the options of attn_options.cuh) that paged_attention.cu and
// attn_prefill*.cu serve for bf16 pools and head sizes up to 256: one CTA per (row, query head), scores and softmax in
// 32-bit.  The 32-bit engines run on it, and head sizes that the tiled kernels do not take.
#include "attn_options.cuh"
#include "ps_common.cuh"

namespace ps {

struct AttnAppendArgs {
    const uint4* proj; int ld16;                 // row pitch in 16-byte units
    int q16, head16, Hkv;                        // 16-byte units of the query columns and of one key head
    uint4* q_out; uint4* k_pool; uint4* v_pool;   // v_pool null: the keys are the values
    const int* row_slot; const int* row_pos; const int* block_table; int max_blocks, page_tokens, num_pages;
    uint32_t* status;
};

__global__ void attn_append_kernel(const AttnAppendArgs a) {
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int row = blockIdx.x;
    const uint4* src = a.proj + (size_t)row * a.ld16;
    for (int i = threadIdx.x; i < a.q16; i += blockDim.x) a.q_out[(size_t)row * a.q16 + i] = src[i];
    if (a.Hkv == 0) return;                      // the layer reads another one's keys
    const int slot = a.row_slot[row], pos = a.row_pos[row];
    if (slot < 0 || pos < 0) return;             // padding row
    const int blk = pos / a.page_tokens, off = pos % a.page_tokens;
    const int page = blk < a.max_blocks ? a.block_table[(size_t)slot * a.max_blocks + blk] : -1;
    if (page < 0 || page >= a.num_pages) { if (threadIdx.x == 0) set_status(a.status, PS_DEV_BAD_INDEX); return; }
    for (int i = threadIdx.x; i < a.Hkv * a.head16; i += blockDim.x) {
        const int head = i / a.head16, c = i % a.head16;
        const size_t at = (((size_t)page * a.Hkv + head) * a.page_tokens + off) * a.head16 + c;
        a.k_pool[at] = src[a.q16 + i];
        if (a.v_pool != nullptr) a.v_pool[at] = src[a.q16 + a.Hkv * a.head16 + i];
    }
}

template <typename T> __device__ __forceinline__ T ar_cast(float v);
template <> __device__ __forceinline__ float ar_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ar_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

struct AttnRowsArgs {
    const void* q; const void* k_pool; const void* v_pool;
    const int* block_table; int max_blocks, page_tokens, num_pages;
    const int* row_slot; const int* row_pos;
    int Hq, Hkv, D; float scale; AttnOptions opt;
    const void* gate; int ld_gate, gate_head_stride, gate_offset;    // optional sigmoid gate
    void* out; uint32_t* status;
};

constexpr int kArThreads = 128, kArTile = 128, kArMaxD = 2048;

// grid = (Hq, rows)
template <typename T>
__global__ void __launch_bounds__(kArThreads) attn_rows_kernel(const AttnRowsArgs a) {
    __shared__ float s_q[kArMaxD], s_o[kArMaxD], s_p[kArTile], red[32];
    __shared__ int s_page[kArTile];
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int h = blockIdx.x, row = blockIdx.y, D = a.D, t = threadIdx.x, warp = t >> 5, lane = t & 31;
    const int pos = a.row_pos[row], slot = a.row_slot[row];
    T* out = reinterpret_cast<T*>(a.out) + ((size_t)row * a.Hq + h) * D;
    if (pos < 0 || slot < 0) {                                       // padding row
        for (int d = t; d < D; d += kArThreads) out[d] = ar_cast<T>(0.f);
        return;
    }
    const int kvh = h / (a.Hq / a.Hkv);
    for (int d = t; d < D; d += kArThreads) {
        s_q[d] = (float)reinterpret_cast<const T*>(a.q)[((size_t)row * a.Hq + h) * D + d];
        s_o[d] = 0.f;
    }
    const int lo = attn_first(a.opt, pos);
    const float scale = a.scale * attn_temperature(a.opt, pos);
    float m = a.opt.sink != nullptr ? a.opt.sink[h] : -3.0e38f;
    float l = a.opt.sink != nullptr ? 1.f : 0.f;
    // the kept first positions, then the run up to the query itself
    const int kept = min(a.opt.keep_first, lo);
    for (int t0 = kept > 0 ? 0 : lo, t1; t0 <= pos; t0 = t1) {
        const int end = t0 < kept ? kept : pos + 1, n = min(kArTile, end - t0);
        t1 = t0 + n == kept ? lo : t0 + n;
        __syncthreads();
        if (t < n) {
            const int tok = t0 + t, page = a.block_table[(size_t)slot * a.max_blocks + tok / a.page_tokens];
            const bool ok = page >= 0 && page < a.num_pages;
            if (!ok) set_status(a.status, PS_DEV_BAD_INDEX);
            s_page[t] = ok ? page : -1;
        }
        __syncthreads();
        for (int j = warp; j < n; j += kArThreads / 32) {            // a warp per key
            float s = 0.f;
            if (s_page[j] >= 0) {
                const T* k = reinterpret_cast<const T*>(a.k_pool) + (((size_t)s_page[j] * a.Hkv + kvh) * a.page_tokens + (t0 + j) % a.page_tokens) * D;
                for (int d = lane; d < D; d += 32) s = fmaf(s_q[d], (float)k[d], s);
            }
            s = warp_sum(s);
            if (lane == 0) s_p[j] = s_page[j] >= 0 ? fmaf(s, scale, attn_bias(a.opt, h, pos - t0 - j)) : -INFINITY;
        }
        __syncthreads();
        const float s = t < n ? s_p[t] : -INFINITY;
        const float m_new = fmaxf(m, block_max(s, red));
        const float p = t < n ? expf(s - m_new) : 0.f;
        const float alpha = expf(m - m_new);
        const float sum = block_sum(p, red);
        l = l * alpha + sum;
        m = m_new;
        s_p[t] = p;
        __syncthreads();
        for (int d = t; d < D; d += kArThreads) {
            float o = s_o[d] * alpha;
            for (int j = 0; j < n; ++j) {
                if (s_page[j] < 0) continue;
                const T* v = reinterpret_cast<const T*>(a.v_pool) + (((size_t)s_page[j] * a.Hkv + kvh) * a.page_tokens + (t0 + j) % a.page_tokens) * D;
                o = fmaf(s_p[j], (float)v[d], o);
            }
            s_o[d] = o;
        }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const T* gate = a.gate == nullptr ? nullptr
                                      : reinterpret_cast<const T*>(a.gate) + (size_t)row * a.ld_gate + (size_t)h * a.gate_head_stride + a.gate_offset;
    for (int d = t; d < D; d += kArThreads) {
        float o = s_o[d] * inv;
        if (gate != nullptr) o *= 1.f / (1.f + expf(-(float)gate[a.opt.gate_per_head ? 0 : d]));
        out[d] = ar_cast<T>(o);
    }
}

}  // namespace ps

// proj: rows of [Hq * D queries | Hkv * D keys (| Hkv * D values, with a value pool) | ...] of `esz`-byte elements; D * esz a
// multiple of 16.  Hkv 0: nothing is appended.
PS_API int ps_attn_append(const void* proj, int ld, int esz, int rows, int Hq, int Hkv, int D, const void* row_slot, const void* row_pos,
                          void* q_out, void* k_pool, void* v_pool, const void* block_table, int max_blocks, int page_tokens, int num_pages,
                          void* status, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || Hkv < 0 || (D * esz) % 16 || ((size_t)ld * esz) % 16 ||
        ((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool) % 16)
        return (int)cudaErrorInvalidValue;
    AttnAppendArgs a;
    a.proj = (const uint4*)proj; a.ld16 = (int)((size_t)ld * esz / 16); a.head16 = D * esz / 16; a.q16 = Hq * a.head16; a.Hkv = Hkv;
    a.q_out = (uint4*)q_out; a.k_pool = (uint4*)k_pool; a.v_pool = (uint4*)v_pool; a.row_slot = (const int*)row_slot;
    a.row_pos = (const int*)row_pos; a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.page_tokens = page_tokens;
    a.num_pages = num_pages; a.status = (uint32_t*)status;
    return launch_pdl(attn_append_kernel, dim3(rows), dim3(256), 0, stream, a);
}

// `options`: an AttnOptions or null.  The gate has the pools' element type.
PS_API int ps_attn_rows(const void* q, const void* k_pool, const void* v_pool, int f32, const void* block_table, int max_blocks,
                        int page_tokens, int num_pages, const void* row_slot, const void* row_pos, int rows, int Hq, int Hkv, int D,
                        float scale, const void* options, const void* gate, int ld_gate, int gate_head_stride, int gate_offset,
                        void* out, void* status, cudaStream_t stream) {
    using namespace ps;
    const AttnOptions opt = attn_options(options);
    if (rows <= 0 || rows > 65535 || Hkv <= 0 || (Hq % Hkv) || D <= 0 || D > kArMaxD || !attn_options_ok(opt)) return (int)cudaErrorInvalidValue;
    AttnRowsArgs a;
    a.q = q; a.k_pool = k_pool; a.v_pool = v_pool; a.block_table = (const int*)block_table; a.max_blocks = max_blocks;
    a.page_tokens = page_tokens; a.num_pages = num_pages; a.row_slot = (const int*)row_slot; a.row_pos = (const int*)row_pos;
    a.Hq = Hq; a.Hkv = Hkv; a.D = D; a.scale = scale; a.opt = opt; a.gate = gate; a.ld_gate = ld_gate;
    a.gate_head_stride = gate_head_stride; a.gate_offset = gate_offset; a.out = out; a.status = (uint32_t*)status;
    if (f32) return launch_pdl(attn_rows_kernel<float>, dim3(Hq, rows), dim3(kArThreads), 0, stream, a);
    return launch_pdl(attn_rows_kernel<__nv_bfloat16>, dim3(Hq, rows), dim3(kArThreads), 0, stream, a);
}
