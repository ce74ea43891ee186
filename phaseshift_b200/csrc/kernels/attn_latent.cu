// Latent attention around its core: latents to the cache, rotation of query parts, and prefill-sized steps over expanded keys
// and values.
//
// A cached row is [latent | rotated key part] (one "head" of the paged pool).  ps_latent_down norms both latents of a projection
// row, turns the shared key part and appends.  ps_latent_turn turns the rotated query parts.  For many rows, keys and values per
// head are products of the latent: ps_latent_gather brings the tokens that the step's long sequences see from their pages into
// consecutive rows, one GEMM expands them, and ps_latent_prefill attends over the result on the tensor cores (attn_tc.cuh).
// Rows of short sequences attend in the latent space instead (attn_latent_decode.cu).
#include "attn_tc.cuh"
#include "turn_angle.cuh"

namespace ps {

template <typename T> __device__ __forceinline__ T la_cast(float v);
template <> __device__ __forceinline__ float la_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 la_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }

struct LatentDownArgs {
    const void* proj; int ld;                    // rows of [query latent: QR | latent: KR | rotated part: R | ...]
    int QR, KR, R, q_true, kv_true, pairs;       // engine sizes, the sizes the norms divide by, pairs that turn
    const float* q_norm; const float* kv_norm; float eps; const double* inv_freq;
    void* cq; void* pool;                        // [rows, QR]; [pages, page_tokens, KR + R]
    const int* row_slot; const int* row_pos; const int* block_table; int max_blocks, page_tokens, num_pages;
    uint32_t* status;
};

// four elements at once (16- or 8-byte accesses)
__device__ __forceinline__ float4 la_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 la_load4(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf16x2_bits_to_f32x2(v.x), b = bf16x2_bits_to_f32x2(v.y);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void la_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void la_store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(f32x2_to_bf16x2_bits(v.x, v.y), f32x2_to_bf16x2_bits(v.z, v.w));
}
__device__ __forceinline__ float la_sq4(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }
__device__ __forceinline__ float4 la_scale4(float4 v, float s, float4 w) { return make_float4(v.x * s * w.x, v.y * s * w.y, v.z * s * w.z, v.w * s * w.w); }

// one CTA per row; QR, KR, R and the row pitch are multiples of 4
template <typename T>
__global__ void __launch_bounds__(256) latent_down_kernel(const LatentDownArgs a) {
    __shared__ float red[64];
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int row = blockIdx.x, t = threadIdx.x, n = blockDim.x;
    const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld;
    const T* lat = src + a.QR;
    const T* rot = lat + a.KR;
    const int slot = a.row_slot[row], pos = a.row_pos[row], blk = pos / a.page_tokens;
    const bool real = slot >= 0 && pos >= 0;                                      // (not a padding row)
    const int page = real && blk < a.max_blocks ? a.block_table[(size_t)slot * a.max_blocks + blk] : -1;
    float ss[2] = {0.f, 0.f};
    for (int i = 4 * t; i < a.QR; i += 4 * n) ss[0] += la_sq4(la_load4(src + i));
    for (int i = 4 * t; i < a.KR; i += 4 * n) ss[1] += la_sq4(la_load4(lat + i));
    block_sum_n<2>(ss, red);
    const float iq = rsqrtf(ss[0] / (float)a.q_true + a.eps), ik = rsqrtf(ss[1] / (float)a.kv_true + a.eps);
    T* cq = reinterpret_cast<T*>(a.cq) + (size_t)row * a.QR;
    for (int i = 4 * t; i < a.QR; i += 4 * n) la_store4(cq + i, la_scale4(la_load4(src + i), iq, *reinterpret_cast<const float4*>(a.q_norm + i)));
    if (!real) return;
    if (page < 0 || page >= a.num_pages) { if (t == 0) set_status(a.status, PS_DEV_BAD_INDEX); return; }
    T* dst = reinterpret_cast<T*>(a.pool) + ((size_t)page * a.page_tokens + pos % a.page_tokens) * (a.KR + a.R);
    for (int i = 4 * t; i < a.KR; i += 4 * n) la_store4(dst + i, la_scale4(la_load4(lat + i), ik, *reinterpret_cast<const float4*>(a.kv_norm + i)));
    for (int i = n - 1 - t; i < a.R / 2; i += n) {                                // from the last thread on: the first ones have the latents
        float u = (float)rot[2 * i], v = (float)rot[2 * i + 1];
        if (i < a.pairs) {
            float s, c;
            turn_angle(pos, a.inv_freq[i], &s, &c);
            const float w = u * c - v * s;
            v = v * c + u * s; u = w;
        }
        dst[a.KR + 2 * i] = la_cast<T>(u); dst[a.KR + 2 * i + 1] = la_cast<T>(v);
    }
}

struct LatentTurnArgs {
    const void* q; int ld, head, off;            // row pitch, head pitch, offset of the rotated part in a head (elements)
    void* out; int ldo, ohead, ooff;
    int H, R, pairs; const double* inv_freq; const int* row_pos;
};

// one CTA per row; `out` may be `q` itself
template <typename T>
__global__ void __launch_bounds__(256) latent_turn_kernel(const LatentTurnArgs a) {
    __shared__ float s_sin[256], s_cos[256];
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int row = blockIdx.x, half = a.R / 2, pos = max(a.row_pos[row], 0);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float s = 0.f, c = 1.f;
        if (i < a.pairs) turn_angle(pos, a.inv_freq[i], &s, &c);
        s_sin[i] = s; s_cos[i] = c;
    }
    __syncthreads();
    const int quads = half / 2;                                                   // two pairs at once
    for (int i = threadIdx.x; i < a.H * quads; i += blockDim.x) {
        const int h = i / quads, j = 2 * (i % quads);
        const float4 x = la_load4(reinterpret_cast<const T*>(a.q) + (size_t)row * a.ld + (size_t)h * a.head + a.off + 2 * j);
        la_store4(reinterpret_cast<T*>(a.out) + (size_t)row * a.ldo + (size_t)h * a.ohead + a.ooff + 2 * j,
                  make_float4(x.x * s_cos[j] - x.y * s_sin[j], x.y * s_cos[j] + x.x * s_sin[j],
                              x.z * s_cos[j + 1] - x.w * s_sin[j + 1], x.w * s_cos[j + 1] + x.z * s_sin[j + 1]));
    }
}

struct LatentGatherArgs {
    const uint4* pool; int row16, lat16;         // 16-byte units of a cached row and of its latent
    const int* block_table; int max_blocks, page_tokens, num_pages;
    const int* seqs; int n_seqs, min_rows; AttnOptions opt;
    uint4* lat; uint4* rot;                      // [rows, KR], [rows, R]
    uint32_t* status;
};

// one warp per gathered row; rows behind a sequence's last token become zero
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherArgs a) {
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    int at = 0, s = 0;
    for (; s < a.n_seqs; ++s) {
        const int n = expanded_rows(a.seqs + 4 * s, a.min_rows, a.opt);
        if (r < at + n) break;
        at += n;
    }
    if (s >= a.n_seqs) return;
    const int* sd = a.seqs + 4 * s;
    const int tok = expanded_first(sd, a.opt) + r - at;
    int page = -1;
    if (tok < sd[3] + sd[1]) {
        page = a.block_table[(size_t)sd[2] * a.max_blocks + tok / a.page_tokens];
        if (page < 0 || page >= a.num_pages) { if (lane == 0) set_status(a.status, PS_DEV_BAD_INDEX); page = -1; }
    }
    const uint4* src = a.pool + ((size_t)max(page, 0) * a.page_tokens + tok % a.page_tokens) * a.row16;
    const int rot16 = a.row16 - a.lat16;
    for (int i = lane; i < a.row16; i += 32) {
        const uint4 v = page >= 0 ? src[i] : make_uint4(0, 0, 0, 0);
        if (i < a.lat16) a.lat[(size_t)r * a.lat16 + i] = v;
        else a.rot[(size_t)r * rot16 + i - a.lat16] = v;
    }
}

template <int DK>
static int launch_latent_prefill(int DV, dim3 grid, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mr,
                                 const AttnTcArgs& a, cudaStream_t stream) {
    switch (DV) {
        case 64: return launch_attn_tc<DK, 64, false, false, false, true>(grid, mq, mk, mv, mr, a, stream);
        case 128: return launch_attn_tc<DK, 128, false, false, false, true>(grid, mq, mk, mv, mr, a, stream);
        case 192: return launch_attn_tc<DK, 192, false, false, false, true>(grid, mq, mk, mv, mr, a, stream);
        case 256: return launch_attn_tc<DK, 256, false, false, false, true>(grid, mq, mk, mv, mr, a, stream);
        default: return (int)cudaErrorInvalidValue;
    }
}

}  // namespace ps

PS_API int ps_latent_down(const void* proj, int ld, int f32, int rows, int QR, int KR, int R, int q_true, int kv_true, int pairs,
                          const void* q_norm, const void* kv_norm, float eps, const void* inv_freq, void* cq, void* pool,
                          const void* row_slot, const void* row_pos, const void* block_table, int max_blocks, int page_tokens,
                          int num_pages, void* status, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || QR <= 0 || KR <= 0 || R < 0 || ((QR | KR | R | ld) & 3) || 2 * pairs > R || q_true <= 0 || kv_true <= 0 || ld < QR + KR + R ||
        (((uintptr_t)proj | (uintptr_t)cq | (uintptr_t)pool | (uintptr_t)q_norm | (uintptr_t)kv_norm) % 16))
        return (int)cudaErrorInvalidValue;
    LatentDownArgs a;
    a.proj = proj; a.ld = ld; a.QR = QR; a.KR = KR; a.R = R; a.q_true = q_true; a.kv_true = kv_true; a.pairs = pairs;
    a.q_norm = (const float*)q_norm; a.kv_norm = (const float*)kv_norm; a.eps = eps; a.inv_freq = (const double*)inv_freq;
    a.cq = cq; a.pool = pool; a.row_slot = (const int*)row_slot; a.row_pos = (const int*)row_pos; a.block_table = (const int*)block_table;
    a.max_blocks = max_blocks; a.page_tokens = page_tokens; a.num_pages = num_pages; a.status = (uint32_t*)status;
    return f32 ? launch_pdl(latent_down_kernel<float>, dim3(rows), dim3(256), 0, stream, a)
               : launch_pdl(latent_down_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, a);
}

// Rotated parts (R columns at `off` of every head) of rows of H heads, from `q` to `out` (its own layout; may be the same).
PS_API int ps_latent_turn(const void* q, int ld, int head, int off, void* out, int ldo, int ohead, int ooff, int f32, int rows, int H, int R,
                          int pairs, const void* inv_freq, const void* row_pos, cudaStream_t stream) {
    using namespace ps;
    if (rows <= 0 || H <= 0 || R <= 0 || R > 512 || 2 * pairs > R || ((R | ld | head | off | ldo | ohead | ooff) & 3) ||
        (((uintptr_t)q | (uintptr_t)out) % 16))
        return (int)cudaErrorInvalidValue;
    LatentTurnArgs a;
    a.q = q; a.ld = ld; a.head = head; a.off = off; a.out = out; a.ldo = ldo; a.ohead = ohead; a.ooff = ooff; a.H = H; a.R = R;
    a.pairs = pairs; a.inv_freq = (const double*)inv_freq; a.row_pos = (const int*)row_pos;
    return f32 ? launch_pdl(latent_turn_kernel<float>, dim3(rows), dim3(256), 0, stream, a)
               : launch_pdl(latent_turn_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, stream, a);
}

// Tokens per tile of the expanded rows: a sequence's first gathered token is a multiple of it, and so is its number of rows.
PS_API int ps_latent_tile(void) { return ps::kTcTok; }

// bf16 pool [pages, page_tokens, KR + R]; `rows` gathered rows in all (of sequences with more than `min_rows` rows in the step).
PS_API int ps_latent_gather(const void* pool, int KR, int R, const void* block_table, int max_blocks, int page_tokens, int num_pages,
                            const void* seqs, int n_seqs, int min_rows, const void* options, int rows, void* lat, void* rot, void* status,
                            cudaStream_t stream) {
    using namespace ps;
    const AttnOptions opt = attn_options(options);
    if (rows <= 0 || rows % kTcTok || n_seqs <= 0 || KR % 8 || R % 8 || !attn_options_ok(opt) || opt.keep_first > 0) return (int)cudaErrorInvalidValue;
    LatentGatherArgs a;
    a.pool = (const uint4*)pool; a.row16 = (KR + R) / 8; a.lat16 = KR / 8; a.block_table = (const int*)block_table; a.max_blocks = max_blocks;
    a.page_tokens = page_tokens; a.num_pages = num_pages; a.seqs = (const int*)seqs; a.n_seqs = n_seqs; a.min_rows = min_rows; a.opt = opt;
    a.lat = (uint4*)lat; a.rot = (uint4*)rot; a.status = (uint32_t*)status;
    return launch_pdl(latent_gather_kernel, dim3(rows / 8), dim3(256), 0, stream, a);
}

// Whether the expanded form has a kernel for heads of `dim` + R query / key columns and `vdim` value columns.
PS_API int ps_latent_prefill_ok(int dim, int R, int vdim) {
    return dim > 0 && R > 0 && dim % 64 == 0 && R % 64 == 0 && dim + R <= 256 && vdim % 64 == 0 && vdim >= 64 && vdim <= 256;
}

// q [q_rows, H * (dim + R)] (rotated parts turned); `kv` [rows, H * dim | H * vdim] and `rot` [rows, R] as gathered and expanded;
// out [q_rows, H * vdim].  `max_seq_rows` bounds the rows of a sequence; gate elementwise.
PS_API int ps_latent_prefill(const void* q, int q_rows, const void* kv, const void* rot, int rows, const void* seqs, int n_seqs,
                             int max_seq_rows, int min_rows, int H, int dim, int R, int vdim, float scale, const void* options,
                             const void* gate, int ld_gate, int gate_head_stride, int gate_offset, void* out, void* status,
                             cudaStream_t stream) {
    using namespace ps;
    const AttnOptions opt = attn_options(options);
    if (!ps_latent_prefill_ok(dim, R, vdim) || q_rows <= 0 || rows <= 0 || n_seqs <= 0 || max_seq_rows <= 0 || H <= 0 || H > 65535 ||
        !attn_options_ok(opt) || opt.keep_first > 0 || attn_transforms_scores(opt) || (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)rot) % 16) ||
        (gate != nullptr && (opt.gate_per_head || ((uintptr_t)gate % 16) || ld_gate % 8 || gate_head_stride % 8 || gate_offset % 8)))
        return (int)cudaErrorInvalidValue;
    const int DK = dim + R;
    const uint64_t ldk = (uint64_t)H * (dim + vdim);
    CUtensorMap mq, mk, mr;
    int err = attn_map_2d(&mq, q, (uint64_t)q_rows, (uint64_t)H * DK, (uint64_t)H * DK, kTcRows);
    if (err) return err;
    if ((err = attn_map_2d(&mk, kv, (uint64_t)rows, ldk, ldk, kTcTok))) return err;
    if ((err = attn_map_2d(&mr, rot, (uint64_t)rows, (uint64_t)R, (uint64_t)R, kTcTok))) return err;
    AttnTcArgs a = {};
    a.page_tokens = kTcTok; a.seqs = (const int*)seqs; a.Hq = H; a.Hkv = H; a.scale_log2 = scale * 1.4426950408889634f; a.min_rows = min_rows;
    a.gate = (const __nv_bfloat16*)gate; a.ld_gate = ld_gate; a.gate_head_stride = gate_head_stride; a.gate_offset = gate_offset;
    a.out = (__nv_bfloat16*)out; a.status = (uint32_t*)status; a.budget = g_ps_wait_budget_cycles; a.opt = opt;
    a.k_groups = dim / 64; a.k_head = dim; a.v_off = H * dim; a.v_head = vdim;
    const dim3 grid((max_seq_rows + kTcRows - 1) / kTcRows, H, n_seqs);
    switch (DK) {
        case 128: return launch_latent_prefill<128>(vdim, grid, mq, mk, mk, mr, a, stream);
        case 192: return launch_latent_prefill<192>(vdim, grid, mq, mk, mk, mr, a, stream);
        case 256: return launch_latent_prefill<256>(vdim, grid, mq, mk, mk, mr, a, stream);
        default: return (int)cudaErrorInvalidValue;
    }
}
