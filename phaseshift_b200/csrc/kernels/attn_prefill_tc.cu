// Launchers of the tensor-core attention over paged pools (attn_tc.cuh): prefill-sized steps, and split-KV partials of decode
// and verify rows.  FP8 pools are widened into a bf16 scratch pool first.
#include "attn_tc.cuh"

namespace ps {

// FP8 pools: the sequences' pages are widened once per layer and step into a bf16 scratch pool of the same page shape
// (values times their per-token scale), with its own block table (scratch page = running index) and sequence descriptors
// (slot = sequence index), and the tensor-core kernel runs on that.  The copy moves 3 bytes per cached element; the
// attention it feeds is an order of magnitude faster than the mma.sync kernel on FP8 pages.
constexpr int kDeqD = 256;     // the only head size whose FP8 pools come this way
struct AttnDeqArgs {
    const uint8_t* k_pool; const uint8_t* v_pool; const float* k_scale; const float* v_scale;
    const int* block_table; int max_blocks; int num_pages; int page_tokens; int Hkv;
    const int* seqs; int n_seqs; int min_rows;
    __nv_bfloat16* k_out; __nv_bfloat16* v_out; int out_pages;
    int* bt_out;                 // [n_seqs][max_blocks]
    int* seqs_out;               // [n_seqs][4]
    uint32_t* status;
};

// grid = (scratch pages, Hkv), block = 256
__global__ void __launch_bounds__(256) attn_kv_dequant_kernel(const AttnDeqArgs a) {
    const int p = blockIdx.x, kvh = blockIdx.y, pt = a.page_tokens;
    // which sequence and block this scratch page belongs to
    int base = 0, s = 0, blk = -1, kv_end = 0, slot = -1;
    for (; s < a.n_seqs; ++s) {
        const int* sd = a.seqs + 4 * s;
        const int n_rows = sd[1];
        if (sd[2] < 0 || n_rows <= a.min_rows) continue;
        const int end = sd[3] + n_rows, np = (end + pt - 1) / pt;
        if (p < base + np) { blk = p - base; kv_end = end; slot = sd[2]; break; }
        base += np;
    }
    if (p == 0 && kvh == 0) {
        for (int i = threadIdx.x; i < a.n_seqs; i += blockDim.x) {
            const int* sd = a.seqs + 4 * i;
            a.seqs_out[4 * i + 0] = sd[0]; a.seqs_out[4 * i + 1] = sd[1]; a.seqs_out[4 * i + 2] = sd[2] < 0 ? -1 : i; a.seqs_out[4 * i + 3] = sd[3];
        }
    }
    if (blk < 0) return;
    if (kvh == 0 && threadIdx.x == 0) a.bt_out[(size_t)s * a.max_blocks + blk] = p;
    const int page = a.block_table[(size_t)slot * a.max_blocks + blk];
    const bool ok = page >= 0 && page < a.num_pages;
    if (!ok && threadIdx.x == 0) set_status(a.status, PS_DEV_BAD_INDEX);
    const size_t src = ((size_t)(ok ? page : 0) * a.Hkv + kvh) * pt;          // token rows of the source page
    const size_t dst = ((size_t)p * a.Hkv + kvh) * pt;
    for (int i = threadIdx.x; i < pt * (kDeqD / 16); i += blockDim.x) {
        const int tok = i / (kDeqD / 16), c = i % (kDeqD / 16);
        const bool live = ok && blk * pt + tok < kv_end;
#pragma unroll
        for (int which = 0; which < 2; ++which) {
            const uint8_t* pool = which ? a.v_pool : a.k_pool;
            const float* sp = which ? a.v_scale : a.k_scale;
            __nv_bfloat16* out = which ? a.v_out : a.k_out;
            uint32_t o[8] = {0, 0, 0, 0, 0, 0, 0, 0};
            if (live) {
                const uint4 v = __ldg(reinterpret_cast<const uint4*>(pool + (src + tok) * kDeqD) + c);
                const float sc = sp[src + tok];
                const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float lo = e4m3_to_f32((w[j >> 1] >> ((j & 1) * 16)) & 0xff) * sc;
                    const float hi = e4m3_to_f32((w[j >> 1] >> ((j & 1) * 16 + 8)) & 0xff) * sc;
                    o[j] = f32x2_to_bf16x2_bits(lo, hi);
                }
            }
            uint4* d = reinterpret_cast<uint4*>(out + (dst + tok) * kDeqD + c * 16);
            d[0] = make_uint4(o[0], o[1], o[2], o[3]);
            d[1] = make_uint4(o[4], o[5], o[6], o[7]);
        }
    }
}

static long long* g_attn_tc_prof = nullptr;

// True when the tensor-core kernel can take the call (the caller falls back to the mma.sync kernel otherwise).
bool attn_prefill_tc_supported(int D, int page_tokens, int kv_fp8, const void* q, const void* k_pool, const void* v_pool,
                               const void* gate, int ld_gate, int gate_head_stride, int gate_offset, const void* deq_k, const AttnOptions& opt) {
    static int enabled = -1;
    if (enabled < 0) {
        const char* e = getenv("PS_ATTN_PREFILL");                 // "legacy": always the mma.sync kernel
        enabled = (e != nullptr && e[0] == 'l') ? 0 : 1;
    }
    if (!enabled || D % 64 || D < 64 || D > 256 || (page_tokens != 16 && page_tokens != 32 && page_tokens != 64) || (kv_fp8 && (deq_k == nullptr || D != kDeqD))) return false;
    if (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool) % 16) return false;
    if (k_pool == v_pool && attn_transforms_scores(opt)) return false;
    if (gate != nullptr && !opt.gate_per_head && (((uintptr_t)gate % 16) || (ld_gate % 8) || (gate_head_stride % 8) || (gate_offset % 8))) return false;
    return true;
}

template <int D, bool DEC>
static int launch_attn_tc_size(bool shared, bool transform, dim3 grid, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv,
                               const AttnTcArgs& a, cudaStream_t stream) {
    if (shared && transform) return (int)cudaErrorInvalidValue;          // no design has both; the callers take another kernel
    if (shared) return launch_attn_tc<D, D, DEC, true, false, false>(grid, mq, mk, mv, mk, a, stream);
    if (transform) return launch_attn_tc<D, D, DEC, false, true, false>(grid, mq, mk, mv, mk, a, stream);
    return launch_attn_tc<D, D, DEC, false, false, false>(grid, mq, mk, mv, mk, a, stream);
}
template <bool DEC>
static int launch_attn_tc_any(int D, bool shared, dim3 grid, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv,
                              const AttnTcArgs& a, cudaStream_t stream) {
    const bool tr = attn_transforms_scores(a.opt);
    switch (D) {
        case 64: return launch_attn_tc_size<64, DEC>(shared, tr, grid, mq, mk, mv, a, stream);
        case 128: return launch_attn_tc_size<128, DEC>(shared, tr, grid, mq, mk, mv, a, stream);
        case 192: return launch_attn_tc_size<192, DEC>(shared, tr, grid, mq, mk, mv, a, stream);
        case 256: return launch_attn_tc_size<256, DEC>(shared, tr, grid, mq, mk, mv, a, stream);
        default: return (int)cudaErrorInvalidValue;
    }
}

int launch_attn_prefill_tc(const void* q, int q_rows, const void* k_pool, const void* v_pool, const void* k_scale, const void* v_scale,
                           int kv_fp8, const void* block_table, int max_blocks, int num_pages, int page_tokens, const void* seqs,
                           int n_seqs, int max_seq_rows, int min_rows, int Hq, int Hkv, int D, float sm_scale, const void* gate, int ld_gate,
                           int gate_head_stride, int gate_offset, void* deq_k, void* deq_v, int deq_pages, void* deq_bt, void* deq_seqs,
                           void* out, void* status, const AttnOptions& opt, cudaStream_t stream) {
    if (kv_fp8) {
        // widen the step's pages into the bf16 scratch pool, then attend over that
        if (deq_k == nullptr || deq_v == nullptr || deq_bt == nullptr || deq_seqs == nullptr || deq_pages <= 0) return (int)cudaErrorInvalidValue;
        AttnDeqArgs d;
        d.k_pool = (const uint8_t*)k_pool; d.v_pool = (const uint8_t*)v_pool; d.k_scale = (const float*)k_scale; d.v_scale = (const float*)v_scale;
        d.block_table = (const int*)block_table; d.max_blocks = max_blocks; d.num_pages = num_pages; d.page_tokens = page_tokens; d.Hkv = Hkv;
        d.seqs = (const int*)seqs; d.n_seqs = n_seqs; d.min_rows = min_rows; d.k_out = (__nv_bfloat16*)deq_k; d.v_out = (__nv_bfloat16*)deq_v;
        d.out_pages = deq_pages; d.bt_out = (int*)deq_bt; d.seqs_out = (int*)deq_seqs; d.status = (uint32_t*)status;
        attn_kv_dequant_kernel<<<dim3(deq_pages, Hkv), 256, 0, stream>>>(d);
        int e = PS_LAUNCH_CHECK();
        if (e) return e;
        k_pool = deq_k; v_pool = deq_v; block_table = deq_bt; seqs = deq_seqs; num_pages = deq_pages;
    }
    CUtensorMap mq, mk, mv;
    int err = attn_map_2d(&mq, q, (uint64_t)q_rows, (uint64_t)Hq * D, (uint64_t)Hq * D, kTcRows);
    if (err) return err;
    const uint64_t pool_rows = (uint64_t)num_pages * Hkv * page_tokens;
    if ((err = attn_map_2d(&mk, k_pool, pool_rows, D, D, (uint32_t)page_tokens))) return err;
    if ((err = attn_map_2d(&mv, v_pool, pool_rows, D, D, (uint32_t)page_tokens))) return err;
    AttnTcArgs a;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.num_pages = num_pages; a.page_tokens = page_tokens; a.seqs = (const int*)seqs;
    a.Hq = Hq; a.Hkv = Hkv; a.scale_log2 = sm_scale * 1.4426950408889634f; a.min_rows = min_rows;
    a.gate = (const __nv_bfloat16*)gate; a.ld_gate = ld_gate; a.gate_head_stride = gate_head_stride; a.gate_offset = gate_offset;
    a.out = (__nv_bfloat16*)out; a.status = (uint32_t*)status; a.budget = g_ps_wait_budget_cycles; a.prof = g_attn_tc_prof;
    a.split_tokens = 0; a.max_splits = 0; a.dec_max_rows = 0; a.part_acc = nullptr; a.part_ml = nullptr;
    a.opt = opt; a.k_groups = a.k_head = a.v_off = a.v_head = 0;
    const int tiles = (max_seq_rows + kTcRows - 1) / kTcRows;
    return launch_attn_tc_any<false>(D, k_pool == v_pool, dim3(tiles, Hq, n_seqs), mq, mk, mv, a, stream);
}

}  // namespace ps

// Decode / verify attention on the tensor cores (bf16 pools, head dim 64 / 128 / 192 / 256, pages of 16 / 32 / 64 tokens, at most 8 query
// heads per KV head): split-KV partials for every sequence of the step with at most `dec_max_rows` (<= 16) rows, in the
// layout of ps_paged_attention's merge pass (`part_acc` [rows, Hq, max_splits, D] fp32, `part_ml` [rows, Hq, max_splits, 2]);
// the caller runs ps_paged_attention_merge afterwards.  `split_tokens` is a multiple of 64, `q` is [q_rows, Hq, D] bf16.
// Reference: src/phaseshift/models/qwen35/kernels/optimized/attention/paged_decode.hip (split-KV decode); the grouped-query
// packing onto one MMA tile has no counterpart there.
// `options`: an AttnOptions (attn_options.cuh) or null; pass the same ones to the merge pass, which applies sink and gate.
PS_API int ps_attn_decode_tc_ex(const void* q, int q_rows, const void* k_pool, const void* v_pool, const void* block_table,
                             int max_blocks, int page_tokens, int num_pages, const void* seqs, int n_seqs, int dec_max_rows,
                             int Hq, int Hkv, int D, float sm_scale, int split_tokens, int max_splits, int max_visible,
                             void* part_acc, void* part_ml, void* status, const void* options, cudaStream_t stream) {
    using namespace ps;
    const AttnOptions opt = attn_options(options);
    if (!attn_options_ok(opt) || (k_pool == v_pool && attn_transforms_scores(opt)) || D % 64 || D < 64 || D > 256 || (page_tokens != 16 && page_tokens != 32 && page_tokens != 64) || Hkv <= 0 || (Hq % Hkv) || Hq / Hkv > 8 ||
        dec_max_rows < 1 || dec_max_rows > 16 || split_tokens < kTcTok || (split_tokens % kTcTok) || n_seqs <= 0 ||
        (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)part_acc) % 16))
        return (int)cudaErrorInvalidValue;
    int n_splits = (max_visible + split_tokens - 1) / split_tokens;
    if (n_splits < 1) n_splits = 1;
    if (n_splits > max_splits) return (int)cudaErrorInvalidValue;
    CUtensorMap mq, mk, mv;
    int err = attn_map_2d(&mq, q, (uint64_t)q_rows * Hq, D, D, 8);                 // the [rows * Hq, D] view, 8-row boxes
    if (err) return err;
    const uint64_t pool_rows = (uint64_t)num_pages * Hkv * page_tokens;
    if ((err = attn_map_2d(&mk, k_pool, pool_rows, D, D, (uint32_t)page_tokens))) return err;
    if ((err = attn_map_2d(&mv, v_pool, pool_rows, D, D, (uint32_t)page_tokens))) return err;
    AttnTcArgs a;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.num_pages = num_pages; a.page_tokens = page_tokens; a.seqs = (const int*)seqs;
    a.Hq = Hq; a.Hkv = Hkv; a.scale_log2 = sm_scale * 1.4426950408889634f; a.min_rows = 0;
    a.gate = nullptr; a.ld_gate = 0; a.gate_head_stride = 0; a.gate_offset = 0; a.out = nullptr;
    a.status = (uint32_t*)status; a.budget = g_ps_wait_budget_cycles; a.prof = nullptr;
    a.split_tokens = split_tokens; a.max_splits = max_splits; a.dec_max_rows = dec_max_rows;
    a.part_acc = (float*)part_acc; a.part_ml = (float*)part_ml; a.opt = opt; a.k_groups = a.k_head = a.v_off = a.v_head = 0;
    return launch_attn_tc_any<true>(D, k_pool == v_pool, dim3(n_splits, Hkv, n_seqs), mq, mk, mv, a, stream);
}

PS_API int ps_attn_decode_tc(const void* q, int q_rows, const void* k_pool, const void* v_pool, const void* block_table,
                             int max_blocks, int page_tokens, int num_pages, const void* seqs, int n_seqs, int dec_max_rows,
                             int Hq, int Hkv, int D, float sm_scale, int split_tokens, int max_splits, int max_visible,
                             void* part_acc, void* part_ml, void* status, cudaStream_t stream) {
    return ps_attn_decode_tc_ex(q, q_rows, k_pool, v_pool, block_table, max_blocks, page_tokens, num_pages, seqs, n_seqs,
                                dec_max_rows, Hq, Hkv, D, sm_scale, split_tokens, max_splits, max_visible, part_acc, part_ml,
                                status, nullptr, stream);
}

// Timing aid: a device buffer of 32 x 16 int64 that CTA (0, 0, 0) of later launches fills with cycle stamps of its softmax
// thread 0 (slots 0-7: tile start, scores ready, scores loaded, row maximum exchanged, probabilities computed, stored,
// proxy fence done, arrived) and of the issuing threads (slots 8-10: score issuer at its tile's start, operands ready,
// issued; 11-12: output issuer with probabilities ready, issued; slot 15 of tiles 0 and 1: start and end of the CTA).  nullptr switches it off.
PS_API void ps_attn_prefill_tc_set_prof(void* buf) { ps::g_attn_tc_prof = (long long*)buf; }
