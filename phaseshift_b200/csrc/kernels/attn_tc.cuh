// Causal paged attention for prefill-sized steps on the fifth-generation tensor cores (head dims 64, 128, 192 and 256, bf16
// pools, pages of 16, 32 or 64 tokens): one CTA = 128 consecutive query rows of one sequence and one query head.  With the
// options of attn_options.cuh (block-local or windowed masks, sinks, query temperature, distance bias, gates), and optionally with
// keys that are the values.
// Described for head dim 256; other sizes have fewer 64-column groups:
//
//   warp 8   TMA producer for Q (once) and the K tiles: a 64-token tile is four pages, each fetched as four
//            64-column boxes (128-byte swizzle) straight from the paged pool through a tensor map over
//            [pages * kv heads * page tokens, D] (one, two or four pages per tile for 64-, 32-, 16-token pages); two stages.
//   warp 9   TMA producer for the V tiles (same boxes, two stages).
//   warps 10, 11  one thread each issues S(t) = Q K(t)^T (tcgen05.mma, 16 products of 128 x 64 x 16) into one of two
//            64-column accumulators, warp 10 for even t and warp 11 for odd t, as soon as the K stage and the
//            accumulator are free, so the tensor core computes the next scores while the softmax warps work on
//            the current ones.
//   warp 12  one thread issues O += P(t) V(t) into a 256-column accumulator.  V is consumed as it lies in the
//            pool (token rows, dims contiguous): an MN-major B operand.
//   warps 0-7  softmax: two threads own a query row (= TMEM lane), 32 score columns each.  Scores come back with
//            tcgen05.ld (both threads read the whole row for its maximum: no shuffles, no exchange), probabilities go
//            to shared memory as a bf16 K-major A operand (swizzled by hand), and the output accumulator is
//            rescaled in tensor memory only when a row's maximum has grown
//            by more than 2^8 since the reference used for its exponents (the sum absorbs the difference, so the
//            result is the exact softmax).  The epilogue normalises, applies the sigmoid output gate and writes
//            bf16 through shared memory with coalesced 16-byte stores.
//
// Keys that are the values (SHARED, one pool): every tile is fetched once into one of four stages, read by S(t) as the K-major
// operand and by P V(t) as the MN-major one, and freed by the latter; warp 9 has nothing to do.
//
// Every wait is bounded; a timeout raises the CTA's abort flag, every role unwinds, outstanding copies get a
// bounded chance to land, tensor memory is freed and PS_DEV_WAIT_TIMEOUT is recorded.  Token rows of the last
// tile that lie beyond the sequence's end are zeroed in shared memory before the P V product (their
// probabilities are zero, but stale pool contents must not be able to inject NaNs).
//
// The reference's prefill attention (src/phaseshift/models/qwen35/kernels/optimized/attention/
// paged_prefill.hip:408-874) tiles 16 query rows per wave on WMMA; FP8 pools, other head sizes and other page
// sizes stay on the mma.sync kernel (attn_prefill.cu).  Launchers: attn_prefill_tc.cu (paged pools), attn_latent.cu (expanded
// latent attention).
#pragma once

#include <cuda.h>

#include "attn_options.cuh"
#include "ps_common.cuh"
#include "ps_tcgen05.cuh"

namespace ps {

constexpr int kTcRows = 128, kTcTok = 64;
constexpr int kTcThreads = 416;                      // warps 0-7 softmax, 8 Q / K producer, 9 V producer, 10-11 S issuers, 12 P V issuer
constexpr int kTcPBuf = kTcRows * kTcTok * 2;         // 16 KB: 128 rows x 64 tokens
template <int DK, int DV> struct TcShape {                           // query / key size, value size
    static_assert(DK % 64 == 0 && DK >= 64 && DK <= 256 && DV % 64 == 0 && DV >= 64 && DV <= 256, "head dims of 64-column groups");
    static constexpr int kGroups = DK / 64, kVGroups = DV / 64;   // 64-column boxes per row
    static constexpr int kQBytes = kTcRows * DK * 2;              // 256: 64 KB, four 64-column boxes of 128 rows
    static constexpr int kKStage = kTcTok * DK * 2;               // 256: 32 KB, four 64-column boxes of 64 tokens
    static constexpr int kVStage = kTcTok * DV * 2;
    static constexpr int kSmem = kQBytes + 2 * kKStage + 2 * kVStage + 2 * kTcPBuf;
    static constexpr int kOutPitch = DV + 8;                      // staging pitch of the epilogue (elements)
    static constexpr uint32_t kTmemCols = DV <= 128 ? 256 : 512;  // S0 | S1 (64 each) | O (DV)
    static_assert(kTcRows * kOutPitch * 2 <= kSmem, "the output staging lies inside the tile buffers");
};

struct AttnTcArgs {
    const int* block_table; int max_blocks; int num_pages; int page_tokens;     // page_tokens: 16, 32 or 64
    const int* seqs;             // [n_seqs][4] = row_start, n_rows, slot, pos_start
    int Hq, Hkv; float scale_log2;
    int min_rows;                // sequences with at most this many rows in the step are left to the split-KV kernel
    const __nv_bfloat16* gate; int ld_gate; int gate_head_stride; int gate_offset;
    __nv_bfloat16* out;          // [rows, Hq * D]
    uint32_t* status;
    long long budget;
    // decode / verify variant (DEC): split-KV partials in the layout of the per-row kernel's merge pass
    int split_tokens; int max_splits; int dec_max_rows;
    float* part_acc; float* part_ml;
    AttnOptions opt;             // (sink and gate: the merge pass applies them for DEC)
    // expanded keys and values (EXPANDED): rows of consecutive tokens; columns of a head's keys, first column of its values
    int k_groups, k_head, v_off, v_head;
    long long* prof;             // optional cycle stamps of CTA (0, 0, 0): [32 tiles][16], softmax slots 0-7, issuer slots 8-12
};

namespace tc {
// Shared-memory descriptor of an MN-major operand (rows = K index, 128 bytes = 64 MN elements per row, 128-byte
// swizzle): `lbo` bytes between 64-element groups along MN, `sbo` bytes between 8-row groups along K.
__device__ __forceinline__ uint64_t smem_desc_sw128_mn(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
    uint64_t d = 0;
    d |= (uint64_t)((smem_addr >> 4) & 0x3FFF);
    d |= (uint64_t)((lbo >> 4) & 0x3FFF) << 16;
    d |= (uint64_t)((sbo >> 4) & 0x3FFF) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// kind::f16, A = bf16 K-major, B = bf16 MN-major, D = fp32.
__host__ __device__ constexpr uint32_t idesc_bf16_f32_bmn(int M, int N) {
    return (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(N >> 3) << 17) | ((uint32_t)(M >> 4) << 24);
}
__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
        ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
          "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
          "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
          "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
}
}  // namespace tc

__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// sigmoid(x) = 0.5 + 0.5 tanh(x / 2) with the hardware tanh (one special-function operation instead of an exponential and a
// reciprocal; absolute error about 5e-4, a fraction of the bf16 rounding step of the gated output).  A full-precision
// division here made the epilogue the longest phase of a short CTA.
__device__ __forceinline__ float sigmoid_fast(float x) {
    float t;
    asm("tanh.approx.f32 %0, %1;" : "=f"(t) : "f"(0.5f * x));
    return fmaf(0.5f, t, 0.5f);
}

// Expanded keys and values of a step (EXPANDED): the sequences with more than `min_rows` rows follow one another, each with the
// tokens its rows see, from a multiple of the tile on.
__device__ __forceinline__ int expanded_first(const int* sd, const AttnOptions& o) { return attn_first(o, sd[3]) / kTcTok * kTcTok; }
__device__ __forceinline__ int expanded_rows(const int* sd, int min_rows, const AttnOptions& o) {
    if (sd[2] < 0 || sd[1] <= min_rows) return 0;
    return (sd[3] + sd[1] - expanded_first(sd, o) + kTcTok - 1) / kTcTok * kTcTok;
}
// Row that position 0 of sequence `s` would have.
__device__ __forceinline__ int expanded_row0(const int* seqs, int s, int min_rows, const AttnOptions& o) {
    int at = 0;
    for (int i = 0; i < s; ++i) at += expanded_rows(seqs + 4 * i, min_rows, o);
    return at - expanded_first(seqs + 4 * s, o);
}

// Prefill (DEC = false): grid = (q tiles of 128 rows, Hq, n_seqs); the heaviest (latest) query tiles are scheduled first.
// Decode / verify (DEC = true): grid = (KV splits, Hkv, n_seqs).  A CTA serves one sequence with at most 16 rows in the step
// and one KV head: tile row 8 r + g is query head g of that KV head for the sequence's row r (grouped-query packing: the G <= 8
// heads that share the KV head ride in one MMA tile, so K and V are read once for all of them), over the tokens of its
// split; it leaves unnormalised partial outputs and (maximum, sum) pairs for the merge pass of paged_attention.cu.
// TRANSFORM: query temperature and distance bias, applied to the scores before the maximum.
// EXPANDED: keys and values were expanded per query head into rows of consecutive tokens (attn_latent.cu), the last 64-column
// groups of the keys (`map_r`) are shared by all heads.
template <int DK, int DV, bool DEC, bool SHARED, bool TRANSFORM, bool EXPANDED>
__global__ void __launch_bounds__(kTcThreads, 1)
attn_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
               const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_r, const AttnTcArgs a) {
    static_assert(!SHARED || DK == DV, "keys that are the values have their size");
    static_assert(!EXPANDED || (!DEC && !SHARED), "expanded keys and values are for prefill-sized steps");
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    using Shape = TcShape<DK, DV>;
    constexpr int kTcQBytes = Shape::kQBytes, kTcKStage = Shape::kKStage, kTcVStage = Shape::kVStage, kTcOutPitch = Shape::kOutPitch;
    constexpr int kNB = Shape::kGroups, kNBV = Shape::kVGroups;
    constexpr uint32_t kTcTmemCols = Shape::kTmemCols;
    constexpr int kStageMask = SHARED ? 3 : 1;       // stages of one operand (a shared tile's four stages cover both operands' space)
    constexpr int kStageLog = SHARED ? 2 : 1;
    // Q, two K and two V stages, two P buffers: 224 KB at D = 256, which with the static part below is the whole 227 KB of the SM;
    // the swizzled tiles need the 1024-byte alignment that the declaration asks for (checked, not assumed)
    unsigned char* smem = smem_raw;
    if ((tc::smem_u32(smem) & 1023u) != 0) {
        if (threadIdx.x == 0) set_status(a.status, PS_DEV_BAD_INDEX);
        return;
    }
    unsigned char* sQ = smem;
    unsigned char* sK = sQ + kTcQBytes;
    unsigned char* sV = sK + 2 * kTcKStage;
    unsigned char* sP = sV + 2 * kTcVStage;
    __shared__ __align__(8) uint64_t q_full, k_full[4], v_full[2], s_full[2], p_full[2], pv_done[2], kv_free[4];
    __shared__ float s_l[2][kTcRows];            // row sums of the two column halves, exchanged once at the end
    __shared__ uint32_t tmem_base_slot;
    __shared__ int s_abort, s_bad, k_issued, k_consumed, v_issued, v_consumed, q_issued, q_consumed;

    const int* sd = a.seqs + 4 * blockIdx.z;
    const int row_start = sd[0], n_rows = sd[1], slot = sd[2], pos_start = sd[3];
    const int G = a.Hq / a.Hkv;
    // tiles of the CTA: `n_keep` tiles of kept first positions from tile `keep0` on, then those from `t_first` on, T in all
    int r_begin, nq, h, kvh, pos_q0, kv_end, t_first, T, keep0 = 0, n_keep = 0;
    const int keep_tiles = EXPANDED ? 0 : (a.opt.keep_first + kTcTok - 1) / kTcTok;
    if constexpr (DEC) {
        if (slot < 0 || n_rows <= 0 || n_rows > a.dec_max_rows) return;
        r_begin = 0; nq = 8 * n_rows; kvh = blockIdx.y; h = kvh * G;
        pos_q0 = pos_start; kv_end = pos_start + n_rows;
        const int tps = a.split_tokens / kTcTok;                         // tiles per split
        const int t_lo = attn_first(a.opt, pos_q0) / kTcTok;             // tile of the first token any row sees
        const int t_end = min((kv_end + kTcTok - 1) / kTcTok, ((int)blockIdx.x + 1) * tps);
        keep0 = (int)blockIdx.x * tps;
        t_first = max(keep0, t_lo);
        n_keep = max(0, min(min(keep_tiles, t_lo), keep0 + tps) - keep0);
        T = n_keep + max(0, t_end - t_first);
        if (T <= 0) return;
    } else {
        const int tile = (int)gridDim.x - 1 - (int)blockIdx.x;
        r_begin = tile * kTcRows;
        if (r_begin >= n_rows || slot < 0 || n_rows <= a.min_rows) return;
        nq = min(kTcRows, n_rows - r_begin);
        h = blockIdx.y; kvh = h / G;
        pos_q0 = pos_start + r_begin;
        kv_end = pos_q0 + nq;
        t_first = attn_first(a.opt, pos_q0) / kTcTok;
        n_keep = min(keep_tiles, t_first);
        T = n_keep + (kv_end + kTcTok - 1) / kTcTok - t_first;
    }
    auto tile_of = [&](int t) { return t < n_keep ? keep0 + t : t_first - n_keep + t; };
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool cta_stamp = a.prof != nullptr && threadIdx.x == 0 && blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0;
    if (cta_stamp) a.prof[15] = clock64();

    if (threadIdx.x == 0) {
        tc::mbar_init(&q_full, 1);
        for (int s = 0; s < 2; ++s) {
            tc::mbar_init(&k_full[s], 1); tc::mbar_init(&v_full[s], 1); tc::mbar_init(&s_full[s], 1);
            tc::mbar_init(&p_full[s], 8); tc::mbar_init(&pv_done[s], 1);
        }
        if constexpr (SHARED) {
            tc::mbar_init(&k_full[2], 1); tc::mbar_init(&k_full[3], 1);
            for (int s = 0; s < 4; ++s) tc::mbar_init(&kv_free[s], 1);
        }
        tc::fence_barrier_init();
        s_abort = 0; s_bad = 0; k_issued = k_consumed = v_issued = v_consumed = q_issued = q_consumed = 0;
        tc::tma_prefetch_desc(&map_q); tc::tma_prefetch_desc(&map_k); tc::tma_prefetch_desc(&map_v);
    }
    if (warp == 12) {
        tc::tmem_alloc(&tmem_base_slot, kTcTmemCols);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem = tmem_base_slot;
    const uint32_t tmem_o = tmem + 128;

    int exp_row0 = 0;            // EXPANDED: row of the sequence's position 0, were it there
    if constexpr (EXPANDED) exp_row0 = expanded_row0(a.seqs, (int)blockIdx.z, a.min_rows, a.opt);

    if (SHARED && warp == 9) {
        // the values arrive with the keys
    } else if (warp == 8 || warp == 9) {
        // ------------------------------------------------ TMA producers: warp 8 = Q and K, warp 9 = V.  One lane per box (a
        // tile is up to 16 boxes: pages x four 64-column groups): issuing them from one thread one after the other costs
        // more than a thousand cycles, and the stage's consumer is waiting for them.
        const bool isK = warp == 8;
        if (isK) {
            if constexpr (DEC) {
                // one 8-row box per (row of the sequence, 64-column group): the G heads of this KV head are consecutive rows
                // of the [rows * Hq, D] view of q; tile rows 8 r + g with g >= G hold other heads' values and are never used
                if (lane == 0) tc::mbar_expect_tx(&q_full, (uint32_t)n_rows * (uint32_t)kNB * 1024u);
                __syncwarp();
                for (int i = lane; i < kNB * n_rows; i += 32) {
                    const int r = i / kNB, c4 = i % kNB;
                    tc::tma_load_2d(sQ + c4 * (kTcRows * 128) + (8 * r) * 128, &map_q, c4 * 64, (row_start + r) * a.Hq + h, &q_full);
                }
            } else {
                if (lane == 0) tc::mbar_expect_tx(&q_full, kTcQBytes);
                __syncwarp();
                if (lane < kNB) tc::tma_load_2d(sQ + lane * (kTcRows * 128), &map_q, h * DK + lane * 64, row_start + r_begin, &q_full);
            }
            if (lane == 0) q_issued = 1;
        }
        const int* bt = a.block_table + (size_t)slot * a.max_blocks;
        const int pt = a.page_tokens, ppt = kTcTok / pt;            // a page is one box of pt token rows per 64-column group
        const int nb = isK ? kNB : kNBV, stage_bytes = isK ? kTcKStage : kTcVStage;
        const int pg = lane / nb, cb = lane % nb;
        const bool active = pg < (EXPANDED ? 1 : ppt);
        unsigned char* stage0 = isK ? sK : sV;
        uint64_t* full = isK ? k_full : v_full;
        uint64_t* freed = isK ? s_full : pv_done;                   // a K stage is free once S(t) has read it, a V stage after P V(t)
        const CUtensorMap* map = isK ? &map_k : &map_v;
        int x = cb * 64;                                            // column of this lane's box
        if constexpr (EXPANDED) {
            if (!isK) x += a.v_off + h * a.v_head;
            else if (cb < a.k_groups) x += h * a.k_head;
            else { map = &map_r; x -= a.k_groups * 64; }
        }
        for (int t = 0; t < T; ++t) {
            const int b = t & kStageMask;
            int page = 0;
            const int blk = tile_of(t) * ppt + pg;
            if (!EXPANDED && active && blk * pt < kv_end) {
                page = bt[blk];
                if (page < 0 || page >= a.num_pages) { s_bad = 1; page = 0; }
            }
            if constexpr (SHARED) {
                if (t >= 4 && !__all_sync(0xffffffffu, tc::mbar_wait_abortable(&kv_free[b], (uint32_t)((t - 4) >> 2) & 1u, a.budget, &s_abort))) break;
            } else {
                if (t >= 2 && !__all_sync(0xffffffffu, tc::mbar_wait_abortable(&freed[b], (uint32_t)((t - 2) >> 1) & 1u, a.budget, &s_abort))) break;
            }
            if (lane == 0) tc::mbar_expect_tx(&full[b], stage_bytes);
            __syncwarp();
            if (active)
                tc::tma_load_2d(stage0 + b * stage_bytes + cb * (kTcTok * 128) + pg * (pt * 128), map, x,
                                EXPANDED ? exp_row0 + (t_first + t) * kTcTok : (page * a.Hkv + kvh) * pt, &full[b]);
            if (lane == 0) { if (isK) k_issued = t + 1; else v_issued = t + 1; }
        }
    } else if (warp == 10 || warp == 11) {
        // ------------------------------------------------ score issuers: warp 10 issues S(t) for even t, warp 11 for odd t.
        // A tcgen05.mma costs its issuing thread about 80 cycles whatever its size, and a 128 x 64 x 16 product is only 32
        // cycles of tensor work, so one thread cannot keep the pipe fed; two threads take turns.
        if (lane == 0) {
            constexpr uint32_t idesc_s = tc::idesc_bf16_f32(kTcRows, kTcTok);
            const int b = warp - 10;
            const uint32_t q_addr = tc::smem_u32(sQ), k_addr0 = tc::smem_u32(sK);
            bool ok = tc::mbar_wait_abortable(&q_full, 0, a.budget, &s_abort);
            if (ok) q_consumed = 1;
            for (int t = b; t < T && ok; t += 2) {
                const uint32_t ph = (uint32_t)(t >> 1) & 1u;
                const bool stamp = a.prof != nullptr && blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0 && t < 32;
                if (stamp) a.prof[t * 16 + 8] = clock64();
                // the score buffer is free once the softmax warps have read S(t - 2), which they signal with P(t - 2)
                if (t >= 2 && !tc::mbar_wait_abortable(&p_full[b], ph ^ 1u, a.budget, &s_abort)) { ok = false; break; }
                const int ks_ = t & kStageMask;                                          // the tile's stage
                const uint32_t k_addr = k_addr0 + ks_ * kTcKStage;
                if (!tc::mbar_wait_abortable(&k_full[ks_], (uint32_t)(t >> kStageLog) & 1u, a.budget, &s_abort)) { ok = false; break; }
                if (stamp) a.prof[t * 16 + 9] = clock64();
                atomicMax(&k_consumed, t + 1);
                tc::fence_after_sync();
#pragma unroll
                for (int ks = 0; ks < DK / 16; ++ks) {
                    const uint64_t adesc = tc::smem_desc_sw128(q_addr + (ks >> 2) * (kTcRows * 128) + (ks & 3) * 32);
                    const uint64_t bdesc = tc::smem_desc_sw128(k_addr + (ks >> 2) * (kTcTok * 128) + (ks & 3) * 32);
                    tc::mma_bf16_ss(tmem + b * kTcTok, adesc, bdesc, idesc_s, ks > 0 ? 1u : 0u);
                }
                tc::mma_commit(&s_full[b]);
                if (stamp) a.prof[t * 16 + 10] = clock64();
            }
        }
    } else if (warp == 12) {
        // ------------------------------------------------ output issuer: O += P(t) V(t)
        if (lane == 0) {
            constexpr uint32_t idesc_o = tc::idesc_bf16_f32_bmn(kTcRows, DV);
            const uint32_t v_addr0 = tc::smem_u32(SHARED ? sK : sV), p_addr = tc::smem_u32(sP);
            for (int t = 0; t < T; ++t) {
                const int b = t & 1;
                const uint32_t ph = (uint32_t)(t >> 1) & 1u;
                const bool stamp = a.prof != nullptr && blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0 && t < 32;
                if (!tc::mbar_wait_abortable(&p_full[b], ph, a.budget, &s_abort)) break;
                if (stamp) a.prof[t * 16 + 11] = clock64();
                const uint32_t v_addr = v_addr0 + (t & kStageMask) * kTcVStage;
                if (!tc::mbar_wait_abortable(SHARED ? &k_full[t & 3] : &v_full[b], SHARED ? (uint32_t)(t >> 2) & 1u : ph, a.budget, &s_abort)) break;
                v_consumed = t + 1;
                tc::fence_after_sync();
#pragma unroll
                for (int kk = 0; kk < kTcTok / 16; ++kk) {
                    const uint64_t adesc = tc::smem_desc_sw128(p_addr + b * kTcPBuf + kk * 32);
                    const uint64_t bdesc = tc::smem_desc_sw128_mn(v_addr + kk * (16 * 128), kTcTok * 128, 1024);
                    tc::mma_bf16_ss(tmem_o, adesc, bdesc, idesc_o, (t > 0 || kk > 0) ? 1u : 0u);
                }
                if constexpr (SHARED) tc::mma_commit(&kv_free[t & 3]);
                tc::mma_commit(&pv_done[b]);
                if (stamp) a.prof[t * 16 + 12] = clock64();
            }
        }
    } else {
        // ------------------------------------------------ softmax warps 0-7: two threads per query row.  Warp w works on
        // TMEM lanes 32 (w % 4) .. + 31 (the quadrant a warp may touch) and on score columns 32 (w / 4) .. + 31 of the tile.
        const int quad = warp & 3, half = warp >> 2;
        const int row = quad * 32 + lane;
        const uint32_t lane_base = (uint32_t)(quad * 32) << 16;
        const int rp = DEC ? pos_q0 + (row >> 3) : pos_q0 + row;     // position of this thread's query row
        const float sc = a.scale_log2;
        const int lo = attn_first(a.opt, rp);                        // first token this row sees
        const int lo_max = attn_first(a.opt, kv_end - 1);            // ... and the largest of any row
        const int keep = EXPANDED ? 0 : a.opt.keep_first;
        [[maybe_unused]] float row_scale = sc, bias_far = 0.f;
        [[maybe_unused]] const float* bias = nullptr;                // this row's head, by distance
        if constexpr (TRANSFORM) {
            row_scale = sc * attn_temperature(a.opt, rp);
            if (a.opt.bias != nullptr) {
                bias = a.opt.bias + (size_t)(DEC ? min(h + (row & 7), a.Hq - 1) : h) * a.opt.bias_len;
                bias_far = bias[a.opt.bias_len - 1] * 1.4426950408889634f;
            }
        }
        float m_ref = 0.f, l_run = 0.f;
        bool fresh = true;                                            // this row has not seen a token yet: m_ref is a placeholder
        bool ok = true;
        // the epilogue reads this tile's gate values (one 512-byte run per row): ask for them now, so that they come from
        // L2 then
        if (!DEC && a.gate != nullptr && !a.opt.gate_per_head && half == 0 && row < nq)
            tc::bulk_prefetch_l2(a.gate + (size_t)(row_start + r_begin + row) * a.ld_gate + (size_t)h * a.gate_head_stride + a.gate_offset, DV * 2);
        for (int t = 0; t < T; ++t) {
            const int b = t & 1;
            const uint32_t ph = (uint32_t)(t >> 1) & 1u;
            const int tt = tile_of(t);                                // tile index within the sequence
            const int t0 = tt * kTcTok + half * 32;                   // first token of this thread's columns
            const bool stamp = a.prof != nullptr && threadIdx.x == 0 && blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0 && t < 32;
            if (stamp) a.prof[t * 16 + 0] = clock64();
            ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&s_full[b], ph, a.budget, &s_abort));
            if (!ok) break;
            tc::fence_after_sync();
            if (stamp) a.prof[t * 16 + 1] = clock64();
            // both threads of a row read all 64 scores and take the maximum themselves (cheaper than an exchange through
            // shared memory); each then exponentiates its own 32 columns
            uint32_t sr[32], so[32];
            tc::tmem_ld_32x32(tmem + lane_base + b * kTcTok + half * 32, sr);
            tc::tmem_ld_32x32(tmem + lane_base + b * kTcTok + (half ^ 1) * 32, so);
            tc::tmem_ld_wait();
            if (stamp) a.prof[t * 16 + 2] = clock64();
            if constexpr (TRANSFORM) {
                const int to = tt * kTcTok + (half ^ 1) * 32;
                if (bias == nullptr || rp - tt * kTcTok - (kTcTok - 1) >= a.opt.bias_len - 1) {      // the whole tile is far away
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        sr[j] = __float_as_uint(fmaf(__uint_as_float(sr[j]), row_scale, bias_far));
                        so[j] = __float_as_uint(fmaf(__uint_as_float(so[j]), row_scale, bias_far));
                    }
                } else {
                    const int far = a.opt.bias_len - 1;
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        const float br = __ldg(bias + min(max(rp - t0 - j, 0), far)) * 1.4426950408889634f;
                        const float bo = __ldg(bias + min(max(rp - to - j, 0), far)) * 1.4426950408889634f;
                        sr[j] = __float_as_uint(fmaf(__uint_as_float(sr[j]), row_scale, br));
                        so[j] = __float_as_uint(fmaf(__uint_as_float(so[j]), row_scale, bo));
                    }
                }
            }
            if (tt * kTcTok < lo_max) {                               // tokens before some row's block
                const int to = tt * kTcTok + (half ^ 1) * 32;
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    if (t0 + j < lo && t0 + j >= keep) sr[j] = 0xff800000u;
                    if (to + j < lo && to + j >= keep) so[j] = 0xff800000u;
                }
            }
            if (tt * kTcTok + kTcTok - 1 > pos_q0) {                  // some row of the tile does not see every token
                const int to = tt * kTcTok + (half ^ 1) * 32;
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    if (t0 + j > rp) sr[j] = 0xff800000u;             // -inf
                    if (to + j > rp) so[j] = 0xff800000u;
                }
            }
            float mq[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int j = 0; j < 32; ++j) mq[j & 3] = fmaxf(mq[j & 3], fmaxf(__uint_as_float(sr[j]), __uint_as_float(so[j])));
            float mx = fmaxf(fmaxf(mq[0], mq[1]), fmaxf(mq[2], mq[3]));
            if constexpr (!TRANSFORM) mx *= sc;                       // scale > 0, so the maximum commutes with it
            if (stamp) a.prof[t * 16 + 3] = clock64();
            float alpha = 1.f;
            if (fresh) {                                              // (a row that sees nothing yet keeps a finite reference)
                if (mx != -INFINITY) { m_ref = mx; fresh = false; }
            }
            else if (mx > m_ref + 8.f) { alpha = ex2_approx(m_ref - mx); m_ref = mx; }
            const bool rescale = __any_sync(0xffffffffu, alpha != 1.f);
            float sq[4] = {0.f, 0.f, 0.f, 0.f};
            uint32_t pk[16];
#pragma unroll
            for (int j = 0; j < 32; j += 2) {
                const float s0 = __uint_as_float(sr[j]), s1 = __uint_as_float(sr[j + 1]);
                const float p0 = ex2_approx(TRANSFORM ? s0 - m_ref : fmaf(s0, sc, -m_ref));
                const float p1 = ex2_approx(TRANSFORM ? s1 - m_ref : fmaf(s1, sc, -m_ref));
                sq[(j >> 1) & 3] += p0 + p1;
                pk[j >> 1] = f32x2_to_bf16x2_bits(p0, p1);
            }
            l_run = l_run * alpha + ((sq[0] + sq[1]) + (sq[2] + sq[3]));
            if (t >= 2) {                                             // P buffer b was read by P V(t - 2)
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[b], (uint32_t)((t - 2) >> 1) & 1u, a.budget, &s_abort));
                if (!ok) break;
            }
            if (stamp) a.prof[t * 16 + 4] = clock64();
            unsigned char* prow = sP + b * kTcPBuf + row * 128;
#pragma unroll
            for (int c = 0; c < 4; ++c)
                *reinterpret_cast<uint4*>(prow + (((half * 4 + c) ^ (row & 7)) << 4)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
            if (t == T - 1 && kv_end < (tt + 1) * kTcTok) {
                // token rows of the last V tile beyond the sequence's end: zero them (whole 128-byte rows, so the swizzle
                // does not matter)
                // (a shared tile has been read by S(t) already: the scores are here)
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(SHARED ? &k_full[t & 3] : &v_full[b], SHARED ? (uint32_t)(t >> 2) & 1u : ph,
                                                                     a.budget, &s_abort));
                if (!ok) break;
                const int jz = kv_end - tt * kTcTok;
                unsigned char* vs = (SHARED ? sK : sV) + (t & kStageMask) * kTcVStage;
                for (int i = (int)threadIdx.x; i < (kTcTok - jz) * kNBV * 8; i += 2 * kTcRows) {
                    const int r = jz + i / (kNBV * 8), cb = i % (kNBV * 8) >> 3, c = i & 7;
                    *reinterpret_cast<uint4*>(vs + cb * (kTcTok * 128) + r * 128 + c * 16) = make_uint4(0, 0, 0, 0);
                }
            }
            if (stamp) a.prof[t * 16 + 5] = clock64();
            tc::fence_proxy_async_smem();
            if (stamp) a.prof[t * 16 + 6] = clock64();
            if (rescale) {                                            // t >= 1: O must be complete up to P V(t - 1)
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[b ^ 1], (uint32_t)((t - 1) >> 1) & 1u, a.budget, &s_abort));
                if (!ok) break;
                tc::fence_after_sync();
#pragma unroll 1
                for (int c0 = half * (DV / 2); c0 < (half + 1) * (DV / 2); c0 += 32) {
                    uint32_t r[32];
                    tc::tmem_ld_32x32(tmem_o + lane_base + c0, r);
                    tc::tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * alpha);
                    tc::tmem_st_32x32(tmem_o + lane_base + c0, r);
                }
                tc::tmem_st_wait();
            }
            tc::fence_before_sync();
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&p_full[b]);
            if (stamp) a.prof[t * 16 + 7] = clock64();
        }
        // ---- epilogue: O / l -> bf16 rows staged in shared memory (Q and K stages are free once the last P V is done)
        if (ok) ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[(T - 1) & 1], (uint32_t)((T - 1) >> 1) & 1u, a.budget, &s_abort));
        if (cta_stamp) a.prof[2 * 16 + 15] = clock64();
        s_l[half][row] = l_run;
        asm volatile("bar.sync 1, 256;" ::: "memory");               // the eight softmax warps only; every one of them gets here
        if (cta_stamp) a.prof[3 * 16 + 15] = clock64();
        if constexpr (DEC) {
            // partial result of this split for query row (r, g): unnormalised output, reference maximum (natural-log units, as
            // the merge pass expects) and sum
            const int r = row >> 3, g = row & 7;
            const bool mine = row < nq && g < G;
            if (ok && quad * 32 < nq) {                              // warp-uniform: the tensor-memory loads are collective
                tc::fence_after_sync();
                const size_t idx = ((size_t)(row_start + (mine ? r : 0)) * a.Hq + h + (mine ? g : 0)) * a.max_splits + blockIdx.x;
                float* dst = a.part_acc + idx * DV;
#pragma unroll 1
                for (int c0 = half * (DV / 2); c0 < (half + 1) * (DV / 2); c0 += 32) {
                    uint32_t rr[32];
                    tc::tmem_ld_32x32(tmem_o + lane_base + c0, rr);
                    tc::tmem_ld_wait();
                    if (mine) {
#pragma unroll
                        for (int jj = 0; jj < 32; jj += 4)
                            *reinterpret_cast<uint4*>(dst + c0 + jj) = make_uint4(rr[jj], rr[jj + 1], rr[jj + 2], rr[jj + 3]);
                    }
                }
                if (mine && half == 0) {
                    const float l = l_run + s_l[1][row];
                    a.part_ml[idx * 2] = l > 0.f ? m_ref * 0.6931471805599453f : -3.0e38f;
                    a.part_ml[idx * 2 + 1] = l;
                }
            }
        } else {
        if (ok) {
            tc::fence_after_sync();
            float l = l_run + s_l[half ^ 1][row];
            if (a.opt.sink != nullptr) l += ex2_approx(fmaf(a.opt.sink[h], 1.4426950408889634f, -m_ref));
            float inv = l > 0.f ? 1.f / l : 0.f;
            if (a.gate != nullptr && a.opt.gate_per_head && row < nq)
                inv *= sigmoid_f(bf16_to_f32(a.gate[(size_t)(row_start + r_begin + row) * a.ld_gate + (size_t)h * a.gate_head_stride + a.gate_offset]));
            __nv_bfloat16* stg = reinterpret_cast<__nv_bfloat16*>(smem) + row * kTcOutPitch;
#pragma unroll 1
            for (int c0 = half * (DV / 2); c0 < (half + 1) * (DV / 2); c0 += 32) {
                uint32_t r[32];
                tc::tmem_ld_32x32(tmem_o + lane_base + c0, r);
                tc::tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; j += 8) {
                    uint32_t w[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        w[e] = f32x2_to_bf16x2_bits(__uint_as_float(r[j + 2 * e]) * inv, __uint_as_float(r[j + 2 * e + 1]) * inv);
                    *reinterpret_cast<uint4*>(stg + c0 + j) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        }
        if (cta_stamp) a.prof[4 * 16 + 15] = clock64();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (cta_stamp) a.prof[5 * 16 + 15] = clock64();
        if (ok) {
            // 16-byte pieces, four per thread and pass so that the gate loads of a pass are in flight together
            const __nv_bfloat16* stg0 = reinterpret_cast<const __nv_bfloat16*>(smem);
            const int n_items = nq * (DV / 8);
            const bool elementwise = a.gate != nullptr && !a.opt.gate_per_head;
            for (int i0 = (int)threadIdx.x; i0 < n_items; i0 += 8 * kTcRows) {
                uint4 g[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const int i = i0 + u * 2 * kTcRows;
                    g[u] = make_uint4(0, 0, 0, 0);
                    if (elementwise && i < n_items)
                        g[u] = __ldg(reinterpret_cast<const uint4*>(a.gate + (size_t)(row_start + r_begin + i / (DV / 8)) * a.ld_gate +
                                                                    (size_t)h * a.gate_head_stride + a.gate_offset + i % (DV / 8) * 8));
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    const int i = i0 + u * 2 * kTcRows;
                    if (i >= n_items) break;
                    const int r = i / (DV / 8), c = i % (DV / 8);
                    uint4 v = *reinterpret_cast<const uint4*>(stg0 + r * kTcOutPitch + c * 8);
                    if (elementwise) {
                        const uint32_t vw[4] = {v.x, v.y, v.z, v.w}, gw[4] = {g[u].x, g[u].y, g[u].z, g[u].w};
                        uint32_t o[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float2 vv = bf16x2_bits_to_f32x2(vw[e]), gg = bf16x2_bits_to_f32x2(gw[e]);
                            o[e] = f32x2_to_bf16x2_bits(vv.x * sigmoid_fast(gg.x), vv.y * sigmoid_fast(gg.y));
                        }
                        v = make_uint4(o[0], o[1], o[2], o[3]);
                    }
                    *reinterpret_cast<uint4*>(a.out + ((size_t)(row_start + r_begin + r) * a.Hq + h) * DV + c * 8) = v;
                }
            }
        }
        }   // prefill epilogue
    }
    if (cta_stamp) a.prof[6 * 16 + 15] = clock64();
    tc::fence_before_sync();
    __syncthreads();
    if (threadIdx.x == 0) {
        if (s_bad != 0) set_status(a.status, PS_DEV_BAD_INDEX);
        if (s_abort != 0) {
            set_status(a.status, PS_DEV_WAIT_TIMEOUT);
            // copies still in flight get a bounded chance to land before the shared memory goes back to the next CTA
            const long long bd = a.budget < 4000000ll ? a.budget : 4000000ll;
            if (q_issued > q_consumed) tc::mbar_wait(&q_full, 0, bd);
            for (int c = k_consumed; c < k_issued; ++c) tc::mbar_wait(&k_full[c & kStageMask], (uint32_t)(c >> kStageLog) & 1u, bd);
            for (int c = v_consumed; c < v_issued; ++c) tc::mbar_wait(&v_full[c & 1], (uint32_t)(c >> 1) & 1u, bd);
        }
    }
    __syncthreads();
    if (cta_stamp) a.prof[16 + 15] = clock64();
    if (warp == 12) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem, kTcTmemCols);
    }
}

typedef CUresult (*EncodeTiledFnA)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                   const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                   CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static EncodeTiledFnA attn_encode_fn() {
    static EncodeTiledFnA fn = nullptr;
    if (fn == nullptr) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult qres;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &qres) == cudaSuccess &&
            qres == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<EncodeTiledFnA>(p);
    }
    return fn;
}

// bf16 row-major [rows, cols] (leading dimension in elements) with a (box_rows x 64) box and the 128-byte swizzle.
static int attn_map_2d(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint64_t ld_elems, uint32_t box_rows) {
    EncodeTiledFnA enc = attn_encode_fn();
    if (enc == nullptr) return (int)cudaErrorNotSupported;
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {ld_elems * 2};
    const cuuint32_t box[2] = {64, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                     CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                     CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : (int)cudaErrorInvalidValue;
}

template <int DK, int DV, bool DEC, bool SHARED, bool TRANSFORM, bool EXPANDED>
static int launch_attn_tc(dim3 grid, const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const CUtensorMap& mr,
                          const AttnTcArgs& a, cudaStream_t stream) {
    constexpr size_t smem = TcShape<DK, DV>::kSmem;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(attn_tc_kernel<DK, DV, DEC, SHARED, TRANSFORM, EXPANDED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        set = true;
    }
    attn_tc_kernel<DK, DV, DEC, SHARED, TRANSFORM, EXPANDED><<<grid, kTcThreads, smem, stream>>>(mq, mk, mv, mr, a);
    return PS_LAUNCH_CHECK();
}

}  // namespace ps
