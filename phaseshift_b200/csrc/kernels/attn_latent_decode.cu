// Latent attention for decode rows and short portions, in the latent space: all heads share the cached rows [latent | rotated
// part] as keys, and the latent part as values (bf16 pool, one head per token, pages of 16, 32 or 64 tokens).
//
// One CTA = up to 128 (row, head) pairs of one sequence as one MMA tile -- tile row r * hp + g is head g of the CTA's row r; rows
// beyond the used ones read whatever lies behind the queries in shared memory, and nobody reads their results --, one KV split, and up to 256 of the value columns (tensor memory holds 128 score columns and 256 output columns; wider latents
// take two CTAs that both compute the scores):
//
//   warp 4   TMA producer: the queries once, then per tile of 64 tokens every 64-column group of the cached rows, once, into a
//            ring of 8 KB stages (a group is one box per page).  The groups that are this CTA's values come last.
//   warps 5, 7 one thread each issues S(t) += Q_g K_g^T group by group as they land (tcgen05.mma) into one of two score
//            accumulators, warp 5 for even t and warp 7 for odd t (rings of fewer than two tiles: warp 5 for all); a group that
//            is no value gives its stage back at once.
//   warp 6   one thread issues O_g += P(t) V_g for the value groups, still in their stages (an MN-major operand), and gives these
//            back.
//   warps 0-3 softmax: one thread per (row, head) with its window, reference maximum and sum in 32-bit; probabilities go to
//            shared memory as a bf16 operand; the output accumulator is rescaled only when the maximum has grown by 2^8.
//
// The result is a partial output per (row, head, split) in the layout of paged_attention.cu's merge pass, splits counted from
// position 0 and kept in a ring, since a row of a windowed sequence sees only a few of them.  Which tokens form a split does not
// depend on the batch.  Every wait is bounded; a timeout unwinds all roles as in attn_tc.cuh.
#include "attn_tc.cuh"

namespace ps {

constexpr int kLdThreads = 256, kLdGroup = kTcTok * 64 * 2, kLdMaxStages = 24;

struct LatentDecodeArgs {
    const int* block_table; int max_blocks, num_pages, page_tokens;
    const int* seqs;             // [n_seqs][4] = row_start, n_rows, slot, pos_start
    int H, heads_per_tile, hp, rows_per_tile, row_tiles, head_tiles;
    int ng, krg;                 // 64-column groups of a cached row, of its latent
    int stages, q_group;         // stages of the ring; bytes of the queries' rows of one group
    float scale_log2; AttnOptions opt;
    int split_tokens, ring, max_rows;
    float* part_acc; float* part_ml;
    uint32_t* status; long long budget;
};

// grid = (splits, value parts * head tiles, sequences * row tiles)
__global__ void __launch_bounds__(kLdThreads, 1)
attn_latent_decode_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv, const LatentDecodeArgs a) {
    extern __shared__ __align__(1024) unsigned char smem[];
    __shared__ __align__(8) uint64_t q_full, full[kLdMaxStages], freed[kLdMaxStages], s_full[2], p_full[2], pv_done[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int s_abort, s_bad, s_issued, s_consumed, q_issued, q_consumed;

    const int vp = (int)blockIdx.y / a.head_tiles, ht = (int)blockIdx.y % a.head_tiles;
    const int seq = (int)blockIdx.z / a.row_tiles, r0 = ((int)blockIdx.z % a.row_tiles) * a.rows_per_tile;
    cudaTriggerProgrammaticLaunchCompletion();
    const int* sd = a.seqs + 4 * seq;            // the step's descriptors were uploaded before any kernel of the step
    const int row_start = sd[0], n_rows = sd[1], slot = sd[2], pos_start = sd[3];
    if (slot < 0 || n_rows <= r0 || n_rows > a.max_rows) { cudaGridDependencySynchronize(); return; }
    const int nr = min(a.rows_per_tile, n_rows - r0), pos0 = pos_start + r0, kv_end = pos0 + nr;
    const int h0 = ht * a.heads_per_tile, nh = min(a.heads_per_tile, a.H - h0);
    const int tps = a.split_tokens / kTcTok;
    const int t_lo = attn_first(a.opt, pos0) / kTcTok;
    const int split = t_lo / tps + (int)blockIdx.x;
    const int t_first = max(split * tps, t_lo), t_end = min((kv_end + kTcTok - 1) / kTcTok, (split + 1) * tps);
    if (t_first >= t_end) { cudaGridDependencySynchronize(); return; }
    const int T = t_end - t_first, ng = a.ng, ns = a.stages;
    const int nv = min(4, a.krg - 4 * vp);       // value groups of this CTA
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if ((tc::smem_u32(smem) & 1023u) != 0) {
        if (threadIdx.x == 0) set_status(a.status, PS_DEV_BAD_INDEX);
        return;
    }
    unsigned char* sQ = smem;                    // ng groups of the used rows x 64 columns (the MMA reads 128 rows from each)
    unsigned char* sP = sQ + (size_t)ng * a.q_group;
    unsigned char* sS = sP + kTcPBuf;

    if (threadIdx.x == 0) {
        tc::mbar_init(&q_full, 1);
        for (int s = 0; s < ns; ++s) { tc::mbar_init(&full[s], 1); tc::mbar_init(&freed[s], 1); }
        for (int s = 0; s < 2; ++s) { tc::mbar_init(&s_full[s], 1); tc::mbar_init(&p_full[s], 4); tc::mbar_init(&pv_done[s], 1); }
        tc::fence_barrier_init();
        s_abort = 0; s_bad = 0; s_issued = s_consumed = q_issued = q_consumed = 0;
        tc::tma_prefetch_desc(&map_q); tc::tma_prefetch_desc(&map_kv);
    }
    if (warp == 6) {
        tc::tmem_alloc(&tmem_slot, 512);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem = tmem_slot, tmem_o = tmem + 128;
    cudaGridDependencySynchronize();

    if (warp == 4) {
        // ------------------------------------------------ producer
        const int blocks = (nh + 7) / 8;                                          // boxes of 8 heads per row and group
        const int n_box = nr * blocks * ng;
        if (lane == 0) tc::mbar_expect_tx(&q_full, (uint32_t)n_box * 1024u);
        __syncwarp();
        for (int i = lane; i < n_box; i += 32) {
            const int g = i % ng, rb = i / ng, r = rb / blocks, b8 = rb % blocks;
            tc::tma_load_2d(sQ + (size_t)g * a.q_group + (r * a.hp + 8 * b8) * 128, &map_q, g * 64,
                            (row_start + r0 + r) * a.H + h0 + 8 * b8, &q_full);
        }
        if (lane == 0) q_issued = 1;
        const int* bt = a.block_table + (size_t)slot * a.max_blocks;
        const int pt = a.page_tokens, ppt = kTcTok / pt;
        int p = 0;
        bool ok = true;
        for (int t = 0; t < T && ok; ++t) {
            int page = 0;
            const int blk = (t_first + t) * ppt + lane;
            if (lane < ppt && blk * pt < kv_end) {
                page = bt[blk];
                if (page < 0 || page >= a.num_pages) { s_bad = 1; page = 0; }
            }
            for (int i = 0; i < ng; ++i, ++p) {
                const int st = p % ns;
                const int g = i < 4 * vp ? i : i < ng - nv ? i + nv : 4 * vp + i - (ng - nv);     // values last
                if (p >= ns) {
                    ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&freed[st], (uint32_t)(p / ns - 1) & 1u, a.budget, &s_abort));
                    if (!ok) break;
                }
                if (lane == 0) tc::mbar_expect_tx(&full[st], kLdGroup);
                __syncwarp();
                if (lane < ppt) tc::tma_load_2d(sS + st * kLdGroup + lane * (pt * 128), &map_kv, g * 64, page * pt, &full[st]);
                if (lane == 0) s_issued = p + 1;
            }
        }
    } else if (warp == 5 || warp == 7) {
        // ------------------------------------------------ scores
        if (lane == 0) {
            constexpr uint32_t idesc = tc::idesc_bf16_f32(kTcRows, kTcTok);
            const uint32_t q_addr = tc::smem_u32(sQ), s_addr = tc::smem_u32(sS);
            // A wait for a stage's next fill must not begin before its last one has landed (the parity would read as done).  A fill
            // of tile t replaces one of tile t - 2 or earlier in a ring of two tiles, and P(t - 2) has been waited for; a smaller
            // ring has one issuer, which takes the fills in order.
            const int issuers = ns >= 2 * ng ? 2 : 1;
            bool ok = (warp == 5 || issuers == 2) && tc::mbar_wait_abortable(&q_full, 0, a.budget, &s_abort);
            if (ok) q_consumed = 1;
            for (int t = warp == 5 ? 0 : 1; t < T && ok; t += issuers) {
                const int b = t & 1;
                // the accumulator is free once the softmax warps have read S(t - 2), which they signal with P(t - 2)
                if (t >= 2 && !tc::mbar_wait_abortable(&p_full[b], ((uint32_t)(t >> 1) & 1u) ^ 1u, a.budget, &s_abort)) break;
                for (int i = 0; i < ng; ++i) {
                    const int p = t * ng + i, st = p % ns;
                    const int g = i < 4 * vp ? i : i < ng - nv ? i + nv : 4 * vp + i - (ng - nv);
                    if (!tc::mbar_wait_abortable(&full[st], (uint32_t)(p / ns) & 1u, a.budget, &s_abort)) { ok = false; break; }
                    atomicMax(&s_consumed, p + 1);
                    tc::fence_after_sync();
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)
                        tc::mma_bf16_ss(tmem + b * kTcTok, tc::smem_desc_sw128(q_addr + g * a.q_group + kk * 32),
                                        tc::smem_desc_sw128(s_addr + st * kLdGroup + kk * 32), idesc, (i > 0 || kk > 0) ? 1u : 0u);
                    if (i < ng - nv) tc::mma_commit(&freed[st]);
                }
                if (ok) tc::mma_commit(&s_full[b]);
            }
        }
    } else if (warp == 6) {
        // ------------------------------------------------ outputs
        if (lane == 0) {
            constexpr uint32_t idesc = tc::idesc_bf16_f32_bmn(kTcRows, 64);
            const uint32_t p_addr = tc::smem_u32(sP), s_addr = tc::smem_u32(sS);
            for (int t = 0; t < T; ++t) {
                const int b = t & 1;
                if (!tc::mbar_wait_abortable(&p_full[b], (uint32_t)(t >> 1) & 1u, a.budget, &s_abort)) break;
                bool ok = true;
                for (int j = 0; j < nv && ok; ++j) {
                    const int p = t * ng + ng - nv + j, st = p % ns;
                    ok = tc::mbar_wait_abortable(&full[st], (uint32_t)(p / ns) & 1u, a.budget, &s_abort);      // landed: S(t) has read it
                    if (!ok) break;
                    tc::fence_after_sync();
#pragma unroll
                    for (int kk = 0; kk < kTcTok / 16; ++kk)
                        tc::mma_bf16_ss(tmem_o + j * 64, tc::smem_desc_sw128(p_addr + kk * 32),
                                        tc::smem_desc_sw128_mn(s_addr + st * kLdGroup + kk * (16 * 128), kTcTok * 128, 1024), idesc,
                                        (t > 0 || kk > 0) ? 1u : 0u);
                    tc::mma_commit(&freed[st]);
                }
                if (!ok) break;
                tc::mma_commit(&pv_done[b]);
            }
        }
    } else {
        // ------------------------------------------------ softmax: thread = tile row = TMEM lane
        const int row = warp * 32 + lane, r = row / a.hp, g = row % a.hp;
        const bool mine = r < nr && g < nh;
        const bool live = warp * 32 < nr * a.hp;                                  // warp-uniform: some lane may have work
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        const int rp = pos0 + min(r, nr - 1), lo = attn_first(a.opt, rp);
        const float sc = a.scale_log2;
        float m_ref = 0.f, l_run = 0.f;
        bool fresh = true, ok = true;
        for (int t = 0; t < T; ++t) {
            const int b = t & 1, tok0 = (t_first + t) * kTcTok;
            ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&s_full[b], (uint32_t)(t >> 1) & 1u, a.budget, &s_abort));
            if (!ok) break;
            tc::fence_after_sync();
            float alpha = 1.f;
            uint32_t pk[32];
            if (live) {
                uint32_t s0[32], s1[32];
                tc::tmem_ld_32x32(tmem + lane_base + b * kTcTok, s0);
                tc::tmem_ld_32x32(tmem + lane_base + b * kTcTok + 32, s1);
                tc::tmem_ld_wait();
                if (tok0 < lo || tok0 + kTcTok - 1 > rp) {
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        if (tok0 + j < lo || tok0 + j > rp) s0[j] = 0xff800000u;                    // -inf
                        if (tok0 + 32 + j < lo || tok0 + 32 + j > rp) s1[j] = 0xff800000u;
                    }
                }
                float mq[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int j = 0; j < 32; ++j) mq[j & 3] = fmaxf(mq[j & 3], fmaxf(__uint_as_float(s0[j]), __uint_as_float(s1[j])));
                const float mx = fmaxf(fmaxf(mq[0], mq[1]), fmaxf(mq[2], mq[3])) * sc;              // scale > 0
                if (fresh) {                                                      // (a row that sees nothing yet keeps a finite reference)
                    if (mx != -INFINITY) { m_ref = mx; fresh = false; }
                } else if (mx > m_ref + 8.f) { alpha = ex2_approx(m_ref - mx); m_ref = mx; }
                float sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int j = 0; j < 32; j += 2) {
                    const float a0 = ex2_approx(fmaf(__uint_as_float(s0[j]), sc, -m_ref)), a1 = ex2_approx(fmaf(__uint_as_float(s0[j + 1]), sc, -m_ref));
                    const float b0 = ex2_approx(fmaf(__uint_as_float(s1[j]), sc, -m_ref)), b1 = ex2_approx(fmaf(__uint_as_float(s1[j + 1]), sc, -m_ref));
                    sq[(j >> 1) & 3] += (a0 + a1) + (b0 + b1);
                    pk[j >> 1] = f32x2_to_bf16x2_bits(a0, a1);
                    pk[16 + (j >> 1)] = f32x2_to_bf16x2_bits(b0, b1);
                }
                l_run = l_run * alpha + ((sq[0] + sq[1]) + (sq[2] + sq[3]));
            }
            if (t >= 1) {                                                         // P V(t - 1) has read P, and O is complete up to it
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[b ^ 1], (uint32_t)((t - 1) >> 1) & 1u, a.budget, &s_abort));
                if (!ok) break;
                tc::fence_after_sync();
            }
            if (live) {
                unsigned char* prow = sP + row * 128;
#pragma unroll
                for (int c = 0; c < 8; ++c)
                    *reinterpret_cast<uint4*>(prow + ((c ^ (row & 7)) << 4)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
            }
            if (t == T - 1 && kv_end < tok0 + kTcTok) {
                // token rows behind the last one: zero them in the value groups (S(t) has read them; whole 128-byte rows)
                const int jz = kv_end - tok0, per = (kTcTok - jz) * 8;
                for (int i = (int)threadIdx.x; i < nv * per; i += kTcRows) {
                    const int st = (t * ng + ng - nv + i / per) % ns, k = i % per;
                    *reinterpret_cast<uint4*>(sS + st * kLdGroup + (jz + (k >> 3)) * 128 + (k & 7) * 16) = make_uint4(0, 0, 0, 0);
                }
            }
            tc::fence_proxy_async_smem();
            if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll 1
                for (int c0 = 0; c0 < nv * 64; c0 += 32) {
                    uint32_t o[32];
                    tc::tmem_ld_32x32(tmem_o + lane_base + c0, o);
                    tc::tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
                    tc::tmem_st_32x32(tmem_o + lane_base + c0, o);
                }
                tc::tmem_st_wait();
            }
            tc::fence_before_sync();
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&p_full[b]);
        }
        if (ok) ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[(T - 1) & 1], (uint32_t)((T - 1) >> 1) & 1u, a.budget, &s_abort));
        if (ok && live) {
            tc::fence_after_sync();
            const size_t idx = ((size_t)(row_start + r0 + (mine ? r : 0)) * a.H + h0 + (mine ? g : 0)) * a.ring + split % a.ring;
            float* dst = a.part_acc + idx * (size_t)(a.krg * 64) + vp * 256;
#pragma unroll 1
            for (int c0 = 0; c0 < nv * 64; c0 += 32) {
                uint32_t o[32];
                tc::tmem_ld_32x32(tmem_o + lane_base + c0, o);
                tc::tmem_ld_wait();
                if (mine) {
#pragma unroll
                    for (int j = 0; j < 32; j += 4) *reinterpret_cast<uint4*>(dst + c0 + j) = make_uint4(o[j], o[j + 1], o[j + 2], o[j + 3]);
                }
            }
            if (mine && vp == 0) {
                a.part_ml[idx * 2] = l_run > 0.f ? m_ref * 0.6931471805599453f : -3.0e38f;         // natural units, as the merge pass expects
                a.part_ml[idx * 2 + 1] = l_run;
            }
        }
    }
    tc::fence_before_sync();
    __syncthreads();
    if (threadIdx.x == 0) {
        if (s_bad != 0) set_status(a.status, PS_DEV_BAD_INDEX);
        if (s_abort != 0) {
            set_status(a.status, PS_DEV_WAIT_TIMEOUT);
            // copies still in flight get a bounded chance to land before the shared memory goes back to the next CTA
            const long long bd = a.budget < 4000000ll ? a.budget : 4000000ll;
            if (q_issued > q_consumed) tc::mbar_wait(&q_full, 0, bd);
            for (int c = s_consumed; c < s_issued; ++c) tc::mbar_wait(&full[c % ns], (uint32_t)(c / ns) & 1u, bd);
        }
    }
    __syncthreads();
    if (warp == 6) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem, 512);
    }
}

// Stages beside `rows` query rows per group; the 2 KB are the static part.
static int latent_decode_stages(int ng, int rows) {
    const int left = 227 * 1024 - 2048 - kTcPBuf - ng * rows * 128;
    const int n = left / kLdGroup;
    return n > kLdMaxStages ? kLdMaxStages : n;
}

}  // namespace ps

// Whether a cached row of KR + R elements fits the kernel (queries and at least two free stages beside the value groups).
PS_API int ps_latent_decode_ok(int KR, int R, int page_tokens) {
    return KR > 0 && R > 0 && KR % 64 == 0 && R % 64 == 0 && (page_tokens == 16 || page_tokens == 32 || page_tokens == 64) &&
           ps::latent_decode_stages((KR + R) / 64, ps::kTcRows) >= 6;
}

// CTAs of one split (value parts x head tiles x row tiles of `max_rows` rows) per sequence: what a caller sizes splits with.
PS_API int ps_latent_decode_ctas(int H, int KR, int max_rows) {
    const int ht = (H + 127) / 128, per = (H + ht - 1) / ht, hp = (per + 7) / 8 * 8, rpt = 128 / hp;
    return ht * ((KR / 64 + 3) / 4) * ((max_rows + rpt - 1) / rpt);
}

// q [q_rows, H, KR + R] bf16 (latent queries, turned rotated parts); partial outputs part_acc [q_rows, H, ring, KR] f32 and part_ml
// [q_rows, H, ring, 2] of every sequence with at most `max_rows` (<= 16) rows in the step; `splits` splits are launched from the
// one that holds the first visible token of a tile's first row on; ring >= the splits that a tile's rows see.  The caller
// runs ps_paged_attention_merge_ex with the same split length, ring and options.
PS_API int ps_latent_decode(const void* q, int q_rows, const void* pool, const void* block_table, int max_blocks, int page_tokens,
                            int num_pages, const void* seqs, int n_seqs, int max_rows, int H, int KR, int R, float scale, int split_tokens,
                            int splits, int ring, const void* options, void* part_acc, void* part_ml, void* status, cudaStream_t stream) {
    using namespace ps;
    const AttnOptions opt = attn_options(options);
    if (!ps_latent_decode_ok(KR, R, page_tokens) || q_rows <= 0 || n_seqs <= 0 || max_rows < 1 || max_rows > 16 || H <= 0 || split_tokens < kTcTok ||
        split_tokens % kTcTok || splits < 1 || ring < 1 || splits > ring || !attn_options_ok(opt) || attn_transforms_scores(opt) || !(scale > 0.f) ||
        (((uintptr_t)q | (uintptr_t)pool | (uintptr_t)part_acc) % 16))
        return (int)cudaErrorInvalidValue;
    LatentDecodeArgs a;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.num_pages = num_pages; a.page_tokens = page_tokens;
    a.seqs = (const int*)seqs; a.H = H;
    a.head_tiles = (H + kTcRows - 1) / kTcRows;
    a.heads_per_tile = (H + a.head_tiles - 1) / a.head_tiles;
    a.hp = (a.heads_per_tile + 7) / 8 * 8;
    a.rows_per_tile = kTcRows / a.hp < max_rows ? kTcRows / a.hp : max_rows;
    a.q_group = a.rows_per_tile * a.hp * 128;
    a.row_tiles = (max_rows + a.rows_per_tile - 1) / a.rows_per_tile;
    a.ng = (KR + R) / 64; a.krg = KR / 64; a.stages = latent_decode_stages(a.ng, a.rows_per_tile * a.hp);
    a.scale_log2 = scale * 1.4426950408889634f; a.opt = opt; a.split_tokens = split_tokens; a.ring = ring; a.max_rows = max_rows;
    a.part_acc = (float*)part_acc; a.part_ml = (float*)part_ml; a.status = (uint32_t*)status; a.budget = g_ps_wait_budget_cycles;
    CUtensorMap mq, mkv;
    int err = attn_map_2d(&mq, q, (uint64_t)q_rows * H, (uint64_t)(KR + R), (uint64_t)(KR + R), 8);
    if (err) return err;
    if ((err = attn_map_2d(&mkv, pool, (uint64_t)num_pages * page_tokens, (uint64_t)(KR + R), (uint64_t)(KR + R), (uint32_t)page_tokens))) return err;
    const size_t smem = (size_t)a.ng * a.q_group + kTcPBuf + (size_t)a.stages * kLdGroup;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(attn_latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024);
        attr_set = true;
    }
    const int vparts = (a.krg + 3) / 4;
    return launch_pdl(attn_latent_decode_kernel, dim3(splits, vparts * a.head_tiles, n_seqs * a.row_tiles), dim3(kLdThreads), smem, stream, mq, mkv, a);
}
