// Latent attention for decode rows and short portions, in the latent space: all heads share the cached rows [latent | rotated
// part] as keys, and the latent part as values (bf16 pool, one head per token, pages of 16, 32 or 64 tokens).
//
// One CTA = up to 128 (row, head) pairs of one sequence as one MMA tile (fewer with wide rows: two tiles of the ring come first) --
// tile row r * hp + g is head g of the CTA's row r; rows beyond the used ones read whatever lies behind the queries in shared
// memory, and nobody reads their results --, one KV split, and up to 256 of the value columns (tensor memory holds four score
// accumulators and 256 output columns; wider latents take two CTAs that both compute the scores):
//
//   warps 4-7 TMA producers: the queries once, then per tile of 64 tokens every 64-column group of the cached rows, once, into a
//            ring of 8 KB stages (a group is one box per page).  The groups that are this CTA's values come last.  Fills take
//            turns among the four warps (waiting, arming and issuing one costs several hundred cycles); the ring is a multiple
//            of four stages, so a stage always belongs to the same warp.
//   warps 8, 9 one thread each issues half of S(t) = sum_g Q_g K_g^T (every other group, as they land) into an accumulator of
//            its own, since issuing a product costs a thread more than the product itself; the softmax adds the two.  Two pairs
//            of accumulators take turns.  A group that is no value gives its stage back at once.
//   warp 10  one thread issues O_g += P(t) V_g for the value groups, still in their stages (an MN-major operand), and gives these
//            back.
//   warps 0-3 softmax: one thread per (row, head) with its window, reference maximum and sum in 32-bit; probabilities go to
//            shared memory as a bf16 operand; the output accumulator is rescaled only when the maximum has grown by 2^8.
//
// The result is a partial output per (row, head, split) in the layout of paged_attention.cu's merge pass, splits counted from
// position 0 and kept in a ring, since a row of a windowed sequence sees only a few of them.  Which tokens form a split does not
// depend on the batch.  Every wait is bounded; a timeout unwinds all roles as in attn_tc.cuh.
#include "attn_tc.cuh"

namespace ps {

constexpr int kLdThreads = 352, kLdProducers = 4, kLdGroup = kTcTok * 64 * 2, kLdMaxStages = 24;

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
    __shared__ __align__(8) uint64_t q_full, full[kLdMaxStages], freed[kLdMaxStages], s_full[2], s_free[2], p_full[2], pv_done[2];
    __shared__ uint32_t tmem_slot;
    __shared__ int s_abort, s_bad, s_fills[kLdMaxStages], q_issued;

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
    unsigned char* sP = sQ + (size_t)ng * a.q_group;             // two buffers of the used rows x 64 tokens
    unsigned char* sS = sP + 2 * a.q_group;

    if (threadIdx.x == 0) {
        tc::mbar_init(&q_full, 1);
        for (int s = 0; s < ns; ++s) { tc::mbar_init(&full[s], 1); tc::mbar_init(&freed[s], 1); }
        for (int s = 0; s < 2; ++s) {
            tc::mbar_init(&s_full[s], 2); tc::mbar_init(&s_free[s], 4); tc::mbar_init(&p_full[s], 4); tc::mbar_init(&pv_done[s], 1);
        }
        tc::fence_barrier_init();
        for (int s = 0; s < ns; ++s) s_fills[s] = 0;
        s_abort = 0; s_bad = 0; q_issued = 0;
        tc::tma_prefetch_desc(&map_q); tc::tma_prefetch_desc(&map_kv);
    }
    if (warp == 10) {
        tc::tmem_alloc(&tmem_slot, 512);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem = tmem_slot, tmem_o = tmem + 256;
    cudaGridDependencySynchronize();

    // group of the cached row that comes i-th in a tile: values last
    auto group_at = [&](int i) { return i < 4 * vp ? i : i < ng - nv ? i + nv : 4 * vp + i - (ng - nv); };
    if (warp >= 4 && warp < 4 + kLdProducers) {
        // ------------------------------------------------ producers
        if (warp == 4) {
            const int blocks = (nh + 7) / 8;                                      // boxes of 8 heads per row and group
            const int n_box = nr * blocks * ng;
            if (lane == 0) tc::mbar_expect_tx(&q_full, (uint32_t)n_box * 1024u);
            __syncwarp();
            for (int i = lane; i < n_box; i += 32) {
                const int g = i % ng, rb = i / ng, r = rb / blocks, b8 = rb % blocks;
                tc::tma_load_2d(sQ + (size_t)g * a.q_group + (r * a.hp + 8 * b8) * 128, &map_q, g * 64,
                                (row_start + r0 + r) * a.H + h0 + 8 * b8, &q_full);
            }
            if (lane == 0) q_issued = 1;
        }
        const int* bt = a.block_table + (size_t)slot * a.max_blocks;
        const int pt = a.page_tokens, ppt = kTcTok / pt;
        auto page_of = [&](int t) {                                               // this lane's page of tile t
            const int blk = (t_first + t) * ppt + lane;
            if (t >= T || lane >= ppt || blk * pt >= kv_end) return 0;
            const int page = bt[blk];
            if (page < 0 || page >= a.num_pages) { s_bad = 1; return 0; }
            return page;
        };
        int i = warp - 4, st = warp - 4, fill = 0, t = 0;
        while (i >= ng) { i -= ng; ++t; }
        int page = page_of(t), next = page_of(t + 1);
        while (t < T) {
            if (fill > 0 && !__all_sync(0xffffffffu, tc::mbar_wait_abortable(&freed[st], (uint32_t)(fill - 1) & 1u, a.budget, &s_abort))) break;
            if (lane == 0) tc::mbar_expect_tx(&full[st], kLdGroup);
            __syncwarp();
            if (lane < ppt) tc::tma_load_2d(sS + st * kLdGroup + lane * (pt * 128), &map_kv, group_at(i) * 64, page * pt, &full[st]);
            if (lane == 0) s_fills[st] = fill + 1;
            st += kLdProducers;
            if (st >= ns) { st -= ns; ++fill; }
            i += kLdProducers;
            while (i >= ng) { i -= ng; ++t; page = next; next = page_of(t + 1); }
        }
    } else if (warp == 8 || warp == 9) {
        // ------------------------------------------------ scores
        if (lane == 0) {
            constexpr uint32_t idesc = tc::idesc_bf16_f32(kTcRows, kTcTok);
            const uint32_t q_addr = tc::smem_u32(sQ), s_addr = tc::smem_u32(sS);
            bool ok = tc::mbar_wait_abortable(&q_full, 0, a.budget, &s_abort);
            const int mine = warp - 8;
            int st0 = 0;                                                          // stage and phase of the tile's first group
            uint32_t ph0 = 0;
            for (int t = 0; t < T && ok; ++t) {
                const int b = t & 1;
                const uint32_t acc = tmem + b * (2 * kTcTok) + mine * kTcTok;
                // The accumulators are free once the softmax warps have read S(t - 2).  The same wait keeps the ones below from
                // beginning before a stage's last fill has landed (the parity would read as done): the ring holds two tiles, so a
                // fill of tile t replaces one of tile t - 2 or earlier.
                if (t >= 2 && !tc::mbar_wait_abortable(&s_free[b], ((uint32_t)(t >> 1) & 1u) ^ 1u, a.budget, &s_abort)) break;
                for (int i = mine; i < ng; i += 2) {
                    const int st = st0 + i < ns ? st0 + i : st0 + i - ns;
                    if (!tc::mbar_wait_abortable(&full[st], st0 + i < ns ? ph0 : ph0 ^ 1u, a.budget, &s_abort)) { ok = false; break; }
                    tc::fence_after_sync();
                    const uint32_t qa = q_addr + group_at(i) * a.q_group, ka = s_addr + st * kLdGroup;
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)
                        tc::mma_bf16_ss(acc, tc::smem_desc_sw128(qa + kk * 32), tc::smem_desc_sw128(ka + kk * 32), idesc,
                                        (i > mine || kk > 0) ? 1u : 0u);
                    if (i < ng - nv) tc::mma_commit(&freed[st]);
                }
                if (ok) tc::mma_commit(&s_full[b]);
                st0 += ng;
                while (st0 >= ns) { st0 -= ns; ph0 ^= 1u; }
            }
        }
    } else if (warp == 10) {
        // ------------------------------------------------ outputs
        if (lane == 0) {
            const uint32_t idesc_all = tc::idesc_bf16_f32_bmn(kTcRows, 64 * nv);
            constexpr uint32_t idesc_one = tc::idesc_bf16_f32_bmn(kTcRows, 64);
            const uint32_t p_addr = tc::smem_u32(sP), s_addr = tc::smem_u32(sS);
            int st = ng - nv;
            uint32_t ph = 0;
            while (st >= ns) { st -= ns; ph ^= 1u; }
            for (int t = 0; t < T; ++t) {
                const int b = t & 1;
                if (!tc::mbar_wait_abortable(&p_full[b], (uint32_t)(t >> 1) & 1u, a.budget, &s_abort)) break;
                const uint32_t pa = p_addr + b * a.q_group;
                const bool together = st + nv <= ns;                              // the value groups' stages follow one another: one wide product
                const int first = st;
                bool ok = true;
                for (int j = 0; j < nv && ok; ++j) {
                    ok = tc::mbar_wait_abortable(&full[st], ph, a.budget, &s_abort);                  // landed: S(t) has read it
                    if (!ok) break;
                    tc::fence_after_sync();
                    if (!together || j == nv - 1) {
                        const uint32_t va = s_addr + (together ? first : st) * kLdGroup, o = tmem_o + (together ? 0 : j * 64);
#pragma unroll
                        for (int kk = 0; kk < kTcTok / 16; ++kk)
                            tc::mma_bf16_ss(o, tc::smem_desc_sw128(pa + kk * 32), tc::smem_desc_sw128_mn(va + kk * (16 * 128), kTcTok * 128, 1024),
                                            together ? idesc_all : idesc_one, (t > 0 || kk > 0) ? 1u : 0u);
                        if (together) { for (int k = first; k < first + nv; ++k) tc::mma_commit(&freed[k]); }
                        else tc::mma_commit(&freed[st]);
                    }
                    if (++st == ns) { st = 0; ph ^= 1u; }
                }
                if (!ok) break;
                tc::mma_commit(&pv_done[b]);
                st += ng - nv;
                while (st >= ns) { st -= ns; ph ^= 1u; }
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
            uint32_t pk[32], s0[32], s1[32];
            if (live) {
                const uint32_t acc = tmem + lane_base + b * (2 * kTcTok);
                uint32_t h[32];
                tc::tmem_ld_32x32(acc, s0);
                tc::tmem_ld_32x32(acc + kTcTok, h);
                tc::tmem_ld_32x32(acc + 32, s1);
                tc::tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; ++j) s0[j] = __float_as_uint(__uint_as_float(s0[j]) + __uint_as_float(h[j]));
                tc::tmem_ld_32x32(acc + kTcTok + 32, h);
                tc::tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 32; ++j) s1[j] = __float_as_uint(__uint_as_float(s1[j]) + __uint_as_float(h[j]));
                tc::fence_before_sync();
            }
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&s_free[b]);                           // the accumulators may take S(t + 2)
            if (live) {
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
            const bool rescale = t >= 1 && __any_sync(0xffffffffu, alpha != 1.f);
            if (t >= 2) {                                                         // P V(t - 2) has read this buffer
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[b], (uint32_t)((t - 2) >> 1) & 1u, a.budget, &s_abort));
                if (!ok) break;
            }
            if (row * 128 < a.q_group) {                                          // (rows behind the used ones have no place)
                unsigned char* prow = sP + b * a.q_group + row * 128;
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
            if (rescale) {                                                        // O must be complete up to P V(t - 1)
                ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&pv_done[b ^ 1], (uint32_t)((t - 1) >> 1) & 1u, a.budget, &s_abort));
                if (!ok) break;
                tc::fence_after_sync();
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
            if (q_issued) tc::mbar_wait(&q_full, 0, bd);
            for (int s = 0; s < ns; ++s)
                if (s_fills[s] > 0) tc::mbar_wait(&full[s], (uint32_t)(s_fills[s] - 1) & 1u, bd);
        }
    }
    __syncthreads();
    if (warp == 10) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem, 512);
    }
}

constexpr int kLdSmem = 225 * 1024;              // of the 227 KB; the rest is the static part

// Query rows (a multiple of 8) that leave room for a ring of two tiles: they take ng query groups and two probability buffers.
static int latent_decode_rows(int ng) {
    const int ring = (2 * ng + kLdProducers - 1) / kLdProducers * kLdProducers;
    const int rows = (kLdSmem - ring * kLdGroup) / (128 * (ng + 2)) / 8 * 8;
    return rows > kTcRows ? kTcRows : rows;
}
static int latent_decode_stages(int ng, int rows) {
    const int n = (kLdSmem - (ng + 2) * rows * 128) / kLdGroup / kLdProducers * kLdProducers;
    return n > kLdMaxStages ? kLdMaxStages : n;
}
struct LatentDecodeTile { int heads, hp, rows, row_tiles, head_tiles; };
static LatentDecodeTile latent_decode_tile(int H, int ng, int max_rows) {
    LatentDecodeTile t;
    const int room = latent_decode_rows(ng);
    t.head_tiles = (H + room - 1) / room;
    t.heads = (H + t.head_tiles - 1) / t.head_tiles;
    t.hp = (t.heads + 7) / 8 * 8;
    t.rows = room / t.hp < max_rows ? room / t.hp : max_rows;
    t.row_tiles = (max_rows + t.rows - 1) / t.rows;
    return t;
}

}  // namespace ps

// Whether a cached row of KR + R elements fits the kernel (a ring of two tiles beside at least eight query rows).
PS_API int ps_latent_decode_ok(int KR, int R, int page_tokens) {
    return KR > 0 && R > 0 && KR % 64 == 0 && R % 64 == 0 && (page_tokens == 16 || page_tokens == 32 || page_tokens == 64) &&
           2 * ((KR + R) / 64) <= ps::kLdMaxStages && ps::latent_decode_rows((KR + R) / 64) >= 8;
}

// CTAs of one split (value parts x head tiles x row tiles of `max_rows` rows) per sequence: what a caller sizes splits with.
PS_API int ps_latent_decode_ctas(int H, int KR, int R, int max_rows) {
    const ps::LatentDecodeTile t = ps::latent_decode_tile(H, (KR + R) / 64, max_rows);
    return t.head_tiles * t.row_tiles * ((KR / 64 + 3) / 4);
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
        split_tokens % kTcTok || splits < 1 || ring < 1 || splits > ring || !attn_options_ok(opt) || opt.keep_first > 0 || attn_transforms_scores(opt) || !(scale > 0.f) ||
        (((uintptr_t)q | (uintptr_t)pool | (uintptr_t)part_acc) % 16))
        return (int)cudaErrorInvalidValue;
    LatentDecodeArgs a;
    a.block_table = (const int*)block_table; a.max_blocks = max_blocks; a.num_pages = num_pages; a.page_tokens = page_tokens;
    a.seqs = (const int*)seqs; a.H = H;
    a.ng = (KR + R) / 64; a.krg = KR / 64;
    const LatentDecodeTile tile = latent_decode_tile(H, a.ng, max_rows);
    a.head_tiles = tile.head_tiles; a.heads_per_tile = tile.heads; a.hp = tile.hp; a.rows_per_tile = tile.rows; a.row_tiles = tile.row_tiles;
    a.q_group = tile.rows * tile.hp * 128;
    a.stages = latent_decode_stages(a.ng, tile.rows * tile.hp);
    a.scale_log2 = scale * 1.4426950408889634f; a.opt = opt; a.split_tokens = split_tokens; a.ring = ring; a.max_rows = max_rows;
    a.part_acc = (float*)part_acc; a.part_ml = (float*)part_ml; a.status = (uint32_t*)status; a.budget = g_ps_wait_budget_cycles;
    CUtensorMap mq, mkv;
    int err = attn_map_2d(&mq, q, (uint64_t)q_rows * H, (uint64_t)(KR + R), (uint64_t)(KR + R), 8);
    if (err) return err;
    if ((err = attn_map_2d(&mkv, pool, (uint64_t)num_pages * page_tokens, (uint64_t)(KR + R), (uint64_t)(KR + R), (uint32_t)page_tokens))) return err;
    const size_t smem = (size_t)(a.ng + 2) * a.q_group + (size_t)a.stages * kLdGroup;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(attn_latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kLdSmem);
        attr_set = true;
    }
    const int vparts = (a.krg + 3) / 4;
    return launch_pdl(attn_latent_decode_kernel, dim3(splits, vparts * a.head_tiles, n_seqs * a.row_tiles), dim3(kLdThreads), smem, stream, mq, mkv, a);
}
