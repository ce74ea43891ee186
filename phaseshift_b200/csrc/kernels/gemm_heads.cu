// One small projection per head: out[m, h, n] = sum_k x[m, h, k] W[h, n, k], optionally times sigmoid(gate[m, h, n]) -- the
// products that take queries of a latent attention into the latent space and its outputs back to the heads.
//
// Operands are swapped as in gemm_smallm.cu: 128 weight rows are the M side of `tcgen05.mma`, up to 64 rows of x the N side, so
// the stages hold mostly weights.  One CTA per (128 weight rows, head, 64 rows); K (64 to 512 here) runs through a four-stage TMA
// ring and the accumulator in tensor memory goes straight to the output, lane = weight row.  The weight tiles of the first stages
// are requested before the predecessor kernel has finished (programmatic dependent launch).  Every wait is bounded.
//
// With `turn_r`, one more CTA per head and 64 rows copies the rotated part of x's head (behind its K columns) behind the head's
// outputs, turned by the row's position, so that the latent queries leave this kernel complete.
#include "ps_tcgen05.cuh"
#include "turn_angle.cuh"

namespace ps {

constexpr int kGhM = 128, kGhRows = 64, kGhK = 64, kGhStages = 4, kGhThreads = 192;

struct GemmHeadsArgs {
    int M, N, K, x_head;         // rows, outputs and inputs per head, columns of x between heads
    int nb, box_rows;            // MMA N; rows of an x box
    __nv_bfloat16* out; int ldo, o_head;
    const __nv_bfloat16* gate; int ldg, g_head;
    int turn_r, turn_pairs; const double* inv_freq; const int* row_pos; const __nv_bfloat16* x; int ldx;
    uint32_t* status; long long budget;
};

__global__ void __launch_bounds__(kGhThreads, 2)
gemm_heads_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const GemmHeadsArgs g) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    constexpr int kW = kGhM * kGhK * 2, kX = kGhRows * kGhK * 2;
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    unsigned char* sW = smem;
    unsigned char* sX = smem + kGhStages * kW;
    __shared__ __align__(8) uint64_t full[kGhStages], empty[kGhStages], acc_bar;
    __shared__ uint32_t tmem_slot;
    __shared__ int s_abort, s_issued, s_consumed;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = blockIdx.x * kGhM, h = blockIdx.y, m0 = blockIdx.z * kGhRows, iters = g.K / kGhK;

    cudaTriggerProgrammaticLaunchCompletion();
    if (g.turn_r > 0 && blockIdx.x == gridDim.x - 1) {
        cudaGridDependencySynchronize();
        const int half = g.turn_r / 2;
        for (int i = threadIdx.x; i < min(kGhRows, g.M - m0) * half; i += kGhThreads) {
            const int m = m0 + i / half, j = i % half;
            const float2 v = bf16x2_bits_to_f32x2(*reinterpret_cast<const uint32_t*>(g.x + (size_t)m * g.ldx + (size_t)h * g.x_head + g.K + 2 * j));
            float s = 0.f, c = 1.f;
            if (j < g.turn_pairs) turn_angle(max(g.row_pos[m], 0), g.inv_freq[j], &s, &c);
            *reinterpret_cast<uint32_t*>(g.out + (size_t)m * g.ldo + (size_t)h * g.o_head + g.N + 2 * j) = f32x2_to_bf16x2_bits(v.x * c - v.y * s, v.y * c + v.x * s);
        }
        return;
    }
    if (threadIdx.x == 0) {
        for (int s = 0; s < kGhStages; ++s) { tc::mbar_init(&full[s], 1); tc::mbar_init(&empty[s], 1); }
        tc::mbar_init(&acc_bar, 1);
        tc::fence_barrier_init();
        s_abort = 0; s_issued = 0; s_consumed = 0;
        tc::tma_prefetch_desc(&map_w); tc::tma_prefetch_desc(&map_x);
    }
    if (warp == 1) {
        tc::tmem_alloc(&tmem_slot, 64);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem = tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            const int early = min(iters, kGhStages);
            const uint32_t bytes = kW + g.box_rows * kGhK * 2;
            for (int it = 0; it < early; ++it) {
                tc::mbar_expect_tx(&full[it], bytes);
                tc::tma_load_2d(sW + it * kW, &map_w, it * kGhK, h * g.N + n0, &full[it]);
            }
            cudaGridDependencySynchronize();
            for (int it = 0; it < iters; ++it) {
                const int s = it % kGhStages;
                if (it >= kGhStages) {
                    if (!tc::mbar_wait_abortable(&empty[s], (uint32_t)((it - kGhStages) / kGhStages) & 1u, g.budget, &s_abort)) break;
                    tc::mbar_expect_tx(&full[s], bytes);
                    tc::tma_load_2d(sW + s * kW, &map_w, it * kGhK, h * g.N + n0, &full[s]);
                }
                tc::tma_load_2d(sX + s * kX, &map_x, h * g.x_head + it * kGhK, m0, &full[s]);
                s_issued = it + 1;
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = tc::idesc_bf16_f32(kGhM, g.nb);
            for (int it = 0; it < iters; ++it) {
                const int s = it % kGhStages;
                if (!tc::mbar_wait_abortable(&full[s], (uint32_t)(it / kGhStages) & 1u, g.budget, &s_abort)) break;
                s_consumed = it + 1;
                tc::fence_after_sync();
                const uint32_t w = tc::smem_u32(sW + s * kW), x = tc::smem_u32(sX + s * kX);
#pragma unroll
                for (int kk = 0; kk < kGhK / 16; ++kk)
                    tc::mma_bf16_ss(tmem, tc::smem_desc_sw128(w + kk * 32), tc::smem_desc_sw128(x + kk * 32), idesc, (it > 0 || kk > 0) ? 1u : 0u);
                tc::mma_commit(&empty[s]);
            }
            tc::mma_commit(&acc_bar);
        }
    } else {
        cudaGridDependencySynchronize();                 // the gate, and the readers of the previous contents of `out`
        const int quad = warp & 3, n = n0 + quad * 32 + lane, rows = min(kGhRows, g.M - m0);
        // the gate values of 16 rows at once, asked for before the accumulator is waited for
        float gate[16];
        auto load_gate = [&](int c0) {
#pragma unroll
            for (int j = 0; j < 16; ++j)
                gate[j] = c0 + j < rows && n < g.N ? bf16_to_f32(g.gate[(size_t)(m0 + c0 + j) * g.ldg + (size_t)h * g.g_head + n]) : 0.f;
        };
        if (g.gate != nullptr) load_gate(0);
        const bool done = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&acc_bar, 0, g.budget, &s_abort));
        tc::fence_after_sync();
        if (done && s_abort == 0) {
            for (int c0 = 0; c0 < g.nb; c0 += 16) {
                uint32_t r[16];
                tc::tmem_ld_32x16(tmem + ((uint32_t)(quad * 32) << 16) + (uint32_t)c0, r);
                tc::tmem_ld_wait();
                if (g.gate != nullptr) {
#pragma unroll
                    for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * sigmoid_f(gate[j]));
                    if (c0 + 16 < g.nb) load_gate(c0 + 16);
                }
#pragma unroll
                for (int j = 0; j < 16; ++j)
                    if (c0 + j < rows && n < g.N) g.out[(size_t)(m0 + c0 + j) * g.ldo + (size_t)h * g.o_head + n] = f32_to_bf16(__uint_as_float(r[j]));
            }
        }
    }
    tc::fence_before_sync();
    __syncthreads();
    if (s_abort != 0 && threadIdx.x == 0) {
        set_status(g.status, PS_DEV_WAIT_TIMEOUT);
        // copies still in flight get a bounded chance to land before the shared memory goes back to the next CTA
        const long long b = g.budget < 4000000ll ? g.budget : 4000000ll;
        for (int c = s_consumed; c < s_issued; ++c) tc::mbar_wait(&full[c % kGhStages], (uint32_t)(c / kGhStages) & 1u, b);
    }
    __syncthreads();
    if (warp == 1) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem, 64);
    }
}

typedef CUresult (*GhEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                               const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static int gh_map_2d(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows) {
    static GhEncodeFn enc = nullptr;
    if (enc == nullptr) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
            enc = reinterpret_cast<GhEncodeFn>(p);
        if (enc == nullptr) return (int)cudaErrorNotSupported;
    }
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kGhK, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
               ? 0 : (int)cudaErrorInvalidValue;
}

}  // namespace ps

// x [M, ldx] bf16, head h at column h * x_head; w [heads * N, K] bf16 row-major; out [M, ldo], head h at column h * o_head; gate
// (optional) likewise.  K, x_head multiples of 64, ldx of 8, 16-byte aligned bases.  `turn_r` > 0 columns behind each head's K are
// turned by the row's position (pairs of neighbours, `inv_freq` f64 radians per position) and stored behind its N outputs.
PS_API int ps_gemm_heads(const void* x, int ldx, int x_head, const void* w, int heads, int M, int N, int K, const void* gate, int ldg,
                         int g_head, void* out, int ldo, int o_head, int turn_r, int turn_pairs, const void* inv_freq, const void* row_pos,
                         void* status, cudaStream_t stream) {
    using namespace ps;
    if (heads <= 0 || heads > 65535 || M <= 0 || N <= 0 || K <= 0 || K % kGhK || x_head % kGhK || ldx % 8 || ldx < (heads - 1) * x_head + K + turn_r ||
        turn_r < 0 || (turn_r & 1) || 2 * turn_pairs > turn_r || (turn_r > 0 && ((ldo | o_head | N) & 1)) ||
        (((uintptr_t)x | (uintptr_t)w) % 16))
        return (int)cudaErrorInvalidValue;
    GemmHeadsArgs g;
    g.M = M; g.N = N; g.K = K; g.x_head = x_head; g.out = (__nv_bfloat16*)out; g.ldo = ldo; g.o_head = o_head;
    const int rows = M < kGhRows ? M : kGhRows;
    g.nb = rows <= 16 ? 16 : rows <= 32 ? 32 : 64;
    g.box_rows = (rows + 7) / 8 * 8;
    g.gate = (const __nv_bfloat16*)gate; g.ldg = ldg; g.g_head = g_head; g.status = (uint32_t*)status; g.budget = g_ps_wait_budget_cycles;
    g.turn_r = turn_r; g.turn_pairs = turn_pairs; g.inv_freq = (const double*)inv_freq; g.row_pos = (const int*)row_pos;
    g.x = (const __nv_bfloat16*)x; g.ldx = ldx;
    CUtensorMap mw, mx;
    int err = gh_map_2d(&mw, w, (uint64_t)heads * N, (uint64_t)K, (uint64_t)K, kGhM);
    if (err) return err;
    if ((err = gh_map_2d(&mx, x, (uint64_t)M, (uint64_t)ldx, (uint64_t)ldx, (uint32_t)g.box_rows))) return err;
    const size_t smem = (size_t)kGhStages * (kGhM + kGhRows) * kGhK * 2 + 1024;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(gemm_heads_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        attr_set = true;
    }
    return launch_pdl(gemm_heads_kernel, dim3((N + kGhM - 1) / kGhM + (turn_r > 0 ? 1 : 0), heads, (M + kGhRows - 1) / kGhRows), dim3(kGhThreads), smem, stream,
                      mw, mx, g);
}
