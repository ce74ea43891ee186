// Matrix products of a mixture of experts: out[r, :] = epilogue(W_e x[r, :]) for rows r sorted by expert, e the row's expert, over
// the tile list that moe_route.cu leaves.
//
// bf16: the operands are swapped relative to the plain prefill GEMM: 128 rows of the expert's weights are the M side of
// `tcgen05.mma`, up to NB sorted rows the N side, so that a tile with few rows (decode: every active expert has a handful)
// streams weights at full width and one with many is an ordinary tensor-core product.  Both operands come by TMA (128-byte swizzle,
// no multicast) into a ring; the accumulator (128 lanes = output features, NB columns = rows) lives in tensor memory.  The
// epilogue reads it with `tcgen05.ld`, a lane per feature: a gated activation (SwiGLU, or g sigmoid(1.702 g) (u + 1) with g and u
// limited) takes its (gate, up) pair from two neighbouring lanes, which share the work of two rows; stores of a warp are whole sectors.  Columns behind a tile's rows hold other experts' rows and are not
// stored.  Every wait is bounded (abort flag, bounded drain, tensor memory freed).
//
// 32-bit: the same list on the CUDA cores, 64 x 64 tiles.
#include "ps_tcgen05.cuh"

namespace ps {

constexpr int kMgM = 128, kMgK = 64, kMgThreads = 192;

struct MoeGemmArgs {
    const int* tiles;            // [0]: number of tiles; from [4] on (expert, first row, rows, 0)
    int N, K, gated;             // N: weight rows per expert; gated 0 store, 1 SwiGLU, 2 limited gate
    void* out; int ldo;          // gated: bf16 [rows, N / 2]; else fp32 [rows, N]
    float limit;
    uint32_t* status;
    long long budget;
};

__device__ __forceinline__ float mg_limited(float gate, float up, float limit) {
    const float g = fminf(gate, limit);
    return g / (1.f + expf(-1.702f * g)) * (fminf(fmaxf(up, -limit), limit) + 1.f);
}

// grid = (weight tiles, tiles of the list at most)
template <int NB, int STAGES>
__global__ void __launch_bounds__(kMgThreads, 2)
moe_gemm_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const MoeGemmArgs g) {
    extern __shared__ __align__(1024) unsigned char smem_raw[];
    constexpr int kWBytes = kMgM * kMgK * 2, kXBytes = NB * kMgK * 2;
    constexpr uint32_t kCols = NB < 32 ? 32 : NB;
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    if ((int)blockIdx.y >= g.tiles[0]) return;
    const int4 tile = reinterpret_cast<const int4*>(g.tiles)[1 + blockIdx.y];
    unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    unsigned char* sW = smem;
    unsigned char* sX = smem + STAGES * kWBytes;
    __shared__ __align__(8) uint64_t full_bar[STAGES], empty_bar[STAGES], acc_bar;
    __shared__ uint32_t tmem_base_slot;
    __shared__ int s_abort, s_issued, s_consumed;      // stages handed to TMA / waited for by the MMA thread

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = blockIdx.x * kMgM, k_iters = (g.K + kMgK - 1) / kMgK;
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) { tc::mbar_init(&full_bar[s], 1); tc::mbar_init(&empty_bar[s], 1); }
        tc::mbar_init(&acc_bar, 1);
        tc::fence_barrier_init();
        s_abort = 0; s_issued = 0; s_consumed = 0;
        tc::tma_prefetch_desc(&map_w);
        tc::tma_prefetch_desc(&map_x);
    }
    if (warp == 1) {
        tc::tmem_alloc(&tmem_base_slot, kCols);
        tc::tmem_relinquish();
    }
    tc::fence_before_sync();
    __syncthreads();
    tc::fence_after_sync();
    const uint32_t tmem_acc = tmem_base_slot;

    if (warp == 0) {
        if (lane == 0) {
            for (int it = 0; it < k_iters; ++it) {
                const int s = it % STAGES;
                const uint32_t ph = (uint32_t)(it / STAGES) & 1u;
                if (it >= STAGES && !tc::mbar_wait_abortable(&empty_bar[s], ph ^ 1u, g.budget, &s_abort)) break;
                tc::mbar_expect_tx(&full_bar[s], kWBytes + kXBytes);
                tc::tma_load_2d(sW + s * kWBytes, &map_w, it * kMgK, tile.x * g.N + n0, &full_bar[s]);
                tc::tma_load_2d(sX + s * kXBytes, &map_x, it * kMgK, tile.y, &full_bar[s]);
                s_issued = it + 1;
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = tc::idesc_bf16_f32(kMgM, (tile.z + 15) / 16 * 16);
            bool ok = true;
            for (int it = 0; it < k_iters && ok; ++it) {
                const int s = it % STAGES;
                const uint32_t ph = (uint32_t)(it / STAGES) & 1u;
                if (!tc::mbar_wait_abortable(&full_bar[s], ph, g.budget, &s_abort)) { ok = false; break; }
                s_consumed = it + 1;
                tc::fence_after_sync();
                const uint32_t w_addr = tc::smem_u32(sW + s * kWBytes), x_addr = tc::smem_u32(sX + s * kXBytes);
#pragma unroll
                for (int kk = 0; kk < kMgK / 16; ++kk)
                    tc::mma_bf16_ss(tmem_acc, tc::smem_desc_sw128(w_addr + kk * 32), tc::smem_desc_sw128(x_addr + kk * 32), idesc,
                                    (it > 0 || kk > 0) ? 1u : 0u);
                tc::mma_commit(&empty_bar[s]);
            }
            tc::mma_commit(&acc_bar);
        }
    } else {
        const int quad = warp & 3;
        const bool done = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&acc_bar, 0, g.budget, &s_abort));
        tc::fence_after_sync();
        const int n = n0 + quad * 32 + lane;
        constexpr int CW = NB < 32 ? 16 : 32;            // columns per load
        if (done && s_abort == 0) {
            for (int c0 = 0; c0 < tile.z; c0 += CW) {
                uint32_t r[CW];
                if constexpr (CW == 16) tc::tmem_ld_32x16(tmem_acc + ((uint32_t)(quad * 32) << 16) + (uint32_t)c0, r);
                else tc::tmem_ld_32x32(tmem_acc + ((uint32_t)(quad * 32) << 16) + (uint32_t)c0, r);
                tc::tmem_ld_wait();
                if (g.gated) {
                    // lanes 2i, 2i + 1 hold gate and up of one feature: the even lane finishes row c, the odd one row c + 1
                    __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(g.out) + (n >> 1);
                    const bool odd = lane & 1;
#pragma unroll
                    for (int c = 0; c < CW; c += 2) {
                        const float mine = __uint_as_float(odd ? r[c + 1] : r[c]), give = __uint_as_float(odd ? r[c] : r[c + 1]);
                        const float got = __shfl_xor_sync(0xffffffffu, give, 1);
                        const float gt = bf16_to_f32(f32_to_bf16(odd ? got : mine)), up = bf16_to_f32(f32_to_bf16(odd ? mine : got));
                        const int row = c0 + c + (odd ? 1 : 0);
                        if (row < tile.z && n < g.N) o[(size_t)(tile.y + row) * g.ldo] = f32_to_bf16(g.gated == 2 ? mg_limited(gt, up, g.limit) : silu_f(gt) * up);
                    }
                } else {
                    float* o = reinterpret_cast<float*>(g.out) + n;
#pragma unroll
                    for (int c = 0; c < CW; ++c)
                        if (c0 + c < tile.z && n < g.N) o[(size_t)(tile.y + c0 + c) * g.ldo] = __uint_as_float(r[c]);
                }
            }
        }
    }
    tc::fence_before_sync();
    __syncthreads();
    if (s_abort != 0 && threadIdx.x == 0) {
        set_status(g.status, PS_DEV_WAIT_TIMEOUT);
        // copies still in flight get a bounded chance to land before the shared memory goes back to the next CTA
        const long long b = g.budget < 4000000ll ? g.budget : 4000000ll;
        for (int c = s_consumed; c < s_issued; ++c) tc::mbar_wait(&full_bar[c % STAGES], (uint32_t)((c / STAGES) & 1), b);
    }
    __syncthreads();
    if (warp == 1) {
        tc::fence_after_sync();
        tc::tmem_dealloc(tmem_acc, kCols);
    }
}

// bf16 row-major [rows, cols] (contiguous) with a (box_rows x 64) box and the 128-byte swizzle.
static int mg_map_2d(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint32_t box_rows) {
    typedef CUresult (*Fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                           const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
    static Fn fn = nullptr;
    if (fn == nullptr) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
            return (int)cudaErrorNotSupported;
        fn = reinterpret_cast<Fn>(p);
    }
    const cuuint64_t dims[2] = {cols, rows};
    const cuuint64_t strides[1] = {cols * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kMgK, box_rows};
    const cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
              CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
               ? 0 : (int)cudaErrorInvalidValue;
}

template <int NB, int STAGES>
static int launch_moe_gemm(const CUtensorMap& map_w, const CUtensorMap& map_x, int max_tiles, const MoeGemmArgs& g, cudaStream_t stream) {
    constexpr size_t smem = (size_t)STAGES * (kMgM + NB) * kMgK * 2 + 1024;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(moe_gemm_kernel<NB, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cudaFuncSetAttribute(moe_gemm_kernel<NB, STAGES>, cudaFuncAttributePreferredSharedMemoryCarveout, (int)cudaSharedmemCarveoutMaxShared);
        set = true;
    }
    return launch_pdl(moe_gemm_kernel<NB, STAGES>, dim3((g.N + kMgM - 1) / kMgM, max_tiles), dim3(kMgThreads), smem, stream, map_w, map_x, g);
}

constexpr int kMfT = 64, kMfK = 16;

struct MoeGemmF32Args {
    const int* tiles; const float* x; const float* w; int N, K, gated; float* out; int ldo; float limit;
};

// grid = (column tiles, tiles of the list at most)
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const MoeGemmF32Args g) {
    __shared__ float sa[kMfK][kMfT + 4], sw[kMfK][kMfT + 4];
    if ((int)blockIdx.y >= g.tiles[0]) return;
    const int4 tile = reinterpret_cast<const int4*>(g.tiles)[1 + blockIdx.y];
    const int n0 = blockIdx.x * kMfT, t = threadIdx.x, tx = t & 15, ty = t >> 4;
    const float* x = g.x + (size_t)tile.y * g.K;
    const float* w = g.w + (size_t)tile.x * g.N * g.K;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < g.K; k0 += kMfK) {
        for (int i = t; i < kMfT * kMfK; i += 256) {
            const int r = i / kMfK, k = i % kMfK;
            const bool kin = k0 + k < g.K;
            sa[k][r] = kin && r < tile.z ? x[(size_t)r * g.K + k0 + k] : 0.f;
            sw[k][r] = kin && n0 + r < g.N ? w[(size_t)(n0 + r) * g.K + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kMfK; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&sa[k][ty * 4]), wv = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
            const float ar[4] = {av.x, av.y, av.z, av.w}, wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], wr[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = ty * 4 + i;
        if (r >= tile.z) continue;
        float* o = g.out + (size_t)(tile.y + r) * g.ldo;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= g.N) continue;
            if (!g.gated) o[n] = acc[i][j];
            else if (!(j & 1)) o[n >> 1] = g.gated == 2 ? mg_limited(acc[i][j], acc[i][j + 1], g.limit) : acc[i][j] / (1.f + expf(-acc[i][j])) * acc[i][j + 1];
        }
    }
}

}  // namespace ps

// Sorted rows `x` [x_rows, K] (x_rows: at least the last tile's first row + tile_rows, whatever lies behind the sorted rows), weights
// `w` [E * N, K], both bf16 and contiguous, K a multiple of 8, N even; `gated` and `limit` as in MoeGemmArgs.  `tile_rows` (16, 32, 64 or 128): the list's tile size.
PS_API int ps_moe_gemm(const void* x, int x_rows, const void* w, int E, int N, int K, int gated, float limit, const void* tiles, int tile_rows,
                       int max_tiles, void* out, int ldo, void* status, cudaStream_t stream) {
    using namespace ps;
    if (x_rows <= 0 || E <= 0 || N <= 0 || (N & 1) || K <= 0 || K % 8 || max_tiles < 1 || max_tiles > 65535 ||
        ((uintptr_t)x | (uintptr_t)w | (uintptr_t)tiles) % 16)
        return (int)cudaErrorInvalidValue;
    CUtensorMap mw, mx;
    int err = mg_map_2d(&mw, w, (uint64_t)E * N, K, kMgM);
    if (err) return err;
    if ((err = mg_map_2d(&mx, x, (uint64_t)x_rows, K, (uint32_t)tile_rows))) return err;
    MoeGemmArgs g{(const int*)tiles, N, K, gated, out, ldo, limit, (uint32_t*)status, g_ps_wait_budget_cycles};
    switch (tile_rows) {
        case 16: return launch_moe_gemm<16, 5>(mw, mx, max_tiles, g, stream);
        case 32: return launch_moe_gemm<32, 5>(mw, mx, max_tiles, g, stream);
        case 64: return launch_moe_gemm<64, 4>(mw, mx, max_tiles, g, stream);
        case 128: return launch_moe_gemm<128, 3>(mw, mx, max_tiles, g, stream);
        default: return (int)cudaErrorInvalidValue;
    }
}

// The same in fp32 over tiles of 64 rows; the gated output is fp32 too.
PS_API int ps_moe_gemm_f32(const void* x, const void* w, int N, int K, int gated, float limit, const void* tiles, int max_tiles, void* out, int ldo,
                           cudaStream_t stream) {
    using namespace ps;
    if (N <= 0 || (N & 1) || K <= 0 || max_tiles < 1 || max_tiles > 65535 || (uintptr_t)tiles % 16) return (int)cudaErrorInvalidValue;
    MoeGemmF32Args g{(const int*)tiles, (const float*)x, (const float*)w, N, K, gated, (float*)out, ldo, limit};
    moe_gemm_f32_kernel<<<dim3((N + kMfT - 1) / kMfT, max_tiles), 256, 0, stream>>>(g);
    return PS_LAUNCH_CHECK();
}
