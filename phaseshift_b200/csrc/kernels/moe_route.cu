// Routing of a mixture of experts: router logits to every row's experts and weights, and the rows sorted by expert.
//
// Per row (a warp): scores = softmax (or sigmoids) over experts and, behind them, identity experts; choice = score + correction; only
// experts of the best groups (a group counts as its best member, or as the sum of its two best) can be chosen; the `top` largest
// choices are taken and weighted by their scores, which may be divided by their sum.  All in 32-bit; ties go to the lower index.
//
// Steps of at most 64 rows run one launch: every CTA routes all rows (a bit per row and expert, so that ranks are population
// counts and every CTA computes the same order) and copies its share of the input rows to their sorted places.  Longer steps
// route in one launch, counting per expert with atomics, and sort in a second; a row's result does not depend on its place.
// Both leave the list of (expert, first sorted row, rows) tiles that the experts' kernels (moe_gemm.cu) run over.
#include "ps_common.cuh"

namespace ps {

constexpr int kRtSmallRows = 64, kRtMaxTop = 32, kRtMaxChoices = 1024, kRtWarps = 16;

struct RouteArgs {
    const float* z; int ldz; const float* correction; const int* row_slot;
    int rows, E, n, top, groups, keep;           // E experts, n = E + identity experts
    int sigmoid, group_top, renormalize;
    int* index; float* weight; float* identity;  // [rows, top], [rows, top], [rows]
    const uint4* h; int h16; uint4* xs;          // input rows of h16 16-byte units, sorted copies
    int* tiles; int tile_rows;                   // [0]: number of tiles; from [4] on (expert, first row, rows, 0)
    int2* pairs; int* counts;                    // long steps: (expert, rank) per row and place; rows per expert
    uint32_t* status;
};

// Order-preserving integer of a float (NaN: below everything that counts).
__device__ __forceinline__ uint32_t rt_key(float v) {
    const uint32_t u = __float_as_uint(v);
    return v == v ? (u & 0x80000000u ? ~u : u | 0x80000000u) : 0u;
}
constexpr uint32_t kRtNone = 0x007fffffu;            // rt_key(-infinity): nothing above it is left

// The `k` largest of v[0 .. n), one after the other; ties go to the lower index.  Every lane keeps the best of its own elements
// (lane, lane + 32, ...), only the lane that loses one looks again.  Taken elements become minus infinity; `take(place, index)` runs
// on all lanes, index -1: nothing is left.
template <typename F>
__device__ __forceinline__ void rt_top(float* v, int n, int k, F take) {
    const int lane = threadIdx.x & 31;
    uint32_t best = 0;
    int at = 0;
    auto look = [&] {
        best = 0;
        for (int i = lane; i < n; i += 32) {
            const uint32_t key = rt_key(v[i]);
            if (key > best) { best = key; at = i; }
        }
    };
    look();
    for (int place = 0; place < k; ++place) {
        const uint32_t top = __reduce_max_sync(0xffffffffu, best);
        const uint32_t who = __reduce_min_sync(0xffffffffu, best == top ? (uint32_t)at : 0xffffffffu);
        const bool some = top > kRtNone;
        take(place, some ? (int)who : -1);
        if (some && best == top && (uint32_t)at == who) { v[at] = -INFINITY; look(); }
    }
    __syncwarp();
}

// One row by one warp; `s` is 3 n floats of its own.  Lane k < top returns place k's choice (-1 when the logits are not finite) and
// weight.
__device__ __forceinline__ void route_row(const RouteArgs& a, int row, float* s, int& id, float& weight) {
    const int lane = threadIdx.x & 31, n = a.n;
    float* score = s;
    float* choice = s + n;
    float* group = s + 2 * n;
    const float* z = a.z + (size_t)row * a.ldz;
    float sum = 1.f;
    if (a.sigmoid) {
        for (int i = lane; i < n; i += 32) score[i] = 1.f / (1.f + expf(-z[i]));
    } else {
        float m = -INFINITY;
        for (int i = lane; i < n; i += 32) m = fmaxf(m, z[i]);
        m = warp_max(m);
        sum = 0.f;
        for (int i = lane; i < n; i += 32) { const float e = expf(z[i] - m); score[i] = e; sum += e; }
        sum = warp_sum(sum);
    }
    for (int i = lane; i < n; i += 32) { const float p = score[i] / sum; score[i] = p; choice[i] = a.correction != nullptr ? p + a.correction[i] : p; }
    __syncwarp();
    if (a.keep < a.groups) {
        const int size = n / a.groups;
        for (int g = lane; g < a.groups; g += 32) {
            float b = -INFINITY, second = -INFINITY;
            for (int i = g * size; i < (g + 1) * size; ++i) {
                second = fmaxf(second, fminf(b, choice[i]));
                b = fmaxf(b, choice[i]);
            }
            group[g] = a.group_top > 1 && size > 1 ? b + second : b;
        }
        __syncwarp();
        rt_top(group, a.groups, a.keep, [](int, int) {});              // kept groups end as minus infinity
        for (int i = lane; i < n; i += 32)
            if (group[i / size] != -INFINITY) choice[i] = -INFINITY;
        __syncwarp();
    }
    id = -1; weight = 0.f;
    float total = 0.f;
    rt_top(choice, n, a.top, [&](int place, int at) {
        if (at < 0) return;
        const float w = score[at];
        if (lane == place) { id = at; weight = w; }
        total += w;
    });
    if (lane < a.top && id < 0) set_status(a.status, PS_DEV_NONFINITE);
    if (a.renormalize) weight /= total + 1e-20f;
}

// Exclusive prefix sums of rows and tiles per expert by one warp; `count(e)` gives an expert's rows.
template <typename F>
__device__ __forceinline__ void route_prefix(const RouteArgs& a, F count, int* first, bool write_tiles) {
    const int lane = threadIdx.x & 31;
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < a.E; e0 += 32) {
        const int e = e0 + lane, c = e < a.E ? count(e) : 0, nt = (c + a.tile_rows - 1) / a.tile_rows;
        const int per = nt > 0 ? ((c + nt - 1) / nt + 15) / 16 * 16 : 0;                 // an expert's tiles are about equal
        int r = c, t = nt;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int pr = __shfl_up_sync(0xffffffffu, r, o), pt = __shfl_up_sync(0xffffffffu, t, o);
            if (lane >= o) { r += pr; t += pt; }
        }
        if (e < a.E) first[e] = rows + r - c;
        if (write_tiles)
            for (int i = 0; i < nt; ++i)
                reinterpret_cast<int4*>(a.tiles)[1 + tiles + t - nt + i] =
                    make_int4(e, rows + r - c + i * per, max(0, min(per, c - i * per)), 0);
        rows += __shfl_sync(0xffffffffu, r, 31);
        tiles += __shfl_sync(0xffffffffu, t, 31);
    }
    if (write_tiles && lane == 0) a.tiles[0] = tiles;
}

// at most 64 rows; grid of any size
__global__ void __launch_bounds__(kRtWarps * 32) moe_route_small_kernel(const RouteArgs a) {
    extern __shared__ __align__(16) unsigned char rt_smem[];
    unsigned long long* seen = reinterpret_cast<unsigned long long*>(rt_smem);         // [E] a bit per row
    int* first = reinterpret_cast<int*>(seen + a.E);                                   // [E]
    int* ids = first + a.E;                                                            // [rows * top]
    float* work = reinterpret_cast<float*>(ids + kRtSmallRows * a.top);                // 3 n per warp
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int e = threadIdx.x; e < a.E; e += blockDim.x) seen[e] = 0ull;
    cudaTriggerProgrammaticLaunchCompletion();
    cudaGridDependencySynchronize();
    __syncthreads();
    for (int row = warp; row < a.rows; row += kRtWarps) {
        int id = -1;
        float w = 0.f;
        if (a.row_slot[row] >= 0) route_row(a, row, work + (size_t)warp * 3 * a.n, id, w);
        if (lane < a.top) {
            ids[row * a.top + lane] = id;
            if (id >= 0 && id < a.E) atomicOr(&seen[id], 1ull << row);
        }
        if (blockIdx.x == 0) {
            if (lane < a.top) a.weight[row * a.top + lane] = w;
            const float same = warp_sum(lane < a.top && id >= a.E ? w : 0.f);
            if (lane == 0) a.identity[row] = same;
        }
    }
    __syncthreads();
    if (warp == 0) route_prefix(a, [&](int e) { return __popcll(seen[e]); }, first, blockIdx.x == 0);
    __syncthreads();
    auto place = [&](int p) {
        const int e = ids[p];
        return e >= 0 && e < a.E ? first[e] + __popcll(seen[e] & ((1ull << (p / a.top)) - 1ull)) : -1;
    };
    if (blockIdx.x == 0)
        for (int p = threadIdx.x; p < a.rows * a.top; p += blockDim.x) a.index[p] = place(p);
    for (int p = blockIdx.x; p < a.rows * a.top; p += gridDim.x) {
        const int to = place(p);
        if (to < 0) continue;
        const uint4* src = a.h + (size_t)(p / a.top) * a.h16;
        for (int i = threadIdx.x; i < a.h16; i += blockDim.x) a.xs[(size_t)to * a.h16 + i] = src[i];
    }
}

// a warp per row
__global__ void __launch_bounds__(256) moe_route_kernel(const RouteArgs a) {
    extern __shared__ __align__(16) unsigned char rt_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = blockIdx.x * 8 + warp;
    if (row >= a.rows) return;
    int id = -1;
    float w = 0.f;
    if (a.row_slot[row] >= 0) route_row(a, row, reinterpret_cast<float*>(rt_smem) + (size_t)warp * 3 * a.n, id, w);
    if (lane < a.top) {
        const bool real = id >= 0 && id < a.E;
        a.pairs[row * a.top + lane] = make_int2(real ? id : -1, real ? atomicAdd(&a.counts[id], 1) : 0);
        a.weight[row * a.top + lane] = w;
    }
    const float same = warp_sum(lane < a.top && id >= a.E ? w : 0.f);
    if (lane == 0) a.identity[row] = same;
}

// a CTA per row
__global__ void __launch_bounds__(256) moe_sort_kernel(const RouteArgs a) {
    extern __shared__ __align__(16) unsigned char rt_smem[];
    int* first = reinterpret_cast<int*>(rt_smem);
    const int row = blockIdx.x;
    if (threadIdx.x < 32) route_prefix(a, [&](int e) { return a.counts[e]; }, first, row == 0);
    __syncthreads();
    const uint4* src = a.h + (size_t)row * a.h16;
    for (int k = 0; k < a.top; ++k) {
        const int2 p = a.pairs[row * a.top + k];
        const int to = p.x >= 0 ? first[p.x] + p.y : -1;
        if (threadIdx.x == 0) a.index[row * a.top + k] = to;
        if (to >= 0)
            for (int i = threadIdx.x; i < a.h16; i += blockDim.x) a.xs[(size_t)to * a.h16 + i] = src[i];
    }
}

}  // namespace ps

// `h`, `xs`: rows of `row_bytes` (a multiple of 16); `tiles`: 4 + 4 * (rows * top / tile_rows + min(E, rows * top)) ints; `pairs`
// (2 ints per row and place) and `counts` ([E]) are scratch of steps longer than 64 rows.  `correction` may be null; `group_top` 1 or 2.
PS_API int ps_moe_route(const void* z, int ldz, const void* correction, const void* row_slot, int rows, int E, int identity, int top,
                        int groups, int keep, int sigmoid, int group_top, int renormalize, void* index, void* weight, void* same, const void* h, int row_bytes, void* xs, void* tiles,
                        int tile_rows, void* pairs, void* counts, void* status, cudaStream_t stream) {
    using namespace ps;
    const int n = E + identity;
    if (rows <= 0 || E <= 0 || identity < 0 || n > kRtMaxChoices || top < 1 || top > kRtMaxTop || groups < 1 || n % groups || keep < 1 || keep > groups ||
        group_top < 1 || group_top > 2 || top > keep * (n / groups) || ldz < n || row_bytes % 16 || tile_rows < 1 || ((uintptr_t)h | (uintptr_t)xs | (uintptr_t)tiles) % 16)
        return (int)cudaErrorInvalidValue;
    RouteArgs a;
    a.z = (const float*)z; a.ldz = ldz; a.correction = (const float*)correction; a.row_slot = (const int*)row_slot; a.rows = rows; a.E = E;
    a.n = n; a.top = top; a.groups = groups; a.keep = keep; a.sigmoid = sigmoid; a.group_top = group_top; a.renormalize = renormalize; a.index = (int*)index; a.weight = (float*)weight; a.identity = (float*)same;
    a.h = (const uint4*)h; a.h16 = row_bytes / 16; a.xs = (uint4*)xs; a.tiles = (int*)tiles; a.tile_rows = tile_rows;
    a.pairs = (int2*)pairs; a.counts = (int*)counts; a.status = (uint32_t*)status;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(moe_route_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024);
        cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);
        set = true;
    }
    if (rows <= kRtSmallRows) {
        const size_t smem = (size_t)E * 12 + (size_t)kRtSmallRows * top * 4 + (size_t)kRtWarps * 3 * n * 4;
        const int ctas = rows * top < 148 ? rows * top : 148;
        return launch_pdl(moe_route_small_kernel, dim3(ctas), dim3(kRtWarps * 32), smem, stream, a);
    }
    if (pairs == nullptr || counts == nullptr) return (int)cudaErrorInvalidValue;
    int err = (int)cudaMemsetAsync(counts, 0, (size_t)E * 4, stream);
    if (err) return err;
    moe_route_kernel<<<(rows + 7) / 8, 256, (size_t)8 * 3 * n * 4, stream>>>(a);
    if ((err = PS_LAUNCH_CHECK())) return err;
    moe_sort_kernel<<<rows, 256, (size_t)E * 4, stream>>>(a);
    return PS_LAUNCH_CHECK();
}
