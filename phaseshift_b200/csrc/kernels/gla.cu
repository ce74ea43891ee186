// Gated linear attention with a decay per key channel: everything between the input projection and the output projection.
//
// Per head, with log-decay la = log(sigmoid(z)) / tau, z = a2 . a1 + bias (a1 = the row's low-rank decay input):
//     S_t = diag(exp(la_t)) S_{t-1} + k_t v_t^T ,   o_t = S_t^T (q_t * q_scale) ,   out = (rms(o) * w) * silu(g)
// The decays, their logarithms and sums, the state and everything multiplied into it are fp32.
// FORGET variants (linear attention whose forget gate is its key): z is a column of the projection per head and channel (+ bias),
//     f = lower + (1 - lower) sigmoid(z),  la = log(f),  k = 1 - f,  q = silu(q) * q_scale
// and there may be no output gate.
//
// ps_gla_rows     row-sequential: one CTA per (sequence, head), state read and written once per launch.  Decode, short
//                 portions, and the 32-bit engines.  Sizes 128 x 128 and 64 x 64 keep the state in registers, others update
//                 it in place.
// ps_gla_chunked  portions of many rows, in blocks of C = 64 rows that are independent of each other except for the state:
//   gla_prepare   per (block, head): z, la and their running sums B inside the block; the 64 x 64 matrix
//                 A[i][j] = sum_d q_i[d] k_j[d] exp(B_i[d] - B_j[d]) (j <= i); A v; the decayed queries q exp(B); and the
//                 block's own contribution to the state, U = sum_j exp(B_end - B_j) k_j v_j^T
//   gla_scan      S_{c+1} = exp(B_end) S_c + U_c over the blocks of a sequence, elementwise; leaves S_c in U's place
//   gla_output    o = A v + (q exp(B)) S_c, head norm, gate
// No exponential of a positive number is ever formed, whatever the decays: A is cut into 16-row sub-blocks; off the diagonal
// exp(B_i - B_j) factors through the end of the key's sub-block and of the sub-block before the query's (all three factors
// are at most 1), on the diagonal it is evaluated pair by pair.
// (Secondary chunking of this kind is described in "Gated Linear Attention Transformers with Hardware-Efficient Training" by
// Songlin Yang, Bailin Wang, Yikang Shen, Rameswar Panda and Yoon Kim.)
// Products run on TF32 mma.sync with every fp32 operand split into two TF32 terms (values and keys come from bf16 and are
// exact), which keeps fp32-level accuracy; the hybrid decoder's chunked recurrence is in gdn_chunked.cu.
#include "ps_common.cuh"

namespace ps {

struct GlaSeq { int row_start, n_rows, slot, pos_start; };

struct GlaArgs {
    const void* proj; int ld, H, dk, dv, dv_true;
    int q_off, k_off, v_off, g_off, a_off, rank;
    float q_scale, inv_tau, eps;
    const void* a2; const float* a2_bias; const float* norm_w;
    const float* lower;                // FORGET: [H * dk]
    float* state;                      // [slots, H, dk, dv]
    const GlaSeq* seqs; int n_seqs;
    void* out;                         // [rows, H * dv]
    int rows_limit;                    // rows kernel: skip sequences with more rows; chunked: skip sequences with at most that many
    // chunked scratch
    float* qd;                         // [blocks, H, 64, dk]  decayed queries
    float* oi;                         // [blocks, H, 64, dv]  A v
    float* u;                          // [blocks, H, dk, dv]
    float* dec;                        // [blocks, H, dk]      exp(B_end)
};

__device__ __forceinline__ float gla_log_decay(float z, float inv_tau) {
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau;
}
// Forget gate: how much is written, and the logarithm of what is kept (bounded, so that sums stay finite).
__device__ __forceinline__ float gla_forget(float z, float lower, float& log_keep) {
    const float e = expf(-fabsf(z)), s = 1.f / (1.f + e), neg = z > 0.f ? e * s : s;            // sigmoid(-z)
    const float k = (1.f - lower) * neg;
    log_keep = fmaxf(k < 0.5f ? log1pf(-k) : logf(lower + (1.f - lower) * (z > 0.f ? s : e * s)), -100.f);
    return k;
}
template <typename T> __device__ __forceinline__ T gla_cast(float v);
template <> __device__ __forceinline__ float gla_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 gla_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }
__device__ __forceinline__ float gla_silu(float x) { return x / (1.f + expf(-x)); }

// ------------------------------------------------------------------------------------------------ row-sequential form
template <typename T, int DK, int DV, bool FORGET>
__global__ void __launch_bounds__(256) gla_rows_kernel(const GlaArgs a) {
    extern __shared__ __align__(16) float gla_smem[];
    const int dk = DK > 0 ? DK : a.dk, dv = DV > 0 ? DV : a.dv;
    const int CG = dv / 4, RG = 256 / CG;          // column groups of four, row groups
    float* s_q = gla_smem;                         // [dk]
    float* s_k = s_q + dk;
    float* s_al = s_k + dk;
    float* s_v = s_al + dk;                        // [dv]
    float* s_part = s_v + dv;                      // [RG][dv], at most 1024
    __shared__ float red[32];
    const int h = blockIdx.x;
    const GlaSeq sd = a.seqs[blockIdx.y];
    if (sd.n_rows <= 0 || sd.slot < 0 || (a.rows_limit > 0 && sd.n_rows > a.rows_limit)) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows) && sd.pos_start >= 0);
    const int t = threadIdx.x, cg = t % CG, rg = t / CG;
    const bool active = rg < RG;
    constexpr int kR = DK > 0 ? DK * DV / 1024 : 1;
    float* sp = a.state + ((size_t)sd.slot * a.H + h) * dk * dv;
    cudaTriggerProgrammaticLaunchCompletion();
    float S[kR][4];
    if constexpr (DK > 0) {
        // the state was last written by an earlier step (or layer pass), not by the stream predecessor
#pragma unroll
        for (int r = 0; r < kR; ++r) {
            const float4 x = *reinterpret_cast<const float4*>(sp + (size_t)(rg + RG * r) * DV + cg * 4);
            S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
        }
    }
    cudaGridDependencySynchronize();
    for (int i = 0; i < sd.n_rows; ++i) {
        const int row = sd.row_start + i;
        const T* pr = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld;
        for (int d = t; d < dk; d += 256) {
            float z = a.a2_bias[h * dk + d];
            const float q = (float)pr[a.q_off + h * dk + d];
            if constexpr (FORGET) {
                float la;
                z += (float)pr[a.a_off + h * dk + d];
                const float k = gla_forget(z, a.lower[h * dk + d], la);
                s_k[d] = k;
                s_al[d] = 1.f - k;
                s_q[d] = gla_silu(q) * a.q_scale;
            } else {
                const T* w = reinterpret_cast<const T*>(a.a2) + (size_t)(h * dk + d) * a.rank;
                for (int r = 0; r < a.rank; ++r) z = fmaf((float)w[r], (float)pr[a.a_off + r], z);
                s_al[d] = expf(gla_log_decay(z, a.inv_tau));
                s_q[d] = q * a.q_scale;
                s_k[d] = (float)pr[a.k_off + h * dk + d];
            }
        }
        for (int d = t; d < dv; d += 256) s_v[d] = (float)pr[a.v_off + h * dv + d];
        __syncthreads();
        if (active) {
            const float4 v = *reinterpret_cast<const float4*>(s_v + cg * 4);
            float p[4] = {0.f, 0.f, 0.f, 0.f};
            if constexpr (DK > 0) {
#pragma unroll
                for (int r = 0; r < kR; ++r) {
                    const int d = rg + RG * r;
                    const float al = s_al[d], k = s_k[d], q = s_q[d];
                    S[r][0] = fmaf(S[r][0], al, k * v.x); S[r][1] = fmaf(S[r][1], al, k * v.y);
                    S[r][2] = fmaf(S[r][2], al, k * v.z); S[r][3] = fmaf(S[r][3], al, k * v.w);
#pragma unroll
                    for (int c = 0; c < 4; ++c) p[c] = fmaf(S[r][c], q, p[c]);
                }
            } else {
                for (int d = rg; d < dk; d += RG) {
                    float4* s4 = reinterpret_cast<float4*>(sp + (size_t)d * dv + cg * 4);
                    float4 x = *s4;
                    const float al = s_al[d], k = s_k[d], q = s_q[d];
                    x.x = fmaf(x.x, al, k * v.x); x.y = fmaf(x.y, al, k * v.y);
                    x.z = fmaf(x.z, al, k * v.z); x.w = fmaf(x.w, al, k * v.w);
                    *s4 = x;
                    p[0] = fmaf(x.x, q, p[0]); p[1] = fmaf(x.y, q, p[1]); p[2] = fmaf(x.z, q, p[2]); p[3] = fmaf(x.w, q, p[3]);
                }
            }
            *reinterpret_cast<float4*>(s_part + rg * dv + cg * 4) = make_float4(p[0], p[1], p[2], p[3]);
        }
        __syncthreads();
        float ss = 0.f;
        for (int d = t; d < dv; d += 256) {
            float o = 0.f;
            for (int r = 0; r < RG; ++r) o += s_part[r * dv + d];
            s_v[d] = o;                            // each thread re-reads only its own entries
            ss = fmaf(o, o, ss);
        }
        ss = block_sum(ss, red);
        const float inv = rsqrtf(ss / (float)a.dv_true + a.eps);
        T* out = reinterpret_cast<T*>(a.out) + (size_t)row * a.H * dv + h * dv;
        for (int d = t; d < dv; d += 256)
            out[d] = gla_cast<T>(s_v[d] * inv * a.norm_w[d] * (FORGET && a.g_off < 0 ? 1.f : gla_silu((float)pr[a.g_off + h * dv + d])));
        __syncthreads();
    }
    if constexpr (DK > 0) {
#pragma unroll
        for (int r = 0; r < kR; ++r)
            *reinterpret_cast<float4*>(sp + (size_t)(rg + RG * r) * DV + cg * 4) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    }
}

// ------------------------------------------------------------------------------------------------ chunked form (bf16)
constexpr int kGC = 64;                 // rows of a block
constexpr int kGPrepThreads = 512, kGOutThreads = 256;
constexpr int kGAPitch = kGC + 4;

__device__ __forceinline__ uint32_t to_tf32(float x) { uint32_t r; asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x)); return r; }
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
    hi = to_tf32(x);
    lo = to_tf32(x - __uint_as_float(hi));
}
__device__ __forceinline__ void mma_tf32_1688(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Which sequence and which of its blocks a global block index is; false: none.
__device__ __forceinline__ bool gla_find_block(const GlaArgs& a, int blk, int& seq, int& row0, int& n) {
    int base = 0;
    for (int s = 0; s < a.n_seqs; ++s) {
        const int rows = a.seqs[s].n_rows;
        if (rows <= a.rows_limit || a.seqs[s].slot < 0) continue;
        const int nb = (rows + kGC - 1) / kGC;
        if (blk < base + nb) {
            seq = s;
            row0 = a.seqs[s].row_start + (blk - base) * kGC;
            n = min(kGC, rows - (blk - base) * kGC);
            return true;
        }
        base += nb;
    }
    return false;
}

__host__ __device__ inline size_t gla_prep_smem_floats(int dk, int dv) {
    const size_t pq = dk + 4, pk = dk + 8, pv = (size_t)(dv + 16) / 2;                  // v rows are bf16
    const size_t b = kGC * (pq > pv ? pq : pv);                                         // B, later v
    return kGC * pq + kGC * pk + b + (size_t)kGC * kGAPitch + 4 * dk;
}

// grid = (blocks, H)
template <int DKT, int DVT, bool FORGET>
__global__ void __launch_bounds__(kGPrepThreads) gla_prepare_kernel(const GlaArgs a) {
    extern __shared__ __align__(16) float gla_smem[];
    const int dk = DKT > 0 ? DKT : a.dk, dv = DVT > 0 ? DVT : a.dv;
    const int PQ = dk + 4, PK = dk + 8, PV = dv + 16;
    float* sQ = gla_smem;                               // [64][PQ]
    float* sK = sQ + kGC * PQ;                          // [64][PK]
    float* sB = sK + kGC * PK;                          // [64][PQ]; its place holds v afterwards
    __nv_bfloat16* sV = reinterpret_cast<__nv_bfloat16*>(sB);       // [64][PV]
    float* sA = sB + kGC * max(PQ, PV / 2);             // [64][68]
    float* sE = sA + kGC * kGAPitch;                    // [4][dk]  B at the end of each 16-row sub-block
    int seq, row0, n;
    if (!gla_find_block(a, blockIdx.x, seq, row0, n)) return;
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const size_t bh = (size_t)blockIdx.x * a.H + h;
    const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj) + (size_t)row0 * a.ld;

    if constexpr (FORGET) {
        // ---- log-decays and keys from the gate's columns
        for (int i = t; i < kGC * (dk / 8); i += kGPrepThreads) {
            const int r = i / (dk / 8), c = (i % (dk / 8)) * 8;
            float la[8], k[8];
            if (r < n) {
                const uint4 zr = *reinterpret_cast<const uint4*>(proj + (size_t)r * a.ld + a.a_off + h * dk + c);
                const uint32_t zw[4] = {zr.x, zr.y, zr.z, zr.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 z = bf16x2_bits_to_f32x2(zw[e]);
                    const int d = h * dk + c + 2 * e;
                    k[2 * e] = gla_forget(z.x + a.a2_bias[d], a.lower[d], la[2 * e]);
                    k[2 * e + 1] = gla_forget(z.y + a.a2_bias[d + 1], a.lower[d + 1], la[2 * e + 1]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) la[e] = k[e] = 0.f;
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) { sB[r * PQ + c + e] = la[e]; sK[r * PK + c + e] = k[e]; }
        }
        __syncthreads();
    } else
    // ---- log-decays: a1 rows and this head's slice of a2 share the q / k buffers, which are not filled yet
    {
        float* s1 = sQ;                                 // [64][rank]
        const int pw = a.rank + 1;
        float* s2 = sQ + kGC * a.rank;                  // [dk][rank + 1]
        for (int i = t; i < kGC * a.rank; i += kGPrepThreads) {
            const int r = i / a.rank, c = i % a.rank;
            s1[i] = r < n ? bf16_to_f32(proj[(size_t)r * a.ld + a.a_off + c]) : 0.f;
        }
        const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.a2) + (size_t)h * dk * a.rank;
        for (int i = t; i < dk * a.rank; i += kGPrepThreads) s2[(i / a.rank) * pw + i % a.rank] = bf16_to_f32(w[i]);
        __syncthreads();
        if constexpr (DKT > 0) {
            // a thread owns one channel and every (512 / dk)-th row: eight weights at a time in registers, a1 as broadcast vectors
            constexpr int kStep = kGPrepThreads / DKT, kRows = kGC / kStep;
            const int d = t % DKT, r0 = t / DKT;
            float z[kRows];
#pragma unroll
            for (int j = 0; j < kRows; ++j) z[j] = a.a2_bias[h * dk + d];
            for (int c0 = 0; c0 < a.rank; c0 += 8) {
                float wv[8];
#pragma unroll
                for (int c = 0; c < 8; ++c) wv[c] = s2[d * pw + c0 + c];
#pragma unroll
                for (int j = 0; j < kRows; ++j) {
                    const float4 x = *reinterpret_cast<const float4*>(s1 + (r0 + j * kStep) * a.rank + c0);
                    const float4 y = *reinterpret_cast<const float4*>(s1 + (r0 + j * kStep) * a.rank + c0 + 4);
                    float acc = z[j];
                    acc = fmaf(wv[0], x.x, acc); acc = fmaf(wv[1], x.y, acc); acc = fmaf(wv[2], x.z, acc); acc = fmaf(wv[3], x.w, acc);
                    acc = fmaf(wv[4], y.x, acc); acc = fmaf(wv[5], y.y, acc); acc = fmaf(wv[6], y.z, acc); acc = fmaf(wv[7], y.w, acc);
                    z[j] = acc;
                }
            }
#pragma unroll
            for (int j = 0; j < kRows; ++j) {
                const int r = r0 + j * kStep;
                sB[r * PQ + d] = r < n ? gla_log_decay(z[j], a.inv_tau) : 0.f;
            }
        } else
        for (int i = t; i < kGC * dk; i += kGPrepThreads) {
            const int r = i / dk, d = i % dk;
            float la = 0.f;
            if (r < n) {
                float z = a.a2_bias[h * dk + d];
                for (int c = 0; c < a.rank; ++c) z = fmaf(s2[d * pw + c], s1[r * a.rank + c], z);
                la = gla_log_decay(z, a.inv_tau);
            }
            sB[r * PQ + d] = la;
        }
        __syncthreads();
    }
    // ---- running sums, 16 rows at a time, then the sub-blocks' offsets; meanwhile q and k arrive
    for (int i = t; i < 4 * dk; i += kGPrepThreads) {
        const int blk = i / dk, d = i % dk;
        float s = 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) { s += sB[(blk * 16 + r) * PQ + d]; sB[(blk * 16 + r) * PQ + d] = s; }
        sE[i] = s;
    }
    for (int i = t; i < kGC * (dk / 8); i += kGPrepThreads) {
        const int r = i / (dk / 8), c = (i % (dk / 8)) * 8;
        uint4 q = make_uint4(0, 0, 0, 0), k = q;
        if (r < n) {
            q = *reinterpret_cast<const uint4*>(proj + (size_t)r * a.ld + a.q_off + h * dk + c);
            if constexpr (!FORGET) k = *reinterpret_cast<const uint4*>(proj + (size_t)r * a.ld + a.k_off + h * dk + c);
        }
        const uint32_t qw[4] = {q.x, q.y, q.z, q.w}, kw[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 qf = bf16x2_bits_to_f32x2(qw[e]);
            if constexpr (FORGET) {
                sQ[r * PQ + c + 2 * e] = silu_f(qf.x) * a.q_scale; sQ[r * PQ + c + 2 * e + 1] = silu_f(qf.y) * a.q_scale;
            } else {
                const float2 kf = bf16x2_bits_to_f32x2(kw[e]);
                sQ[r * PQ + c + 2 * e] = qf.x * a.q_scale; sQ[r * PQ + c + 2 * e + 1] = qf.y * a.q_scale;
                sK[r * PK + c + 2 * e] = kf.x; sK[r * PK + c + 2 * e + 1] = kf.y;
            }
        }
    }
    __syncthreads();
    // ---- diagonal sub-blocks, pair by pair (sums local to the sub-block suffice: only differences enter)
#pragma unroll 1
    for (int blk = 0; blk < 4; ++blk) {
        const int il = (blk & 1) ? 15 - warp : warp, i = blk * 16 + il;
        if constexpr (DKT > 0) {
            constexpr int kU = DKT / 32;                // consecutive channels of a lane
            const int d = lane * kU;
            float qi[kU], bi[kU];
#pragma unroll
            for (int u = 0; u < kU; ++u) { qi[u] = sQ[i * PQ + d + u]; bi[u] = sB[i * PQ + d + u]; }
            for (int jl = 0; jl <= il; ++jl) {
                const int j = blk * 16 + jl;
                float kj[kU], bj[kU], s = 0.f;
                if constexpr (kU == 4) {
                    *reinterpret_cast<float4*>(kj) = *reinterpret_cast<const float4*>(sK + j * PK + d);
                    *reinterpret_cast<float4*>(bj) = *reinterpret_cast<const float4*>(sB + j * PQ + d);
                } else {
#pragma unroll
                    for (int u = 0; u < kU; ++u) { kj[u] = sK[j * PK + d + u]; bj[u] = sB[j * PQ + d + u]; }
                }
#pragma unroll
                for (int u = 0; u < kU; ++u) s = fmaf(qi[u] * kj[u], __expf(bi[u] - bj[u]), s);
                s = warp_sum(s);
                if (lane == 0) sA[i * kGAPitch + j] = s;
            }
        } else {
        constexpr int kU = 8;
        float qi[kU], bi[kU];
#pragma unroll
        for (int u = 0; u < kU; ++u) {
            const int d = lane + 32 * u;
            qi[u] = d < dk ? sQ[i * PQ + d] : 0.f;
            bi[u] = d < dk ? sB[i * PQ + d] : 0.f;
        }
        for (int jl = 0; jl <= il; ++jl) {
            const int j = blk * 16 + jl;
            float s = 0.f;
#pragma unroll
            for (int u = 0; u < kU; ++u) {
                const int d = lane + 32 * u;
                if (d < dk) s = fmaf(qi[u] * sK[j * PK + d], __expf(bi[u] - sB[j * PQ + d]), s);
            }
            s = warp_sum(s);
            if (lane == 0) sA[i * kGAPitch + j] = s;
        }
        }
        if (lane > il && lane < 16) sA[i * kGAPitch + blk * 16 + lane] = 0.f;
    }
    __syncthreads();
    // ---- scale in place: q by the decay since the start of its sub-block, k by the decay up to the end of its own
    for (int i = t; i < kGC * dk; i += kGPrepThreads) {
        const int r = i / dk, d = i % dk;
        const float bl = sB[r * PQ + d];
        sQ[r * PQ + d] *= __expf(bl);
        sK[r * PK + d] *= __expf(sE[(r >> 4) * dk + d] - bl);
    }
    __syncthreads();
    for (int d = t; d < dk; d += kGPrepThreads) {                // sub-block totals -> running sums at the sub-blocks' ends
        const float e1 = sE[d] + sE[dk + d], e2 = e1 + sE[2 * dk + d], e3 = e2 + sE[3 * dk + d];
        sE[dk + d] = e1; sE[2 * dk + d] = e2; sE[3 * dk + d] = e3;
        a.dec[bh * dk + d] = expf(e3);
    }
    for (int i = t; i < kGC * (dv / 8); i += kGPrepThreads) {    // B has been used up
        const int r = i / (dv / 8), c = (i % (dv / 8)) * 8;
        *reinterpret_cast<uint4*>(sV + r * PV + c) =
            r < n ? *reinterpret_cast<const uint4*>(proj + (size_t)r * a.ld + a.v_off + h * dv + c) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    // ---- sub-blocks below the diagonal: (query block, key block) pairs x two halves of eight keys
    if (warp < 12) {
        const int pair = warp >> 1, half = warp & 1;
        const int qi = pair < 1 ? 1 : (pair < 3 ? 2 : 3), kj = pair < 1 ? 0 : (pair < 3 ? pair - 1 : pair - 3);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const float* q0 = sQ + (qi * 16 + g) * PQ + tq;
        const float* k0 = sK + (kj * 16 + half * 8 + g) * PK + tq;
        for (int k = 0; k < dk; k += 8) {
            float f0 = 1.f, f1 = 1.f;                            // decay from the end of the key's block to the start of the query's
            if (qi - 1 > kj) {
                f0 = __expf(sE[(qi - 1) * dk + k + tq] - sE[kj * dk + k + tq]);
                f1 = __expf(sE[(qi - 1) * dk + k + tq + 4] - sE[kj * dk + k + tq + 4]);
            }
            uint32_t ah[4], al[4], bh2[2], bl2[2];
            split_tf32(q0[k] * f0, ah[0], al[0]);
            split_tf32(q0[8 * PQ + k] * f0, ah[1], al[1]);
            split_tf32(q0[k + 4] * f1, ah[2], al[2]);
            split_tf32(q0[8 * PQ + k + 4] * f1, ah[3], al[3]);
            split_tf32(k0[k], bh2[0], bl2[0]);
            split_tf32(k0[k + 4], bh2[1], bl2[1]);
            mma_tf32_1688(acc, al, bh2[0], bh2[1]);
            mma_tf32_1688(acc, ah, bl2[0], bl2[1]);
            mma_tf32_1688(acc, ah, bh2[0], bh2[1]);
        }
        float* dst = sA + (qi * 16 + g) * kGAPitch + kj * 16 + half * 8 + 2 * tq;
        dst[0] = acc[0]; dst[1] = acc[1]; dst[8 * kGAPitch] = acc[2]; dst[8 * kGAPitch + 1] = acc[3];
    }
    // ---- queries decayed from the block's start (the state is read with them)
    {
        float* qd = a.qd + bh * kGC * dk;
        for (int i = t; i < kGC * dk; i += kGPrepThreads) {
            const int r = i / dk, d = i % dk;
            const float f = r >= 16 ? __expf(sE[((r >> 4) - 1) * dk + d]) : 1.f;
            qd[i] = sQ[r * PQ + d] * f;
        }
    }
    __syncthreads();
    // ---- A v: a warp takes query blocks p and 3 - p (equal work) and every eighth column tile
    {
        float* oi = a.oi + bh * kGC * dv;
        for (int half = 0; half < 2; ++half) {
            const int m = half == 0 ? (warp & 1) : 3 - (warp & 1);
            for (int nt = warp >> 1; nt < dv / 8; nt += 8) {
                float acc[4] = {0.f, 0.f, 0.f, 0.f};
                for (int k = 0; k < 16 * (m + 1); k += 8) {
                    uint32_t ah[4], al[4];
                    const float* ap = sA + (m * 16 + g) * kGAPitch + k + tq;
                    split_tf32(ap[0], ah[0], al[0]);
                    split_tf32(ap[8 * kGAPitch], ah[1], al[1]);
                    split_tf32(ap[4], ah[2], al[2]);
                    split_tf32(ap[8 * kGAPitch + 4], ah[3], al[3]);
                    const uint32_t b0 = __float_as_uint(bf16_to_f32(sV[(k + tq) * PV + nt * 8 + g]));
                    const uint32_t b1 = __float_as_uint(bf16_to_f32(sV[(k + tq + 4) * PV + nt * 8 + g]));
                    mma_tf32_1688(acc, al, b0, b1);
                    mma_tf32_1688(acc, ah, b0, b1);
                }
                float* o = oi + (size_t)(m * 16 + g) * dv + nt * 8 + 2 * tq;
                *reinterpret_cast<float2*>(o) = make_float2(acc[0], acc[1]);
                *reinterpret_cast<float2*>(o + 8 * dv) = make_float2(acc[2], acc[3]);
            }
        }
    }
    // ---- U = (k decayed to the block's end)^T v: 16 channels x 64 columns per task
    {
        float* u = a.u + bh * dk * dv;
        const int mt = dk / 16, ng = (dv + 63) / 64;
        for (int task = warp; task < mt * ng; task += kGPrepThreads / 32) {
            const int m = task % mt, nb = task / mt * 8, ne = min(8, dv / 8 - nb);
            float acc[8][4];
#pragma unroll
            for (int j = 0; j < 8; ++j) { acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f; }
            const int c0 = m * 16 + g, c1 = c0 + 8;
            const float e0 = sE[3 * dk + c0], e1 = sE[3 * dk + c1];
#pragma unroll 2
            for (int k = 0; k < kGC; k += 8) {
                const int kb = k >> 4;
                const float f0 = kb < 3 ? __expf(e0 - sE[kb * dk + c0]) : 1.f, f1 = kb < 3 ? __expf(e1 - sE[kb * dk + c1]) : 1.f;
                uint32_t ah[4], al[4];
                split_tf32(sK[(k + tq) * PK + c0] * f0, ah[0], al[0]);
                split_tf32(sK[(k + tq) * PK + c1] * f1, ah[1], al[1]);
                split_tf32(sK[(k + tq + 4) * PK + c0] * f0, ah[2], al[2]);
                split_tf32(sK[(k + tq + 4) * PK + c1] * f1, ah[3], al[3]);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    if (j < ne) {
                        const uint32_t b0 = __float_as_uint(bf16_to_f32(sV[(k + tq) * PV + (nb + j) * 8 + g]));
                        const uint32_t b1 = __float_as_uint(bf16_to_f32(sV[(k + tq + 4) * PV + (nb + j) * 8 + g]));
                        mma_tf32_1688(acc[j], al, b0, b1);
                        mma_tf32_1688(acc[j], ah, b0, b1);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                if (j < ne) {
                    float* o = u + (size_t)c0 * dv + (nb + j) * 8 + 2 * tq;
                    *reinterpret_cast<float2*>(o) = make_float2(acc[j][0], acc[j][1]);
                    *reinterpret_cast<float2*>(o + 8 * dv) = make_float2(acc[j][2], acc[j][3]);
                }
            }
        }
    }
}

// grid = (ceil(H * dk * dv / 4 / 256), n_seqs): a thread carries four state elements through the sequence's blocks.
__global__ void __launch_bounds__(256) gla_scan_kernel(const GlaArgs a) {
    const GlaSeq sd = a.seqs[blockIdx.y];
    if (sd.slot < 0 || sd.n_rows <= a.rows_limit) return;
    const size_t per = (size_t)a.H * a.dk * a.dv;
    const size_t e = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
    if (e >= per) return;
    int base = 0;
    for (int s = 0; s < (int)blockIdx.y; ++s)
        if (a.seqs[s].slot >= 0 && a.seqs[s].n_rows > a.rows_limit) base += (a.seqs[s].n_rows + kGC - 1) / kGC;
    const int nb = (sd.n_rows + kGC - 1) / kGC;
    float4* st = reinterpret_cast<float4*>(a.state + (size_t)sd.slot * per + e);
    float4 S = *st;
    const size_t hd = e / a.dv;                            // head * dk + channel
    float* u = a.u + (size_t)base * per + e;
    const float* dc = a.dec + (size_t)base * a.H * a.dk + hd;
    float4 un = *reinterpret_cast<const float4*>(u);
    float dn = *dc;
    for (int c = 0; c < nb; ++c) {
        const float4 uc = un;
        const float d = dn;
        if (c + 1 < nb) {
            un = *reinterpret_cast<const float4*>(u + (size_t)(c + 1) * per);
            dn = dc[(size_t)(c + 1) * a.H * a.dk];
        }
        *reinterpret_cast<float4*>(u + (size_t)c * per) = S;
        S.x = fmaf(S.x, d, uc.x); S.y = fmaf(S.y, d, uc.y); S.z = fmaf(S.z, d, uc.z); S.w = fmaf(S.w, d, uc.w);
    }
    *st = S;
}

__device__ __forceinline__ void gla_cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// grid = (blocks, H)
template <int DKT, int DVT, bool FORGET>
__global__ void __launch_bounds__(kGOutThreads) gla_output_kernel(const GlaArgs a) {
    extern __shared__ __align__(16) float gla_smem[];
    __shared__ float s_ss[2][kGC];
    const int dk = DKT > 0 ? DKT : a.dk, dv = DVT > 0 ? DVT : a.dv;
    const int PQ = dk + 4, PS = dv + 8;
    float* sQ = gla_smem;                                  // [64][PQ]
    float* sS = sQ + kGC * PQ;                             // [dk][PS]
    int seq, row0, n;
    if (!gla_find_block(a, blockIdx.x, seq, row0, n)) return;
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const size_t bh = (size_t)blockIdx.x * a.H + h;
    const float* qd = a.qd + bh * kGC * dk;
    for (int i = t; i < kGC * dk / 4; i += kGOutThreads) {
        const int r = i / (dk / 4), c = (i % (dk / 4)) * 4;
        gla_cp_async16(sQ + r * PQ + c, qd + r * dk + c);
    }
    const float* S = a.u + bh * dk * dv;
    for (int i = t; i < dk * dv / 4; i += kGOutThreads) {
        const int r = i / (dv / 4), c = (i % (dv / 4)) * 4;
        gla_cp_async16(sS + r * PS + c, S + (size_t)r * dv + c);
    }
    constexpr int kNT = DVT > 0 ? DVT / 16 : 16;           // column tiles of eight per warp (half of the head)
    const int m = warp & 3, half = warp >> 2, nt = dv / 16;
    float acc[kNT][4];
    const float* oi = a.oi + bh * kGC * dv + (size_t)(m * 16 + g) * dv + half * (dv / 2) + 2 * tq;
#pragma unroll
    for (int j = 0; j < kNT; ++j) {
        if (j < nt) {
            const float2 x = *reinterpret_cast<const float2*>(oi + j * 8), y = *reinterpret_cast<const float2*>(oi + 8 * dv + j * 8);
            acc[j][0] = x.x; acc[j][1] = x.y; acc[j][2] = y.x; acc[j][3] = y.y;
        } else acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const float* q0 = sQ + (m * 16 + g) * PQ + tq;
    const float* s0 = sS + tq * PS + half * (dv / 2) + g;
    for (int k = 0; k < dk; k += 8) {
        uint32_t ah[4], al[4];
        split_tf32(q0[k], ah[0], al[0]);
        split_tf32(q0[8 * PQ + k], ah[1], al[1]);
        split_tf32(q0[k + 4], ah[2], al[2]);
        split_tf32(q0[8 * PQ + k + 4], ah[3], al[3]);
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            if (j < nt) {
                uint32_t bh0, bl0, bh1, bl1;
                split_tf32(s0[k * PS + j * 8], bh0, bl0);
                split_tf32(s0[(k + 4) * PS + j * 8], bh1, bl1);
                mma_tf32_1688(acc[j], al, bh0, bh1);
                mma_tf32_1688(acc[j], ah, bl0, bl1);
                mma_tf32_1688(acc[j], ah, bh0, bh1);
            }
        }
    }
    // ---- head norm over both column halves, gate, store
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < kNT; ++j) {
        ss[0] += acc[j][0] * acc[j][0] + acc[j][1] * acc[j][1];
        ss[1] += acc[j][2] * acc[j][2] + acc[j][3] * acc[j][3];
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
        if (tq == 0) s_ss[half][m * 16 + g + 8 * r] = ss[r];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int lr = m * 16 + g + 8 * r;
        if (lr >= n) continue;
        const float inv = rsqrtf((s_ss[0][lr] + s_ss[1][lr]) / (float)a.dv_true + a.eps);
        const size_t row = (size_t)row0 + lr;
        const __nv_bfloat16* gp = reinterpret_cast<const __nv_bfloat16*>(a.proj) + row * a.ld + a.g_off + h * dv;
        __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + row * a.H * dv + h * dv;
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            if (j < nt) {
                const int d = half * (dv / 2) + j * 8 + 2 * tq;
                const float2 wv = *reinterpret_cast<const float2*>(a.norm_w + d);
                float gx = 1.f, gy = 1.f;
                if (!FORGET || a.g_off >= 0) {
                    const float2 gv = bf16x2_bits_to_f32x2(*reinterpret_cast<const uint32_t*>(gp + d));
                    gx = silu_f(gv.x); gy = silu_f(gv.y);
                }
                *reinterpret_cast<uint32_t*>(out + d) = f32x2_to_bf16x2_bits(acc[j][2 * r] * inv * wv.x * gx, acc[j][2 * r + 1] * inv * wv.y * gy);
            }
        }
    }
}

template <int DKT, int DVT, bool FORGET>
static int launch_gla_chunked(const GlaArgs& a, int blocks, cudaStream_t stream) {
    const size_t s1 = gla_prep_smem_floats(a.dk, a.dv) * 4, s2 = ((size_t)kGC * (a.dk + 4) + (size_t)a.dk * (a.dv + 8)) * 4;
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(gla_prepare_kernel<DKT, DVT, FORGET>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        cudaFuncSetAttribute(gla_output_kernel<DKT, DVT, FORGET>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        set = true;
    }
    gla_prepare_kernel<DKT, DVT, FORGET><<<dim3(blocks, a.H), kGPrepThreads, s1, stream>>>(a);
    int e = PS_LAUNCH_CHECK();
    if (e) return e;
    const long long groups = (long long)a.H * a.dk * a.dv / 4;
    gla_scan_kernel<<<dim3((unsigned)((groups + 255) / 256), a.n_seqs), 256, 0, stream>>>(a);
    if ((e = PS_LAUNCH_CHECK())) return e;
    gla_output_kernel<DKT, DVT, FORGET><<<dim3(blocks, a.H), kGOutThreads, s2, stream>>>(a);
    return PS_LAUNCH_CHECK();
}

template <bool FORGET>
static int launch_gla(const GlaArgs& a, int chunked, int f32, int blocks, cudaStream_t stream) {
    const int dk = a.dk, dv = a.dv;
    if (chunked) {
        if (dk == 128 && dv == 128) return launch_gla_chunked<128, 128, FORGET>(a, blocks, stream);
        if (dk == 64 && dv == 64) return launch_gla_chunked<64, 64, FORGET>(a, blocks, stream);
        return launch_gla_chunked<0, 0, FORGET>(a, blocks, stream);
    }
    const size_t smem = ((size_t)3 * dk + dv + 1024) * 4;
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(a.H, a.n_seqs);
    if (f32) return launch_pdl(gla_rows_kernel<float, 0, 0, FORGET>, grid, dim3(256), smem, stream, a);
    if (dk == 128 && dv == 128) return launch_pdl(gla_rows_kernel<__nv_bfloat16, 128, 128, FORGET>, grid, dim3(256), smem, stream, a);
    if (dk == 64 && dv == 64) return launch_pdl(gla_rows_kernel<__nv_bfloat16, 64, 64, FORGET>, grid, dim3(256), smem, stream, a);
    return launch_pdl(gla_rows_kernel<__nv_bfloat16, 0, 0, FORGET>, grid, dim3(256), smem, stream, a);
}

}  // namespace ps

PS_DEFINE_LIMITS_SETTER(gla)

// Rows of the chunked path's blocks, and whether it takes a head geometry (shared-memory plan and tile multiples).
PS_API int ps_gla_block_rows() { return ps::kGC; }
PS_API int ps_gla_chunked_ok(int dk, int dv, int rank) {
    if (dk % 16 || dv % 32 || dk > 256 || dv > 256 || rank < 0) return 0;
    if (ps::gla_prep_smem_floats(dk, dv) * 4 > 226 * 1024 || ((size_t)ps::kGC * (dk + 4) + (size_t)dk * (dv + 8)) * 4 > 226 * 1024) return 0;
    return (size_t)ps::kGC * rank + (size_t)dk * (rank + 1) <= (size_t)ps::kGC * (2 * dk + 12) ? 1 : 0;
}

// `chunked` = 0: every sequence with at most `rows_limit` rows (0 = all) row by row, bf16 or (`f32`) 32-bit;
// `chunked` = 1: the sequences with more than `rows_limit` rows, `blocks` = the sum of their ceil(rows / 64), bf16 only, scratch
// sizes as in GlaArgs.  dk a multiple of 16, dv of 32 (at most 1024), row pitch and offsets multiples of 8 elements.
// `lower` not null: the FORGET variants (`rank` 0, `a2` null, z at `a_off`, `k_off` unused); `g_off` -1 there: no output gate.
// Both forms may load a slot's state before the stream predecessor has finished (see ps_gdn_rows).
PS_API int ps_gla(int chunked, const void* proj, int ld, int f32, int H, int dk, int dv, int dv_true, int q_off, int k_off, int v_off,
                  int g_off, int a_off, int rank, float q_scale, float inv_tau, float eps, const void* a2, const void* a2_bias,
                  const void* norm_w, const void* lower, void* state, const void* seqs, int n_seqs, int rows_limit, void* out, int blocks, void* qd,
                  void* oi, void* u, void* dec, cudaStream_t stream) {
    using namespace ps;
    if (n_seqs <= 0 || H <= 0 || dk <= 0 || dk % 16 || dv <= 0 || dv % 32 || dv > 1024 || dv_true < 1 || dv_true > dv || rank < (lower != nullptr ? 0 : 1) ||
        rank % 8 || ((ld | q_off | k_off | v_off | a_off) % 8) || (lower != nullptr && g_off < 0 ? false : g_off % 8 != 0) || ((uintptr_t)proj | (uintptr_t)state) % 16)
        return (int)cudaErrorInvalidValue;
    GlaArgs a;
    a.proj = proj; a.ld = ld; a.H = H; a.dk = dk; a.dv = dv; a.dv_true = dv_true; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off;
    a.g_off = g_off; a.a_off = a_off; a.rank = rank; a.q_scale = q_scale; a.inv_tau = inv_tau; a.eps = eps; a.a2 = a2;
    a.a2_bias = (const float*)a2_bias; a.norm_w = (const float*)norm_w; a.lower = (const float*)lower; a.state = (float*)state; a.seqs = (const GlaSeq*)seqs;
    a.n_seqs = n_seqs; a.out = out; a.rows_limit = rows_limit; a.qd = (float*)qd; a.oi = (float*)oi; a.u = (float*)u; a.dec = (float*)dec;
    if (chunked && (f32 || blocks <= 0 || !ps_gla_chunked_ok(dk, dv, rank) || qd == nullptr || oi == nullptr || u == nullptr || dec == nullptr))
        return (int)cudaErrorInvalidValue;
    return lower != nullptr ? launch_gla<true>(a, chunked, f32, blocks, stream) : launch_gla<false>(a, chunked, f32, blocks, stream);
}
