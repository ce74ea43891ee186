// Delta rule with a decay per head and key channel: everything between the input projection and the output projection.
//
// Per value head (consecutive ones share a query / key head), with x the causal convolution + silu of a projected channel:
//     q = x_q / |x_q| / sqrt(dk),  k = x_k / |x_k|,  v = x_v,  beta = sigmoid(b),  g = exp(-rate softplus(a2 a + dt_bias))
//     S <- diag(g) S ;  u = beta (v - S^T k) ;  S <- S + k u^T ;  o = S^T q ;  out = rms(o) * w * sigmoid(g2 gi)
// (a, gi: the row's low-rank inputs of decay and gate).  All of it is fp32 from the projection on, the state too.
//
// The convolution's history is state: [slots, taps - 1, heads, 2 dk + dv], the projected row of position p in row p % (taps - 1).
// Every value head has a copy of its query and key channels, so heads share nothing.
//
// ps_delta_rows: row-sequential, one CTA per (sequence, head).  Decode, short portions, and the 32-bit engines.  Heads of 64 or 128
// channels keep the state in registers, others update it in place.
//
// ps_delta_chunked: portions of many rows, heads of 64 or 128 channels, in blocks of C = 64 rows.  With B_t the running sum of the
// log-decays in the block (a vector over the key channels), S0 the state before it and
//     A[t][s] = beta_t sum_d k_t k_s exp(B_t - B_s)  (s < t),   M[t][s] = sum_d q_t k_s exp(B_t - B_s)  (s <= t),
// the recurrence is (I + A) Delta = diag(beta) (V - (k exp(B)) S0),  o_t = (q_t exp(B_t)) S0 + M Delta,
// S_end = diag(exp(B_end)) S0 + (k exp(B_end - B))^T Delta.  With T = (I + A)^-1 everything but the state is independent of it:
//   delta_prepare  per (block, head): convolutions, unit vectors, decays; M, T, W = T diag(beta) (k exp(B)), U = T diag(beta) V and the
//                  decayed queries and keys
//   delta_scan     per (sequence, head, 32 value columns): Delta = U - W S0,  o = Qd S0 + M Delta,  S = diag(dec) S0 + Kd^T Delta
//   delta_finish   per (block, head): head norm, output gate, and the convolution's history
// No exponential of a positive number is formed, whatever the decays: the triangles are cut into 16-row sub-blocks; off the diagonal
// exp(B_t - B_s) factors through the end of the key's sub-block and of the sub-block before the query's, on the diagonal it is
// evaluated pair by pair.  (The triangular form is that of "Parallelizing Linear Transformers with the Delta Rule over Sequence Length"
// by Songlin Yang, Bailin Wang, Yu Zhang, Yikang Shen and Yoon Kim; sub-blocks as in gla.cu.)
// The products of delta_prepare run on TF32 mma.sync with both operands split into two terms, those of the scan on bf16 mma.sync with
// both operands split into two bf16 terms (16 bits of mantissa); sums and the state are fp32.
#include "ps_common.cuh"

namespace ps {

struct DeltaSeq { int row_start, n_rows, slot, pos_start; };

struct DeltaArgs {
    const void* proj; int ld, H, G, dk, dv, dk_true, dv_true;
    int q_off, b_off, a_off, g_off, ra, rg, taps;
    float eps;
    const void* conv;                  // [taps, 2 G dk + H dv]
    const void* a2; const float* dt_bias; const float* rate; const void* g2; const float* norm_w;
    void* history;
    float* state;                      // [slots, H, dk, dv]
    const DeltaSeq* seqs; int n_seqs;
    void* out;                         // [rows, H * dv]
    int rows_limit;                    // rows kernel: skip sequences with more rows (0: none); chunked: skip those with at most that many
};

template <typename T> __device__ __forceinline__ T dr_cast(float v);
template <> __device__ __forceinline__ float dr_cast<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 dr_cast<__nv_bfloat16>(float v) { return f32_to_bf16(v); }
__device__ __forceinline__ float dr_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float dr_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// sum over eight elements of w * x
__device__ __forceinline__ float dr_dot8(const __nv_bfloat16* w, const float* x, float acc) {
    const uint4 v = *reinterpret_cast<const uint4*>(w);
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = bf16x2_bits_to_f32x2(u[i]);
        acc = fmaf(f.x, x[2 * i], acc);
        acc = fmaf(f.y, x[2 * i + 1], acc);
    }
    return acc;
}
__device__ __forceinline__ float dr_dot8(const float* w, const float* x, float acc) {
#pragma unroll
    for (int i = 0; i < 8; ++i) acc = fmaf(w[i], x[i], acc);
    return acc;
}
__device__ __forceinline__ void dr_prefetch(const void* p, size_t bytes) {
    for (size_t i = (size_t)threadIdx.x * 128; i < bytes; i += (size_t)blockDim.x * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(p) + i));
}

// Column of the projection (from q_off on: the convolution's channel) that channel c of value head h reads.
__device__ __forceinline__ int dr_column(const DeltaArgs& a, int h, int c) {
    const int hk = h / (a.H / a.G);
    if (c < a.dk) return hk * a.dk + c;
    if (c < 2 * a.dk) return (a.G + hk) * a.dk + c - a.dk;
    return 2 * a.G * a.dk + h * a.dv + c - 2 * a.dk;
}

// The portion's last rows replace the history (every thread of the CTA; all reads of it lie before).
template <typename T>
__device__ __forceinline__ void dr_store_history(const DeltaArgs& a, const DeltaSeq& sd, int h) {
    const int back = a.taps - 1, CH = 2 * a.dk + a.dv;
    for (int r = max(0, sd.n_rows - back); r < sd.n_rows; ++r) {
        const T* src = reinterpret_cast<const T*>(a.proj) + (size_t)(sd.row_start + r) * a.ld + a.q_off;
        T* dst = reinterpret_cast<T*>(a.history) + (((size_t)sd.slot * back + (sd.pos_start + r) % back) * a.H + h) * CH;
        for (int c = threadIdx.x; c < CH; c += blockDim.x) dst[c] = src[dr_column(a, h, c)];
    }
}

// ------------------------------------------------------------------------------------------------ row-sequential form
template <typename T, int DK, int DV>
__global__ void __launch_bounds__(256, 2) delta_rows_kernel(const DeltaArgs a) {
    extern __shared__ __align__(16) float dr_smem[];
    const int dk = DK > 0 ? DK : a.dk, dv = DV > 0 ? DV : a.dv, CH = 2 * dk + dv;
    const int CG = dv / 4, RG = 256 / CG;              // column groups of four, row groups
    float* s_x = dr_smem;                              // [2 dk + dv]: q, k, v behind convolution and silu
    float* s_al = s_x + CH;                            // [dk]
    float* s_gate = s_al + dk;                         // [dv]
    float* s_low = s_gate + dv;                        // [ra + rg]
    float* s_u = s_low + a.ra + a.rg;                  // [dv]
    float* s_pk = s_u + dv;                            // [RG][dv], at most 1024
    float* s_pq = s_pk + 1024;
    __shared__ float red[96];
    const int h = blockIdx.x, t = threadIdx.x;
    const DeltaSeq sd = a.seqs[blockIdx.y];
    if (sd.n_rows <= 0 || sd.slot < 0 || (a.rows_limit > 0 && sd.n_rows > a.rows_limit)) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows) && sd.pos_start >= 0);
    const int cg = t % CG, rg = t / CG, C = 2 * a.G * dk + a.H * dv, back = a.taps - 1;
    const bool active = rg < RG;
    constexpr int kR = DK > 0 ? DK * DV / 1024 : 1;
    float* sp = a.state + ((size_t)sd.slot * a.H + h) * dk * dv;
    const T* a2 = reinterpret_cast<const T*>(a.a2) + (size_t)h * dk * a.ra;
    const T* g2 = reinterpret_cast<const T*>(a.g2) + (size_t)h * dv * a.rg;
    const T* conv = reinterpret_cast<const T*>(a.conv);
    cudaTriggerProgrammaticLaunchCompletion();
    dr_prefetch(a2, (size_t)dk * a.ra * sizeof(T));
    dr_prefetch(g2, (size_t)dv * a.rg * sizeof(T));
    float S[kR][4];
    if constexpr (DK > 0) {
        // the state was last written by an earlier step, not by the stream predecessor
#pragma unroll
        for (int r = 0; r < kR; ++r) {
            const float4 x = *reinterpret_cast<const float4*>(sp + (size_t)(rg + RG * r) * DV + cg * 4);
            S[r][0] = x.x; S[r][1] = x.y; S[r][2] = x.z; S[r][3] = x.w;
        }
    }
    const float rate = a.rate[h];
    cudaGridDependencySynchronize();
    const T* hist = reinterpret_cast<const T*>(a.history) + ((size_t)sd.slot * back * a.H + h) * CH;
    for (int i = 0; i < sd.n_rows; ++i) {
        const int row = sd.row_start + i, pos = sd.pos_start + i;
        const T* pr = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.ld;
        for (int c = t; c < CH; c += 256) {
            const int col = dr_column(a, h, c);
            float y = 0.f;
            for (int j = min(back, pos); j >= 0; --j) {
                const float x = j <= i ? (float)pr[a.q_off + col - (ptrdiff_t)j * a.ld] : (float)hist[(size_t)((pos - j) % back) * a.H * CH + c];
                y = fmaf((float)conv[(size_t)(back - j) * C + col], x, y);
            }
            s_x[c] = dr_silu(y);
        }
        for (int r = t; r < a.ra + a.rg; r += 256) s_low[r] = (float)pr[r < a.ra ? a.a_off + r : a.g_off + r - a.ra];
        __syncthreads();
        // decay and gate: two threads per channel, each every other group of eight
        for (int e = t; e < 2 * dk; e += 256) {
            float z = 0.f;
            for (int r = (e & 1) * 8; r < a.ra; r += 16) z = dr_dot8(a2 + (size_t)(e >> 1) * a.ra + r, s_low + r, z);
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            if (!(e & 1)) s_al[e >> 1] = expf(-rate * dr_softplus(z + a.dt_bias[h * dk + (e >> 1)]));
        }
        for (int e = t; e < 2 * dv; e += 256) {
            float z = 0.f;
            for (int r = (e & 1) * 8; r < a.rg; r += 16) z = dr_dot8(g2 + (size_t)(e >> 1) * a.rg + r, s_low + a.ra + r, z);
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            if (!(e & 1)) s_gate[e >> 1] = dr_sigmoid(z);
        }
        float s3[3] = {0.f, 0.f, 0.f};
        for (int d = t; d < dk; d += 256) {
            const float q = s_x[d], k = s_x[dk + d];
            s3[0] = fmaf(q, q, s3[0]); s3[1] = fmaf(k, k, s3[1]); s3[2] = fmaf(q, k, s3[2]);
        }
        block_sum_n<3>(s3, red);                       // (its barriers publish the decays and gates too)
        const float qn = rsqrtf(s3[0] + 1e-6f) * rsqrtf((float)a.dk_true), kn = rsqrtf(s3[1] + 1e-6f), kq = s3[2] * qn * kn;
        const float beta = dr_sigmoid((float)pr[a.b_off + h]);
        // one pass over the decayed state: S^T k and S^T q
        float pk[4] = {0.f, 0.f, 0.f, 0.f}, pq[4] = {0.f, 0.f, 0.f, 0.f};
        if (active) {
            if constexpr (DK > 0) {
#pragma unroll
                for (int r = 0; r < kR; ++r) {
                    const int d = rg + RG * r;
                    const float al = s_al[d], k = s_x[dk + d] * kn, q = s_x[d] * qn;
#pragma unroll
                    for (int c = 0; c < 4; ++c) { S[r][c] *= al; pk[c] = fmaf(S[r][c], k, pk[c]); pq[c] = fmaf(S[r][c], q, pq[c]); }
                }
            } else {
                for (int d = rg; d < dk; d += RG) {
                    const float4 x = *reinterpret_cast<const float4*>(sp + (size_t)d * dv + cg * 4);
                    const float al = s_al[d], k = s_x[dk + d] * kn, q = s_x[d] * qn;
                    const float y[4] = {x.x * al, x.y * al, x.z * al, x.w * al};
#pragma unroll
                    for (int c = 0; c < 4; ++c) { pk[c] = fmaf(y[c], k, pk[c]); pq[c] = fmaf(y[c], q, pq[c]); }
                }
            }
            *reinterpret_cast<float4*>(s_pk + rg * dv + cg * 4) = make_float4(pk[0], pk[1], pk[2], pk[3]);
            *reinterpret_cast<float4*>(s_pq + rg * dv + cg * 4) = make_float4(pq[0], pq[1], pq[2], pq[3]);
        }
        __syncthreads();
        // u = beta (v - S^T k);  o = (S + k u^T)^T q = S^T q + (k . q) u
        float ss = 0.f;
        for (int d = t; d < dv; d += 256) {
            float kv = 0.f, qv = 0.f;
            for (int r = 0; r < RG; ++r) { kv += s_pk[r * dv + d]; qv += s_pq[r * dv + d]; }
            const float u = beta * (s_x[2 * dk + d] - kv), o = fmaf(kq, u, qv);
            s_u[d] = u;
            s_pq[d] = o;                               // this thread alone has read and reads column d
            ss = fmaf(o, o, ss);
        }
        ss = block_sum(ss, red);                       // (publishes u)
        const float inv = rsqrtf(ss / (float)a.dv_true + a.eps);
        T* out = reinterpret_cast<T*>(a.out) + (size_t)row * a.H * dv + h * dv;
        for (int d = t; d < dv; d += 256) out[d] = dr_cast<T>(s_pq[d] * inv * a.norm_w[d] * s_gate[d]);
        if (active) {
            const float4 u = *reinterpret_cast<const float4*>(s_u + cg * 4);
            if constexpr (DK > 0) {
#pragma unroll
                for (int r = 0; r < kR; ++r) {
                    const float k = s_x[dk + rg + RG * r] * kn;
                    S[r][0] = fmaf(k, u.x, S[r][0]); S[r][1] = fmaf(k, u.y, S[r][1]); S[r][2] = fmaf(k, u.z, S[r][2]); S[r][3] = fmaf(k, u.w, S[r][3]);
                }
            } else {
                for (int d = rg; d < dk; d += RG) {
                    float4* s4 = reinterpret_cast<float4*>(sp + (size_t)d * dv + cg * 4);
                    float4 x = *s4;
                    const float al = s_al[d], k = s_x[dk + d] * kn;
                    x.x = fmaf(k, u.x, x.x * al); x.y = fmaf(k, u.y, x.y * al); x.z = fmaf(k, u.z, x.z * al); x.w = fmaf(k, u.w, x.w * al);
                    *s4 = x;
                }
            }
        }
        __syncthreads();                               // the next row rewrites the shared buffers
    }
    if constexpr (DK > 0) {
#pragma unroll
        for (int r = 0; r < kR; ++r)
            *reinterpret_cast<float4*>(sp + (size_t)(rg + RG * r) * DV + cg * 4) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    }
    if (back > 0) dr_store_history<T>(a, sd, h);
}

// ------------------------------------------------------------------------------------------------ chunked form (bf16 engines)
constexpr int kDC = 64;                 // rows of a block
constexpr int kDPrepThreads = 512, kDScanThreads = 256, kDFinThreads = 256;
constexpr int kDSlice = 32;             // value columns of a scan CTA
constexpr int kDTP = kDC + 4;

struct DeltaChunkArgs {
    DeltaArgs a;
    __nv_bfloat16* mats;                // per (block, head): W, Qd, Kd [64, dk] and M [64, 64], each as a high and a low part
    float* u;                           // per (block, head): [64, dv]
    float* dec;                         // per (block, head): [dk]
    float* o;                           // [rows, H * dv]
};
__host__ __device__ constexpr size_t delta_mats(int dk) { return (size_t)2 * (3 * kDC * dk + kDC * kDC); }

// Which sequence and block of it a global block index is; false: none.
__device__ __forceinline__ bool delta_find_block(const DeltaArgs& a, int blk, DeltaSeq& sd, int& chunk) {
    int base = 0;
    for (int s = 0; s < a.n_seqs; ++s) {
        const DeltaSeq d = a.seqs[s];
        if (d.n_rows <= a.rows_limit || d.slot < 0) continue;
        const int nb = (d.n_rows + kDC - 1) / kDC;
        if (blk < base + nb) { sd = d; chunk = blk - base; return true; }
        base += nb;
    }
    return false;
}

__device__ __forceinline__ uint32_t dr_tf32(float x) { uint32_t r; asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x)); return r; }
__device__ __forceinline__ void dr_split(float x, uint32_t& hi, uint32_t& lo) {
    hi = dr_tf32(x);
    lo = dr_tf32(x - __uint_as_float(hi));
}
__device__ __forceinline__ void dr_mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dr_mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dr_ldsm(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void dr_ldsm_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)) : "memory");
}
__device__ __forceinline__ void dr_cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
// Two neighbouring values as bf16 pairs: rounded, and what is left.
__device__ __forceinline__ void dr_halves(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = f32x2_to_bf16x2_bits(x, y);
    const float2 f = bf16x2_bits_to_f32x2(hi);
    lo = f32x2_to_bf16x2_bits(x - f.x, y - f.y);
}
__device__ __forceinline__ void dr_widen(const uint4& v, float (&f)[8]) {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 t = bf16x2_bits_to_f32x2(u[i]); f[2 * i] = t.x; f[2 * i + 1] = t.y; }
}

// Convolution + silu of eight channels over four consecutive rows of a block.  `src`: row 0 of the block at the channels, `hist`: the
// head's history at the channels (rows of `hist_ld`), `w`: the taps at the channels (rows of C); rows from n on become zero.
template <int TAPS>
__device__ __forceinline__ void delta_conv(const __nv_bfloat16* src, int ld, const __nv_bfloat16* hist, size_t hist_ld, const __nv_bfloat16* w, int C,
                                           int taps, int r0, int n, int before, int pos0, float* dst, int pitch) {
    constexpr int kRun = 4;
    const int T = TAPS > 0 ? TAPS : taps, back = T - 1;
    auto row = [&](int r) {                            // `before`: rows of the portion ahead of the block
        if (r >= n || pos0 + r < 0) return make_uint4(0, 0, 0, 0);
        if (r + before >= 0) return *reinterpret_cast<const uint4*>(src + (ptrdiff_t)r * ld);
        return *reinterpret_cast<const uint4*>(hist + (size_t)((pos0 + r) % back) * hist_ld);
    };
    float y[kRun][8];
#pragma unroll
    for (int i = 0; i < kRun; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = 0.f;
    if constexpr (TAPS > 0) {
        uint4 x[kRun + TAPS - 1];
#pragma unroll
        for (int i = 0; i < kRun + TAPS - 1; ++i) x[i] = row(r0 + i - (TAPS - 1));
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {               // tap j meets the row TAPS - 1 - j before
            float wv[8];
            dr_widen(*reinterpret_cast<const uint4*>(w + (size_t)j * C), wv);
#pragma unroll
            for (int i = 0; i < kRun; ++i) {
                float xv[8];
                dr_widen(x[i + j], xv);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[i][e] = fmaf(wv[e], xv[e], y[i][e]);
            }
        }
    } else {
        for (int j = 0; j < T; ++j) {
            float wv[8];
            dr_widen(*reinterpret_cast<const uint4*>(w + (size_t)j * C), wv);
#pragma unroll
            for (int i = 0; i < kRun; ++i) {
                float xv[8];
                dr_widen(row(r0 + i - (back - j)), xv);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[i][e] = fmaf(wv[e], xv[e], y[i][e]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
        if (r0 + i >= n) {
#pragma unroll
            for (int e = 0; e < 8; ++e) y[i][e] = 0.f;
        }
#pragma unroll
        for (int e = 0; e < 8; e += 4)
            *reinterpret_cast<float4*>(dst + (r0 + i) * pitch + e) = make_float4(silu_f(y[i][e]), silu_f(y[i][e + 1]), silu_f(y[i][e + 2]), silu_f(y[i][e + 3]));
    }
}

__host__ __device__ constexpr size_t delta_prep_floats(int dk, int dv) {
    return (size_t)3 * kDC * (dk + 4) + (size_t)kDC * (dv + 8) + 3 * kDC * kDTP + 3 * 16 * 17 + 4 * dk + kDC;
}

// grid = (blocks, H)
template <int DK, int DV, int TAPS>
__global__ void __launch_bounds__(kDPrepThreads, 1) delta_prepare_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) float dr_smem[];
    const DeltaArgs& a = c.a;
    constexpr int P = DK + 4, PV = DV + 8, NW = kDPrepThreads / 32;
    float* sQ = dr_smem;                                // [64][P]
    float* sK = sQ + kDC * P;                           // [64][P]  k, later decayed to the end of its sub-block
    float* sB = sK + kDC * P;                           // [64][P]  running log-decays, later k decayed from the start
    float* sV = sB + kDC * P;                           // [64][PV]
    float* sA = sV + kDC * PV;                          // [64][68]
    float* sM = sA + kDC * kDTP;                        // [64][68]
    float* sT = sM + kDC * kDTP;                        // [64][68]
    float* sX = sT + kDC * kDTP;                        // [3][16][17]
    float* sE = sX + 3 * 16 * 17;                       // [4][DK]  log-decay sums of the sub-blocks, then up to their ends
    float* sBeta = sE + 4 * DK;                         // [64]
    DeltaSeq sd; int chunk;
    if (!delta_find_block(a, blockIdx.x, sd, chunk)) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows) && sd.pos_start >= 0);
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const int before = chunk * kDC, n = min(kDC, sd.n_rows - before), pos0 = sd.pos_start + before, back = a.taps - 1;
    const size_t bh = (size_t)blockIdx.x * a.H + h;
    const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj) + (size_t)(sd.row_start + before) * a.ld;
    const __nv_bfloat16* conv = reinterpret_cast<const __nv_bfloat16*>(a.conv);
    const int CH = 2 * DK + DV, C = 2 * a.G * DK + a.H * DV;

    // ---- convolutions
    for (int i = t; i < kDC / 4 * (CH / 8); i += kDPrepThreads) {
        const int ch = i % (CH / 8) * 8, r0 = i / (CH / 8) * 4, col = dr_column(a, h, ch);
        const __nv_bfloat16* hist = reinterpret_cast<const __nv_bfloat16*>(a.history) + ((size_t)sd.slot * back * a.H + h) * CH + ch;
        const bool is_v = ch >= 2 * DK;
        float* dst = is_v ? sV + ch - 2 * DK : ch < DK ? sQ + ch : sK + ch - DK;
        delta_conv<TAPS>(proj + a.q_off + col, a.ld, hist, (size_t)a.H * CH, conv + col, C, a.taps, r0, n, before, pos0, dst, is_v ? PV : P);
    }
    if (t < kDC) sBeta[t] = t < n ? dr_sigmoid(bf16_to_f32(proj[(size_t)t * a.ld + a.b_off + h])) : 0.f;
    // ---- log-decays: rows of low-rank inputs times the head's rows of a2, on the tensor cores; a warp has 16 rows and DK / 4 channels
    {
        constexpr int kNT = DK / 32;
        const int m = warp & 3, n0 = (warp >> 2) * (DK / 4);
        float z[kNT][4];
#pragma unroll
        for (int j = 0; j < kNT; ++j) z[j][0] = z[j][1] = z[j][2] = z[j][3] = 0.f;
        const int rlo = min(m * 16 + g, n - 1), rhi = min(m * 16 + g + 8, n - 1);        // (rows behind the last are not used)
        const __nv_bfloat16* lo = proj + (size_t)rlo * a.ld + a.a_off + 2 * tq;
        const __nv_bfloat16* hi = proj + (size_t)rhi * a.ld + a.a_off + 2 * tq;
        const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.a2) + ((size_t)h * DK + n0 + g) * a.ra + 2 * tq;
        for (int k = 0; k < a.ra; k += 16) {
            const uint32_t af[4] = {*reinterpret_cast<const uint32_t*>(lo + k), *reinterpret_cast<const uint32_t*>(hi + k),
                                    *reinterpret_cast<const uint32_t*>(lo + k + 8), *reinterpret_cast<const uint32_t*>(hi + k + 8)};
#pragma unroll
            for (int j = 0; j < kNT; ++j) {
                const __nv_bfloat16* wp = w + (size_t)j * 8 * a.ra + k;
                dr_mma_bf16(z[j], af, *reinterpret_cast<const uint32_t*>(wp), *reinterpret_cast<const uint32_t*>(wp + 8));
            }
        }
        const float rate = a.rate[h];
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            const int d = n0 + j * 8 + 2 * tq;
            const float b0 = a.dt_bias[h * DK + d], b1 = a.dt_bias[h * DK + d + 1];
            const int r0 = m * 16 + g, r1 = r0 + 8;
            *reinterpret_cast<float2*>(sB + r0 * P + d) = r0 < n ? make_float2(-rate * dr_softplus(z[j][0] + b0), -rate * dr_softplus(z[j][1] + b1)) : make_float2(0.f, 0.f);
            *reinterpret_cast<float2*>(sB + r1 * P + d) = r1 < n ? make_float2(-rate * dr_softplus(z[j][2] + b0), -rate * dr_softplus(z[j][3] + b1)) : make_float2(0.f, 0.f);
        }
    }
    __syncthreads();
    // ---- running sums, 16 rows at a time; unit vectors
    if (t < 4 * DK) {
        const int blk = t / DK, d = t % DK;
        float s = 0.f;
#pragma unroll
        for (int r = 0; r < 16; ++r) { s += sB[(blk * 16 + r) * P + d]; sB[(blk * 16 + r) * P + d] = s; }
        sE[t] = s;
    }
    {
        constexpr int kU = DK / 32;
        const float qs = rsqrtf((float)a.dk_true);
#pragma unroll
        for (int i = 0; i < kDC / NW; ++i) {
            const int r = warp * (kDC / NW) + i;
            float q[kU], k[kU], qq = 0.f, kk = 0.f;
#pragma unroll
            for (int u = 0; u < kU; ++u) {
                q[u] = sQ[r * P + lane + 32 * u]; k[u] = sK[r * P + lane + 32 * u];
                qq = fmaf(q[u], q[u], qq); kk = fmaf(k[u], k[u], kk);
            }
            const float fq = rsqrtf(warp_sum(qq) + 1e-6f) * qs, fk = rsqrtf(warp_sum(kk) + 1e-6f);
#pragma unroll
            for (int u = 0; u < kU; ++u) { sQ[r * P + lane + 32 * u] = q[u] * fq; sK[r * P + lane + 32 * u] = k[u] * fk; }
        }
    }
    __syncthreads();
    // ---- diagonal sub-blocks, pair by pair, two keys at a time (sums local to the sub-block suffice: only differences enter)
#pragma unroll 1
    for (int blk = 0; blk < 4; ++blk) {
        constexpr int kU = DK / 32;
        const int il = (blk & 1) ? 15 - warp : warp, i = blk * 16 + il, d = lane * kU;
        auto load = [&](const float* p, float (&v)[kU]) {
            if constexpr (kU == 4) *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
            else *reinterpret_cast<float2*>(v) = *reinterpret_cast<const float2*>(p);
        };
        float qi[kU], ki[kU], bi[kU];
        load(sQ + i * P + d, qi); load(sK + i * P + d, ki); load(sB + i * P + d, bi);
        for (int jl = 0; jl <= il; jl += 2) {
            float v[4];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int j = blk * 16 + min(jl + e, il);
                float kj[kU], bj[kU], s0 = 0.f, s1 = 0.f;
                load(sK + j * P + d, kj); load(sB + j * P + d, bj);
#pragma unroll
                for (int u = 0; u < kU; ++u) {
                    const float f = kj[u] * __expf(bi[u] - bj[u]);
                    s0 = fmaf(qi[u], f, s0); s1 = fmaf(ki[u], f, s1);
                }
                v[2 * e] = s0; v[2 * e + 1] = s1;
            }
            // four sums over the warp at once: lanes 0, 8, 16, 24 end with one each
            const bool up = lane & 16, odd = lane & 8;
            float x = (up ? v[2] : v[0]) + __shfl_xor_sync(0xffffffffu, up ? v[0] : v[2], 16);
            float y = (up ? v[3] : v[1]) + __shfl_xor_sync(0xffffffffu, up ? v[1] : v[3], 16);
            float s = (odd ? y : x) + __shfl_xor_sync(0xffffffffu, odd ? x : y, 8);
            s += __shfl_xor_sync(0xffffffffu, s, 4);
            s += __shfl_xor_sync(0xffffffffu, s, 2);
            s += __shfl_xor_sync(0xffffffffu, s, 1);
            const int j = jl + (up ? 1 : 0);
            if ((lane & 7) == 0 && j <= il) {
                if (!odd) sM[i * kDTP + blk * 16 + j] = s;
                else sA[i * kDTP + blk * 16 + j] = sBeta[i] * s;
            }
        }
    }
    __syncthreads();
    // ---- queries and keys decayed from the start of their sub-block, keys decayed to its end
    for (int i = t; i < kDC * DK / 4; i += kDPrepThreads) {
        const int r = i / (DK / 4), d = i % (DK / 4) * 4;
        float4 b = *reinterpret_cast<float4*>(sB + r * P + d), q = *reinterpret_cast<float4*>(sQ + r * P + d), k = *reinterpret_cast<float4*>(sK + r * P + d);
        const float4 e = *reinterpret_cast<const float4*>(sE + (r >> 4) * DK + d);
        const float4 f = make_float4(__expf(b.x), __expf(b.y), __expf(b.z), __expf(b.w));
        *reinterpret_cast<float4*>(sQ + r * P + d) = make_float4(q.x * f.x, q.y * f.y, q.z * f.z, q.w * f.w);
        *reinterpret_cast<float4*>(sB + r * P + d) = make_float4(k.x * f.x, k.y * f.y, k.z * f.z, k.w * f.w);
        *reinterpret_cast<float4*>(sK + r * P + d) = make_float4(k.x * __expf(e.x - b.x), k.y * __expf(e.y - b.y), k.z * __expf(e.z - b.z), k.w * __expf(e.w - b.w));
    }
    __syncthreads();
    if (t < DK) {                                       // sub-block totals -> sums up to the sub-blocks' ends
        const float e1 = sE[t] + sE[DK + t], e2 = e1 + sE[2 * DK + t], e3 = e2 + sE[3 * DK + t];
        sE[DK + t] = e1; sE[2 * DK + t] = e2; sE[3 * DK + t] = e3;
        c.dec[bh * DK + t] = expf(e3);
    }
    __syncthreads();
    // ---- below the diagonal: (query sub-block, key sub-block) x two halves of eight keys, for queries and keys at once; the solve of
    // the diagonal sub-blocks of T (thread: sub-block, column) by the last two warps
    if (warp < 12) {
        const int pair = warp >> 1, half = warp & 1;
        const int qi = pair < 1 ? 1 : (pair < 3 ? 2 : 3), kj = pair < 1 ? 0 : (pair < 3 ? pair - 1 : pair - 3);
        float am[4] = {0.f, 0.f, 0.f, 0.f}, aa[4] = {0.f, 0.f, 0.f, 0.f};
        const float* q0 = sQ + (qi * 16 + g) * P + tq;
        const float* p0 = sB + (qi * 16 + g) * P + tq;
        const float* k0 = sK + (kj * 16 + half * 8 + g) * P + tq;
#pragma unroll 2
        for (int k = 0; k < DK; k += 8) {
            float f0 = 1.f, f1 = 1.f;                   // decay from the end of the key's sub-block to the start of the query's
            if (qi - 1 > kj) {
                f0 = __expf(sE[(qi - 1) * DK + k + tq] - sE[kj * DK + k + tq]);
                f1 = __expf(sE[(qi - 1) * DK + k + tq + 4] - sE[kj * DK + k + tq + 4]);
            }
            uint32_t bh2[2], bl2[2], ah[4], al[4];
            dr_split(k0[k] * f0, bh2[0], bl2[0]);
            dr_split(k0[k + 4] * f1, bh2[1], bl2[1]);
            dr_split(q0[k], ah[0], al[0]); dr_split(q0[8 * P + k], ah[1], al[1]);
            dr_split(q0[k + 4], ah[2], al[2]); dr_split(q0[8 * P + k + 4], ah[3], al[3]);
            dr_mma_tf32(am, al, bh2[0], bh2[1]); dr_mma_tf32(am, ah, bl2[0], bl2[1]); dr_mma_tf32(am, ah, bh2[0], bh2[1]);
            dr_split(p0[k], ah[0], al[0]); dr_split(p0[8 * P + k], ah[1], al[1]);
            dr_split(p0[k + 4], ah[2], al[2]); dr_split(p0[8 * P + k + 4], ah[3], al[3]);
            dr_mma_tf32(aa, al, bh2[0], bh2[1]); dr_mma_tf32(aa, ah, bl2[0], bl2[1]); dr_mma_tf32(aa, ah, bh2[0], bh2[1]);
        }
        const int r0 = qi * 16 + g, at = r0 * kDTP + kj * 16 + half * 8 + 2 * tq;
        const float b0 = sBeta[r0], b1 = sBeta[r0 + 8];
        sM[at] = am[0]; sM[at + 1] = am[1]; sM[at + 8 * kDTP] = am[2]; sM[at + 8 * kDTP + 1] = am[3];
        sA[at] = b0 * aa[0]; sA[at + 1] = b0 * aa[1]; sA[at + 8 * kDTP] = b1 * aa[2]; sA[at + 8 * kDTP + 1] = b1 * aa[3];
    } else if (warp >= 14) {
        const int b = (t - 14 * 32) >> 4, j = t & 15;
        const float* Ab = sA + (16 * b) * kDTP + 16 * b;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s0 = i == j ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
            for (int k = 0; k < i; ++k) { if (k & 1) s1 = fmaf(-Ab[i * kDTP + k], x[k], s1); else s0 = fmaf(-Ab[i * kDTP + k], x[k], s0); }
            x[i] = s0 + s1;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) sT[(16 * b + i) * kDTP + 16 * b + j] = x[i];
    }
    __syncthreads();
    // ---- everything that is ready goes out: Qd, Kd, M; k decayed from the block's start replaces k decayed from the sub-block's
    __nv_bfloat16* mats = c.mats + bh * delta_mats(DK);
    uint32_t* gW = reinterpret_cast<uint32_t*>(mats);                   // pairs of columns; high part, then low part
    constexpr int kMat = kDC * DK / 2;
    uint32_t* gQ = gW + 2 * kMat;
    uint32_t* gK = gQ + 2 * kMat;
    uint32_t* gM = gK + 2 * kMat;
    for (int i = t; i < kMat / 2; i += kDPrepThreads) {
        const int r = i / (DK / 4), d = i % (DK / 4) * 4, blk = r >> 4;
        const float4 q = *reinterpret_cast<const float4*>(sQ + r * P + d), k = *reinterpret_cast<const float4*>(sK + r * P + d);
        float f[4], e[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            f[u] = blk > 0 ? __expf(sE[(blk - 1) * DK + d + u]) : 1.f;
            e[u] = blk < 3 ? __expf(sE[3 * DK + d + u] - sE[blk * DK + d + u]) : 1.f;
        }
        uint2 hi, lo;
        dr_halves(q.x * f[0], q.y * f[1], hi.x, lo.x); dr_halves(q.z * f[2], q.w * f[3], hi.y, lo.y);
        reinterpret_cast<uint2*>(gQ)[i] = hi; reinterpret_cast<uint2*>(gQ + kMat)[i] = lo;
        dr_halves(k.x * e[0], k.y * e[1], hi.x, lo.x); dr_halves(k.z * e[2], k.w * e[3], hi.y, lo.y);
        reinterpret_cast<uint2*>(gK)[i] = hi; reinterpret_cast<uint2*>(gK + kMat)[i] = lo;
        float4* p = reinterpret_cast<float4*>(sB + r * P + d);
        const float4 b = *p;
        *p = make_float4(b.x * f[0], b.y * f[1], b.z * f[2], b.w * f[3]);
    }
    for (int i = t; i < kDC * kDC / 2; i += kDPrepThreads) {
        const int r = i / (kDC / 2), s = i % (kDC / 2) * 2;
        uint32_t hi, lo;
        dr_halves(s <= r ? sM[r * kDTP + s] : 0.f, s + 1 <= r ? sM[r * kDTP + s + 1] : 0.f, hi, lo);
        gM[i] = hi; gM[kDC * kDC / 2 + i] = lo;
    }
    // ---- T, block rows 1 .. 3: T_ij = -T_ii (sum_{k = j .. i-1} A_ik T_kj) for all j < i at once
    for (int bi = 1; bi < 4; ++bi) {
        for (int e = t; e < bi * 256; e += kDPrepThreads) {
            const int bj = e >> 8, r = (e >> 4) & 15, cc = e & 15;
            const float* Ar = sA + (16 * bi + r) * kDTP;
            float s0 = 0.f, s1 = 0.f;
            for (int k = 16 * bj; k < 16 * bi; k += 2) {
                s0 = fmaf(Ar[k], sT[k * kDTP + 16 * bj + cc], s0);
                s1 = fmaf(Ar[k + 1], sT[(k + 1) * kDTP + 16 * bj + cc], s1);
            }
            sX[(bj * 16 + r) * 17 + cc] = s0 + s1;
        }
        __syncthreads();
        for (int e = t; e < bi * 256; e += kDPrepThreads) {
            const int bj = e >> 8, r = (e >> 4) & 15, cc = e & 15;
            const float* Tr = sT + (16 * bi + r) * kDTP + 16 * bi;
            float s = 0.f;
#pragma unroll
            for (int k = 0; k < 16; ++k) s = fmaf(Tr[k], sX[(bj * 16 + k) * 17 + cc], s);        // T_ii is zero above its diagonal
            sT[(16 * bi + r) * kDTP + 16 * bj + cc] = -s;
        }
        __syncthreads();
    }
    // ---- W = T diag(beta) K (warps 0-7) and U = T diag(beta) V (warps 8-15): a warp has 16 rows and half the columns; T is lower
    // triangular, so steps beyond the row tile are skipped
    {
        const int m = warp & 3, half = (warp >> 2) & 1;
        const bool isW = warp < NW / 2;
        constexpr int kNT = (DK > DV ? DK : DV) / 16;
        const int nt = (isW ? DK : DV) / 16, col0 = half * (isW ? DK : DV) / 2;
        const float* src = isW ? sB : sV;
        const int pitch = isW ? P : PV;
        float acc[kNT][4];
#pragma unroll
        for (int j = 0; j < kNT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        const float* tr = sT + (16 * m + g) * kDTP + tq;
        for (int k = 0; k < 16 * (m + 1); k += 8) {
            uint32_t ah[4], al[4];
            dr_split(tr[k], ah[0], al[0]); dr_split(tr[8 * kDTP + k], ah[1], al[1]);
            dr_split(tr[k + 4], ah[2], al[2]); dr_split(tr[8 * kDTP + k + 4], ah[3], al[3]);
            const float f0 = sBeta[k + tq], f1 = sBeta[k + tq + 4];
            const float* b0p = src + (k + tq) * pitch + col0 + g;
            const float* b1p = b0p + 4 * pitch;
#pragma unroll
            for (int j = 0; j < kNT; ++j) {
                if (j < nt) {
                    uint32_t bh0, bl0, bh1, bl1;
                    dr_split(b0p[8 * j] * f0, bh0, bl0);
                    dr_split(b1p[8 * j] * f1, bh1, bl1);
                    dr_mma_tf32(acc[j], al, bh0, bh1);
                    dr_mma_tf32(acc[j], ah, bl0, bl1);
                    dr_mma_tf32(acc[j], ah, bh0, bh1);
                }
            }
        }
        const int r0 = 16 * m + g;
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            if (j >= nt) continue;
            const int d = col0 + 8 * j + 2 * tq;
            if (isW) {
                uint32_t hi, lo;
                dr_halves(acc[j][0], acc[j][1], hi, lo);
                gW[(r0 * DK + d) / 2] = hi; gW[kMat + (r0 * DK + d) / 2] = lo;
                dr_halves(acc[j][2], acc[j][3], hi, lo);
                gW[((r0 + 8) * DK + d) / 2] = hi; gW[kMat + ((r0 + 8) * DK + d) / 2] = lo;
            } else {
                float* u = c.u + bh * kDC * DV;
                *reinterpret_cast<float2*>(u + (size_t)r0 * DV + d) = make_float2(acc[j][0], acc[j][1]);
                *reinterpret_cast<float2*>(u + (size_t)(r0 + 8) * DV + d) = make_float2(acc[j][2], acc[j][3]);
            }
        }
    }
}

// Shared-memory rows of the scan are padded so that eight rows of a fragment load fall into different banks.
__host__ __device__ constexpr int delta_pk(int dk) { return dk + 8; }
__host__ __device__ constexpr size_t delta_scan_bytes(int dk) {
    return (size_t)2 * 2 * (3 * kDC * delta_pk(dk) + kDC * (kDC + 8) + (dk + kDC) * (kDSlice + 8)) + (size_t)4 * kDC * (kDSlice + 8);
}

// grid = (DV / 32, H, n_seqs): a CTA walks the sequence's blocks with 32 columns of the state in its accumulator registers.
template <int DK>
__global__ void __launch_bounds__(kDScanThreads, 1) delta_scan_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) unsigned char ds_smem[];
    typedef __nv_bfloat16 bf;
    const DeltaArgs& a = c.a;
    constexpr int PK = delta_pk(DK), PM = kDC + 8, PS = kDSlice + 8, NT = kDSlice / 8, PU = kDSlice + 8;
    bf* sW = reinterpret_cast<bf*>(ds_smem);            // [2][64][PK], high and low part
    bf* sQ = sW + 2 * kDC * PK;
    bf* sK = sQ + 2 * kDC * PK;
    bf* sM = sK + 2 * kDC * PK;                         // [2][64][PM]
    bf* sS = sM + 2 * kDC * PM;                         // [2][DK][PS]  operand copy of the state
    bf* sD = sS + 2 * DK * PS;                          // [2][64][PS]  Delta
    float* sU = reinterpret_cast<float*>(sD + 2 * kDC * PS);             // [64][PU]
    const DeltaSeq sd = a.seqs[blockIdx.z];
    if (sd.slot < 0 || sd.n_rows <= a.rows_limit) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows));
    int blk = 0;
    for (int s = 0; s < (int)blockIdx.z; ++s) {
        const DeltaSeq d = a.seqs[s];
        if (d.n_rows > a.rows_limit && d.slot >= 0) blk += (d.n_rows + kDC - 1) / kDC;
    }
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const int c0 = blockIdx.x * kDSlice, dv = a.dv, m = warp & 3;
    const bool own = warp < DK / 16;                    // this warp keeps state rows 16 warp .. 16 warp + 15
    float* state = a.state + ((size_t)sd.slot * a.H + h) * DK * dv + c0;
    float S[NT][4];
    auto publish = [&]() {                              // the state as a high and a low part
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            uint32_t hi, lo;
            bf* p = sS + (16 * warp + g) * PS + 8 * j + 2 * tq;
            dr_halves(S[j][0], S[j][1], hi, lo);
            *reinterpret_cast<uint32_t*>(p) = hi; *reinterpret_cast<uint32_t*>(p + DK * PS) = lo;
            dr_halves(S[j][2], S[j][3], hi, lo);
            *reinterpret_cast<uint32_t*>(p + 8 * PS) = hi; *reinterpret_cast<uint32_t*>(p + (DK + 8) * PS) = lo;
        }
    };
    if (own) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const float2 x = *reinterpret_cast<const float2*>(state + (size_t)(16 * warp + g) * dv + 8 * j + 2 * tq);
            const float2 y = *reinterpret_cast<const float2*>(state + (size_t)(16 * warp + g + 8) * dv + 8 * j + 2 * tq);
            S[j][0] = x.x; S[j][1] = x.y; S[j][2] = y.x; S[j][3] = y.y;
        }
        publish();
    }
    auto copy = [&](bf* dst, const bf* src, int cols, int pitch) {       // both parts of a [64, cols] matrix
        const int per = cols / 8;
        for (int i = t; i < 2 * kDC * per; i += kDScanThreads) dr_cp16(dst + (i / per) * pitch + i % per * 8, src + (size_t)i * 8);
    };
    auto commit = []() { asm volatile("cp.async.commit_group;" ::: "memory"); };
    auto fetch_first = [&](int b) {                     // what the first products of a block read
        const bf* src = c.mats + ((size_t)b * a.H + h) * delta_mats(DK);
        copy(sW, src, DK, PK);
        copy(sQ, src + 2 * kDC * DK, DK, PK);
        const float* u = c.u + ((size_t)b * a.H + h) * kDC * dv + c0;
        for (int i = t; i < kDC * kDSlice / 4; i += kDScanThreads) {
            const int r = i / (kDSlice / 4), cc = i % (kDSlice / 4) * 4;
            dr_cp16(sU + r * PU + cc, u + (size_t)r * dv + cc);
        }
        commit();
    };
    // one product with split operands: the low parts' product is left out
    auto mma3 = [](float (&acc)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
        dr_mma_bf16(acc, al, bh0, bh1);
        dr_mma_bf16(acc, ah, bl0, bl1);
        dr_mma_bf16(acc, ah, bh0, bh1);
    };
    fetch_first(blk);
    for (int r0 = 0; r0 < sd.n_rows; r0 += kDC, ++blk) {
        const int n = min(kDC, sd.n_rows - r0);
        const float* dec = c.dec + ((size_t)blk * a.H + h) * DK;
        float d0 = 0.f, d1 = 0.f;
        if (own) { d0 = dec[16 * warp + g]; d1 = dec[16 * warp + g + 8]; }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();                                // W, Qd, U and the state's copy are there; Kd and M of the last block are free
        {
            const bf* src = c.mats + ((size_t)blk * a.H + h) * delta_mats(DK) + 4 * kDC * DK;
            copy(sM, src + 2 * kDC * DK, kDC, PM);
            copy(sK, src, DK, PK);
            commit();
        }
        // ---- warps 0-3: W S0, warps 4-7: Qd S0; 16 rows x 32 columns each
        float acc[NT][4];
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        {
            const bf* ap = (warp < 4 ? sW : sQ) + (16 * m + (lane & 15)) * PK + (lane >> 4) * 8;
            const bf* bp = sS + (lane & 15) * PS + (lane >> 4) * 8;
#pragma unroll
            for (int k = 0; k < DK; k += 16) {
                uint32_t ah[4], al[4];
                dr_ldsm(ah, ap + k); dr_ldsm(al, ap + kDC * PK + k);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t bh[4], bl[4];
                    dr_ldsm_t(bh, bp + k * PS + j * 8); dr_ldsm_t(bl, bp + (DK + k) * PS + j * 8);
                    mma3(acc[j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma3(acc[j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
            }
        }
        if (warp < 4) {
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int r = 16 * m + g, cc = 8 * j + 2 * tq;
                const float2 u0 = *reinterpret_cast<const float2*>(sU + r * PU + cc), u1 = *reinterpret_cast<const float2*>(sU + (r + 8) * PU + cc);
                uint32_t hi, lo;
                bf* p = sD + r * PS + cc;
                dr_halves(u0.x - acc[j][0], u0.y - acc[j][1], hi, lo);
                *reinterpret_cast<uint32_t*>(p) = hi; *reinterpret_cast<uint32_t*>(p + kDC * PS) = lo;
                dr_halves(u1.x - acc[j][2], u1.y - acc[j][3], hi, lo);
                *reinterpret_cast<uint32_t*>(p + 8 * PS) = hi; *reinterpret_cast<uint32_t*>(p + (kDC + 8) * PS) = lo;
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();                                // Delta, Kd and M are there; W, Qd, U and the state's copy are free
        if (r0 + kDC < sd.n_rows) fetch_first(blk + 1);
        // ---- o = Qd S0 + M Delta (steps above the diagonal are skipped)
        if (warp >= 4) {
            const bf* ap = sM + (16 * m + (lane & 15)) * PM + (lane >> 4) * 8;
            const bf* bp = sD + (lane & 15) * PS + (lane >> 4) * 8;
            for (int k = 0; k < 16 * (m + 1); k += 16) {
                uint32_t ah[4], al[4];
                dr_ldsm(ah, ap + k); dr_ldsm(al, ap + kDC * PM + k);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t bh[4], bl[4];
                    dr_ldsm_t(bh, bp + k * PS + j * 8); dr_ldsm_t(bl, bp + (kDC + k) * PS + j * 8);
                    mma3(acc[j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma3(acc[j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
            }
            const int lo = 16 * m + g, hi = lo + 8;
            float* o = c.o + (size_t)(sd.row_start + r0) * a.H * dv + (size_t)h * dv + c0;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int cc = 8 * j + 2 * tq;
                if (lo < n) *reinterpret_cast<float2*>(o + (size_t)lo * a.H * dv + cc) = make_float2(acc[j][0], acc[j][1]);
                if (hi < n) *reinterpret_cast<float2*>(o + (size_t)hi * a.H * dv + cc) = make_float2(acc[j][2], acc[j][3]);
            }
        }
        // ---- S = diag(dec) S0 + Kd^T Delta
        if (own) {
#pragma unroll
            for (int j = 0; j < NT; ++j) { S[j][0] *= d0; S[j][1] *= d0; S[j][2] *= d1; S[j][3] *= d1; }
            const bf* ap = sK + ((lane & 7) + ((lane >> 4) & 1) * 8) * PK + 16 * warp + ((lane >> 3) & 1) * 8;
            const bf* bp = sD + (lane & 15) * PS + (lane >> 4) * 8;
#pragma unroll
            for (int k = 0; k < kDC; k += 16) {
                uint32_t ah[4], al[4];
                dr_ldsm_t(ah, ap + k * PK); dr_ldsm_t(al, ap + (kDC + k) * PK);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    uint32_t bh[4], bl[4];
                    dr_ldsm_t(bh, bp + k * PS + j * 8); dr_ldsm_t(bl, bp + (kDC + k) * PS + j * 8);
                    mma3(S[j], ah, al, bh[0], bh[1], bl[0], bl[1]);
                    mma3(S[j + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
                }
            }
            publish();                                  // (nobody reads the copy between the two barriers)
        }
    }
    if (own) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            *reinterpret_cast<float2*>(state + (size_t)(16 * warp + g) * dv + 8 * j + 2 * tq) = make_float2(S[j][0], S[j][1]);
            *reinterpret_cast<float2*>(state + (size_t)(16 * warp + g + 8) * dv + 8 * j + 2 * tq) = make_float2(S[j][2], S[j][3]);
        }
    }
}

// grid = (blocks, H): head norm and output gate (low-rank inputs times the head's rows of g2, on the tensor cores)
template <int DV>
__global__ void __launch_bounds__(kDFinThreads) delta_finish_kernel(const DeltaChunkArgs c) {
    __shared__ float s_ss[2][kDC];
    const DeltaArgs& a = c.a;
    DeltaSeq sd; int chunk;
    if (!delta_find_block(a, blockIdx.x, sd, chunk)) return;
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const int before = chunk * kDC, n = min(kDC, sd.n_rows - before);
    const size_t row0 = (size_t)sd.row_start + before;
    const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj) + row0 * a.ld;
    constexpr int kNT = DV / 16;
    const int m = warp & 3, half = warp >> 2, col0 = half * (DV / 2);
    const int rlo = m * 16 + g, rhi = rlo + 8;
    const float* o = c.o + row0 * a.H * DV + (size_t)h * DV + col0 + 2 * tq;
    float2 v[kNT][2];
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < kNT; ++j) {
        v[j][0] = rlo < n ? *reinterpret_cast<const float2*>(o + (size_t)rlo * a.H * DV + 8 * j) : make_float2(0.f, 0.f);
        v[j][1] = rhi < n ? *reinterpret_cast<const float2*>(o + (size_t)rhi * a.H * DV + 8 * j) : make_float2(0.f, 0.f);
#pragma unroll
        for (int r = 0; r < 2; ++r) ss[r] += v[j][r].x * v[j][r].x + v[j][r].y * v[j][r].y;
    }
    float z[kNT][4];
#pragma unroll
    for (int j = 0; j < kNT; ++j) z[j][0] = z[j][1] = z[j][2] = z[j][3] = 0.f;
    const __nv_bfloat16* lo = proj + (size_t)min(rlo, n - 1) * a.ld + a.g_off + 2 * tq;
    const __nv_bfloat16* hi = proj + (size_t)min(rhi, n - 1) * a.ld + a.g_off + 2 * tq;
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.g2) + ((size_t)h * DV + col0 + g) * a.rg + 2 * tq;
    for (int k = 0; k < a.rg; k += 16) {
        const uint32_t af[4] = {*reinterpret_cast<const uint32_t*>(lo + k), *reinterpret_cast<const uint32_t*>(hi + k),
                                *reinterpret_cast<const uint32_t*>(lo + k + 8), *reinterpret_cast<const uint32_t*>(hi + k + 8)};
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            const __nv_bfloat16* wp = w + (size_t)j * 8 * a.rg + k;
            dr_mma_bf16(z[j], af, *reinterpret_cast<const uint32_t*>(wp), *reinterpret_cast<const uint32_t*>(wp + 8));
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
        ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
        if (tq == 0) s_ss[half][rlo + 8 * r] = ss[r];
    }
    __syncthreads();
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + row0 * a.H * DV + (size_t)h * DV + col0 + 2 * tq;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int row = rlo + 8 * r;
        if (row >= n) continue;
        const float inv = rsqrtf((s_ss[0][row] + s_ss[1][row]) / (float)a.dv_true + a.eps);
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            const float2 nw = *reinterpret_cast<const float2*>(a.norm_w + col0 + 8 * j + 2 * tq);
            *reinterpret_cast<uint32_t*>(out + (size_t)row * a.H * DV + 8 * j) =
                f32x2_to_bf16x2_bits(v[j][r].x * inv * nw.x * dr_sigmoid(z[j][2 * r]), v[j][r].y * inv * nw.y * dr_sigmoid(z[j][2 * r + 1]));
        }
    }
    if (chunk == 0 && a.taps > 1) dr_store_history<__nv_bfloat16>(a, sd, h);      // delta_prepare has read it
}

template <int DK, int DV>
static int launch_delta_chunked(const DeltaChunkArgs& c, int blocks, cudaStream_t stream) {
    constexpr size_t s1 = delta_prep_floats(DK, DV) * 4, s2 = delta_scan_bytes(DK);
    static_assert(s1 <= 226 * 1024 && s2 <= 226 * 1024, "shared memory of the chunked kernels");
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(delta_prepare_kernel<DK, DV, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        cudaFuncSetAttribute(delta_prepare_kernel<DK, DV, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        cudaFuncSetAttribute(delta_scan_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
        set = true;
    }
    const DeltaArgs& a = c.a;
    if (a.taps == 4) delta_prepare_kernel<DK, DV, 4><<<dim3(blocks, a.H), kDPrepThreads, s1, stream>>>(c);
    else delta_prepare_kernel<DK, DV, 0><<<dim3(blocks, a.H), kDPrepThreads, s1, stream>>>(c);
    int e = PS_LAUNCH_CHECK();
    if (e) return e;
    delta_scan_kernel<DK><<<dim3(DV / kDSlice, a.H, a.n_seqs), kDScanThreads, s2, stream>>>(c);
    if ((e = PS_LAUNCH_CHECK())) return e;
    delta_finish_kernel<DV><<<dim3(blocks, a.H), kDFinThreads, 0, stream>>>(c);
    return PS_LAUNCH_CHECK();
}

}  // namespace ps

PS_DEFINE_LIMITS_SETTER(delta_rule)

static int delta_args(ps::DeltaArgs& a, const void* proj, int ld, int H, int G, int dk, int dv, int dk_true, int dv_true, int q_off, int b_off,
                      int a_off, int g_off, int ra, int rg, int taps, float eps, const void* conv, const void* a2, const void* dt_bias,
                      const void* rate, const void* g2, const void* norm_w, void* history, void* state, const void* seqs, int n_seqs, void* out) {
    if (n_seqs <= 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dk % 16 || dv <= 0 || dv % 32 || dv > 1024 || dk_true < 1 || dk_true > dk ||
        dv_true < 1 || dv_true > dv || ra < 8 || ra % 8 || rg < 8 || rg % 8 || taps < 1 || (taps > 1 && history == nullptr) ||
        (ld | q_off | a_off | g_off) % 8 || b_off < 0 ||
        ((uintptr_t)proj | (uintptr_t)conv | (uintptr_t)a2 | (uintptr_t)g2 | (uintptr_t)history | (uintptr_t)state | (uintptr_t)out) % 16)
        return (int)cudaErrorInvalidValue;
    a.proj = proj; a.ld = ld; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.dk_true = dk_true; a.dv_true = dv_true; a.q_off = q_off; a.b_off = b_off;
    a.a_off = a_off; a.g_off = g_off; a.ra = ra; a.rg = rg; a.taps = taps; a.eps = eps; a.conv = conv; a.a2 = a2; a.dt_bias = (const float*)dt_bias;
    a.rate = (const float*)rate; a.g2 = g2; a.norm_w = (const float*)norm_w; a.history = history; a.state = (float*)state;
    a.seqs = (const ps::DeltaSeq*)seqs; a.n_seqs = n_seqs; a.out = out; a.rows_limit = 0;
    return 0;
}

// Every sequence with at most `rows_limit` rows (0 = all) row by row, bf16 or (`f32`) 32-bit.  dk a multiple of 16, dv of 32 (at most
// 1024), ranks, row pitch and offsets (of the q, k, v columns and the low-rank inputs) multiples of 8 elements.
// The kernel may load a slot's state before the stream predecessor has finished (see ps_gdn_rows).
PS_API int ps_delta_rows(const void* proj, int ld, int f32, int H, int G, int dk, int dv, int dk_true, int dv_true, int q_off, int b_off, int a_off,
                         int g_off, int ra, int rg, int taps, float eps, const void* conv, const void* a2, const void* dt_bias, const void* rate,
                         const void* g2, const void* norm_w, void* history, void* state, const void* seqs, int n_seqs, void* out, int rows_limit,
                         cudaStream_t stream) {
    using namespace ps;
    DeltaArgs a;
    const int err = delta_args(a, proj, ld, H, G, dk, dv, dk_true, dv_true, q_off, b_off, a_off, g_off, ra, rg, taps, eps, conv, a2, dt_bias, rate,
                               g2, norm_w, history, state, seqs, n_seqs, out);
    if (err) return err;
    a.rows_limit = rows_limit;
    const size_t smem = ((size_t)3 * dk + 3 * dv + ra + rg + 2048) * 4;
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(H, n_seqs);
#define PS_DELTA_ROWS(T, K, V)                                                                                                         \
    do {                                                                                                                               \
        static bool set = false;                                                                                                       \
        if (!set) { cudaFuncSetAttribute(delta_rows_kernel<T, K, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); set = true; } \
        return launch_pdl(delta_rows_kernel<T, K, V>, grid, dim3(256), smem, stream, a);                                               \
    } while (0)
    if (f32) PS_DELTA_ROWS(float, 0, 0);
    if (dk == 128 && dv == 128) PS_DELTA_ROWS(__nv_bfloat16, 128, 128);
    if (dk == 128 && dv == 64) PS_DELTA_ROWS(__nv_bfloat16, 128, 64);
    if (dk == 64 && dv == 128) PS_DELTA_ROWS(__nv_bfloat16, 64, 128);
    if (dk == 64 && dv == 64) PS_DELTA_ROWS(__nv_bfloat16, 64, 64);
    PS_DELTA_ROWS(__nv_bfloat16, 0, 0);
#undef PS_DELTA_ROWS
}

// Rows of the chunked form's blocks, and whether it takes a head geometry.
PS_API int ps_delta_block_rows() { return ps::kDC; }
PS_API int ps_delta_chunked_ok(int dk, int dv, int ra, int rg) {
    return (dk == 64 || dk == 128) && (dv == 64 || dv == 128) && ra % 16 == 0 && rg % 16 == 0 ? 1 : 0;
}
PS_API long long ps_delta_mats(int dk) { return (long long)ps::delta_mats(dk); }

// The sequences with more than `rows_limit` rows, `blocks` = the sum of their ceil(rows / 64); bf16.  `mats`: ps_delta_mats(dk) bf16 per
// block and head, `u`: 64 * dv, `dec`: dk floats per block and head, `o`: [rows, H * dv] floats; all 16-byte aligned.
PS_API int ps_delta_chunked(const void* proj, int ld, int H, int G, int dk, int dv, int dk_true, int dv_true, int q_off, int b_off, int a_off,
                            int g_off, int ra, int rg, int taps, float eps, const void* conv, const void* a2, const void* dt_bias, const void* rate,
                            const void* g2, const void* norm_w, void* history, void* state, const void* seqs, int n_seqs, void* out, int rows_limit,
                            int blocks, void* mats, void* u, void* dec, void* o, cudaStream_t stream) {
    using namespace ps;
    DeltaChunkArgs c;
    const int err = delta_args(c.a, proj, ld, H, G, dk, dv, dk_true, dv_true, q_off, b_off, a_off, g_off, ra, rg, taps, eps, conv, a2, dt_bias, rate,
                               g2, norm_w, history, state, seqs, n_seqs, out);
    if (err) return err;
    if (blocks <= 0 || rows_limit < 1 || !ps_delta_chunked_ok(dk, dv, ra, rg) || mats == nullptr || u == nullptr || dec == nullptr || o == nullptr ||
        ((uintptr_t)mats | (uintptr_t)u | (uintptr_t)o) % 16)
        return (int)cudaErrorInvalidValue;
    c.a.rows_limit = rows_limit;
    c.mats = (__nv_bfloat16*)mats; c.u = (float*)u; c.dec = (float*)dec; c.o = (float*)o;
    if (dk == 128) return dv == 128 ? launch_delta_chunked<128, 128>(c, blocks, stream) : launch_delta_chunked<128, 64>(c, blocks, stream);
    return dv == 128 ? launch_delta_chunked<64, 128>(c, blocks, stream) : launch_delta_chunked<64, 64>(c, blocks, stream);
}
