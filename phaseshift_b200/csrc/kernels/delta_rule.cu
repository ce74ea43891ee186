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
//   delta_scan     per (sequence, head, 16 value columns): Delta = U - W S0,  o = Qd S0 + M Delta,  S = diag(dec) S0 + Kd^T Delta
//   delta_finish   per (block, head): head norm, output gate, and the convolution's history
// No exponential of a positive number is formed, whatever the decays: the triangles are cut into 16-row sub-blocks; off the diagonal
// exp(B_t - B_s) factors through the end of the key's sub-block and of the sub-block before the query's, on the diagonal it is
// evaluated pair by pair.  (The triangular form is that of "Parallelizing Linear Transformers with the Delta Rule over Sequence Length"
// by Songlin Yang, Bailin Wang, Yu Zhang, Yikang Shen and Yoon Kim; sub-blocks as in gla.cu.)
// The products run on bf16 mma.sync with both operands split into two terms (16 bits of mantissa); sums and the state are fp32.
#include "ps_tcgen05.cuh"

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
constexpr int kDPrepThreads = 512, kDFinThreads = 256;
constexpr int kDTP = kDC + 4;
template <int N> struct DeltaInt { static constexpr int value = N; };

struct DeltaChunkArgs {
    DeltaArgs a;
    unsigned char* mats;                // per (block, head), as the scan's shared memory holds it: -W and Qd, then Kd, M and the decay
    float* u;                           // per (block, head): U transposed, [dv, 64]
    float* o;                           // [rows, H * dv]
    uint32_t* status; long long budget;
};
// -W, Qd, Kd [64, dk] and M [64, 64] as a high and a low part of bf16, rows padded by eight elements so that eight rows of a fragment
// load fall into different banks; dec [dk] fp32.
constexpr int kDMPitch = kDC + 8;
__host__ __device__ constexpr size_t delta_mat_bytes(int dk) { return (size_t)2 * 2 * kDC * (dk + 8); }
__host__ __device__ constexpr size_t delta_early_bytes(int dk) { return 2 * delta_mat_bytes(dk); }
__host__ __device__ constexpr size_t delta_late_bytes(int dk) { return delta_mat_bytes(dk) + (size_t)2 * 2 * kDC * kDMPitch + (size_t)4 * dk; }
__host__ __device__ constexpr size_t delta_mats(int dk) { return delta_early_bytes(dk) + delta_late_bytes(dk); }

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

__device__ __forceinline__ float dr_ex2(float x) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x)); return r; }
// Products with operands split into a high and a low part, n column tiles of eight; the low parts' product is left out.  Every round
// runs over all accumulators, so that neighbouring instructions do not wait for each other.
template <int N>
__device__ __forceinline__ void dr_mma3(float (&acc)[N][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[N / 2][4],
                                        const uint32_t (&bl)[N / 2][4]) {
#pragma unroll
    for (int j = 0; j < N; ++j) dr_mma_bf16(acc[j], al, bh[j / 2][j % 2 * 2], bh[j / 2][j % 2 * 2 + 1]);
#pragma unroll
    for (int j = 0; j < N; ++j) dr_mma_bf16(acc[j], ah, bl[j / 2][j % 2 * 2], bl[j / 2][j % 2 * 2 + 1]);
#pragma unroll
    for (int j = 0; j < N; ++j) dr_mma_bf16(acc[j], ah, bh[j / 2][j % 2 * 2], bh[j / 2][j % 2 * 2 + 1]);
}

// log(1 + exp(x)) from the series of the inverse hyperbolic tangent: log(1 + e) = 2 artanh(e / (2 + e)), e <= 1
__device__ __forceinline__ float dr_softplus_fast(float x) {
    const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
    float p = 1.f / 15.f;
    p = fmaf(p, q, 1.f / 13.f); p = fmaf(p, q, 1.f / 11.f); p = fmaf(p, q, 1.f / 9.f); p = fmaf(p, q, 1.f / 7.f);
    p = fmaf(p, q, 1.f / 5.f); p = fmaf(p, q, 1.f / 3.f); p = fmaf(p, q, 1.f);
    return fmaf(2.f * s, p, fmaxf(x, 0.f));
}

// Convolution + silu of eight channels over the RUN rows from r0 on of a block; rows from n on become zero.  `row(r)`: the projected
// channels of row r (negative: before the block; zero before the sequence), `weight(j)`: those of tap j.
template <int TAPS, int RUN, typename Row, typename Weight>
__device__ __forceinline__ void delta_conv(int taps, int r0, int n, Row row, Weight weight, float (&y)[RUN][8]) {
    const int T = TAPS > 0 ? TAPS : taps;
#pragma unroll
    for (int i = 0; i < RUN; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = 0.f;
    if constexpr (TAPS > 0) {
        uint4 x[RUN - 1 + TAPS];
        float wv[TAPS][8];
#pragma unroll
        for (int i = 0; i < RUN - 1 + TAPS; ++i) x[i] = row(r0 + i - (TAPS - 1));
#pragma unroll
        for (int j = 0; j < TAPS; ++j) dr_widen(weight(j), wv[j]);
#pragma unroll
        for (int k = 0; k < RUN - 1 + TAPS; ++k) {           // row k of the run meets tap k - i of output i
            float xv[8];
            dr_widen(x[k], xv);
#pragma unroll
            for (int i = 0; i < RUN; ++i) {
                const int j = k - i;
                if (j < 0 || j >= TAPS) continue;
#pragma unroll
                for (int e = 0; e < 8; ++e) y[i][e] = fmaf(wv[j][e], xv[e], y[i][e]);
            }
        }
    } else {
        for (int j = 0; j < T; ++j) {                  // tap j meets the row T - 1 - j before
            float wv[8];
            dr_widen(weight(j), wv);
#pragma unroll
            for (int i = 0; i < RUN; ++i) {
                float xv[8];
                dr_widen(row(r0 + i - (T - 1 - j)), xv);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[i][e] = fmaf(wv[e], xv[e], y[i][e]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < RUN; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = r0 + i < n ? __fdividef(y[i][e], 1.f + __expf(-y[i][e])) : 0.f;
}

// Shared memory of delta_prepare in bytes: [fp32 q, k, decays | later their bf16 pairs], v pairs, A, M, T, small tables.
constexpr int kDRel = 6;                // (query sub-block, key sub-block) below the diagonal
constexpr int kDStageTaps = 7;          // longest convolution whose rows are staged in shared memory
constexpr int kDLow = 128;              // low-rank columns staged at a time
constexpr int kDLowPitch = kDLow + 8;
__host__ __device__ constexpr size_t delta_prep_region(int dk, int dv) {
    const size_t f = (size_t)3 * kDC * (dk + 4) * 4, h = (size_t)2 * 2 * (2 * kDC + kDRel * 16) * (dk + 8);
    const size_t r = (size_t)2 * kDC * (dk + 4) * 4 + (size_t)(kDC + kDStageTaps - 1) * (2 * dk + dv) * 2;
    return f > h ? (f > r ? f : r) : (h > r ? h : r);
}
__host__ __device__ constexpr size_t delta_prep_bytes(int dk, int dv) {
    return delta_prep_region(dk, dv) + (size_t)2 * 2 * kDC * (dv + 8) + 4 * ((size_t)3 * kDC * kDTP + 3 * 16 * 17 + 4 * dk + 10 * dk + kDC);
}

// grid = (blocks, H)
template <int DK, int DV, int TAPS>
__global__ void __launch_bounds__(kDPrepThreads, 1) delta_prepare_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) unsigned char dp_smem[];
    typedef __nv_bfloat16 bf;
    const DeltaArgs& a = c.a;
    constexpr int P = DK + 4, PB = DK + 8, PV = DV + 8, NW = kDPrepThreads / 32, PT = kDC + 8;
    float* sQ = reinterpret_cast<float*>(dp_smem);      // [64][P]
    float* sK = sQ + kDC * P;                           // [64][P]
    float* sB = sK + kDC * P;                           // [64][P]  log2-decays, then their running sums in a sub-block
    bf* hQ = reinterpret_cast<bf*>(dp_smem);            // later [2][64][PB]: q decayed from the start of its sub-block, high and low part
    bf* hR = hQ + 2 * kDC * PB;                         // [2][64][PB]: k likewise, then from the start of the block
    bf* hC = hR + 2 * kDC * PB;                         // [2][96][PB]: k decayed to the start of a later sub-block
    bf* hT = hQ;                                        // [2][64][PT]: T diag(beta), when hQ has been used up
    bf* sRaw = reinterpret_cast<bf*>(sB);               // first of all [64 + taps - 1][CH]: projected rows, from taps - 1 before the block on
    bf* hV = reinterpret_cast<bf*>(dp_smem + delta_prep_region(DK, DV));  // [2][64][PV]
    float* sA = reinterpret_cast<float*>(hV + 2 * kDC * PV);              // [64][68]
    float* sM = sA + kDC * kDTP;                        // [64][68]
    float* sT = sM + kDC * kDTP;                        // [64][68]
    bf* sLow = reinterpret_cast<bf*>(sA);               // at first [64][136] low-rank inputs and [DK][136] rows of a2
    float* sX = sT + kDC * kDTP;                        // [3][16][17]
    bf* sConv = reinterpret_cast<bf*>(sX);              // at first [taps][CH]: the convolutions
    float* sE = sX + 3 * 16 * 17;                       // [4][DK]  log2-decay sums of the sub-blocks
    float* sF = sE + 4 * DK;                            // [4][DK] decay up to a sub-block's start, [6][DK] between two sub-blocks' ends
    float* sBeta = sF + 10 * DK;                        // [64]
    DeltaSeq sd; int chunk;
    if (!delta_find_block(a, blockIdx.x, sd, chunk)) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows) && sd.pos_start >= 0);
    const int h = blockIdx.y, t = threadIdx.x, warp = t >> 5, lane = t & 31, g = lane >> 2, tq = lane & 3;
    const int before = chunk * kDC, n = min(kDC, sd.n_rows - before), pos0 = sd.pos_start + before, back = a.taps - 1;
    const size_t bh = (size_t)blockIdx.x * a.H + h;
    const bf* proj = reinterpret_cast<const bf*>(a.proj) + (size_t)(sd.row_start + before) * a.ld;
    const bf* conv = reinterpret_cast<const bf*>(a.conv);
    constexpr int CH = 2 * DK + DV;
    const int C = 2 * a.G * DK + a.H * DV;

    static_assert((size_t)kDStageTaps * CH * 2 <= (size_t)4 * (3 * 16 * 17 + 4 * DK + 10 * DK) && (kDC + DK) * kDLowPitch * 2 <= 4 * 3 * kDC * kDTP,
                  "staged operands");
    const bf* a2 = reinterpret_cast<const bf*>(a.a2) + (size_t)h * DK * a.ra;
    auto stage_low = [&](int k0) {                      // columns k0 .. of the low-rank inputs (rows behind the last are not used) and of a2
        const int d = lane * 8;
        if (d >= min(kDLow, a.ra - k0)) return;
        for (int r = warp; r < kDC; r += NW) dr_cp16(sLow + r * kDLowPitch + d, proj + (size_t)min(r, n - 1) * a.ld + a.a_off + k0 + d);
        for (int r = warp; r < DK; r += NW) dr_cp16(sLow + (kDC + r) * kDLowPitch + d, a2 + (size_t)r * a.ra + k0 + d);
    };
    // ---- convolutions, out of staged rows
    const bf* hist = reinterpret_cast<const bf*>(a.history) + ((size_t)sd.slot * back * a.H + h) * CH;
    // columns of the head's three runs of channels, less the channel
    const int hk = h / (a.H / a.G), col_q = hk * DK, col_k = (a.G + hk - 1) * DK, col_v = 2 * a.G * DK + h * DV - 2 * DK;
    auto column = [&](int ch) { return ch + (ch < DK ? col_q : ch < 2 * DK ? col_k : col_v); };
    auto row_source = [&](int r, bool& mine) -> const bf* {              // row r: null: zero, `mine`: the projection's columns
        mine = r + before >= 0;
        if (r >= n || pos0 + r < 0) return nullptr;
        return mine ? proj + (ptrdiff_t)r * a.ld + a.q_off : hist + (size_t)((pos0 + r) % back) * a.H * CH;
    };
    const bool staged = a.taps <= kDStageTaps;
    if (staged) {
        for (int r = warp; r < kDC + back; r += NW) {
            bool mine;
            const bf* src = row_source(r - back, mine);
            for (int ch = lane * 8; ch < CH; ch += 256) {
                if (src != nullptr) dr_cp16(sRaw + r * CH + ch, src + (mine ? column(ch) : ch));
                else *reinterpret_cast<uint4*>(sRaw + r * CH + ch) = make_uint4(0, 0, 0, 0);
            }
        }
        for (int j = warp; j < a.taps; j += NW)
            for (int ch = lane * 8; ch < CH; ch += 256) dr_cp16(sConv + j * CH + ch, conv + (size_t)j * C + column(ch));
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    stage_low(0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (t < kDC) sBeta[t] = t < n ? dr_sigmoid(bf16_to_f32(proj[(size_t)t * a.ld + a.b_off + h])) : 0.f;
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    auto convolve = [&](auto run, int r0, int ch, float (&y)[decltype(run)::value][8]) {
        if (TAPS > 0 || staged)
            delta_conv<TAPS>(a.taps, r0, n, [&](int r) { return *reinterpret_cast<const uint4*>(sRaw + (r + back) * CH + ch); },
                             [&](int j) { return *reinterpret_cast<const uint4*>(sConv + j * CH + ch); }, y);
        else
            delta_conv<0>(a.taps, r0, n, [&](int r) {
                bool mine;
                const bf* p = row_source(r, mine);
                return p != nullptr ? *reinterpret_cast<const uint4*>(p + (mine ? column(ch) : ch)) : make_uint4(0, 0, 0, 0);
            }, [&](int j) { return *reinterpret_cast<const uint4*>(conv + (size_t)j * C + column(ch)); }, y);
    };
    for (int i = t; i < kDC / 4 * (2 * DK / 8); i += kDPrepThreads) {        // queries and keys
        const int ch = i % (2 * DK / 8) * 8, r0 = i / (2 * DK / 8) * 4;
        float y[4][8];
        convolve(DeltaInt<4>{}, r0, ch, y);
        float* dst = (ch < DK ? sQ + ch : sK + ch - DK) + r0 * P;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            *reinterpret_cast<float4*>(dst + r * P) = make_float4(y[r][0], y[r][1], y[r][2], y[r][3]);
            *reinterpret_cast<float4*>(dst + r * P + 4) = make_float4(y[r][4], y[r][5], y[r][6], y[r][7]);
        }
    }
    for (int i = t; i < kDC / 2 * (DV / 8); i += kDPrepThreads) {            // values
        const int ch = i % (DV / 8) * 8, r0 = i / (DV / 8) * 2;
        float y[2][8];
        convolve(DeltaInt<2>{}, r0, 2 * DK + ch, y);
        bf* dst = hV + r0 * PV + ch;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            uint4 hi, lo;
            dr_halves(y[r][0], y[r][1], hi.x, lo.x); dr_halves(y[r][2], y[r][3], hi.y, lo.y);
            dr_halves(y[r][4], y[r][5], hi.z, lo.z); dr_halves(y[r][6], y[r][7], hi.w, lo.w);
            *reinterpret_cast<uint4*>(dst + r * PV) = hi;
            *reinterpret_cast<uint4*>(dst + (kDC + r) * PV) = lo;
        }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();                                    // (the staged rows have been read too)
    // ---- log2-decays: rows of low-rank inputs times the head's rows of a2, on the tensor cores; a warp has 16 rows and DK / 4 channels
    {
        constexpr int kNT = DK / 32;
        const int m = warp & 3, n0 = (warp >> 2) * (DK / 4);
        float z[kNT][4];
#pragma unroll
        for (int j = 0; j < kNT; ++j) z[j][0] = z[j][1] = z[j][2] = z[j][3] = 0.f;
        const bf* ap = sLow + (16 * m + (lane & 15)) * kDLowPitch + (lane >> 4) * 8;
        const bf* bp = sLow + (kDC + n0 + (lane & 7) + (lane >> 4) * 8) * kDLowPitch + ((lane >> 3) & 1) * 8;
        for (int k0 = 0; k0 < a.ra; k0 += kDLow) {
            if (k0 > 0) {
                __syncthreads();
                stage_low(k0);
                asm volatile("cp.async.wait_all;" ::: "memory");
                __syncthreads();
            }
            const int cols = min(kDLow, a.ra - k0);
            for (int k = 0; k < cols; k += 16) {
                uint32_t af[4];
                dr_ldsm(af, ap + k);
#pragma unroll
                for (int j = 0; j < kNT; j += 2) {
                    uint32_t wf[4];
                    dr_ldsm(wf, bp + j * 8 * kDLowPitch + k);
                    dr_mma_bf16(z[j], af, wf[0], wf[1]);
                    dr_mma_bf16(z[j + 1], af, wf[2], wf[3]);
                }
            }
        }
        const float rate = -1.4426950408889634f * a.rate[h];
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
            const int d = n0 + j * 8 + 2 * tq;
            const float b0 = a.dt_bias[h * DK + d], b1 = a.dt_bias[h * DK + d + 1];
            const int r0 = m * 16 + g, r1 = r0 + 8;
            *reinterpret_cast<float2*>(sB + r0 * P + d) = r0 < n ? make_float2(rate * dr_softplus_fast(z[j][0] + b0), rate * dr_softplus_fast(z[j][1] + b1)) : make_float2(0.f, 0.f);
            *reinterpret_cast<float2*>(sB + r1 * P + d) = r1 < n ? make_float2(rate * dr_softplus_fast(z[j][2] + b0), rate * dr_softplus_fast(z[j][3] + b1)) : make_float2(0.f, 0.f);
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
    // ---- diagonal sub-blocks (sums local to the sub-block suffice: only differences enter).  Rows 8 - 15 against keys 0 - 7: both
    // sides factor through row 7; a warp has a quarter of the channels of one sub-block, rows 0 - 7 of its tile are queries, 8 - 15 keys
    {
        const int blk = warp >> 2, part = warp & 3;
        const float* ref = sB + (blk * 16 + 7) * P;
        const float* q = sQ + (blk * 16 + 8 + g) * P;
        const float* k = sK + (blk * 16 + 8 + g) * P;
        const float* bi = sB + (blk * 16 + 8 + g) * P;
        const float* kj = sK + (blk * 16 + g) * P;
        const float* bj = sB + (blk * 16 + g) * P;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k0 = part * (DK / 4); k0 < (part + 1) * (DK / 4); k0 += 16) {
            uint32_t ah[4], al[4], xh[2], xl[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int d = k0 + 8 * e + 2 * tq;
                const float2 r = *reinterpret_cast<const float2*>(ref + d), b = *reinterpret_cast<const float2*>(bi + d), u = *reinterpret_cast<const float2*>(bj + d);
                const float2 qv = *reinterpret_cast<const float2*>(q + d), kv = *reinterpret_cast<const float2*>(k + d), jv = *reinterpret_cast<const float2*>(kj + d);
                const float f0 = dr_ex2(b.x - r.x), f1 = dr_ex2(b.y - r.y);
                dr_halves(qv.x * f0, qv.y * f1, ah[2 * e], al[2 * e]);
                dr_halves(kv.x * f0, kv.y * f1, ah[2 * e + 1], al[2 * e + 1]);
                dr_halves(jv.x * dr_ex2(r.x - u.x), jv.y * dr_ex2(r.y - u.y), xh[e], xl[e]);
            }
            dr_mma_bf16(acc, al, xh[0], xh[1]);
            dr_mma_bf16(acc, ah, xl[0], xl[1]);
            dr_mma_bf16(acc, ah, xh[0], xh[1]);
        }
        float* dst = sT + (warp * 16 + g) * 8 + 2 * tq;      // partial sums of the four quarters
        *reinterpret_cast<float2*>(dst) = make_float2(acc[0], acc[1]);
        *reinterpret_cast<float2*>(dst + 64) = make_float2(acc[2], acc[3]);
    }
    // the eight 8 x 8 triangles on the diagonal pair by pair, two keys at a time
#pragma unroll 1
    for (int u = 0; u < 4; ++u) {
        constexpr int kU = DK / 32;
        const int il = (u & 1) ? 7 - (warp & 7) : warp & 7, first = ((warp >> 3) + 2 * u) * 8, i = first + il, d = lane * kU;
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
                const int j = first + min(jl + e, il);
                float kj[kU], bj[kU], s0 = 0.f, s1 = 0.f;
                load(sK + j * P + d, kj); load(sB + j * P + d, bj);
#pragma unroll
                for (int x = 0; x < kU; ++x) {
                    const float f = kj[x] * dr_ex2(bi[x] - bj[x]);
                    s0 = fmaf(qi[x], f, s0); s1 = fmaf(ki[x], f, s1);
                }
                v[2 * e] = s0; v[2 * e + 1] = s1;
            }
            // four sums over the warp at once: lanes 0, 8, 16, 24 end with one each
            const bool up = lane & 16, odd = lane & 8;
            const float x = (up ? v[2] : v[0]) + __shfl_xor_sync(0xffffffffu, up ? v[0] : v[2], 16);
            const float y = (up ? v[3] : v[1]) + __shfl_xor_sync(0xffffffffu, up ? v[1] : v[3], 16);
            float s = (odd ? y : x) + __shfl_xor_sync(0xffffffffu, odd ? x : y, 8);
            s += __shfl_xor_sync(0xffffffffu, s, 4);
            s += __shfl_xor_sync(0xffffffffu, s, 2);
            s += __shfl_xor_sync(0xffffffffu, s, 1);
            const int jj = jl + (up ? 1 : 0), j = first + jj;
            if ((lane & 7) == 0 && jj <= il) {
                if (!odd) sM[i * kDTP + j] = s;
                else sA[i * kDTP + j] = sBeta[i] * s;
            }
        }
    }
    // ---- decay factors: up to the sub-blocks' starts, and between the ends of two sub-blocks
    if (t < DK) {
        const float e0 = sE[t], e1 = sE[DK + t], e2 = sE[2 * DK + t], e3 = sE[3 * DK + t];
        sF[t] = 1.f; sF[DK + t] = dr_ex2(e0); sF[2 * DK + t] = dr_ex2(e0 + e1); sF[3 * DK + t] = dr_ex2(e0 + e1 + e2);
        float* rel = sF + 4 * DK + t;                   // ends of sub-blocks (1, 0), (2, 0), (2, 1), (3, 0), (3, 1), (3, 2)
        rel[0] = dr_ex2(e1); rel[DK] = dr_ex2(e1 + e2); rel[2 * DK] = dr_ex2(e2);
        rel[3 * DK] = dr_ex2(e1 + e2 + e3); rel[4 * DK] = dr_ex2(e2 + e3); rel[5 * DK] = dr_ex2(e3);
        reinterpret_cast<float*>(c.mats + (bh + 1) * delta_mats(DK))[t - DK] = exp2f(e0 + e1 + e2 + e3);
    }
    // ---- a thread's elements of q, k and the sums move to registers; their place takes the bf16 pairs
    constexpr int kQ4 = kDC * DK / 4 / kDPrepThreads;
    float4 rq[kQ4], rk[kQ4], rb[kQ4];
#pragma unroll
    for (int u = 0; u < kQ4; ++u) {
        const int i = t + u * kDPrepThreads, at = i / (DK / 4) * P + i % (DK / 4) * 4;
        rq[u] = *reinterpret_cast<const float4*>(sQ + at); rk[u] = *reinterpret_cast<const float4*>(sK + at); rb[u] = *reinterpret_cast<const float4*>(sB + at);
    }
    __syncthreads();
    if (t < 256) {                                      // the quarters of the 8 x 8 squares
        const int blk = t >> 6, il = (t >> 3) & 7, j = t & 7, i = blk * 16 + 8 + il, at = i * kDTP + blk * 16 + j;
        float m = 0.f, k = 0.f;
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            m += sT[((blk * 4 + p) * 16 + il) * 8 + j];
            k += sT[((blk * 4 + p) * 16 + 8 + il) * 8 + j];
        }
        sM[at] = m;
        sA[at] = sBeta[i] * k;
    }
    constexpr int kMat = kDC * PB;                      // elements of a matrix: the high part, then the low part
    bf* gW = reinterpret_cast<bf*>(c.mats + bh * delta_mats(DK));
    bf* gQ = gW + 2 * kMat;
    bf* gK = gQ + 2 * kMat;
    bf* gM = gK + 2 * kMat;
    auto pair4 = [](float4 v, uint2& hi, uint2& lo) { dr_halves(v.x, v.y, hi.x, lo.x); dr_halves(v.z, v.w, hi.y, lo.y); };
    auto mul4 = [](float4 x, float4 y) { return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w); };
    auto put = [&](bf* dst, int part, float4 v) {
        uint2 hi, lo;
        pair4(v, hi, lo);
        *reinterpret_cast<uint2*>(dst) = hi;
        *reinterpret_cast<uint2*>(dst + part) = lo;
    };
#pragma unroll
    for (int u = 0; u < kQ4; ++u) {
        const int i = t + u * kDPrepThreads, r = i / (DK / 4), d = i % (DK / 4) * 4, blk = r >> 4;
        const float4 b = rb[u], e = *reinterpret_cast<const float4*>(sE + blk * DK + d);
        const float4 f = make_float4(dr_ex2(b.x), dr_ex2(b.y), dr_ex2(b.z), dr_ex2(b.w));
        const float4 q = mul4(rq[u], f), k = mul4(rk[u], make_float4(dr_ex2(e.x - b.x), dr_ex2(e.y - b.y), dr_ex2(e.z - b.z), dr_ex2(e.w - b.w)));
        put(hQ + r * PB + d, kDC * PB, q);
        put(hR + r * PB + d, kDC * PB, mul4(rk[u], f));
        put(gQ + r * PB + d, kMat, mul4(q, *reinterpret_cast<const float4*>(sF + blk * DK + d)));
        const float* rel = sF + 4 * DK + d;
        if (blk < 3) {
            // to the start of sub-block qi = blk + 1, ..., 3 (places qi (qi - 1) / 2 + blk), and to the block's end
            bf* dst = hC + (r & 15) * PB + d;
            constexpr int part = kDRel * 16 * PB;
            put(dst + (blk + 1) * (blk) / 2 * 16 * PB + blk * 16 * PB, part, k);
            for (int qi = blk + 2; qi <= 3; ++qi) {
                const int x = (qi - 1) * (qi - 2) / 2 + blk;                       // (qi - 1, blk) among the pairs of ends
                put(dst + (qi * (qi - 1) / 2 + blk) * 16 * PB, part, mul4(k, *reinterpret_cast<const float4*>(rel + x * DK)));
            }
            put(gK + r * PB + d, kMat, mul4(k, *reinterpret_cast<const float4*>(rel + (3 + blk) * DK)));
        } else
            put(gK + r * PB + d, kMat, k);
    }
    __syncthreads();
    // ---- below the diagonal: a warp has one (query sub-block, key sub-block) for queries or for keys; the solve of T's diagonal
    // sub-blocks (thread: sub-block, column) by the last two warps
    if (warp < 12) {
        const int x = warp >> 1, qi = x < 1 ? 1 : (x < 3 ? 2 : 3), kj = x - qi * (qi - 1) / 2;
        const bool keys = warp & 1;
        float acc[2][4] = {};
        const bf* ap = (keys ? hR : hQ) + (qi * 16 + (lane & 15)) * PB + (lane >> 4) * 8;
        const bf* bp = hC + (x * 16 + (lane & 7) + (lane >> 4) * 8) * PB + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int k = 0; k < DK; k += 16) {
            uint32_t ah[4], al[4], bh[1][4], bl[1][4];
            dr_ldsm(ah, ap + k); dr_ldsm(al, ap + kDC * PB + k);
            dr_ldsm(bh[0], bp + k); dr_ldsm(bl[0], bp + kDRel * 16 * PB + k);
            dr_mma3<2>(acc, ah, al, bh, bl);
        }
        const int r0 = qi * 16 + g;
        const float f0 = keys ? sBeta[r0] : 1.f, f1 = keys ? sBeta[r0 + 8] : 1.f;
        float* dst = (keys ? sA : sM) + r0 * kDTP + kj * 16 + 2 * tq;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            *reinterpret_cast<float2*>(dst + 8 * j) = make_float2(f0 * acc[j][0], f0 * acc[j][1]);
            *reinterpret_cast<float2*>(dst + 8 * kDTP + 8 * j) = make_float2(f1 * acc[j][2], f1 * acc[j][3]);
        }
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
    // ---- M goes out; k decayed from the block's start replaces k decayed from the sub-block's
    for (int i = t; i < kDC * kDC / 4; i += kDPrepThreads) {
        const int r = i / (kDC / 4), s = i % (kDC / 4) * 4;
        const float* p = sM + r * kDTP + s;
        put(gM + r * kDMPitch + s, kDC * kDMPitch, make_float4(s <= r ? p[0] : 0.f, s + 1 <= r ? p[1] : 0.f, s + 2 <= r ? p[2] : 0.f, s + 3 <= r ? p[3] : 0.f));
    }
#pragma unroll
    for (int u = 0; u < kQ4; ++u) {
        const int i = t + u * kDPrepThreads, r = i / (DK / 4), d = i % (DK / 4) * 4, blk = r >> 4;
        const float4 b = rb[u], p = *reinterpret_cast<const float4*>(sF + blk * DK + d);
        put(hR + r * PB + d, kDC * PB, mul4(mul4(rk[u], make_float4(dr_ex2(b.x), dr_ex2(b.y), dr_ex2(b.z), dr_ex2(b.w))), p));
    }
    // ---- T, block rows 1 .. 3: T_ij = -T_ii (sum_{k = j .. i-1} A_ik T_kj) for all j < i at once
    for (int bi = 1; bi < 4; ++bi) {
        for (int e = t; e < bi * 256; e += kDPrepThreads) {
            const int bj = e >> 8, r = (e >> 4) & 15, cc = e & 15;
            const float* Ar = sA + (16 * bi + r) * kDTP;
            float s0 = 0.f, s1 = 0.f;
            for (int k = 16 * bj; k < 16 * bi; k += 4) {
                const float4 x = *reinterpret_cast<const float4*>(Ar + k);
                const float* tp = sT + k * kDTP + 16 * bj + cc;
                s0 = fmaf(x.x, tp[0], s0); s1 = fmaf(x.y, tp[kDTP], s1); s0 = fmaf(x.z, tp[2 * kDTP], s0); s1 = fmaf(x.w, tp[3 * kDTP], s1);
            }
            sX[(bj * 16 + r) * 17 + cc] = s0 + s1;
        }
        __syncthreads();
        for (int e = t; e < bi * 256; e += kDPrepThreads) {
            const int bj = e >> 8, r = (e >> 4) & 15, cc = e & 15;
            const float* Tr = sT + (16 * bi + r) * kDTP + 16 * bi;
            float s = 0.f;
#pragma unroll
            for (int k = 0; k < 16; k += 4) {                        // T_ii is zero above its diagonal
                const float4 x = *reinterpret_cast<const float4*>(Tr + k);
                const float* xp = sX + (bj * 16 + k) * 17 + cc;
                s = fmaf(x.x, xp[0], s); s = fmaf(x.y, xp[17], s); s = fmaf(x.z, xp[34], s); s = fmaf(x.w, xp[51], s);
            }
            sT[(16 * bi + r) * kDTP + 16 * bj + cc] = -s;
        }
        __syncthreads();
    }
    for (int i = t; i < kDC * kDC / 4; i += kDPrepThreads) {
        const int r = i / (kDC / 4), s = i % (kDC / 4) * 4;
        if (s >> 4 > r >> 4) continue;                  // blocks above the diagonal are not read
        put(hT + r * PT + s, kDC * PT, mul4(*reinterpret_cast<const float4*>(sT + r * kDTP + s), *reinterpret_cast<const float4*>(sBeta + s)));
    }
    __syncthreads();
    // ---- W = T diag(beta) K (warps 0-7) and U = T diag(beta) V (warps 8-15): a warp has 16 rows and half the columns; T is lower
    // triangular, so steps beyond the row tile are skipped
    auto product = [&](auto cols, const bf* src, auto store) {
        constexpr int D = decltype(cols)::value, pitch = D + 8, kN = D / 16;
        const int m = warp & 3, col0 = ((warp >> 2) & 1) * (D / 2);
        float acc[kN][4];
#pragma unroll
        for (int j = 0; j < kN; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        const bf* ap = hT + (16 * m + (lane & 15)) * PT + (lane >> 4) * 8;
        const bf* bp = src + (lane & 15) * pitch + col0 + (lane >> 4) * 8;
        for (int k = 0; k < 16 * (m + 1); k += 16) {
            uint32_t ah[4], al[4], bh[kN / 2][4], bl[kN / 2][4];
            dr_ldsm(ah, ap + k); dr_ldsm(al, ap + kDC * PT + k);
#pragma unroll
            for (int j = 0; j < kN / 2; ++j) { dr_ldsm_t(bh[j], bp + k * pitch + 16 * j); dr_ldsm_t(bl[j], bp + (kDC + k) * pitch + 16 * j); }
            dr_mma3<kN>(acc, ah, al, bh, bl);
        }
#pragma unroll
        for (int j = 0; j < kN; ++j) {
            store(16 * m + g, col0 + 8 * j + 2 * tq, acc[j][0], acc[j][1]);
            store(16 * m + g + 8, col0 + 8 * j + 2 * tq, acc[j][2], acc[j][3]);
        }
    };
    if (warp < NW / 2) {
        product(DeltaInt<DK>{}, hR, [&](int r, int d, float x, float y) {
            uint32_t hi, lo;
            dr_halves(-x, -y, hi, lo);
            *reinterpret_cast<uint32_t*>(gW + r * PB + d) = hi; *reinterpret_cast<uint32_t*>(gW + kMat + r * PB + d) = lo;
        });
    } else {
        float* u = c.u + bh * kDC * DV;
        product(DeltaInt<DV>{}, hV, [&](int r, int d, float x, float y) { u[d * kDC + r] = x; u[(d + 1) * kDC + r] = y; });
    }
}

// grid = (DV / (16 NW), H, n_seqs).  Everything runs transposed: a warp has 16 value columns of a sequence's head and keeps their state,
// Delta and outputs in accumulator registers, which are also the left operands of the next products; only W, Qd, Kd and M come from
// shared memory.  One more warp copies them there: -W and Qd of two blocks, Kd, M and the decays of one.
template <int DK, int NW>
__global__ void __launch_bounds__(32 * NW + 32, 1) delta_scan_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) unsigned char ds_smem[];
    typedef __nv_bfloat16 bf;
    const DeltaArgs& a = c.a;
    constexpr int PB = DK + 8, kMat = kDC * PB, ND = DK / 8;
    constexpr uint32_t kEarly = (uint32_t)delta_early_bytes(DK), kLate = (uint32_t)delta_late_bytes(DK);
    __shared__ __align__(8) uint64_t full_e[2], empty_e[2], full_l, empty_l;
    __shared__ int s_abort;
    const DeltaSeq sd = a.seqs[blockIdx.z];
    if (sd.slot < 0 || sd.n_rows <= a.rows_limit) return;
    PS_CHECK(PS_SLOT_OK(sd.slot) && PS_ROWS_OK(sd.row_start, sd.n_rows));
    int first = 0;
    for (int s = 0; s < (int)blockIdx.z; ++s) {
        const DeltaSeq d = a.seqs[s];
        if (d.n_rows > a.rows_limit && d.slot >= 0) first += (d.n_rows + kDC - 1) / kDC;
    }
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3, dv = a.dv;
    const int n_blocks = (sd.n_rows + kDC - 1) / kDC;
    if (threadIdx.x == 0) {
        for (int i = 0; i < 2; ++i) { tc::mbar_init(&full_e[i], 1); tc::mbar_init(&empty_e[i], NW); }
        tc::mbar_init(&full_l, 1);
        tc::mbar_init(&empty_l, NW);
        tc::fence_barrier_init();
        s_abort = 0;
    }
    __syncthreads();
    unsigned char* late = ds_smem + 2 * kEarly;
    if (warp == NW) {
        if (lane == 0) {
            int early = 0, lates = 0;                   // copies handed out
            bool ok = true;
            auto fetch_early = [&](int i) {
                ok = ok && (i < 2 || tc::mbar_wait_abortable(&empty_e[i & 1], (uint32_t)((i >> 1) - 1) & 1u, c.budget, &s_abort));
                if (!ok) return;
                tc::mbar_expect_tx(&full_e[i & 1], kEarly);
                tc::bulk_load(ds_smem + (i & 1) * kEarly, c.mats + ((size_t)(first + i) * a.H + h) * delta_mats(DK), kEarly, &full_e[i & 1]);
                ++early;
            };
            fetch_early(0);
            for (int i = 0; i < n_blocks && ok; ++i) {
                if (i + 1 < n_blocks) fetch_early(i + 1);
                ok = ok && (i < 1 || tc::mbar_wait_abortable(&empty_l, (uint32_t)(i - 1) & 1u, c.budget, &s_abort));
                if (!ok) break;
                tc::mbar_expect_tx(&full_l, kLate);
                tc::bulk_load(late, c.mats + ((size_t)(first + i) * a.H + h) * delta_mats(DK) + kEarly, kLate, &full_l);
                ++lates;
            }
            if (!ok) {
                // copies still in flight get a bounded chance to land before the shared memory goes back to the next CTA
                const long long b = c.budget < 4000000ll ? c.budget : 4000000ll;
                for (int i = max(0, early - 2); i < early; ++i) tc::mbar_wait(&full_e[i & 1], (uint32_t)(i >> 1) & 1u, b);
                if (lates > 0) tc::mbar_wait(&full_l, (uint32_t)(lates - 1) & 1u, b);
            }
        }
    } else {
        const int v0 = (blockIdx.x * NW + warp) * 16 + g;            // this thread's value columns: v0 and v0 + 8
        float* state = a.state + ((size_t)sd.slot * a.H + h) * DK * dv + v0;
        float S[ND][4], D[8][4], R[8][4];
#pragma unroll
        for (int j = 0; j < ND; ++j) {
            const float* p = state + (size_t)(8 * j + 2 * tq) * dv;
            S[j][0] = p[0]; S[j][1] = p[dv]; S[j][2] = p[8]; S[j][3] = p[dv + 8];
        }
        auto load_u = [&](int i) {
            const float* u = c.u + (((size_t)(first + i) * a.H + h) * dv + v0) * kDC + 2 * tq;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float2 x = *reinterpret_cast<const float2*>(u + 8 * j), y = *reinterpret_cast<const float2*>(u + 8 * kDC + 8 * j);
                D[j][0] = x.x; D[j][1] = x.y; D[j][2] = y.x; D[j][3] = y.y;
            }
        };
        // accumulator tiles 2 k and 2 k + 1 as the left operand of a product's step k
        auto operand = [](const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
            dr_halves(x[0], x[1], hi[0], lo[0]); dr_halves(x[2], x[3], hi[1], lo[1]);
            dr_halves(y[0], y[1], hi[2], lo[2]); dr_halves(y[2], y[3], hi[3], lo[3]);
        };
        load_u(0);
        const int row_n = (lane & 7) + (lane >> 4) * 8, col_n = ((lane >> 3) & 1) * 8;     // right operand from rows of columns
        bool ok = true;
        for (int i = 0; i < n_blocks; ++i) {
            const int n = min(kDC, sd.n_rows - i * kDC);
            ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&full_e[i & 1], (uint32_t)(i >> 1) & 1u, c.budget, &s_abort));
            if (!ok) break;
            // ---- Delta^T = U^T - S^T W^T, and the state's part of the outputs
#pragma unroll
            for (int j = 0; j < 8; ++j) R[j][0] = R[j][1] = R[j][2] = R[j][3] = 0.f;
            {
                const bf* wp = reinterpret_cast<const bf*>(ds_smem + (i & 1) * kEarly) + row_n * PB + col_n;
                const bf* qp = wp + 2 * kMat;
#pragma unroll
                for (int k = 0; k < DK / 16; ++k) {
                    uint32_t ah[4], al[4], bh[4][4], bl[4][4];
                    operand(S[2 * k], S[2 * k + 1], ah, al);
#pragma unroll
                    for (int j = 0; j < 4; ++j) { dr_ldsm(bh[j], wp + 16 * j * PB + 16 * k); dr_ldsm(bl[j], wp + kMat + 16 * j * PB + 16 * k); }
                    dr_mma3<8>(D, ah, al, bh, bl);
#pragma unroll
                    for (int j = 0; j < 4; ++j) { dr_ldsm(bh[j], qp + 16 * j * PB + 16 * k); dr_ldsm(bl[j], qp + kMat + 16 * j * PB + 16 * k); }
                    dr_mma3<8>(R, ah, al, bh, bl);
                }
            }
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&empty_e[i & 1]);
            uint32_t dh[4][4], dl[4][4];
#pragma unroll
            for (int k = 0; k < 4; ++k) operand(D[2 * k], D[2 * k + 1], dh[k], dl[k]);
            if (i + 1 < n_blocks) load_u(i + 1);
            ok = __all_sync(0xffffffffu, tc::mbar_wait_abortable(&full_l, (uint32_t)i & 1u, c.budget, &s_abort));
            if (!ok) break;
            // ---- o^T += Delta^T M^T (tokens after the row are skipped)
            {
                const bf* mp = reinterpret_cast<const bf*>(late) + 2 * kMat + row_n * kDMPitch + col_n;
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    uint32_t bh[4][4], bl[4][4];
#pragma unroll
                    for (int j = k; j < 4; ++j) {
                        dr_ldsm(bh[j], mp + 16 * j * kDMPitch + 16 * k);
                        dr_ldsm(bl[j], mp + kDC * kDMPitch + 16 * j * kDMPitch + 16 * k);
                    }
#pragma unroll
                    for (int j = 2 * k; j < 8; ++j) dr_mma_bf16(R[j], dl[k], bh[j / 2][j % 2 * 2], bh[j / 2][j % 2 * 2 + 1]);
#pragma unroll
                    for (int j = 2 * k; j < 8; ++j) dr_mma_bf16(R[j], dh[k], bl[j / 2][j % 2 * 2], bl[j / 2][j % 2 * 2 + 1]);
#pragma unroll
                    for (int j = 2 * k; j < 8; ++j) dr_mma_bf16(R[j], dh[k], bh[j / 2][j % 2 * 2], bh[j / 2][j % 2 * 2 + 1]);
                }
            }
            {
                float* o = c.o + (size_t)(sd.row_start + i * kDC) * a.H * dv + (size_t)h * dv + v0;
                const size_t ld = (size_t)a.H * dv;
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int r = 8 * j + 2 * tq;
                    if (r < n) { o[r * ld] = R[j][0]; o[r * ld + 8] = R[j][2]; }
                    if (r + 1 < n) { o[(r + 1) * ld] = R[j][1]; o[(r + 1) * ld + 8] = R[j][3]; }
                }
            }
            // ---- S^T = S^T diag(dec) + Delta^T Kd
            {
                const float* dec = reinterpret_cast<const float*>(late + kLate) - DK;
#pragma unroll
                for (int j = 0; j < ND; ++j) {
                    const float2 d = *reinterpret_cast<const float2*>(dec + 8 * j + 2 * tq);
                    S[j][0] *= d.x; S[j][1] *= d.y; S[j][2] *= d.x; S[j][3] *= d.y;
                }
                const bf* kp = reinterpret_cast<const bf*>(late) + (lane & 15) * PB + (lane >> 4) * 8;
#pragma unroll
                for (int x = 0; x < ND; x += 8) {
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        uint32_t bh[4][4], bl[4][4];
#pragma unroll
                        for (int j = 0; j < 4; ++j) {
                            dr_ldsm_t(bh[j], kp + 16 * k * PB + 8 * x + 16 * j);
                            dr_ldsm_t(bl[j], kp + kMat + 16 * k * PB + 8 * x + 16 * j);
                        }
                        dr_mma3<8>(reinterpret_cast<float (&)[8][4]>(S[x]), dh[k], dl[k], bh, bl);
                    }
                }
            }
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&empty_l);
        }
        if (ok) {
#pragma unroll
            for (int j = 0; j < ND; ++j) {
                float* p = state + (size_t)(8 * j + 2 * tq) * dv;
                p[0] = S[j][0]; p[dv] = S[j][1]; p[8] = S[j][2]; p[dv + 8] = S[j][3];
            }
        }
    }
    __syncthreads();
    if (threadIdx.x == 0 && s_abort != 0) set_status(c.status, PS_DEV_WAIT_TIMEOUT);
}

// grid = (blocks, H): head norm and output gate (low-rank inputs times the head's rows of g2, on the tensor cores)
template <int DV>
__global__ void __launch_bounds__(kDFinThreads, 2) delta_finish_kernel(const DeltaChunkArgs c) {
    extern __shared__ __align__(16) unsigned char df_smem[];
    constexpr int PG = kDLowPitch;
    __nv_bfloat16* s_in = reinterpret_cast<__nv_bfloat16*>(df_smem);      // [64][136]
    __nv_bfloat16* s_w = s_in + kDC * PG;                                 // [DV][136]
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
    const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(a.g2) + (size_t)h * DV * a.rg;
    auto stage = [&](int k0) {                          // (rows behind the last are not used)
        const int per = min(kDLow, a.rg - k0) / 8;
        for (int i = t; i < (kDC + DV) * per; i += kDFinThreads) {
            const int r = i / per, d = i % per * 8;
            if (r < kDC) dr_cp16(s_in + r * PG + d, proj + (size_t)min(r, n - 1) * a.ld + a.g_off + k0 + d);
            else dr_cp16(s_w + (r - kDC) * PG + d, w + (size_t)(r - kDC) * a.rg + k0 + d);
        }
    };
    stage(0);
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
    for (int k0 = 0; k0 < a.rg; k0 += kDLow) {
        const int cols = min(kDLow, a.rg - k0);
        if (k0 > 0) {
            __syncthreads();
            stage(k0);
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        const __nv_bfloat16* ap = s_in + (16 * m + (lane & 15)) * PG + (lane >> 4) * 8;
        const __nv_bfloat16* bp = s_w + (col0 + (lane & 7) + (lane >> 4) * 8) * PG + ((lane >> 3) & 1) * 8;
        for (int k = 0; k < cols; k += 16) {
            uint32_t af[4];
            dr_ldsm(af, ap + k);
#pragma unroll
            for (int j = 0; j < kNT; j += 2) {
                uint32_t wf[4];
                dr_ldsm(wf, bp + j * 8 * PG + k);
                dr_mma_bf16(z[j], af, wf[0], wf[1]);
                dr_mma_bf16(z[j + 1], af, wf[2], wf[3]);
            }
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
    constexpr size_t s1 = delta_prep_bytes(DK, DV), s2 = 2 * delta_early_bytes(DK) + delta_late_bytes(DK), s4 = (size_t)(kDC + DV) * kDLowPitch * 2;
    static_assert(s1 <= 226 * 1024 && s2 <= 226 * 1024, "shared memory of the chunked kernels");
    static bool set = false;
    if (!set) {
        cudaFuncSetAttribute(delta_prepare_kernel<DK, DV, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        cudaFuncSetAttribute(delta_prepare_kernel<DK, DV, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
        cudaFuncSetAttribute(delta_finish_kernel<DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s4);
        cudaFuncSetAttribute(delta_scan_kernel<DK, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
        cudaFuncSetAttribute(delta_scan_kernel<DK, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
        set = true;
    }
    const DeltaArgs& a = c.a;
    if (a.taps == 4) delta_prepare_kernel<DK, DV, 4><<<dim3(blocks, a.H), kDPrepThreads, s1, stream>>>(c);
    else delta_prepare_kernel<DK, DV, 0><<<dim3(blocks, a.H), kDPrepThreads, s1, stream>>>(c);
    int e = PS_LAUNCH_CHECK();
    if (e) return e;
    // one CTA per SM: two warps each while all CTAs are resident at once
    if (a.H * a.n_seqs * (DV / 32) <= 148) delta_scan_kernel<DK, 2><<<dim3(DV / 32, a.H, a.n_seqs), 96, s2, stream>>>(c);
    else delta_scan_kernel<DK, 4><<<dim3(DV / 64, a.H, a.n_seqs), 160, s2, stream>>>(c);
    if ((e = PS_LAUNCH_CHECK())) return e;
    delta_finish_kernel<DV><<<dim3(blocks, a.H), kDFinThreads, s4, stream>>>(c);
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

// The sequences with more than `rows_limit` rows, `blocks` = the sum of their ceil(rows / 64); bf16.  `mats`: ps_delta_mats(dk) bytes per
// block and head, `u`: 64 * dv floats per block and head, `o`: [rows, H * dv] floats; all 16-byte aligned.
PS_API int ps_delta_chunked(const void* proj, int ld, int H, int G, int dk, int dv, int dk_true, int dv_true, int q_off, int b_off, int a_off,
                            int g_off, int ra, int rg, int taps, float eps, const void* conv, const void* a2, const void* dt_bias, const void* rate,
                            const void* g2, const void* norm_w, void* history, void* state, const void* seqs, int n_seqs, void* out, int rows_limit,
                            int blocks, void* mats, void* u, void* o, void* status, cudaStream_t stream) {
    using namespace ps;
    DeltaChunkArgs c;
    const int err = delta_args(c.a, proj, ld, H, G, dk, dv, dk_true, dv_true, q_off, b_off, a_off, g_off, ra, rg, taps, eps, conv, a2, dt_bias, rate,
                               g2, norm_w, history, state, seqs, n_seqs, out);
    if (err) return err;
    if (blocks <= 0 || rows_limit < 1 || !ps_delta_chunked_ok(dk, dv, ra, rg) || mats == nullptr || u == nullptr || o == nullptr ||
        ((uintptr_t)mats | (uintptr_t)u | (uintptr_t)o) % 16)
        return (int)cudaErrorInvalidValue;
    c.a.rows_limit = rows_limit;
    c.mats = (unsigned char*)mats; c.u = (float*)u; c.o = (float*)o; c.status = (uint32_t*)status; c.budget = g_ps_wait_budget_cycles;
    if (dk == 128) return dv == 128 ? launch_delta_chunked<128, 128>(c, blocks, stream) : launch_delta_chunked<128, 64>(c, blocks, stream);
    return dv == 128 ? launch_delta_chunked<64, 128>(c, blocks, stream) : launch_delta_chunked<64, 64>(c, blocks, stream);
}
