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
__global__ void __launch_bounds__(256) delta_rows_kernel(const DeltaArgs a) {
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
