// 32-bit projection of the float32 engines: out[M,N] = epilogue(A[M,K] . W[N,K]^T), fp32 multiply-adds on the CUDA cores
// (no TF32).  Several products of one shape (one per head) run as one batched launch.  64 x 64 tiles, 4 x 4 outputs per thread; the gated epilogues combine interleaved (gate, up) columns as the
// bf16 kernels do.  A precision mode, not a fast path.
#include "ps_common.cuh"

namespace ps {

constexpr int kFT = 64, kFK = 16;

__device__ __forceinline__ float gelu_f32(float z) { return z / (1.f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z))); }

struct GemmF32Args {
    const float* a; int lda; const float* w; int ldw;
    int M, N, K, epilogue;             // 0 store, 2 SwiGLU, 3 ReGLU, 4 tanh-gelu, 5 GeGLU
    float* out; int ldo;
    long long stride_a, stride_w, stride_o;                   // elements from one product of the batch to the next
    const float* gate; int ldg; long long stride_g;           // optional: the stored value is multiplied by sigmoid(gate)
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(GemmF32Args g) {
    __shared__ float sa[kFK][kFT + 4], sw[kFK][kFT + 4];
    const int m0 = blockIdx.y * kFT, n0 = blockIdx.x * kFT, t = threadIdx.x, tx = t & 15, ty = t >> 4;
    g.a += blockIdx.z * g.stride_a; g.w += blockIdx.z * g.stride_w; g.out += blockIdx.z * g.stride_o;
    if (g.gate != nullptr) g.gate += blockIdx.z * g.stride_g;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < g.K; k0 += kFK) {
        for (int i = t; i < kFT * kFK; i += 256) {
            const int r = i / kFK, k = i % kFK;
            const bool kin = k0 + k < g.K;
            sa[k][r] = kin && m0 + r < g.M ? g.a[(size_t)(m0 + r) * g.lda + k0 + k] : 0.f;
            sw[k][r] = kin && n0 + r < g.N ? g.w[(size_t)(n0 + r) * g.ldw + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kFK; ++k) {
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
        const int m = m0 + ty * 4 + i;
        if (m >= g.M) continue;
        if (g.epilogue == 2 || g.epilogue == 3 || g.epilogue == 5) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tx * 4 + j;
                if (n + 1 < g.N) {
                    const float gate = acc[i][j];
                    const float act = g.epilogue == 3 ? fmaxf(gate, 0.f) : g.epilogue == 5 ? gelu_f32(gate) : gate / (1.f + expf(-gate));
                    g.out[(size_t)m * g.ldo + (n >> 1)] = act * acc[i][j + 1];
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int n = n0 + tx * 4 + j;
                if (n >= g.N) continue;
                float v = acc[i][j];
                if (g.epilogue == 4) v = gelu_f32(v);
                if (g.gate != nullptr) v *= 1.f / (1.f + expf(-g.gate[(size_t)m * g.ldg + n]));
                g.out[(size_t)m * g.ldo + n] = v;
            }
        }
    }
}

}  // namespace ps

PS_API int ps_gemm_f32(const void* a, int lda, const void* w, int ldw, int M, int N, int K, int epilogue, void* out, int ldo,
                       cudaStream_t stream) {
    using namespace ps;
    if (M <= 0 || N <= 0 || K <= 0 || epilogue < 0 || epilogue == 1 || epilogue > 5 || ((epilogue == 2 || epilogue == 3 || epilogue == 5) && (N & 1)))
        return (int)cudaErrorInvalidValue;
    GemmF32Args g{(const float*)a, lda, (const float*)w, ldw, M, N, K, epilogue, (float*)out, ldo, 0, 0, 0, nullptr, 0, 0};
    gemm_f32_kernel<<<dim3((N + kFT - 1) / kFT, (M + kFT - 1) / kFT), 256, 0, stream>>>(g);
    return PS_LAUNCH_CHECK();
}

// `batch` products out_b[M,N] = A_b[M,K] . W_b[N,K]^T (times sigmoid(gate_b[M,N])), operand b at b * stride elements.
PS_API int ps_gemm_f32_batched(const void* a, int lda, long long stride_a, const void* w, int ldw, long long stride_w, int batch, int M,
                               int N, int K, const void* gate, int ldg, long long stride_g, void* out, int ldo, long long stride_o,
                               cudaStream_t stream) {
    using namespace ps;
    if (batch <= 0 || batch > 65535 || M <= 0 || N <= 0 || K <= 0) return (int)cudaErrorInvalidValue;
    GemmF32Args g{(const float*)a, lda, (const float*)w, ldw, M, N, K, 0, (float*)out, ldo, stride_a, stride_w, stride_o,
                  (const float*)gate, ldg, stride_g};
    gemm_f32_kernel<<<dim3((N + kFT - 1) / kFT, (M + kFT - 1) / kFT, batch), 256, 0, stream>>>(g);
    return PS_LAUNCH_CHECK();
}
