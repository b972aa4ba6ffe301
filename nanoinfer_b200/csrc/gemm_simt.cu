// The general matrix product of the engine: C[M,N] = A[M,K] . W[N,K]^T (+ bias), any M, N, K,
// 32-bit accumulation on the CUDA cores. It is the true 32-bit path (no reduced-precision matrix
// mode) and the fallback of the bfloat16 path for shapes the tensor-core kernel refuses.
//
// Every output element is accumulated by one thread over k = 0..K-1 in ascending order, so a row's
// result does not depend on how many other rows the call has (the reference guarantees the same:
// cpp/src/cuda/cuda_gemm.cu:37-45). Tiling after cpp/src/cuda/cuda_gemm.cu:80-150 in spirit only.
//
// Epilogues: STORE (T out = acc + bias), ADD (float out += acc + bias: the residual sum),
// F32 (float out = acc + bias: logits), SWIGLU (two accumulators, W rows n and n + N:
// T out = silu(gate) * up, silu(g) = g / (1 + exp(-g)), cpp/src/ops.cpp:86-93), GLU (the same with limits and constants),
// GEGLU (gelu(gate) * up).
#include "common.cuh"

template <typename T, int EPI>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ W, const float* __restrict__ bias,
                 void* __restrict__ out, int M, int N, int K, int lda, int ldo, const NibGlu glu) {
    constexpr int BM = 64, BN = 64, BK = 16, TM = 4, TN = 4;
    constexpr bool DUAL = epi_dual(EPI);
    __shared__ float As[BK][BM + 1];
    __shared__ float Ws[BK][BN + 1];
    __shared__ float Us[DUAL ? BK : 1][DUAL ? BN + 1 : 1];

    const int tid = threadIdx.x;
    const int tx = tid % 16, ty = tid / 16;     // thread's 4x4 micro tile: rows ty*4.., cols tx*4..
    const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;

    float acc[TM][TN];
    float acc2[DUAL ? TM : 1][DUAL ? TN : 1];
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN; ++j) acc[i][j] = 0.f;
    if (DUAL) {
#pragma unroll
        for (int i = 0; i < (DUAL ? TM : 1); ++i)
#pragma unroll
            for (int j = 0; j < (DUAL ? TN : 1); ++j) acc2[i][j] = 0.f;
    }

    for (int k0 = 0; k0 < K; k0 += BK) {
        // 64 rows x 16 k = 1024 elements per operand, 4 per thread
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int e = tid + i * 256;
            const int r = e / BK, kk = e % BK;
            const int gk = k0 + kk;
            float a = 0.f, w = 0.f, u = 0.f;
            if (gk < K) {
                if (m0 + r < M) a = Elem<T>::load(A + (size_t)(m0 + r) * lda + gk);
                if (n0 + r < N) {
                    w = Elem<T>::load(W + (size_t)(n0 + r) * K + gk);
                    if (DUAL) u = Elem<T>::load(W + (size_t)(N + n0 + r) * K + gk);
                }
            }
            As[kk][r] = a;
            Ws[kk][r] = w;
            if (DUAL) Us[kk][r] = u;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < BK; ++kk) {
            float a[TM], w[TN];
#pragma unroll
            for (int i = 0; i < TM; ++i) a[i] = As[kk][ty * TM + i];
#pragma unroll
            for (int j = 0; j < TN; ++j) w[j] = Ws[kk][tx * TN + j];
#pragma unroll
            for (int i = 0; i < TM; ++i)
#pragma unroll
                for (int j = 0; j < TN; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
            if (DUAL) {
                float u[TN];
#pragma unroll
                for (int j = 0; j < TN; ++j) u[j] = Us[kk][tx * TN + j];
#pragma unroll
                for (int i = 0; i < (DUAL ? TM : 1); ++i)
#pragma unroll
                    for (int j = 0; j < (DUAL ? TN : 1); ++j) acc2[i][j] = fmaf(a[i], u[j], acc2[i][j]);
            }
        }
        __syncthreads();
    }

#pragma unroll
    for (int i = 0; i < TM; ++i) {
        const int m = m0 + ty * TM + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < TN; ++j) {
            const int n = n0 + tx * TN + j;
            if (n >= N) continue;
            float v = acc[i][j] + (bias ? bias[n] : 0.f);
            const size_t o = (size_t)m * ldo + n;
            if (EPI == EPI_STORE) {
                Elem<T>::store((T*)out + o, v);
            } else if (EPI == EPI_ADD) {
                ((float*)out)[o] += v;
            } else if (EPI == EPI_F32) {
                ((float*)out)[o] = v;
            } else {
                const float g = v, u = acc2[DUAL ? i : 0][DUAL ? j : 0];
                Elem<T>::store((T*)out + o, EPI == EPI_GLU ? nib_glu_exact(glu, g, u) : EPI == EPI_GEGLU ? nib_geglu_exact(g, u) : g / (1.0f + expf(-g)) * u);
            }
        }
    }
}

template <typename T>
static int launch_simt(const void* A, const void* W, const float* bias, void* out, int M, int N, int K,
                       int lda, int ldo, int epi, const NibGlu& glu, cudaStream_t stream) {
    dim3 grid(ceil_div(N, 64), ceil_div(M, 64));
    dim3 block(256);
    switch (epi) {
        case EPI_STORE: gemm_simt_kernel<T, EPI_STORE><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        case EPI_ADD: gemm_simt_kernel<T, EPI_ADD><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        case EPI_F32: gemm_simt_kernel<T, EPI_F32><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        case EPI_SWIGLU: gemm_simt_kernel<T, EPI_SWIGLU><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        case EPI_GLU: gemm_simt_kernel<T, EPI_GLU><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        case EPI_GEGLU: gemm_simt_kernel<T, EPI_GEGLU><<<grid, block, 0, stream>>>((const T*)A, (const T*)W, bias, out, M, N, K, lda, ldo, glu); break;
        default: nib_set_error("gemm: unknown epilogue %d", epi); return 1;
    }
    NIB_LAUNCH_CHECK();
    return 0;
}

// A [M, K] with row stride lda; W [N, K] (SWIGLU: [2N, K], gate rows then up rows); out [M, N] with
// row stride ldo. epi: 0 store, 1 add into float, 2 store float, 3 swiglu, 5 the gated form with the constants glu, 6 geglu.
NIB_API int nib_gemm_simt(const void* A, const void* W, const float* bias, void* out, int M, int N, int K,
                          int lda, int ldo, int epi, int dtype, const NibGlu* glu, cudaStream_t stream) {
    NIB_REQUIRE(M >= 0 && N > 0 && K > 0 && lda >= K && ldo >= N, "gemm: bad sizes M=%d N=%d K=%d lda=%d ldo=%d", M, N, K, lda, ldo);
    NIB_REQUIRE(!epi_dual(epi) || bias == nullptr, "gemm: the gated epilogues take no bias");
    NIB_REQUIRE(epi != EPI_GLU || glu != nullptr, "gemm: the gated epilogue needs its constants");
    const NibGlu constants = glu != nullptr ? *glu : NibGlu{};
    if (M == 0) return 0;
    NIB_REQUIRE(ceil_div(M, 64) <= 65535, "gemm: M=%d is too large for one launch", M);
    if (dtype == NIB_F32) return launch_simt<float>(A, W, bias, out, M, N, K, lda, ldo, epi, constants, stream);
    if (dtype == NIB_BF16) return launch_simt<__nv_bfloat16>(A, W, bias, out, M, N, K, lda, ldo, epi, constants, stream);
    NIB_REQUIRE(false, "gemm: unknown dtype %d", dtype);
}

// ---------------------------------------------------------------------------------- block-diagonal product, few tokens
// out[b, t, n] = bias[b, n] + sum_k a[b, t, k] * w[b, n, k] for `blocks` independent square-ish blocks and a handful
// of tokens: one warp per (block, output feature) keeps its weight row in registers and walks the tokens, so a
// decode step reads every weight once and needs one launch for all blocks. a: [blocks, tokens, k] of T,
// w: [blocks, n, k] of T, bias: [blocks, n] floats or null, out: [blocks, tokens, n] floats.
template <typename T>
__global__ void __launch_bounds__(128)
block_diag_smallm_kernel(const T* __restrict__ a, const T* __restrict__ w, const float* __restrict__ bias, float* __restrict__ out,
                         int blocks, int tokens, int n, int k) {
    pdl_launch_dependents();
    pdl_wait();      // the activations come from the kernel before
    const long long wid = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (wid >= (long long)blocks * n) return;
    const int b = (int)(wid / n), f = (int)(wid % n);
    const T* wr = w + ((size_t)b * n + f) * k;
    const float bv = bias ? bias[(size_t)b * n + f] : 0.f;
    for (int t = 0; t < tokens; ++t) {
        const T* ar = a + ((size_t)b * tokens + t) * k;
        float acc = 0.f;
        for (int c = lane; c < k; c += 32) acc = fmaf(Elem<T>::load(wr + c), Elem<T>::load(ar + c), acc);
        acc = warp_sum(acc);
        if (lane == 0) out[((size_t)b * tokens + t) * n + f] = acc + bv;
    }
}

NIB_API int nib_block_diag_smallm(const void* a, const void* w, const float* bias, float* out, int blocks, int tokens, int n, int k,
                                  int dtype, cudaStream_t stream) {
    NIB_REQUIRE(blocks > 0 && tokens >= 0 && n > 0 && k > 0, "block-diagonal product: bad sizes");
    if (tokens == 0) return 0;
    const int grid = ceil_div((long long)blocks * n, 4);
    if (dtype == NIB_F32)
        NIB_CUDA(launch_pdl(block_diag_smallm_kernel<float>, dim3(grid), dim3(128), (size_t)0, stream, (const float*)a, (const float*)w, bias, out, blocks, tokens, n, k));
    else if (dtype == NIB_BF16)
        NIB_CUDA(launch_pdl(block_diag_smallm_kernel<__nv_bfloat16>, dim3(grid), dim3(128), (size_t)0, stream, (const __nv_bfloat16*)a, (const __nv_bfloat16*)w, bias, out, blocks, tokens, n, k));
    else
        NIB_REQUIRE(false, "block-diagonal product: unknown dtype %d", dtype);
    NIB_LAUNCH_CHECK();
    return 0;
}
