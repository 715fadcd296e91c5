// Plain matrix product on the CUDA cores, any sizes and any mix of 32-bit and bfloat16
// storage:  C[M, N] = A[M, K] . W[N, K]^T, every product and sum in 32-bit (FFMA; no tensor
// cores, no TF32).  It is the float32 path's matrix product (bfloat16 weights are widened
// exactly on the fly, so the weights are kept once) and the bfloat16 path's fallback for
// shapes the tensor-core kernel refuses.  Each output element is one thread's sum over k in
// ascending order, so a row's result does not depend on M or on what else is in the batch.
// The reference's counterpart on this path is its CPU Linear (spymaster2h/spyinfer
// src/backends/cpu/x64/kernels.cpp:95-166); its CUDA path calls cuBLAS in half precision.
#include "common.cuh"

SPY_MODULE(spy_gemm_simt)

constexpr int BM = 64, BN = 64, BK = 16, TM = 4, TN = 4;

template <typename TA, typename TW, typename TC>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const TA* __restrict__ A, long long lda, const TW* __restrict__ W, long long ldw, TC* __restrict__ C, long long ldc,
                 int M, int N, int K)
{
    __shared__ float As[BK][BM + 4];
    __shared__ float Ws[BK][BN + 4];
    pdl_enter();
    const int tid = threadIdx.x;
    const int tx = tid % 16, ty = tid / 16;
    const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
    // each thread stages four consecutive k of one row of each tile
    const int lr = tid / 4, lk = (tid % 4) * 4;
    float acc[TM][TN];
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
        for (int j = 0; j < TN; ++j) acc[i][j] = 0.f;

    for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int k = k0 + lk + i;
            const int m = m0 + lr, n = n0 + lr;
            As[lk + i][lr] = (m < M && k < K) ? to_f32(A[(size_t)m * lda + k]) : 0.f;
            Ws[lk + i][lr] = (n < N && k < K) ? to_f32(W[(size_t)n * ldw + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < BK; ++k) {
            float a[TM], w[TN];
#pragma unroll
            for (int i = 0; i < TM; ++i) a[i] = As[k][ty * TM + i];
#pragma unroll
            for (int j = 0; j < TN; ++j) w[j] = Ws[k][tx * TN + j];
#pragma unroll
            for (int i = 0; i < TM; ++i)
#pragma unroll
                for (int j = 0; j < TN; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
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
            if (n < N) C[(size_t)m * ldc + n] = from_f32<TC>(acc[i][j]);
        }
    }
}

// Row strides lda/ldw/ldc are in elements.

// A product with few output columns (a router, a gate of one number a token): a block of eight warps owns one row of A (or four) and
// up to SKINNY_NG columns at a time; its threads stride over k, so every load is a run of consecutive elements and many are
// under way at once, and the threads' sums are added in a fixed order.  A row's result does not depend on M either.
constexpr int SKINNY_N = 32, SKINNY_NG = 16, SKINNY_THREADS = 256;

// ROWS rows of A a block (every weight element a block fetches serves ROWS of them; a row's sums are formed in the same order
// whatever ROWS is).  One row a block is what runs: four rows a block, tried for steps of many rows, were no faster (the weights of
// a product this narrow stay in L1/L2, and the accumulators of four rows cost occupancy).
template <typename TA, typename TW, typename TC, int ROWS>
__global__ void __launch_bounds__(SKINNY_THREADS)
gemm_skinny_kernel(const TA* __restrict__ A, long long lda, const TW* __restrict__ W, long long ldw, TC* __restrict__ C, long long ldc,
                   int M, int N, int K)
{
    __shared__ float part[ROWS][SKINNY_THREADS / 32][SKINNY_NG];
    pdl_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long m0 = (long long)blockIdx.x * ROWS;
    const TA* a[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) a[r] = A + (m0 + r < M ? m0 + r : m0) * lda;      // rows beyond the last: the first again, never stored
    for (int n0 = 0; n0 < N; n0 += SKINNY_NG) {
        float acc[ROWS][SKINNY_NG];
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
#pragma unroll
            for (int j = 0; j < SKINNY_NG; ++j) acc[r][j] = 0.f;
#pragma unroll(ROWS == 1 ? 4 : 2)
        for (int k = threadIdx.x; k < K; k += SKINNY_THREADS) {
            float av[ROWS];
#pragma unroll
            for (int r = 0; r < ROWS; ++r) av[r] = to_f32(a[r][k]);
#pragma unroll
            for (int j = 0; j < SKINNY_NG; ++j)
                if (n0 + j < N) {
                    const float w = to_f32(W[(size_t)(n0 + j) * ldw + k]);
#pragma unroll
                    for (int r = 0; r < ROWS; ++r) acc[r][j] = fmaf(av[r], w, acc[r][j]);
                }
        }
#pragma unroll
        for (int r = 0; r < ROWS; ++r)
#pragma unroll
            for (int j = 0; j < SKINNY_NG; ++j) {
                if (n0 + j >= N) break;                   // the same for every thread
                const float sum = warp_sum(acc[r][j]);
                if (lane == 0) part[r][warp][j] = sum;
            }
        __syncthreads();
        for (int i = threadIdx.x; i < ROWS * SKINNY_NG; i += SKINNY_THREADS) {
            const int r = i / SKINNY_NG, j = i % SKINNY_NG;
            if (m0 + r < M && n0 + j < N) {
                float sum = 0.f;
#pragma unroll
                for (int w = 0; w < SKINNY_THREADS / 32; ++w) sum += part[r][w][j];
                C[(m0 + r) * ldc + n0 + j] = from_f32<TC>(sum);
            }
        }
        __syncthreads();
    }
}

// The same in runs of four (16-byte accesses of 32-bit rows, 8-byte ones of bfloat16 rows) where the rows allow it.
__device__ __forceinline__ void load4(const float* p, float (&v)[4])
{
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&v)[4])
{
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x), b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
    v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
}

template <typename TA, typename TW, typename TC, int NG>
__global__ void __launch_bounds__(SKINNY_THREADS)
gemm_skinny_quads_kernel(const TA* __restrict__ A, long long lda, const TW* __restrict__ W, long long ldw, TC* __restrict__ C, long long ldc, int N, int K)
{
    __shared__ float part[SKINNY_THREADS / 32][NG];
    pdl_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const long long m = blockIdx.x;
    const TA* a = A + m * lda;
    for (int n0 = 0; n0 < N; n0 += NG) {
        float acc[NG];
#pragma unroll
        for (int j = 0; j < NG; ++j) acc[j] = 0.f;
        for (int k = 4 * threadIdx.x; k < K; k += 4 * SKINNY_THREADS) {
            float av[4];
            load4(a + k, av);
#pragma unroll
            for (int j = 0; j < NG; ++j)
                if (n0 + j < N) {
                    float w[4];
                    load4(W + (size_t)(n0 + j) * ldw + k, w);
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[j] = fmaf(av[e], w[e], acc[j]);
                }
        }
#pragma unroll
        for (int j = 0; j < NG; ++j) {
            if (n0 + j >= N) break;                       // the same for every thread
            const float sum = warp_sum(acc[j]);
            if (lane == 0) part[warp][j] = sum;
        }
        __syncthreads();
        if (threadIdx.x < NG && n0 + threadIdx.x < N) {
            float sum = 0.f;
#pragma unroll
            for (int w = 0; w < SKINNY_THREADS / 32; ++w) sum += part[w][threadIdx.x];
            C[m * ldc + n0 + threadIdx.x] = from_f32<TC>(sum);
        }
        __syncthreads();
    }
}

extern "C" int spy_gemm_simt(const void* A, int a_dtype, long long lda, const void* W, int w_dtype, long long ldw, void* C, int c_dtype,
                             long long ldc, int M, int N, int K, cudaStream_t stream)
{
    if (M <= 0 || N <= 0) return 0;
    if (K <= 0) SPY_FAIL("gemm: K %d must be positive", K);
    if (lda < K || ldw < K || ldc < N) SPY_FAIL("gemm: row strides %lld/%lld/%lld are shorter than the rows", lda, ldw, ldc);
    if (N <= SKINNY_N) {                                      // chosen by the weight's shape alone, as every choice of a product is
        SPY_DISPATCH_DTYPE(a_dtype, TA, {
            SPY_DISPATCH_DTYPE(w_dtype, TW, {
                SPY_DISPATCH_DTYPE(c_dtype, TC, {
                    const bool quads = K % 4 == 0 && lda % 4 == 0 && ldw % 4 == 0 && reinterpret_cast<uintptr_t>(A) % (4 * sizeof(TA)) == 0
                                       && reinterpret_cast<uintptr_t>(W) % (4 * sizeof(TW)) == 0;
                    if (quads && N <= 8)
                        spy_launch(gemm_skinny_quads_kernel<TA, TW, TC, 8>, dim3((unsigned)M), dim3(SKINNY_THREADS), 0, stream, (const TA*)A, lda,
                                   (const TW*)W, ldw, (TC*)C, ldc, N, K);
                    else if (quads)
                        spy_launch(gemm_skinny_quads_kernel<TA, TW, TC, 16>, dim3((unsigned)M), dim3(SKINNY_THREADS), 0, stream, (const TA*)A, lda,
                                   (const TW*)W, ldw, (TC*)C, ldc, N, K);
                    else
                        spy_launch(gemm_skinny_kernel<TA, TW, TC, 1>, dim3((unsigned)M), dim3(SKINNY_THREADS), 0, stream, (const TA*)A, lda,
                               (const TW*)W, ldw, (TC*)C, ldc, M, N, K);
                })
            })
        })
        SPY_CHECK_LAUNCH("gemm_skinny");
        return 0;
    }
    const long long gy = ((long long)M + BM - 1) / BM;
    if (gy > 65535) SPY_FAIL("gemm: M %d exceeds the grid limit of this kernel (%d rows)", M, 65535 * BM);
    dim3 grid((N + BN - 1) / BN, (unsigned)gy);
    SPY_DISPATCH_DTYPE(a_dtype, TA, {
        SPY_DISPATCH_DTYPE(w_dtype, TW, {
            SPY_DISPATCH_DTYPE(c_dtype, TC, {
                spy_launch(gemm_simt_kernel<TA, TW, TC>, grid, dim3(256), 0, stream, (const TA*)A, lda, (const TW*)W, ldw, (TC*)C, ldc, M, N, K);
            })
        })
    })
    SPY_CHECK_LAUNCH("gemm_simt");
    return 0;
}
