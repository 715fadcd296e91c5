// Per-head bfloat16 products on the 5th-generation tensor cores, the two of attention through a latent:
//     out[t, h * out_head_stride + n] = sum_k in[t, h * in_head_stride + k] * W[h, n, k],   n < N, k < K,
// 32-bit accumulation.  Options as head_product (latent.cu) has them: `tail` elements that follow each head's K inputs go, rotated by a
// (cos, sin) table at the token's position (pairs (j, j + r) or (2j, 2j + 1)), to the columns after its N results; a gate multiplies
// the results by sigmoid(gate[t, gate_off + h * N + n]).
//
// A block takes 128 tokens of one head and 128 of its outputs: K blocks of 64 of both operands by TMA (the inputs as a tensor [tokens]
// [heads][K], so that what follows a head's K inputs is never read as one of them; the weights [heads][N][K]; what lies beyond any
// of the three sizes arrives as zero), tcgen05.mma 128 x 128 x 16 into tensor memory, and an epilogue of one thread a token.  The weights'
// tiles are requested before the wait for the kernels ahead.  K, strides and pitches are multiples of 8 (16-byte TMA coordinates).
#include <cuda.h>

#include "common.cuh"
#include "tcgen05.cuh"

SPY_MODULE(spy_head_gemm)

namespace {

using namespace tc;

constexpr int BM = 128, BN = 128, BK = 64, UMMA_K = 16;
constexpr int NUM_THREADS = 192;   // warp 0: TMA, warp 1: MMA + TMEM, warps 2..5: epilogue
constexpr int MAX_STAGES = 4;
constexpr int X_BYTES = BM * BK * 2, STAGE_BYTES = 2 * X_BYTES;

struct Args {
    const bf16* in;  long long in_ld;  int in_head_stride, K, k_blocks, stages;
    bf16* out;       long long out_ld; int out_head_stride, N;
    int tail;
    const float* rope; int rot_half, table_rows, interleaved; const int* positions;
    const void* gate; int gate_dtype; long long gate_ld; int gate_off;
    int T;
    int* status;
};

// element j of the rotated vector x[0 .. n) at a position whose table row is cs (cos, sin pairs)
__device__ __forceinline__ float rotated(const bf16* x, int j, int rot_half, int interleaved, const float* cs)
{
    if (j >= 2 * rot_half) return to_f32(x[j]);
    const int a = interleaved ? j >> 1 : (j < rot_half ? j : j - rot_half);
    const bool first = interleaved ? (j & 1) == 0 : j < rot_half;
    const float u = to_f32(x[interleaved ? 2 * a : a]), v = to_f32(x[interleaved ? 2 * a + 1 : a + rot_half]);
    const float c = cs[2 * a], s = cs[2 * a + 1];
    return first ? u * c - v * s : v * c + u * s;
}

// eight neighbouring elements from a 16-byte border
__device__ __forceinline__ void load8(const bf16* p, float (&v)[8])
{
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        v[2 * i] = __uint_as_float(w[i] << 16);
        v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8])
{
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8])
{
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}

// The rotated tail of one token's head.  `vec`: the tail, its rotated pairs and the rows are multiples of eight elements.
__device__ __forceinline__ void store_tail(const Args& A, const bf16* x, bf16* out, const float* cs, bool vec)
{
    if (!vec) {
        for (int j = 0; j < A.tail; ++j) out[j] = __float2bfloat16_rn(rotated(x, j, A.rot_half, A.interleaved, cs));
        return;
    }
    float c[2][8];
    if (!A.interleaved) {
        for (int a = 0; a < A.rot_half; a += 8) {
            float u[8], v[8], ru[8], rv[8];
            load8(x + a, u);
            load8(x + A.rot_half + a, v);
            load8(cs + 2 * a, c[0]);
            load8(cs + 2 * a + 8, c[1]);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float co = c[i >> 2][2 * (i & 3)], si = c[i >> 2][2 * (i & 3) + 1];
                ru[i] = u[i] * co - v[i] * si;
                rv[i] = v[i] * co + u[i] * si;
            }
            store8(out + a, ru);
            store8(out + A.rot_half + a, rv);
        }
    } else {
        for (int j = 0; j < 2 * A.rot_half; j += 8) {
            float u[8], ru[8];
            load8(x + j, u);
            load8(cs + j, c[0]);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                ru[2 * i] = u[2 * i] * c[0][2 * i] - u[2 * i + 1] * c[0][2 * i + 1];
                ru[2 * i + 1] = u[2 * i + 1] * c[0][2 * i] + u[2 * i] * c[0][2 * i + 1];
            }
            store8(out + j, ru);
        }
    }
    for (int j = 2 * A.rot_half; j < A.tail; j += 8) *reinterpret_cast<uint4*>(out + j) = *reinterpret_cast<const uint4*>(x + j);
}

__global__ void __launch_bounds__(NUM_THREADS)
head_gemm_kernel(const __grid_constant__ CUtensorMap map_in, const __grid_constant__ CUtensorMap map_w, const Args A)
{
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + (size_t)A.stages * STAGE_BYTES);
    uint64_t* empty_bar = full_bar + MAX_STAGES;
    uint64_t* acc_full = empty_bar + MAX_STAGES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_full + 1);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * BM, h = blockIdx.y, n0 = blockIdx.z * BN;

    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int s = 0; s < MAX_STAGES; ++s) {
            mbar_init(full_bar + s, 1);
            mbar_init(empty_bar + s, 1);
        }
        mbar_init(acc_full, 1);
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, BN);
    fence_before_sync();
    __syncthreads();
    fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            const int ahead = min(A.stages, A.k_blocks);
            for (int kb = 0; kb < ahead; ++kb) {
                mbar_expect_tx(full_bar + kb, STAGE_BYTES);
                tma_load_3d(smem_u32(smem + (size_t)kb * STAGE_BYTES + X_BYTES), &map_w, kb * BK, n0, h, full_bar + kb);
            }
            pdl_wait();
            for (int kb = 0; kb < ahead; ++kb) tma_load_3d(smem_u32(smem + (size_t)kb * STAGE_BYTES), &map_in, kb * BK, h, t0, full_bar + kb);
            for (int kb = ahead; kb < A.k_blocks; ++kb) {
                const int s = kb % A.stages;
                if (!mbar_wait(empty_bar + s, (uint32_t)(kb / A.stages - 1) & 1, abort_flag)) break;
                mbar_expect_tx(full_bar + s, STAGE_BYTES);
                tma_load_3d(smem_u32(smem + (size_t)s * STAGE_BYTES + X_BYTES), &map_w, kb * BK, n0, h, full_bar + s);
                tma_load_3d(smem_u32(smem + (size_t)s * STAGE_BYTES), &map_in, kb * BK, h, t0, full_bar + s);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const uint32_t idesc = instr_desc_bf16(BM, BN, false, false);
            bool ok = true;
            for (int kb = 0; kb < A.k_blocks; ++kb) {
                const int s = kb % A.stages;
                ok = mbar_wait(full_bar + s, (uint32_t)(kb / A.stages) & 1, abort_flag);
                if (!ok) break;
                fence_after_sync();
                const uint32_t xs = smem_u32(smem + (size_t)s * STAGE_BYTES);
#pragma unroll
                for (int k = 0; k < BK / UMMA_K; ++k)
                    umma(tmem_base, desc_k_major(xs + k * UMMA_K * 2), desc_k_major(xs + X_BYTES + k * UMMA_K * 2), idesc, (kb > 0 || k > 0) ? 1u : 0u);
                umma_commit(empty_bar + s);
            }
            if (ok) umma_commit(acc_full);
        }
    } else {
        const int quarter = warp & 3, t = t0 + quarter * 32 + lane;
        const bool row_ok = t < A.T;
        pdl_wait();
        bf16* out = A.out + (size_t)(row_ok ? t : 0) * A.out_ld + (size_t)h * A.out_head_stride;
        if (A.tail > 0 && blockIdx.z == 0 && row_ok) {
            const int pos = A.positions[t];
            if (A.rot_half > 0 && (pos < 0 || pos >= A.table_rows)) report_status(A.status, SPY_STATUS_BAD_POSITION, t);
            else {
                const bf16* x = A.in + (size_t)t * A.in_ld + (size_t)h * A.in_head_stride + A.K;
                const float* cs = A.rope + (size_t)(A.rot_half ? pos : 0) * A.rot_half * 2;
                const bool vec = A.tail % 8 == 0 && A.rot_half % 8 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out + A.N) | reinterpret_cast<uintptr_t>(cs)) & 15) == 0;
                store_tail(A, x, out + A.N, cs, vec);
            }
        }
        if (mbar_wait(acc_full, 0, abort_flag)) {
            fence_after_sync();
            const size_t gate_at = (size_t)(row_ok ? t : 0) * A.gate_ld + A.gate_off + (size_t)h * A.N;
#pragma unroll 1
            for (int c = 0; c < BN && n0 + c < A.N; c += 32) {
                uint32_t r[32];
                tmem_load<32>(tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)c, r);
                tmem_wait_ld();
                if (!row_ok) continue;
                const int valid = min(32, A.N - n0 - c);
                const size_t gate_c = gate_at + n0 + c;
                const bool gate_bf16 = A.gate_dtype == SPY_BF16;
                if (A.gate != nullptr && valid == 32 && (((reinterpret_cast<uintptr_t>(A.gate) + gate_c * (gate_bf16 ? 2 : 4)) & 15) == 0)) {
                    float g[4][8];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (gate_bf16) load8((const bf16*)A.gate + gate_c + 8 * i, g[i]);
                        else load8((const float*)A.gate + gate_c + 8 * i, g[i]);
                    }
#pragma unroll
                    for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * (1.0f / (1.0f + expf(-g[i >> 3][i & 7]))));
                } else if (A.gate != nullptr) {
#pragma unroll
                    for (int i = 0; i < 32; ++i) {
                        if (i < valid) {
                            const size_t at = gate_at + n0 + c + i;
                            const float g = A.gate_dtype == SPY_BF16 ? to_f32(((const bf16*)A.gate)[at]) : ((const float*)A.gate)[at];
                            r[i] = __float_as_uint(__uint_as_float(r[i]) / (1.0f + expf(-g)));
                        }
                    }
                }
                bf16* dst = out + n0 + c;
                if (valid == 32 && (reinterpret_cast<uintptr_t>(dst) & 15) == 0) {
#pragma unroll
                    for (int i = 0; i < 4; ++i)
                        reinterpret_cast<uint4*>(dst)[i] = make_uint4(pack_bf16(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1])),
                                                                      pack_bf16(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3])),
                                                                      pack_bf16(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5])),
                                                                      pack_bf16(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7])));
                } else {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (i < valid) dst[i] = __float2bfloat16_rn(__uint_as_float(r[i]));
                }
            }
        }
    }

    fence_before_sync();
    __syncthreads();
    if (*abort_flag) {
        if (threadIdx.x == 0) {
            const unsigned long long start = global_timer();
            while (global_timer() - start < 2000000ull) { }   // let copies in flight land before the shared memory is released
            report_status(A.status, SPY_STATUS_WAIT_TIMEOUT, (int)blockIdx.x);
        }
        __syncthreads();
    }
    if (warp == 1) {
        fence_after_sync();
        tmem_dealloc(tmem_base, BN);
    }
}

int make_map(CUtensorMap* map, const void* ptr, long long d0, long long d1, long long d2, long long pitch1, long long pitch2, int box1, int box2)
{
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn) SPY_FAIL("head_gemm: cuTensorMapEncodeTiled is not available from the driver");
    cuuint64_t dims[3] = {(cuuint64_t)d0, (cuuint64_t)d1, (cuuint64_t)d2};
    cuuint64_t strides[2] = {(cuuint64_t)pitch1 * 2, (cuuint64_t)pitch2 * 2};
    cuuint32_t box[3] = {(cuuint32_t)BK, (cuuint32_t)box1, (cuuint32_t)box2};
    cuuint32_t elem[3] = {1, 1, 1};
    CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) SPY_FAIL("head_gemm: cuTensorMapEncodeTiled failed with code %d (%lld x %lld x %lld, pitches %lld and %lld)", (int)r, d0, d1, d2, pitch1, pitch2);
    return 0;
}

}  // namespace

// in [tokens, in_ld]: head h's K inputs (and `tail` more) start at column h * in_head_stride.  W [heads][N][K].  out [tokens, out_ld]: head
// h's N results (and the rotated tail) start at column h * out_head_stride.  gate [tokens, gate_ld] of gate_dtype, or null.
extern "C" int spy_head_gemm(const void* in, long long in_ld, int in_head_stride, int K, const void* W, int N, void* out, long long out_ld,
                             int out_head_stride, int tail, const float* rope, int rot_half, int table_rows, int interleaved, const int* positions,
                             const void* gate, int gate_dtype, long long gate_ld, int gate_off, int tokens, int heads, int* status, cudaStream_t stream)
{
    if (tokens <= 0) return 0;
    if (heads <= 0 || heads > 65535 || K <= 0 || N <= 0 || tail < 0 || (N + BN - 1) / BN > 65535) SPY_FAIL("head_gemm: %d heads, K %d, N %d, tail %d", heads, K, N, tail);
    if (K % 8 != 0 || in_ld % 8 != 0 || in_head_stride % 8 != 0 || ((reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(W)) & 15) != 0)
        SPY_FAIL("head_gemm: heads must start on 16-byte borders (K %d, pitch %lld, head stride %d)", K, in_ld, in_head_stride);
    if (tail > 0 && (positions == nullptr || 2 * rot_half > tail || (rot_half > 0 && rope == nullptr))) SPY_FAIL("head_gemm: the rotated tail needs positions and a table that fits it");
    if (in_head_stride < K + tail || out_head_stride < N + tail) SPY_FAIL("head_gemm: a head's columns overlap the next head's");
    CUtensorMap mi, mw;
    if (make_map(&mi, in, K, heads, tokens, in_head_stride, in_ld, 1, BM) || make_map(&mw, W, K, N, heads, K, (long long)N * K, BN, 1)) return 1;
    const int k_blocks = (K + BK - 1) / BK, stages = k_blocks < MAX_STAGES ? k_blocks : MAX_STAGES;
    const Args A = {(const bf16*)in, in_ld, in_head_stride, K, k_blocks, stages, (bf16*)out, out_ld, out_head_stride, N, tail, rope, rot_half, table_rows,
                    interleaved, positions, gate, gate_dtype, gate_ld, gate_off, tokens, status};
    const size_t smem = (size_t)stages * STAGE_BYTES + 1024 /* alignment slack */ + 128 /* barriers */;
    SPY_ONCE_PER_DEVICE {
        SPY_CUDA(cudaFuncSetAttribute(head_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_STAGES * STAGE_BYTES + 1024 + 128));
    }
    spy_launch(head_gemm_kernel, dim3((tokens + BM - 1) / BM, heads, (N + BN - 1) / BN), dim3(NUM_THREADS), smem, stream, mi, mw, A);
    SPY_CHECK_LAUNCH("head_gemm");
    return 0;
}
