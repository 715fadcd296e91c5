// Grouped bfloat16 product on the 5th-generation tensor cores, for the experts of a mixture: rows sorted by expert, every expert's run
// padded to whole tiles of TILE_ROWS rows, each tile multiplied with its own expert's part of one fused weight,
//     C[r, n] = sum_k A[r, k] * W[expert * row_step + n, expert * col_step + k],   n < N, k < K,
// 32-bit accumulation in tensor memory.  `tile_expert` [row tiles] lives on the device (-1: a tile behind the last row): the number of
// rows an expert got is not known on the host, nothing is read back, and the launch is the same for every batch of one size.
//
// The main loop is the one of the product for many tokens: a cluster of two blocks on one 256 x 256 tile (tcgen05.mma with
// cta_group::2, each block loading its 128 rows of both operands by TMA, without multicast), a ring of six stages that runs on across
// tiles, two accumulators in tensor memory so that a tile's epilogue runs beside the next tile's main loop, one cluster per pair of SMs
// walking the tiles with the row tiles fastest (clusters side by side share an expert's weight tile in L2).  The end of K is zero-filled
// by TMA on the A side, so what W holds beyond an expert's columns counts for nothing (it is the next expert's, finite); columns beyond
// N are not stored.  K, col_step and W's row pitch are multiples of 8 (16-byte TMA coordinates).
#include <cuda.h>

#include "common.cuh"
#include "tcgen05.cuh"

SPY_MODULE(spy_gemm_grouped)

namespace {

using namespace tc;

constexpr int BM = 128, BK = 64, BN = 256, UMMA_K = 16;
constexpr int TILE_ROWS = 2 * BM;
constexpr int NUM_THREADS = 192;   // warp 0: TMA, warp 1: MMA + TMEM, warps 2..5: epilogue
constexpr int STAGES = 6;
constexpr int X_BYTES = BM * BK * 2, STAGE_BYTES = 2 * X_BYTES;      // 128 rows of A and 128 of W
constexpr size_t SMEM = (size_t)STAGES * STAGE_BYTES + 1024 /* alignment slack */ + 256 /* barriers */;

// Stores 32 consecutive columns of one row, in 16-byte pieces where the row allows it.
template <typename TC>
__device__ __forceinline__ void store_row32(TC* dst, const uint32_t (&r)[32], int valid)
{
    if (valid >= 32 && (reinterpret_cast<uintptr_t>(dst) & 15) == 0) {
        if constexpr (sizeof(TC) == 4) {
#pragma unroll
            for (int i = 0; i < 8; ++i)
                reinterpret_cast<float4*>(dst)[i] = make_float4(__uint_as_float(r[4 * i]), __uint_as_float(r[4 * i + 1]), __uint_as_float(r[4 * i + 2]),
                                                                __uint_as_float(r[4 * i + 3]));
        } else {
#pragma unroll
            for (int i = 0; i < 4; ++i)
                reinterpret_cast<uint4*>(dst)[i] = make_uint4(pack_bf16(__uint_as_float(r[8 * i]), __uint_as_float(r[8 * i + 1])),
                                                              pack_bf16(__uint_as_float(r[8 * i + 2]), __uint_as_float(r[8 * i + 3])),
                                                              pack_bf16(__uint_as_float(r[8 * i + 4]), __uint_as_float(r[8 * i + 5])),
                                                              pack_bf16(__uint_as_float(r[8 * i + 6]), __uint_as_float(r[8 * i + 7])));
        }
    } else {
#pragma unroll
        for (int i = 0; i < 32; ++i)
            if (i < valid) dst[i] = from_f32<TC>(__uint_as_float(r[i]));
    }
}

// The tiles of a cluster, in the order it walks them: number t is row tile t % row_tiles, column tile t / row_tiles.
struct Walk {
    int t, step, tiles, row_tiles;
    const int* tile_expert;
    int row_tile, col_tile, expert;
    __device__ Walk(int cluster, int clusters, int row_tiles_, int tiles_, const int* te) : t(cluster), step(clusters), tiles(tiles_), row_tiles(row_tiles_), tile_expert(te) {}
    __device__ bool next(int experts)
    {
        for (; t < tiles; t += step) {
            row_tile = t % row_tiles;
            expert = tile_expert[row_tile];
            if (expert < 0 || expert >= experts) continue;       // behind the last row
            col_tile = t / row_tiles;
            t += step;
            return true;
        }
        return false;
    }
};

template <typename TC>
__global__ void __launch_bounds__(NUM_THREADS, 1)
gemm_grouped_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, TC* __restrict__ out, long long ld,
                    const int* __restrict__ tile_expert, int experts, int row_tiles, int tiles, int N, int k_blocks, int row_step, int col_step, int* status)
{
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* tiles_s = smem;
    uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + (size_t)STAGES * STAGE_BYTES);   // the leader's are used
    uint64_t* empty_bar = full_bar + STAGES;   // every block's own
    uint64_t* acc_full = empty_bar + STAGES;   // [2] every block's own
    uint64_t* acc_empty = acc_full + 2;             // [2] the leader's are used: 256 arrivals
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t rank = cluster_ctarank();
    const int cluster = blockIdx.x >> 1, clusters = gridDim.x >> 1;
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(full_bar + s, 1);
            mbar_init(empty_bar + s, 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(acc_full + b, 1);
            mbar_init(acc_empty + b, 256);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc_pair(tmem_slot, 2u * BN);
    fence_before_sync();
    __syncthreads();
    cluster_sync();   // both blocks' barriers are initialised and their tensor memory is allocated before either is used from the other side
    fence_after_sync();
    const uint32_t tmem_base = *tmem_slot;

    pdl_launch_dependents();
    pdl_wait();                     // which expert a tile belongs to was worked out by a kernel ahead
    Walk walk(cluster, clusters, row_tiles, tiles, tile_expert);
    if (warp == 0) {
        if (lane == 0) {
            long long g = 0;
            bool ok = true;
            while (ok && walk.next(experts)) {
                const int a_row = walk.row_tile * TILE_ROWS + (int)rank * BM;
                const int w_row = walk.expert * row_step + walk.col_tile * BN + (int)rank * (BN / 2), w_col = walk.expert * col_step;
                for (int kb = 0; kb < k_blocks; ++kb, ++g) {
                    const int s = (int)(g % STAGES);
                    const uint32_t phase = (uint32_t)(g / STAGES) & 1;
                    if (g >= STAGES && !mbar_wait(empty_bar + s, phase ^ 1, abort_flag)) { ok = false; break; }
                    uint8_t* xs = tiles_s + (size_t)s * STAGE_BYTES;
                    if (rank == 0) mbar_expect_tx(full_bar + s, 2 * STAGE_BYTES);   // both blocks' bytes
                    const uint32_t leader_full = map_to_rank(smem_u32(full_bar + s), 0);
                    tma_load_2d_pair(smem_u32(xs), &map_a, kb * BK, a_row, leader_full);
                    tma_load_2d_pair(smem_u32(xs + X_BYTES), &map_w, w_col + kb * BK, w_row, leader_full);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0 && rank == 0) {
            const uint32_t idesc = instr_desc_bf16(2 * BM, BN, false, false);
            long long g = 0;
            bool ok = true;
            for (int i = 0; ok && walk.next(experts); ++i) {
                const int buf = i & 1;
                const uint32_t aph = (uint32_t)(i >> 1) & 1;
                if (i >= 2) ok = mbar_wait(acc_empty + buf, aph ^ 1, abort_flag);   // both blocks' epilogues have read this buffer's last tile
                if (!ok) break;
                fence_after_sync();
                const uint32_t acc = tmem_base + (uint32_t)buf * BN;
                for (int kb = 0; kb < k_blocks; ++kb, ++g) {
                    const int s = (int)(g % STAGES);
                    const uint32_t phase = (uint32_t)(g / STAGES) & 1;
                    ok = mbar_wait(full_bar + s, phase, abort_flag);
                    if (!ok) break;
                    fence_after_sync();
                    const uint8_t* xs = tiles_s + (size_t)s * STAGE_BYTES;
                    const uint64_t dx = desc_k_major(smem_u32(xs)), dy = desc_k_major(smem_u32(xs + X_BYTES));
#pragma unroll
                    for (int k = 0; k < BK / UMMA_K; ++k) {
                        const uint64_t adv = (uint64_t)((k * UMMA_K * 2) >> 4);
                        umma_pair(acc, dx + adv, dy + adv, idesc, (kb > 0 || k > 0) ? 1u : 0u);
                    }
                    umma_commit_pair(empty_bar + s);
                }
                if (ok) umma_commit_pair(acc_full + buf);
            }
        }
    } else {
        const int quarter = warp & 3;
        bool ok = true;
        for (int i = 0; ok && walk.next(experts); ++i) {
            const int buf = i & 1;
            const uint32_t aph = (uint32_t)(i >> 1) & 1;
            ok = mbar_wait(acc_full + buf, aph, abort_flag);
            if (!ok) break;
            fence_after_sync();
            const size_t row = (size_t)walk.row_tile * TILE_ROWS + rank * BM + quarter * 32 + lane;
            const int n0 = walk.col_tile * BN;
#pragma unroll 1
            for (int c = 0; c < BN && n0 + c < N; c += 32) {
                uint32_t r[32];
                tmem_load<32>(tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(buf * BN + c), r);
                tmem_wait_ld();
                store_row32<TC>(out + row * ld + n0 + c, r, min(32, N - n0 - c));
            }
            fence_before_sync();
            if (rank == 0) mbar_arrive(acc_empty + buf);
            else mbar_arrive_cluster(map_to_rank(smem_u32(acc_empty + buf), 0));
        }
    }

    fence_before_sync();
    __syncthreads();
    if (*abort_flag) {
        if (threadIdx.x == 0) {
            const unsigned long long t0 = global_timer();
            while (global_timer() - t0 < 2000000ull) { }
            report_status(status, SPY_STATUS_WAIT_TIMEOUT, (int)blockIdx.x);
        }
        __syncthreads();
    }
    cluster_sync();   // neither block leaves (and frees tensor memory the pair shares) while the other may still use it
    if (warp == 1) {
        fence_after_sync();
        tmem_dealloc_pair(tmem_base, 2u * BN);
    }
}

int make_map(CUtensorMap* map, const void* ptr, long long rows, long long cols, long long ld)
{
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn) SPY_FAIL("gemm_grouped: cuTensorMapEncodeTiled is not available from the driver");
    cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    cuuint32_t box[2] = {(cuuint32_t)BK, (cuuint32_t)BM};
    cuuint32_t elem[2] = {1, 1};
    CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) SPY_FAIL("gemm_grouped: cuTensorMapEncodeTiled failed with code %d (rows %lld, columns %lld, pitch %lld)", (int)r, rows, cols, ld);
    return 0;
}

template <typename TC>
int launch(const CUtensorMap& ma, const CUtensorMap& mw, void* C, long long ldc, const int* tile_expert, int experts, int row_tiles, int N, int k_blocks,
           int row_step, int col_step, int* status, cudaStream_t stream)
{
    static int clusters_of_device[SPY_MAX_DEVICES] = {};
    int& clusters_max = clusters_of_device[spy_device()];
    if (clusters_max == 0) {
        SPY_CUDA(cudaFuncSetAttribute(gemm_grouped_kernel<TC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM));
        const int sms = spy_sm_count();
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(sms / 2 * 2);
        cfg.blockDim = dim3(NUM_THREADS);
        cfg.dynamicSmemBytes = SMEM;
        cudaLaunchAttribute attr[1];
        attr[0].id = cudaLaunchAttributeClusterDimension;
        attr[0].val.clusterDim.x = 2;
        attr[0].val.clusterDim.y = 1;
        attr[0].val.clusterDim.z = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 1;
        int active = 0;
        SPY_CUDA(cudaOccupancyMaxActiveClusters(&active, gemm_grouped_kernel<TC>, &cfg));
        if (active <= 0) SPY_FAIL("gemm_grouped: no cluster of two blocks fits the device");
        clusters_max = active < sms / 2 ? active : sms / 2;
    }
    const long long tiles = (long long)row_tiles * ((N + BN - 1) / BN);
    if (tiles > 0x7fffffffLL) SPY_FAIL("gemm_grouped: %lld tiles exceed the kernel's range", tiles);
    const int clusters = (int)(tiles < clusters_max ? tiles : clusters_max);
    spy_launch_cluster(gemm_grouped_kernel<TC>, dim3(2 * clusters), dim3(NUM_THREADS), SMEM, stream, 2u, ma, mw, (TC*)C, ldc, tile_expert, experts, row_tiles,
                       (int)tiles, N, k_blocks, row_step, col_step, status);
    SPY_CHECK_LAUNCH("gemm_grouped");
    return 0;
}

}  // namespace

extern "C" int spy_gemm_grouped_tile_rows() { return TILE_ROWS; }

// A [rows, K] with row pitch lda (rows a multiple of TILE_ROWS), W [w_rows, w_cols] with row pitch ldw, C [rows, N] with pitch ldc;
// tile_expert [rows / TILE_ROWS] on the device.
extern "C" int spy_gemm_grouped(const void* A, long long lda, int rows, int K, const void* W, long long ldw, int w_rows, int w_cols, void* C, int c_dtype,
                                long long ldc, int N, const int* tile_expert, int experts, int row_step, int col_step, int* status, cudaStream_t stream)
{
    if (rows <= 0 || N <= 0) return 0;
    if (rows % TILE_ROWS != 0 || K <= 0 || experts <= 0) SPY_FAIL("gemm_grouped: %d rows, K %d, %d experts", rows, K, experts);
    if (K % 8 != 0 || lda % 8 != 0 || ldw % 8 != 0 || col_step % 8 != 0 || ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(W)) & 15) != 0)
        SPY_FAIL("gemm_grouped: rows and columns must start on 16-byte borders (K %d, pitches %lld and %lld, column step %d)", K, lda, ldw, col_step);
    if ((long long)(experts - 1) * row_step + N > w_rows || (long long)(experts - 1) * col_step + K > w_cols)
        SPY_FAIL("gemm_grouped: %d experts' parts of %d x %d do not fit a weight of %d x %d", experts, N, K, w_rows, w_cols);
    CUtensorMap ma, mw;
    if (make_map(&ma, A, rows, K, lda) || make_map(&mw, W, w_rows, w_cols, ldw)) return 1;
    const int k_blocks = (K + BK - 1) / BK, row_tiles = rows / TILE_ROWS;
    if (c_dtype == SPY_F32) return launch<float>(ma, mw, C, ldc, tile_expert, experts, row_tiles, N, k_blocks, row_step, col_step, status, stream);
    if (c_dtype == SPY_BF16) return launch<bf16>(ma, mw, C, ldc, tile_expert, experts, row_tiles, N, k_blocks, row_step, col_step, status, stream);
    SPY_FAIL("gemm_grouped: unknown dtype code %d", c_dtype);
}
