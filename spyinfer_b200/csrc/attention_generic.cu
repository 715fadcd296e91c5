// Attention over the paged cache for any mix of queries: one block per (query token, head).
// This is the plain kernel: it takes every head size (a multiple of 4 elements), every page
// size, 32-bit or bfloat16 storage, and computes everything in 32-bit with expf.  It is the
// engine's float32 path and the fallback of the bfloat16 path for sizes its fast kernels
// refuse.  A cache of one plane (`planes` = 1) holds keys only and the values are the keys
// themselves (a latent that both are made of): V rows are then read from the K plane.  Head
// sizes that are no multiple of 4 take element-wise loads.
//
// A query at position p of sequence s sees the keys j with lo <= j <= p, lo = 0 or
// p - window + 1; key j lies in page block_table[s, j / page_size], slot j % page_size.
// kv head = head / (nh / nkv); score = (q . k) * scale; p = exp(score - max) / sum;
// o = sum p v.  Formula: spymaster2h/spyinfer src/backends/cpu/cpu_attention.cpp:89-135.
// Keys are processed in chunks of 128 that start at multiples of 128 of the absolute
// position, so the result of a query does not depend on how the batch was cut.
// Two options of the mask and the softmax: with a window, `keep_first` > 0 lets every query also see
// the keys at the sequence's first keep_first positions (at their true positions); `sink` != 0 adds one
// to the softmax's denominator (a key of score 0 that has no value): p = exp(score) / (1 + sum exp(score)).
// SpyScores (common.cuh) caps the scores, takes a distance bias off, adds a learned sink a head, scales the result.
#include "common.cuh"

SPY_MODULE(spy_attention_generic)

constexpr int CHUNK = 128;
constexpr int ACC = 8;       // output elements a thread owns: head sizes up to ACC * CHUNK

template <typename T> struct Vec4;
template <> struct Vec4<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4])
    {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
};
template <> struct Vec4<bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[4])
    {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x);
        const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    }
};

template <typename TA, typename TC>
__global__ void __launch_bounds__(CHUNK)
attention_generic_kernel(const TA* __restrict__ q, long long q_row_stride, TA* __restrict__ out, const TC* __restrict__ pages,
                         const int* __restrict__ block_table, int table_width, int page_size, int num_pages, int nh, int nkv, int hd,
                         const int* __restrict__ positions, const int* __restrict__ seq_of_token, int window, float scale, int* status, int planes,
                         int keep_first, int sink, SpyScores sc)
{
    extern __shared__ float smem[];
    pdl_enter();
    float* q_s = smem;                       // hd
    float* p_s = q_s + hd;                   // CHUNK
    long long* row_s = (long long*)(p_s + CHUNK + (hd & 1));  // CHUNK offsets of K rows (elements); 8-byte aligned: hd + (hd & 1) and CHUNK are even
    float* scratch = (float*)(row_s + CHUNK);      // 33

    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int pos = positions[t];
    const int seq = seq_of_token[t];
    const int kvh = h / (nh / nkv);
    const int* bt = block_table + (size_t)seq * table_width;
    const long long v_offset = planes == 2 ? (long long)nkv * page_size * hd : 0;  // from a K row to its V row (one plane: the values are the keys)
    const bool quads = (hd & 3) == 0;

    const TA* q_row = q + (size_t)t * q_row_stride + (size_t)h * hd;
    for (int d = tid; d < hd; d += CHUNK) q_s[d] = to_f32(q_row[d]);

    const int lo = spy_first_key(pos, window);
    float m = -INFINITY, l = 0.f;
    float acc[ACC];                       // dims tid, tid + 128, tid + 256, ...
#pragma unroll
    for (int r = 0; r < ACC; ++r) acc[r] = 0.f;
    __syncthreads();

    const int kept = min(keep_first, lo);             // the keys 0 .. kept - 1 lie before the window and are seen all the same
    const int kept_chunks = (kept + CHUNK - 1) / CHUNK;
    for (int c = 0; c <= pos / CHUNK; ++c) {
        if (c >= kept_chunks && c < lo / CHUNK) {
            c = lo / CHUNK - 1;                       // nothing to see between the kept keys and the window
            continue;
        }
        const int j = c * CHUNK + tid;
        bool valid = (j >= lo || j < kept) && j <= pos;
        long long row = 0;
        if (valid) {
            const int lp = j / page_size;
            const int page = lp < table_width ? bt[lp] : -1;
            if (page < 0 || page >= num_pages) {
                report_status(status, SPY_STATUS_BAD_PAGE, t);
                valid = false;
            } else {
                row = ((((long long)page * planes) * nkv + kvh) * page_size + j % page_size) * hd;
            }
        }
        float s = -INFINITY;
        if (valid) {
            const TC* k = pages + row;
            float dot = 0.f;
            if (quads) {
                for (int d = 0; d < hd; d += 4) {
                    float kv[4];
                    Vec4<TC>::load(k + d, kv);
                    dot = fmaf(q_s[d], kv[0], dot);
                    dot = fmaf(q_s[d + 1], kv[1], dot);
                    dot = fmaf(q_s[d + 2], kv[2], dot);
                    dot = fmaf(q_s[d + 3], kv[3], dot);
                }
            } else {
                for (int d = 0; d < hd; ++d) dot = fmaf(q_s[d], to_f32(k[d]), dot);
            }
            s = dot * scale;
            if (sc.softcap > 0.f) s = sc.softcap * tanhf(s / sc.softcap);
            if (sc.slopes != nullptr) s -= sc.slopes[h] * (float)(pos - j);
        }
        const float chunk_max = block_max(s, scratch);
        const float m_new = fmaxf(m, chunk_max);
        if (m_new == -INFINITY) continue;  // every key of the chunk was refused: nothing to add (uniform over the block)
        const float p = valid ? expf(s - m_new) : 0.f;
        const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
        p_s[tid] = p;
        row_s[tid] = row;
        const float chunk_sum = block_sum(p, scratch);  // its barriers also publish p_s and row_s
        l = l * alpha + chunk_sum;
        m = m_new;
        const int first = (c < kept_chunks ? 0 : max(lo, c * CHUNK) - c * CHUNK), last = min(pos, c * CHUNK + CHUNK - 1) - c * CHUNK;
        const int gap_first = c < kept_chunks ? kept - c * CHUNK : CHUNK, gap_end = c < kept_chunks ? lo - c * CHUNK : 0;   // [gap_first, gap_end): unseen keys inside the chunk
#pragma unroll
        for (int r = 0; r < ACC; ++r) {
            const int d = tid + r * CHUNK;
            if (d < hd) {
                float a = acc[r] * alpha;
                for (int jj = first; jj <= last; ++jj) {
                    if (jj >= gap_first && jj < gap_end) continue;
                    a = fmaf(p_s[jj], to_f32(pages[row_s[jj] + v_offset + d]), a);
                }
                acc[r] = a;
            }
        }
        __syncthreads();  // p_s and row_s are rewritten by the next chunk
    }
    if (sink) l += m == -INFINITY ? 1.f : expf(-m);      // the key of score 0 without a value
    if (sc.sinks != nullptr) l += m == -INFINITY ? 1.f : expf(sc.sinks[h] - m);      // (too large for 32-bit: the result is 0, as it should be)
    const float os = sc.out_scale != nullptr ? sc.out_scale[(size_t)t * nh + h] : 1.f;
    TA* o_row = out + ((size_t)t * nh + h) * hd;
#pragma unroll
    for (int r = 0; r < ACC; ++r) {
        const int d = tid + r * CHUNK;
        if (d < hd) o_row[d] = from_f32<TA>(l > 0.f ? acc[r] / l * os : 0.f);
    }
}

// q: [T, ...] rows of q_row_stride elements whose first nh*hd elements are the query heads;
// out: [T, nh*hd]; pages: one cache [num_pages][planes][nkv][page_size][hd] of cache_dtype.
extern "C" int spy_attention_generic(const void* q, long long q_row_stride, void* out, int act_dtype, const void* pages, int cache_dtype,
                                     const int* block_table, int table_width, int page_size, int num_pages, int nh, int nkv, int hd,
                                     const int* positions, const int* seq_of_token, int tokens, int window, float scale, int* status,
                                     cudaStream_t stream, int planes, int keep_first, int sink, float softcap, const float* slopes, const float* sinks,
                                     const float* out_scale)
{
    if (softcap < 0.f) SPY_FAIL("attention: a cap of %g on the scores", softcap);
    const SpyScores scores = {softcap, slopes, sinks, out_scale};
    if (keep_first < 0 || (keep_first > 0 && window <= 0)) SPY_FAIL("attention: kept first keys (%d) go with a window", keep_first);
    if (tokens <= 0) return 0;
    if (nh <= 0 || nkv <= 0 || nh % nkv != 0) SPY_FAIL("attention: %d query heads do not group over %d key/value heads", nh, nkv);
    if (hd <= 0 || hd > ACC * CHUNK) SPY_FAIL("attention: head_dim %d must be positive and at most %d", hd, ACC * CHUNK);
    if (planes != 1 && planes != 2) SPY_FAIL("attention: a cache of %d planes (1: keys that are the values too, 2: keys and values)", planes);
    if (page_size <= 0 || num_pages <= 0 || table_width <= 0) SPY_FAIL("attention: page_size, num_pages and table_width must be positive");
    if (nh > 65535) SPY_FAIL("attention: %d heads exceed the grid limit", nh);
    const size_t smem = (size_t)(hd + (hd & 1) + CHUNK + 33) * sizeof(float) + (size_t)CHUNK * sizeof(long long);
    dim3 grid(tokens, nh);
    SPY_DISPATCH_DTYPE(act_dtype, TA, {
        SPY_DISPATCH_DTYPE(cache_dtype, TC, {
            spy_launch(attention_generic_kernel<TA, TC>, grid, dim3(CHUNK), smem, stream,
                (const TA*)q, q_row_stride, (TA*)out, (const TC*)pages, block_table, table_width, page_size, num_pages, nh, nkv, hd,
                positions, seq_of_token, window, scale, status, planes, keep_first, sink, scores);
        })
    })
    SPY_CHECK_LAUNCH("attention_generic");
    return 0;
}
