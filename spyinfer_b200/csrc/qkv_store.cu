// The steps around the attention kernels for attention without norms on queries and keys.
//
// qkv_store: from the rows of a fused projection (q | k | v at given columns; possibly a stack of split-K partial sums, added in
//   order) to queries and cache rows: an optional bias, rotation of the first 2 * rot_half elements of every query and key head by a
//   (cos, sin) table (pairs (2i, 2i + 1) or (i, i + rot_half)), queries to q_out [T, heads, hd], keys and values through the block
//   table into pages of rows hd >= max(dim, vdim).  What lies beyond a row's content is zero.
// gate_heads: out[t, h, e] = attn[t, h, e] * sigmoid(gate[t, col + h * vdim + e]) for e < vdim, from rows of hd to rows of vdim; the
//   gate is a part of the same projection (possibly a stack).
// All arithmetic in 32-bit.
#include "common.cuh"

SPY_MODULE(spy_qkv_store)

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
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16* p, const float (&v)[4])
{
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 x;
    x.x = *reinterpret_cast<uint32_t*>(&a);
    x.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = x;
}

// four (or one) neighbouring columns of a projection row, its parts summed, the bias added
template <typename TP>
__device__ __forceinline__ void columns4(const TP* __restrict__ row, int splits, long long split_stride, const float* __restrict__ bias, int col, float (&v)[4])
{
    load4(row + col, v);
    float p[4];
#pragma unroll 4
    for (int s = 1; s < splits; ++s) {
        load4(row + s * split_stride + col, p);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] += p[e];
    }
    if (bias != nullptr) {
        load4(bias + col, p);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] += p[e];
    }
}
template <typename TP>
__device__ __forceinline__ float column(const TP* __restrict__ row, int splits, long long split_stride, const float* __restrict__ bias, int col)
{
    float v = to_f32(row[col]);
    for (int s = 1; s < splits; ++s) v += to_f32(row[s * split_stride + col]);
    return bias != nullptr ? v + bias[col] : v;
}

struct StoreArgs {
    long long ld, split_stride;
    int splits, q_col, k_col, v_col;
    const float* bias;
    const float* rope;
    int rot_half, table_rows, half_pairs;
    const int* positions;
    const int* seq_of_token;
    const int* block_table;
    int table_width, page_size, num_pages, heads, kv_heads, dim, vdim, hd;
    int* status;
};

// Grid: x = token, y = piece of the token's rows.  VEC: sizes, columns and pitches are multiples of four, the pairs are neighbours
// (or nothing is rotated) and rot_half is even: a thread takes four neighbouring elements of a row of hd.  Else one element a thread.
template <typename TP, typename TQ, bool VEC>
__global__ void __launch_bounds__(128)
qkv_store_kernel(const TP* __restrict__ proj, TQ* __restrict__ q_out, TQ* __restrict__ pages, StoreArgs A)
{
    pdl_enter();
    const int t = blockIdx.x;
    const int pos = A.positions[t];
    const bool pos_ok = A.rot_half == 0 || (pos >= 0 && pos < A.table_rows);
    if (!pos_ok && threadIdx.x == 0 && blockIdx.y == 0) report_status(A.status, SPY_STATUS_BAD_POSITION, t);
    const int lp = pos >= 0 ? pos / A.page_size : -1;
    const int page = (lp >= 0 && lp < A.table_width) ? A.block_table[(long long)A.seq_of_token[t] * A.table_width + lp] : -1;
    const bool page_ok = page >= 0 && page < A.num_pages;
    if (!page_ok && threadIdx.x == 0 && blockIdx.y == 0) report_status(A.status, SPY_STATUS_BAD_PAGE, t);
    const int slot = page_ok ? pos % A.page_size : 0;
    const TP* row = proj + (long long)t * A.ld;
    const int V = VEC ? 4 : 1, per_head = A.hd / V, rows = A.heads + 2 * A.kv_heads;
    const int item = blockIdx.y * blockDim.x + threadIdx.x;
    if (item >= rows * per_head) return;
    const int r = item / per_head, e0 = (item - r * per_head) * V;
    const int kind = r < A.heads ? 0 : (r < A.heads + A.kv_heads ? 1 : 2);          // query, key, value
    const int head = kind == 0 ? r : (kind == 1 ? r - A.heads : r - A.heads - A.kv_heads);
    const int width = kind == 2 ? A.vdim : A.dim;
    const int col = (kind == 0 ? A.q_col : (kind == 1 ? A.k_col : A.v_col)) + head * width;
    TQ* dst;
    if (kind == 0) dst = q_out + ((long long)t * A.heads + head) * A.hd + e0;
    else if (page_ok) dst = pages + ((((long long)page * 2 + (kind - 1)) * A.kv_heads + head) * A.page_size + slot) * A.hd + e0;
    else return;
    if constexpr (VEC) {
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if (e0 < width) {
            columns4(row, A.splits, A.split_stride, A.bias, col + e0, o);
            const int p = e0 / 2;
            if (kind != 2 && p < A.rot_half && pos_ok) {
                float cs[4];
                load4(A.rope + ((long long)pos * A.rot_half + p) * 2, cs);
                const float a0 = o[0] * cs[0] - o[1] * cs[1], b0 = o[1] * cs[0] + o[0] * cs[1];
                const float a1 = o[2] * cs[2] - o[3] * cs[3], b1 = o[3] * cs[2] + o[2] * cs[3];
                o[0] = a0; o[1] = b0; o[2] = a1; o[3] = b1;
            }
        }
        store4(dst, o);
    } else {
        float o = 0.f;
        if (e0 < width) {
            o = column(row, A.splits, A.split_stride, A.bias, col + e0);
            if (kind != 2 && e0 < 2 * A.rot_half && pos_ok) {
                const int p = A.half_pairs ? e0 % A.rot_half : e0 / 2;
                const bool second = A.half_pairs ? e0 >= A.rot_half : (e0 & 1);
                const int other = A.half_pairs ? (second ? e0 - A.rot_half : e0 + A.rot_half) : e0 ^ 1;
                const float x = column(row, A.splits, A.split_stride, A.bias, col + other);
                const float c = A.rope[((long long)pos * A.rot_half + p) * 2], s = A.rope[((long long)pos * A.rot_half + p) * 2 + 1];
                o = second ? o * c + x * s : o * c - x * s;
            }
        }
        dst[0] = from_f32<TQ>(o);
    }
}

// proj [splits][T, ld]; bias [ld] float32 or null; rope [table_rows, rot_half, 2] float32 (null with rot_half 0); q_out [T, heads * hd];
// pages [num_pages][2][kv_heads][page_size][hd] of the queries' type.
extern "C" int spy_qkv_store(const void* proj, int proj_dtype, long long ld, int splits, long long split_stride, int q_col, int k_col, int v_col,
                             const float* bias, const float* rope, int rot_half, int table_rows, int half_pairs, const int* positions,
                             const int* seq_of_token, void* q_out, int q_dtype, const int* block_table, int table_width, void* pages, int page_size,
                             int num_pages, int tokens, int heads, int kv_heads, int dim, int vdim, int hd, int* status, cudaStream_t stream)
{
    if (tokens <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || hd < dim || hd < vdim || splits < 1)
        SPY_FAIL("qkv_store: %d heads, %d key/value heads, dim %d, vdim %d do not fit rows of %d", heads, kv_heads, dim, vdim, hd);
    if (rot_half < 0 || 2 * rot_half > dim || (rot_half > 0 && rope == nullptr)) SPY_FAIL("qkv_store: %d rotated pairs do not fit a head of %d elements", rot_half, dim);
    if (page_size <= 0 || num_pages <= 0 || table_width <= 0 || block_table == nullptr || pages == nullptr)
        SPY_FAIL("qkv_store: page_size, num_pages and table_width must be positive");
    const StoreArgs A = {ld, split_stride, splits, q_col, k_col, v_col, bias, rope, rot_half, table_rows, half_pairs, positions, seq_of_token,
                         block_table, table_width, page_size, num_pages, heads, kv_heads, dim, vdim, hd, status};
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = dim % 4 == 0 && vdim % 4 == 0 && hd % 4 == 0 && q_col % 4 == 0 && k_col % 4 == 0 && v_col % 4 == 0 && ld % 4 == 0
                     && split_stride % 4 == 0 && rot_half % 2 == 0 && (rot_half == 0 || !half_pairs) && aligned(proj) && aligned(bias) && aligned(q_out)
                     && aligned(pages) && aligned(rope);
    const long long items = (long long)(heads + 2 * kv_heads) * hd / (vec ? 4 : 1);
    const int threads = 128;
    if ((items + threads - 1) / threads > 65535) SPY_FAIL("qkv_store: %lld elements a token exceed the grid", items);
    const dim3 grid(tokens, (unsigned)((items + threads - 1) / threads));
    SPY_DISPATCH_DTYPE(proj_dtype, TP, {
        SPY_DISPATCH_DTYPE(q_dtype, TQ, {
            if (vec) spy_launch(qkv_store_kernel<TP, TQ, true>, grid, dim3(threads), 0, stream, (const TP*)proj, (TQ*)q_out, (TQ*)pages, A);
            else spy_launch(qkv_store_kernel<TP, TQ, false>, grid, dim3(threads), 0, stream, (const TP*)proj, (TQ*)q_out, (TQ*)pages, A);
        })
    })
    SPY_CHECK_LAUNCH("qkv_store");
    return 0;
}

template <typename TA, typename TG, bool VEC>
__global__ void __launch_bounds__(128)
gate_heads_kernel(const TA* __restrict__ attn, int hd, const TG* __restrict__ gate, long long gate_ld, int splits, long long split_stride, int gate_col,
                  TA* __restrict__ out, int heads, int vdim)
{
    pdl_enter();
    const int V = VEC ? 4 : 1;
    const int t = blockIdx.x, i = (blockIdx.y * blockDim.x + threadIdx.x) * V, n = heads * vdim;
    if (i >= n) return;
    const int h = i / vdim, e = i - h * vdim;
    const TG* g_row = gate + (long long)t * gate_ld;
    const TA* a = attn + ((long long)t * heads + h) * hd + e;
    TA* o = out + (long long)t * n + i;
    if constexpr (VEC) {
        float g[4], v[4];
        columns4(g_row, splits, split_stride, (const float*)nullptr, gate_col + i, g);
        load4(a, v);
#pragma unroll
        for (int k = 0; k < 4; ++k) v[k] = v[k] / (1.0f + expf(-g[k]));
        store4(o, v);
    } else {
        const float g = column(g_row, splits, split_stride, (const float*)nullptr, gate_col + i);
        o[0] = from_f32<TA>(to_f32(a[0]) / (1.0f + expf(-g)));
    }
}

// attn [T, heads * hd] (the first vdim elements of each head's row are read), gate [splits][T, gate_ld] from column gate_col, out [T, heads * vdim].
extern "C" int spy_gate_heads(const void* attn, int act_dtype, int hd, const void* gate, int gate_dtype, long long gate_ld, int splits, long long split_stride,
                              int gate_col, void* out, int tokens, int heads, int vdim, cudaStream_t stream)
{
    if (tokens <= 0) return 0;
    if (heads <= 0 || vdim <= 0 || hd < vdim || splits < 1) SPY_FAIL("gate_heads: %d heads of %d values do not fit rows of %d", heads, vdim, hd);
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = vdim % 4 == 0 && hd % 4 == 0 && gate_ld % 4 == 0 && gate_col % 4 == 0 && split_stride % 4 == 0 && aligned(attn) && aligned(gate) && aligned(out);
    const long long items = (long long)heads * vdim / (vec ? 4 : 1);
    if ((items + 127) / 128 > 65535) SPY_FAIL("gate_heads: %lld elements a token exceed the grid", items);
    const dim3 grid(tokens, (unsigned)((items + 127) / 128));
    SPY_DISPATCH_DTYPE(act_dtype, TA, {
        SPY_DISPATCH_DTYPE(gate_dtype, TG, {
            if (vec)
                spy_launch(gate_heads_kernel<TA, TG, true>, grid, dim3(128), 0, stream, (const TA*)attn, hd, (const TG*)gate, gate_ld, splits, split_stride,
                           gate_col, (TA*)out, heads, vdim);
            else
                spy_launch(gate_heads_kernel<TA, TG, false>, grid, dim3(128), 0, stream, (const TA*)attn, hd, (const TG*)gate, gate_ld, splits, split_stride,
                           gate_col, (TA*)out, heads, vdim);
        })
    })
    SPY_CHECK_LAUNCH("gate_heads");
    return 0;
}
