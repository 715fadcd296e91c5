// Attention whose queries, keys and values go through a short causal convolution over time: from the rows of a fused projection
// to queries and cache rows in one pass.
//
//   y_t[c] = sum_j kernel[j, c] * u_(t - taps + 1 + j)[c]     on every channel c of q | k | v (zeros before a sequence's start)
//
// u is the projection (possibly a stack of split-K partial sums, added in order).  Queries are multiplied by a factor of their
// position p, 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1) (temp_every 0: none), and go to q_out [T, heads, hd]; keys and
// values go through the block table into pages of rows hd >= max(dim, vdim); what lies beyond a row's content is zero.  One more
// group of columns, a gate a head, becomes gate_out[t, h] = sigmoid(u[gate_col + h]) (gate_out null: none).
//
// The `taps - 1` projected values ahead of a step's run of tokens lie in state[slot] (float32 [taps - 1, channels], oldest first,
// zero for a new request) and the run's last ones go there.  Grid: x = request x piece of `PIECE` tokens, y = elements of a token's
// rows; a thread owns V neighbouring channels of one piece and walks its tokens with the last inputs in registers.  Only the thread
// of a run's first piece reads and writes the state of its (request, channels), so no thread reads what another writes.  All
// arithmetic in 32-bit.
#include "common.cuh"

SPY_MODULE(spy_conv_qkv)

// tokens a thread walks: at least taps - 1, so that only a run's first piece needs the state
constexpr int piece_of(int max_taps) { return max_taps <= 4 ? 8 : 16; }

template <int V, typename T>
__device__ __forceinline__ void take(const T* p, float (&v)[V])
{
    if constexpr (V == 1) v[0] = to_f32(*p);
    else if constexpr (sizeof(T) == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    } else {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x), b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    }
}
template <int V, typename T>
__device__ __forceinline__ void put(T* p, const float (&v)[V])
{
    if constexpr (V == 1) *p = from_f32<T>(v[0]);
    else if constexpr (sizeof(T) == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x;
        x.x = *reinterpret_cast<uint32_t*>(&a);
        x.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = x;
    }
}

struct ConvArgs {
    long long ld, split_stride;
    int splits;
    const float* kernel;           // [taps, channels]
    float* state;                  // [slots, taps - 1, channels]
    const int* q_start;
    const int* state_slot;
    const int* positions;
    const int* block_table;
    int table_width, page_size, num_pages, heads, kv_heads, dim, vdim, hd, taps, pieces;
    float temp_coef, temp_every;
    int gate_col;
    float* gate_out;
    int* status;
};

// V neighbouring columns of a projection row, its parts summed
template <int V, typename TP>
__device__ __forceinline__ void columns(const TP* __restrict__ row, int splits, long long split_stride, float (&v)[V])
{
    take<V>(row, v);
    float p[V];
#pragma unroll 4
    for (int s = 1; s < splits; ++s) {
        take<V>(row + s * split_stride, p);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] += p[e];
    }
}

template <typename TP, typename TQ, int V, int MAXT>
__global__ void __launch_bounds__(128)
conv_qkv_kernel(const TP* __restrict__ proj, TQ* __restrict__ q_out, TQ* __restrict__ pages, ConvArgs A)
{
    constexpr int PIECE = piece_of(MAXT);
    __shared__ float temp_s[PIECE];          // what a token's queries are multiplied by
    __shared__ long long page_s[PIECE];      // its place in the pages: page * 2 * kv_heads * page_size + slot, or below zero
    pdl_enter();
    const int seq = blockIdx.x / A.pieces, piece = blockIdx.x % A.pieces;
    const int start = A.q_start[seq], end = A.q_start[seq + 1];
    const int t0 = start + piece * PIECE, t1 = min(end, t0 + PIECE);
    if (t0 >= end) return;
    if (threadIdx.x < PIECE && t0 + (int)threadIdx.x < t1) {
        const int t = t0 + threadIdx.x, pos = A.positions[t];
        const int lp = pos >= 0 ? pos / A.page_size : -1;
        const int page = (lp >= 0 && lp < A.table_width) ? A.block_table[(long long)seq * A.table_width + lp] : -1;
        const bool ok = page >= 0 && page < A.num_pages;
        if (!ok && blockIdx.y == 0) report_status(A.status, SPY_STATUS_BAD_PAGE, t);
        page_s[threadIdx.x] = ok ? (long long)page * 2 * A.kv_heads * A.page_size + (pos - lp * A.page_size) : -1;
        temp_s[threadIdx.x] = A.temp_every > 0.f ? 1.0f + A.temp_coef * logf(floorf((float)(pos + 1) / A.temp_every) + 1.0f) : 1.0f;
    }
    __syncthreads();
    const int per_head = A.hd / V, rows = A.heads + 2 * A.kv_heads;
    int item = blockIdx.y * blockDim.x + threadIdx.x;
    if (item >= rows * per_head) {
        item -= rows * per_head;
        if (A.gate_out == nullptr || item >= A.heads) return;
        for (int t = t0; t < t1; ++t) {
            float g[1];
            columns<1>(proj + (long long)t * A.ld + A.gate_col + item, A.splits, A.split_stride, g);
            A.gate_out[(long long)t * A.heads + item] = 1.0f / (1.0f + expf(-g[0]));
        }
        return;
    }
    const int r = item / per_head, e0 = (item - r * per_head) * V;
    const int kind = r < A.heads ? 0 : (r < A.heads + A.kv_heads ? 1 : 2);          // query, key, value
    const int head = kind == 0 ? r : (kind == 1 ? r - A.heads : r - A.heads - A.kv_heads);
    const int width = kind == 2 ? A.vdim : A.dim;
    const int channels = A.heads * A.dim + A.kv_heads * (A.dim + A.vdim);
    const int c = (kind == 0 ? 0 : (kind == 1 ? A.heads * A.dim : (A.heads + A.kv_heads) * A.dim)) + head * width + e0;
    const int hist_n = A.taps - 1, pad = MAXT - A.taps;          // fewer taps than MAXT: the oldest ones weigh nothing
    const long long row_at = (long long)(kind == 2 ? A.kv_heads + head : head) * A.page_size;      // a key or value head's rows within a page
    auto place = [&](int t) -> TQ* {
        if (kind == 0) return q_out + ((long long)t * A.heads + head) * A.hd + e0;
        return page_s[t - t0] >= 0 ? pages + (page_s[t - t0] + row_at) * A.hd + e0 : nullptr;
    };
    if (e0 >= width) {                                            // behind a row's content
        const float zero[V] = {};
        for (int t = t0; t < t1; ++t)
            if (TQ* dst = place(t)) put<V>(dst, zero);
        return;
    }
    // buf: the MAXT - 1 inputs ahead of a group of AHEAD tokens, and theirs; all of a group's loads are under way together
    constexpr int AHEAD = MAXT <= 4 ? PIECE : 4, HIST = MAXT - 1;
    float k[MAXT][V], buf[HIST + AHEAD][V];
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
#pragma unroll
        for (int e = 0; e < V; ++e) k[j][e] = 0.f;
        if (j >= pad) take<V>(A.kernel + (long long)(j - pad) * channels + c, k[j]);
    }
    const TP* in = proj + c;
    float* st = piece == 0 && hist_n > 0 ? A.state + (long long)A.state_slot[seq] * hist_n * channels + c : nullptr;
#pragma unroll
    for (int i = 0; i < HIST; ++i) {
#pragma unroll
        for (int e = 0; e < V; ++e) buf[i][e] = 0.f;
        if (i >= pad) {
            if (piece == 0) take<V>(st + (long long)(i - pad) * channels, buf[i]);
            else columns<V>(in + (long long)(t0 - HIST + i) * A.ld, A.splits, A.split_stride, buf[i]);
        }
    }
    for (int tb = t0; tb < t1; tb += AHEAD) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (tb + u < t1) columns<V>(in + (long long)(tb + u) * A.ld, A.splits, A.split_stride, buf[HIST + u]);
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (tb + u < t1) {
                float acc[V];
#pragma unroll
                for (int e = 0; e < V; ++e) acc[e] = k[0][e] * buf[u][e];
#pragma unroll
                for (int j = 1; j < MAXT; ++j)
#pragma unroll
                    for (int e = 0; e < V; ++e) acc[e] = fmaf(k[j][e], buf[u + j][e], acc[e]);
                if (kind == 0) {
                    const float f = temp_s[tb + u - t0];
#pragma unroll
                    for (int e = 0; e < V; ++e) acc[e] *= f;
                }
                if (TQ* dst = place(tb + u)) put<V>(dst, acc);
            }
        }
#pragma unroll
        for (int i = 0; i < HIST; ++i)
#pragma unroll
            for (int e = 0; e < V; ++e) buf[i][e] = buf[AHEAD + i][e];
    }
    if (piece == 0) {
        // what the next step will find: the inputs at the run's last taps - 1 places, older ones moved up from the old state
        const int n = end - start;
        for (int i = 0; i < hist_n; ++i) {
            const int t = end - hist_n + i;
            float v[V];
            if (t >= start) columns<V>(in + (long long)t * A.ld, A.splits, A.split_stride, v);
            else take<V>(st + (long long)(i + n) * channels, v);
            put<V>(st + (long long)i * channels, v);
        }
    }
}

// proj [splits][T, ld]: q (heads x dim), k (kv_heads x dim) and v (kv_heads x vdim) from column 0 on; kernel [taps, channels] float32;
// q_out [T, heads * hd]; pages [num_pages][2][kv_heads][page_size][hd] of the queries' type.  `longest`: no request brings more tokens.
extern "C" int spy_conv_qkv_store(const void* proj, int proj_dtype, long long ld, int splits, long long split_stride, const float* kernel, int taps,
                                  float* state, const int* q_start, const int* state_slot, int seqs, int longest, float temp_coef, float temp_every,
                                  int gate_col, float* gate_out, const int* positions, void* q_out, int q_dtype,
                                  const int* block_table, int table_width, void* pages, int page_size, int num_pages, int heads, int kv_heads, int dim,
                                  int vdim, int hd, int* status, cudaStream_t stream)
{
    if (seqs <= 0 || longest <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || hd < dim || hd < vdim || splits < 1)
        SPY_FAIL("conv_qkv: %d heads, %d key/value heads, dim %d, vdim %d do not fit rows of %d", heads, kv_heads, dim, vdim, hd);
    if (taps < 1 || taps > 16 || kernel == nullptr || (taps > 1 && state == nullptr)) SPY_FAIL("conv_qkv: %d taps (1 to 16; more than one need a state)", taps);
    if (page_size <= 0 || num_pages <= 0 || table_width <= 0 || block_table == nullptr || pages == nullptr)
        SPY_FAIL("conv_qkv: page_size, num_pages and table_width must be positive");
    if (temp_every < 0.f) SPY_FAIL("conv_qkv: a query temperature every %g positions", temp_every);
    const int piece = taps <= 4 ? piece_of(4) : piece_of(16), pieces = (longest + piece - 1) / piece;
    const ConvArgs A = {ld, split_stride, splits, kernel, state, q_start, state_slot, positions, block_table, table_width, page_size, num_pages,
                        heads, kv_heads, dim, vdim, hd, taps, pieces, temp_coef, temp_every, gate_col, gate_out, status};
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = taps <= 4 && dim % 4 == 0 && vdim % 4 == 0 && hd % 4 == 0 && ld % 4 == 0 && split_stride % 4 == 0 && aligned(proj) && aligned(kernel) && aligned(state)
                     && aligned(q_out) && aligned(pages);
    const long long items = (long long)(heads + 2 * kv_heads) * hd / (vec ? 4 : 1) + (gate_out != nullptr ? heads : 0), blocks = (long long)seqs * pieces;
    if ((items + 127) / 128 > 65535 || blocks > 0x7fffffffLL) SPY_FAIL("conv_qkv: %lld elements a token, %d requests of up to %d tokens exceed the grid", items, seqs, longest);
    const dim3 grid((unsigned)blocks, (unsigned)((items + 127) / 128));
    SPY_DISPATCH_DTYPE(proj_dtype, TP, {
        SPY_DISPATCH_DTYPE(q_dtype, TQ, {
            auto run = [&](auto f) { spy_launch(f, grid, dim3(128), 0, stream, (const TP*)proj, (TQ*)q_out, (TQ*)pages, A); };
            if (vec) run(conv_qkv_kernel<TP, TQ, 4, 4>);
            else if (taps <= 4) run(conv_qkv_kernel<TP, TQ, 1, 4>);
            else run(conv_qkv_kernel<TP, TQ, 1, 16>);
        })
    })
    SPY_CHECK_LAUNCH("conv_qkv");
    return 0;
}
