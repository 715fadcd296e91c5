// The residual sum of a block whose norm sits on the sublayer's OUTPUT:  h += rms_norm(y) * w,  h the 32-bit residual stream.
//   v   = y[row], itself possibly a sum of split-K partial products            32-bit sums
//   h[row] += v * (1 / sqrt(mean(v^2) + eps)) * w                              32-bit statistics; w as stored or as (offset + w)
//   copy[row] = h[row] in the activations' type                                what the next sublayer's products read (optional)
// With y absent the kernel only makes the copy (the embedding's rows for the first sublayer).
// One block a row.  Rows of up to 16 K elements (a multiple of 4) stay in registers; other rows wait in shared memory
// between the two passes.
#include "common.cuh"

SPY_MODULE(spy_residual_norm)

template <typename TY, typename TW, typename TC>
__global__ void __launch_bounds__(256) residual_norm_kernel(float* __restrict__ h, const TY* __restrict__ y, int splits, long long split_stride,
                                                            const TW* __restrict__ w, float w_offset, TC* __restrict__ copy, int len, float eps)
{
    extern __shared__ float row_buf[];   // len floats, then 33 of scratch
    pdl_enter();
    float* scratch = row_buf + len;
    const size_t base = (size_t)blockIdx.x * len;
    if (y != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < len; i += blockDim.x) {
            float v = 0.f;
            for (int s = 0; s < splits; ++s) v += to_f32(y[(size_t)s * split_stride + base + i]);   // the parts in their order
            row_buf[i] = v;
            ss = fmaf(v, v, ss);
        }
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)len + eps);
        for (int i = threadIdx.x; i < len; i += blockDim.x) {
            const float r = h[base + i] + (row_buf[i] * inv) * (w_offset + to_f32(w[i]));
            h[base + i] = r;
            if (copy != nullptr) copy[base + i] = from_f32<TC>(r);
        }
    } else if (copy != nullptr) {
        for (int i = threadIdx.x; i < len; i += blockDim.x) copy[base + i] = from_f32<TC>(h[base + i]);
    }
}

template <typename T> struct Quad;
template <> struct Quad<float> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4])
    {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Quad<bf16> {
    static __device__ __forceinline__ void load(const bf16* p, float (&v)[4])
    {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x), b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
        v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
    }
    static __device__ __forceinline__ void store(bf16* p, const float (&v)[4])
    {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x;
        x.x = *reinterpret_cast<uint32_t*>(&a);
        x.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = x;
    }
};

// Rows whose length is a multiple of 4 and at most 16 K stay in registers: a thread owns NQ quads of the row (quad
// tid + j * blockDim.x), the weight's quads are loaded before the wait for the kernels ahead, the stream's and every
// part's loads are under way together, and the sums over the parts keep their order.
template <typename TY, typename TW, typename TC, int NQ, int MAXT>
__global__ void __launch_bounds__(MAXT) residual_norm_row_kernel(float* __restrict__ h, const TY* __restrict__ y, int splits, long long split_stride,
                                                                 const TW* __restrict__ w, float w_offset, TC* __restrict__ copy, int len, float eps)
{
    __shared__ float scratch[33];
    pdl_launch_dependents();
    float wv[NQ][4];
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
        const int i = 4 * ((int)threadIdx.x + j * (int)blockDim.x);
        if (i < len) Quad<TW>::load(w + i, wv[j]);
    }
    pdl_wait();
    const size_t base = (size_t)blockIdx.x * len;
    float hv[NQ][4], v[NQ][4];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
        const int i = 4 * ((int)threadIdx.x + j * (int)blockDim.x);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[j][e] = 0.f;
        if (i < len) {
            Quad<float>::load(h + base + i, hv[j]);
            for (int s0 = 0; s0 < splits; s0 += 4) {
                float d[4][4];
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (s0 + k < splits) Quad<TY>::load(y + (size_t)(s0 + k) * split_stride + base + i, d[k]);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    if (s0 + k < splits) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) v[j][e] += d[k][e];
                    }
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) ss = fmaf(v[j][e], v[j][e], ss);
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)len + eps);
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
        const int i = 4 * ((int)threadIdx.x + j * (int)blockDim.x);
        if (i < len) {
            float r[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) r[e] = hv[j][e] + (v[j][e] * inv) * (w_offset + wv[j][e]);
            Quad<float>::store(h + base + i, r);
            if (copy != nullptr) Quad<TC>::store(copy + base + i, r);
        }
    }
}

// h [rows, len] float32; y [rows, len] or a stack [splits, rows, len] (y_dtype), or null; w [len] (w_dtype); copy [rows, len] (copy_dtype) or null.
extern "C" int spy_residual_norm(float* h, const void* y, int y_dtype, int splits, long long split_stride, const void* w, int w_dtype, float w_offset,
                                 void* copy, int copy_dtype, int rows, int len, float eps, cudaStream_t stream)
{
    if (rows <= 0) return 0;
    if (len <= 0) SPY_FAIL("residual_norm: row length %d must be positive", len);
    if (y != nullptr && (splits <= 0 || w == nullptr)) SPY_FAIL("residual_norm: a result to add needs its parts' count and the norm's weight");
    const size_t smem = (size_t)(len + 33) * sizeof(float);
    if (smem > 200 * 1024) SPY_FAIL("residual_norm: a row of %d does not fit a block's shared memory", len);
    if (y == nullptr) { y_dtype = SPY_F32; w_dtype = SPY_F32; }
    const bool aligned = (reinterpret_cast<uintptr_t>(h) & 15) == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0 &&
                         (reinterpret_cast<uintptr_t>(copy) & 15) == 0 && (split_stride & 3) == 0;
    if (y != nullptr && len % 4 == 0 && len <= 16384 && aligned) {
        const int quads = len / 4;
        int nq = rows >= 4 * spy_sm_count() ? 4 : 1;            // many rows: fewer, fatter threads; few rows (decoding): the whole block on one row
        while (quads > nq * 1024) nq *= 2;
        int threads = ((quads + nq - 1) / nq + 31) / 32 * 32;
        SPY_DISPATCH_DTYPE(y_dtype, TY, {
            SPY_DISPATCH_DTYPE(w_dtype, TW, {
                SPY_DISPATCH_DTYPE(copy_dtype, TC, {
                    if (nq == 1) spy_launch(residual_norm_row_kernel<TY, TW, TC, 1, 1024>, dim3(rows), dim3(threads), 0, stream, h, (const TY*)y, splits, split_stride, (const TW*)w, w_offset, (TC*)copy, len, eps);
                    else if (nq == 2) spy_launch(residual_norm_row_kernel<TY, TW, TC, 2, 1024>, dim3(rows), dim3(threads), 0, stream, h, (const TY*)y, splits, split_stride, (const TW*)w, w_offset, (TC*)copy, len, eps);
                    else if (threads <= 256) spy_launch(residual_norm_row_kernel<TY, TW, TC, 4, 256>, dim3(rows), dim3(threads), 0, stream, h, (const TY*)y, splits, split_stride, (const TW*)w, w_offset, (TC*)copy, len, eps);
                    else spy_launch(residual_norm_row_kernel<TY, TW, TC, 4, 1024>, dim3(rows), dim3(threads), 0, stream, h, (const TY*)y, splits, split_stride, (const TW*)w, w_offset, (TC*)copy, len, eps);
                })
            })
        })
        SPY_CHECK_LAUNCH("residual_norm");
        return 0;
    }
    SPY_DISPATCH_DTYPE(y_dtype, TY, {
        SPY_DISPATCH_DTYPE(w_dtype, TW, {
            SPY_DISPATCH_DTYPE(copy_dtype, TC, {
                auto kernel = residual_norm_kernel<TY, TW, TC>;
                if (smem > 48 * 1024) SPY_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
                spy_launch(kernel, dim3(rows), dim3(256), smem, stream, h, (const TY*)y, splits, split_stride, (const TW*)w, w_offset, (TC*)copy, len, eps);
            })
        })
    })
    SPY_CHECK_LAUNCH("residual_norm");
    return 0;
}

// out = a_scale * rms_norm(a) * a_weight + b_scale * rms_norm(b) * b_weight, row by row: two sublayer outputs side by side, each normed over
// the whole row (each possibly a stack of split-K partial sums).  One block a row; both rows stay in shared memory between the passes.
template <typename T, int V> __device__ __forceinline__ void load_run(const T* p, float (&v)[V])
{
    if constexpr (V == 1) {
        v[0] = to_f32(p[0]);
    } else if constexpr (sizeof(T) == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    } else {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 c = *reinterpret_cast<const __nv_bfloat162*>(&x.x), d = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
        v[0] = __low2float(c); v[1] = __high2float(c); v[2] = __low2float(d); v[3] = __high2float(d);
    }
}

// V = 4: runs of four where rows, parts and tensors allow them
template <typename TA, typename TB, int V>
__global__ void normed_sum_kernel(float* __restrict__ out, const TA* __restrict__ a, int a_splits, long long a_stride, const float* __restrict__ a_weight,
                                  float a_scale, const TB* __restrict__ b, int b_splits, long long b_stride, const float* __restrict__ b_weight, float b_scale,
                                  int len, float eps)
{
    extern __shared__ __align__(16) float rows_s[];
    __shared__ float scratch[33];
    pdl_enter();
    const long long at = (long long)blockIdx.x * len;
    float *ra = rows_s, *rb = rows_s + (len + 3) / 4 * 4;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x * V; i < len; i += blockDim.x * V) {
        float va[V], vb[V], p[V];
        load_run<TA, V>(a + at + i, va);
        load_run<TB, V>(b + at + i, vb);
#pragma unroll 4
        for (int s = 1; s < a_splits; ++s) {
            load_run<TA, V>(a + s * a_stride + at + i, p);
#pragma unroll
            for (int e = 0; e < V; ++e) va[e] += p[e];
        }
#pragma unroll 4
        for (int s = 1; s < b_splits; ++s) {
            load_run<TB, V>(b + s * b_stride + at + i, p);
#pragma unroll
            for (int e = 0; e < V; ++e) vb[e] += p[e];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            ra[i + e] = va[e];
            rb[i + e] = vb[e];
            sa = fmaf(va[e], va[e], sa);
            sb = fmaf(vb[e], vb[e], sb);
        }
    }
    sa = block_sum(sa, scratch);
    sb = block_sum(sb, scratch);
    const float ia = a_scale / sqrtf(sa / (float)len + eps), ib = b_scale / sqrtf(sb / (float)len + eps);
    for (int i = threadIdx.x * V; i < len; i += blockDim.x * V) {
        float wa[V], wb[V], o[V];
        load_run<float, V>(a_weight + i, wa);
        load_run<float, V>(b_weight + i, wb);
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = ra[i + e] * ia * wa[e] + rb[i + e] * ib * wb[e];
        if constexpr (V == 4) *reinterpret_cast<float4*>(out + at + i) = make_float4(o[0], o[1], o[2], o[3]);
        else out[at + i] = o[0];
    }
}

extern "C" int spy_normed_sum(float* out, const void* a, int a_dtype, int a_splits, long long a_stride, const float* a_weight, float a_scale, const void* b,
                              int b_dtype, int b_splits, long long b_stride, const float* b_weight, float b_scale, int rows, int len, float eps,
                              cudaStream_t stream)
{
    if (rows <= 0) return 0;
    if (len <= 0 || a_splits < 1 || b_splits < 1) SPY_FAIL("normed_sum: rows of %d elements, %d and %d parts", len, a_splits, b_splits);
    const size_t smem = 2 * (((size_t)len + 3) / 4 * 4) * sizeof(float);
    if (smem > 220 * 1024) SPY_FAIL("normed_sum: two rows of %d elements do not fit a block's shared memory", len);
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = len % 4 == 0 && a_stride % 4 == 0 && b_stride % 4 == 0 && aligned(out) && aligned(a) && aligned(b) && aligned(a_weight) && aligned(b_weight);
    const int per = vec ? len / 4 : len, threads = per >= 512 ? 256 : 128;
    SPY_DISPATCH_DTYPE(a_dtype, TA, {
        SPY_DISPATCH_DTYPE(b_dtype, TB, {
            auto kernel = vec ? normed_sum_kernel<TA, TB, 4> : normed_sum_kernel<TA, TB, 1>;
            if (smem > 48 * 1024) SPY_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            spy_launch(kernel, dim3(rows), dim3(threads), smem, stream, out, (const TA*)a, a_splits, a_stride, a_weight, a_scale, (const TB*)b, b_splits,
                       b_stride, b_weight, b_scale, len, eps);
        })
    })
    SPY_CHECK_LAUNCH("normed_sum");
    return 0;
}

template <int V, typename T>
__device__ __forceinline__ void sum_load(const T* p, float (&v)[V])
{
    if constexpr (V == 4) Quad<T>::load(p, v);
    else v[0] = to_f32(*p);
}
template <int V, typename T>
__device__ __forceinline__ void sum_store(T* p, const float (&v)[V])
{
    if constexpr (V == 4) Quad<T>::store(p, v);
    else *p = from_f32<T>(v[0]);
}

// hidden += a (+ b), each a result [rows, len] or a stack of split-K partial sums, and (optionally) the sum's copy in the type the
// next product reads: what a block does whose two sublayers read one norm.  V elements a thread.
template <typename TA, typename TB, typename TC, int V>
__global__ void __launch_bounds__(256)
stream_sum_kernel(float* __restrict__ hidden, const TA* __restrict__ a, int a_splits, long long a_stride, const TB* __restrict__ b, int b_splits,
                  long long b_stride, TC* __restrict__ copy, long long n)
{
    pdl_enter();
    const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    float h[V];
    sum_load<V>(hidden + i, h);
    float t[V], u[V];
    sum_load<V>(a + i, t);
#pragma unroll 4
    for (int s = 1; s < a_splits; ++s) {
        sum_load<V>(a + s * a_stride + i, u);
#pragma unroll
        for (int e = 0; e < V; ++e) t[e] += u[e];
    }
    if (b != nullptr) {
        float w[V];
        sum_load<V>(b + i, w);
#pragma unroll 4
        for (int s = 1; s < b_splits; ++s) {
            sum_load<V>(b + s * b_stride + i, u);
#pragma unroll
            for (int e = 0; e < V; ++e) w[e] += u[e];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) t[e] += w[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) h[e] += t[e];
    sum_store<V>(hidden + i, h);
    if (copy != nullptr) sum_store<V>(copy + i, h);
}

extern "C" int spy_stream_sum(float* hidden, const void* a, int a_dtype, int a_splits, long long a_stride, const void* b, int b_dtype, int b_splits,
                              long long b_stride, void* copy, int copy_dtype, long long n, cudaStream_t stream)
{
    if (n <= 0) return 0;
    if (hidden == nullptr || a == nullptr || a_splits < 1 || (b != nullptr && b_splits < 1)) SPY_FAIL("stream_sum: a stream and a result are needed");
    if (b == nullptr) b_dtype = SPY_F32;
    if (copy == nullptr) copy_dtype = SPY_BF16;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = n % 4 == 0 && a_stride % 4 == 0 && b_stride % 4 == 0 && aligned(hidden) && aligned(a) && aligned(b) && aligned(copy);
    const long long blocks = (n / (vec ? 4 : 1) + 255) / 256;
    if (blocks > 0x7fffffffLL) SPY_FAIL("stream_sum: %lld elements exceed the grid", n);
    SPY_DISPATCH_DTYPE(a_dtype, TA, {
        SPY_DISPATCH_DTYPE(b_dtype, TB, {
            SPY_DISPATCH_DTYPE(copy_dtype, TC, {
                if (vec)
                    spy_launch(stream_sum_kernel<TA, TB, TC, 4>, dim3((unsigned)blocks), dim3(256), 0, stream, hidden, (const TA*)a, a_splits, a_stride, (const TB*)b,
                               b_splits, b_stride, (TC*)copy, n);
                else
                    spy_launch(stream_sum_kernel<TA, TB, TC, 1>, dim3((unsigned)blocks), dim3(256), 0, stream, hidden, (const TA*)a, a_splits, a_stride, (const TB*)b,
                               b_splits, b_stride, (TC*)copy, n);
            })
        })
    })
    SPY_CHECK_LAUNCH("stream_sum");
    return 0;
}
