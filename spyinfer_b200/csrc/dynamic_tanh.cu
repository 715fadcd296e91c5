// Dynamic Tanh, a norm without statistics: dyt(x) = tanh(alpha * x) * w + b, element by element with one alpha for the tensor and a
// weight and a bias along the row, around the 32-bit residual stream.  One launch does, per element, either or both of
//   1. hidden += y_scale * dyt_y(y)      (y: a sublayer's output, possibly a stack of split-K partial sums added in order)
//   2. out = dyt(hidden)                  (what the next sublayer reads, or the rows the head reads)
// in 32-bit.  With `rows` the listed rows are gathered, put into out[0 .. n) and nothing is written back.  Nothing is shared
// between elements, so a thread takes V of them with all its loads under way together, and a row is spread over as many blocks
// as it has pieces of THREADS * V elements.
#include "common.cuh"

SPY_MODULE(spy_dynamic_tanh)

constexpr int THREADS = 128;

template <typename T, int V> struct Run;
template <typename T> struct Run<T, 1> {
    static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32(p[0]); }
    static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { p[0] = from_f32<T>(v[0]); }
};
template <> struct Run<float, 4> {
    static __device__ __forceinline__ void load(const float* p, float (&v)[4])
    {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
    static __device__ __forceinline__ void store(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <> struct Run<bf16, 4> {
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

// the four tensors of one dyt: alpha is read from the device
struct Tanh {
    const float* alpha;
    const void* w;
    const void* b;
};

// ROWS rows a block (1; 4 when there are many): a thread's weights are loaded once for all of them, and their inputs are under way together.
template <typename TY, typename TW, typename TO, int V, int ROWS>
__global__ void __launch_bounds__(THREADS)
dynamic_tanh_kernel(float* __restrict__ hidden, const TY* __restrict__ y, int splits, long long split_stride, Tanh ty, float y_scale,
                    const int* __restrict__ rows, Tanh tx, TO* __restrict__ out, int n, int len, int write_back)
{
    pdl_launch_dependents();
    const int i = (blockIdx.y * THREADS + threadIdx.x) * V;
    float wy[V], by[V], wx[V], bx[V];
    float ay = 0.f, ax = 0.f;
    if (i < len) {                                   // weights: no kernel of a step writes them
        if (y != nullptr) {
            ay = *ty.alpha;
            Run<TW, V>::load((const TW*)ty.w + i, wy);
            Run<TW, V>::load((const TW*)ty.b + i, by);
        }
        if (out != nullptr) {
            ax = *tx.alpha;
            Run<TW, V>::load((const TW*)tx.w + i, wx);
            Run<TW, V>::load((const TW*)tx.b + i, bx);
        }
    }
    pdl_wait();
    if (i >= len) return;
    const int r0 = blockIdx.x * ROWS, live = min(ROWS, n - r0);
    long long at[ROWS];
    float h[ROWS][V], v[ROWS][V];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        if (j >= live) break;
        at[j] = (long long)(rows != nullptr ? rows[r0 + j] : r0 + j) * len + i;
        Run<float, V>::load(hidden + at[j], h[j]);
        if (y != nullptr) Run<TY, V>::load(y + at[j], v[j]);
    }
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        if (j >= live) break;
        if (y != nullptr) {
            float p[V];
#pragma unroll 4
            for (int s = 1; s < splits; ++s) {
                Run<TY, V>::load(y + s * split_stride + at[j], p);
#pragma unroll
                for (int e = 0; e < V; ++e) v[j][e] += p[e];
            }
#pragma unroll
            for (int e = 0; e < V; ++e) h[j][e] += y_scale * fmaf(tanhf(ay * v[j][e]), wy[e], by[e]);
            if (write_back) Run<float, V>::store(hidden + at[j], h[j]);
        }
        if (out == nullptr) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) h[j][e] = fmaf(tanhf(ax * h[j][e]), wx[e], bx[e]);
        Run<TO, V>::store(out + (long long)(r0 + j) * len + i, h[j]);
    }
}

// hidden [*, len] float32.  y (optional): [splits][rows][len] of y_dtype with its alpha, weight, bias and scale.  alpha/weight/
// bias/out (optional): dyt of the (new) stream rows into out [n, len] of out_dtype.  Weights and biases have weight_dtype, the
// alphas are float32 numbers on the device.
extern "C" int spy_dynamic_tanh(float* hidden, const void* y, int y_dtype, int splits, long long split_stride, const float* y_alpha, const void* y_weight,
                                const void* y_bias, float y_scale, const int* rows, const float* alpha, const void* weight, const void* bias,
                                int weight_dtype, void* out, int out_dtype, int n, int len, int write_back, cudaStream_t stream)
{
    if (n <= 0) return 0;
    if (len <= 0) SPY_FAIL("dynamic_tanh: rows of %d elements", len);
    if (y == nullptr && out == nullptr) return 0;
    if (y != nullptr && (y_alpha == nullptr || y_weight == nullptr || y_bias == nullptr || splits < 1))
        SPY_FAIL("dynamic_tanh: a sublayer output needs its alpha, weight, bias and at least one part");
    if (out != nullptr && (alpha == nullptr || weight == nullptr || bias == nullptr)) SPY_FAIL("dynamic_tanh: the norm of the stream needs its alpha, weight and bias");
    if (y == nullptr) y_dtype = SPY_F32;
    if (out == nullptr) out_dtype = SPY_F32;
    auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool vec = len % 4 == 0 && split_stride % 4 == 0 && aligned(hidden) && aligned(y) && aligned(y_weight) && aligned(y_bias) && aligned(weight)
                     && aligned(bias) && aligned(out);
    const int per_block = THREADS * (vec ? 4 : 1), pieces = (len + per_block - 1) / per_block;
    if (pieces > 65535) SPY_FAIL("dynamic_tanh: rows of %d elements exceed the grid", len);
    const Tanh ty = {y_alpha, y_weight, y_bias}, tx = {alpha, weight, bias};
    SPY_DISPATCH_DTYPE(y_dtype, TY, {
        SPY_DISPATCH_DTYPE(weight_dtype, TW, {
            SPY_DISPATCH_DTYPE(out_dtype, TO, {
                const bool many = n >= 512;
                auto kernel = vec ? (many ? dynamic_tanh_kernel<TY, TW, TO, 4, 4> : dynamic_tanh_kernel<TY, TW, TO, 4, 1>)
                                  : (many ? dynamic_tanh_kernel<TY, TW, TO, 1, 4> : dynamic_tanh_kernel<TY, TW, TO, 1, 1>);
                spy_launch(kernel, dim3(many ? (n + 3) / 4 : n, pieces), dim3(THREADS), 0, stream, hidden, (const TY*)y, splits, split_stride, ty, y_scale, rows,
                           tx, (TO*)out, n, len, write_back);
            })
        })
    })
    SPY_CHECK_LAUNCH("dynamic_tanh");
    return 0;
}
