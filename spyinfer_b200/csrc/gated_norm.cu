// What follows a recurrence: norms with a gate.
//   gated_head_norm: each head's output divided by its root mean square, times a weight, times a gate (sigmoid or SiLU);
//   gate_group_norm: the gate (SiLU) first, then a norm in equal parts of the row, times a weight.
// The gate's pre-activation is columns of a 32-bit projection.  All arithmetic in 32-bit.
#include "common.cuh"

SPY_MODULE(spy_gated_norm)

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }

// Unit root mean square per head, a weight, a gate.
// One warp a (token, head) row, eight rows a block: the row's sum of squares is a sum inside the warp.
template <typename TO> __device__ __forceinline__ void store4(TO* p, const float (&v)[4])
{
    if constexpr (sizeof(TO) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
        uint2 x;
        x.x = *reinterpret_cast<uint32_t*>(&a);
        x.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = x;
    }
}

// VEC: head sizes, pitch and columns are multiples of four; a row of up to 512 elements stays in registers between the two passes
template <typename TO, bool VEC>
__global__ void gated_head_norm_kernel(const float* __restrict__ o, const float* __restrict__ proj, long long ld, int off_g, const float* __restrict__ weight,
                                       TO* __restrict__ out, long long rows, int H, int dv, float eps, int gate_act)
{
    pdl_enter();
    const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (row >= rows) return;
    const int lane = threadIdx.x & 31;
    const long long t = row / H;
    const int h = (int)(row - t * H);
    const float* src = o + row * dv;
    float ss = 0.f;
    const float* g = proj + t * ld + off_g + h * dv;
    if constexpr (VEC) {
        float4 v[4], gv[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * lane + 128 * i;
            v[i] = c < dv ? *reinterpret_cast<const float4*>(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            gv[i] = c < dv ? *reinterpret_cast<const float4*>(g + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        ss = warp_sum(ss);
        const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
        auto gated = [&](float x, float w, float z) {
            const float s = sigmoidf_(z);
            return x * inv * w * (gate_act == 1 ? z * s : s);
        };
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = 4 * lane + 128 * i;
            if (c >= dv) break;
            const float4 w = *reinterpret_cast<const float4*>(weight + h * dv + c);
            const float o4[4] = {gated(v[i].x, w.x, gv[i].x), gated(v[i].y, w.y, gv[i].y), gated(v[i].z, w.z, gv[i].z), gated(v[i].w, w.w, gv[i].w)};
            store4<TO>(out + row * dv + c, o4);
        }
        return;
    }
    for (int c = lane; c < dv; c += 32) ss += src[c] * src[c];
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int c = lane; c < dv; c += 32) {
        const float gate = gate_act == 1 ? g[c] * sigmoidf_(g[c]) : sigmoidf_(g[c]);
        out[row * dv + c] = from_f32<TO>(((src[c] * inv) * weight[h * dv + c]) * gate);
    }
}

extern "C" int spy_gated_head_norm(const float* o, const float* proj, long long ld, int off_g, const float* weight, void* out, int out_dtype, int tokens,
                                   int H, int dv, float eps, cudaStream_t stream, int gate_act)
{
    if (gate_act != 0 && gate_act != 1) SPY_FAIL("gated_head_norm: gate activation %d (0: sigmoid, 1: SiLU)", gate_act);
    if (tokens <= 0) return 0;
    if (H <= 0 || dv <= 0) SPY_FAIL("gated_head_norm: %d heads of %d", H, dv);
    const bool vec = dv % 4 == 0 && dv <= 512 && ld % 4 == 0 && off_g % 4 == 0
                     && ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
    const long long rows = (long long)tokens * H, blocks = (rows + 7) / 8;
    if (blocks > 0x7fffffffLL) SPY_FAIL("gated_head_norm: %lld rows exceed the grid limit", rows);
    SPY_DISPATCH_DTYPE(out_dtype, TO, {
        auto kernel = vec ? gated_head_norm_kernel<TO, true> : gated_head_norm_kernel<TO, false>;
        spy_launch(kernel, dim3((unsigned)blocks), dim3(256), 0, stream, o, proj, ld, off_g, weight, (TO*)out, rows, H, dv, eps, gate_act);
    })
    SPY_CHECK_LAUNCH("gated_head_norm");
    return 0;
}

// The gate ahead of the norm: y = o * silu(gate), cut into `groups` equal parts a row, each divided by its own root mean square, times a
// weight.  One block a (token, part); the products stay in shared memory between the two passes.
template <typename TO, int V>
__global__ void __launch_bounds__(256)
gate_group_norm_kernel(const float* __restrict__ o, const float* __restrict__ proj, long long ld, int off_g, const float* __restrict__ weight,
                       TO* __restrict__ out, int size, int groups, float eps)
{
    extern __shared__ __align__(16) float y_s[];
    __shared__ float scratch[33];
    pdl_enter();
    const long long t = blockIdx.x;
    const int part = size / groups, c0 = blockIdx.y * part;
    const float* src = o + t * size + c0;
    const float* g = proj + t * ld + off_g + c0;
    float ss = 0.f;
    for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
        float a[V], b[V];
        if (V == 4) {
            *reinterpret_cast<float4*>(a) = *reinterpret_cast<const float4*>(src + c);
            *reinterpret_cast<float4*>(b) = *reinterpret_cast<const float4*>(g + c);
        } else {
            a[0] = src[c];
            b[0] = g[c];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float y = a[e] * (b[e] * sigmoidf_(b[e]));
            y_s[c + e] = y;
            ss = fmaf(y, y, ss);
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)part + eps);
    for (int c = threadIdx.x * V; c < part; c += blockDim.x * V) {
#pragma unroll
        for (int e = 0; e < V; ++e) out[t * size + c0 + c + e] = from_f32<TO>(y_s[c + e] * inv * weight[c0 + c + e]);
    }
}

extern "C" int spy_gate_group_norm(const float* o, const float* proj, long long ld, int off_g, const float* weight, void* out, int out_dtype, int tokens,
                                   int size, int groups, float eps, cudaStream_t stream)
{
    if (tokens <= 0) return 0;
    if (size <= 0 || groups <= 0 || size % groups != 0 || groups > 65535) SPY_FAIL("gate_group_norm: rows of %d in %d parts", size, groups);
    const int part = size / groups;
    const size_t smem = (size_t)part * sizeof(float);
    if (smem > 200 * 1024) SPY_FAIL("gate_group_norm: a part of %d elements does not fit a block's shared memory", part);
    const bool vec = part % 4 == 0 && ld % 4 == 0 && off_g % 4 == 0 && ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(proj)) & 15) == 0;
    const int per = part / (vec ? 4 : 1);
    const int threads = per >= 256 ? 256 : per >= 128 ? 128 : per >= 64 ? 64 : 32;
    SPY_DISPATCH_DTYPE(out_dtype, TO, {
        auto kernel = vec ? gate_group_norm_kernel<TO, 4> : gate_group_norm_kernel<TO, 1>;
        if (smem > 48 * 1024) SPY_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        spy_launch(kernel, dim3(tokens, groups), dim3(threads), smem, stream, o, proj, ld, off_g, weight, (TO*)out, size, groups, eps);
    })
    SPY_CHECK_LAUNCH("gate_group_norm");
    return 0;
}
