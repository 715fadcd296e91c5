// Linear recurrences over a matrix state [dk, dv] per (request, head) with ONE decay a head and token, carried from token to token in
// 32-bit, q and k shared by groups of heads:
//   * the gated delta rule:        S = g S,  u = beta (v - S^T k),  S = S + k u^T,  o = S^T q,
//                                  g = exp(-exp(A_log) softplus(za + dt_bias)), beta = sigmoid(zb), q and k unit vectors made here
//                                  (x / sqrt(sum x^2 + 1e-6), q also times q_scale);
//   * the state-space dual scan:   S = exp(-exp(A_log) dt) S + dt k v^T,  o = S^T q + D v,  dt = softplus(zd + dt_bias)
//                                  (k and q are its B and C).
//
// Steps with prompt portions (head_scan_kernel): a block owns a tile of value columns of one (request, head) and keeps its part of S in
// registers for the whole run.  Tokens are taken U = 8 at a time.  With S0 the state ahead of the eight, D(t, s) the product of the
// decays of s + 1 .. t and g_t that of 0 .. t:
//     x_t = S0^T k_t,   y_t = S0^T q_t                                       (all eight against the same state: one pass, no chain)
//     w_t = beta_t (v_t - g_t x_t - sum_{s<t} D(t,s) (k_t . k_s) w_s)        (delta rule; else w_t = dt_t v_t)
//     o_t = g_t y_t + sum_{s<=t} D(t,s) (q_t . k_s) w_s                      (+ D v_t)
//     S  <- g_7 S0 + sum_s D(7,s) k_s w_s^T
// which is the token-by-token walk with its sums in another order.  Only products of decays occur, no quotients.  A column's own chain
// of eight is walked by the lanes that hold it.  So a token costs three multiply-adds an element of the state (two without the delta
// rule; packed two to an instruction), the lanes' sums over the rows run for eight tokens together, and nothing waits for one token.
// The coefficients (dot products among the eight tokens' keys and queries, their decays) are the same for every column of a head:
// a kernel ahead (head_table_kernel) makes them once, a warp for every eight tokens of a key head.
//
// Steps in which every request brings one token (head_decode_kernel): a block takes whole rows of a state (contiguous memory), asks for
// all of its part before it waits for the kernels ahead in the stream, and holds it in registers between reading and writing.
//
// q, k and v are columns of one 32-bit matrix `proj` [T, ld], the gates' pre-activations of another, `gates` [T, gates_ld].
#include "common.cuh"

SPY_MODULE(spy_head_scan)

constexpr int U = 8;              // tokens taken together
constexpr int WARPS = 4;          // of a block of the kernel for portions
constexpr int THREADS = 32 * WARPS;
// groups of eight in shared memory (keys of KS elements): one that is walked, the others on their way
__host__ __device__ constexpr int ring_of(int KS) { return KS > 512 ? 2 : 4; }
constexpr int TABLE = 64 + 64 + 5 * U;   // floats of a group's coefficients: among the tokens (removal, read-out), then per token

struct HeadScanArgs {
    const float* proj;
    long long ld;
    int off_q, off_k, off_v;
    const float* gates;
    long long gates_ld;
    int off_rate, off_decay;      // columns of the rate's (delta rule) and the decay's or step's pre-activations, one a head
    const float *a_log, *dt_bias, *d_skip;
    float* state;                 // [slots, H, dk, dv]
    int num_slots;
    const int* q_start;           // [S + 1]
    const int* state_slot;        // [S]
    float* out;                   // [T, H * dv]
    int H, share, dk, dv;
    float q_scale;
    int* status;
    float* tables;                // [T / U + S][H][TABLE]: the coefficients of every eight tokens (steps with portions)
};

// where a request's groups of eight tokens lie among the tables
__device__ __forceinline__ int first_group(int q_start, int seq) { return q_start / U + seq; }

__device__ __forceinline__ float sigmoidf_(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplusf_(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ void cp_async16(float* smem_dst, const float* src)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(float* smem_dst, const float* src)
{
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// two 32-bit floats side by side: one instruction for both
typedef unsigned long long f2;
__device__ __forceinline__ f2 pair2(float a, float b)
{
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void split2(f2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c)
{
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b)
{
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}

// v[0 .. 2M) of every lane -> v[0 .. M): lanes whose `bit` of `off` is 0 keep the first half, the others the second, each summed with
// the partner's half
template <int M> __device__ __forceinline__ void halve(float* v, int off, bool upper)
{
#pragma unroll
    for (int i = 0; i < M; ++i) {
        const float keep = upper ? v[i + M] : v[i], send = upper ? v[i] : v[i + M];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
    }
}
// 32 values a lane, summed over the warp: lane l ends with the sum of the values numbered l
__device__ __forceinline__ float transpose_sum32(float (&v)[32], int lane)
{
    halve<16>(v, 16, lane & 16);
    halve<8>(v, 8, lane & 8);
    halve<4>(v, 4, lane & 4);
    halve<2>(v, 2, lane & 2);
    halve<1>(v, 1, lane & 1);
    return v[0];
}

// The coefficients of eight tokens, by one warp for all heads that share the keys:
//   table[t * 8 + s]        delta rule: beta_t D(t,s) (k_t . k_s) for s < t, else 0
//   table[64 + t * 8 + s]   D(t,s) (q_t . k_s) (times dt_s without the delta rule) for s <= t, else 0
//   table[128 + i * 8 + t]  0: beta_t  1: beta_t g_t on x_t  2: g_t on y_t  3: D(7,t) on k_t's update (times dt_t without the delta rule)
//                           4 (t = 0): g_7
// with the unit vectors' factors folded in.  Tokens behind a run's end keep everything and add nothing.
constexpr int TABLE_WARPS = 4;
template <bool DELTA, int V>
__global__ void __launch_bounds__(32 * TABLE_WARPS) head_table_kernel(HeadScanArgs A, int num_seqs, int num_groups)
{
    __shared__ float raw_all[TABLE_WARPS][96];
    pdl_enter();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, hk = blockIdx.y;
    const int gi = blockIdx.x * TABLE_WARPS + warp;
    if (gi >= num_groups) return;
    // the request whose groups hold number gi: the last one that starts at or before it
    int lo = 0, hi = num_seqs - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) / 2;
        if (first_group(A.q_start[mid], mid) <= gi) lo = mid;
        else hi = mid - 1;
    }
    const int start = A.q_start[lo], t0 = start + (gi - first_group(start, lo)) * U, n_tok = min(U, A.q_start[lo + 1] - t0);
    if (n_tok <= 0) return;
    float* raw = raw_all[warp];
    const int dk = A.dk;
    float dots[64], diag[32];
#pragma unroll
    for (int i = 0; i < 64; ++i) dots[i] = 0.f;
#pragma unroll
    for (int i = 0; i < 32; ++i) diag[i] = 0.f;
    for (int e = lane * V; e < dk; e += 32 * V) {
        float k[U][V], q[U][V];
#pragma unroll
        for (int t = 0; t < U; ++t) {
            const float* row = A.proj + (size_t)(t0 + t) * A.ld + hk * dk + e;
#pragma unroll
            for (int j = 0; j < V; ++j) k[t][j] = q[t][j] = 0.f;
            if (t < n_tok) {
                if (V == 4) {
                    *reinterpret_cast<float4*>(k[t]) = *reinterpret_cast<const float4*>(row + A.off_k);
                    *reinterpret_cast<float4*>(q[t]) = *reinterpret_cast<const float4*>(row + A.off_q);
                } else {
                    k[t][0] = row[A.off_k];
                    q[t][0] = row[A.off_q];
                }
            }
        }
#pragma unroll
        for (int t = 0; t < U; ++t)
#pragma unroll
            for (int j = 0; j < V; ++j) {
#pragma unroll
                for (int s = 0; s <= t; ++s) {
                    // row t, column s: k_t . k_s;  row s, column t: q_t . k_s (s < t);  q_t . k_t apart
                    if (DELTA) dots[t * 8 + s] = fmaf(k[t][j], k[s][j], dots[t * 8 + s]);
                    float& d = s < t ? dots[s * 8 + t] : diag[t];
                    d = fmaf(q[t][j], k[s][j], d);
                }
                if (DELTA) diag[8 + t] = fmaf(q[t][j], q[t][j], diag[8 + t]);
            }
    }
    float half[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) half[i] = dots[i];
    raw[lane] = transpose_sum32(half, lane);
#pragma unroll
    for (int i = 0; i < 32; ++i) half[i] = dots[32 + i];
    raw[32 + lane] = transpose_sum32(half, lane);
    raw[64 + lane] = transpose_sum32(diag, lane);
    __syncwarp();
    // the unit vectors' factors: lane t the key's, lane 8 + t the query's
    float unit = 1.f;
    if (DELTA && lane < 16) unit = (lane < 8 ? 1.0f : A.q_scale) / sqrtf(raw[lane < 8 ? 9 * lane : 64 + lane] + 1e-6f);
    const float unit_q = __shfl_sync(0xffffffffu, unit, 8 + (lane & 7));
    float rk[2], rq[2];                              // this lane's two entries (t = lane / 8 + 4 j, s = lane % 8): k_t . k_s and q_t . k_s of unit vectors
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int t = (lane >> 3) + 4 * j, s = lane & 7;
        const float ik_s = __shfl_sync(0xffffffffu, unit, s), ik_t = __shfl_sync(0xffffffffu, unit, t), iq_t = __shfl_sync(0xffffffffu, unit, 8 + t);
        rk[j] = DELTA && s < t ? raw[t * 8 + s] * (ik_t * ik_s) : 0.f;
        rq[j] = s < t ? raw[s * 8 + t] : s == t ? raw[64 + t] : 0.f;
        if (DELTA) rq[j] *= iq_t * ik_s;
    }
    for (int h = hk * A.share; h < (hk + 1) * A.share; ++h) {
        float keep = 1.f, add = 0.f;                 // of token lane % 8
        if ((lane & 7) < n_tok) {
            const float* row = A.gates + (size_t)(t0 + (lane & 7)) * A.gates_ld + h;
            const float dt = softplusf_(row[A.off_decay] + A.dt_bias[h]);
            keep = expf(-expf(A.a_log[h]) * dt);
            add = DELTA ? sigmoidf_(row[A.off_rate]) : dt;
        }
        float kp[U];
#pragma unroll
        for (int i = 0; i < U; ++i) kp[i] = __shfl_sync(0xffffffffu, keep, i);
        auto decay = [&](int t, int s) {             // product over s + 1 .. t
            float d = 1.f;
#pragma unroll
            for (int i = 0; i < U; ++i)
                if (i > s && i <= t) d *= kp[i];
            return d;
        };
        float* table = A.tables + ((size_t)gi * A.H + h) * TABLE;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = (lane >> 3) + 4 * j, s = lane & 7;
            const float d = s <= t ? decay(t, s) : 0.f;
            const float add_t = __shfl_sync(0xffffffffu, add, t), add_s = add;
            if (DELTA) table[t * 8 + s] = add_t * d * rk[j];
            table[64 + t * 8 + s] = DELTA ? d * rq[j] : d * rq[j] * add_s;
        }
        if (lane < U) {
            const float g = decay(lane, -1), rest = decay(U - 1, lane);
            if (DELTA) {
                table[128 + lane] = add;
                table[136 + lane] = add * g * unit;
            }
            table[144 + lane] = DELTA ? g * unit_q : g;
            table[152 + lane] = DELTA ? rest * unit : rest * add;
            if (lane == U - 1) table[160] = g;
        }
    }
}

// A thread's rows: quads qd * 4 RG + 4 rg .. + 3 (qd < NR / 4) of RG * NR >= dk; its columns: NC neighbours.  RG row groups share a
// warp's lanes (rg = lane / CG), so a warp owns (32 / RG) * NC columns and a block four times that.
template <bool DELTA, int RG, int NR, int NC>
__global__ void __launch_bounds__(THREADS, 2) head_scan_kernel(HeadScanArgs A)
{
    constexpr int NQ = NR / 4, KS = RG * NR, CG = 32 / RG, WC = CG * NC, CTB = WARPS * WC, NREP = RG / NC;
    static_assert(RG >= NC && NC >= 2, "the columns of a thread are dealt out over its row groups");
    extern __shared__ __align__(16) float sm[];
    // in plain stream order (spy_launch_in_order): it runs long on about a block an SM
    pdl_wait();
    constexpr int RING = ring_of(KS), STAGE = U * (2 * KS + CTB) + TABLE;            // floats of a group: keys, queries, values, coefficients
    float* w_s = sm + RING * STAGE;                          // [WARPS][U][WC]

    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CTB, hk = h / A.share;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dk = A.dk, dv = A.dv;
    const int t_begin = A.q_start[seq], t_end = A.q_start[seq + 1];
    if (t_begin >= t_end) return;
    const int slot = A.state_slot[seq];
    if (slot < 0 || slot >= A.num_slots) {
        if (tid == 0) report_status(A.status, SPY_STATUS_BAD_PAGE, t_begin);
        return;
    }
    const float* my_tables = A.tables + ((size_t)first_group(t_begin, seq) * A.H + h) * TABLE;
    const bool aligned = (dk & 3) == 0 && (A.ld & 3) == 0 && ((A.off_k | A.off_q) & 3) == 0 && (reinterpret_cast<uintptr_t>(A.proj) & 15) == 0;
    const bool v_aligned = (dv & 3) == 0 && (A.ld & 3) == 0 && (A.off_v & 3) == 0 && (reinterpret_cast<uintptr_t>(A.proj) & 15) == 0;
    const int n_groups = (t_end - t_begin + U - 1) / U;
    // Requests a group's rows (a warp a token) and coefficients: a few copies a warp and group, so that the walk's own traffic with shared
    // memory never waits behind many of them.  Zeros behind a row's end and the run's.
    auto request = [&](int g) {
        if (g < n_groups) {
            const int t0 = t_begin + g * U, n_tok = min(U, t_end - t0);
            float* k_s = sm + (g % RING) * STAGE;
            float* q_s = k_s + U * KS;
            float* v_s = q_s + U * KS;
#pragma unroll
            for (int tt = warp; tt < U; tt += WARPS) {
                const float* row = A.proj + (size_t)(t0 + tt) * A.ld;
                const bool in = tt < n_tok;
                const float *ks = row + A.off_k + hk * dk, *qs = row + A.off_q + hk * dk, *vs = row + A.off_v + h * dv + c0;
                if (aligned) {
#pragma unroll
                    for (int e = 4 * lane; e < KS; e += 128) {
                        if (in && e < dk) {
                            cp_async16(k_s + tt * KS + e, ks + e);
                            cp_async16(q_s + tt * KS + e, qs + e);
                        } else {
                            *reinterpret_cast<float4*>(k_s + tt * KS + e) = make_float4(0.f, 0.f, 0.f, 0.f);
                            *reinterpret_cast<float4*>(q_s + tt * KS + e) = make_float4(0.f, 0.f, 0.f, 0.f);
                        }
                    }
                } else {
                    for (int e = lane; e < KS; e += 32) {
                        if (in && e < dk) {
                            cp_async4(k_s + tt * KS + e, ks + e);
                            cp_async4(q_s + tt * KS + e, qs + e);
                        } else {
                            k_s[tt * KS + e] = q_s[tt * KS + e] = 0.f;
                        }
                    }
                }
                if (v_aligned) {
                    for (int c = 4 * lane; c < CTB; c += 128) {
                        if (in && c0 + c < dv) cp_async16(v_s + tt * CTB + c, vs + c);
                        else *reinterpret_cast<float4*>(v_s + tt * CTB + c) = make_float4(0.f, 0.f, 0.f, 0.f);
                    }
                } else {
                    for (int c = lane; c < CTB; c += 32) {
                        if (in && c0 + c < dv) cp_async4(v_s + tt * CTB + c, vs + c);
                        else v_s[tt * CTB + c] = 0.f;
                    }
                }
            }
            if (warp == (g & (WARPS - 1))) {
                const float* src = my_tables + (size_t)g * A.H * TABLE;
                for (int e = 4 * lane + (DELTA ? 0 : 64); e < TABLE; e += 128) cp_async16(v_s + U * CTB + e, src + e);
            }
        }
        cp_async_commit();                         // one group of copies a call, empty behind the last
    };
#pragma unroll
    for (int g = 0; g < RING - 1; ++g) request(g);
    const int rg = lane / CG, cg = lane % CG;
    const int col0 = c0 + warp * WC + cg * NC;                   // the thread's first column
    float* st = A.state + ((size_t)slot * A.H + h) * dk * dv;
    f2 S[NR / 2][NC];                                            // rows 2 i and 2 i + 1 of the thread's, one column
#pragma unroll
    for (int i = 0; i < NR / 2; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const int r = (i / 2) * 4 * RG + 4 * rg + 2 * (i % 2);
            const bool in = col0 + c < dv;
            S[i][c] = pair2(in && r < dk ? st[(size_t)r * dv + col0 + c] : 0.f, in && r + 1 < dk ? st[(size_t)(r + 1) * dv + col0 + c] : 0.f);
        }
    // which column of the thread's row groups this lane sums and walks, and (NREP lanes walk the same column) which copy it is
    const bool b0 = rg & 1, b1 = rg & 2;
    const int own = NC == 4 ? (b0 ? 2 : 0) + (b1 ? 1 : 0) : (b0 ? 1 : 0), rep = rg / NC;
    const int own_col = warp * WC + cg * NC + own;               // within the block's tile
    const float d_skip = DELTA ? 0.f : A.d_skip[h];
    float* wb = w_s + warp * U * WC;
    // the copies of a column share its tokens out
    const int t_own = NREP >= 8 ? (rep & 1) * 4 + (rep & 2) + ((rep & 4) >> 2) : NREP >= 4 ? (rep & 1) * 4 + (rep & 2) : NREP >= 2 ? (rep & 1) * 4 : 0;
    constexpr int N_OWN = NREP >= U ? 1 : U / NREP;
    const bool stores = c0 + own_col < dv && (NREP < 16 || rep < 8);
    for (int g = 0; g < n_groups; ++g) {
        cp_async_wait<RING - 2>();
        __syncthreads();                           // this group has landed; every warp is past the one before, whose place is free
        request(g + RING - 1);
        {
            const int t0 = t_begin + g * U, n_tok = t_end - t0;
            const float* kg = sm + (g % RING) * STAGE + 4 * rg;
            const float* qg = kg + U * KS;
            const float* vg = sm + (g % RING) * STAGE + 2 * U * KS;
            const float* tab = vg + U * CTB;
            float w[U];                            // the column's own values: what each token writes
            float x[DELTA ? NC * U : 1], y[NC * U];     // [column][token]
            constexpr int PART = NC == 4 ? 4 : U;      // tokens whose sums are under way together
#pragma unroll
            for (int u0 = 0; u0 < U; u0 += PART) {
                f2 x2[DELTA ? NC * PART : 1], y2[NC * PART];
#pragma unroll
                for (int j = 0; j < NC * PART; ++j) {
                    if (DELTA) x2[j] = 0ull;
                    y2[j] = 0ull;
                }
#pragma unroll
                for (int u = 0; u < PART; ++u)
#pragma unroll
                    for (int qd = 0; qd < NQ; ++qd) {
                        ulonglong2 kk, qq;
                        if (DELTA) kk = *reinterpret_cast<const ulonglong2*>(kg + (u0 + u) * KS + qd * 4 * RG);
                        qq = *reinterpret_cast<const ulonglong2*>(qg + (u0 + u) * KS + qd * 4 * RG);
#pragma unroll
                        for (int c = 0; c < NC; ++c) {
                            if (DELTA) x2[c * PART + u] = fma2(kk.x, S[qd * 2][c], x2[c * PART + u]);
                            y2[c * PART + u] = fma2(qq.x, S[qd * 2][c], y2[c * PART + u]);
                        }
#pragma unroll
                        for (int c = 0; c < NC; ++c) {
                            if (DELTA) x2[c * PART + u] = fma2(kk.y, S[qd * 2 + 1][c], x2[c * PART + u]);
                            y2[c * PART + u] = fma2(qq.y, S[qd * 2 + 1][c], y2[c * PART + u]);
                        }
                    }
#pragma unroll
                for (int c = 0; c < NC; ++c)
#pragma unroll
                    for (int u = 0; u < PART; ++u) {
                        float p, q;
                        if constexpr (DELTA) {
                            split2(x2[c * PART + u], p, q);
                            x[c * U + u0 + u] = p + q;
                        }
                        split2(y2[c * PART + u], p, q);
                        y[c * U + u0 + u] = p + q;
                    }
            }
            if constexpr (DELTA) halve<NC * U / 2>(x, CG, b0);
            if constexpr (DELTA && NC == 4) halve<U>(x, 2 * CG, b1);
            if constexpr (DELTA) {
#pragma unroll
                for (int o = NC * CG; o <= 16; o <<= 1)
#pragma unroll
                    for (int u = 0; u < U; ++u) x[u] += __shfl_xor_sync(0xffffffffu, x[u], o);
            }
            if constexpr (DELTA) {
#pragma unroll
                for (int t = 0; t < U; ++t) {
                    float a[U];
                    *reinterpret_cast<float4*>(a) = *reinterpret_cast<const float4*>(tab + t * 8);
                    if (t > 4) *reinterpret_cast<float4*>(a + 4) = *reinterpret_cast<const float4*>(tab + t * 8 + 4);
                    float r = fmaf(tab[128 + t], vg[t * CTB + own_col], -tab[136 + t] * x[t]);
#pragma unroll
                    for (int s = 0; s < t; ++s) r = fmaf(-a[s], w[s], r);
                    w[t] = r;
                }
                __syncwarp();                      // the group before has been read
                // the copies of a column share its tokens out
                constexpr int EACH = NREP >= U ? U : NREP;
#pragma unroll
                for (int j = 0; j < U / EACH; ++j) {
                    const int mine = rep % EACH, t = j * EACH + mine;
                    float v = w[j * EACH];
#pragma unroll
                    for (int r = 1; r < EACH; ++r) v = r == mine ? w[j * EACH + r] : v;
                    wb[t * WC + cg * NC + own] = tab[152 + t] * v;
                }
                __syncwarp();
            } else {
#pragma unroll
                for (int t = 0; t < U; ++t) w[t] = vg[t * CTB + own_col];       // the step is in the table
            }
            const f2 g_all = pair2(tab[160], tab[160]);
#pragma unroll
            for (int j = 0; j < NR / 2; ++j)
#pragma unroll
                for (int c = 0; c < NC; ++c) S[j][c] = mul2(S[j][c], g_all);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                float ww[NC];
                const float* src = DELTA ? wb + u * WC + cg * NC : vg + u * CTB + warp * WC + cg * NC;
                if (NC == 4) *reinterpret_cast<float4*>(ww) = *reinterpret_cast<const float4*>(src);
                else *reinterpret_cast<float2*>(ww) = *reinterpret_cast<const float2*>(src);
                f2 w2[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const float v = DELTA ? ww[c] : ww[c] * tab[152 + u];
                    w2[c] = pair2(v, v);
                }
#pragma unroll
                for (int qd = 0; qd < NQ; ++qd) {
                    const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(kg + u * KS + qd * 4 * RG);
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        S[qd * 2][c] = fma2(kk.x, w2[c], S[qd * 2][c]);
                        S[qd * 2 + 1][c] = fma2(kk.y, w2[c], S[qd * 2 + 1][c]);
                    }
                }
            }
            // the read-outs, which nothing of the state waits for
            halve<NC * U / 2>(y, CG, b0);
            if constexpr (NC == 4) halve<U>(y, 2 * CG, b1);
            if (NREP >= 2) halve<4>(y, NC * CG, rep & 1);
            if (NREP >= 4) halve<2>(y, 2 * NC * CG, rep & 2);
            if (NREP >= 8) halve<1>(y, 4 * NC * CG, rep & 4);
            if (NREP >= 16) y[0] += __shfl_xor_sync(0xffffffffu, y[0], 16);
#pragma unroll
            for (int j = 0; j < N_OWN; ++j) {
                const int t = t_own + j;
                float p[U];
                *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(tab + 64 + t * 8);
                *reinterpret_cast<float4*>(p + 4) = *reinterpret_cast<const float4*>(tab + 64 + t * 8 + 4);
                float o = tab[144 + t] * y[j];
#pragma unroll
                for (int s = 0; s < U; ++s) o = fmaf(p[s], w[s], o);
                if (!DELTA) o = fmaf(d_skip, vg[t * CTB + own_col], o);
                if (stores && t < n_tok) A.out[(size_t)(t0 + t) * A.H * dv + h * dv + c0 + own_col] = o;
            }
        }
    }
#pragma unroll
    for (int i = 0; i < NR / 2; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            const int r = (i / 2) * 4 * RG + 4 * rg + 2 * (i % 2);
            float p, q;
            split2(S[i][c], p, q);
            if (col0 + c < dv && r < dk) st[(size_t)r * dv + col0 + c] = p;
            if (col0 + c < dv && r + 1 < dk) st[(size_t)(r + 1) * dv + col0 + c] = q;
        }
    pdl_launch_dependents();
}

// Decoding.  A block of DT threads owns `cols` (a multiple of V) columns of one (request, head): cols / V threads across, the rest down
// the rows; thread row `down` holds the rows down, down + n_down, ...  (at most NI of them).  cols / V is a power of two, at most 32.
constexpr int DT = 256;
template <bool DELTA, int V, int NI>
__global__ void __launch_bounds__(DT, NI * V <= 32 ? 3 : NI * V <= 64 ? 2 : 1) head_decode_kernel(HeadScanArgs A, int cols)
{
    extern __shared__ __align__(16) float sm[];
    __shared__ float sums[3][DT / 32];
    pdl_launch_dependents();
    const int seq = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * cols, hk = h / A.share;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, dk = A.dk, dv = A.dv;
    // the batch's arrays and this entry's states are written by no kernel of the step: they may be read before the wait
    const int t = A.q_start[seq], n = A.q_start[seq + 1] - t, slot = A.state_slot[seq];
    const bool ok = n > 0 && slot >= 0 && slot < A.num_slots;
    const int across = cols / V, n_down = DT / across, down = tid / across, c = (tid - down * across) * V;
    const bool mine = ok && c0 + c < dv;
    float* st = A.state + ((size_t)(ok ? slot : 0) * A.H + h) * dk * dv + c0 + c;
    float S[NI][V];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int r = down + i * n_down;
#pragma unroll
        for (int e = 0; e < V; ++e) S[i][e] = 0.f;
        if (mine && r < dk) {
            if (V == 4) *reinterpret_cast<float4*>(S[i]) = *reinterpret_cast<const float4*>(st + (size_t)r * dv);
            else S[i][0] = st[(size_t)r * dv];
        }
    }
    float* k_s = sm;                               // dk
    float* q_s = k_s + dk;                         // dk
    float* red = q_s + dk + ((2 * dk) & 3 ? 4 - ((2 * dk) & 3) : 0);      // [warps][cols] (twice), on a 16-byte border
    pdl_wait();
    if (!ok) {
        if (n > 0 && tid == 0) report_status(A.status, SPY_STATUS_BAD_PAGE, t);
        return;
    }
    const float* row = A.proj + (size_t)t * A.ld;
    const float* gt = A.gates + (size_t)t * A.gates_ld + h;
    const float dt = softplusf_(gt[A.off_decay] + A.dt_bias[h]);
    const float keep = expf(-expf(A.a_log[h]) * dt), add = DELTA ? sigmoidf_(gt[A.off_rate]) : dt;
    float v[V];
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = mine ? row[A.off_v + h * dv + c0 + c + e] : 0.f;
    float kk = 0.f, qq = 0.f, qk = 0.f;
    for (int r = tid; r < dk; r += DT) {
        const float k = row[A.off_k + hk * dk + r], q = row[A.off_q + hk * dk + r];
        k_s[r] = k;
        q_s[r] = q;
        kk = fmaf(k, k, kk);
        qq = fmaf(q, q, qq);
        qk = fmaf(q, k, qk);
    }
    kk = warp_sum(kk);
    qq = warp_sum(qq);
    qk = warp_sum(qk);
    if (lane == 0) {
        sums[0][warp] = kk;
        sums[1][warp] = qq;
        sums[2][warp] = qk;
    }
    __syncthreads();
    kk = qq = qk = 0.f;
#pragma unroll
    for (int w = 0; w < DT / 32; ++w) {
        kk += sums[0][w];
        qq += sums[1][w];
        qk += sums[2][w];
    }
    const float ik = DELTA ? 1.0f / sqrtf(kk + 1e-6f) : 1.f, iq = DELTA ? A.q_scale / sqrtf(qq + 1e-6f) : 1.f;
    // x = S^T k and y = S^T q over the old state, both summed over the thread rows through shared memory; then
    // o = keep y + (q . k) w, w = beta (v - keep x) (delta rule) or dt v, and the state takes k w
    float x[V], y[V];
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = y[e] = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int r = down + i * n_down;
        if (r < dk) {
            const float k = k_s[r], q = q_s[r];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                if (DELTA) x[e] = fmaf(k, S[i][e], x[e]);
                y[e] = fmaf(q, S[i][e], y[e]);
            }
        }
    }
    float* red_y = red + (DELTA ? DT / 32 * cols : 0);
    for (int o = across; o < 32; o <<= 1) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            if (DELTA) x[e] += __shfl_xor_sync(0xffffffffu, x[e], o);
            y[e] += __shfl_xor_sync(0xffffffffu, y[e], o);
        }
    }
    if (lane < across) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            if (DELTA) red[warp * cols + c + e] = x[e];
            red_y[warp * cols + c + e] = y[e];
        }
    }
    __syncthreads();
    auto sum_warps = [&](const float* from, float (&out)[V]) {
#pragma unroll
        for (int e = 0; e < V; ++e) out[e] = 0.f;
#pragma unroll
        for (int d = 0; d < DT / 32; ++d) {
            float part[V];
            if (V == 4) *reinterpret_cast<float4*>(part) = *reinterpret_cast<const float4*>(from + d * cols + c);
            else part[0] = from[d * cols + c];
#pragma unroll
            for (int e = 0; e < V; ++e) out[e] += part[e];
        }
    };
    float w[V];
    if (DELTA) sum_warps(red, x);
#pragma unroll
    for (int e = 0; e < V; ++e) w[e] = DELTA ? add * (v[e] - keep * ik * x[e]) : add * v[e];
    if (!mine) return;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int r = down + i * n_down;
        if (r < dk) {
            const float k = k_s[r] * ik;
#pragma unroll
            for (int e = 0; e < V; ++e) S[i][e] = fmaf(k, w[e], keep * S[i][e]);
            if (V == 4) *reinterpret_cast<float4*>(st + (size_t)r * dv) = *reinterpret_cast<const float4*>(S[i]);
            else st[(size_t)r * dv] = S[i][0];
        }
    }
    if (down == 0) {
        sum_warps(red_y, y);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            float o = fmaf(keep * iq, y[e], qk * iq * ik * w[e]);
            if (!DELTA) o = fmaf(A.d_skip[h], v[e], o);
            A.out[(size_t)t * A.H * dv + h * dv + c0 + c + e] = o;
        }
    }
}

template <bool DELTA, int RG, int NR, int NC>
static int launch_portions(const HeadScanArgs& A, int num_seqs, cudaStream_t stream)
{
    constexpr int KS = RG * NR, WC = 32 / RG * NC, CTB = WARPS * WC;
    constexpr size_t smem = (ring_of(KS) * (U * (2 * (size_t)KS + CTB) + TABLE) + (size_t)WARPS * U * WC) * sizeof(float);
    static_assert(smem <= 220 * 1024, "the ring fits a block's shared memory");
    const int tiles = (A.dv + CTB - 1) / CTB;
    if (tiles > 65535) SPY_FAIL("head scan: a value size of %d exceeds the grid limit", A.dv);
    auto kernel = head_scan_kernel<DELTA, RG, NR, NC>;
    if (smem > 48 * 1024) SPY_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    spy_launch_in_order(kernel, dim3(num_seqs, A.H, tiles), dim3(THREADS), smem, stream, A);
    SPY_CHECK_LAUNCH("head scan");
    return 0;
}

template <bool DELTA, int RG, int NR>
static int launch_portions_cols(const HeadScanArgs& A, int num_seqs, cudaStream_t stream)
{
    // four columns a thread where that still gives the SMs enough blocks, else two
    static int forced = -1;                      // SPYINFER_HEAD_SCAN_COLUMNS = 2 or 4 in the environment fixes it (for measurements)
    if (forced < 0) {
        const char* e = getenv("SPYINFER_HEAD_SCAN_COLUMNS");
        forced = e != nullptr ? atoi(e) : 0;
    }
    constexpr int wide = WARPS * (32 / RG) * 4;
    const long long blocks = (long long)num_seqs * A.H * ((A.dv + wide - 1) / wide);
    const bool four = forced == 4 || (forced != 2 && 3 * blocks >= 2LL * spy_sm_count());      // measured: 128 blocks of four 441 us, 256 of two 471; 64 of four 436, 128 of two 371
    if constexpr (NR <= 16) {
        if (four) return launch_portions<DELTA, RG, NR, 4>(A, num_seqs, stream);
    }
    return launch_portions<DELTA, RG, NR, 2>(A, num_seqs, stream);
}

template <bool DELTA, int V>
static int launch_decode(const HeadScanArgs& A, int num_seqs, cudaStream_t stream)
{
    // as many columns as keep a thread's part of the state within 8 loads (at most 128 columns)
    int cols = V == 4 ? 128 : 32;
    while (cols > V && cols / 2 >= A.dv) cols /= 2;
    auto per_thread = [&](int n) { return (A.dk + DT / (n / V) - 1) / (DT / (n / V)); };
    while (cols > V && per_thread(cols) > 8) cols /= 2;
    const int ni = per_thread(cols), tiles = (A.dv + cols - 1) / cols;
    const size_t smem = (2 * (size_t)A.dk + 4 + (DELTA ? 2 : 1) * (size_t)(DT / 32) * cols) * sizeof(float);
    if (ni > 32 || tiles > 65535 || smem > 220 * 1024) SPY_FAIL("head scan: states of %d x %d are not served", A.dk, A.dv);
    void (*kernel)(HeadScanArgs, int) = ni <= 2 ? head_decode_kernel<DELTA, V, 2> : ni <= 4 ? head_decode_kernel<DELTA, V, 4> : ni <= 8 ? head_decode_kernel<DELTA, V, 8>
                                        : ni <= 16 ? head_decode_kernel<DELTA, V, 16> : head_decode_kernel<DELTA, V, 32>;
    if (smem > 48 * 1024) SPY_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    spy_launch(kernel, dim3(num_seqs, A.H, tiles), dim3(DT), smem, stream, A, cols);
    SPY_CHECK_LAUNCH("head scan (decoding)");
    return 0;
}

template <bool DELTA> static int launch_head_scan(const HeadScanArgs& A, int num_seqs, int tokens, int longest, cudaStream_t stream)
{
    if (num_seqs <= 0) return 0;
    if (A.H <= 0 || A.dk <= 0 || A.dv <= 0 || A.share <= 0 || A.H % A.share != 0)
        SPY_FAIL("head scan: %d heads sharing keys by %d, key size %d, value size %d", A.H, A.share, A.dk, A.dv);
    if (A.H > 65535) SPY_FAIL("head scan: %d heads exceed the grid limit", A.H);
    if (longest <= 1) {     // every request brings one token
        const bool vec = A.dv % 4 == 0 && (reinterpret_cast<uintptr_t>(A.state) & 15) == 0;
        return vec ? launch_decode<DELTA, 4>(A, num_seqs, stream) : launch_decode<DELTA, 1>(A, num_seqs, stream);
    }
    if (A.tables == nullptr) SPY_FAIL("head scan: a step with portions needs the coefficients' scratch");
    if (A.dk > 1024) SPY_FAIL("head scan: a key size of %d exceeds the kernel's 1024", A.dk);
    const int num_groups = tokens / U + num_seqs;
    const bool vec = A.dk % 4 == 0 && A.ld % 4 == 0 && A.off_k % 4 == 0 && A.off_q % 4 == 0 && (reinterpret_cast<uintptr_t>(A.proj) & 15) == 0;
    const dim3 grid((num_groups + TABLE_WARPS - 1) / TABLE_WARPS, A.H / A.share), block(32 * TABLE_WARPS);
    if (vec) spy_launch(head_table_kernel<DELTA, 4>, grid, block, 0, stream, A, num_seqs, num_groups);
    else spy_launch(head_table_kernel<DELTA, 1>, grid, block, 0, stream, A, num_seqs, num_groups);
    SPY_CHECK_LAUNCH("head scan (coefficients)");
    if (A.dk <= 32) return launch_portions_cols<DELTA, 4, 8>(A, num_seqs, stream);
    if (A.dk <= 64) return launch_portions_cols<DELTA, 8, 8>(A, num_seqs, stream);
    if (A.dk <= 128) return launch_portions_cols<DELTA, 16, 8>(A, num_seqs, stream);
    if (A.dk <= 256) return launch_portions_cols<DELTA, 32, 8>(A, num_seqs, stream);
    if (A.dk <= 512) return launch_portions_cols<DELTA, 32, 16>(A, num_seqs, stream);
    return launch_portions_cols<DELTA, 32, 32>(A, num_seqs, stream);
}

// Floats of scratch that a step with prompt portions needs (`tables`; it may be null when every request brings one token).
extern "C" long long spy_head_scan_scratch(int tokens, int num_seqs, int H) { return (long long)(tokens / U + num_seqs) * H * TABLE; }

// proj [tokens, ld] holds q, k ([H / share, dk] each) and v ([H, dv]) at `off_*`; gates [tokens, gates_ld] the pre-activations; a_log, dt_bias
// (and d_skip) [H]; state [slots, H, dk, dv]; out [tokens, H * dv].  `longest`: no request brings more tokens than this; 1: each brings one.
extern "C" int spy_gated_delta_scan(const float* proj, long long ld, int off_q, int off_k, int off_v, const float* gates, long long gates_ld, int off_rate,
                                    int off_decay, const float* a_log, const float* dt_bias, float* state, int num_slots, const int* q_start,
                                    const int* state_slot, int num_seqs, int tokens, int longest, float* out, int H, int share, int dk, int dv, float q_scale,
                                    float* tables, int* status, cudaStream_t stream)
{
    const HeadScanArgs A = {proj, ld, off_q, off_k, off_v, gates, gates_ld, off_rate, off_decay, a_log, dt_bias, nullptr, state, num_slots, q_start, state_slot,
                            out, H, share, dk, dv, q_scale, status, tables};
    return launch_head_scan<true>(A, num_seqs, tokens, longest, stream);
}

extern "C" int spy_ssd_scan(const float* proj, long long ld, int off_c, int off_b, int off_x, const float* gates, long long gates_ld, int off_dt,
                            const float* a_log, const float* dt_bias, const float* d_skip, float* state, int num_slots, const int* q_start,
                            const int* state_slot, int num_seqs, int tokens, int longest, float* out, int H, int share, int n, int dv, float* tables, int* status,
                            cudaStream_t stream)
{
    const HeadScanArgs A = {proj, ld, off_c, off_b, off_x, gates, gates_ld, 0, off_dt, a_log, dt_bias, d_skip, state, num_slots, q_start, state_slot,
                            out, H, share, n, dv, 1.0f, status, tables};
    return launch_head_scan<false>(A, num_seqs, tokens, longest, stream);
}
