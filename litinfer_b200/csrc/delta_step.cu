// One token a sequence under the gated delta rule with one decay a head, as one kernel: what li_delta_prepare, li_delta_scan and
// li_gated_rmsnorm do one after the other (recurrent.cu), for steps of single tokens.
//
// A block takes one key head of one sequence with all the heads that use it:
//   1. the convolution of its channels (the last taps - 1 inputs from the request's state, which moves on) and silu;
//   2. q and k as unit vectors, k . q, and per head the decay and beta;
//   3. the heads' states, eight columns a warp at a time: with a column's elements spread over the lanes, the two sums
//      S^T k and S^T q of the state as it was give u = beta (v - g S^T k) and o = g S^T q + u (k . q), and the column goes back
//      as g S + k u;
//   4. per head o / sqrt(mean(o^2) + eps) * w * silu(gate), in the run dtype.
// While the kernel before this one still runs, the block asks for its states' lines.  Everything is float.
#include "common.cuh"

namespace {

constexpr int kThreads = 512, kWarps = kThreads / 32;
constexpr int kCols = 8;

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }

// Sums over the 32 lanes of eight values a lane in nine exchanges; every lane then holds the sum of value
// 4 (lane >> 4 & 1) + 2 (lane >> 3 & 1) + (lane >> 2 & 1).
__device__ __forceinline__ float sum8(const float (&a)[8], int lane) {
    float b[4], c[2];
    const bool up16 = lane & 16, up8 = lane & 8, up4 = lane & 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) b[j] = (up16 ? a[j + 4] : a[j]) + __shfl_xor_sync(0xffffffffu, up16 ? a[j] : a[j + 4], 16);
#pragma unroll
    for (int j = 0; j < 2; ++j) c[j] = (up8 ? b[j + 2] : b[j]) + __shfl_xor_sync(0xffffffffu, up8 ? b[j] : b[j + 2], 8);
    float v = (up4 ? c[1] : c[0]) + __shfl_xor_sync(0xffffffffu, up4 ? c[0] : c[1], 4);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    return v + __shfl_xor_sync(0xffffffffu, v, 1);
}

// E = DP / 32 neighbouring key channels a lane; kWhole: d is DP, so that a lane's elements are one load
template <typename T, int E, bool kWhole>
__global__ void __launch_bounds__(kThreads)
delta_step_kernel(const T* __restrict__ proj, int stride, int col0, int b_off, int a_off, int g_off, const float* __restrict__ conv_w, int taps,
                  float* __restrict__ state, long long state_stride, long long state_off, const int* __restrict__ slots, const float* __restrict__ dt_bias,
                  const float* __restrict__ A_log, float q_scale, float unit_eps, const float* __restrict__ norm_w, float eps, T* __restrict__ y, int heads,
                  int kv_heads, int d, int dv) {
    constexpr int DP = 32 * E;
    extern __shared__ float smem[];
    float* qs = smem;                        // [DP] each, zeros behind d
    float* ks = qs + DP;
    const int rep = heads / kv_heads;
    float* vs = ks + DP;                     // [rep][dv]
    float* os = vs + rep * dv;               // [rep][dv]
    float* gb = os + rep * dv;               // [rep][2] decay and beta
    __shared__ float factors[3];             // of q, of k, and k . q
    const int hk = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* st = state + (size_t)slots[s] * state_stride;
    float* heads_at = st + (size_t)hk * rep * dv * d;
    pdl_launch_dependents();
    for (size_t i = (size_t)tid * 128; i < (size_t)rep * dv * d * sizeof(float); i += kThreads * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"((const char*)heads_at + i));
    pdl_wait();
    const T* row = proj + (size_t)s * stride;
    const int C = 2 * kv_heads * d + heads * dv;
    float* cs = st + state_off;
    for (int i = tid; i < 2 * DP + rep * dv; i += kThreads) {
        // which channel of the convolution, and where its result goes
        const bool is_v = i >= 2 * DP;
        const int j = is_v ? i - 2 * DP : i & (DP - 1);
        if (!is_v && j >= d) {
            smem[i] = 0.0f;
            continue;
        }
        const int c = is_v ? 2 * kv_heads * d + hk * rep * dv + j : (i >= DP ? kv_heads * d : 0) + hk * d + j;
        const float now = to_float(row[col0 + c]);
        float acc = 0.0f;
        for (int k = 0; k + 1 < taps; ++k) {
            const float old = cs[(size_t)k * C + c];
            acc = fmaf(conv_w[(size_t)c * taps + k], old, acc);
            if (k > 0) cs[(size_t)(k - 1) * C + c] = old;                  // oldest first: each input moves one place on
        }
        acc = fmaf(conv_w[(size_t)c * taps + taps - 1], now, acc);
        if (taps > 1) cs[(size_t)(taps - 2) * C + c] = now;
        smem[i] = silu_f(acc);
    }
    if (tid < rep) {
        const int h = hk * rep + tid;
        const float z = to_float(row[a_off + h]) + dt_bias[h];
        const float sp = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
        gb[2 * tid] = expf(-expf(A_log[h]) * sp);
        gb[2 * tid + 1] = 1.0f / (1.0f + expf(-to_float(row[b_off + h])));
    }
    __syncthreads();
    if (warp == 0) {
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const float q = qs[lane + 32 * e], k = ks[lane + 32 * e];
            qq = fmaf(q, q, qq), kk = fmaf(k, k, kk), qk = fmaf(q, k, qk);
        }
        qq = warp_sum(qq), kk = warp_sum(kk), qk = warp_sum(qk);
        if (lane == 0) {
            factors[0] = q_scale / sqrtf(qq + unit_eps);
            factors[1] = 1.0f / sqrtf(kk + unit_eps);
            factors[2] = qk * factors[0] * factors[1];
        }
    }
    __syncthreads();
    float q[E], k[E];
#pragma unroll
    for (int e = 0; e < E; ++e) q[e] = qs[E * lane + e] * factors[0], k[e] = ks[E * lane + e] * factors[1];
    const float kq = factors[2];
    const int groups = (dv + kCols - 1) / kCols;
    for (int job = warp; job < rep * groups; job += kWarps) {
        const int r = job / groups, c0 = (job - r * groups) * kCols;
        float* S_at = heads_at + ((size_t)r * dv + c0) * d;
        float S[kCols][E], sk[kCols], sq[kCols];
#pragma unroll
        for (int j = 0; j < kCols; ++j) {
            const float* p = S_at + (size_t)j * d + E * lane;
            const bool in = c0 + j < dv;
            if constexpr (kWhole && E % 4 == 0) {
#pragma unroll
                for (int f = 0; f < E / 4; ++f) {
                    const float4 x = in ? reinterpret_cast<const float4*>(p)[f] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    S[j][4 * f] = x.x, S[j][4 * f + 1] = x.y, S[j][4 * f + 2] = x.z, S[j][4 * f + 3] = x.w;
                }
            } else {
#pragma unroll
                for (int e = 0; e < E; ++e) S[j][e] = (in && E * lane + e < d) ? p[e] : 0.0f;
            }
        }
#pragma unroll
        for (int j = 0; j < kCols; ++j) {
            sk[j] = sq[j] = 0.0f;
#pragma unroll
            for (int e = 0; e < E; ++e) sk[j] = fmaf(S[j][e], k[e], sk[j]), sq[j] = fmaf(S[j][e], q[e], sq[j]);
        }
        const float g = gb[2 * r], beta = gb[2 * r + 1];
        const int mine = 4 * ((lane >> 4) & 1) + 2 * ((lane >> 3) & 1) + ((lane >> 2) & 1);
        const float skv = g * sum8(sk, lane), sqv = g * sum8(sq, lane);
        const float v = c0 + mine < dv ? vs[r * dv + c0 + mine] : 0.0f;
        const float um = beta * (v - skv);
        if ((lane & 3) == 0 && c0 + mine < dv) os[r * dv + c0 + mine] = fmaf(um, kq, sqv);
#pragma unroll
        for (int j = 0; j < kCols; ++j) {
            const float u = __shfl_sync(0xffffffffu, um, 16 * ((j >> 2) & 1) + 8 * ((j >> 1) & 1) + 4 * (j & 1));
            float* p = S_at + (size_t)j * d + E * lane;
            if (c0 + j >= dv) continue;
            if constexpr (kWhole && E % 4 == 0) {
#pragma unroll
                for (int f = 0; f < E / 4; ++f)
                    reinterpret_cast<float4*>(p)[f] = make_float4(fmaf(k[4 * f], u, g * S[j][4 * f]), fmaf(k[4 * f + 1], u, g * S[j][4 * f + 1]),
                                                                  fmaf(k[4 * f + 2], u, g * S[j][4 * f + 2]), fmaf(k[4 * f + 3], u, g * S[j][4 * f + 3]));
            } else {
#pragma unroll
                for (int e = 0; e < E; ++e)
                    if (E * lane + e < d) p[e] = fmaf(k[e], u, g * S[j][e]);
            }
        }
    }
    __syncthreads();
    for (int r = warp; r < rep; r += kWarps) {
        const int h = hk * rep + r;
        float ss = 0.0f;
        for (int c = lane; c < dv; c += 32) ss = fmaf(os[r * dv + c], os[r * dv + c], ss);
        const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + eps);
        for (int c = lane; c < dv; c += 32)
            y[(size_t)s * heads * dv + (size_t)h * dv + c] =
                from_float<T>(os[r * dv + c] * rinv * norm_w[(size_t)h * dv + c] * silu_f(to_float(row[g_off + (size_t)h * dv + c])));
    }
}

template <typename T, int E>
cudaError_t launch(const void* proj, int stride, int col0, int b_off, int a_off, int g_off, const float* conv_w, int taps, float* state, long long state_stride,
                   long long state_off, const int* slots, const float* dt_bias, const float* A_log, float q_scale, float unit_eps, const float* norm_w, float eps,
                   void* y, int S, int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
    const int rep = heads / kv_heads;
    const size_t smem = ((size_t)2 * 32 * E + 2 * rep * dv + 2 * rep) * sizeof(float);
    const bool whole = d == 32 * E && state_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
    return li_launch_pdl(whole ? delta_step_kernel<T, E, true> : delta_step_kernel<T, E, false>, dim3(kv_heads, S), dim3(kThreads), smem, stream, (const T*)proj, stride,
                         col0, b_off, a_off, g_off, conv_w, taps, state, state_stride, state_off, slots, dt_bias, A_log, q_scale, unit_eps, norm_w, eps, (T*)y, heads,
                         kv_heads, d, dv);
}

}  // namespace

// proj [S, stride], one row a sequence: the convolution's channels q | k | v from column col0, beta's, the decays' and the gate's inputs from
// b_off, a_off and g_off; conv_w [channels, taps] float; state [slots, state_stride] float: the heads' states [heads][dv][d], and at state_off
// the last taps - 1 inputs; norm_w [heads dv]; y [S, heads dv] in the run dtype.  accepts: 1 if the sizes fit.
LI_EXPORT int li_delta_step_accepts(int heads, int kv_heads, int d, int dv) {
    return (heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && d > 0 && d <= 256 && dv > 0 && heads / kv_heads <= kThreads &&
            ((size_t)2 * 256 + 2 * (size_t)(heads / kv_heads) * (dv + 1)) * sizeof(float) <= 48 * 1024) ? 1 : 0;
}

LI_EXPORT int li_delta_step(const void* proj, int dtype, int stride, int col0, int b_off, int a_off, int g_off, const float* conv_w, int taps, float* state,
                            long long state_stride, long long state_off, const int* slots, const float* dt_bias, const float* A_log, float q_scale, float unit_eps,
                            const float* norm_w, float eps, void* y, int S, int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
    LI_REQUIRE(li_delta_step_accepts(heads, kv_heads, d, dv), "delta step: refuses %d heads on %d key heads of %d x %d", heads, kv_heads, d, dv);
    LI_REQUIRE(taps >= 1 && conv_w != nullptr, "delta step: a convolution of %d taps", taps);
    LI_REQUIRE(col0 >= 0 && col0 + 2 * kv_heads * d + heads * dv <= stride && b_off >= 0 && b_off + heads <= stride && a_off >= 0 && a_off + heads <= stride &&
                   g_off >= 0 && g_off + heads * dv <= stride, "delta step: the projections' columns do not fit rows of %d", stride);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "delta step: unknown dtype %d", dtype);
    if (S == 0) return 0;
    LI_REQUIRE(S <= 65535, "delta step: %d sequences in one launch", S);
    cudaError_t e;
#define LI_STEP(E_)                                                                                                                                   \
    e = dtype == LI_F32 ? launch<float, E_>(proj, stride, col0, b_off, a_off, g_off, conv_w, taps, state, state_stride, state_off, slots, dt_bias, A_log,  \
                                            q_scale, unit_eps, norm_w, eps, y, S, heads, kv_heads, d, dv, stream)                                        \
                        : launch<bf16, E_>(proj, stride, col0, b_off, a_off, g_off, conv_w, taps, state, state_stride, state_off, slots, dt_bias, A_log,   \
                                           q_scale, unit_eps, norm_w, eps, y, S, heads, kv_heads, d, dv, stream)
    if (d <= 32) LI_STEP(1);
    else if (d <= 64) LI_STEP(2);
    else if (d <= 128) LI_STEP(4);
    else LI_STEP(8);
#undef LI_STEP
    if (e != cudaSuccess) return li_fail("delta_step: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("delta_step");
}
