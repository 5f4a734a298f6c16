// The gated delta rule with one decay a head, for long portions: chunks of 64 tokens as matrix products in float.
//
// Per head, with g_t the token's decay, beta_t its step size, and S [d, dv] the state before the chunk:
//     S_t = g_t S_(t-1) + k_t u_t^T,   u_t = beta_t (v_t - g_t S_(t-1)^T k_t),   o_t = S_t^T q_t.
// With c_t = g_1 ... g_t inside the chunk, unrolling S_t gives  u_t = beta_t (v_t - c_t S^T k_t - sum_(s<t) (c_t / c_s) (k_t . k_s) u_s),
// a triangular system: (I + A) U = diag(beta) V - diag(beta c) K S with A_ts = beta_t (c_t / c_s) (k_t . k_s), s < t.  So
//     U = X - W S,   X = (I + A)^-1 diag(beta) V,   W = (I + A)^-1 diag(beta c) K      (X, W: nothing of the state),
//     O = diag(c) Q S + P U,   P_ts = (c_t / c_s) (q_t . k_s), s <= t,
//     S <- c_C S + K^T diag(c_C / c_t) U.
// Three kernels over what li_delta_prepare made (recurrent.cu):
//   * delta_chunk_solve: every chunk and head by itself: A, P, and the two triangular solves, a thread a column;
//   * delta_chunk_carry: the chunks of a sequence in order, for a head and 16 columns of the values: U, the state before every
//     chunk, and the sequence's last state back into its slot.  The only part that walks, and it walks chunks;
//   * delta_chunk_output: every chunk and head by itself: O, with the norm over the head, its weight and the silu gate.
// Ratios of decays are exponentials of differences of summed logarithms (double), so nothing overflows however fast a head forgets.
// Everything is float on the multiply-add pipes; the results differ from the walk's by rounding.
#include "common.cuh"

namespace {

constexpr int kC = 64;              // tokens of a chunk
constexpr int kLA = kC + 4;         // a row of a [.., tokens] tile in shared memory
constexpr int kThreads = 256;
constexpr int kMultiprocessors = 148;
constexpr size_t kMoreThanHalf = 120 * 1024;      // of a multiprocessor's shared memory
constexpr int kSlice = 16;          // value columns a block of the carry takes
constexpr int kCols = 128;          // value columns a block of the output takes at a time
constexpr int kRowsB = 16;          // rows of its second operand that it stages at a time

__device__ __forceinline__ void copy16(float* dst, const float* src, bool valid) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    const int bytes = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes));
}
__device__ __forceinline__ void copies_done() { asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory"); }

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// Two multiply-adds in one instruction, each rounded like fmaf.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    float2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;"
        : "=l"(*reinterpret_cast<unsigned long long*>(&d))
        : "l"(*reinterpret_cast<unsigned long long*>(&a)), "l"(*reinterpret_cast<unsigned long long*>(&b)), "l"(*reinterpret_cast<unsigned long long*>(&c)));
    return d;
}
__device__ __forceinline__ float2 lo2(float4 v) { return make_float2(v.x, v.y); }
__device__ __forceinline__ float2 hi2(float4 v) { return make_float2(v.z, v.w); }
__device__ __forceinline__ float2 dot4(float4 a, float4 b, float2 c) { return fma2(lo2(a), lo2(b), fma2(hi2(a), hi2(b), c)); }

// columns of the values in the workspace: rows of whole 16-byte pieces
__host__ __device__ constexpr int padded(int dv) { return (dv + 3) / 4 * 4; }

template <int DP>
__host__ __device__ constexpr size_t solve_smem() { return ((size_t)2 * kC * (DP + 4) + 2 * kC * kLA + 4 * kC) * sizeof(float); }

// prep_qk [T, kv_heads, 2 DP + 4] (q | k | k . q), prep_g [T, heads, 4] (g | beta | log g), v [T, heads dv]; seg: a chunk's first token,
// end, number, slot.  Out, per chunk and head: wm [64, DP] and xm [64, dv] (W and X), pt [64, 64] (P transposed), sums [2, 64] (c_t, and
// c_64 / c_t).
template <int DP>
__global__ void __launch_bounds__(kThreads, DP <= 128 ? 2 : 1)
delta_chunk_solve_kernel(const float* __restrict__ prep_qk, const float* __restrict__ prep_g, const float* __restrict__ v, const int4* __restrict__ seg,
                         float* __restrict__ wm, float* __restrict__ xm, float* __restrict__ pt, float* __restrict__ sums, int heads, int kv_heads, int dv) {
    constexpr int LD = DP + 4, RQ = 2 * DP + 4;
    extern __shared__ __align__(16) float smem[];
    float* Ks = smem;                       // [64][LD]
    float* Qs = Ks + kC * LD;
    float* At = Qs + kC * LD;               // [s][t]
    float* Ps = At + kC * kLA;              // [s][t]
    float* cum = Ps + kC * kLA;             // [64] log(c_t), as a sum of two floats: heads that forget at once reach hundreds, and
    float* low = cum + kC;                  //      what counts are differences
    float* beta = low + kC;
    float* bc = beta + kC;                  // beta_t c_t
    pdl_wait();
    const int h = blockIdx.x, hk = h / (heads / kv_heads);
    const int4 sg = seg[blockIdx.y];
    const int q0 = sg.x, n = min(sg.y - sg.x, kC);
    const size_t unit = (size_t)sg.z * heads + h;
    const int tid = threadIdx.x, lane = tid & 31;
    for (int idx = tid; idx < kC * (DP / 4); idx += kThreads) {
        const int t = idx / (DP / 4), i = idx - t * (DP / 4);
        const float* row = prep_qk + ((size_t)(q0 + (t < n ? t : 0)) * kv_heads + hk) * RQ + 4 * i;
        copy16(Qs + t * LD + 4 * i, row, t < n);
        copy16(Ks + t * LD + 4 * i, row + DP, t < n);
    }
    if (tid < 32) {
        double a[2];
        float b[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = lane + 32 * j;
            const float4 g = t < n ? ld4(prep_g + ((size_t)(q0 + t) * heads + h) * 4) : make_float4(1.0f, 0.0f, 0.0f, 0.0f);
            a[j] = (double)g.z;
            b[j] = g.y;
        }
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double x = __shfl_up_sync(0xffffffffu, a[0], o), y = __shfl_up_sync(0xffffffffu, a[1], o);
            if (lane >= o) a[0] += x, a[1] += y;
        }
        a[1] += __shfl_sync(0xffffffffu, a[0], 31);
        const double end = __shfl_sync(0xffffffffu, a[1], 31);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = lane + 32 * j;
            const float c = expf((float)a[j]);
            cum[t] = (float)a[j];
            low[t] = (float)(a[j] - (double)(float)a[j]);
            beta[t] = b[j];
            bc[t] = b[j] * c;
            sums[(unit * 2) * kC + t] = c;
            sums[(unit * 2 + 1) * kC + t] = expf((float)(end - a[j]));
        }
    }
    copies_done();
    __syncthreads();
    // the products of keys with keys and of queries with keys: a thread takes tokens ty + 16 i against those of tx + 16 j, j <= i
    {
        const int tx = tid & 15, ty = tid >> 4;
        const int blocks = (n + 15) >> 4;
        float2 kk[4][4], qk[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) kk[i][j] = qk[i][j] = make_float2(0.0f, 0.0f);
#pragma unroll 1
        for (int k = 0; k < DP; k += 4) {
            float4 col[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) col[j] = ld4(Ks + (tx + 16 * j) * LD + k);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (i < blocks) {
                    const float4 kr = ld4(Ks + (ty + 16 * i) * LD + k), qr = ld4(Qs + (ty + 16 * i) * LD + k);
#pragma unroll
                    for (int j = 0; j <= i; ++j) {
                        kk[i][j] = dot4(kr, col[j], kk[i][j]);
                        qk[i][j] = dot4(qr, col[j], qk[i][j]);
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int t = ty + 16 * i, s = tx + 16 * j;
                const float f = s <= t ? expf((cum[t] - cum[s]) + (low[t] - low[s])) : 0.0f;
                At[s * kLA + t] = s < t ? beta[t] * f * (kk[i][j].x + kk[i][j].y) : 0.0f;
                Ps[s * kLA + t] = f * (qk[i][j].x + qk[i][j].y);
            }
    }
    __syncthreads();
    for (int idx = tid; idx < kC * (kC / 4); idx += kThreads) {
        const int s = idx / (kC / 4), i = idx - s * (kC / 4);
        *reinterpret_cast<float4*>(pt + (unit * kC + s) * kC + 4 * i) = ld4(Ps + s * kLA + 4 * i);
    }
    // the triangular solves, a column a thread: as soon as x_s is known it is taken off the rows behind it
    const int dvp = padded(dv);
    for (int c = tid; c < DP + dvp; c += kThreads) {
        float2 x[kC / 2];
        if (c < DP) {
#pragma unroll
            for (int t = 0; t < kC; t += 2) x[t / 2] = make_float2(bc[t] * Ks[t * LD + c], bc[t + 1] * Ks[(t + 1) * LD + c]);
        } else {
            const bool real = c - DP < dv;
            const float* col = v + (size_t)q0 * heads * dv + (size_t)h * dv + (real ? c - DP : 0);
#pragma unroll
            for (int t = 0; t < kC; t += 2)
                x[t / 2] = make_float2(real && t < n ? beta[t] * col[(size_t)t * heads * dv] : 0.0f, real && t + 1 < n ? beta[t + 1] * col[(size_t)(t + 1) * heads * dv] : 0.0f);
        }
#pragma unroll
        for (int s8 = 0; s8 < kC; s8 += 8) {
            if (s8 < n) {
#pragma unroll
                for (int s = s8; s < s8 + 8; ++s) {
                    const float xs = (s & 1) ? -x[s / 2].y : -x[s / 2].x;
                    const float2 both = make_float2(xs, xs);
#pragma unroll
                    for (int t4 = (s + 1) / 4 * 4; t4 < kC; t4 += 4) {
                        const float4 a = ld4(At + s * kLA + t4);         // (zeros where t <= s)
                        x[t4 / 2] = fma2(lo2(a), both, x[t4 / 2]);
                        x[t4 / 2 + 1] = fma2(hi2(a), both, x[t4 / 2 + 1]);
                    }
                }
            }
        }
        float* out = c < DP ? wm + unit * kC * DP + c : xm + unit * kC * dvp + (c - DP);
        const int ld = c < DP ? DP : dvp;
#pragma unroll
        for (int t = 0; t < kC; t += 2) {
            out[(size_t)t * ld] = x[t / 2].x;
            out[(size_t)(t + 1) * ld] = x[t / 2].y;
        }
    }
    pdl_launch_dependents();
}

constexpr int kCarryScratch = kThreads * 16;
constexpr int kUs = kSlice + 2;     // numbers (twice each) of a row of U in shared memory
template <int DP>
__host__ __device__ constexpr size_t carry_smem() {
    return ((size_t)kC * (DP + 4) + kC * (DP + 16) + 2 * (kC * kSlice + 2 * kC) + kSlice * (DP + 4) + kCarryScratch + 2 * kC * kUs) * sizeof(float);
}

// runs: triples (first chunk, chunks, slot).  s0 [chunk, head, DP, dv]: the state before every chunk; u [chunk, head, 64, dv].  A block
// takes 16 columns of a head's values.  W of the next chunk is on its way from the moment this chunk's W has been used, K likewise, so
// that one buffer each is enough and two blocks can share a multiprocessor.  Both products give a thread eight rows by four columns,
// summed over a part of the third index; lanes 16 apart hold neighbouring parts and add up first, the rest goes through shared memory.
template <int DP>
__global__ void __launch_bounds__(kThreads, DP <= 128 ? 2 : 1)
delta_chunk_carry_kernel(const float* __restrict__ prep_qk, const int4* __restrict__ seg, const int* __restrict__ runs, const float* __restrict__ wm,
                         const float* __restrict__ xm, const float* __restrict__ sums, float* __restrict__ state, long long state_stride,
                         float* __restrict__ s0, float* __restrict__ u, int heads, int kv_heads, int d, int dv) {
    constexpr int RQ = 2 * DP + 4, LD = DP + 4, LK = DP + 16;
    constexpr int NW = DP / 32, PH = 8 / NW, TB = DP / 2;               // K^T U: warps side by side over the key channels, parts, tiles
    constexpr int kXBuf = kC * kSlice + 2 * kC;
    extern __shared__ __align__(16) float smem[];
    float* W = smem;                                    // [64][LD]
    float* Kb = W + kC * LD;                            // [64][LK]
    float* Xs = Kb + kC * LK;                           // [2]: X [64][16], then sums [2][64]
    float* S = Xs + 2 * kXBuf;                          // [16][LD]: a column of the state after the other
    float* red = S + kSlice * LD;
    float2* Us = reinterpret_cast<float2*>(red + kCarryScratch);        // [64][kUs]: U with the decay to the chunk's end, every number twice
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, ct = lane & 3, quarter = (lane >> 2) & 3, pb = lane >> 4;
    const int h = blockIdx.y, hk = h / (heads / kv_heads), c0 = blockIdx.x * kSlice, dvp = padded(dv);
    pdl_wait();
    const int first = runs[3 * blockIdx.z], count = runs[3 * blockIdx.z + 1], slot = runs[3 * blockIdx.z + 2];
    float* st = state + (size_t)slot * state_stride + (size_t)h * dv * d;
    auto stage_w = [&](int j) {
        if (j < count) {
            const size_t unit = (size_t)(first + j) * heads + h;
            float* X = Xs + (j & 1) * kXBuf;
#pragma unroll 4
            for (int idx = tid; idx < kC * (DP / 4); idx += kThreads) {
                const int t = idx / (DP / 4), i = idx - t * (DP / 4);
                copy16(W + t * LD + 4 * i, wm + unit * kC * DP + 4 * idx, true);
            }
            {
                const int t = tid >> 2, c = 4 * (tid & 3);
                copy16(X + t * kSlice + c, xm + (unit * kC + t) * dvp + (c0 + c < dvp ? c0 + c : 0), c0 + c < dvp);
            }
            if (tid < 2 * kC / 4) copy16(X + kC * kSlice + 4 * tid, sums + unit * 2 * kC + 4 * tid, true);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto stage_k = [&](int j, int4 sg) {
        if (j < count) {
            const int n = min(sg.y - sg.x, kC);
            const float* from = prep_qk + ((size_t)sg.x * kv_heads + hk) * RQ + DP;
#pragma unroll 4
            for (int idx = tid; idx < kC * (DP / 4); idx += kThreads) {
                const int t = idx / (DP / 4), i = idx - t * (DP / 4);
                copy16(Kb + t * LK + 4 * i, from + (size_t)(t < n ? t : 0) * kv_heads * RQ + 4 * i, t < n);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage_w(0);
    stage_k(0, seg[first]);
    for (int idx = tid; idx < DP * kSlice; idx += kThreads) {
        const int c = idx / DP, k = idx - c * DP;
        S[c * LD + k] = (k < d && c0 + c < dv) ? st[(size_t)(c0 + c) * d + k] : 0.0f;
    }
    for (int j = 0; j < count; ++j) {
        const size_t unit = (size_t)(first + j) * heads + h;
        const float* X = Xs + (j & 1) * kXBuf;
        const float* cm = X + kC * kSlice;
        const int4 after = seg[first + min(j + 1, count - 1)];      // the next chunk's tokens: asked for long before they are needed
        asm volatile("cp.async.wait_group 1;" ::: "memory");        // W and X of this chunk (its K may still be on its way)
        __syncthreads();
        // the state before this chunk, for the outputs
        for (int idx = tid; idx < DP * 4; idx += kThreads) {
            const int k = idx >> 2, c = 4 * (idx & 3);
            if (c0 + c < dvp)
                *reinterpret_cast<float4*>(s0 + (unit * DP + k) * dvp + c0 + c) = make_float4(S[c * LD + k], S[(c + 1) * LD + k], S[(c + 2) * LD + k], S[(c + 3) * LD + k]);
        }
        // W S: tokens tt + 8 i by columns ct + 4 q a thread, an eighth of the key channels each
        {
            const int tt = quarter + 4 * (warp & 1), ph = warp >> 1, part = 2 * ph + pb;
            float2 acc[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i)
#pragma unroll
                for (int q = 0; q < 4; ++q) acc[i][q] = make_float2(0.0f, 0.0f);
            const float* w0 = W + tt * LD + part * (DP / 8);
            const float* sp = S + ct * LD + part * (DP / 8);
#pragma unroll 1
            for (int k = 0; k < DP / 8; k += 4) {
                float4 s[4];
#pragma unroll
                for (int q = 0; q < 4; ++q) s[q] = ld4(sp + 4 * q * LD + k);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const float4 w = ld4(w0 + 8 * i * LD + k);
#pragma unroll
                    for (int q = 0; q < 4; ++q) acc[i][q] = dot4(w, s[q], acc[i][q]);
                }
            }
            float* to = red + (ph * 32 + 16 * pb) * 32 + ct + 4 * tt;
#pragma unroll
            for (int e = 0; e < 16; ++e) {
                // this lane keeps rows i = 4 pb .. 4 pb + 3; the other half's go to the lane 16 away
                const float2 a = acc[e >> 2][e & 3], b = acc[4 + (e >> 2)][e & 3];
                const float lo = a.x + a.y, hi = b.x + b.y;
                const float other = __shfl_xor_sync(0xffffffffu, pb ? lo : hi, 16);
                to[e * 32] = (pb ? hi : lo) + other;
            }
        }
        __syncthreads();
        stage_w(j + 1);
#pragma unroll
        for (int o = tid; o < kC * kSlice; o += kThreads) {
            const int e = o >> 5, tile = o & 31, t = (tile >> 2) + 8 * (e >> 2), c = (tile & 3) + 4 * (e & 3);
            const float val = X[t * kSlice + c] - ((red[o] + red[1024 + o]) + (red[2048 + o] + red[3072 + o]));
            if (c0 + c < dvp) u[(unit * kC + t) * dvp + c0 + c] = val;
            const float f = cm[kC + t] * val;
            Us[t * kUs + c] = make_float2(f, f);
        }
        asm volatile("cp.async.wait_group 1;" ::: "memory");        // K of this chunk (the next W may still be on its way)
        __syncthreads();
        // the state behind the chunk: key channels 4 kt .. and DP / 2 + 4 kt .. by columns 4 ct .. a thread, a part of the tokens each
        {
            const int kt = quarter + 4 * (warp % NW), ph = warp / NW;
            float2 acc[4][4];                                           // [column][pair of key channels]
#pragma unroll
            for (int q = 0; q < 4; ++q)
#pragma unroll
                for (int p = 0; p < 4; ++p) acc[q][p] = make_float2(0.0f, 0.0f);
            const float* kp = Kb + (ph * (kC / PH) + pb) * LK + 4 * kt;
            const float2* up = Us + (ph * (kC / PH) + pb) * kUs + 4 * ct;
#pragma unroll 4
            for (int i = 0; i < kC / PH / 2; ++i) {
                const float4 ka = ld4(kp + 2 * i * LK), kb = ld4(kp + 2 * i * LK + DP / 2);
                const float* us = reinterpret_cast<const float*>(up + 2 * i * kUs);
                const float4 u01 = ld4(us), u23 = ld4(us + 4);
                const float2 uu[4] = {lo2(u01), hi2(u01), lo2(u23), hi2(u23)};
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    acc[q][0] = fma2(lo2(ka), uu[q], acc[q][0]);
                    acc[q][1] = fma2(hi2(ka), uu[q], acc[q][1]);
                    acc[q][2] = fma2(lo2(kb), uu[q], acc[q][2]);
                    acc[q][3] = fma2(hi2(kb), uu[q], acc[q][3]);
                }
            }
            float* to = red + (ph * 32 + 16 * pb) * TB + ct + 4 * kt;
#pragma unroll
            for (int e = 0; e < 16; ++e) {
                // columns 2 pb and 2 pb + 1 stay with this lane
                const float2 a = acc[e >> 3][(e >> 1) & 3], b = acc[2 + (e >> 3)][(e >> 1) & 3];
                const float lo = (e & 1) ? a.y : a.x, hi = (e & 1) ? b.y : b.x;
                const float other = __shfl_xor_sync(0xffffffffu, pb ? lo : hi, 16);
                to[e * TB] = (pb ? hi : lo) + other;
            }
        }
        __syncthreads();
        const float f = cm[kC - 1];
#pragma unroll
        for (int o = tid; o < 32 * TB; o += kThreads) {
            const int e = o / TB, tile = o - e * TB, c = 4 * (tile & 3) + (e >> 3), kk = e & 7, k = 4 * (tile >> 2) + (kk & 3) + (kk >> 2) * (DP / 2);
            float sum = red[o];
#pragma unroll
            for (int ph = 1; ph < PH; ++ph) sum += red[ph * 32 * TB + o];
            S[c * LD + k] = fmaf(f, S[c * LD + k], sum);
        }
        stage_k(j + 1, after);
    }
    pdl_launch_dependents();
    __syncthreads();
    for (int idx = tid; idx < DP * kSlice; idx += kThreads) {
        const int c = idx / DP, k = idx - c * DP;
        if (k < d && c0 + c < dv) st[(size_t)(c0 + c) * d + k] = S[c * LD + k];
    }
}

template <int DP>
__host__ __device__ constexpr size_t output_smem() { return ((size_t)(DP + kC) * kLA + 2 * kRowsB * kCols) * sizeof(float); }

// o = diag(c) Q S + P U as one product over DP + 64 rows.  norm_w given (dv at most 128): y = o / sqrt(mean(o^2) + eps) * norm_w * silu(gate),
// in the run dtype; else out takes o as it is.
template <typename T, int DP>
__global__ void __launch_bounds__(kThreads, DP <= 128 ? 3 : 2)
delta_chunk_output_kernel(const float* __restrict__ prep_qk, const int4* __restrict__ seg, const float* __restrict__ pt, const float* __restrict__ sums,
                          const float* __restrict__ s0, const float* __restrict__ u, float* __restrict__ out, const T* __restrict__ gate, int gate_ld,
                          int gate_off, const float* __restrict__ norm_w, float eps, T* __restrict__ y, int heads, int kv_heads, int dv) {
    constexpr int RQ = 2 * DP + 4;
    extern __shared__ __align__(16) float smem[];
    float* At = smem;                        // [DP + 64][68]: rows of Q^T with the decay, then of P^T
    float* B = At + (DP + kC) * kLA;         // [2][16][128]
    pdl_wait();
    const int h = blockIdx.x, hk = h / (heads / kv_heads), dvp = padded(dv);
    const int4 sg = seg[blockIdx.y];
    const int q0 = sg.x, n = min(sg.y - sg.x, kC);
    const size_t unit = (size_t)sg.z * heads + h;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, t0 = 8 * warp;
    constexpr int kBlocks = (DP + kC) / kRowsB;
    auto stage = [&](int b, int kb, int cb) {
#pragma unroll
        for (int idx = tid; idx < kRowsB * (kCols / 4); idx += kThreads) {
            const int r = idx / (kCols / 4), c = 4 * (idx - r * (kCols / 4));
            const int k = kb * kRowsB + r, col = cb + c;
            const float* row = k < DP ? s0 + (unit * DP + k) * dvp : u + (unit * kC + (k - DP)) * dvp;
            copy16(B + (b * kRowsB + r) * kCols + c, row + (col < dvp ? col : 0), col < dvp);
        }
    };
    stage(0, 0, 0);
    for (int idx = tid; idx < kC * (DP / 4); idx += kThreads) {
        const int i = idx / kC, t = idx - i * kC;
        float4 q = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (t < n) {
            q = ld4(prep_qk + ((size_t)(q0 + t) * kv_heads + hk) * RQ + 4 * i);
            const float f = sums[unit * 2 * kC + t];
            q.x *= f, q.y *= f, q.z *= f, q.w *= f;
        }
        float* to = At + 4 * i * kLA + t;
        to[0] = q.x, to[kLA] = q.y, to[2 * kLA] = q.z, to[3 * kLA] = q.w;
    }
    for (int idx = tid; idx < kC * (kC / 4); idx += kThreads) {
        const int s = idx / (kC / 4), i = idx - s * (kC / 4);
        copy16(At + (DP + s) * kLA + 4 * i, pt + (unit * kC + s) * kC + 4 * i, true);
    }
    for (int cb = 0; cb < dv; cb += kCols) {
        float2 acc[4][4];                    // tokens t0 + 2 a and t0 + 2 a + 1 by four columns
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[a][q] = make_float2(0.0f, 0.0f);
        for (int kb = 0; kb < kBlocks; ++kb) {
            const int b = kb & 1;
            copies_done();
            __syncthreads();
            if (kb + 1 < kBlocks) stage(b ^ 1, kb + 1, cb);
            // (rows of P^T: a token sees those up to its own; tokens behind the portion's end see nothing)
            if (t0 < n && kb * kRowsB <= DP + t0 + 7) {
#pragma unroll 4
                for (int r = 0; r < kRowsB; ++r) {
                    const float* at = At + (kb * kRowsB + r) * kLA + t0;
                    const float4 a0 = ld4(at), a1 = ld4(at + 4), bv = ld4(B + (b * kRowsB + r) * kCols + 4 * lane);
                    const float2 av[4] = {lo2(a0), hi2(a0), lo2(a1), hi2(a1)};
                    const float2 bb[4] = {make_float2(bv.x, bv.x), make_float2(bv.y, bv.y), make_float2(bv.z, bv.z), make_float2(bv.w, bv.w)};
#pragma unroll
                    for (int a = 0; a < 4; ++a)
#pragma unroll
                        for (int q = 0; q < 4; ++q) acc[a][q] = fma2(av[a], bb[q], acc[a][q]);
                }
            }
        }
        const int col = cb + 4 * lane;
#pragma unroll
        for (int a = 0; a < 8; ++a) {
            const int t = t0 + a;
            if (t >= n) break;                                     // (the same for the whole warp)
            float o[4];
#pragma unroll
            for (int q = 0; q < 4; ++q) o[q] = (a & 1) ? acc[a / 2][q].y : acc[a / 2][q].x;
            if (norm_w) {
                float ss = 0.0f;
#pragma unroll
                for (int q = 0; q < 4; ++q) ss = fmaf(o[q], o[q], ss);                     // (zeros behind the last column)
                const float rinv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + eps);
                const T* gr = gate + (size_t)(q0 + t) * gate_ld + gate_off + (size_t)h * dv + col;
                T* to = y + (size_t)(q0 + t) * heads * dv + (size_t)h * dv + col;
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (col + q < dv) {
                        const float g = to_float(gr[q]);
                        to[q] = from_float<T>(o[q] * rinv * norm_w[h * dv + col + q] * (g / (1.0f + expf(-g))));
                    }
            } else {
                float* to = out + (size_t)(q0 + t) * heads * dv + (size_t)h * dv + col;
#pragma unroll
                for (int q = 0; q < 4; ++q)
                    if (col + q < dv) to[q] = o[q];
            }
        }
        __syncthreads();                                           // everybody has left the last rows staged
        if (cb + kCols < dv) stage(0, 0, cb + kCols);
    }
    pdl_launch_dependents();
}

template <typename K>
int raise_smem(K kernel, size_t bytes, const char* what) {
    if (bytes <= 48 * 1024) return 0;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    return e == cudaSuccess ? 0 : li_fail("%s: cannot raise shared memory to %zu: %s", what, bytes, cudaGetErrorString(e));
}

template <int DP>
int launch(const float* prep_qk, const float* prep_g, const float* v, float* state, long long state_stride, const int* seg, int chunks, const int* runs,
           int nruns, float* wm, float* xm, float* pt, float* sums, float* s0, float* u, float* out, const void* gate, int dtype, int gate_ld, int gate_off,
           const float* norm_w, float eps, void* y, int heads, int kv_heads, int d, int dv, cudaStream_t stream) {
    static bool raised = false;
    if (!raised) {
        if (int rc = raise_smem(delta_chunk_solve_kernel<DP>, solve_smem<DP>(), "delta chunks")) return rc;
        if (int rc = raise_smem(delta_chunk_carry_kernel<DP>, carry_smem<DP>() > kMoreThanHalf ? carry_smem<DP>() : kMoreThanHalf, "delta chunks")) return rc;
        if (int rc = raise_smem(delta_chunk_output_kernel<float, DP>, output_smem<DP>(), "delta chunks")) return rc;
        if (int rc = raise_smem(delta_chunk_output_kernel<bf16, DP>, output_smem<DP>(), "delta chunks")) return rc;
        raised = true;
    }
    cudaError_t e = li_launch_pdl(delta_chunk_solve_kernel<DP>, dim3(heads, chunks), dim3(kThreads), solve_smem<DP>(), stream, prep_qk, prep_g, v, (const int4*)seg,
                                  wm, xm, pt, sums, heads, kv_heads, dv);
    if (e == cudaSuccess) {
        // The walk lasts as long as its slowest block: while there is a multiprocessor for each, none shares one (blocks are placed as the
        // kernel before drains, two at a time where two fit; more shared memory than half of a multiprocessor's keeps them apart).
        const dim3 grid(ceil_div(dv, kSlice), heads, nruns);
        const bool apart = (long long)grid.x * heads * nruns <= kMultiprocessors;
        const size_t bytes = apart && carry_smem<DP>() < kMoreThanHalf ? kMoreThanHalf : carry_smem<DP>();
        e = li_launch_pdl(delta_chunk_carry_kernel<DP>, grid, dim3(kThreads), bytes, stream, prep_qk, (const int4*)seg, runs, wm, xm, sums, state, state_stride, s0, u, heads,
                          kv_heads, d, dv);
    }
    if (e == cudaSuccess) {
        if (dtype == LI_F32)
            e = li_launch_pdl(delta_chunk_output_kernel<float, DP>, dim3(heads, chunks), dim3(kThreads), output_smem<DP>(), stream, prep_qk, (const int4*)seg, pt,
                              sums, s0, u, out, (const float*)gate, gate_ld, gate_off, norm_w, eps, (float*)y, heads, kv_heads, dv);
        else
            e = li_launch_pdl(delta_chunk_output_kernel<bf16, DP>, dim3(heads, chunks), dim3(kThreads), output_smem<DP>(), stream, prep_qk, (const int4*)seg, pt,
                              sums, s0, u, out, (const bf16*)gate, gate_ld, gate_off, norm_w, eps, (bf16*)y, heads, kv_heads, dv);
    }
    if (e != cudaSuccess) return li_fail("delta chunks: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("delta chunks");
}

}  // namespace

// seg [chunks] quadruples (first token, end, chunk, slot), at most 64 tokens each; runs [nruns] triples (first chunk, chunks, slot).
// Workspace, float, with DP = 32, 64, 128 or 256 (the first that holds d) and dv rounded up to a multiple of 4: wm [chunks, heads, 64, DP],
// xm [chunks, heads, 64, dv], pt [chunks, heads, 64, 64], sums [chunks, heads, 2, 64], s0 [chunks, heads, DP, dv], u [chunks, heads, 64, dv].  norm_w [heads dv] (may be NULL; dv at most 128): y [T, heads dv] in the run dtype takes
// the normed and gated outputs, gate [T, gate_ld] from column gate_off; without it out [T, heads dv] float takes the outputs.
LI_EXPORT int li_delta_chunks(const float* prep_qk, const float* prep_g, const float* v, float* state, long long state_stride, const int* seg, int chunks,
                              const int* runs, int nruns, float* wm, float* xm, float* pt, float* sums, float* s0, float* u, float* out, const void* gate,
                              int dtype, int gate_ld, int gate_off, const float* norm_w, float eps, void* y, int heads, int kv_heads, int d, int dv,
                              cudaStream_t stream) {
    LI_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && d > 0 && d <= 256 && dv > 0, "delta chunks: %d heads on %d key heads of %d x %d (keys of at most 256)",
               heads, kv_heads, d, dv);
    LI_REQUIRE(chunks >= 0 && nruns >= 0 && chunks <= 65535 && nruns <= 65535 && heads <= 65535, "delta chunks: %d chunks of %d sequences in one launch", chunks, nruns);
    LI_REQUIRE(norm_w != nullptr ? (dv <= kCols && y != nullptr && gate != nullptr && gate_off >= 0 && gate_off + heads * dv <= gate_ld) : out != nullptr,
               "delta chunks: outputs of %d columns a head, gate at column %d of %d", dv, gate_off, gate_ld);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "delta chunks: unknown dtype %d", dtype);
    LI_REQUIRE(((uintptr_t)prep_qk | (uintptr_t)prep_g | (uintptr_t)seg | (uintptr_t)wm | (uintptr_t)xm | (uintptr_t)pt | (uintptr_t)sums | (uintptr_t)s0 | (uintptr_t)u) % 16 == 0,
               "delta chunks: an operand is not on a 16-byte boundary");
    if (chunks == 0 || nruns == 0) return 0;
#define LI_CHUNKS(DP)                                                                                                                                  \
    return launch<DP>(prep_qk, prep_g, v, state, state_stride, seg, chunks, runs, nruns, wm, xm, pt, sums, s0, u, out, gate, dtype, gate_ld, gate_off, norm_w, eps, \
                      y, heads, kv_heads, d, dv, stream)
    if (d <= 32) LI_CHUNKS(32);
    if (d <= 64) LI_CHUNKS(64);
    if (d <= 128) LI_CHUNKS(128);
    LI_CHUNKS(256);
#undef LI_CHUNKS
}
