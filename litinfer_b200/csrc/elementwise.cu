// Embedding gather, RMSNorm (plain, fused with the residual add, gathered
// rows), residual add and SwiGLU.
//
// RMSNorm per row: ss = sum x_j^2; r = 1 / sqrt(ss / H + eps); y_j = (w_j x_j) r,
// all in float, one rounding of y (LitInfer: src/ops/rms_norm/op.cpp:13-24).
// SwiGLU: up * gate / (1 + exp(-gate)) (src/ops/swiglu/op.cpp:17-23).
// One block per row; every thread owns the elements j = tid, tid + B, ... in
// both passes, so the second pass re-reads only what the same thread wrote.
#include "common.cuh"

namespace {

constexpr int kRowThreads = 256;

template <typename T>
__global__ void embedding_kernel(const T* __restrict__ table, const int* __restrict__ ids, float* __restrict__ out, int H, int V, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);          // ids are validated on the host; never read outside the table
    const T* row = table + (size_t)id * H;
    float* dst = out + (size_t)t * H;
    for (int j = threadIdx.x; j < H; j += blockDim.x) dst[j] = to_float(row[j]) * scale;
}

// x[t] += pairs[row of (previous token, token)]; the previous token of a portion's first token is the sequence's state.
template <typename T>
__global__ void add_pair_rows_kernel(float* __restrict__ x, const T* __restrict__ pairs, const int* __restrict__ ids,
                                     const int* __restrict__ positions, const int* __restrict__ q_start, const int* __restrict__ seq_of_token,
                                     const int* __restrict__ slots, int* __restrict__ state, long long state_stride, int buckets,
                                     long long mul_prev, long long mul_cur, int H) {
    __shared__ int row_s;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    if (threadIdx.x == 0) {
        const int s = seq_of_token[t];
        const int first = q_start[s], end = q_start[s + 1];
        int* st = state + (size_t)slots[s] * state_stride;
        int row = buckets;                                      // a sequence's first token
        if (positions[t] > 0) {
            const long long prev = t > first ? ids[t - 1] : *st;
            long long r = (prev * mul_prev + (long long)ids[t] * mul_cur) % buckets;
            row = (int)(r < 0 ? r + buckets : r);
        }
        // the portion's first token is the only reader of the state, so it also moves it on: to the portion's last token
        if (t == first) *st = ids[end - 1];
        row_s = row;
    }
    __syncthreads();
    const T* src = pairs + (size_t)row_s * H;
    float* dst = x + (size_t)t * H;
    for (int j = threadIdx.x; j < H; j += blockDim.x) dst[j] += to_float(src[j]);
}

// mode 0: y = norm(x[row]); mode 1: x[row] += delta[row] first (stored back).
template <typename T, bool kAdd>
__global__ void rmsnorm_kernel(float* __restrict__ x, const T* __restrict__ delta, const int* __restrict__ rows,
                               const float* __restrict__ w, float eps, T* __restrict__ out, int H, int T_rows) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    int src = rows ? rows[r] : r;
    if (src < 0 || src >= T_rows) src = 0;
    float* xr = x + (size_t)src * H;
    float ss = 0.0f;
    for (int j = threadIdx.x; j < H; j += blockDim.x) {
        float v = xr[j];
        if (kAdd) {
            v += to_float(delta[(size_t)src * H + j]);
            xr[j] = v;
        }
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float rinv = 1.0f / sqrtf(ss / (float)H + eps);
    T* o = out + (size_t)r * H;
    for (int j = threadIdx.x; j < H; j += blockDim.x) o[j] = from_float<T>((w[j] * xr[j]) * rinv);
}

// The same for widths that are a multiple of 4 and fit 4 float4 a thread: the row stays in
// registers between the sum of squares and the scaling, and all loads are 16 bytes wide.
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&r.x), b = *reinterpret_cast<const __nv_bfloat162*>(&r.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 r;
    r.x = *reinterpret_cast<const unsigned*>(&a);
    r.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
}

constexpr int kVecPerThread = 4;

template <typename T, bool kAdd>
__global__ void rmsnorm_vec_kernel(float* __restrict__ x, const T* __restrict__ delta, const int* __restrict__ rows,
                                   const float* __restrict__ w, float eps, T* __restrict__ out, int H, int T_rows) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    int src = rows ? rows[r] : r;
    if (src < 0 || src >= T_rows) src = 0;
    float* xr = x + (size_t)src * H;
    const int nvec = H >> 2;
    float4 v[kVecPerThread];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kVecPerThread; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        if (q < nvec) {
            v[i] = load4(xr + 4 * q);
            if (kAdd) {
                const float4 d = load4(delta + (size_t)src * H + 4 * q);
                v[i].x += d.x; v[i].y += d.y; v[i].z += d.z; v[i].w += d.w;
                store4(xr + 4 * q, v[i]);
            }
            ss += v[i].x * v[i].x;
            ss += v[i].y * v[i].y;
            ss += v[i].z * v[i].z;
            ss += v[i].w * v[i].w;
        }
    }
    ss = block_sum(ss, scratch);
    const float rinv = 1.0f / sqrtf(ss / (float)H + eps);
    T* o = out + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < kVecPerThread; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        if (q < nvec) {
            const float4 ww = load4(w + 4 * q);
            store4(o + 4 * q, make_float4((ww.x * v[i].x) * rinv, (ww.y * v[i].y) * rinv, (ww.z * v[i].z) * rinv, (ww.w * v[i].w) * rinv));
        }
    }
}

template <typename T>
__global__ void residual_add_kernel(float* __restrict__ x, const T* __restrict__ delta, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < n; i += stride) x[i] += to_float(delta[i]);
}

template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int I, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < n; i += stride) {
        const long long t = i / I;
        const int j = (int)(i - t * I);
        const float g = to_float(gate_up[t * 2 * I + j]);
        const float u = to_float(gate_up[t * 2 * I + I + j]);
        out[i] = from_float<T>(swiglu_of<T>(g, u));
    }
}

int grid_for(long long n, int threads) {
    long long b = ceil_div_ll(n, threads);
    if (b > 148LL * 16) b = 148LL * 16;
    return (int)(b < 1 ? 1 : b);
}

}  // namespace

LI_EXPORT int li_add_pair_rows(float* x, const void* pairs, int dtype, const int* ids, const int* positions, const int* q_start,
                               const int* seq_of_token, const int* slots, int* state, long long state_stride, int buckets, long long mul_prev,
                               long long mul_cur, int T, int H, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && H > 0 && buckets > 0 && state_stride > 0, "add_pair_rows: bad sizes T=%d H=%d buckets=%d", T, H, buckets);
    if (T == 0) return 0;
    if (dtype == LI_F32)
        li_launch_pdl(add_pair_rows_kernel<float>, dim3(T), dim3(kRowThreads), 0, stream, x, (const float*)pairs, ids, positions, q_start, seq_of_token,
                      slots, state, state_stride, buckets, mul_prev, mul_cur, H);
    else if (dtype == LI_BF16)
        li_launch_pdl(add_pair_rows_kernel<bf16>, dim3(T), dim3(kRowThreads), 0, stream, x, (const bf16*)pairs, ids, positions, q_start, seq_of_token,
                      slots, state, state_stride, buckets, mul_prev, mul_cur, H);
    else
        return li_fail("add_pair_rows: unknown dtype %d", dtype);
    return li_check_launch("add_pair_rows");
}

LI_EXPORT int li_embedding(const void* table, int dtype, const int* ids, float* out, int T, int H, int V, float scale, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && H > 0 && V > 0, "embedding: bad sizes T=%d H=%d V=%d", T, H, V);
    if (T == 0) return 0;
    if (dtype == LI_F32)
        li_launch_pdl(embedding_kernel<float>, dim3(T), dim3(kRowThreads), 0, stream, (const float*)table, ids, out, H, V, scale);
    else if (dtype == LI_BF16)
        li_launch_pdl(embedding_kernel<bf16>, dim3(T), dim3(kRowThreads), 0, stream, (const bf16*)table, ids, out, H, V, scale);
    else
        return li_fail("embedding: unknown dtype %d", dtype);
    return li_check_launch("embedding");
}

template <bool kAdd>
static int launch_norm(float* x, const void* delta, int dtype, const int* rows, const float* w, float eps, void* out, int R, int T,
                       int H, cudaStream_t stream, const char* what) {
    LI_REQUIRE(R >= 0 && H > 0, "%s: bad sizes rows=%d H=%d", what, R, H);
    if (R == 0) return 0;
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "%s: unknown dtype %d", what, dtype);
    const bool aligned = ((uintptr_t)x % 16 == 0) && ((uintptr_t)out % 16 == 0) && ((uintptr_t)w % 16 == 0) && ((uintptr_t)delta % 16 == 0);
    if (H % 4 == 0 && H / 4 <= 1024 * kVecPerThread && aligned) {
        int threads = ceil_div(H / 4, kVecPerThread);
        threads = ceil_div(threads, 32) * 32;
        if (threads < 64) threads = 64;
        if (dtype == LI_F32)
            li_launch_pdl(rmsnorm_vec_kernel<float, kAdd>, dim3(R), dim3(threads), 0, stream, x, (const float*)delta, rows, w, eps, (float*)out, H, T);
        else
            li_launch_pdl(rmsnorm_vec_kernel<bf16, kAdd>, dim3(R), dim3(threads), 0, stream, x, (const bf16*)delta, rows, w, eps, (bf16*)out, H, T);
        return li_check_launch(what);
    }
    if (dtype == LI_F32)
        li_launch_pdl(rmsnorm_kernel<float, kAdd>, dim3(R), dim3(kRowThreads), 0, stream, x, (const float*)delta, rows, w, eps, (float*)out, H, T);
    else
        li_launch_pdl(rmsnorm_kernel<bf16, kAdd>, dim3(R), dim3(kRowThreads), 0, stream, x, (const bf16*)delta, rows, w, eps, (bf16*)out, H, T);
    return li_check_launch(what);
}

LI_EXPORT int li_rmsnorm(const float* x, const float* w, float eps, void* out, int dtype, int T, int H, cudaStream_t stream) {
    return launch_norm<false>(const_cast<float*>(x), nullptr, dtype, nullptr, w, eps, out, T, T, H, stream, "rmsnorm");
}

LI_EXPORT int li_add_rmsnorm(float* x, const void* delta, int dtype, const float* w, float eps, void* out, int T, int H,
                             cudaStream_t stream) {
    return launch_norm<true>(x, delta, dtype, nullptr, w, eps, out, T, T, H, stream, "add_rmsnorm");
}

LI_EXPORT int li_gather_rmsnorm(const float* x, const int* rows, const float* w, float eps, void* out, int dtype, int R, int T, int H,
                                cudaStream_t stream) {
    return launch_norm<false>(const_cast<float*>(x), nullptr, dtype, rows, w, eps, out, R, T, H, stream, "gather_rmsnorm");
}

LI_EXPORT int li_residual_add(float* x, const void* delta, int dtype, long long n, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (dtype == LI_F32)
        residual_add_kernel<float><<<grid_for(n, 256), 256, 0, stream>>>(x, (const float*)delta, n);
    else if (dtype == LI_BF16)
        residual_add_kernel<bf16><<<grid_for(n, 256), 256, 0, stream>>>(x, (const bf16*)delta, n);
    else
        return li_fail("residual_add: unknown dtype %d", dtype);
    return li_check_launch("residual_add");
}

// The device's resident copy of the requests' block tables (a row per state slot) and the step's view of it.  `updates`
// (from the host runtime's packer): a count, then triples (slot, logical page, page id).  CTA s brings the row of
// sequence s up to date (the triples of its slot; two sequences of one request write the same values) and copies its
// first max_blocks entries into the step's table, the sink page beyond the row's width.  LitInfer builds and uploads a
// table per layer and step (src/llaisys/models/qwen2.cpp:993-1003); here a step uploads what changed.
namespace {
__global__ void table_gather_kernel(int* __restrict__ resident, int rows, int cols, const int* __restrict__ updates, int update_cap,
                                    const int* __restrict__ slots, int* __restrict__ out, int max_blocks, int trash_page) {
    const int s = blockIdx.x;
    int slot = slots[s];
    if (slot < 0 || slot >= rows) slot = rows - 1;                  // the last row is never written: all sink page
    int n = updates[0];
    if (n > update_cap) n = update_cap;
    int* row = resident + (size_t)slot * cols;
    if (slot != rows - 1)
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const int* u = updates + 1 + 3 * i;
            if (u[0] == slot && u[1] >= 0 && u[1] < cols) row[u[1]] = u[2];
        }
    __syncthreads();
    for (int b = threadIdx.x; b < max_blocks; b += blockDim.x) out[(size_t)s * max_blocks + b] = b < cols ? row[b] : trash_page;
}
}  // namespace

LI_EXPORT int li_table_gather(int* resident, int rows, int cols, const int* updates, int update_cap, const int* slots, int* out, int S,
                              int max_blocks, int trash_page, cudaStream_t stream) {
    LI_REQUIRE(rows >= 1 && cols >= 1 && S >= 0 && max_blocks >= 1 && update_cap >= 0, "table_gather: bad sizes rows=%d cols=%d S=%d max_blocks=%d cap=%d",
               rows, cols, S, max_blocks, update_cap);
    if (S == 0) return 0;
    table_gather_kernel<<<S, 128, 0, stream>>>(resident, rows, cols, updates, update_cap, slots, out, max_blocks, trash_page);
    return li_check_launch("table_gather");
}

// x *= factor (an embedding scale) and x = cap * tanh(x / cap) (a cap on the logits), in place on float32.
namespace {
__global__ void scale_kernel(float* __restrict__ x, long long n, float factor) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] *= factor;
}
__global__ void logit_cap_kernel(float* __restrict__ x, long long n, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) x[i] = cap * tanhf(x[i] / cap);
}
}  // namespace

namespace {
// out[r, :] = src[rows[r], :] for float rows (the wanted logits out of a captured step's fixed layout)
__global__ void gather_rows_kernel(const float* __restrict__ src, const int* __restrict__ rows, float* __restrict__ out, int n_src, long long width) {
    pdl_launch_dependents();
    pdl_wait();
    int r = rows[blockIdx.y];
    r = r < 0 ? 0 : (r >= n_src ? n_src - 1 : r);          // validated on the host; never read outside the source
    const float* s = src + (size_t)r * width;
    float* o = out + (size_t)blockIdx.y * width;
    for (long long j = (long long)blockIdx.x * blockDim.x + threadIdx.x; j < width; j += (long long)gridDim.x * blockDim.x) o[j] = s[j];
}
}  // namespace

LI_EXPORT int li_gather_rows(const float* src, const int* rows, float* out, int n_src, int n_rows, long long width, cudaStream_t stream) {
    LI_REQUIRE(n_src >= 1 && n_rows >= 0 && n_rows <= 65535 && width >= 1, "gather_rows: bad sizes (%d source rows, %d rows, width %lld)", n_src, n_rows, width);
    if (n_rows == 0) return 0;
    const unsigned bx = (unsigned)((width + 1023) / 1024 < 64 ? (width + 1023) / 1024 : 64);
    li_launch_pdl(gather_rows_kernel, dim3(bx, n_rows), dim3(256), 0, stream, src, rows, out, n_src, width);
    return li_check_launch("gather_rows");
}

LI_EXPORT int li_scale_inplace(float* x, long long n, float factor, cudaStream_t stream) {
    LI_REQUIRE(n >= 0 && n <= (1LL << 40), "scale: bad size %lld", n);
    if (n == 0) return 0;
    li_launch_pdl(scale_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, x, n, factor);
    return li_check_launch("scale");
}

LI_EXPORT int li_logit_cap(float* x, long long n, float cap, cudaStream_t stream) {
    LI_REQUIRE(n >= 0 && n <= (1LL << 40), "logit_cap: bad size %lld", n);
    LI_REQUIRE(cap > 0.0f, "logit_cap: the cap must be positive, got %g", (double)cap);
    if (n == 0) return 0;
    li_launch_pdl(logit_cap_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, x, n, cap);
    return li_check_launch("logit_cap");
}

LI_EXPORT int li_swiglu(const void* gate_up, void* out, int dtype, int T, int I, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && I > 0, "swiglu: bad sizes T=%d I=%d", T, I);
    const long long n = (long long)T * I;
    if (n == 0) return 0;
    if (dtype == LI_F32)
        swiglu_kernel<float><<<grid_for(n, 256), 256, 0, stream>>>((const float*)gate_up, (float*)out, I, n);
    else if (dtype == LI_BF16)
        swiglu_kernel<bf16><<<grid_for(n, 256), 256, 0, stream>>>((const bf16*)gate_up, (bf16*)out, I, n);
    else
        return li_fail("swiglu: unknown dtype %d", dtype);
    return li_check_launch("swiglu");
}

// out = sa * a + sb * b over n elements of the run dtype, the sum in float.
namespace {
template <typename T>
__global__ void weighted_sum2_kernel(const T* __restrict__ a, const T* __restrict__ b, float sa, float sb, T* __restrict__ out, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < n; i += stride) out[i] = from_float<T>(fmaf(sa, to_float(a[i]), sb * to_float(b[i])));
}
}  // namespace

LI_EXPORT int li_weighted_sum2(const void* a, const void* b, float sa, float sb, void* out, int dtype, long long n, cudaStream_t stream) {
    if (n == 0) return 0;
    if (dtype == LI_F32)
        weighted_sum2_kernel<float><<<grid_for(n, 256), 256, 0, stream>>>((const float*)a, (const float*)b, sa, sb, (float*)out, n);
    else if (dtype == LI_BF16)
        weighted_sum2_kernel<bf16><<<grid_for(n, 256), 256, 0, stream>>>((const bf16*)a, (const bf16*)b, sa, sb, (bf16*)out, n);
    else
        return li_fail("weighted_sum2: unknown dtype %d", dtype);
    return li_check_launch("weighted_sum2");
}

// A gated unit with bounded operands: g = min(gate, limit), u = clamp(up, -limit, limit),
// out = g / (1 + exp(-alpha g)) * (u + 1); gate_up [T, 2 I] as gate | up.  Float arithmetic, one rounding.
namespace {
template <typename T>
__global__ void glu_clamped_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int I, long long n, float limit, float alpha) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < n; i += stride) {
        const long long t = i / I;
        const int j = (int)(i - t * I);
        const float g = fminf(to_float(gate_up[t * 2 * I + j]), limit);
        const float u = fminf(fmaxf(to_float(gate_up[t * 2 * I + I + j]), -limit), limit);
        out[i] = from_float<T>(g / (1.0f + expf(-alpha * g)) * (u + 1.0f));
    }
}
}  // namespace

LI_EXPORT int li_glu_clamped(const void* gate_up, void* out, int dtype, int T, int I, float limit, float alpha, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && I > 0, "glu_clamped: bad sizes T=%d I=%d", T, I);
    const long long n = (long long)T * I;
    if (n == 0) return 0;
    if (dtype == LI_F32)
        glu_clamped_kernel<float><<<grid_for(n, 256), 256, 0, stream>>>((const float*)gate_up, (float*)out, I, n, limit, alpha);
    else if (dtype == LI_BF16)
        glu_clamped_kernel<bf16><<<grid_for(n, 256), 256, 0, stream>>>((const bf16*)gate_up, (bf16*)out, I, n, limit, alpha);
    else
        return li_fail("glu_clamped: unknown dtype %d", dtype);
    return li_check_launch("glu_clamped");
}

// up * gelu(gate), the tanh form; gate_up [T, 2 I] as gate | up.  Float arithmetic, one rounding.
namespace {
template <typename T>
__global__ void geglu_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int I, long long n) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < n; i += stride) {
        const long long t = i / I;
        const int j = (int)(i - t * I);
        out[i] = from_float<T>(geglu_of<T>(to_float(gate_up[t * 2 * I + j]), to_float(gate_up[t * 2 * I + I + j])));
    }
}
}  // namespace

LI_EXPORT int li_geglu(const void* gate_up, void* out, int dtype, int T, int I, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && I > 0, "geglu: bad sizes T=%d I=%d", T, I);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "geglu: unknown dtype %d", dtype);
    const long long n = (long long)T * I;
    if (n == 0) return 0;
    cudaError_t e;
    if (dtype == LI_F32) e = li_launch_pdl(geglu_kernel<float>, dim3(grid_for(n, 256)), dim3(256), 0, stream, (const float*)gate_up, (float*)out, I, n);
    else e = li_launch_pdl(geglu_kernel<bf16>, dim3(grid_for(n, 256)), dim3(256), 0, stream, (const bf16*)gate_up, (bf16*)out, I, n);
    if (e != cudaSuccess) return li_fail("geglu: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("geglu");
}

// A gate that opens a token's row of a table: out[t, i] = gelu(z[t, i]) * table[ids[t], col + i], the tanh form of gelu.  z float
// (a product's sums as they are), table and out in the run dtype; float arithmetic, one rounding.
namespace {
template <typename T>
__global__ void gelu_token_rows_kernel(const float* __restrict__ z, const T* __restrict__ table, long long ld, int col, int rows, const int* __restrict__ ids,
                                       T* __restrict__ out, int n, long long total) {
    pdl_launch_dependents();
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const long long t = i / n;
    int id = ids[t];
    if (id < 0 || id >= rows) id = 0;                  // validated on the host; keep the read inside the table
    out[i] = from_float<T>(geglu_of<T>(z[i], to_float(table[id * ld + col + (int)(i - t * n)])));
}
}  // namespace

LI_EXPORT int li_gelu_token_rows(const float* z, const void* table, int dtype, long long ld, int col, int rows, const int* ids, void* out, int T, int n,
                                 cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && n > 0 && rows > 0 && col >= 0 && col + n <= ld, "gelu_token_rows: columns %d .. %d of rows of %lld", col, col + n, ld);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "gelu_token_rows: unknown dtype %d", dtype);
    if (T == 0) return 0;
    const long long total = (long long)T * n;
    const dim3 grid((unsigned)ceil_div_ll(total, 128));
    cudaError_t e;
    if (dtype == LI_F32)
        e = li_launch_pdl(gelu_token_rows_kernel<float>, grid, dim3(128), 0, stream, z, (const float*)table, ld, col, rows, ids, (float*)out, n, total);
    else
        e = li_launch_pdl(gelu_token_rows_kernel<bf16>, grid, dim3(128), 0, stream, z, (const bf16*)table, ld, col, rows, ids, (bf16*)out, n, total);
    if (e != cudaSuccess) return li_fail("gelu_token_rows: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("gelu_token_rows");
}

// The gate's product and the opening of the row as one kernel, for few tokens: out[t, i] = gelu(x[t] . w[i]) * table[ids[t], col + i], a
// block per column i, eight tokens at a time, 16-byte loads, float sums.
namespace {
template <typename T>
__device__ __forceinline__ void unpack16(float (&v)[16 / sizeof(T)], uint4 u) {
    const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
        if constexpr (sizeof(T) == 2) v[2 * k] = __uint_as_float(w[k] << 16), v[2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
        else v[k] = __uint_as_float(w[k]);
    }
}

constexpr int kGateWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kGateWarps * 32)
token_gate_kernel(const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ table, long long ld, int col, int rows, const int* __restrict__ ids,
                  T* __restrict__ out, int tokens, int H, int n) {
    constexpr int V = 16 / (int)sizeof(T), TK = 8;
    __shared__ float part[kGateWarps][TK];
    const int i = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_launch_dependents();
    const T* wr = w + (size_t)i * H;
    // the weights do not depend on the kernel before this one: asked for while that still runs
    for (int k = threadIdx.x * (128 / (int)sizeof(T)); k < H; k += kGateWarps * 32 * (128 / (int)sizeof(T))) asm volatile("prefetch.global.L2 [%0];" ::"l"(wr + k));
    pdl_wait();
    for (int t0 = 0; t0 < tokens; t0 += TK) {
        float acc[TK];
#pragma unroll
        for (int j = 0; j < TK; ++j) acc[j] = 0.0f;
        for (int k = V * threadIdx.x; k < H; k += kGateWarps * 32 * V) {
            const uint4 wu = __ldg(reinterpret_cast<const uint4*>(wr + k));
            uint4 xu[TK];
#pragma unroll
            for (int j = 0; j < TK; ++j) xu[j] = *reinterpret_cast<const uint4*>(x + (size_t)min(t0 + j, tokens - 1) * H + k);
            float wv[V];
            unpack16<T>(wv, wu);
#pragma unroll
            for (int j = 0; j < TK; ++j) {
                float xv[V];
                unpack16<T>(xv, xu[j]);
#pragma unroll
                for (int q = 0; q < V; ++q) acc[j] = fmaf(xv[q], wv[q], acc[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < TK; ++j) {
            const float z = warp_sum(acc[j]);
            if (lane == j) part[warp][j] = z;
        }
        __syncthreads();
        if (threadIdx.x < TK && t0 + (int)threadIdx.x < tokens) {
            const int t = t0 + threadIdx.x;
            float z = 0.0f;
#pragma unroll
            for (int p = 0; p < kGateWarps; ++p) z += part[p][threadIdx.x];
            int id = ids[t];
            if (id < 0 || id >= rows) id = 0;
            out[(size_t)t * n + i] = from_float<T>(geglu_of<T>(z, to_float(table[id * ld + col + i])));
        }
        __syncthreads();
    }
}
}  // namespace

LI_EXPORT int li_token_gate_accepts(int dtype, int T, int H) { return (T >= 1 && T <= 16 && H > 0 && H % (dtype == LI_F32 ? 4 : 8) == 0) ? 1 : 0; }

LI_EXPORT int li_token_gate(const void* x, const void* w, const void* table, int dtype, long long ld, int col, int rows, const int* ids, void* out, int T, int H,
                            int n, cudaStream_t stream) {
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "token_gate: unknown dtype %d", dtype);
    LI_REQUIRE(li_token_gate_accepts(dtype, T, H) && ((uintptr_t)x % 16) == 0 && ((uintptr_t)w % 16) == 0, "token_gate: refuses %d tokens of %d", T, H);
    LI_REQUIRE(n > 0 && rows > 0 && col >= 0 && col + n <= ld, "token_gate: columns %d .. %d of rows of %lld", col, col + n, ld);
    const dim3 grid(n);
    const cudaError_t e = dtype == LI_F32
        ? li_launch_pdl(token_gate_kernel<float>, grid, dim3(kGateWarps * 32), 0, stream, (const float*)x, (const float*)w, (const float*)table, ld, col, rows, ids, (float*)out, T, H, n)
        : li_launch_pdl(token_gate_kernel<bf16>, grid, dim3(kGateWarps * 32), 0, stream, (const bf16*)x, (const bf16*)w, (const bf16*)table, ld, col, rows, ids, (bf16*)out, T, H, n);
    if (e != cudaSuccess) return li_fail("token_gate: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("token_gate");
}

// PolyNorm and a sigmoid gate.
//   li_polynorm: per token row z [n]: out = a N(z) + b N(z^2) + c N(z^3) + e with powers element by element and
//     N(v) = v / sqrt(mean(v^2) + eps); coef = {a, b, c, e} float on the device.  The three means are taken in one pass (the row
//     in registers up to 16,384 elements, else read again), everything in float, one rounding.
//   li_mul_sigmoid: x[t, i] *= sigmoid(gate[t, gate_off + i / group]) in float, one rounding (an output gate per element, or
//     with group = a head's width one per head).
namespace {
constexpr int kPolyRegs = 16;

template <typename T>
__global__ void polynorm_kernel(const T* __restrict__ z, const float* __restrict__ coef, float eps, T* __restrict__ out, int n) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const T* row = z + (size_t)blockIdx.x * n;
    T* dst = out + (size_t)blockIdx.x * n;
    const bool held = n <= kPolyRegs * (int)blockDim.x;
    float v[kPolyRegs];
    float s2 = 0.0f, s4 = 0.0f, s6 = 0.0f;
    if (held) {
#pragma unroll
        for (int k = 0; k < kPolyRegs; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            v[k] = i < n ? to_float(row[i]) : 0.0f;
            const float p2 = v[k] * v[k];
            s2 += p2; s4 = fmaf(p2, p2, s4); s6 = fmaf(p2 * p2, p2, s6);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const float x = to_float(row[i]), p2 = x * x;
            s2 += p2; s4 = fmaf(p2, p2, s4); s6 = fmaf(p2 * p2, p2, s6);
        }
    }
    s2 = block_sum(s2, scratch); s4 = block_sum(s4, scratch); s6 = block_sum(s6, scratch);
    const float inv_n = 1.0f / (float)n;
    const float a = coef[0] / sqrtf(s2 * inv_n + eps), b = coef[1] / sqrtf(s4 * inv_n + eps), c = coef[2] / sqrtf(s6 * inv_n + eps), e = coef[3];
    if (held) {
#pragma unroll
        for (int k = 0; k < kPolyRegs; ++k) {
            const int i = threadIdx.x + k * blockDim.x;
            if (i < n) dst[i] = from_float<T>(fmaf(v[k], fmaf(v[k], fmaf(v[k], c, b), a), e));
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const float x = to_float(row[i]);
            dst[i] = from_float<T>(fmaf(x, fmaf(x, fmaf(x, c, b), a), e));
        }
    }
}

template <typename T>
__global__ void mul_sigmoid_kernel(T* __restrict__ x, const T* __restrict__ gate, int gate_stride, int gate_off, int group, int n, long long total) {
    pdl_launch_dependents();
    pdl_wait();
    long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (; i < total; i += stride) {
        const long long t = i / n;
        const int j = (int)(i - t * n);
        const float g = to_float(gate[t * gate_stride + gate_off + j / group]);
        x[i] = from_float<T>(to_float(x[i]) / (1.0f + expf(-g)));
    }
}
}  // namespace

LI_EXPORT int li_polynorm(const void* z, int dtype, const float* coef, float eps, void* out, int T, int n, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && n > 0 && coef != nullptr, "polynorm: bad sizes T=%d n=%d", T, n);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "polynorm: unknown dtype %d", dtype);
    if (T == 0) return 0;
    int threads = ((ceil_div(n, kPolyRegs) + 31) / 32) * 32;
    threads = threads < 64 ? 64 : threads > 1024 ? 1024 : threads;
    cudaError_t e;
    if (dtype == LI_F32) e = li_launch_pdl(polynorm_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)z, coef, eps, (float*)out, n);
    else e = li_launch_pdl(polynorm_kernel<bf16>, dim3(T), dim3(threads), 0, stream, (const bf16*)z, coef, eps, (bf16*)out, n);
    if (e != cudaSuccess) return li_fail("polynorm: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("polynorm");
}

LI_EXPORT int li_mul_sigmoid(void* x, const void* gate, int dtype, int gate_stride, int gate_off, int group, int T, int n, cudaStream_t stream) {
    LI_REQUIRE(T >= 0 && n > 0 && group > 0 && n % group == 0 && gate_off >= 0 && gate_off + n / group <= gate_stride, "mul_sigmoid: bad sizes T=%d n=%d (gate at %d of %d)", T, n, gate_off, gate_stride);
    LI_REQUIRE(dtype == LI_F32 || dtype == LI_BF16, "mul_sigmoid: unknown dtype %d", dtype);
    const long long total = (long long)T * n;
    if (total == 0) return 0;
    cudaError_t e;
    if (dtype == LI_F32) e = li_launch_pdl(mul_sigmoid_kernel<float>, dim3(grid_for(total, 256)), dim3(256), 0, stream, (float*)x, (const float*)gate, gate_stride, gate_off, group, n, total);
    else e = li_launch_pdl(mul_sigmoid_kernel<bf16>, dim3(grid_for(total, 256)), dim3(256), 0, stream, (bf16*)x, (const bf16*)gate, gate_stride, gate_off, group, n, total);
    if (e != cudaSuccess) return li_fail("mul_sigmoid: launch failed: %s", cudaGetErrorString(e));
    return li_check_launch("mul_sigmoid");
}

// out[tok, :] = hprime[tok, :] / sqrt(sum of ssq[:, tok] / width + eps): the normalised activation itself, for a
// consumer that cannot take the factor into its own product (row_scale.cuh).  bfloat16.
namespace {
__global__ void apply_row_scale_kernel(const bf16* __restrict__ hprime, const float* __restrict__ ssq, int nparts, float width, float eps,
                                       bf16* __restrict__ out, int M, int H) {
    __shared__ float factor;
    pdl_launch_dependents();
    pdl_wait();
    const int tok = blockIdx.x;
    if (threadIdx.x < 32) {
        float s = 0.0f;
        for (int p = threadIdx.x; p < nparts; p += 32) s += ssq[(size_t)tok * nparts + p];
        s = warp_sum(s);
        if (threadIdx.x == 0) factor = 1.0f / sqrtf(s / width + eps);
    }
    __syncthreads();
    const float f = factor;
    for (int j = threadIdx.x; j < H; j += blockDim.x) out[(size_t)tok * H + j] = __float2bfloat16_rn(__bfloat162float(hprime[(size_t)tok * H + j]) * f);
}
}  // namespace

LI_EXPORT int li_apply_row_scale(const void* hprime, const float* ssq, int nparts, int width, float eps, void* out, int M, int H,
                                 cudaStream_t stream) {
    LI_REQUIRE(M >= 0 && H > 0 && nparts >= 1 && width >= 1, "apply_row_scale: bad sizes M=%d H=%d parts=%d width=%d", M, H, nparts, width);
    if (M == 0) return 0;
    li_launch_pdl(apply_row_scale_kernel, dim3(M), dim3(256), 0, stream, (const bf16*)hprime, ssq, nparts, (float)width, eps, (bf16*)out, M, H);
    return li_check_launch("apply_row_scale");
}
