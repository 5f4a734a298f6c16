// Causal grouped-query attention of a ragged batch over the paged cache:
// the general kernel.  It serves the true 32-bit path for every batch shape
// and is the fall-back of the bfloat16 path for head sizes the tensor-core
// kernels refuse.
//
// One warp per (token, query head).  The token at position p of sequence s
// reads keys lo..p of s with lo = max(0, p - window + 1) (window 0: lo = 0),
// one key after the other in ascending order, with the online-softmax
// recurrence of LitInfer's kernel (src/ops/paged_attention/op.cpp:194-234):
//   m' = max(m, s_t); alpha = exp(m - m'); e = exp(s_t - m');
//   l = l alpha + e;  acc = acc alpha + e v_t;  out = acc / l.
// Scores, exponentials, sums and the weighted values are float.  The order of
// the keys and of the lanes' partial sums is fixed, so a token's output does
// not depend on what else is in the batch or on how its sequence was cut.
//
// Cache layout: keys [page][kv_head][offset][head_dim], values transposed
// [page][kv_head][head_dim][offset]; the page of key t of sequence s is
// block_table[s][t / page_size].  Any head_dim up to 512.
//
// Optional changes of the scores and the output (all off when zero / null):
//   softcap > 0:  s <- softcap * tanh(s / softcap) after the scale;
//   slopes [nh]:  s <- s - slopes[h] * (p - key), a penalty linear in the distance;
//   gate:         the head's output is multiplied by 1 / (1 + exp(-g)), g one number a head or one an output element.
// Optional changes of what is seen and of the softmax's denominator:
//   chunk > 0:    keys below p - p % chunk are not seen (p sees its own chunk only);
//   keep_first > 0 (with a window): keys 0 .. keep_first - 1 stay visible behind the window, at their own positions;
//   sinks [nh]:   exp(sinks[h]) joins the denominator of head h once; it has no key and no value and is not scaled.
// maps > 1: a query row of head_dim elements stands for `maps` heads (attention_mma.cuh: ScoreMod); qkv then holds nh / maps of them.
#include "attention_options.h"
#include "common.cuh"

namespace {

constexpr int kWarpsPerBlock = 4;
constexpr int kMaxPerLane = 16;       // head_dim <= 512

template <typename T>
__global__ void __launch_bounds__(kWarpsPerBlock * 32)
attention_generic_kernel(const T* __restrict__ qkv, T* __restrict__ out, const T* __restrict__ kcache, const T* __restrict__ vcache,
                         const int* __restrict__ block_table, int max_blocks, const int* __restrict__ seq_of_token,
                         const int* __restrict__ positions, int total, int nh, int nkv, int dh, int page_size, int num_pages,
                         float scale, int window, AttentionOptions opt) {
    const int warp = blockIdx.x * kWarpsPerBlock + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (warp >= total) return;
    const int t = warp / nh, h = warp - t * nh;
    const int kvh = h / (nh / nkv);
    const int s = seq_of_token[t];
    const int p = positions[t];
    const int lo = first_seen_key(p, window, opt.chunk), maps = opt.maps;
    const size_t row = opt.q_ld > 0 ? opt.q_ld : (nh / maps + 2 * nkv) * dh;
    const T* q = qkv + t * row + (h / maps) * dh;
    const int per = (dh + 31) >> 5;
    const int part = dh / maps, part_lo = (h % maps) * part, part_hi = part_lo + part;

    float qr[kMaxPerLane], acc[kMaxPerLane];
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
        const int d = lane + 32 * i;
        qr[i] = (i < per && d >= part_lo && d < part_hi) ? to_float(q[d]) : 0.0f;
        acc[i] = 0.0f;
    }
    float m = -INFINITY, l = 0.0f;
    const float slope = opt.slopes ? opt.slopes[h] : 0.0f, softcap = opt.softcap;
    const int keep_first = window > 0 ? opt.keep_first : 0;
    const int* bt = block_table + (size_t)s * max_blocks;
    // the kept first keys that lie behind the window come first, then the window: ascending order either way
    const int kept = keep_first < lo ? keep_first : lo;
    for (int key = kept > 0 ? 0 : lo; key <= p; ++key) {
        if (key == kept && key < lo) key = lo;
        const int lb = key / page_size;
        int page = bt[lb];
        if (page < 0 || page >= num_pages) page = 0;      // host-validated; keep the read inside the cache
        const int off = key - lb * page_size;
        const size_t base = (((size_t)page * nkv + kvh) * page_size + off) * dh;
        const size_t vbase = ((size_t)page * nkv + kvh) * dh * page_size + off;
        float dot = 0.0f;
#pragma unroll
        for (int i = 0; i < kMaxPerLane; ++i) {
            const int d = lane + 32 * i;
            if (i < per && d >= part_lo && d < part_hi) dot = fmaf(qr[i], to_float(kcache[base + d]), dot);
        }
        float sc = warp_sum(dot) * scale;
        if (softcap > 0.0f) sc = softcap * tanhf(sc / softcap);
        sc -= slope * (float)(p - key);
        const float mn = fmaxf(m, sc);
        const float alpha = expf(m - mn);
        const float e = expf(sc - mn);
        l = l * alpha + e;
#pragma unroll
        for (int i = 0; i < kMaxPerLane; ++i) {
            const int d = lane + 32 * i;
            if (i < per && d < dh) acc[i] = acc[i] * alpha + e * to_float(vcache[vbase + (size_t)d * page_size]);
        }
        m = mn;
    }
    T* o = out + (size_t)t * nh * dh + h * dh;
    if (opt.sinks) {
        const float sk = opt.sinks[h];
        const float mn = fmaxf(m, sk);
        const float alpha = expf(m - mn);
        l = l * alpha + expf(sk - mn);
#pragma unroll
        for (int i = 0; i < kMaxPerLane; ++i) acc[i] *= alpha;
    }
    float inv = l > 0.0f ? 1.0f / l : 0.0f;
    const T* gate = opt.gate ? (const T*)opt.gate + (size_t)t * opt.gate_ld : nullptr;
    if (gate && !opt.gate_elements) inv *= 1.0f / (1.0f + expf(-to_float(gate[h])));
#pragma unroll
    for (int i = 0; i < kMaxPerLane; ++i) {
        const int d = lane + 32 * i;
        if (i < per && d < dh) {
            float r = acc[i] * inv;
            if (gate && opt.gate_elements) r *= 1.0f / (1.0f + expf(-to_float(gate[(size_t)h * dh + d])));
            o[d] = from_float<T>(r);
        }
    }
}

}  // namespace

int li_attention_generic(const void* qkv, void* out, const void* kcache, const void* vcache, int dtype, const int* block_table,
                         int max_blocks, const int* seq_of_token, const int* positions, int T, int nh, int nkv, int dh,
                         int page_size, int num_pages, float scale, int window, const AttentionOptions& opt, cudaStream_t stream) {
    LI_REQUIRE(dh <= 32 * kMaxPerLane, "attention: head_dim %d is larger than %d", dh, 32 * kMaxPerLane);
    const long long total = (long long)T * nh;
    LI_REQUIRE(total < (1LL << 31), "attention: too many (token, head) pairs");
    const int blocks = (int)ceil_div_ll(total, kWarpsPerBlock);
    if (dtype == LI_F32)
        attention_generic_kernel<float><<<blocks, kWarpsPerBlock * 32, 0, stream>>>(
            (const float*)qkv, (float*)out, (const float*)kcache, (const float*)vcache, block_table, max_blocks, seq_of_token, positions,
            (int)total, nh, nkv, dh, page_size, num_pages, scale, window, opt);
    else if (dtype == LI_BF16)
        attention_generic_kernel<bf16><<<blocks, kWarpsPerBlock * 32, 0, stream>>>(
            (const bf16*)qkv, (bf16*)out, (const bf16*)kcache, (const bf16*)vcache, block_table, max_blocks, seq_of_token, positions,
            (int)total, nh, nkv, dh, page_size, num_pages, scale, window, opt);
    else
        return li_fail("attention: unknown dtype %d", dtype);
    return li_check_launch("attention (generic)");
}
