// What may change attention over the paged cache, as one bundle that the launchers hand on.  Everything is off by default.
#pragma once

struct AttentionOptions {
    float softcap = 0.0f;            // > 0: a score s becomes softcap * tanh(s / softcap), after the scale
    const float* slopes = nullptr;   // [heads]: slopes[h] * (p - key) is taken off
    const void* gate = nullptr;      // run dtype: the output is multiplied by its sigmoid, one number a head (gate[t gate_ld + h]) ...
    long long gate_ld = 0;
    int gate_elements = 0;           // ... or one an output element (gate[t gate_ld + h dh + d])
    int keep_first = 0;              // with a window: these first keys stay visible behind it
    const float* sinks = nullptr;    // [heads]: exp(sinks[h]) joins the denominator
    int maps = 1;                    // heads that a query row stands for
    int chunk = 0;                   // > 0: position p sees keys of its own chunk only, those from p - p % chunk on
    int q_ld = 0;                    // elements of a row of the queries' tensor (0: q|k|v rows)
};

// The first key that a query at position p sees behind the kept ones: of the last `window`, of its own chunk (0: no bound).
#ifdef __CUDACC__
__host__ __device__
#endif
inline int first_seen_key(int p, int window, int chunk) {
    int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
    if (chunk > 0 && p >= chunk) {
        const int c = p - p % chunk;
        lo = lo > c ? lo : c;
    }
    return lo;
}
