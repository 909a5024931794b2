// Shared pieces of the mixture-of-experts kernels (experts.cu, experts_tc.cu).
//
// Routing leaves the (token, choice) pairs sorted by expert: position i of the sorted order belongs to
// pair slot[i] = token * top + choice with weight scale[i]; expert e has positions [offsets[e], offsets[e + 1]).
#pragma once

#include "vec_io.cuh"

namespace nckv {

// The two products of all experts.  UP: act[i] = silu(s g) * (s u) with [g; u] = W_e h[token], s = scale[i] (the
// weight multiplies the expert's input, which for a product without bias is its output).  Otherwise
// y[slot[i]] = W_e act[i].
struct ExpertParams {
    const void *a;         // UP: h (rows, K); else act (R, K)
    const void *w;         // UP: (E, 2 N, K) gate rows, then up rows; else (E, N, K)
    void *out;             // UP: act (R, N); else y (R, N) by slot
    const int32_t *offsets, *slot;
    const float *scale;
    int32_t *status;
    int R, E, top, N, K;
};

cudaError_t experts_tc(const ExpertParams &p, bool up, cudaStream_t s, int *rc);  // tcgen05 form, many rows

}  // namespace nckv
