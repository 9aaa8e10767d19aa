// Routing of one token over a mixture of experts: softmax over the logits, the largest top_k, renormalised.
#pragma once
#include <math_constants.h>
#include <stdint.h>

namespace nnq {

constexpr int kMaxExperts = 256;
constexpr int kMaxTopK = 16;
constexpr int kLaneExperts = kMaxExperts / 32;   // logits held by a lane of the routing warp

// Softmax over the E logits of one token (lg, generic address) and top-k selection by one warp.
__device__ __forceinline__ void route_token(const float *lg, int E, int top_k, int tok, int *__restrict__ idx,
                                            float *__restrict__ wt, int lane) {
    // lane l holds the logits of experts l, l + 32, ...
    float p[kLaneExperts];
    float mx = -CUDART_INF_F;
#pragma unroll
    for (int k = 0; k < kLaneExperts; k++) {
        p[k] = -1.0f;
        if (32 * k >= E) continue;   // (the same in every lane: few experts cost few steps)
        p[k] = lane + 32 * k < E ? lg[lane + 32 * k] : -CUDART_INF_F;
        mx = fmaxf(mx, p[k]);
    }
    // softmax over the E experts (max-subtracted, f32)
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
    float sum = 0.0f;
#pragma unroll
    for (int k = 0; k < kLaneExperts; k++) {
        if (32 * k >= E) continue;
        p[k] = lane + 32 * k < E ? expf(p[k] - mx) : 0.0f;
        sum += p[k];
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, off);
#pragma unroll
    for (int k = 0; k < kLaneExperts; k++)
        if (32 * k < E) p[k] = lane + 32 * k < E ? p[k] / sum : -1.0f;
    // top-k: k rounds of (largest probability, lowest index) selection
    float sel_p = 0.0f, wsum = 0.0f;
    int sel_e = 0;
    for (int s = 0; s < top_k; s++) {
        float best = p[0];
        int be = lane;
#pragma unroll
        for (int k = 1; k < kLaneExperts; k++)
            if (32 * k < E && p[k] > best) {
                best = p[k];
                be = lane + 32 * k;
            }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) {
            float ob = __shfl_xor_sync(0xFFFFFFFFu, best, off);
            int oe = __shfl_xor_sync(0xFFFFFFFFu, be, off);
            if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
        }
#pragma unroll
        for (int k = 0; k < kLaneExperts; k++)
            if (be == lane + 32 * k) p[k] = -1.0f;
        if (lane == s) { sel_p = best; sel_e = be; }
        wsum += best;
    }
    if (lane < top_k) {
        idx[(int64_t)tok * top_k + lane] = sel_e;
        wt[(int64_t)tok * top_k + lane] = sel_p / wsum;
    }
}

}  // namespace nnq
