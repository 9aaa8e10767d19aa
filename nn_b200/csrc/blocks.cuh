// Device side of blocks.h shared by the mixer kernels.
#pragma once
#include "blocks.h"
#include "decoder_common.cuh"

namespace nnq {

__device__ __forceinline__ int span_pos(const RowSpan &s) { return s.state ? s.state[1] : s.pos0; }

// CTAs [first, gridDim.x) of a launch cover the act columns right of the mixer's, 16 bytes per thread and
// turn where the segment allows it
__device__ __forceinline__ void ffn_part(const FfnPart &f, int n, int first) {
    const int cols = f.out_k - f.mix;
    const long long total = (long long)n * cols;
    const long long step = (long long)(gridDim.x - first) * blockDim.x;
    for (long long i = (long long)(blockIdx.x - first) * blockDim.x + threadIdx.x; i < total; i += step) {
        const int row = (int)(i / cols), c = f.mix + (int)(i - (long long)row * cols);
        const int j = c - f.c_ffn;
        float v = 0.0f;
        if (j >= 0 && j < f.ffn) {
            const float *p = f.proj + (size_t)row * f.in_cols;
            v = silu_f32(p[f.c_gate + j]) * p[f.c_up + j];
        }
        store_act(f.act, f.act_dt, (size_t)row * f.out_k + c, v);
    }
}

inline int ffn_ctas(const FfnPart &f, int n, int threads, int sm_count) {
    const long long total = (long long)n * (f.out_k - f.mix);
    const long long want = (total + 4LL * threads - 1) / (4LL * threads);
    return (int)(want < 8LL * sm_count ? want : 8LL * sm_count);
}

// half-split rotation of dimension d of a vector held at x (any address space); cs / sn: this position's row
__device__ __forceinline__ float rotated(const float *x, int d, int rot, const float *cs, const float *sn) {
    const int half = rot >> 1;
    if (d >= rot) return x[d];
    if (d < half) return x[d] * cs[d] - x[d + half] * sn[d];
    const int i = d - half;
    return x[d] * cs[i] + x[i] * sn[i];
}

}  // namespace nnq
