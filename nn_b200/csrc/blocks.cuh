// Device side of blocks.h shared by the mixer kernels.
#pragma once
#include "blocks.h"
#include "decoder_common.cuh"

namespace nnq {

__device__ __forceinline__ int span_pos(const RowSpan &s) { return s.state ? s.state[1] : s.pos0; }

// bf16 results are rounded to eight bits anyway: the fast exponential and division are enough for them
template <bool FAST>
__device__ __forceinline__ float silu_act(float x) { return FAST ? __fdividef(x, 1.0f + __expf(-x)) : silu_f32(x); }

// eight columns of the feed-forward activation from column j on; columns past its width are zero
template <bool FAST>
__device__ __forceinline__ void ffn_eight(const FfnPart &f, const float *p, int j, float *v) {
    const float *g = p + f.c_gate + j, *u = p + f.c_up + j;
    if (j + 8 <= f.ffn) {
        const float4 g0 = reinterpret_cast<const float4 *>(g)[0], g1 = reinterpret_cast<const float4 *>(g)[1];
        const float4 u0 = reinterpret_cast<const float4 *>(u)[0], u1 = reinterpret_cast<const float4 *>(u)[1];
        v[0] = silu_act<FAST>(g0.x) * u0.x; v[1] = silu_act<FAST>(g0.y) * u0.y; v[2] = silu_act<FAST>(g0.z) * u0.z; v[3] = silu_act<FAST>(g0.w) * u0.w;
        v[4] = silu_act<FAST>(g1.x) * u1.x; v[5] = silu_act<FAST>(g1.y) * u1.y; v[6] = silu_act<FAST>(g1.z) * u1.z; v[7] = silu_act<FAST>(g1.w) * u1.w;
    } else {
#pragma unroll
        for (int i = 0; i < 8; i++) v[i] = j + i < f.ffn ? silu_act<FAST>(g[i]) * u[i] : 0.0f;
    }
}

// CTAs [first, gridDim.x) of a launch cover the act columns right of the mixer's, eight columns per thread and
// turn (all segments start at multiples of eight columns, rows are multiples of 64)
__device__ __forceinline__ void ffn_part(const FfnPart &f, int n, int first) {
    const unsigned units = (unsigned)(f.out_k - f.c_ffn) >> 3, total = n * units;
    const unsigned step = (gridDim.x - first) * blockDim.x;
    for (unsigned i = (blockIdx.x - first) * blockDim.x + threadIdx.x; i < total; i += step) {
        const unsigned row = i / units, j = (i - row * units) * 8;
        const float *p = f.proj + (size_t)row * f.in_cols;
        const size_t at = (size_t)row * f.out_k + f.c_ffn + j;
        float v[8];
        if (f.act_dt == NNQ_F32) {
            ffn_eight<false>(f, p, j, v);
            float4 *d = reinterpret_cast<float4 *>(reinterpret_cast<float *>(f.act) + at);
            d[0] = make_float4(v[0], v[1], v[2], v[3]);
            d[1] = make_float4(v[4], v[5], v[6], v[7]);
        } else {
            ffn_eight<true>(f, p, j, v);
            uint32_t q[4];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
                q[k] = *reinterpret_cast<const uint32_t *>(&b);
            }
            *reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(f.act) + at) = make_uint4(q[0], q[1], q[2], q[3]);
        }
        if (j == 0)   // the gap between the mixer's columns and the feed-forward's
            for (int c = f.mix; c < f.c_ffn; c++) store_act(f.act, f.act_dt, (size_t)row * f.out_k + c, 0.0f);
    }
}

inline int ffn_ctas(const FfnPart &f, int n, int threads, int sm_count) {
    const long long total = (long long)n * ((f.out_k - f.c_ffn) >> 3);
    const long long want = (total + threads - 1) / threads;
    return (int)(want < 16LL * sm_count ? want : 16LL * sm_count);
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
