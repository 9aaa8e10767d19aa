// Device side of a block decoder's residual update and norms, shared by the norm kernels and the row product that
// has a norm in its prologue.
#pragma once
#include <cuda_bf16.h>

#include "blocks.h"
#include "decoder_common.cuh"

namespace nnq {

// One row: x = embedding rows, or alpha h_in + delta; with post_w given x <- LN(x). h_out (NULL to drop it)
// receives x. What the products read is x itself, RMSNorm(x) w or LN(x) w + b (in.kind).
struct NormRow {
    const float *h_in, *delta;          // delta NULL: alpha h_in
    float *h_out;
    const __nv_bfloat16 *e0, *e1;       // e0 given: x = e0 (+ e1)
    float alpha;
    const float *post_w, *post_b;
    InNorm in;
    float eps;
    int hidden;
};

__device__ __forceinline__ long long pair_row(const PairTable &p, int prev, int tok, int pos) {
    return pos == 0 ? p.buckets : ((long long)prev * p.mul_prev + (long long)tok * p.mul_cur) % p.buckets;
}

__device__ __forceinline__ float4 bf4(const __nv_bfloat16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xFFFF0000u));
}

// Asks L2 for the weights and biases of the norms (constants: also before the kernel in front has ended).
template <int K>
__device__ __forceinline__ void norm_prefetch(const NormRow &r) {
    const float *p[4] = {r.post_w, r.post_b, r.in.kind == kNormNone ? nullptr : r.in.w, r.in.kind == kNormLayer ? r.in.b : nullptr};
#pragma unroll
    for (int j = 0; j < 4; j++)
#pragma unroll
        for (int k = 0; k < K; k++) {
            const int i = 4 * (threadIdx.x + blockDim.x * k);
            if (p[j] && i < r.hidden && (threadIdx.x & 7) == 0) asm volatile("prefetch.global.L2 [%0];" ::"l"(p[j] + i));
        }
}

// The row as units of four elements, unit threadIdx.x + blockDim.x * k in v[k] (hidden a multiple of 4 and at most
// 4 * K * blockDim.x; units past the end are zero). Every thread of the block calls it; red: 32 floats.
template <int K>
__device__ __forceinline__ void norm_units(const NormRow &r, float4 (&v)[K], float *red) {
    const float n = (float)r.hidden;
#pragma unroll
    for (int k = 0; k < K; k++) {
        const int i = 4 * (threadIdx.x + blockDim.x * k);
        v[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (i >= r.hidden) continue;
        if (r.e0) {
            v[k] = bf4(r.e0 + i);
            if (r.e1) {
                const float4 b = bf4(r.e1 + i);
                v[k].x += b.x; v[k].y += b.y; v[k].z += b.z; v[k].w += b.w;
            }
        } else {
            const float4 a = *reinterpret_cast<const float4 *>(r.h_in + i);
            const float4 b = r.delta ? *reinterpret_cast<const float4 *>(r.delta + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            v[k] = make_float4(fmaf(r.alpha, a.x, b.x), fmaf(r.alpha, a.y, b.y), fmaf(r.alpha, a.z, b.z), fmaf(r.alpha, a.w, b.w));
        }
    }
    auto squares = [&](float m) {   // sum of the squared deviations from m
        float ss = 0.0f;
#pragma unroll
        for (int k = 0; k < K; k++) {
            if (4 * (threadIdx.x + blockDim.x * k) >= r.hidden) continue;
            const float a = v[k].x - m, b = v[k].y - m, c = v[k].z - m, d = v[k].w - m;
            ss = fmaf(a, a, fmaf(b, b, fmaf(c, c, fmaf(d, d, ss))));
        }
        return block_sum(ss, red);
    };
    auto layer_norm = [&](const float *w, const float *b) {
        float4 g[K], o[K];   // (asked for before the sums are formed)
#pragma unroll
        for (int k = 0; k < K; k++) {
            const int i = 4 * (threadIdx.x + blockDim.x * k);
            g[k] = o[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (i >= r.hidden) continue;
            g[k] = *reinterpret_cast<const float4 *>(w + i);
            o[k] = *reinterpret_cast<const float4 *>(b + i);
        }
        float s = 0.0f;
#pragma unroll
        for (int k = 0; k < K; k++) s += (v[k].x + v[k].y) + (v[k].z + v[k].w);
        const float mean = block_sum(s, red) / n;
        const float inv = 1.0f / sqrtf(squares(mean) / n + r.eps);
#pragma unroll
        for (int k = 0; k < K; k++) {
            const int i = 4 * (threadIdx.x + blockDim.x * k);
            if (i >= r.hidden) continue;
            v[k] = make_float4(fmaf((v[k].x - mean) * inv, g[k].x, o[k].x), fmaf((v[k].y - mean) * inv, g[k].y, o[k].y), fmaf((v[k].z - mean) * inv, g[k].z, o[k].z),
                               fmaf((v[k].w - mean) * inv, g[k].w, o[k].w));
        }
    };
    if (r.post_w) layer_norm(r.post_w, r.post_b);
    if (r.h_out) {
#pragma unroll
        for (int k = 0; k < K; k++) {
            const int i = 4 * (threadIdx.x + blockDim.x * k);
            if (i < r.hidden) *reinterpret_cast<float4 *>(r.h_out + i) = v[k];
        }
    }
    if (r.in.kind == kNormRms) {
        float4 g[K];
#pragma unroll
        for (int k = 0; k < K; k++) {
            const int i = 4 * (threadIdx.x + blockDim.x * k);
            g[k] = i < r.hidden ? *reinterpret_cast<const float4 *>(r.in.w + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        const float rms = sqrtf(squares(0.0f) / n + r.eps);
#pragma unroll
        for (int k = 0; k < K; k++) {
            if (4 * (threadIdx.x + blockDim.x * k) >= r.hidden) continue;
            v[k] = make_float4(v[k].x / rms * g[k].x, v[k].y / rms * g[k].y, v[k].z / rms * g[k].z, v[k].w / rms * g[k].w);
        }
    } else if (r.in.kind == kNormLayer) {
        layer_norm(r.in.w, r.in.b);
    }
}

// The same for any width, one element at a time; out(i, value) takes the elements in front of hidden.
template <typename Out>
__device__ __forceinline__ void norm_elements(const NormRow &r, float *red, Out out) {
    const float n = (float)r.hidden;
    auto x0 = [&](int i) {
        if (r.e0) return __bfloat162float(r.e0[i]) + (r.e1 ? __bfloat162float(r.e1[i]) : 0.0f);
        return fmaf(r.alpha, r.h_in[i], r.delta ? r.delta[i] : 0.0f);
    };
    auto sum = [&](auto f) {
        float s = 0.0f;
        for (int i = threadIdx.x; i < r.hidden; i += blockDim.x) s += f(i);
        return block_sum(s, red);
    };
    float m0 = 0.0f, d0 = 1.0f, m1 = 0.0f, d1 = 1.0f;
    if (r.post_w) {
        m0 = sum(x0) / n;
        d0 = sqrtf(sum([&](int i) { const float d = x0(i) - m0; return d * d; }) / n + r.eps);
    }
    auto x1 = [&](int i) { return r.post_w ? fmaf((x0(i) - m0) / d0, r.post_w[i], r.post_b[i]) : x0(i); };
    if (r.in.kind != kNormNone) {
        if (r.in.kind == kNormLayer) m1 = sum(x1) / n;
        d1 = sqrtf(sum([&](int i) { const float d = x1(i) - m1; return d * d; }) / n + r.eps);
    }
    for (int i = threadIdx.x; i < r.hidden; i += blockDim.x) {
        const float x = x1(i);
        if (r.h_out) r.h_out[i] = x;
        if (r.in.kind == kNormRms) out(i, x / d1 * r.in.w[i]);
        else if (r.in.kind == kNormLayer) out(i, fmaf((x - m1) / d1, r.in.w[i], r.in.b[i]));
        else out(i, x);
    }
}

}  // namespace nnq
