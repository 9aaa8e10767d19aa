// Residual add + RMSNorm of a block decoder, for the row of a decode step and for a block of rows. The normed
// rows may be wider than the model (zero columns up to the products' k step).
#include "blocks.h"
#include "decoder_common.cuh"

namespace nnq {

// h = embedding row of the current token, or h += delta; xn = RMSNorm(h) * w, zeros from hidden to xn_ld.
// One CTA; every thread keeps its (up to 8) elements in registers between the two phases.
__global__ void __launch_bounds__(1024)
norm_step_kernel(float *__restrict__ h, const float *__restrict__ delta, const __nv_bfloat16 *__restrict__ embed,
                 const int *__restrict__ state, const float *__restrict__ w, float eps, void *__restrict__ xn, int act_dt,
                 int hidden, int embed_ld, int xn_ld) {
    pdl_prologue();
    pdl_release();
    __shared__ float red[32];
    const int tok = embed ? state[0] : 0;
    float v[8], wv[8];
    float ss = 0.0f;
#pragma unroll
    for (int r = 0; r < 8; r++) {
        const int i = threadIdx.x + r * 1024;
        v[r] = 0.0f;
        wv[r] = 0.0f;
        if (i < hidden) {
            v[r] = embed ? __bfloat162float(embed[(size_t)tok * embed_ld + i]) : h[i] + delta[i];
            wv[r] = w[i];
            h[i] = v[r];
            ss = fmaf(v[r], v[r], ss);
        }
    }
    for (int i = threadIdx.x + 8 * 1024; i < hidden; i += 1024) {   // wider models: the tail goes through memory
        const float t = embed ? __bfloat162float(embed[(size_t)tok * embed_ld + i]) : h[i] + delta[i];
        h[i] = t;
        ss = fmaf(t, t, ss);
    }
    const float mean = block_sum(ss, red) / (float)hidden;
    const float rms = sqrtf(mean + eps);
#pragma unroll
    for (int r = 0; r < 8; r++) {
        const int i = threadIdx.x + r * 1024;
        if (i < hidden) store_act(xn, act_dt, i, (v[r] / rms) * wv[r]);
    }
    for (int i = threadIdx.x + 8 * 1024; i < hidden; i += 1024) store_act(xn, act_dt, i, (h[i] / rms) * w[i]);
    for (int i = hidden + threadIdx.x; i < xn_ld; i += 1024) store_act(xn, act_dt, i, 0.0f);
}

// row r: h = embedding of tokens[r] or h += delta; xn = RMSNorm(h) * w, zeros from hidden to
// xn_ld. One CTA per row. With `rows` given CTA i norms row rows[i] into row i of xn and leaves h as it is.
__global__ void __launch_bounds__(256)
norm_rows_kernel(float *__restrict__ h, const float *__restrict__ delta, const __nv_bfloat16 *__restrict__ embed,
                 const int *__restrict__ tokens, const float *__restrict__ w, float eps, void *__restrict__ xn, int act_dt,
                 int hidden, int embed_ld, int xn_ld, const int *__restrict__ rows) {
    __shared__ float red[32];
    const size_t r = rows ? rows[blockIdx.x] : blockIdx.x;
    float *hr = h + r * hidden;
    const float *dr = delta ? delta + r * hidden : nullptr;
    const __nv_bfloat16 *er = embed ? embed + (size_t)tokens[r] * embed_ld : nullptr;
    float ss = 0.0f;
    if (!er && hidden % 4 == 0 && hidden <= 256 * 4 * 8) {
        float4 v[8];
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = 4 * (threadIdx.x + 256 * k);
            v[k] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (i < hidden) {
                const float4 a = *reinterpret_cast<const float4 *>(hr + i), b = *reinterpret_cast<const float4 *>(dr + i);
                v[k] = make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
                if (!rows) *reinterpret_cast<float4 *>(hr + i) = v[k];
            }
            ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, ss))));
        }
        const float rms = sqrtf(block_sum(ss, red) / (float)hidden + eps);
        char *xr = reinterpret_cast<char *>(xn) + (size_t)blockIdx.x * xn_ld * (act_dt == NNQ_F32 ? 4 : 2);
#pragma unroll
        for (int k = 0; k < 8; k++) {
            const int i = 4 * (threadIdx.x + 256 * k);
            if (i >= hidden) continue;
            const float4 g = *reinterpret_cast<const float4 *>(w + i);
            const float y0 = v[k].x / rms * g.x, y1 = v[k].y / rms * g.y, y2 = v[k].z / rms * g.z, y3 = v[k].w / rms * g.w;
            if (act_dt == NNQ_F32) {
                reinterpret_cast<float4 *>(xr)[i >> 2] = make_float4(y0, y1, y2, y3);
            } else {
                const __nv_bfloat162 a = __floats2bfloat162_rn(y0, y1), b = __floats2bfloat162_rn(y2, y3);
                reinterpret_cast<uint2 *>(xr)[i >> 2] = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
            }
        }
        for (int i = hidden + threadIdx.x; i < xn_ld; i += blockDim.x) store_act(xr, act_dt, i, 0.0f);
        return;
    }
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = er ? __bfloat162float(er[i]) : hr[i] + dr[i];
        if (!rows) hr[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float rms = sqrtf(block_sum(ss, red) / (float)hidden + eps);
    char *xr = reinterpret_cast<char *>(xn) + (size_t)blockIdx.x * xn_ld * (act_dt == NNQ_F32 ? 4 : 2);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) store_act(xr, act_dt, i, ((rows ? hr[i] + dr[i] : hr[i]) / rms) * w[i]);
    for (int i = hidden + threadIdx.x; i < xn_ld; i += blockDim.x) store_act(xr, act_dt, i, 0.0f);
}

nnq_status launch_norm_step(nnq_ctx *ctx, const NormRows &a, const int *state, cudaStream_t st) {
    launch_pdl(norm_step_kernel, dim3(1), dim3(1024), st, a.h, a.delta, a.embed, state, a.w, a.eps, a.xn, a.act_dt, a.hidden, a.embed_ld, a.xn_ld);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "norm launch");
}

nnq_status launch_norm_rows(nnq_ctx *ctx, const NormRows &a, int n, const int *tokens, const int *rows, cudaStream_t st) {
    norm_rows_kernel<<<n, 256, 0, st>>>(a.h, a.delta, a.embed, tokens, a.w, a.eps, a.xn, a.act_dt, a.hidden, a.embed_ld, a.xn_ld, rows);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "norm launch");
}

}  // namespace nnq
