// Residual update + norm of a block decoder, for the row of a decode step and for a block of rows, and the small
// row kernels around the products (gated activation of an interleaved product, logit cap). The normed rows may be
// wider than the model (zero columns up to the products' k step).
#include "block_norm.cuh"
#include "blocks.cuh"

namespace nnq {

template <int K>
__device__ __forceinline__ void store_units(const NormRow &r, void *xn, int act_dt, float *red) {
    float4 v[K];
    norm_units(r, v, red);
#pragma unroll
    for (int k = 0; k < K; k++) {
        const int u = threadIdx.x + blockDim.x * k;
        if (4 * u >= r.hidden) continue;
        if (act_dt == NNQ_F32) {
            reinterpret_cast<float4 *>(xn)[u] = v[k];
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v[k].x, v[k].y), b = __floats2bfloat162_rn(v[k].z, v[k].w);
            reinterpret_cast<uint2 *>(xn)[u] = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
        }
    }
}

// One CTA of 256 per row (the row of a step: `state` given, token state[0], position state[1], the token before it
// state[4]). With `rows` given CTA i norms row rows[i] into row i of xn and leaves h as it is. K: units of four elements
// per thread, 0: any width, element by element.
template <int K>
__global__ void __launch_bounds__(256) norm_rows_kernel(const NormRows a, const int *__restrict__ tokens, int pos0, const int *__restrict__ rows,
                                                        const int *__restrict__ state) {
    pdl_prologue();
    pdl_release();
    __shared__ float red[32];
    const size_t r = rows ? rows[blockIdx.x] : blockIdx.x;
    NormRow n;
    n.h_in = a.h + r * a.hidden;
    n.h_out = rows ? nullptr : a.h + r * a.hidden;
    n.delta = a.delta ? a.delta + r * a.delta_ld : nullptr;
    n.e0 = n.e1 = nullptr;
    if (a.embed) {
        const int tok = state ? state[0] : tokens[(int)r], pos = state ? state[1] : pos0 + (int)r;
        n.e0 = a.embed + (size_t)tok * a.embed_ld;
        if (a.pairs.table) {
            const int prev = pos == 0 ? 0 : (state ? state[4] : tokens[(int)r - 1]);   // (tokens[-1]: the one in front of this block)
            n.e1 = a.pairs.table + pair_row(a.pairs, prev, tok, pos) * a.embed_ld;
        }
    }
    n.alpha = a.alpha;
    n.post_w = a.post_w;
    n.post_b = a.post_b;
    n.in = a.in;
    n.eps = a.eps;
    n.hidden = a.hidden;
    char *xr = reinterpret_cast<char *>(a.xn) + (size_t)blockIdx.x * a.xn_ld * (a.act_dt == NNQ_F32 ? 4 : 2);
    if constexpr (K > 0) store_units<K>(n, xr, a.act_dt, red);
    else norm_elements(n, red, [&](int i, float v) { store_act(xr, a.act_dt, i, v); });
    for (int i = a.hidden + threadIdx.x; i < a.xn_ld; i += blockDim.x) store_act(xr, a.act_dt, i, 0.0f);
}

static void go_norm(const NormRows &a, int n, const int *tokens, int pos0, const int *rows, const int *state, cudaStream_t st) {
    const dim3 grid(n), block(256);
    if (a.hidden % 4 || a.hidden > 8192) launch_pdl(norm_rows_kernel<0>, grid, block, st, a, tokens, pos0, rows, state);
    else if (a.hidden <= 2048) launch_pdl(norm_rows_kernel<2>, grid, block, st, a, tokens, pos0, rows, state);
    else if (a.hidden <= 4096) launch_pdl(norm_rows_kernel<4>, grid, block, st, a, tokens, pos0, rows, state);
    else launch_pdl(norm_rows_kernel<8>, grid, block, st, a, tokens, pos0, rows, state);
}

nnq_status launch_norm_step(nnq_ctx *ctx, const NormRows &a, const int *state, cudaStream_t st) {
    go_norm(a, 1, nullptr, 0, nullptr, state, st);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "norm launch");
}

nnq_status launch_norm_rows(nnq_ctx *ctx, const NormRows &a, int n, const int *tokens, int pos0, const int *rows, cudaStream_t st) {
    go_norm(a, n, tokens, pos0, rows, nullptr, st);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "norm launch");
}

// act[row, j] = f(proj[row, 2 j]) * proj[row, 2 j + 1], zeros from ffn to act_ld; four columns per thread
__global__ void __launch_bounds__(256) pair_act_kernel(const float *__restrict__ proj, int proj_ld, int ffn, int kind, void *__restrict__ act, int act_dt,
                                                       int act_ld, long long total) {
    pdl_prologue();
    pdl_release();
    const int units = act_ld >> 2;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < total; i += (long long)gridDim.x * 256) {
        const int row = (int)(i / units), j = (int)(i - (long long)row * units) * 4;
        const float4 *p = reinterpret_cast<const float4 *>(proj + (size_t)row * proj_ld + 2 * j);
        float v[4];
        if (j + 4 <= ffn) {
            const float4 a = p[0], b = p[1];
            v[0] = gate_act(kind, a.x) * a.y; v[1] = gate_act(kind, a.z) * a.w; v[2] = gate_act(kind, b.x) * b.y; v[3] = gate_act(kind, b.z) * b.w;
        } else {
            const float *q = reinterpret_cast<const float *>(p);
#pragma unroll
            for (int e = 0; e < 4; e++) v[e] = j + e < ffn ? gate_act(kind, q[2 * e]) * q[2 * e + 1] : 0.0f;
        }
        const size_t at = (size_t)row * act_ld + j;
        if (act_dt == NNQ_F32) {
            *reinterpret_cast<float4 *>(reinterpret_cast<float *>(act) + at) = make_float4(v[0], v[1], v[2], v[3]);
        } else {
            const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
            *reinterpret_cast<uint2 *>(reinterpret_cast<__nv_bfloat16 *>(act) + at) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
        }
    }
}

nnq_status launch_pair_act(nnq_ctx *ctx, const float *proj, int proj_ld, int n, int ffn, int kind, void *act, int act_dt, int act_ld, cudaStream_t st) {
    const long long total = (long long)n * (act_ld >> 2), want = (total + 255) / 256, most = 16LL * ctx->sm_count;
    launch_pdl(pair_act_kernel, dim3((unsigned)(want < most ? want : most)), dim3(256), st, proj, proj_ld, ffn, kind, act, act_dt, act_ld, total);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "activation launch");
}

__global__ void __launch_bounds__(256) logit_cap_kernel(float *__restrict__ z, float cap, long long n) {
    pdl_prologue();
    pdl_release();
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) z[i] = cap * tanhf(z[i] / cap);
}

nnq_status launch_logit_cap(nnq_ctx *ctx, float *z, float cap, long long n, cudaStream_t st) {
    const long long want = (n + 255) / 256, most = 8LL * ctx->sm_count;
    launch_pdl(logit_cap_kernel, dim3((unsigned)(want < most ? want : most)), dim3(256), st, z, cap, n);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "logit cap launch");
}

}  // namespace nnq
