// y = x W^T (+ bias) for unquantized weights with f32 products and f32 sums: no operand is rounded to a
// shorter format. Up to eight rows run on the row kernel (also f32 throughout); more rows on 64 x 64
// register-tiled output tiles.
#include <cuda_bf16.h>

#include "blocks.h"

namespace nnq {

constexpr int kSgTile = 64, kSgK = 16, kSgLd = kSgTile + 4;

template <bool BF16W>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const uint8_t *__restrict__ w, const float *__restrict__ x, const float *__restrict__ bias, void *__restrict__ y, int M, int N,
                  int K, int y_dt) {
    __shared__ __align__(16) float xs[kSgK][kSgLd], ws[kSgK][kSgLd];
    const int tid = threadIdx.x, m0 = blockIdx.y * kSgTile, n0 = blockIdx.x * kSgTile;
    const int tx = tid & 15, ty = tid >> 4;            // 4 output columns / rows each
    const int lr = tid >> 2, lk = (tid & 3) * 4;       // staging: row of the tile, four consecutive k
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += kSgK) {             // K is a multiple of 32
        float4 xv = make_float4(0.0f, 0.0f, 0.0f, 0.0f), wv = xv;
        if (m0 + lr < M) xv = *reinterpret_cast<const float4 *>(x + (size_t)(m0 + lr) * K + k0 + lk);
        if (n0 + lr < N) {
            const size_t at = (size_t)(n0 + lr) * K + k0 + lk;
            if (BF16W) {
                const uint2 u = *reinterpret_cast<const uint2 *>(w + at * 2);
                wv = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16),
                                 __uint_as_float(u.y & 0xFFFF0000u));
            } else {
                wv = *reinterpret_cast<const float4 *>(w + at * 4);
            }
        }
        __syncthreads();
        xs[lk][lr] = xv.x; xs[lk + 1][lr] = xv.y; xs[lk + 2][lr] = xv.z; xs[lk + 3][lr] = xv.w;
        ws[lk][lr] = wv.x; ws[lk + 1][lr] = wv.y; ws[lk + 2][lr] = wv.z; ws[lk + 3][lr] = wv.w;
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kSgK; k++) {
            const float4 a = *reinterpret_cast<const float4 *>(&xs[k][4 * ty]), b = *reinterpret_cast<const float4 *>(&ws[k][4 * tx]);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + 4 * ty + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + 4 * tx + j;
            if (n >= N) continue;
            const float v = acc[i][j] + (bias ? __ldg(bias + n) : 0.0f);
            if (y_dt == NNQ_F32) reinterpret_cast<float *>(y)[(size_t)m * N + n] = v;
            else reinterpret_cast<__nv_bfloat16 *>(y)[(size_t)m * N + n] = __float2bfloat16_rn(v);
        }
    }
}

nnq_status launch_linear_f32(nnq_ctx *ctx, const LinearArgs &a, cudaStream_t stream) {
    if (a.m == 0 || a.n == 0) return NNQ_OK;
    if (a.x_dt != NNQ_F32) return fail(ctx, NNQ_ERR_UNSUPPORTED, "the f32 path takes f32 activations");
    if (a.m <= 8 || (a.fmt != NNQ_BF16_DENSE && a.fmt != NNQ_F32_DENSE)) return launch_linear_generic(ctx, a, stream);
    const dim3 grid((unsigned)((a.n + kSgTile - 1) / kSgTile), (unsigned)((a.m + kSgTile - 1) / kSgTile));
    if (a.fmt == NNQ_BF16_DENSE)
        linear_f32_kernel<true><<<grid, 256, 0, stream>>>(a.w, (const float *)a.x, a.bias, a.y, (int)a.m, (int)a.n, (int)a.k, a.y_dt);
    else
        linear_f32_kernel<false><<<grid, 256, 0, stream>>>(a.w, (const float *)a.x, a.bias, a.y, (int)a.m, (int)a.n, (int)a.k, a.y_dt);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "f32 product launch");
}

}  // namespace nnq
