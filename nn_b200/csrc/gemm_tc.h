// Tensor-core (tcgen05 / TMEM) prefill product: internal declarations.
#pragma once
#include <cuda_bf16.h>

#include "blocks.h"
#include "nnq_internal.h"

namespace nnq {

struct TcArgs {
    const uint8_t *w;       // raw blocks [N, K]
    const uint8_t *scales;  // separate scale bytes or NULL
    const void *x;
    const float *bias;
    void *y;
    int64_t m, n, k;
    int fmt, x_dt, y_dt;
};

// Grouped variant for the expert products of a mixture-of-experts block: the rows of x are sorted
// by expert (device-side offsets[e] .. offsets[e+1]), expert e multiplies its rows with the weight
// at w + e * w_stride (scales + e * s_stride) and adds bias + e * n. x is bf16 [rows_upper, k]
// (rows beyond offsets[experts] are never stored), y is f32 [rows_upper, n].
struct TcGroupArgs {
    const uint8_t *w, *scales;
    size_t w_stride, s_stride;
    const void *x_bf16;
    const float *bias;      // [experts][n] or NULL
    float *y;
    const int *offsets;     // device, [experts + 1]
    int experts;
    int64_t rows_upper;     // upper bound of offsets[experts] (allocation size of x and y in rows)
    int64_t n, k;
    int fmt;
    // decode-once path only: with h_out given and an MXFP4 format the product is the gate / up product
    // of an expert block (n = 2 * inter, gate rows first) and its epilogue writes
    // h_out[row, j] = clamp(silu(gate_j), +-swiglu_limit) * up_j in bf16 instead of y
    // (gemm_dense_grouped_fuses_swiglu tells)
    __nv_bfloat16 *h_out = nullptr;
    float swiglu_limit = 0.0f;
    // decode-once path only: the experts are nn-gptoss [experts, K, N] MXFP4 tensors (codes [E, K, N / 2],
    // scale bytes [E, K, N / 32], blocks along N); the decode transposes them into the [N, K] copy
    bool kn = false;
    // bf16 experts whose gate and up rows alternate (row 2j: gate j): multiplied in place, with h_out given the epilogue
    // forms the activation as above
    bool pairs = false;
};
bool gemm_dense_grouped_fuses_swiglu(const TcGroupArgs &g);
nnq_status launch_gemm_tc_grouped(nnq_ctx *ctx, const TcGroupArgs &a, cudaStream_t stream);

// K must be a multiple of 64 (one 128-byte swizzle row of bf16 per stage).
bool gemm_tc_supported(const nnq_weight *w, int64_t m);
nnq_status launch_gemm_tc(nnq_ctx *ctx, const TcArgs &a, cudaStream_t stream);

// Large prefill (M >= 256, bf16 activations, K a multiple of 64): decode the weight to bf16 in the
// context's scratch, then a persistent TMA + tcgen05 GEMM (gemm_dense.cu).
bool gemm_dense_supported(const nnq_ctx *ctx, const nnq_weight *w, int64_t m, int x_dt);
nnq_status dense_scratch_reserve(nnq_ctx *ctx, int64_t n, int64_t k);
nnq_status launch_gemm_dense(nnq_ctx *ctx, const TcArgs &a, cudaStream_t stream);
// the GEMM alone over an already decoded bf16 [n, k] weight (a.w / a.fmt are not read)
nnq_status launch_gemm_dense_bf16(nnq_ctx *ctx, const void *w_bf16, const TcArgs &a, cudaStream_t stream);
// gate / up product of a bf16 weight with alternating gate and up rows (n = 2 * width): h_out[m, width] = f(gate) * up in
// bf16, f = gate_kind (nnq_gate_act); gemm_dense_supported tells whether it runs, a.y is not written
nnq_status launch_gemm_dense_pairs(nnq_ctx *ctx, const TcArgs &a, __nv_bfloat16 *h_out, int gate_kind, cudaStream_t stream);
// dense_gemv.cu: one to four bf16 rows against an unquantized bf16 weight
bool dense_gemv_supported(const nnq_weight *w, int64_t m, int x_dt);
nnq_status launch_dense_gemv(nnq_ctx *ctx, const TcArgs &a, cudaStream_t stream);
// The same for one row that the kernel forms itself: h = alpha h_in + delta, or the embedding row of token state[0]
// (plus its pair row: previous token state[4], position state[1]), post-normed where post_w is given; x = in(h). h_out
// (not h_in) receives h, xn_out x as bf16 [k], NULL to drop them. a.x is not read; a.k >= hidden, columns from hidden on
// are zero.
struct GemvNorm {
    const float *h_in, *delta;    // delta NULL: alpha h_in
    float *h_out;
    __nv_bfloat16 *xn_out;
    float alpha;
    const __nv_bfloat16 *embed;   // NULL: alpha h_in + delta
    PairTable pairs;
    int embed_ld;
    const int *state;
    const float *post_w, *post_b;
    InNorm in;
    float eps;
    int hidden;
    bool half;                    // half of the warps and of the ring: products whose weight is a few hundred kilobytes per SM
    int xn_at;                    // (set by the launcher)
};
bool dense_gemv_norm_supported(const nnq_weight *w, int hidden);
// pair_act > 0: rows 2j and 2j + 1 of the weight are a gate and an up row, and y (bf16, n / 2 columns and zeros up to y_ld)
// receives f(gate) * up, f = nnq_gate_act pair_act - 1
nnq_status launch_dense_gemv_norm(nnq_ctx *ctx, const TcArgs &a, const GemvNorm &norm, int pair_act, int y_ld, cudaStream_t stream);
// Products of one row with the experts it is routed to, bf16 [experts, N, K] weights.
// Every CTA routes the row (logits f32 [experts]).
//   up    slot s, row pair j of its expert: y[s * inter + j] = weight_s * silu(gate) * up in bf16
//   down  y[n] (f32) = sum over the slots of W[expert of s][n, :] . x[s * inter ..]; routes before it waits for the kernel in
//         front, so that kernel must not be the one that forms the logits
struct GemvExperts {
    const void *w;
    int experts, top, inter, hidden;
    const float *logits;
    const __nv_bfloat16 *x;
    void *y;
};
nnq_status launch_dense_gemv_experts(nnq_ctx *ctx, const GemvExperts &g, bool up, cudaStream_t stream);
bool gemm_dense_shape_ok(const nnq_ctx *ctx, int64_t m, int64_t n, int64_t k, int x_dt);
// the expert products of a prefill-sized MoE call: all local experts decoded at once
bool gemm_dense_grouped_supported(const nnq_ctx *ctx, const TcGroupArgs &g);
nnq_status launch_gemm_dense_grouped(nnq_ctx *ctx, const TcGroupArgs &g, cudaStream_t stream);

}  // namespace nnq
