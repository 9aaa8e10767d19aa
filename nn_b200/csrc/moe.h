// Mixture-of-experts block: internal declarations.
#pragma once
#include "gemm_tc.h"
#include "nnq_internal.h"

struct nnq_moe {
    nnq_ctx *ctx;
    int n_experts, hidden, inter, top_k;
    int e_begin, e_local;  // experts held by this device: [e_begin, e_begin + e_local)
    float limit;
    int layout;            // nnq_moe_layout
    int fmt;               // nnq_format of the expert weights
    float *d_router_w, *d_router_b;
    nnq_weight *router;    // bf16 copy of the router where it is exact (NNQ_MOE_NK_PAIRS), else NULL
    uint8_t *d_gu, *d_gu_scales, *d_dn, *d_dn_scales;
    size_t gu_bytes, gu_scale_bytes, dn_bytes, dn_scale_bytes;   // per tensor (all experts)
    float *d_gu_bias, *d_dn_bias;
    // tiled copies of the expert weights for the grouped token-column kernel ([N, K] layouts whose
    // format and K have a tiled layout); NULL otherwise
    uint8_t *d_gu_tiled, *d_dn_tiled;
    size_t gu_tile_stride, dn_tile_stride;   // bytes per expert
};

namespace nnq {

// moe.cu, for a decoder's blocks: scratch for calls of up to `rows` tokens, and the block over `rows` tokens (y: [rows,
// hidden]). exact: every product in f32 (f32 activations only).
nnq_status moe_reserve(nnq_ctx *ctx, const nnq_moe *m, int64_t rows);
// NNQ_MOE_NK_PAIRS, one bf16 row: the norm in front (norm.xn_out is set here), the router and the experts in three launches
bool moe_step_supported(const nnq_moe *m, int hidden);
nnq_status moe_step(nnq_ctx *ctx, const nnq_moe *m, const GemvNorm &norm, float *y, cudaStream_t st);
nnq_status moe_rows(nnq_ctx *ctx, const nnq_moe *m, const void *x, nnq_dtype x_dt, int64_t rows, bool exact, float *y, cudaStream_t st);

}  // namespace nnq
