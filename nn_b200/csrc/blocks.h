// Mixers of a block decoder (attn_window.cu, recurrent.cu): kernel arguments and launchers.
//
// A block reads one normed row h per token. Everything that multiplies h sits in ONE projection row,
// proj[row, :] = [q | k | v | g | a1 | gate | up] (f32, segments at multiples of 8 columns), and
// everything that is projected back to the model width sits in ONE row act[row, :] = [mixer output |
// feed-forward activation] (f32 or bf16), so that a block is two products with the mixer between them.
// Every launcher serves both a block of prompt rows (n rows from position pos0) and a decode step
// (n = 1, the position is read from state[1] so that the launch can be replayed from a graph).
#pragma once
#include <cuda_bf16.h>

#include "nnq_internal.h"

namespace nnq {

constexpr int kAttnMaxDim = 256;        // key and value dimensions of an attention head
constexpr int kRecMaxKeyDim = 256;      // key rows of a state tile held in a thread's registers

inline int round_up(int v, int m) { return (v + m - 1) / m * m; }

// where the rows of this launch are in the sequence
struct RowSpan {
    int n;              // rows
    int pos0;           // position of the first row (state == NULL)
    const int *state;   // decode step: state[1] is the position (n = 1)
};

// block_norm.cu: h <- h + delta (or the embedding rows), xn <- RMSNorm(h) * w
struct NormRows {
    float *h;
    const float *delta;
    const __nv_bfloat16 *embed;   // NULL: h + delta
    const float *w;
    float eps;
    void *xn;
    int act_dt, hidden, embed_ld, xn_ld;
};
nnq_status launch_norm_step(nnq_ctx *ctx, const NormRows &a, const int *state, cudaStream_t st);   // one row, token in state[0]
// n rows of tokens[]; with `rows` given, n rows picked by index (h is left as it is)
nnq_status launch_norm_rows(nnq_ctx *ctx, const NormRows &a, int n, const int *tokens, const int *rows, cudaStream_t st);

// silu(gate) * up of the feed-forward, and zeros in the columns of act that belong to neither part
struct FfnPart {
    const float *proj;
    int in_cols, c_gate, c_up, ffn;
    void *act;
    int act_dt, out_k, mix, c_ffn;   // act[:, 0, mix) is the mixer's, [c_ffn, c_ffn + ffn) the feed-forward's
};

struct WindowAttn {
    RowSpan span;
    FfnPart ffn;
    int heads, kv_heads, dim, vdim, dim_ld, vdim_ld;   // _ld: rounded up to 4
    int c_q, c_k, c_v, c_g;         // columns of proj
    int gated;                      // multiply the output with sigmoid(proj[c_g ..])
    // short causal convolution over the rows of proj, before the rotation
    int taps;                       // 0 = none
    const float *conv;              // [channels, taps], channels ordered q | k | v
    float *conv_ring;               // [taps, channels]: projected values of position p at slot p % taps
    // rotation of the first rot_dims dimensions, half-split pairs
    int rot_dims;
    const float *cosv, *sinv;       // [max_seq, rot_dims / 2]
    // value mixing with the values of an earlier layer for the same token
    int mix_mode;                   // 0 none, 1 store into vfirst, 2 v = (1 - lambda) v + lambda vfirst
    float lambda;
    float *vfirst;                  // [rows, kv_heads * vdim]
    float scale;
    int window;                     // position i sees j with 0 <= i - j < window
    float *qrot;                    // [rows, heads, dim_ld]
    float *kcache, *vcache;         // [kv_heads, cap, dim_ld / vdim_ld], position p at slot p % cap
    int cap;
    // decode step: keys a window can hold, key ranges per (kv head, head tile), records of the ranges and their
    // arrival counters
    int keys_max;
    int ranges;
    float *part;
    unsigned int *arrived;
};

nnq_status launch_attn_prep(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st);       // convolution, rotation, mixing, cache append, ffn part
nnq_status launch_attn_conv_tail(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st);  // n > 1: the last taps - 1 rows enter the ring
nnq_status launch_attn_rows(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st);       // block of rows
bool attn_tc_supported(const WindowAttn &a);                                           // attn_tc.cu: block of rows on the tensor cores
nnq_status launch_attn_tc(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st);
nnq_status launch_attn_step(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st);       // one row, prologue and feed-forward part included
int attn_step_ranges(int sm_count, int heads, int kv_heads, int window, int max_seq);  // key ranges of the step kernel
size_t attn_step_part_floats(int heads, int kv_heads, int vdim_ld, int ranges);
int attn_step_counters(int heads, int kv_heads);

// S_t = diag(decay_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t per head; then per-head RMS norm of o, times
// silu(g). The decay is a constant per head, or sigmoid(W_2 a1 + b)^(1 / tau) per key channel and token.
struct Recurrence {
    RowSpan span;
    FfnPart ffn;
    int heads, dim, vdim, dim_ld;   // dim_ld: 64, 128 or 256
    int c_q, c_k, c_v, c_g, c_a1;
    float q_scale, k_scale;         // applied after the rotation
    int rot_dims;
    const float *cosv, *sinv;
    int rank;                       // > 0: decay per key channel
    const float *a2t;               // [rank, heads * dim]
    const float *a2b;               // [heads * dim]
    float inv_tau;
    const float *decay;             // [heads] (rank == 0)
    const float *head_norm;         // [vdim] or NULL
    float eps;
    float *state;                   // [heads, dim, vdim] f32
    float *q, *k, *a;               // block of rows: prepared [rows, heads, dim_ld]
    float *o;                       // [rows, heads * vdim]
};

nnq_status launch_rec_rows(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st);
nnq_status launch_rec_step(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st);

// linear_f32.cu: y = x W^T (+ bias) with f32 products and sums for unquantized weights, any row count
nnq_status launch_linear_f32(nnq_ctx *ctx, const LinearArgs &a, cudaStream_t stream);

}  // namespace nnq
