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

// hashed table of token pairs added to the embedding: row (previous * mul_prev + token * mul_cur) mod buckets, row
// `buckets` for the first token of a sequence; rows as wide as the embedding's
struct PairTable {
    const __nv_bfloat16 *table;   // NULL: none
    long long mul_prev, mul_cur, buckets;
};

// what a product reads: x itself, RMSNorm(x) * w or the layer norm (x - mean) / sd * w + b
enum NormKind { kNormNone = 0, kNormRms = 1, kNormLayer = 2 };
struct InNorm {
    int kind;
    const float *w, *b;
};

// block_norm.cu: h <- alpha h + delta, or the embedding rows; with post_w given h <- layer norm of that; xn <- in(h)
struct NormRows {
    float *h;
    const float *delta;
    int delta_ld;
    float alpha;
    const float *post_w, *post_b;
    const __nv_bfloat16 *embed;   // NULL: alpha h + delta
    PairTable pairs;
    InNorm in;
    float eps;
    void *xn;
    int act_dt, hidden, embed_ld, xn_ld;
};
nnq_status launch_norm_step(nnq_ctx *ctx, const NormRows &a, const int *state, cudaStream_t st);   // one row, token in state[0]
// n rows of tokens[] at positions pos0 .. (tokens[-1]: the token in front of them); with `rows` given, n rows picked by
// index (h is left as it is)
nnq_status launch_norm_rows(nnq_ctx *ctx, const NormRows &a, int n, const int *tokens, int pos0, const int *rows, cudaStream_t st);
// act[row, j] = f(proj[row, 2 j]) * proj[row, 2 j + 1] for j < ffn, zeros up to act_ld (a multiple of 4); kind: nnq_gate_act
nnq_status launch_pair_act(nnq_ctx *ctx, const float *proj, int proj_ld, int n, int ffn, int kind, void *act, int act_dt, int act_ld, cudaStream_t st);
nnq_status launch_logit_cap(nnq_ctx *ctx, float *z, float cap, long long n, cudaStream_t st);   // z <- cap tanh(z / cap)

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

// Attention through a latent: per token one normed vector c (kv_rank) and one rotated key part r (rot), kept in a ring;
// a head's key is [W_uk,h c | r], its value W_uv,h c. ukv holds the heads' W_uk rows (dim_ld apart), then their W_uv rows
// (vdim_ld apart), zero rows between. A block of rows expands the keys and values its window reaches (kv = latents ukv^T);
// a decode step moves W_uk to the query and W_uv behind the weighted sum, and reads the latents themselves.
struct LatentAttn {
    RowSpan span;
    int heads, dim, rot, vdim, dim_ld, vdim_ld;   // dim: unrotated part; _ld: rounded up to 64
    int q_rank, q_ld, kv_rank, kv_ld, rot_ld;     // _ld: rounded up to 64
    const float *proj;              // rows of the input product
    int in_cols, c_q, c_kv;         // its columns; c_kv < 0: the ring belongs to an earlier block
    float eps;
    const float *q_norm, *kv_norm;
    const float *cosv, *sinv;       // [max_seq, rot / 2]
    int act_dt;                     // of cq, the rings, kv and out
    void *cq;                       // [rows, q_ld]
    void *ring_c, *ring_r;          // [cap, kv_ld], [cap, rot_ld], position p at slot p % cap
    int cap;
    const float *q;                 // [rows, heads * (dim + rot)] as projected
    float scale;
    int window;
    void *out;                      // [rows, out_ld], heads * vdim columns and zeros
    int out_ld;
    // block of rows: keys first .. pos0 + n - 1 in a row
    int first, keys;
    void *lin_c, *lin_r;            // [keys, kv_ld], [keys, rot_ld] (the ring itself where nothing wraps: linear = 0)
    int linear;                     // copy the ring's older positions
    const void *kv;                 // [keys, heads * (dim_ld + vdim_ld)]
    float *qrot, *kfull, *vfull;    // rows on the general attention kernels: f32 copies with the shared part per head
    // decode step
    const __nv_bfloat16 *ukv;
    float *qlat;                    // queries in the latent space (latent_step_query_floats)
    int ranges, keys_max;
    float *part;                    // [ranges, heads, kv_ld + 4]: maximum, sum, -, -, weighted latents
};

enum { kLatentQueries = 1, kLatentKeys = 2 };
// the normed query latent (cq), the new latents into the ring (and lin), the older ones into lin; n rows
nnq_status launch_latent_prep(nnq_ctx *ctx, const LatentAttn &a, int parts, cudaStream_t st);
nnq_status launch_latent_rows(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st);   // attention of a block of rows (n > 1 or not)
bool latent_tc_supported(int act_dt, int dim, int rot, int vdim);                    // attn_latent_tc.cu: on the tensor cores
nnq_status launch_latent_tc(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st);
nnq_status launch_latent_step(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st);   // one row, appends its latent
size_t latent_step_query_floats(int heads, int kv_ld, int rot_ld);
bool latent_step_supported(int act_dt, int kv_ld, int rot_ld);
int latent_step_ranges(int sm_count, int heads, int window, int max_seq, int act_dt);

// linear_f32.cu: y = x W^T (+ bias) with f32 products and sums for unquantized weights, any row count
nnq_status launch_linear_f32(nnq_ctx *ctx, const LinearArgs &a, cudaStream_t stream);

}  // namespace nnq
