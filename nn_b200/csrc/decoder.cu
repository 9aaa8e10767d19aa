// One decode step (one token, batch 1) of a Qwen3-shaped decoder on the device: embedding row ->
// N x [RMSNorm -> q/k/v products -> per-head QK-norm + half-split RoPE -> KV append -> grouped-query
// attention over the cache -> o product -> residual -> RMSNorm -> gate/up products -> silu * up ->
// down product -> residual] -> final RMSNorm -> vocabulary product -> greedy argmax.
// Follows crates/nn-qwen3/src/layers.rs:40-47,94-167,205-226 (MLP, attention, decoder layer),
// crates/nn-core/src/layers/rms_norm.rs:87-100, layers/attention/rope.rs:78-106 (tables),
// rope_half_split.rs:98-134 (rotation), attention/sdpa.rs:59-71, dyn_tensor/ops/math.rs:140 (silu)
// and layers/generation/autoregressive_sampling.rs:14-21 (argmax: the last of equal maxima).
//
// The quantized products are the library's own (nnq_linear / nnq_linear_batch); this file adds the
// small kernels between them. Token and position live in device memory and are advanced by the
// last kernel of a step, so the launches of one step can be captured once and replayed per token.
//
// A decoder is built either from Qwen3 layers (nnq_decoder_create) or from blocks that each name their own
// mixer (nnq_decoder_create_blocks): norm -> one product for everything that reads the normed row -> mixer
// and feed-forward activation (attn_window.cu, recurrent.cu) -> one product back to the model width. Token
// loop, prompt pass, position keeping, head and greedy commit are the same for both.
#include <cuda_bf16.h>
#include <math.h>
#include <string.h>

#include <new>

#include "blocks.h"
#include "comm.cuh"
#include "decoder_common.cuh"
#include "gemm_tc.h"
#include "moe.h"

namespace nnq {
nnq_status comm_view(nnq_comm *c, CommView *out);   // comm.cu
}

struct nnq_decoder {
    nnq_ctx *ctx;
    nnq_decoder_config cfg;
    struct Layer {
        const nnq_weight *q, *k, *v, *o, *gate, *up, *down;
        float *in_norm, *post_norm, *q_norm, *k_norm;   // device copies
    } *layers;
    const void *d_embed;        // [vocab, hidden] bf16, caller-owned
    float *d_final_norm;
    const nnq_weight *lm_head;
    float *d_cos, *d_sin;       // [max_seq, head_dim / 2]
    float *d_kcache, *d_vcache; // [layers, kv_heads, max_seq, head_dim]
    float *d_h, *d_delta, *d_q, *d_k, *d_v, *d_qrot, *d_g, *d_u, *d_logits, *d_part;
    unsigned int *d_arrived;   // per kv head: attention CTAs that have published their record
    void *d_xn, *d_attn, *d_mid;   // activations fed to the products (f32 or bf16)
    int *d_state;               // [0] token, [1] position, [2] steps taken, [3] context full, [4] token before [0]; then the argmax scratch
    int *d_tokens;              // generated tokens, [max_seq]
    int act_dt;
    int ready;                  // bit set of what has been supplied
    nnq_comm *comm;             // tensor parallel: exchange of the row-parallel products (NULL when tp_world = 1)
    int lh, lkv;                // query / key-value heads held by this rank
    int head_rows, head_row0;   // rows of the vocabulary projection held by this rank and the first of them
    long long host_pos;         // position of the next step as far as the host knows it (-1: unknown)
    // prompt pass: row-major [rows, width] versions of the step's buffers, allocated by the first
    // nnq_decoder_prefill call (pf_rows rows)
    int pf_rows;
    float *pf_h, *pf_delta, *pf_q, *pf_k, *pf_v, *pf_qrot, *pf_g, *pf_u;
    void *pf_xn, *pf_attn, *pf_mid;
    int *pf_tokens;
    int *pf_want;               // rows of a block whose logits are asked for, [kPrefillRows]
    float *d_want_logits;       // [kWantRows, vocab], allocated by the first nnq_decoder_extend that asks for any
    int embed_ld, xn_ld;        // row strides of the embedding table and of the normed rows
    // block decoder: the row buffers above are allocated at creation (pf_rows rows; a step uses row 0)
    struct Block {
        nnq_block_config cfg;
        nnq_block_layout lay;
        const nnq_weight *in, *out;
        float *norm, *bias_in, *bias_out, *conv, *head_norm, *a2t, *a2b, *decay;
        float lambda;
        float *cosv, *sinv;     // rotation tables, owned by the first block with the same base and width
        bool owns_tables;
        int dim_ld, vdim_ld;
        int cap, ranges;        // attention: ring capacity, key ranges of the decode kernel
        float *kcache, *vcache, *conv_ring, *rec_state;
        int mix_mode;
        float *norm_bias;       // post_norm
        const nnq_weight *uq, *ukv;
        const nnq_moe *moe;
        float *q_norm, *kv_norm;
        void *ring_c, *ring_r;  // latents and rotated key parts, owned by the block that forms them
    } *blocks;
    float *b_h2;                // the step's residual row alternates between d_h and this buffer
    float *b_proj, *b_q, *b_k, *b_a, *b_o, *b_vfirst;   // rows of proj; prepared q / k / decay, mixer output, first values
    void *b_act;
    void *b_cq, *b_lin_c, *b_lin_r, *b_kv;              // latent attention: query latents, the window's latents in a row, expanded keys and values
    float *b_q2, *b_qrot, *b_kfull, *b_vfull, *b_qlat;  // its queries; f32 copies for the general kernels; queries in the latent space
    float *final_bias;          // layer norm in front of the head
    float logit_cap;            // 0: none
    nnq::PairTable pairs;
};

namespace nnq {

constexpr int kAttnRanges = 32;   // CTAs per kv head in the decode step's attention
constexpr int kAttnWarps = 4;
// Rows of a prompt that go through the layers together: large enough that the products run on the
// decode-once tensor path with several row tiles per weight tile (about 210 KB of buffers per row at
// the Qwen3-8B shape).
constexpr int kPrefillRows = 1024;
// with experts among the blocks: their weights are read once per block of rows, whatever part of the rows each expert gets
constexpr int kPrefillRowsExperts = 4096;
constexpr int kArgmaxBlocks = 128;
constexpr int kStateWords = 8;    // token, position, steps, context full, previous token
constexpr int kWantRows = 64;     // rows of logits formed together

// h = embedding row of the current token (first layer), or h += delta; xn = RMSNorm(h) * w.
// One CTA; every thread keeps its (up to 8) elements in registers between the two phases.
__global__ void __launch_bounds__(1024)
dec_norm_kernel(float *__restrict__ h, const float *__restrict__ delta, const __nv_bfloat16 *__restrict__ embed,
                const int *__restrict__ state, const float *__restrict__ w, float eps, void *__restrict__ xn, int act_dt,
                int hidden) {
    pdl_prologue();
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
            v[r] = embed ? __bfloat162float(embed[(size_t)tok * hidden + i]) : h[i] + delta[i];
            wv[r] = w[i];
            h[i] = v[r];
            ss = fmaf(v[r], v[r], ss);
        }
    }
    for (int i = threadIdx.x + 8 * 1024; i < hidden; i += 1024) {   // wider models: the tail goes through memory
        const float t = embed ? __bfloat162float(embed[(size_t)tok * hidden + i]) : h[i] + delta[i];
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
}

// One CTA per head (query heads, then key heads, then value heads), one thread per dimension:
// RMSNorm over the head (q, k), half-split rotation at the current position, append k / v.
__global__ void __launch_bounds__(256)
dec_qk_rope_kernel(const float *__restrict__ q, const float *__restrict__ k, const float *__restrict__ v,
                   const float *__restrict__ qw, const float *__restrict__ kw, const float *__restrict__ cosv,
                   const float *__restrict__ sinv, const int *__restrict__ state, float eps, float *__restrict__ qrot,
                   float *__restrict__ kcache, float *__restrict__ vcache, int n_heads, int n_kv, int hd, int max_seq) {
    pdl_prologue();
    __shared__ float red[32];
    __shared__ float xs[256];
    const int head = blockIdx.x, d = threadIdx.x, pos = state[1];
    const int half = hd / 2;
    if (head >= n_heads + n_kv) {   // value head: plain append
        const int kvh = head - n_heads - n_kv;
        if (d < hd) vcache[((size_t)kvh * max_seq + pos) * hd + d] = v[kvh * hd + d];
        return;
    }
    const bool is_q = head < n_heads;
    const float *src = is_q ? q + head * hd : k + (head - n_heads) * hd;
    const float *w = is_q ? qw : kw;
    const float x = d < hd ? src[d] : 0.0f;
    const float mean = block_sum(x * x, red) / (float)hd;
    const float rms = sqrtf(mean + eps);
    if (d < hd) xs[d] = (x / rms) * w[d];
    __syncthreads();
    if (d >= hd) return;
    const int i = d < half ? d : d - half;
    const float c = cosv[(size_t)pos * half + i], s = sinv[(size_t)pos * half + i];
    // y1 = x1 cos - x2 sin; y2 = x1 sin + x2 cos
    const float y = d < half ? xs[d] * c - xs[d + half] * s : xs[d - half] * s + xs[d] * c;
    if (is_q) qrot[head * hd + d] = y;
    else kcache[((size_t)(head - n_heads) * max_seq + pos) * hd + d] = y;
}

// Grouped-query attention over the cache in one launch. The keys are taken in batches of 32; a
// kv head's batches are dealt to kAttnRanges CTAs (contiguous ranges) and inside a CTA to its four
// warps. For a batch, lane j forms the dot products of key j with every query head of the group (the
// query vectors sit in shared memory, the key row is read once for the whole group), the batch joins
// the running softmax of each head (maximum, sum), then the value rows are read coalesced (lane l
// owns dimensions 4l .. 4l+3) and weighted with the probabilities passed by shuffle. The warps of a
// CTA merge through shared memory into one record per head, (m, l, acc[hd]), in global memory; the
// CTA that finishes last for its kv head (an arrival counter, reset by that CTA for the next
// launch) merges the records of all ranges and writes the output rows:
// out[head, d] = sum_s acc_s[d] e^(m_s - M) / sum_s l_s e^(m_s - M).
template <int G>
__global__ void __launch_bounds__(kAttnWarps * 32)
dec_attn_kernel(const float *__restrict__ qrot, const float *__restrict__ kcache, const float *__restrict__ vcache,
                const int *__restrict__ state, float scale, float *__restrict__ part, unsigned int *__restrict__ arrived,
                void *__restrict__ out, int act_dt, int hd, int max_seq) {
    pdl_prologue();
    __shared__ __align__(16) float qs[G][128];
    __shared__ __align__(16) float wacc[kAttnWarps][G][128];
    __shared__ float wm[kAttnWarps][G], wl[kAttnWarps][G];
    __shared__ int s_last;
    const int kvh = blockIdx.x, range = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int ctx = state[1] + 1;
    const int nb = (ctx + 31) >> 5;                              // batches of 32 keys in the context
    const int bper = (nb + kAttnRanges - 1) / kAttnRanges;       // batches per range
    const int used = (nb + bper - 1) / bper;                     // ranges that hold keys
    const int b_lo = range * bper, b_hi = min(nb, b_lo + bper);
    if (b_lo < b_hi) {
        for (int i = threadIdx.x; i < G * 32; i += kAttnWarps * 32)
            *reinterpret_cast<float4 *>(&qs[i >> 5][4 * (i & 31)]) = *reinterpret_cast<const float4 *>(qrot + (kvh * G + (i >> 5)) * hd + 4 * (i & 31));
        __syncthreads();
        float m[G], l[G];
        float4 acc[G];
#pragma unroll
        for (int g = 0; g < G; g++) {
            m[g] = -INFINITY;
            l[g] = 0.0f;
            acc[g] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        const float *kb = kcache + (size_t)kvh * max_seq * hd, *vb = vcache + (size_t)kvh * max_seq * hd;
        for (int b = b_lo + warp; b < b_hi; b += kAttnWarps) {
            const int b0 = b << 5, j1 = min(ctx, b0 + 32);
            const int j = b0 + lane;
            const bool valid = j < j1;
            const float4 *krow = reinterpret_cast<const float4 *>(kb + (size_t)(valid ? j : b0) * hd);
            // the value rows of the batch are wanted after the softmax: ask L2 for them now (lane j: row j)
            if (valid) {
                const char *vrow = reinterpret_cast<const char *>(vb + (size_t)j * hd);
#pragma unroll
                for (int c = 0; c < 4; c++) asm volatile("prefetch.global.L2 [%0];" ::"l"(vrow + 128 * c));
            }
            float dot[G];
#pragma unroll
            for (int g = 0; g < G; g++) dot[g] = 0.0f;
#pragma unroll 16
            for (int d4 = 0; d4 < 32; d4++) {
                const float4 kv = krow[d4];
#pragma unroll
                for (int g = 0; g < G; g++) {
                    const float4 qv = *reinterpret_cast<const float4 *>(&qs[g][4 * d4]);
                    dot[g] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, dot[g]))));
                }
            }
            float p[G];
#pragma unroll
            for (int g = 0; g < G; g++) {
                const float s = valid ? dot[g] * scale : -INFINITY;
                float bm = s;
#pragma unroll
                for (int off = 16; off > 0; off >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xFFFFFFFFu, bm, off));
                const float mn = fmaxf(m[g], bm);   // finite: the batch holds at least one key
                const float corr = expf(m[g] - mn);
                p[g] = expf(s - mn);
                float ps = p[g];
#pragma unroll
                for (int off = 16; off > 0; off >>= 1) ps += __shfl_xor_sync(0xFFFFFFFFu, ps, off);
                l[g] = l[g] * corr + ps;
                acc[g].x *= corr; acc[g].y *= corr; acc[g].z *= corr; acc[g].w *= corr;
                m[g] = mn;
            }
            const int nk = j1 - b0;
#pragma unroll 4
            for (int jj = 0; jj < nk; jj++) {
                const float4 vv = *reinterpret_cast<const float4 *>(vb + (size_t)(b0 + jj) * hd + 4 * lane);
#pragma unroll
                for (int g = 0; g < G; g++) {
                    const float pj = __shfl_sync(0xFFFFFFFFu, p[g], jj);
                    acc[g].x = fmaf(pj, vv.x, acc[g].x);
                    acc[g].y = fmaf(pj, vv.y, acc[g].y);
                    acc[g].z = fmaf(pj, vv.z, acc[g].z);
                    acc[g].w = fmaf(pj, vv.w, acc[g].w);
                }
            }
        }
        // the warps of the CTA -> one record per head
#pragma unroll
        for (int g = 0; g < G; g++) {
            if (lane == 0) {
                wm[warp][g] = m[g];
                wl[warp][g] = l[g];
            }
            *reinterpret_cast<float4 *>(&wacc[warp][g][4 * lane]) = acc[g];
        }
        __syncthreads();
        for (int i = threadIdx.x; i < G * 128; i += kAttnWarps * 32) {
            const int g = i >> 7, dd = i & 127;
            float M = wm[0][g];
#pragma unroll
            for (int w = 1; w < kAttnWarps; w++) M = fmaxf(M, wm[w][g]);   // warp 0 always holds a batch: finite
            float L = 0.0f, a = 0.0f;
#pragma unroll
            for (int w = 0; w < kAttnWarps; w++) {
                const float e = wm[w][g] == -INFINITY ? 0.0f : expf(wm[w][g] - M);
                L = fmaf(wl[w][g], e, L);
                a = fmaf(wacc[w][g][dd], e, a);
            }
            float *o = part + ((size_t)(kvh * kAttnRanges + range) * G + g) * (hd + 4);   // record: m, l, pad, pad, acc[hd]
            if (dd == 0) {
                o[0] = M;
                o[1] = L;
            }
            if (dd < hd) o[4 + dd] = a;
        }
    }
    // arrival: the records above are published before the count, the last CTA reads them after it
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) s_last = atomicAdd(arrived + kvh, 1u) == (unsigned)(kAttnRanges - 1);
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    // a warp per head, a lane per four dimensions; every load of a pass is issued before the first
    // is used (the records sit in L2: the pass costs one round trip, not one per range)
    for (int g = warp; g < G; g += kAttnWarps) {
        const float *rec = part + ((size_t)(kvh * kAttnRanges) * G + g) * (hd + 4);
        const size_t step = (size_t)G * (hd + 4);
        float2 ml[kAttnRanges];
#pragma unroll
        for (int s = 0; s < kAttnRanges; s++)
            ml[s] = s < used ? __ldcg(reinterpret_cast<const float2 *>(rec + s * step)) : make_float2(-INFINITY, 0.0f);
        float M = ml[0].x;
#pragma unroll
        for (int s = 1; s < kAttnRanges; s++) M = fmaxf(M, ml[s].x);
        float L = 0.0f;
#pragma unroll
        for (int s = 0; s < kAttnRanges; s++) {
            ml[s].x = s < used ? expf(ml[s].x - M) : 0.0f;
            L = fmaf(ml[s].y, ml[s].x, L);
        }
        float4 a = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int h = 0; h < kAttnRanges; h += 16) {
            float4 v[16];
#pragma unroll
            for (int s = 0; s < 16; s++)
                v[s] = h + s < used ? __ldcg(reinterpret_cast<const float4 *>(rec + (h + s) * step + 4) + lane) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int s = 0; s < 16; s++) {
                a.x = fmaf(v[s].x, ml[h + s].x, a.x);
                a.y = fmaf(v[s].y, ml[h + s].x, a.y);
                a.z = fmaf(v[s].z, ml[h + s].x, a.z);
                a.w = fmaf(v[s].w, ml[h + s].x, a.w);
            }
        }
        const int at = (kvh * G + g) * hd + 4 * lane;
        store_act(out, act_dt, at, a.x / L);
        store_act(out, act_dt, at + 1, a.y / L);
        store_act(out, act_dt, at + 2, a.z / L);
        store_act(out, act_dt, at + 3, a.w / L);
    }
    if (threadIdx.x == 0) arrived[kvh] = 0;   // the next launch starts after this grid has ended
}

__global__ void dec_silu_mul_kernel(const float *__restrict__ g, const float *__restrict__ u, void *__restrict__ mid,
                                    int act_dt, int n) {
    pdl_prologue();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) {
        const float x = g[i];
        store_act(mid, act_dt, i, (x / (1.0f + expf(-x))) * u[i]);
    }
}

// larger value wins; of equal values the larger index (the reference keeps the last maximum)
__device__ __forceinline__ void arg_better(float &bv, int &bi, float v, int i) {
    if (v > bv || (v == bv && i > bi)) {
        bv = v;
        bi = i;
    }
}

__global__ void __launch_bounds__(256)
dec_argmax_stage1_kernel(float *__restrict__ logits, int n, float cap, float *__restrict__ bv_out, int *__restrict__ bi_out) {
    pdl_prologue();
    __shared__ float sv[8];
    __shared__ int si[8];
    float bv = -INFINITY;
    int bi = -1;
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n; i += gridDim.x * blockDim.x) {
        float z = logits[i];
        if (cap > 0.0f) logits[i] = z = cap * tanhf(z / cap);
        arg_better(bv, bi, z, i);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        const float ov = __shfl_xor_sync(0xFFFFFFFFu, bv, off);
        const int oi = __shfl_xor_sync(0xFFFFFFFFu, bi, off);
        arg_better(bv, bi, ov, oi);
    }
    if ((threadIdx.x & 31) == 0) {
        sv[threadIdx.x >> 5] = bv;
        si[threadIdx.x >> 5] = bi;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < 8; w++) arg_better(bv, bi, sv[w], si[w]);
        bv_out[blockIdx.x] = bv;
        bi_out[blockIdx.x] = bi;
    }
}

// Records the winning token and advances the device-side (token, position) pair. state[3] is set
// by the step that fills the last position; a step that finds it set has nowhere to write:
// it raises the context's status word (2 = context full) and changes nothing.
__device__ __forceinline__ void dec_commit_token(int bi, int *state, int *tokens, int max_seq) {
    if (bi < 0) bi = 0;   // all NaN: the reference returns index 0
    const int pos = state[1];
    tokens[pos] = bi;
    state[4] = state[0];   // the token in front of the next one
    state[0] = bi;
    if (pos + 1 < max_seq) state[1] = pos + 1;
    else state[3] = 1;
    state[2] += 1;
}

// picks the winner among the block maxima
__global__ void dec_argmax_stage2_kernel(const float *__restrict__ bv_in, const int *__restrict__ bi_in, int blocks,
                                         int *__restrict__ state, int *__restrict__ tokens, int max_seq, int *status) {
    pdl_prologue();
    float bv = -INFINITY;   // one warp
    int bi = -1;
    for (int b = threadIdx.x; b < blocks; b += 32) arg_better(bv, bi, bv_in[b], bi_in[b]);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        const float ov = __shfl_xor_sync(0xFFFFFFFFu, bv, off);
        const int oi = __shfl_xor_sync(0xFFFFFFFFu, bi, off);
        arg_better(bv, bi, ov, oi);
    }
    if (threadIdx.x != 0) return;
    if (state[3]) atomicExch(status, 2);
    else dec_commit_token(bi, state, tokens, max_seq);
}

// Vocabulary-parallel head: every rank holds the maximum of its slice of the logits; the ranks
// exchange (value, index) through the last 16 bytes of their communicator slots as two 8-byte
// (payload, sequence number) stores, wait (bounded) for the peers' records and all pick the same
// winner: the larger value, of equal values the larger index -- the reference's "last maximum"
// rule survives the gather because it only depends on (value, index), not on arrival order.
__global__ void dec_argmax_exchange_kernel(const float *__restrict__ bv_in, const int *__restrict__ bi_in, int blocks,
                                           int index_offset, uint8_t *const *peers, int rank, int world, size_t slot_bytes,
                                           int *__restrict__ state, int *__restrict__ tokens, int max_seq, int *status) {
    pdl_prologue();
    if (threadIdx.x != 0 || blockIdx.x != 0) return;
    uint8_t *local = peers[rank];
    const unsigned seq = *reinterpret_cast<volatile unsigned *>(local) + 1u;
    const unsigned limit = comm_spin_limit(local);
    float bv = -INFINITY;
    int bi = -1;
    for (int b = 0; b < blocks; b++) arg_better(bv, bi, bv_in[b], bi_in[b]);
    if (bi >= 0) bi += index_offset;
    const int par = (int)(seq & 1u);
    const size_t mine = comm_data_offset(par, rank, world, slot_bytes) + slot_bytes - 16;
    for (int p = 0; p < world; p++) {
        if (p == rank) continue;
        asm volatile("st.volatile.global.v2.u32 [%0], {%1, %2};" ::"l"(peers[p] + mine), "r"(__float_as_uint(bv)), "r"(seq) : "memory");
        asm volatile("st.volatile.global.v2.u32 [%0], {%1, %2};" ::"l"(peers[p] + mine + 8), "r"((unsigned)bi), "r"(seq) : "memory");
    }
    bool ok = true;
    for (int r = 0; r < world; r++) {
        if (r == rank) continue;
        const uint8_t *src = local + comm_data_offset(par, r, world, slot_bytes) + slot_bytes - 16;
        uint32_t vb = 0, ib = 0, t0 = 0, t1 = 0;
        unsigned spins = 0;
        do {
            asm volatile("ld.volatile.global.v2.u32 {%0, %1}, [%2];" : "=r"(vb), "=r"(t0) : "l"(src) : "memory");
            asm volatile("ld.volatile.global.v2.u32 {%0, %1}, [%2];" : "=r"(ib), "=r"(t1) : "l"(src + 8) : "memory");
        } while ((t0 != seq || t1 != seq) && ++spins <= limit);
        if (t0 != seq || t1 != seq) {
            ok = false;
            continue;
        }
        arg_better(bv, bi, __uint_as_float(vb), (int)ib);
    }
    if (!ok) atomicExch(status, 1);
    if (state[3]) atomicExch(status, 2);
    else dec_commit_token(bi, state, tokens, max_seq);
    *reinterpret_cast<volatile unsigned *>(local) = seq;   // this exchange is complete
}

// ---- prompt pass: the same operations over a block of rows (one row per prompt token) ----

// row r: h = embedding of tokens[r] (first layer) or h += delta; xn = RMSNorm(h) * w. One CTA per row.
__global__ void __launch_bounds__(256)
dec_norm_rows_kernel(float *__restrict__ h, const float *__restrict__ delta, const __nv_bfloat16 *__restrict__ embed,
                     const int *__restrict__ tokens, const float *__restrict__ w, float eps, void *__restrict__ xn, int act_dt,
                     int hidden) {
    __shared__ float red[32];
    const size_t r = blockIdx.x;
    float *hr = h + r * hidden;
    const float *dr = delta ? delta + r * hidden : nullptr;
    const __nv_bfloat16 *er = embed ? embed + (size_t)tokens[r] * hidden : nullptr;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = er ? __bfloat162float(er[i]) : hr[i] + dr[i];
        hr[i] = v;
        ss = fmaf(v, v, ss);
    }
    const float rms = sqrtf(block_sum(ss, red) / (float)hidden + eps);
    char *xr = reinterpret_cast<char *>(xn) + r * hidden * (act_dt == NNQ_F32 ? 4 : 2);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) store_act(xr, act_dt, i, (hr[i] / rms) * w[i]);
}

// grid (heads, rows): per-head RMSNorm + half-split rotation at position pos0 + row, append of k / v
__global__ void __launch_bounds__(256)
dec_qk_rope_rows_kernel(const float *__restrict__ q, const float *__restrict__ k, const float *__restrict__ v,
                        const float *__restrict__ qw, const float *__restrict__ kw, const float *__restrict__ cosv,
                        const float *__restrict__ sinv, int pos0, float eps, float *__restrict__ qrot, float *__restrict__ kcache,
                        float *__restrict__ vcache, int n_heads, int n_kv, int hd, int max_seq) {
    __shared__ float red[32];
    __shared__ float xs[256];
    const int head = blockIdx.x, row = blockIdx.y, d = threadIdx.x, pos = pos0 + row;
    const int half = hd / 2;
    const size_t qoff = (size_t)row * n_heads * hd, kvoff = (size_t)row * n_kv * hd;
    if (head >= n_heads + n_kv) {
        const int kvh = head - n_heads - n_kv;
        if (d < hd) vcache[((size_t)kvh * max_seq + pos) * hd + d] = v[kvoff + kvh * hd + d];
        return;
    }
    const bool is_q = head < n_heads;
    const float *src = is_q ? q + qoff + head * hd : k + kvoff + (head - n_heads) * hd;
    const float *w = is_q ? qw : kw;
    const float x = d < hd ? src[d] : 0.0f;
    const float rms = sqrtf(block_sum(x * x, red) / (float)hd + eps);
    if (d < hd) xs[d] = (x / rms) * w[d];
    __syncthreads();
    if (d >= hd) return;
    const int i = d < half ? d : d - half;
    const float c = cosv[(size_t)pos * half + i], sn = sinv[(size_t)pos * half + i];
    const float y = d < half ? xs[d] * c - xs[d + half] * sn : xs[d - half] * sn + xs[d] * c;
    if (is_q) qrot[qoff + head * hd + d] = y;
    else kcache[((size_t)(head - n_heads) * max_seq + pos) * hd + d] = y;
}

// Causal attention of a block of query rows over the cache: one warp per (kv head, R consecutive
// rows) serves the G query heads of the group for all R rows (G * R = 16 query vectors in shared
// memory), so that a key / value row is read once per R rows; row r sees keys 0 .. pos0 + r (the mask
// of the reference's prompt pass: crates/nn-core/src/layers/attention/sdpa.rs:118-141). Same
// batch-of-32-keys scheme as the decode kernel, normalised output written directly.
template <int G, int R>
__global__ void __launch_bounds__(32)
dec_attn_rows_kernel(const float *__restrict__ qrot, const float *__restrict__ kcache, const float *__restrict__ vcache, int pos0,
                     int n, float scale, void *__restrict__ out, int act_dt, int n_heads, int hd, int max_seq) {
    constexpr int P = G * R;   // pair p = r * G + g
    __shared__ __align__(16) float qs[P][128];
    const int kvh = blockIdx.x, r0 = blockIdx.y * R, lane = threadIdx.x;
    const int rows = min(R, n - r0);
    const int jmax = pos0 + r0 + rows;   // keys the last row of this block sees
#pragma unroll
    for (int p = 0; p < P; p++) {
        const int row = r0 + min(p / G, rows - 1);   // rows past the end repeat the last one; not stored
        *reinterpret_cast<float4 *>(&qs[p][4 * lane]) =
            *reinterpret_cast<const float4 *>(qrot + (size_t)row * n_heads * hd + (kvh * G + p % G) * hd + 4 * lane);
    }
    __syncwarp();
    float m[P], l[P];
    float4 acc[P];
#pragma unroll
    for (int p = 0; p < P; p++) {
        m[p] = -INFINITY;
        l[p] = 0.0f;
        acc[p] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    const float *kb = kcache + (size_t)kvh * max_seq * hd, *vb = vcache + (size_t)kvh * max_seq * hd;
    for (int b0 = 0; b0 < jmax; b0 += 32) {
        const int j = b0 + lane;
        const float4 *krow = reinterpret_cast<const float4 *>(kb + (size_t)(j < jmax ? j : b0) * hd);
        float dot[P];
#pragma unroll
        for (int p = 0; p < P; p++) dot[p] = 0.0f;
#pragma unroll 8
        for (int d4 = 0; d4 < 32; d4++) {
            const float4 kv = krow[d4];
#pragma unroll
            for (int p = 0; p < P; p++) {
                const float4 qv = *reinterpret_cast<const float4 *>(&qs[p][4 * d4]);
                dot[p] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, dot[p]))));
            }
        }
#pragma unroll
        for (int p = 0; p < P; p++) {
            // key j is visible to row r0 + p / G up to position pos0 + row; the first batch holds key 0
            // for every row, so the running maximum is finite from then on
            const bool valid = j <= pos0 + r0 + min(p / G, rows - 1);
            const float sc = valid ? dot[p] * scale : -INFINITY;
            float bm = sc;
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xFFFFFFFFu, bm, off));
            const float mn = fmaxf(m[p], bm);
            const float corr = expf(m[p] - mn);
            dot[p] = expf(sc - mn);   // the probability, kept in place of the score
            float ps = dot[p];
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) ps += __shfl_xor_sync(0xFFFFFFFFu, ps, off);
            l[p] = l[p] * corr + ps;
            acc[p].x *= corr; acc[p].y *= corr; acc[p].z *= corr; acc[p].w *= corr;
            m[p] = mn;
        }
        const int nb = min(32, jmax - b0);
        for (int jj = 0; jj < nb; jj++) {
            const float4 vv = *reinterpret_cast<const float4 *>(vb + (size_t)(b0 + jj) * hd + 4 * lane);
#pragma unroll
            for (int p = 0; p < P; p++) {
                const float pj = __shfl_sync(0xFFFFFFFFu, dot[p], jj);
                acc[p].x = fmaf(pj, vv.x, acc[p].x);
                acc[p].y = fmaf(pj, vv.y, acc[p].y);
                acc[p].z = fmaf(pj, vv.z, acc[p].z);
                acc[p].w = fmaf(pj, vv.w, acc[p].w);
            }
        }
    }
#pragma unroll
    for (int p = 0; p < P; p++) {
        if (p / G >= rows) continue;
        char *orow = reinterpret_cast<char *>(out) + (size_t)(r0 + p / G) * n_heads * hd * (act_dt == NNQ_F32 ? 4 : 2);
        const int base = (kvh * G + p % G) * hd + 4 * lane;
        store_act(orow, act_dt, base, acc[p].x / l[p]);
        store_act(orow, act_dt, base + 1, acc[p].y / l[p]);
        store_act(orow, act_dt, base + 2, acc[p].z / l[p]);
        store_act(orow, act_dt, base + 3, acc[p].w / l[p]);
    }
}

// position of the last prompt token, for the commit of its greedy successor
__global__ void dec_set_pos_kernel(int *state, int pos) {
    if (threadIdx.x == 0 && blockIdx.x == 0) state[1] = pos;
}

}  // namespace nnq

using namespace nnq;

extern "C" {

static nnq_status dev_alloc(nnq_ctx *ctx, void **p, size_t bytes, const char *what) {
    nnq_status s = check_cuda(ctx, cudaMalloc(p, bytes ? bytes : 16), what);
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemset(*p, 0, bytes ? bytes : 16), what);
    return s;
}

nnq_status nnq_decoder_create(nnq_ctx *ctx, const nnq_decoder_config *cfg, nnq_decoder **out) {
    if (!ctx || !cfg || !out) return NNQ_ERR_INVALID_ARG;
    *out = nullptr;
    nnq_decoder_config c = *cfg;
    if (c.tp_world == 0) c.tp_world = 1;   // a zeroed field means no tensor parallelism
    if (c.hidden < 1 || c.n_heads < 1 || c.n_kv_heads < 1 || c.ffn < 1 || c.n_layers < 1 || c.vocab < 1 || c.max_seq < 1)
        return fail(ctx, NNQ_ERR_INVALID_ARG, "bad decoder dimensions");
    if (c.head_dim != 128) return fail(ctx, NNQ_ERR_UNSUPPORTED, "the attention kernel is written for head_dim = 128 (got %d)", c.head_dim);
    const int grp = c.n_heads % c.n_kv_heads ? 0 : c.n_heads / c.n_kv_heads;
    if (grp != 1 && grp != 2 && grp != 4 && grp != 8)
        return fail(ctx, NNQ_ERR_UNSUPPORTED, "query heads per key/value head must be 1, 2, 4 or 8");
    if (c.act_dtype != NNQ_F32 && c.act_dtype != NNQ_BF16) return fail(ctx, NNQ_ERR_INVALID_ARG, "unknown activation dtype");
    if (c.tp_world < 1 || c.tp_world > 8 || c.tp_rank < 0 || c.tp_rank >= c.tp_world)
        return fail(ctx, NNQ_ERR_INVALID_ARG, "bad tensor-parallel rank %d of %d", c.tp_rank, c.tp_world);
    if (c.n_kv_heads % c.tp_world || c.ffn % c.tp_world)
        return fail(ctx, NNQ_ERR_UNSUPPORTED, "key/value heads and the FFN width must divide by the tensor-parallel world size");
    if (!(c.rope_theta > 0.0)) return fail(ctx, NNQ_ERR_INVALID_ARG, "rope_theta must be positive");
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s != NNQ_OK) return s;
    nnq_decoder *d = new (std::nothrow) nnq_decoder();
    if (!d) return fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
    memset(d, 0, sizeof(*d));
    d->ctx = ctx;
    d->cfg = c;
    d->act_dt = c.act_dtype;
    d->embed_ld = d->xn_ld = c.hidden;
    d->lh = c.n_heads / c.tp_world;
    d->lkv = c.n_kv_heads / c.tp_world;
    d->head_rows = c.vocab;
    d->head_row0 = 0;
    d->host_pos = -1;
    d->layers = new (std::nothrow) nnq_decoder::Layer[c.n_layers]();
    if (!d->layers) {
        delete d;
        return fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
    }
    const int hd = c.head_dim, half = hd / 2, qdim = d->lh * hd, kvdim = d->lkv * hd, lffn = c.ffn / c.tp_world;
    const size_t es = c.act_dtype == NNQ_F32 ? 4 : 2;
    const size_t cache = (size_t)c.n_layers * d->lkv * c.max_seq * hd * 4;
    s = dev_alloc(ctx, (void **)&d->d_cos, (size_t)c.max_seq * half * 4, "rope table");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_sin, (size_t)c.max_seq * half * 4, "rope table");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_kcache, cache, "key cache");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_vcache, cache, "value cache");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_h, (size_t)c.hidden * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_delta, (size_t)c.hidden * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_q, (size_t)qdim * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_k, (size_t)kvdim * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_v, (size_t)kvdim * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_qrot, (size_t)qdim * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_g, (size_t)lffn * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_u, (size_t)lffn * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_logits, (size_t)c.vocab * 4, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_part, (size_t)d->lh * kAttnRanges * (hd + 4) * 4, "attention partials");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_arrived, (size_t)(d->lkv > 0 ? d->lkv : 1) * 4, "attention arrival counters");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemset(d->d_arrived, 0, (size_t)(d->lkv > 0 ? d->lkv : 1) * 4), "attention arrival counters clear");
    if (s == NNQ_OK) s = dev_alloc(ctx, &d->d_xn, (size_t)c.hidden * es, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, &d->d_attn, (size_t)qdim * es, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, &d->d_mid, (size_t)lffn * es, "decoder buffer");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_state, (kStateWords + 2 * kArgmaxBlocks) * 4, "decoder state");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_tokens, (size_t)c.max_seq * 4, "token log");
    if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->d_final_norm, (size_t)c.hidden * 4, "final norm");
    for (int l = 0; l < c.n_layers && s == NNQ_OK; l++) {
        nnq_decoder::Layer &L = d->layers[l];
        s = dev_alloc(ctx, (void **)&L.in_norm, (size_t)c.hidden * 4, "norm weight");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&L.post_norm, (size_t)c.hidden * 4, "norm weight");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&L.q_norm, (size_t)hd * 4, "norm weight");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&L.k_norm, (size_t)hd * 4, "norm weight");
    }
    if (s == NNQ_OK) {
        // tables exactly as the reference builds them: inv_freq in f32, the angle rounded to f32
        float *hc = new (std::nothrow) float[(size_t)c.max_seq * half], *hs = new (std::nothrow) float[(size_t)c.max_seq * half];
        if (!hc || !hs) s = fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
        if (s == NNQ_OK) {
            for (int i = 0; i < half; i++) {
                const float inv = (float)(1.0 / pow(c.rope_theta, (double)(2 * i) / (double)hd));
                for (int p = 0; p < c.max_seq; p++) {
                    const float angle = (float)((double)p * (double)inv);
                    hc[(size_t)p * half + i] = cosf(angle);
                    hs[(size_t)p * half + i] = sinf(angle);
                }
            }
            s = check_cuda(ctx, cudaMemcpy(d->d_cos, hc, (size_t)c.max_seq * half * 4, cudaMemcpyHostToDevice), "rope table");
            if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(d->d_sin, hs, (size_t)c.max_seq * half * 4, cudaMemcpyHostToDevice), "rope table");
        }
        delete[] hc;
        delete[] hs;
    }
    if (s != NNQ_OK) {
        nnq_decoder_destroy(d);
        return s;
    }
    *out = d;
    return NNQ_OK;
}

static bool shape_is(const nnq_weight *w, int64_t n, int64_t k) { return w && w->n == n && w->k == k; }

nnq_status nnq_decoder_set_layer(nnq_decoder *d, int layer, const nnq_weight *q, const nnq_weight *k, const nnq_weight *v,
                                 const nnq_weight *o, const nnq_weight *gate, const nnq_weight *up, const nnq_weight *down,
                                 const float *in_norm, const float *post_norm, const float *q_norm, const float *k_norm) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    if (!d->layers) return fail(ctx, NNQ_ERR_INVALID_ARG, "this decoder is made of blocks: use nnq_decoder_set_block");
    if (layer < 0 || layer >= c.n_layers) return fail(ctx, NNQ_ERR_INVALID_ARG, "layer %d out of range", layer);
    if (!in_norm || !post_norm || !q_norm || !k_norm) return fail(ctx, NNQ_ERR_INVALID_ARG, "NULL norm weight");
    // with tensor parallelism: this rank's column shards of q / k / v / gate / up and row shards of o / down
    const int64_t qdim = (int64_t)d->lh * c.head_dim, kvdim = (int64_t)d->lkv * c.head_dim, lffn = c.ffn / c.tp_world;
    if (!shape_is(q, qdim, c.hidden) || !shape_is(k, kvdim, c.hidden) || !shape_is(v, kvdim, c.hidden) ||
        !shape_is(o, c.hidden, qdim) || !shape_is(gate, lffn, c.hidden) || !shape_is(up, lffn, c.hidden) ||
        !shape_is(down, c.hidden, lffn))
        return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "projection shapes of layer %d do not match the configuration", layer);
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s != NNQ_OK) return s;
    nnq_decoder::Layer &L = d->layers[layer];
    L.q = q; L.k = k; L.v = v; L.o = o; L.gate = gate; L.up = up; L.down = down;
    s = check_cuda(ctx, cudaMemcpy(L.in_norm, in_norm, (size_t)c.hidden * 4, cudaMemcpyDefault), "norm weight");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(L.post_norm, post_norm, (size_t)c.hidden * 4, cudaMemcpyDefault), "norm weight");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(L.q_norm, q_norm, (size_t)c.head_dim * 4, cudaMemcpyDefault), "norm weight");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(L.k_norm, k_norm, (size_t)c.head_dim * 4, cudaMemcpyDefault), "norm weight");
    return s;
}

nnq_status nnq_decoder_set_head(nnq_decoder *d, const void *embed_bf16_dev, const float *final_norm, const nnq_weight *lm_head) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    if (!d->layers) return fail(ctx, NNQ_ERR_INVALID_ARG, "this decoder is made of blocks: use nnq_decoder_set_head_weights");
    if (!embed_bf16_dev || !final_norm) return fail(ctx, NNQ_ERR_INVALID_ARG, "NULL tensor");
    // tensor parallel: either the whole [vocab, hidden] projection on every rank, or this rank's
    // rows [rank * vocab / world, (rank + 1) * vocab / world) of it (vocabulary parallel: the ranks
    // then agree on the greedy token through the communicator)
    const nnq_decoder_config &c = d->cfg;
    if (shape_is(lm_head, c.vocab, c.hidden)) {
        d->head_rows = c.vocab;
        d->head_row0 = 0;
    } else if (c.tp_world > 1 && c.vocab % c.tp_world == 0 && shape_is(lm_head, c.vocab / c.tp_world, c.hidden)) {
        d->head_rows = c.vocab / c.tp_world;
        d->head_row0 = c.tp_rank * d->head_rows;
    } else {
        return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "vocabulary projection must be [vocab, hidden] (or this rank's [vocab / world, hidden] rows)");
    }
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s != NNQ_OK) return s;
    d->d_embed = embed_bf16_dev;
    d->lm_head = lm_head;
    d->ready = 1;
    return check_cuda(ctx, cudaMemcpy(d->d_final_norm, final_norm, (size_t)d->cfg.hidden * 4, cudaMemcpyDefault), "final norm");
}

// ---- block decoders ----

static nnq_status check_block(nnq_ctx *ctx, int l, const nnq_block_config &b) {
    if (b.mixer < NNQ_MIXER_ATTENTION || b.mixer > NNQ_MIXER_NONE) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: unknown mixer %d", l, b.mixer);
    if ((b.mixer == NNQ_MIXER_LATENT || b.mixer == NNQ_MIXER_NONE) && !b.post_norm) return fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: this mixer takes post_norm", l);
    if (b.ffn_act != NNQ_ACT_SILU && b.ffn_act != NNQ_ACT_GELU_TANH) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: unknown activation %d", l, b.ffn_act);
    if (b.mixer == NNQ_MIXER_NONE) {
        if (b.experts < 0 || b.ffn < 0 || (b.experts > 0) == (b.ffn > 0)) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: a feed-forward or a mixture of experts", l);
        return NNQ_OK;
    }
    if (b.experts || b.ffn_act != NNQ_ACT_SILU) return fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: experts and other activations than silu stand in blocks without a mixer", l);
    if (b.mixer == NNQ_MIXER_LATENT) {
        if (b.heads < 1 || b.dim < 1 || b.vdim < 1 || b.ffn || b.q_rank < 1 || b.kv_rank < 1 || b.window < 0 || !(b.scale > 0.0f)) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad sizes", l);
        if (b.rot_dims < 0 || b.rot_dims % 2 || (b.rot_dims && !(b.rot_base > 0.0))) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad rotation", l);
        if (b.vdim > kAttnMaxDim || b.dim + b.rot_dims > 2 * kAttnMaxDim) return fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: attention heads of %d + %d / %d are above %d / %d", l, b.dim, b.rot_dims, b.vdim, 2 * kAttnMaxDim, kAttnMaxDim);
        return NNQ_OK;
    }
    if (b.heads < 1 || b.dim < 1 || b.vdim < 1 || b.ffn < 0) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad sizes", l);
    if (b.rot_dims < 0 || b.rot_dims % 2 || b.rot_dims > b.dim || (b.rot_dims && !(b.rot_base > 0.0)))
        return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad rotation (%d of %d dimensions)", l, b.rot_dims, b.dim);
    if (b.mixer == NNQ_MIXER_ATTENTION) {
        if (b.kv_heads < 1 || b.heads % b.kv_heads) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: %d query heads over %d key/value heads", l, b.heads, b.kv_heads);
        if (b.window < 0 || b.conv_taps < 0) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad window or convolution", l);
        if (b.dim > kAttnMaxDim || b.vdim > kAttnMaxDim)
            return fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: attention heads of %d / %d are above %d", l, b.dim, b.vdim, kAttnMaxDim);
    } else {
        if (b.decay_rank < 0 || (b.decay_rank > 0 && !(b.decay_tau > 0.0f))) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d: bad decay", l);
        if (b.dim > kRecMaxKeyDim || b.vdim > 2048)
            return fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: recurrent heads of %d / %d are above %d / 2048", l, b.dim, b.vdim, kRecMaxKeyDim);
    }
    return NNQ_OK;
}

static nnq_block_layout layout_of(const nnq_block_config &b, int hidden) {
    nnq_block_layout y = {};
    y.in_k = round_up(hidden, 64);   // one k step of the tensor-core products
    y.ffn_step = 1;
    if (b.mixer == NNQ_MIXER_LATENT) {
        y.q = 0;
        y.k = b.kv_from < 0 ? round_up(b.q_rank, 8) : -1;
        y.v = y.g = y.a1 = y.gate = y.up = -1;
        y.in_cols = round_up(b.q_rank, 8) + (b.kv_from < 0 ? round_up(b.kv_rank + b.rot_dims, 8) : 0);
        y.q_ld = round_up(b.q_rank, 64);
        y.kv_ld = round_up(b.kv_rank, 64);
        y.dim_ld = round_up(b.dim, 64);
        y.vdim_ld = round_up(b.vdim, 64);
        y.ffn_col = y.out_k = round_up(b.heads * b.vdim, 64);
        return y;
    }
    if (b.mixer == NNQ_MIXER_NONE) {
        y.q = y.k = y.v = y.g = y.a1 = -1;
        y.gate = 0;
        y.up = 1;
        y.ffn_step = 2;
        y.out_k = round_up(b.ffn, 64);
        y.in_cols = 2 * y.out_k;
        return y;
    }
    const bool attn = b.mixer == NNQ_MIXER_ATTENTION;
    const int kvh = attn ? b.kv_heads : b.heads;
    int at = 0;
    auto take = [&](int width) {
        if (width == 0) return -1;
        const int c = at;
        at += round_up(width, 8);
        return c;
    };
    y.q = take(b.heads * b.dim);
    y.k = take(kvh * b.dim);
    y.v = take(kvh * b.vdim);
    y.g = take(!attn || b.out_gate ? b.heads * b.vdim : 0);
    y.a1 = take(attn ? 0 : b.decay_rank);
    y.gate = take(b.ffn);
    y.up = take(b.ffn);
    y.in_cols = at;
    y.ffn_col = round_up(b.heads * b.vdim, 8);
    // (a gap in front of the feed-forward's columns is cleared together with them: there are some then)
    y.out_k = round_up(y.ffn_col + (b.ffn > 0 || y.ffn_col == b.heads * b.vdim ? b.ffn : 8), 64);
    return y;
}

nnq_status nnq_decoder_create_blocks(nnq_ctx *ctx, const nnq_decoder_config *cfg, const nnq_block_config *blocks, int block_rows, nnq_decoder **out) {
    if (!ctx || !cfg || !blocks || !out) return NNQ_ERR_INVALID_ARG;
    *out = nullptr;
    nnq_decoder_config c = *cfg;
    if (c.tp_world == 0) c.tp_world = 1;
    if (c.tp_world != 1) return fail(ctx, NNQ_ERR_UNSUPPORTED, "block decoders run on one device");
    if (c.hidden < 1 || c.n_layers < 1 || c.vocab < 1 || c.max_seq < 1 || block_rows < 0) return fail(ctx, NNQ_ERR_INVALID_ARG, "bad decoder dimensions");
    if (c.act_dtype != NNQ_F32 && c.act_dtype != NNQ_BF16) return fail(ctx, NNQ_ERR_INVALID_ARG, "unknown activation dtype");
    nnq_status s = NNQ_OK;
    int first_mix = -1;
    for (int l = 0; l < c.n_layers; l++) {
        if ((s = check_block(ctx, l, blocks[l])) != NNQ_OK) return s;
        if (blocks[l].mixer == NNQ_MIXER_LATENT && blocks[l].kv_from >= 0) {
            const nnq_block_config &b = blocks[l], *o = b.kv_from < l ? &blocks[b.kv_from] : nullptr;
            if (!o || o->mixer != NNQ_MIXER_LATENT || o->kv_from >= 0 || o->kv_rank != b.kv_rank || o->rot_dims != b.rot_dims || (b.rot_dims && o->rot_base != b.rot_base))
                return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d cannot read the latents of block %d", l, b.kv_from);
        }
        if (blocks[l].mixer != NNQ_MIXER_ATTENTION || !blocks[l].value_mix) continue;
        if (first_mix < 0) first_mix = l;
        else if (blocks[l].kv_heads * blocks[l].vdim != blocks[first_mix].kv_heads * blocks[first_mix].vdim)
            return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d mixes values of another width than block %d", l, first_mix);
    }
    if ((s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice")) != NNQ_OK) return s;
    nnq_decoder *d = new (std::nothrow) nnq_decoder();
    if (!d) return fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
    memset(d, 0, sizeof(*d));
    d->ctx = ctx;
    d->cfg = c;
    d->act_dt = c.act_dtype;
    d->head_rows = c.vocab;
    d->host_pos = -1;
    d->xn_ld = d->embed_ld = round_up(c.hidden, 64);
    d->blocks = new (std::nothrow) nnq_decoder::Block[c.n_layers]();
    if (!d->blocks) {
        delete d;
        return fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
    }
    bool experts = false;
    for (int l = 0; l < c.n_layers; l++) experts = experts || blocks[l].experts > 0;
    const int want_rows = block_rows ? block_rows : (experts ? kPrefillRowsExperts : kPrefillRows);
    const int rows = d->pf_rows = want_rows < c.max_seq ? want_rows : c.max_seq;
    const size_t R = rows, es = c.act_dtype == NNQ_F32 ? 4 : 2;
    size_t proj = 0, act = 0, q = 0, k = 0, o = 0, vf = 0, part = 0, counters = 1;
    size_t cq = 0, lin_c = 0, lin_r = 0, kv = 0, q2 = 0, qrot = 0, kfull = 0, vfull = 0, qlat = 0;
    auto alloc = [&](void *pp, size_t bytes, const char *what) {
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)pp, bytes, what);
    };
    auto most = [](size_t &m, size_t v) { if (v > m) m = v; };
    for (int l = 0; l < c.n_layers && s == NNQ_OK; l++) {
        nnq_decoder::Block &B = d->blocks[l];
        B.cfg = blocks[l];
        B.lay = layout_of(B.cfg, c.hidden);
        const nnq_block_config &b = B.cfg;
        most(proj, B.lay.in_cols);
        most(act, B.lay.out_k);
        alloc(&B.norm, (size_t)c.hidden * 4, "norm weight");
        if (b.post_norm) alloc(&B.norm_bias, (size_t)c.hidden * 4, "norm bias");
        if (b.mixer == NNQ_MIXER_ATTENTION) {
            B.dim_ld = round_up(b.dim, 4);
            B.vdim_ld = round_up(b.vdim, 4);
            // a block of rows writes its keys before it reads: window - 1 older positions stay beside them
            B.cap = b.window > 0 && (long long)b.window - 1 + rows < c.max_seq ? b.window - 1 + rows : c.max_seq;
            B.ranges = attn_step_ranges(ctx->sm_count, b.heads, b.kv_heads, b.window > 0 ? b.window : c.max_seq, c.max_seq);
            B.mix_mode = !b.value_mix ? 0 : (l == first_mix ? 1 : 2);
            const int channels = b.heads * b.dim + b.kv_heads * (b.dim + b.vdim);
            alloc(&B.kcache, (size_t)b.kv_heads * B.cap * B.dim_ld * 4, "key cache");
            alloc(&B.vcache, (size_t)b.kv_heads * B.cap * B.vdim_ld * 4, "value cache");
            if (b.conv_taps > 0) {
                alloc(&B.conv, (size_t)channels * b.conv_taps * 4, "convolution taps");
                alloc(&B.conv_ring, (size_t)channels * b.conv_taps * 4, "convolution state");
            }
            most(q, (size_t)b.heads * B.dim_ld);
            if (b.value_mix) most(vf, (size_t)b.kv_heads * b.vdim);
            most(part, attn_step_part_floats(b.heads, b.kv_heads, B.vdim_ld, B.ranges));
            most(counters, attn_step_counters(b.heads, b.kv_heads));
        } else if (b.mixer == NNQ_MIXER_LATENT) {
            const nnq_block_layout &y = B.lay;
            const int rot_ld = round_up(b.rot_dims, 64), window = b.window > 0 ? b.window : c.max_seq;
            if (!latent_step_supported(c.act_dtype, y.kv_ld, rot_ld)) s = fail(ctx, NNQ_ERR_UNSUPPORTED, "block %d: a latent of %d + %d is too wide", l, b.kv_rank, b.rot_dims);
            alloc(&B.q_norm, (size_t)b.q_rank * 4, "norm weight");
            if (b.kv_from < 0) {
                alloc(&B.kv_norm, (size_t)b.kv_rank * 4, "norm weight");
                long long widest = window;   // the ring serves every block that reads it
                for (int j = l + 1; j < c.n_layers; j++)
                    if (blocks[j].mixer == NNQ_MIXER_LATENT && blocks[j].kv_from == l && (blocks[j].window > 0 ? blocks[j].window : c.max_seq) > widest)
                        widest = blocks[j].window > 0 ? blocks[j].window : c.max_seq;
                B.cap = widest - 1 + rows < c.max_seq ? (int)widest - 1 + rows : c.max_seq;
                alloc(&B.ring_c, (size_t)B.cap * y.kv_ld * es, "latents");
                alloc(&B.ring_r, (size_t)B.cap * rot_ld * es, "rotated key parts");
            } else {
                B.cap = d->blocks[b.kv_from].cap;
                B.ring_c = d->blocks[b.kv_from].ring_c;
                B.ring_r = d->blocks[b.kv_from].ring_r;
            }
            B.ranges = latent_step_ranges(ctx->sm_count, b.heads, window, c.max_seq, c.act_dtype);
            const size_t keys = (long long)window - 1 + rows < c.max_seq ? window - 1 + rows : c.max_seq;
            most(cq, y.q_ld);
            if (B.cap < c.max_seq) {
                most(lin_c, keys * y.kv_ld);
                most(lin_r, keys * rot_ld);
            }
            most(kv, keys * b.heads * (y.dim_ld + y.vdim_ld));
            most(q2, (size_t)b.heads * (b.dim + b.rot_dims));
            if (!latent_tc_supported(c.act_dtype, b.dim, b.rot_dims, b.vdim)) {
                const size_t dl = round_up(b.dim + b.rot_dims, 4), vl = round_up(b.vdim, 4);
                most(qrot, b.heads * dl);
                most(kfull, keys * b.heads * dl);
                most(vfull, keys * b.heads * vl);
            }
            most(qlat, latent_step_query_floats(b.heads, y.kv_ld, rot_ld));
            most(part, (size_t)B.ranges * b.heads * (y.kv_ld + 4));
        } else if (b.mixer == NNQ_MIXER_RECURRENT) {
            B.dim_ld = b.dim <= 64 ? 64 : round_up(b.dim, 128);
            alloc(&B.rec_state, (size_t)b.heads * b.dim * b.vdim * 4, "recurrent state");
            if (b.decay_rank > 0) {
                alloc(&B.a2t, (size_t)b.heads * b.dim * b.decay_rank * 4, "decay weight");
                alloc(&B.a2b, (size_t)b.heads * b.dim * 4, "decay bias");
            } else {
                alloc(&B.decay, (size_t)b.heads * 4, "decay");
            }
            most(q, (size_t)b.heads * B.dim_ld);
            most(k, (size_t)b.heads * B.dim_ld);
            most(o, (size_t)b.heads * b.vdim);
        }
        if (b.rot_dims > 0) {
            for (int j = 0; j < l && !B.cosv; j++)
                if (d->blocks[j].cfg.rot_dims == b.rot_dims && d->blocks[j].cfg.rot_base == b.rot_base) {
                    B.cosv = d->blocks[j].cosv;
                    B.sinv = d->blocks[j].sinv;
                }
            if (!B.cosv) {
                const int half = b.rot_dims / 2;
                const size_t n = (size_t)c.max_seq * half;
                B.owns_tables = true;
                alloc(&B.cosv, n * 4, "rotation table");
                alloc(&B.sinv, n * 4, "rotation table");
                float *hc = new (std::nothrow) float[n], *hs = new (std::nothrow) float[n];
                if (!hc || !hs) s = fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
                if (s == NNQ_OK) {
                    // angles in f64: the tables are the correctly rounded sine and cosine at any position
                    for (int i = 0; i < half; i++) {
                        const double f = pow(b.rot_base, -2.0 * i / b.rot_dims);
                        for (int p = 0; p < c.max_seq; p++) {
                            hc[(size_t)p * half + i] = (float)cos(p * f);
                            hs[(size_t)p * half + i] = (float)sin(p * f);
                        }
                    }
                    s = check_cuda(ctx, cudaMemcpy(B.cosv, hc, n * 4, cudaMemcpyHostToDevice), "rotation table");
                    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(B.sinv, hs, n * 4, cudaMemcpyHostToDevice), "rotation table");
                }
                delete[] hc;
                delete[] hs;
            }
        }
    }
    if (s == NNQ_OK) {
        alloc(&d->b_cq, R * cq * es, "row buffer");
        alloc(&d->b_lin_c, lin_c * es, "row buffer");
        alloc(&d->b_lin_r, lin_r * es, "row buffer");
        alloc(&d->b_kv, kv * es, "expanded keys and values");
        alloc(&d->b_q2, R * q2 * 4, "row buffer");
        alloc(&d->b_qrot, R * qrot * 4, "row buffer");
        alloc(&d->b_kfull, kfull * 4, "expanded keys");
        alloc(&d->b_vfull, vfull * 4, "expanded values");
        alloc(&d->b_qlat, qlat * 4, "row buffer");
    }
    alloc(&d->d_h, (size_t)c.hidden * 4, "decoder buffer");
    alloc(&d->b_h2, (size_t)c.hidden * 4, "decoder buffer");
    alloc(&d->d_delta, (size_t)d->xn_ld * 4, "decoder buffer");
    alloc(&d->d_xn, (size_t)d->xn_ld * es, "decoder buffer");
    alloc(&d->d_logits, (size_t)c.vocab * 4, "decoder buffer");
    alloc(&d->d_final_norm, (size_t)c.hidden * 4, "final norm");
    alloc(&d->d_state, (kStateWords + 2 * kArgmaxBlocks) * 4, "decoder state");
    alloc(&d->d_tokens, (size_t)c.max_seq * 4, "token log");
    alloc(&d->d_part, part * 4, "attention partials");
    alloc(&d->d_arrived, counters * 4, "attention arrival counters");
    alloc(&d->pf_h, R * c.hidden * 4, "row buffer");
    alloc(&d->pf_delta, R * d->xn_ld * 4, "row buffer");   // (the experts' rows are as wide as the products' input)
    alloc(&d->pf_xn, R * d->xn_ld * es, "row buffer");
    alloc(&d->pf_tokens, (R + 1) * 4, "row buffer");   // the token in front of a block of rows, then the block's
    alloc(&d->pf_want, R * 4, "row buffer");
    alloc(&d->b_proj, R * proj * 4, "row buffer");
    alloc(&d->b_act, R * act * es, "row buffer");
    alloc(&d->b_q, R * q * 4, "row buffer");
    alloc(&d->b_k, R * k * 4, "row buffer");
    alloc(&d->b_a, R * k * 4, "row buffer");
    alloc(&d->b_o, R * o * 4, "row buffer");
    alloc(&d->b_vfirst, R * vf * 4, "row buffer");
    if (s != NNQ_OK) {
        nnq_decoder_destroy(d);
        return s;
    }
    *out = d;
    return NNQ_OK;
}

nnq_status nnq_decoder_block_layout(const nnq_decoder *d, int layer, nnq_block_layout *out) {
    if (!d || !out) return NNQ_ERR_INVALID_ARG;
    if (!d->blocks || layer < 0 || layer >= d->cfg.n_layers) return fail(d->ctx, NNQ_ERR_INVALID_ARG, "no block %d", layer);
    *out = d->blocks[layer].lay;
    return NNQ_OK;
}

nnq_status nnq_decoder_set_block(nnq_decoder *d, int layer, const nnq_block_weights *w) {
    if (!d || !w) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    if (!d->blocks || layer < 0 || layer >= c.n_layers) return fail(ctx, NNQ_ERR_INVALID_ARG, "no block %d", layer);
    nnq_decoder::Block &B = d->blocks[layer];
    const nnq_block_config &b = B.cfg;
    if (b.experts) {
        if (!w->moe || w->moe->hidden != B.lay.in_k || w->moe->n_experts != b.experts || w->moe->layout != NNQ_MOE_NK_PAIRS)
            return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "block %d takes %d bf16 experts of width %d", layer, b.experts, B.lay.in_k);
    } else if (!shape_is(w->in, B.lay.in_cols, B.lay.in_k) || !shape_is(w->out, c.hidden, B.lay.out_k))
        return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "products of block %d must be [%d, %d] and [%d, %d]", layer, B.lay.in_cols, B.lay.in_k, c.hidden, B.lay.out_k);
    if (!w->norm || (B.conv && !w->conv) || (B.a2t && (!w->decay_w || !w->decay_b)) || (B.decay && !w->decay))
        return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d lacks a tensor", layer);
    if (b.post_norm && !w->norm_bias) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d lacks a tensor", layer);
    if (b.mixer == NNQ_MIXER_LATENT) {
        if (!w->q_norm || (B.kv_norm && !w->kv_norm)) return fail(ctx, NNQ_ERR_INVALID_ARG, "block %d lacks a tensor", layer);
        if (!shape_is(w->uq, (int64_t)b.heads * (b.dim + b.rot_dims), B.lay.q_ld) || !shape_is(w->ukv, (int64_t)b.heads * (B.lay.dim_ld + B.lay.vdim_ld), B.lay.kv_ld) ||
            w->ukv->fmt != NNQ_BF16_DENSE)
            return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "latent products of block %d must be [%d, %d] and (bf16) [%d, %d]", layer, b.heads * (b.dim + b.rot_dims), B.lay.q_ld,
                        b.heads * (B.lay.dim_ld + B.lay.vdim_ld), B.lay.kv_ld);
    }
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    auto copy = [&](float *dst, const float *src, size_t n, const char *what) {
        if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(dst, src, n * 4, cudaMemcpyDefault), what);
    };
    auto optional = [&](float **dst, const float *src, size_t n, const char *what) {
        if (!src || s != NNQ_OK) return;
        if (!*dst) s = dev_alloc(ctx, (void **)dst, n * 4, what);
        copy(*dst, src, n, what);
    };
    copy(B.norm, w->norm, c.hidden, "norm weight");
    if (b.post_norm) copy(B.norm_bias, w->norm_bias, c.hidden, "norm bias");
    if (B.q_norm) copy(B.q_norm, w->q_norm, b.q_rank, "norm weight");
    if (B.kv_norm) copy(B.kv_norm, w->kv_norm, b.kv_rank, "norm weight");
    if (b.experts && s == NNQ_OK) s = moe_reserve(ctx, w->moe, d->pf_rows);
    optional(&B.bias_in, w->bias_in, B.lay.in_cols, "bias");
    optional(&B.bias_out, w->bias_out, c.hidden, "bias");
    optional(&B.head_norm, b.mixer == NNQ_MIXER_RECURRENT ? w->head_norm : nullptr, b.vdim, "head norm weight");
    if (B.conv) copy(B.conv, w->conv, (size_t)(b.heads * b.dim + b.kv_heads * (b.dim + b.vdim)) * b.conv_taps, "convolution taps");
    if (B.decay) copy(B.decay, w->decay, b.heads, "decay");
    if (B.a2t && s == NNQ_OK) {
        // [channels, rank] -> [rank, channels]: neighbouring channels are neighbouring lanes
        const size_t n = (size_t)b.heads * b.dim, r = b.decay_rank;
        float *src = new (std::nothrow) float[2 * n * r];
        if (!src) return fail(ctx, NNQ_ERR_OUT_OF_MEMORY, "host allocation failed");
        float *t = src + n * r;
        s = check_cuda(ctx, cudaMemcpy(src, w->decay_w, n * r * 4, cudaMemcpyDefault), "decay weight");
        for (size_t i = 0; i < n; i++)
            for (size_t j = 0; j < r; j++) t[j * n + i] = src[i * r + j];
        copy(B.a2t, t, n * r, "decay weight");
        delete[] src;
        copy(B.a2b, w->decay_b, n, "decay bias");
    }
    B.lambda = w->lambda;
    if (s == NNQ_OK) {
        B.in = w->in;
        B.out = w->out;
        B.uq = w->uq;
        B.ukv = w->ukv;
        B.moe = w->moe;
    }
    return s;
}

nnq_status nnq_decoder_set_head_weights(nnq_decoder *d, const nnq_weight *embed, const float *final_norm, const nnq_weight *lm_head) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    if (!d->blocks) return fail(ctx, NNQ_ERR_INVALID_ARG, "not a block decoder: use nnq_decoder_set_head");
    if (!final_norm || !shape_is(embed, c.vocab, d->embed_ld) || embed->fmt != NNQ_BF16_DENSE || !shape_is(lm_head, c.vocab, d->xn_ld))
        return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "embedding (bf16) and vocabulary projection must be [%d, %d]", c.vocab, d->xn_ld);
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(d->d_final_norm, final_norm, (size_t)c.hidden * 4, cudaMemcpyDefault), "final norm");
    if (s != NNQ_OK) return s;
    d->d_embed = embed->d_raw;
    d->lm_head = lm_head;
    d->ready = 1;
    return NNQ_OK;
}

nnq_status nnq_decoder_set_head_options(nnq_decoder *d, const nnq_head_options *o) {
    if (!d || !o) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    if (!d->blocks) return fail(ctx, NNQ_ERR_INVALID_ARG, "not a block decoder");
    if (!(o->logit_cap >= 0.0f)) return fail(ctx, NNQ_ERR_INVALID_ARG, "bad logit cap");
    if (o->pair_table && (o->pair_buckets < 1 || o->pair_buckets >= (1ll << 31) || o->pair_mul_prev < 0 || o->pair_mul_cur < 0 || o->pair_mul_prev >= (1ll << 31) ||
                          o->pair_mul_cur >= (1ll << 31) || !shape_is(o->pair_table, o->pair_buckets + 1, d->embed_ld) || o->pair_table->fmt != NNQ_BF16_DENSE))
        return fail(ctx, NNQ_ERR_SHAPE_MISMATCH, "the pair table must be bf16 [buckets + 1, %d]", d->embed_ld);
    nnq_status s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s == NNQ_OK && o->final_norm_bias) {
        if (!d->final_bias) s = dev_alloc(ctx, (void **)&d->final_bias, (size_t)d->cfg.hidden * 4, "final norm bias");
        if (s == NNQ_OK) s = check_cuda(ctx, cudaMemcpy(d->final_bias, o->final_norm_bias, (size_t)d->cfg.hidden * 4, cudaMemcpyDefault), "final norm bias");
    }
    d->logit_cap = o->logit_cap;
    d->pairs = PairTable{};
    if (o->pair_table) d->pairs = {(const __nv_bfloat16 *)o->pair_table->d_raw, o->pair_mul_prev, o->pair_mul_cur, o->pair_buckets};
    return s;
}

nnq_status nnq_decoder_set_comm(nnq_decoder *d, nnq_comm *comm) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    if (d->cfg.tp_world > 1 && !comm) return fail(d->ctx, NNQ_ERR_INVALID_ARG, "a tensor-parallel decoder needs a communicator");
    d->comm = comm;
    return NNQ_OK;
}

nnq_status nnq_decoder_reset(nnq_decoder *d, int token, int pos, void *stream) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    if (token < 0 || token >= d->cfg.vocab || pos < 0 || pos >= d->cfg.max_seq) return fail(d->ctx, NNQ_ERR_INVALID_ARG, "token or position out of range");
    cudaSetDevice(d->ctx->device);
    const int st[4] = {token, pos, 0, 0};
    nnq_status s = NNQ_OK;
    if (d->blocks && pos != 0) {
        // recurrent state and convolution inputs exist for one position only
        int at = 0;
        if ((s = nnq_decoder_state(d, nullptr, &at, nullptr, stream)) != NNQ_OK) return s;
        if (at != pos) return fail(d->ctx, NNQ_ERR_INVALID_ARG, "the decoder's state is at position %d: it can continue there or restart at 0, not at %d", at, pos);
    }
    d->host_pos = pos;
    s = check_cuda(d->ctx, cudaMemcpyAsync(d->d_state, st, sizeof(st), cudaMemcpyHostToDevice, (cudaStream_t)stream), "decoder state");
    if (s == NNQ_OK) s = check_cuda(d->ctx, cudaStreamSynchronize((cudaStream_t)stream), "decoder state");   // st is on the stack
    return s;
}

nnq_status nnq_decoder_buffers(nnq_decoder *d, float **k_cache, float **v_cache, float **logits, int **tokens) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    if (k_cache) *k_cache = d->d_kcache;
    if (v_cache) *v_cache = d->d_vcache;
    if (logits) *logits = d->d_logits;
    if (tokens) *tokens = d->d_tokens;
    return NNQ_OK;
}

// A product of the decoder: blocks with f32 activations keep f32 operands throughout.
static nnq_status product(nnq_decoder *d, const nnq_weight *w, const void *x, int64_t m, const float *bias, void *y, cudaStream_t st, int y_dt = NNQ_F32) {
    if (!d->blocks || d->act_dt != NNQ_F32) return nnq_linear(d->ctx, w, x, (nnq_dtype)d->act_dt, m, bias, y, (nnq_dtype)y_dt, st);
    LinearArgs a = {w->d_raw, w->d_scales, x, bias, y, m, w->n, w->k, w->fmt, NNQ_F32, y_dt};
    return launch_linear_f32(d->ctx, a, st);
}

// Vocabulary projection of the normed state in d_xn, greedy argmax (exchanged between the ranks
// when the projection is split by rows), commit of the token and advance of the position.
static nnq_status launch_argmax(nnq_decoder *d, bool vocab_parallel, const CommView &cv, cudaStream_t st) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    float *logits = d->d_logits + d->head_row0;
    float *bv = reinterpret_cast<float *>(d->d_state + kStateWords);
    int *bi = d->d_state + kStateWords + kArgmaxBlocks;
    launch_pdl(dec_argmax_stage1_kernel, dim3(kArgmaxBlocks), dim3(256), st, logits, d->head_rows, d->logit_cap, bv, bi);
    if (vocab_parallel)
        launch_pdl(dec_argmax_exchange_kernel, dim3(1), dim3(32), st, bv, bi, kArgmaxBlocks, d->head_row0, cv.peer_table, cv.rank, cv.world,
                   cv.slot_bytes, d->d_state, d->d_tokens, c.max_seq, ctx->d_status);
    else
        launch_pdl(dec_argmax_stage2_kernel, dim3(1), dim3(32), st, bv, bi, kArgmaxBlocks, d->d_state, d->d_tokens, c.max_seq, ctx->d_status);
    ctx->launches += 2;
    return check_cuda(ctx, cudaGetLastError(), "decoder head launch");
}

static nnq_status launch_head(nnq_decoder *d, bool vocab_parallel, const CommView &cv, cudaStream_t st) {
    // the logits of this rank's rows land at their global offsets in the [vocab] buffer
    nnq_status s = product(d, d->lm_head, d->d_xn, 1, nullptr, d->d_logits + d->head_row0, st);
    return s != NNQ_OK ? s : launch_argmax(d, vocab_parallel, cv, st);
}

static nnq_status head_mode(nnq_decoder *d, bool *vocab_parallel, CommView *cv) {
    const nnq_decoder_config &c = d->cfg;
    *vocab_parallel = d->head_rows != c.vocab;
    *cv = CommView{};
    if (*vocab_parallel) {
        nnq_status sv = comm_view(d->comm, cv);
        if (sv != NNQ_OK) return sv;
        if (cv->slot_bytes < (size_t)8 * c.hidden + 16)
            return fail(d->ctx, NNQ_ERR_UNSUPPORTED, "a vocabulary-parallel head needs communicator slots of at least 8 * hidden + 16 bytes (have %zu)", cv->slot_bytes);
    }
    return NNQ_OK;
}

// Measurement aid (builds with -DNNQ_DIAG only): NNQ_DEC_SKIP is a bit mask of step parts that are
// not launched (1 norms, 2 rotation / cache append, 4 attention, 16 SwiGLU, 32 products), to read
// the cost of each part off the time of a replayed step. The results are meaningless with any bit set.
#ifdef NNQ_DIAG
static int dec_skip() {
    static const int v = getenv("NNQ_DEC_SKIP") ? atoi(getenv("NNQ_DEC_SKIP")) : 0;
    return v;
}
#define DEC_RUN(bit, ...) do { if (!(dec_skip() & (bit))) { __VA_ARGS__; } } while (0)
#else
#define DEC_RUN(bit, ...) do { __VA_ARGS__; } while (0)
#endif

static nnq_status ready_to_run(const nnq_decoder *d) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    if (!d->ready) return fail(ctx, NNQ_ERR_INVALID_ARG, "decoder head has not been set");
    if (c.tp_world > 1 && !d->comm) return fail(ctx, NNQ_ERR_INVALID_ARG, "communicator has not been set");
    for (int l = 0; l < c.n_layers; l++)
        if (d->blocks ? !d->blocks[l].in && !d->blocks[l].moe : !d->layers[l].q) return fail(ctx, NNQ_ERR_INVALID_ARG, "layer %d has not been set", l);
    return NNQ_OK;
}

// What the row buffers hold in front of block l (l = n_layers: in front of the head): the last block's sum has not been
// formed yet. h: residual rows, delta: that block's output rows.
static NormRows pending_rows(const nnq_decoder *d, int l, float *h, const float *delta) {
    const nnq_decoder_config &c = d->cfg;
    NormRows r = {};
    r.h = h;
    r.delta = delta;
    r.alpha = 1.0f;
    r.delta_ld = c.hidden;
    if (l == 0) {
        r.embed = (const __nv_bfloat16 *)d->d_embed;
        r.pairs = d->pairs;
    } else if (d->blocks) {
        const nnq_decoder::Block &P = d->blocks[l - 1];
        if (P.moe) r.delta_ld = d->xn_ld;
        if (P.cfg.post_norm) {
            r.alpha = P.cfg.alpha;
            r.post_w = P.norm;
            r.post_b = P.norm_bias;
        }
    }
    if (l == c.n_layers) r.in = {d->final_bias ? kNormLayer : kNormRms, d->d_final_norm, d->final_bias};
    else if (d->blocks && !d->blocks[l].cfg.post_norm) r.in = {kNormRms, d->blocks[l].norm, nullptr};
    r.eps = c.rms_eps;
    r.act_dt = d->act_dt;
    r.hidden = c.hidden;
    r.embed_ld = d->embed_ld;
    r.xn_ld = d->xn_ld;
    return r;
}

static bool fused_steps(const nnq_decoder *d) { return d->act_dt == NNQ_BF16 && d->ctx->path == NNQ_PATH_AUTO; }

// The mixer, the feed-forward activation and the output product of block l for n rows: b_proj -> delta. `state`
// given: a decode step (n = 1, position in state[1]), else rows from position pos0. activated: b_act holds the
// feed-forward activation already.
static nnq_status run_block(nnq_decoder *d, int l, int n, int pos0, const int *state, bool activated, float *delta, cudaStream_t st) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder::Block &B = d->blocks[l];
    const nnq_block_config &k = B.cfg;
    nnq_status s;
    const RowSpan span = {n, pos0, state};
    const FfnPart ffn = {d->b_proj, B.lay.in_cols, B.lay.gate, B.lay.up, k.ffn, d->b_act, d->act_dt, B.lay.out_k, k.heads * k.vdim, B.lay.ffn_col};
    if (k.mixer == NNQ_MIXER_NONE) {
        if (!activated && (s = launch_pair_act(ctx, d->b_proj, B.lay.in_cols, n, k.ffn, k.ffn_act, d->b_act, d->act_dt, B.lay.out_k, st)) != NNQ_OK) return s;
    } else if (k.mixer == NNQ_MIXER_LATENT) {
        LatentAttn a = {};
        a.span = span;
        a.heads = k.heads; a.dim = k.dim; a.rot = k.rot_dims; a.vdim = k.vdim; a.dim_ld = B.lay.dim_ld; a.vdim_ld = B.lay.vdim_ld;
        a.q_rank = k.q_rank; a.q_ld = B.lay.q_ld; a.kv_rank = k.kv_rank; a.kv_ld = B.lay.kv_ld; a.rot_ld = round_up(k.rot_dims, 64);
        a.proj = d->b_proj; a.in_cols = B.lay.in_cols; a.c_q = B.lay.q; a.c_kv = B.lay.k;
        a.eps = d->cfg.rms_eps; a.q_norm = B.q_norm; a.kv_norm = B.kv_norm;
        a.cosv = B.cosv; a.sinv = B.sinv;
        a.act_dt = d->act_dt;
        a.cq = d->b_cq; a.ring_c = B.ring_c; a.ring_r = B.ring_r; a.cap = B.cap;
        a.q = d->b_q2;
        a.scale = k.scale; a.window = k.window > 0 ? k.window : (1 << 30);
        a.out = d->b_act; a.out_ld = B.lay.out_k;
        a.ukv = (const __nv_bfloat16 *)B.ukv->d_raw;
        if (state) {
            a.qlat = d->b_qlat; a.ranges = B.ranges; a.part = d->d_part;
            a.keys_max = k.window > 0 && k.window < d->cfg.max_seq ? k.window : d->cfg.max_seq;
            if (fused_steps(d) && dense_gemv_norm_supported(B.uq, k.q_rank)) {
                // the query latent's norm in the prologue of the product that reads it
                const TcArgs t = {B.uq->d_raw, B.uq->d_scales, nullptr, nullptr, d->b_q2, 1, B.uq->n, B.uq->k, B.uq->fmt, NNQ_BF16, NNQ_F32};
                GemvNorm g = {};
                g.h_in = d->b_proj + B.lay.q;
                g.alpha = 1.0f;
                g.in = {kNormRms, B.q_norm, nullptr};
                g.eps = d->cfg.rms_eps;
                g.hidden = k.q_rank;
                g.half = true;
                s = launch_dense_gemv_norm(ctx, t, g, 0, 0, st);
            } else {
                s = launch_latent_prep(ctx, a, kLatentQueries, st);
                if (s == NNQ_OK) s = product(d, B.uq, d->b_cq, 1, nullptr, d->b_q2, st);
            }
            if (s != NNQ_OK || (s = launch_latent_step(ctx, a, st)) != NNQ_OK) return s;
        } else {
            const size_t es = d->act_dt == NNQ_F32 ? 4 : 2;
            a.first = k.window > 0 && pos0 - k.window + 1 > 0 ? pos0 - k.window + 1 : 0;
            a.keys = pos0 + n - a.first;
            a.linear = a.cap < d->cfg.max_seq;   // a ring that can wrap
            a.lin_c = a.linear ? d->b_lin_c : (char *)a.ring_c + (size_t)a.first * a.kv_ld * es;
            a.lin_r = a.linear ? d->b_lin_r : (char *)a.ring_r + (size_t)a.first * a.rot_ld * es;
            a.kv = d->b_kv;
            a.qrot = d->b_qrot; a.kfull = d->b_kfull; a.vfull = d->b_vfull;
            s = launch_latent_prep(ctx, a, kLatentQueries | kLatentKeys, st);
            if (s == NNQ_OK) s = product(d, B.uq, d->b_cq, n, nullptr, d->b_q2, st);
            if (s == NNQ_OK) s = product(d, B.ukv, a.lin_c, a.keys, nullptr, d->b_kv, st, d->act_dt);
            if (s != NNQ_OK || (s = launch_latent_rows(ctx, a, st)) != NNQ_OK) return s;
        }
    } else if (k.mixer == NNQ_MIXER_ATTENTION) {
        WindowAttn a = {};
        a.span = span;
        a.ffn = ffn;
        a.heads = k.heads; a.kv_heads = k.kv_heads; a.dim = k.dim; a.vdim = k.vdim; a.dim_ld = B.dim_ld; a.vdim_ld = B.vdim_ld;
        a.c_q = B.lay.q; a.c_k = B.lay.k; a.c_v = B.lay.v; a.c_g = B.lay.g;
        a.gated = k.out_gate;
        a.taps = k.conv_taps; a.conv = B.conv; a.conv_ring = B.conv_ring;
        a.rot_dims = k.rot_dims; a.cosv = B.cosv; a.sinv = B.sinv;
        a.mix_mode = B.mix_mode; a.lambda = B.lambda; a.vfirst = d->b_vfirst;
        a.scale = k.scale; a.window = k.window > 0 ? k.window : (1 << 30);
        a.qrot = d->b_q; a.kcache = B.kcache; a.vcache = B.vcache; a.cap = B.cap;
        a.keys_max = k.window > 0 && k.window < d->cfg.max_seq ? k.window : d->cfg.max_seq;
        a.ranges = B.ranges; a.part = d->d_part; a.arrived = d->d_arrived;
        if (state) {
            if ((s = launch_attn_step(ctx, a, st)) != NNQ_OK) return s;
        } else {
            if ((s = launch_attn_prep(ctx, a, st)) != NNQ_OK) return s;
            if ((s = launch_attn_conv_tail(ctx, a, st)) != NNQ_OK) return s;
            if ((s = launch_attn_rows(ctx, a, st)) != NNQ_OK) return s;
        }
    } else {
        Recurrence r = {};
        r.span = span;
        r.ffn = ffn;
        r.heads = k.heads; r.dim = k.dim; r.vdim = k.vdim; r.dim_ld = B.dim_ld;
        r.c_q = B.lay.q; r.c_k = B.lay.k; r.c_v = B.lay.v; r.c_g = B.lay.g; r.c_a1 = B.lay.a1;
        r.q_scale = k.q_scale; r.k_scale = k.k_scale;
        r.rot_dims = k.rot_dims; r.cosv = B.cosv; r.sinv = B.sinv;
        r.rank = k.decay_rank; r.a2t = B.a2t; r.a2b = B.a2b; r.inv_tau = k.decay_rank > 0 ? 1.0f / k.decay_tau : 0.0f; r.decay = B.decay;
        r.head_norm = B.head_norm; r.eps = d->cfg.rms_eps;
        r.state = B.rec_state; r.q = d->b_q; r.k = d->b_k; r.a = d->b_a; r.o = d->b_o;
        if ((s = state ? launch_rec_step(ctx, r, st) : launch_rec_rows(ctx, r, st)) != NNQ_OK) return s;
    }
    return product(d, B.out, d->b_act, n, B.bias_out, delta, st);
}

// The residual update and norm of r for a product kernel that has them in its prologue. The new residual row goes to the
// other of two buffers.
static GemvNorm step_norm(nnq_decoder *d, const NormRows &r) {
    GemvNorm g = {};
    g.h_in = r.h; g.delta = r.delta; g.h_out = d->b_h2; g.alpha = r.alpha;
    g.embed = r.embed; g.pairs = r.pairs; g.embed_ld = r.embed_ld; g.state = d->d_state;
    g.post_w = r.post_w; g.post_b = r.post_b; g.in = r.in; g.eps = r.eps; g.hidden = r.hidden;
    float *t = d->d_h;
    d->d_h = d->b_h2;
    d->b_h2 = t;
    return g;
}

// y = what block l (l = n_layers: the head) reads times w^T for the step's row; where the residual update and the norm
// are part of the product kernel the new residual row goes to the other of two buffers. pair_act: as in
// launch_dense_gemv_norm; *activated tells whether y holds the activation.
static nnq_status step_norm_product(nnq_decoder *d, int l, const nnq_weight *w, const float *bias, float *y, int pair_act, int y_ld, void *act, bool *activated,
                                    cudaStream_t st) {
    const nnq_decoder_config &c = d->cfg;
    NormRows r = pending_rows(d, l, d->d_h, d->d_delta);
    *activated = false;
    if (fused_steps(d) && dense_gemv_norm_supported(w, c.hidden)) {
        const TcArgs a = {w->d_raw, w->d_scales, nullptr, bias, pair_act ? act : y, 1, w->n, w->k, w->fmt, NNQ_BF16, NNQ_F32};
        GemvNorm g = step_norm(d, r);
        g.half = l < c.n_layers && d->blocks[l].cfg.mixer == NNQ_MIXER_LATENT;   // a small product in front of another
        nnq_status s = launch_dense_gemv_norm(d->ctx, a, g, pair_act, y_ld, st);
        *activated = pair_act > 0;
        return s;
    }
    r.xn = d->d_xn;
    const nnq_status s = launch_norm_step(d->ctx, r, d->d_state, st);
    return s == NNQ_OK ? product(d, w, d->d_xn, 1, bias, y, st) : s;
}

static nnq_status step_blocks(nnq_decoder *d, cudaStream_t st) {
    nnq_status s = NNQ_OK;
    for (int l = 0; l < d->cfg.n_layers; l++) {
        const nnq_decoder::Block &B = d->blocks[l];
        if (B.moe) {
            NormRows r = pending_rows(d, l, d->d_h, d->d_delta);
            if (fused_steps(d) && moe_step_supported(B.moe, d->cfg.hidden)) {
                if ((s = moe_step(d->ctx, B.moe, step_norm(d, r), d->d_delta, st)) != NNQ_OK) return s;
                continue;
            }
            r.xn = d->d_xn;
            if ((s = launch_norm_step(d->ctx, r, d->d_state, st)) != NNQ_OK) return s;
            if ((s = moe_rows(d->ctx, B.moe, d->d_xn, (nnq_dtype)d->act_dt, 1, d->act_dt == NNQ_F32, d->d_delta, st)) != NNQ_OK) return s;
            continue;
        }
        bool activated = false;
        const int pair = B.cfg.mixer == NNQ_MIXER_NONE ? 1 + B.cfg.ffn_act : 0;
        if ((s = step_norm_product(d, l, B.in, B.bias_in, d->b_proj, pair, B.lay.out_k, d->b_act, &activated, st)) != NNQ_OK) return s;
        if ((s = run_block(d, l, 1, 0, d->d_state, activated, d->d_delta, st)) != NNQ_OK) return s;
    }
    return NNQ_OK;
}

static nnq_status rows_blocks(nnq_decoder *d, int n, int pos0, cudaStream_t st) {
    const nnq_decoder_config &c = d->cfg;
    for (int l = 0; l < c.n_layers; l++) {
        const nnq_decoder::Block &B = d->blocks[l];
        NormRows r = pending_rows(d, l, d->pf_h, d->pf_delta);
        r.xn = d->pf_xn;
        nnq_status s = launch_norm_rows(d->ctx, r, n, d->pf_tokens + 1, pos0, nullptr, st);
        if (s == NNQ_OK && B.moe) {
            s = moe_rows(d->ctx, B.moe, d->pf_xn, (nnq_dtype)d->act_dt, n, d->act_dt == NNQ_F32, d->pf_delta, st);
        } else {
            // hundreds of rows: the activation in the product's epilogue
            const bool fused = fused_steps(d) && B.cfg.mixer == NNQ_MIXER_NONE && gemm_dense_supported(d->ctx, B.in, n, d->act_dt);
            if (s == NNQ_OK && fused) {
                const TcArgs a = {B.in->d_raw, B.in->d_scales, d->pf_xn, nullptr, nullptr, n, B.in->n, B.in->k, B.in->fmt, NNQ_BF16, NNQ_BF16};
                s = launch_gemm_dense_pairs(d->ctx, a, (__nv_bfloat16 *)d->b_act, B.cfg.ffn_act, st);
            } else if (s == NNQ_OK) {
                s = product(d, B.in, d->pf_xn, n, B.bias_in, d->b_proj, st);
            }
            if (s == NNQ_OK) s = run_block(d, l, n, pos0, nullptr, fused, d->pf_delta, st);
        }
        if (s != NNQ_OK) return s;
    }
    return NNQ_OK;
}

static nnq_status step_qwen3(nnq_decoder *d, cudaStream_t st) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = NNQ_OK;
    const int hd = c.head_dim, group = c.n_heads / c.n_kv_heads, lh = d->lh, lkv = d->lkv, lffn = c.ffn / c.tp_world;
    const nnq_dtype adt = (nnq_dtype)d->act_dt;
    const size_t layer_cache = (size_t)lkv * c.max_seq * hd;
    const float scale = (float)(1.0 / sqrt((double)hd));
    const __nv_bfloat16 *embed = (const __nv_bfloat16 *)d->d_embed;
    for (int l = 0; l < c.n_layers; l++) {
        const nnq_decoder::Layer &L = d->layers[l];
        DEC_RUN(1, launch_pdl(dec_norm_kernel, dim3(1), dim3(1024), st, d->d_h, d->d_delta, l == 0 ? embed : nullptr, d->d_state, L.in_norm, c.rms_eps, d->d_xn, d->act_dt, c.hidden));
        const nnq_weight *w3[3] = {L.q, L.k, L.v};
        const void *x3[3] = {d->d_xn, d->d_xn, d->d_xn};
        void *y3[3] = {d->d_q, d->d_k, d->d_v};
        DEC_RUN(32, if ((s = nnq_linear_batch(ctx, 3, w3, x3, adt, 1, nullptr, y3, NNQ_F32, st)) != NNQ_OK) return s);
        DEC_RUN(2, launch_pdl(dec_qk_rope_kernel, dim3(lh + 2 * lkv), dim3(hd), st, d->d_q, d->d_k, d->d_v, L.q_norm, L.k_norm, d->d_cos, d->d_sin, d->d_state,
                              c.rms_eps, d->d_qrot, d->d_kcache + l * layer_cache, d->d_vcache + l * layer_cache, lh, lkv, hd, c.max_seq));
        DEC_RUN(4, {
            const dim3 ag(lkv, kAttnRanges), ab(kAttnWarps * 32);
            const float *kc = d->d_kcache + l * layer_cache, *vc = d->d_vcache + l * layer_cache;
            switch (group) {
                case 1: launch_pdl(dec_attn_kernel<1>, ag, ab, st, d->d_qrot, kc, vc, d->d_state, scale, d->d_part, d->d_arrived, d->d_attn, d->act_dt, hd, c.max_seq); break;
                case 2: launch_pdl(dec_attn_kernel<2>, ag, ab, st, d->d_qrot, kc, vc, d->d_state, scale, d->d_part, d->d_arrived, d->d_attn, d->act_dt, hd, c.max_seq); break;
                case 4: launch_pdl(dec_attn_kernel<4>, ag, ab, st, d->d_qrot, kc, vc, d->d_state, scale, d->d_part, d->d_arrived, d->d_attn, d->act_dt, hd, c.max_seq); break;
                case 8: launch_pdl(dec_attn_kernel<8>, ag, ab, st, d->d_qrot, kc, vc, d->d_state, scale, d->d_part, d->d_arrived, d->d_attn, d->act_dt, hd, c.max_seq); break;
                default: return fail(ctx, NNQ_ERR_UNSUPPORTED, "query heads per key/value head must be 1, 2, 4 or 8");
            }
        });
        // row-parallel products: with tensor parallelism the partial sums are exchanged inside the kernel
        DEC_RUN(32, s = d->comm ? nnq_comm_linear(d->comm, L.o, d->d_attn, adt, 1, nullptr, d->d_delta, NNQ_F32, st)
                                : nnq_linear(ctx, L.o, d->d_attn, adt, 1, nullptr, d->d_delta, NNQ_F32, st));
        if (s != NNQ_OK) return s;
        DEC_RUN(1, launch_pdl(dec_norm_kernel, dim3(1), dim3(1024), st, d->d_h, d->d_delta, nullptr, d->d_state, L.post_norm, c.rms_eps, d->d_xn, d->act_dt, c.hidden));
        const nnq_weight *w2[2] = {L.gate, L.up};
        const void *x2[2] = {d->d_xn, d->d_xn};
        void *y2[2] = {d->d_g, d->d_u};
        DEC_RUN(32, if ((s = nnq_linear_batch(ctx, 2, w2, x2, adt, 1, nullptr, y2, NNQ_F32, st)) != NNQ_OK) return s);
        DEC_RUN(16, launch_pdl(dec_silu_mul_kernel, dim3((lffn + 255) / 256), dim3(256), st, d->d_g, d->d_u, d->d_mid, d->act_dt, lffn));
        DEC_RUN(32, s = d->comm ? nnq_comm_linear(d->comm, L.down, d->d_mid, adt, 1, nullptr, d->d_delta, NNQ_F32, st)
                                : nnq_linear(ctx, L.down, d->d_mid, adt, 1, nullptr, d->d_delta, NNQ_F32, st));
        if (s != NNQ_OK) return s;
        ctx->launches += 5;
    }
    return NNQ_OK;
}

static nnq_status rows_qwen3(nnq_decoder *d, int n, int pos0, cudaStream_t st) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = NNQ_OK;
    const int hd = c.head_dim, group = c.n_heads / c.n_kv_heads, lh = d->lh, lkv = d->lkv, lffn = c.ffn / c.tp_world;
    const nnq_dtype adt = (nnq_dtype)d->act_dt;
    const size_t layer_cache = (size_t)lkv * c.max_seq * hd;
    const float scale = (float)(1.0 / sqrt((double)hd));
    const __nv_bfloat16 *embed = (const __nv_bfloat16 *)d->d_embed;
    for (int l = 0; l < c.n_layers; l++) {
        const nnq_decoder::Layer &L = d->layers[l];
        float *kc = d->d_kcache + l * layer_cache, *vc = d->d_vcache + l * layer_cache;
        dec_norm_rows_kernel<<<n, 256, 0, st>>>(d->pf_h, l == 0 ? nullptr : d->pf_delta, l == 0 ? embed : nullptr, d->pf_tokens + 1, L.in_norm, c.rms_eps, d->pf_xn, d->act_dt, c.hidden);
        const nnq_weight *w3[3] = {L.q, L.k, L.v};
        const void *x3[3] = {d->pf_xn, d->pf_xn, d->pf_xn};
        void *y3[3] = {d->pf_q, d->pf_k, d->pf_v};
        if ((s = nnq_linear_batch(ctx, 3, w3, x3, adt, n, nullptr, y3, NNQ_F32, st)) != NNQ_OK) return s;
        dec_qk_rope_rows_kernel<<<dim3(lh + 2 * lkv, n), hd, 0, st>>>(d->pf_q, d->pf_k, d->pf_v, L.q_norm, L.k_norm, d->d_cos, d->d_sin, pos0,
                                                                     c.rms_eps, d->pf_qrot, kc, vc, lh, lkv, hd, c.max_seq);
        // 16 query vectors per warp: R = 16 / G rows share each key / value row
        switch (group) {
            case 1: dec_attn_rows_kernel<1, 16><<<dim3(lkv, (n + 15) / 16), 32, 0, st>>>(d->pf_qrot, kc, vc, pos0, n, scale, d->pf_attn, d->act_dt, lh, hd, c.max_seq); break;
            case 2: dec_attn_rows_kernel<2, 8><<<dim3(lkv, (n + 7) / 8), 32, 0, st>>>(d->pf_qrot, kc, vc, pos0, n, scale, d->pf_attn, d->act_dt, lh, hd, c.max_seq); break;
            case 4: dec_attn_rows_kernel<4, 4><<<dim3(lkv, (n + 3) / 4), 32, 0, st>>>(d->pf_qrot, kc, vc, pos0, n, scale, d->pf_attn, d->act_dt, lh, hd, c.max_seq); break;
            case 8: dec_attn_rows_kernel<8, 2><<<dim3(lkv, (n + 1) / 2), 32, 0, st>>>(d->pf_qrot, kc, vc, pos0, n, scale, d->pf_attn, d->act_dt, lh, hd, c.max_seq); break;
            default: return fail(ctx, NNQ_ERR_UNSUPPORTED, "query heads per key/value head must be 1, 2, 4 or 8");
        }
        s = d->comm ? nnq_comm_linear(d->comm, L.o, d->pf_attn, adt, n, nullptr, d->pf_delta, NNQ_F32, st)
                    : nnq_linear(ctx, L.o, d->pf_attn, adt, n, nullptr, d->pf_delta, NNQ_F32, st);
        if (s != NNQ_OK) return s;
        dec_norm_rows_kernel<<<n, 256, 0, st>>>(d->pf_h, d->pf_delta, nullptr, d->pf_tokens, L.post_norm, c.rms_eps, d->pf_xn, d->act_dt, c.hidden);
        const nnq_weight *w2[2] = {L.gate, L.up};
        const void *x2[2] = {d->pf_xn, d->pf_xn};
        void *y2[2] = {d->pf_g, d->pf_u};
        if ((s = nnq_linear_batch(ctx, 2, w2, x2, adt, n, nullptr, y2, NNQ_F32, st)) != NNQ_OK) return s;
        const int total = n * lffn;
        dec_silu_mul_kernel<<<(total + 255) / 256, 256, 0, st>>>(d->pf_g, d->pf_u, d->pf_mid, d->act_dt, total);
        s = d->comm ? nnq_comm_linear(d->comm, L.down, d->pf_mid, adt, n, nullptr, d->pf_delta, NNQ_F32, st)
                    : nnq_linear(ctx, L.down, d->pf_mid, adt, n, nullptr, d->pf_delta, NNQ_F32, st);
        if (s != NNQ_OK) return s;
        ctx->launches += 5;
    }
    return NNQ_OK;
}

nnq_status nnq_decoder_step(nnq_decoder *d, void *stream) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = ready_to_run(d);
    if (s != NNQ_OK) return s;
    // The caches hold max_seq positions and never grow (the reference's KvCacheLayer::append doubles
    // its buffer instead): a step past the last position is refused here, and -- for captured graphs
    // that the host does not see being replayed -- by the device-side flag behind nnq_device_status.
    if (d->host_pos >= c.max_seq)
        return fail(ctx, NNQ_ERR_UNSUPPORTED, "the decoder's context is full (max_seq = %d positions): reset it", c.max_seq);
    if (d->host_pos >= 0) d->host_pos++;
    bool vocab_parallel = false;
    CommView cv = {};
    if ((s = head_mode(d, &vocab_parallel, &cv)) != NNQ_OK) return s;
    s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice");
    if (s != NNQ_OK) return s;
    cudaStream_t st = (cudaStream_t)stream;
    if (d->blocks) {
        if ((s = step_blocks(d, st)) != NNQ_OK) return s;
        bool activated = false;
        if ((s = step_norm_product(d, c.n_layers, d->lm_head, nullptr, d->d_logits, 0, 0, nullptr, &activated, st)) != NNQ_OK) return s;
        return launch_argmax(d, vocab_parallel, cv, st);
    }
    if ((s = step_qwen3(d, st)) != NNQ_OK) return s;
    launch_pdl(dec_norm_kernel, dim3(1), dim3(1024), st, d->d_h, d->d_delta, nullptr, d->d_state, d->d_final_norm, c.rms_eps, d->d_xn, d->act_dt, c.hidden);
    ctx->launches++;
    return launch_head(d, vocab_parallel, cv, st);
}

// Checks of a call that feeds `count` given tokens from position start_pos on.
static nnq_status check_tokens(nnq_decoder *d, const int32_t *tokens_host, int count, int start_pos) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = ready_to_run(d);
    if (s != NNQ_OK) return s;
    if (!tokens_host || count < 1 || start_pos < 0) return fail(ctx, NNQ_ERR_INVALID_ARG, "bad prompt arguments");
    if ((long long)start_pos + count > c.max_seq)
        return fail(ctx, NNQ_ERR_UNSUPPORTED, "a prompt of %d tokens at position %d does not fit max_seq = %d", count, start_pos, c.max_seq);
    for (int i = 0; i < count; i++)
        if (tokens_host[i] < 0 || tokens_host[i] >= c.vocab) return fail(ctx, NNQ_ERR_INVALID_ARG, "prompt token %d out of range", i);
    if (d->blocks && start_pos != 0 && start_pos != d->host_pos)
        return fail(ctx, NNQ_ERR_INVALID_ARG, "the decoder's state is at position %lld: it can continue there or restart at 0, not at %d", d->host_pos, start_pos);
    return NNQ_OK;
}

// Rows that go through the layers together: bounded by the row buffers (allocated here for Qwen3 layers)
// and, with tensor parallelism, by what one exchange carries.
static nnq_status row_buffers(nnq_decoder *d, int *rows_max) {
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = NNQ_OK;
    *rows_max = d->blocks ? d->pf_rows : kPrefillRows;
    if (d->comm) {
        CommView v;
        if ((s = comm_view(d->comm, &v)) != NNQ_OK) return s;
        const size_t fit = v.slot_bytes / ((size_t)c.hidden * 4);
        if (fit < 1) return fail(ctx, NNQ_ERR_UNSUPPORTED, "communicator slots are smaller than one row of the hidden state");
        if ((size_t)*rows_max > fit) *rows_max = (int)fit;
    }
    const int qdim = d->lh * c.head_dim, kvdim = d->lkv * c.head_dim, lffn = d->blocks ? 0 : c.ffn / c.tp_world;
    const size_t es = d->act_dt == NNQ_F32 ? 4 : 2;
    if (!d->pf_h) {
        d->pf_rows = kPrefillRows;
        const size_t R = kPrefillRows;
        s = dev_alloc(ctx, (void **)&d->pf_h, R * c.hidden * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_delta, R * c.hidden * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_q, R * qdim * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_k, R * kvdim * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_v, R * kvdim * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_qrot, R * qdim * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_g, R * lffn * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_u, R * lffn * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, &d->pf_xn, R * c.hidden * es, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, &d->pf_attn, R * qdim * es, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, &d->pf_mid, R * lffn * es, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_tokens, (R + 1) * 4, "prompt buffer");
        if (s == NNQ_OK) s = dev_alloc(ctx, (void **)&d->pf_want, R * 4, "prompt buffer");
        if (s != NNQ_OK) return s;
    }
    return NNQ_OK;
}

// n <= rows_max tokens through the layers: afterwards pf_h + pf_delta are the rows' final residuals.
static nnq_status run_rows(nnq_decoder *d, const int32_t *tokens_host, int n, int pos0, cudaStream_t st) {
    nnq_status s = check_cuda(d->ctx, cudaMemcpyAsync(d->pf_tokens + 1, tokens_host, (size_t)n * 4, cudaMemcpyHostToDevice, st), "prompt tokens");
    if (s != NNQ_OK) return s;
    if (d->blocks) {   // the token in front of the block, and what a later block or step finds as its previous token
        s = check_cuda(d->ctx, cudaMemcpyAsync(d->pf_tokens, d->d_state + 4, 4, cudaMemcpyDeviceToDevice, st), "prompt tokens");
        if (s == NNQ_OK) s = check_cuda(d->ctx, cudaMemcpyAsync(d->d_state + 4, d->pf_tokens + n, 4, cudaMemcpyDeviceToDevice, st), "prompt tokens");
        if (s != NNQ_OK) return s;
    }
    return d->blocks ? rows_blocks(d, n, pos0, st) : rows_qwen3(d, n, pos0, st);
}

nnq_status nnq_decoder_prefill(nnq_decoder *d, const int32_t *tokens_host, int count, int start_pos, void *stream) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = check_tokens(d, tokens_host, count, start_pos);
    if (s != NNQ_OK) return s;
    bool vocab_parallel = false;
    CommView cv = {};
    if ((s = head_mode(d, &vocab_parallel, &cv)) != NNQ_OK) return s;
    if ((s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice")) != NNQ_OK) return s;
    cudaStream_t st = (cudaStream_t)stream;
    int rows_max = 0;
    if ((s = row_buffers(d, &rows_max)) != NNQ_OK) return s;
    d->host_pos = -1;   // until the call has gone through
    int n = 0;
    for (int c0 = 0; c0 < count; c0 += n) {
        n = count - c0 < rows_max ? count - c0 : rows_max;
        if ((s = run_rows(d, tokens_host + c0, n, start_pos + c0, st)) != NNQ_OK) return s;
    }
    // the last prompt token's state: final norm, vocabulary projection, greedy successor
    const int st4[4] = {tokens_host[count - 1], start_pos + count - 1, 0, 0};
    if ((s = check_cuda(ctx, cudaMemcpyAsync(d->d_state, st4, sizeof(st4), cudaMemcpyHostToDevice, st), "decoder state")) != NNQ_OK) return s;
    NormRows r = pending_rows(d, c.n_layers, d->pf_h + (size_t)(n - 1) * c.hidden, d->pf_delta);
    r.delta += (size_t)(n - 1) * r.delta_ld;
    r.xn = d->d_xn;
    s = launch_norm_step(ctx, r, d->d_state, st);
    if (s != NNQ_OK || (s = launch_head(d, vocab_parallel, cv, st)) != NNQ_OK) return s;
    s = check_cuda(ctx, cudaStreamSynchronize(st), "prompt pass");   // tokens_host and st4 are the caller's / the stack's
    if (s == NNQ_OK) d->host_pos = (long long)start_pos + count;
    return s;
}

nnq_status nnq_decoder_extend(nnq_decoder *d, const int32_t *tokens_host, int count, int start_pos, const int32_t *want, int n_want,
                              float *logits_host, void *stream) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    nnq_ctx *ctx = d->ctx;
    const nnq_decoder_config &c = d->cfg;
    nnq_status s = check_tokens(d, tokens_host, count, start_pos);
    if (s != NNQ_OK) return s;
    if (n_want < 0 || (n_want && (!want || !logits_host))) return fail(ctx, NNQ_ERR_INVALID_ARG, "bad list of wanted positions");
    for (int i = 0; i < n_want; i++)
        if (want[i] < 0 || want[i] >= count || (i && want[i] <= want[i - 1])) return fail(ctx, NNQ_ERR_INVALID_ARG, "wanted positions must be ascending and inside the tokens");
    if (d->head_rows != c.vocab) return fail(ctx, NNQ_ERR_UNSUPPORTED, "wanted logits need the whole vocabulary projection on this rank");
    if ((s = check_cuda(ctx, cudaSetDevice(ctx->device), "cudaSetDevice")) != NNQ_OK) return s;
    cudaStream_t st = (cudaStream_t)stream;
    if (count == 1) {
        if ((s = nnq_decoder_reset(d, tokens_host[0], start_pos, stream)) != NNQ_OK) return s;
        if ((s = nnq_decoder_step(d, stream)) != NNQ_OK) return s;
        if (n_want) s = check_cuda(ctx, cudaMemcpyAsync(logits_host, d->d_logits, (size_t)c.vocab * 4, cudaMemcpyDeviceToHost, st), "logits");
        if (s == NNQ_OK) s = check_cuda(ctx, cudaStreamSynchronize(st), "decoder step");
        return s;
    }
    int rows_max = 0;
    if ((s = row_buffers(d, &rows_max)) != NNQ_OK) return s;
    if (n_want && !d->d_want_logits && (s = dev_alloc(ctx, (void **)&d->d_want_logits, (size_t)kWantRows * c.vocab * 4, "logits of wanted rows")) != NNQ_OK) return s;
    d->host_pos = -1;   // until the call has gone through
    int n = 0, w0 = 0;
    for (int c0 = 0; c0 < count; c0 += n) {
        n = count - c0 < rows_max ? count - c0 : rows_max;
        if ((s = run_rows(d, tokens_host + c0, n, start_pos + c0, st)) != NNQ_OK) return s;
        while (w0 < n_want && want[w0] < c0 + n) {
            int32_t rows[kWantRows];
            int m = 0;
            while (m < kWantRows && w0 + m < n_want && want[w0 + m] < c0 + n) {
                rows[m] = want[w0 + m] - c0;
                m++;
            }
            if ((s = check_cuda(ctx, cudaMemcpyAsync(d->pf_want, rows, (size_t)m * 4, cudaMemcpyHostToDevice, st), "wanted rows")) != NNQ_OK) return s;
            NormRows r = pending_rows(d, c.n_layers, d->pf_h, d->pf_delta);
            r.xn = d->pf_xn;
            s = launch_norm_rows(ctx, r, m, nullptr, 0, d->pf_want, st);
            if (s == NNQ_OK) s = product(d, d->lm_head, d->pf_xn, m, nullptr, d->d_want_logits, st);
            if (s == NNQ_OK && d->logit_cap > 0.0f) s = launch_logit_cap(ctx, d->d_want_logits, d->logit_cap, (long long)m * c.vocab, st);
            if (s != NNQ_OK) return s;
            s = check_cuda(ctx, cudaMemcpyAsync(logits_host + (size_t)w0 * c.vocab, d->d_want_logits, (size_t)m * c.vocab * 4, cudaMemcpyDeviceToHost, st), "logits");
            if (s == NNQ_OK) s = check_cuda(ctx, cudaStreamSynchronize(st), "logits");   // rows[] is on the stack
            if (s != NNQ_OK) return s;
            w0 += m;
        }
    }
    const bool full = start_pos + count >= c.max_seq;
    const int st4[4] = {tokens_host[count - 1], full ? c.max_seq - 1 : start_pos + count, 0, full ? 1 : 0};
    s = check_cuda(ctx, cudaMemcpyAsync(d->d_state, st4, sizeof(st4), cudaMemcpyHostToDevice, st), "decoder state");
    if (s == NNQ_OK) s = check_cuda(ctx, cudaStreamSynchronize(st), "prompt pass");
    if (s == NNQ_OK) d->host_pos = (long long)start_pos + count;
    return s;
}

nnq_status nnq_decoder_state(nnq_decoder *d, int *token, int *pos, int *steps, void *stream) {
    if (!d) return NNQ_ERR_INVALID_ARG;
    cudaSetDevice(d->ctx->device);
    int st[4] = {0, 0, 0, 0};
    nnq_status s = check_cuda(d->ctx, cudaMemcpyAsync(st, d->d_state, sizeof(st), cudaMemcpyDeviceToHost, (cudaStream_t)stream), "decoder state");
    if (s == NNQ_OK) s = check_cuda(d->ctx, cudaStreamSynchronize((cudaStream_t)stream), "decoder state");
    if (s == NNQ_OK && (d->host_pos >= 0 || st[2] > 0)) d->host_pos = st[3] ? d->cfg.max_seq : st[1];   // replayed graphs advance it unseen
    if (token) *token = st[0];
    if (pos) *pos = st[1];
    if (steps) *steps = st[2];
    return s;
}

void nnq_decoder_destroy(nnq_decoder *d) {
    if (!d) return;
    cudaSetDevice(d->ctx->device);
    cudaDeviceSynchronize();
    if (d->layers) {
        for (int l = 0; l < d->cfg.n_layers; l++) {
            cudaFree(d->layers[l].in_norm); cudaFree(d->layers[l].post_norm);
            cudaFree(d->layers[l].q_norm); cudaFree(d->layers[l].k_norm);
        }
        delete[] d->layers;
    }
    if (d->blocks) {
        for (int l = 0; l < d->cfg.n_layers; l++) {
            nnq_decoder::Block &B = d->blocks[l];
            cudaFree(B.norm); cudaFree(B.bias_in); cudaFree(B.bias_out); cudaFree(B.conv); cudaFree(B.head_norm);
            cudaFree(B.a2t); cudaFree(B.a2b); cudaFree(B.decay); cudaFree(B.kcache); cudaFree(B.vcache);
            cudaFree(B.conv_ring); cudaFree(B.rec_state); cudaFree(B.norm_bias); cudaFree(B.q_norm); cudaFree(B.kv_norm);
            if (B.cfg.mixer == NNQ_MIXER_LATENT && B.cfg.kv_from < 0) {
                cudaFree(B.ring_c); cudaFree(B.ring_r);
            }
            if (B.owns_tables) {
                cudaFree(B.cosv); cudaFree(B.sinv);
            }
        }
        delete[] d->blocks;
    }
    cudaFree(d->b_h2); cudaFree(d->b_proj); cudaFree(d->b_q); cudaFree(d->b_k); cudaFree(d->b_a); cudaFree(d->b_o); cudaFree(d->b_vfirst); cudaFree(d->b_act);
    cudaFree(d->b_cq); cudaFree(d->b_lin_c); cudaFree(d->b_lin_r); cudaFree(d->b_kv); cudaFree(d->b_q2); cudaFree(d->b_qrot);
    cudaFree(d->b_kfull); cudaFree(d->b_vfull); cudaFree(d->b_qlat); cudaFree(d->final_bias);
    cudaFree(d->pf_want); cudaFree(d->d_want_logits);
    cudaFree(d->d_final_norm); cudaFree(d->d_cos); cudaFree(d->d_sin); cudaFree(d->d_kcache); cudaFree(d->d_vcache);
    cudaFree(d->d_h); cudaFree(d->d_delta); cudaFree(d->d_q); cudaFree(d->d_k); cudaFree(d->d_v); cudaFree(d->d_qrot);
    cudaFree(d->d_g); cudaFree(d->d_u); cudaFree(d->d_logits); cudaFree(d->d_part); cudaFree(d->d_arrived); cudaFree(d->d_xn); cudaFree(d->d_attn);
    cudaFree(d->d_mid); cudaFree(d->d_state); cudaFree(d->d_tokens);
    cudaFree(d->pf_h); cudaFree(d->pf_delta); cudaFree(d->pf_q); cudaFree(d->pf_k); cudaFree(d->pf_v); cudaFree(d->pf_qrot);
    cudaFree(d->pf_g); cudaFree(d->pf_u); cudaFree(d->pf_xn); cudaFree(d->pf_attn); cudaFree(d->pf_mid); cudaFree(d->pf_tokens);
    cudaGetLastError();
    delete d;
}

}  // extern "C"
