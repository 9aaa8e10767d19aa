// Sliding-window grouped-query attention of a block decoder: short causal convolutions on the projected
// q / k / v, half-split rotation, value mixing with an earlier layer, append to a ring of keys and values,
// softmax attention over the window, sigmoid output gate. Any head sizes (value dimension up to 256) and
// any number of query heads per key / value head. Scores, softmax and sums are f32.
#include <math.h>

#include "blocks.cuh"

namespace nnq {

constexpr int kPrepWarps = 4, kPrepRows = 8;

// Projected value (before the convolution) of channel c, column col of proj, `back` rows before row r at
// position pos: rows of this launch come from proj, earlier ones from the ring, positions before 0 are zero.
__device__ __forceinline__ float conv_input(const WindowAttn &a, int channels, int r, int pos, int back, int c, int col) {
    if (r >= back) return a.ffn.proj[(size_t)(r - back) * a.ffn.in_cols + col];
    return pos >= back ? a.conv_ring[(size_t)((pos - back) % a.taps) * channels + c] : 0.0f;
}

// One warp per (head, kPrepRows consecutive rows), heads numbered q | k | v; a lane slides over the rows of its
// channels, so that a projected value is read once. TAPS 0: no convolution; -1: any other number of taps.
// CTAs from prep_ctas on do the feed-forward part.
template <int TAPS>
__global__ void __launch_bounds__(kPrepWarps * 32) attn_prep_kernel(const WindowAttn a, int prep_ctas) {
    pdl_prologue();
    pdl_release();
    extern __shared__ float prep_smem[];
    if ((int)blockIdx.x >= prep_ctas) {
        ffn_part(a.ffn, a.span.n, prep_ctas);
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nh = a.heads + 2 * a.kv_heads, n = a.span.n;
    const int item = blockIdx.x * kPrepWarps + warp;
    const int tile = item / nh, head = item - tile * nh, row0 = tile * kPrepRows;
    if (row0 >= n) return;
    const int rows = min(kPrepRows, n - row0), pos0 = span_pos(a.span) + row0;
    const bool is_q = head < a.heads, is_v = head >= a.heads + a.kv_heads;
    const int h = is_q ? head : (is_v ? head - a.heads - a.kv_heads : head - a.heads);
    const int width = is_v ? a.vdim : a.dim, wmax = max(a.dim, a.vdim);
    const int channels = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
    const int c0 = is_q ? h * a.dim : (is_v ? (a.heads + a.kv_heads) * a.dim + h * a.vdim : (a.heads + h) * a.dim);
    const int col0 = (is_q ? a.c_q : (is_v ? a.c_v : a.c_k)) + h * width;
    float *xs = prep_smem + warp * kPrepRows * wmax;   // [rows, wmax]
    for (int d = lane; d < width; d += 32) {
        float cur[kPrepRows];
#pragma unroll
        for (int r = 0; r < kPrepRows; r++) cur[r] = r < rows ? a.ffn.proj[(size_t)(row0 + r) * a.ffn.in_cols + col0 + d] : 0.0f;
        // one row: this position's slot is read by nobody in this launch (readers look 1 .. taps - 1 back)
        if (TAPS != 0 && n == 1 && a.taps > 1) a.conv_ring[(size_t)(pos0 % a.taps) * channels + c0 + d] = cur[0];
        if constexpr (TAPS > 0) {
            float w[TAPS], u[TAPS];   // u[b]: value b rows back
#pragma unroll
            for (int t = 0; t < TAPS; t++) w[t] = a.conv[(size_t)(c0 + d) * TAPS + t];
#pragma unroll
            for (int b = 1; b < TAPS; b++) u[b] = conv_input(a, channels, row0, pos0, b, c0 + d, col0 + d);
#pragma unroll
            for (int r = 0; r < kPrepRows; r++) {
                u[0] = cur[r];
                float y = 0.0f;
#pragma unroll
                for (int t = 0; t < TAPS; t++) y = fmaf(w[t], u[TAPS - 1 - t], y);
                if (r < rows) xs[r * wmax + d] = y;
#pragma unroll
                for (int b = TAPS - 1; b > 0; b--) u[b] = u[b - 1];
            }
        } else if constexpr (TAPS == 0) {
#pragma unroll
            for (int r = 0; r < kPrepRows; r++)
                if (r < rows) xs[r * wmax + d] = cur[r];
        } else {
            for (int r = 0; r < rows; r++) {
                float y = 0.0f;
                for (int t = 0; t < a.taps; t++)
                    y = fmaf(a.conv[(size_t)(c0 + d) * a.taps + t], conv_input(a, channels, row0 + r, pos0 + r, a.taps - 1 - t, c0 + d, col0 + d), y);
                xs[r * wmax + d] = y;
            }
        }
    }
    __syncwarp();
    const int half = a.rot_dims >> 1;
    for (int r = 0; r < rows; r++) {
        const int pos = pos0 + r, row = row0 + r;
        const float *x = xs + r * wmax;
        if (is_v) {
            const size_t vf = ((size_t)row * a.kv_heads + h) * a.vdim;
            float *dst = a.vcache + ((size_t)h * a.cap + pos % a.cap) * a.vdim_ld;
            for (int d = lane; d < width; d += 32) {
                float v = x[d];
                if (a.mix_mode == 1) a.vfirst[vf + d] = v;
                else if (a.mix_mode == 2) v = (1.0f - a.lambda) * v + a.lambda * a.vfirst[vf + d];
                dst[d] = v;
            }
        } else {
            const float *cs = a.cosv + (size_t)pos * half, *sn = a.sinv + (size_t)pos * half;
            float *dst = is_q ? a.qrot + ((size_t)row * a.heads + h) * a.dim_ld : a.kcache + ((size_t)h * a.cap + pos % a.cap) * a.dim_ld;
            for (int d = lane; d < a.dim_ld; d += 32) dst[d] = d < width ? rotated(x, d, a.rot_dims, cs, sn) : 0.0f;
        }
    }
}

// the last min(n, taps - 1) projected rows of a block of rows enter the ring
__global__ void __launch_bounds__(256) attn_conv_tail_kernel(const WindowAttn a) {
    const int channels = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
    const int rows = min(a.span.n, a.taps - 1);
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= rows * channels) return;
    const int back = i / channels, c = i - back * channels;
    const int row = a.span.n - 1 - back, pos = a.span.pos0 + row;
    const int qn = a.heads * a.dim, kn = a.kv_heads * a.dim;
    const int col = c < qn ? a.c_q + c : (c < qn + kn ? a.c_k + c - qn : a.c_v + c - qn - kn);
    a.conv_ring[(size_t)(pos % a.taps) * channels + c] = a.ffn.proj[(size_t)row * a.ffn.in_cols + col];
}

// ---- softmax attention over the window: a warp, P query vectors, batches of 32 keys ----
//
// Lane j forms the dot products of key j of the batch with the P query vectors (in shared memory), the
// batch joins each vector's running softmax, then the value rows are read coalesced (lane l owns value
// dimensions 4l .. 4l+3, and 128 + 4l .. for VC = 2) and weighted with the probabilities passed by
// shuffle. lo[p] .. hi[p] is what query vector p sees.
template <int P, int VC>
struct WarpSoftmax {
    float m[P], l[P];
    float4 acc[P][VC];

    __device__ __forceinline__ void init() {
#pragma unroll
        for (int p = 0; p < P; p++) {
            m[p] = -INFINITY;
            l[p] = 0.0f;
#pragma unroll
            for (int c = 0; c < VC; c++) acc[p][c] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    }

    // keys b0 .. min(b0 + 31, last); kb / vb: rows of this kv head
    template <typename Visible>
    __device__ __forceinline__ void batch(const WindowAttn &a, const float *qs, const float *kb, const float *vb, int b0, int last, Visible vis) {
        const int lane = threadIdx.x & 31;
        const int nk = min(32, last - b0 + 1);
        const int s0 = b0 % a.cap;
        int slot = s0 + (lane < nk ? lane : 0);
        if (slot >= a.cap) slot -= a.cap;
        const float4 *krow = reinterpret_cast<const float4 *>(kb + (size_t)slot * a.dim_ld);
        const float4 *q4 = reinterpret_cast<const float4 *>(qs);
        const int n4 = a.dim_ld >> 2;
        float dot[P];
#pragma unroll
        for (int p = 0; p < P; p++) dot[p] = 0.0f;
#pragma unroll 8
        for (int d4 = 0; d4 < n4; d4++) {
            const float4 kv = krow[d4];
#pragma unroll
            for (int p = 0; p < P; p++) {
                const float4 qv = q4[p * n4 + d4];
                dot[p] = fmaf(qv.x, kv.x, fmaf(qv.y, kv.y, fmaf(qv.z, kv.z, fmaf(qv.w, kv.w, dot[p]))));
            }
        }
#pragma unroll
        for (int p = 0; p < P; p++) {
            const bool ok = lane < nk && vis(p, b0 + lane);
            const float s = ok ? dot[p] * a.scale : -INFINITY;
            const float mn = fmaxf(m[p], warp_max(s));
            const float corr = m[p] == mn ? 1.0f : expf(m[p] - mn);   // no key of this vector yet: both -inf
            dot[p] = ok ? expf(s - mn) : 0.0f;                        // the weight, in place of the score
            l[p] = l[p] * corr + warp_sum(dot[p]);
#pragma unroll
            for (int c = 0; c < VC; c++) {
                acc[p][c].x *= corr; acc[p][c].y *= corr; acc[p][c].z *= corr; acc[p][c].w *= corr;
            }
            m[p] = mn;
        }
        int s = s0;
#pragma unroll 4
        for (int jj = 0; jj < nk; jj++) {
            const float *vrow = vb + (size_t)s * a.vdim_ld;
            if (++s == a.cap) s = 0;
            float4 vv[VC];
#pragma unroll
            for (int c = 0; c < VC; c++)
                vv[c] = 4 * lane + 128 * c < a.vdim_ld ? *reinterpret_cast<const float4 *>(vrow + 4 * lane + 128 * c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int p = 0; p < P; p++) {
                const float w = __shfl_sync(0xFFFFFFFFu, dot[p], jj);
#pragma unroll
                for (int c = 0; c < VC; c++) {
                    acc[p][c].x = fmaf(w, vv[c].x, acc[p][c].x);
                    acc[p][c].y = fmaf(w, vv[c].y, acc[p][c].y);
                    acc[p][c].z = fmaf(w, vv[c].z, acc[p][c].z);
                    acc[p][c].w = fmaf(w, vv[c].w, acc[p][c].w);
                }
            }
        }
    }
};

// normalised output of (row, head), value dimension d, times its gate
__device__ __forceinline__ void attn_store(const WindowAttn &a, int row, int head, int d, float v) {
    if (d >= a.vdim) return;
    const int c = head * a.vdim + d;
    if (a.gated) v *= sigmoid_f32(a.ffn.proj[(size_t)row * a.ffn.in_cols + a.c_g + c]);
    store_act(a.ffn.act, a.ffn.act_dt, (size_t)row * a.ffn.out_k + c, v);
}

// A warp takes P consecutive (row, query head of the group) pairs of one kv head, so a key / value row is
// read once per P query vectors; pair t is row t / group, head t % group.
template <int P, int VC>
__global__ void __launch_bounds__(32) attn_rows_kernel(const WindowAttn a) {
    extern __shared__ __align__(16) float rows_qs[];
    const int kvh = blockIdx.x, lane = threadIdx.x;
    const int group = a.heads / a.kv_heads, pairs = a.span.n * group;
    const int t0 = blockIdx.y * P;
    const int n4 = a.dim_ld >> 2;
    const int last_pair = min(pairs, t0 + P) - 1;
    int prow[P];
#pragma unroll
    for (int p = 0; p < P; p++) {
        const int t = min(t0 + p, last_pair);   // pairs past the end repeat the last one; not stored
        prow[p] = t / group;
        const float4 *src = reinterpret_cast<const float4 *>(a.qrot + ((size_t)prow[p] * a.heads + kvh * group + t % group) * a.dim_ld);
        for (int i = lane; i < n4; i += 32) reinterpret_cast<float4 *>(rows_qs)[p * n4 + i] = src[i];
    }
    __syncwarp();
    const int pos0 = a.span.pos0;
    const int first = max(0, pos0 + prow[0] - a.window + 1), last = pos0 + prow[P - 1];
    const float *kb = a.kcache + (size_t)kvh * a.cap * a.dim_ld, *vb = a.vcache + (size_t)kvh * a.cap * a.vdim_ld;
    WarpSoftmax<P, VC> ws;
    ws.init();
    for (int b0 = first; b0 <= last; b0 += 32)
        ws.batch(a, rows_qs, kb, vb, b0, last, [&](int p, int j) {
            const int i = pos0 + prow[p];
            return j <= i && i - j < a.window;
        });
#pragma unroll
    for (int p = 0; p < P; p++) {
        const int t = t0 + p;
        if (t > last_pair) continue;
        const int head = kvh * group + t % group;
        const float inv = 1.0f / ws.l[p];
#pragma unroll
        for (int c = 0; c < VC; c++) {
            const int d = 4 * lane + 128 * c;
            attn_store(a, prow[p], head, d, ws.acc[p][c].x * inv);
            attn_store(a, prow[p], head, d + 1, ws.acc[p][c].y * inv);
            attn_store(a, prow[p], head, d + 2, ws.acc[p][c].z * inv);
            attn_store(a, prow[p], head, d + 3, ws.acc[p][c].w * inv);
        }
    }
}

constexpr int kDecWarps = 4;
constexpr int kDecMaxRanges = 32;

// One token: grid (kv head, key range, tile of P query heads of the group). The window's batches of 32
// keys are dealt to the ranges (contiguous) and to a CTA's warps; the warps merge through shared memory.
// With several ranges a CTA publishes a record (m, l, acc) per head and the last CTA of its (kv head,
// tile) to arrive merges the records; the counter is back at zero for the next launch.
template <int P, int VC>
__global__ void __launch_bounds__(kDecWarps * 32) attn_decode_kernel(const WindowAttn a) {
    pdl_prologue();
    pdl_release();
    extern __shared__ __align__(16) float dec_smem[];
    __shared__ float wm[kDecWarps][P], wl[kDecWarps][P];
    __shared__ int s_last;
    const int kvh = blockIdx.x, range = blockIdx.y, tile = blockIdx.z;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int group = a.heads / a.kv_heads, g0 = tile * P, ng = min(P, group - g0);
    const int n4 = a.dim_ld >> 2, vld = a.vdim_ld;
    float *qs = dec_smem;                    // [P, dim_ld]
    float *wacc = dec_smem + P * a.dim_ld;   // [warps, P, vdim_ld]
    const int pos = a.span.state[1];
    const int first = max(0, pos - a.window + 1);
    const int nb = (pos - first + 32) >> 5;                     // batches of 32 keys
    const int bper = (nb + gridDim.y - 1) / gridDim.y;
    const int used = (nb + bper - 1) / bper;                    // ranges that hold keys
    const int b_lo = range * bper, b_hi = min(nb, b_lo + bper);
    const int slot0 = (kvh * gridDim.z + tile) * gridDim.y;     // this tile's records
    const int rec = vld + 4;                                    // m, l, pad, pad, acc
    if (b_lo < b_hi) {
        for (int i = threadIdx.x; i < P * n4; i += kDecWarps * 32) {
            const int p = i / n4, d4 = i - p * n4;
            reinterpret_cast<float4 *>(qs)[i] =
                reinterpret_cast<const float4 *>(a.qrot + (size_t)(kvh * group + g0 + min(p, ng - 1)) * a.dim_ld)[d4];
        }
        __syncthreads();
        const float *kb = a.kcache + (size_t)kvh * a.cap * a.dim_ld, *vb = a.vcache + (size_t)kvh * a.cap * vld;
        WarpSoftmax<P, VC> ws;
        ws.init();
        for (int b = b_lo + warp; b < b_hi; b += kDecWarps)
            ws.batch(a, qs, kb, vb, first + (b << 5), pos, [](int, int) { return true; });
#pragma unroll
        for (int p = 0; p < P; p++) {
            if (lane == 0) {
                wm[warp][p] = ws.m[p];
                wl[warp][p] = ws.l[p];
            }
#pragma unroll
            for (int c = 0; c < VC; c++)
                if (4 * lane + 128 * c < vld) *reinterpret_cast<float4 *>(&wacc[(warp * P + p) * vld + 4 * lane + 128 * c]) = ws.acc[p][c];
        }
        __syncthreads();
        for (int i = threadIdx.x; i < ng * vld; i += kDecWarps * 32) {
            const int p = i / vld, d = i - p * vld;
            float M = wm[0][p];   // warp 0 always holds a batch: finite
#pragma unroll
            for (int w = 1; w < kDecWarps; w++) M = fmaxf(M, wm[w][p]);
            float L = 0.0f, s = 0.0f;
#pragma unroll
            for (int w = 0; w < kDecWarps; w++) {
                const float e = wm[w][p] == -INFINITY ? 0.0f : expf(wm[w][p] - M);
                L = fmaf(wl[w][p], e, L);
                s = fmaf(wacc[(w * P + p) * vld + d], e, s);
            }
            if (used == 1) {
                attn_store(a, 0, kvh * group + g0 + p, d, s / L);
            } else {
                float *o = a.part + ((size_t)(slot0 + range) * P + p) * rec;
                if (d == 0) {
                    o[0] = M;
                    o[1] = L;
                }
                o[4 + d] = s;
            }
        }
    }
    if (used == 1) return;   // the same for every CTA of the launch: nobody counts
    __threadfence();
    __syncthreads();
    unsigned int *cnt = a.arrived + kvh * gridDim.z + tile;
    if (threadIdx.x == 0) s_last = atomicAdd(cnt, 1u) == gridDim.y - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (int i = threadIdx.x; i < ng * vld; i += kDecWarps * 32) {
        const int p = i / vld, d = i - p * vld;
        const float *r0 = a.part + ((size_t)slot0 * P + p) * rec;
        const size_t step = (size_t)P * rec;
        float M = -INFINITY;
        for (int s = 0; s < used; s++) M = fmaxf(M, __ldcg(r0 + s * step));
        float L = 0.0f, v = 0.0f;
#pragma unroll 4
        for (int s = 0; s < used; s++) {
            const float e = expf(__ldcg(r0 + s * step) - M);
            L = fmaf(__ldcg(r0 + s * step + 1), e, L);
            v = fmaf(__ldcg(r0 + s * step + 4 + d), e, v);
        }
        attn_store(a, 0, kvh * group + g0 + p, d, v / L);
    }
    if (threadIdx.x == 0) *cnt = 0;   // the next launch starts after this grid has ended
}

// ---- host side ----

static int dec_tile(int group) { return group > 4 ? 8 : (group > 2 ? 4 : (group > 1 ? 2 : 1)); }

int attn_decode_ranges(int window, int max_seq) {
    const int keys = window < max_seq ? window : max_seq;
    const int per = 32 * kDecWarps;   // one batch per warp
    const int r = (keys + per - 1) / per;
    return r < 1 ? 1 : (r > kDecMaxRanges ? kDecMaxRanges : r);
}

int attn_decode_counters(int heads, int kv_heads) {
    const int group = heads / kv_heads, P = dec_tile(group);
    return kv_heads * ((group + P - 1) / P);
}

size_t attn_decode_part_floats(int heads, int kv_heads, int vdim_ld, int ranges) {
    return (size_t)attn_decode_counters(heads, kv_heads) * ranges * dec_tile(heads / kv_heads) * (vdim_ld + 4);
}

template <typename K>
static nnq_status allow_smem(nnq_ctx *ctx, K kernel, size_t bytes) {
    if (bytes <= 48 * 1024) return NNQ_OK;
    return check_cuda(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes), "attention shared memory");
}

template <int TAPS>
static nnq_status go_prep(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const int items = (a.span.n + kPrepRows - 1) / kPrepRows * (a.heads + 2 * a.kv_heads);
    const int prep = (items + kPrepWarps - 1) / kPrepWarps;
    const int ffn = ffn_ctas(a.ffn, a.span.n, kPrepWarps * 32, ctx->sm_count);
    const size_t smem = (size_t)kPrepWarps * kPrepRows * (a.dim > a.vdim ? a.dim : a.vdim) * sizeof(float);
    nnq_status s = allow_smem(ctx, attn_prep_kernel<TAPS>, smem);
    if (s != NNQ_OK) return s;
    launch_pdl_smem(attn_prep_kernel<TAPS>, dim3(prep + ffn), dim3(kPrepWarps * 32), smem, st, a, prep);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "attention prologue launch");
}

nnq_status launch_attn_prep(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    switch (a.taps) {
        case 0: return go_prep<0>(ctx, a, st);
        case 2: return go_prep<2>(ctx, a, st);
        case 3: return go_prep<3>(ctx, a, st);
        case 4: return go_prep<4>(ctx, a, st);
        default: return go_prep<-1>(ctx, a, st);
    }
}

nnq_status launch_attn_conv_tail(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    if (a.taps < 2 || a.span.n < 2) return NNQ_OK;
    const int channels = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
    const int rows = a.span.n < a.taps - 1 ? a.span.n : a.taps - 1;
    attn_conv_tail_kernel<<<(rows * channels + 255) / 256, 256, 0, st>>>(a);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "convolution tail launch");
}

template <int P, int VC>
static nnq_status go_rows(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const int pairs = a.span.n * (a.heads / a.kv_heads);
    const size_t smem = (size_t)P * a.dim_ld * sizeof(float);
    nnq_status s = allow_smem(ctx, attn_rows_kernel<P, VC>, smem);
    if (s != NNQ_OK) return s;
    attn_rows_kernel<P, VC><<<dim3(a.kv_heads, (pairs + P - 1) / P), 32, smem, st>>>(a);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "window attention launch");
}

nnq_status launch_attn_rows(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    if (attn_tc_supported(a)) return launch_attn_tc(ctx, a, st);
    return a.vdim_ld <= 128 ? go_rows<8, 1>(ctx, a, st) : go_rows<8, 2>(ctx, a, st);
}

template <int P, int VC>
static nnq_status go_decode(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const int group = a.heads / a.kv_heads;
    const size_t smem = (size_t)P * (a.dim_ld + kDecWarps * a.vdim_ld) * sizeof(float);
    nnq_status s = allow_smem(ctx, attn_decode_kernel<P, VC>, smem);
    if (s != NNQ_OK) return s;
    launch_pdl_smem(attn_decode_kernel<P, VC>, dim3(a.kv_heads, a.ranges, (group + P - 1) / P), dim3(kDecWarps * 32), smem, st, a);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "decode attention launch");
}

nnq_status launch_attn_decode(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const bool wide = a.vdim_ld > 128;
    switch (dec_tile(a.heads / a.kv_heads)) {
        case 1: return wide ? go_decode<1, 2>(ctx, a, st) : go_decode<1, 1>(ctx, a, st);
        case 2: return wide ? go_decode<2, 2>(ctx, a, st) : go_decode<2, 1>(ctx, a, st);
        case 4: return wide ? go_decode<4, 2>(ctx, a, st) : go_decode<4, 1>(ctx, a, st);
        default: return wide ? go_decode<8, 2>(ctx, a, st) : go_decode<8, 1>(ctx, a, st);
    }
}

}  // namespace nnq
