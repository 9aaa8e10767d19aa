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

// ---- one token: everything of the layer between its two products in one launch ----
//
// CTA = (kv head, tile of P query heads of its group, range of keys); 256 threads. Before it waits for the product
// in front of it, a CTA asks for the keys and values of its range (they do not depend on this token) and forms the
// part of its convolutions that lies in the past. After the wait: convolution and rotation of its query heads (and
// of the new key and value in the CTAs that hold the current position), scores with a warp per eighth of the
// dimensions, softmax with a lane per two keys, values with a thread per dimension. Ranges are merged by the CTA of
// a (kv head, tile) that finishes last. Further CTAs do the feed-forward part.
constexpr int kStepThreads = 256, kStepKeys = 64, kStepMaxRanges = 64;

struct StepSmem {   // offsets in floats
    int k, v, q, raw, trig, dots, probs, total;
    int k_ld;
};
__host__ __device__ inline StepSmem step_smem(int P, int dim, int dim_ld, int vdim_ld) {
    StepSmem m;
    m.k_ld = dim_ld + 4;   // rows four banks apart: eight lanes reading 16 bytes of eight rows meet no bank twice
    int at = 0;
    auto take = [&](int n) {
        const int o = at;
        at += (n + 3) / 4 * 4;
        return o;
    };
    m.k = take(kStepKeys * m.k_ld);
    m.v = take(kStepKeys * vdim_ld);
    m.q = take(P * dim_ld);
    m.raw = take(P * dim + dim + vdim_ld);        // convolved values before the rotation: query heads, key, value
    m.trig = take(dim);                        // cosines and sines of the current position
    m.dots = take(8 * P * kStepKeys);          // partial scores of the eight warps
    m.probs = take(kStepKeys * P);
    m.total = at;
    return m;
}

__device__ __forceinline__ void cp_async16_attn(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <int P>
__global__ void __launch_bounds__(kStepThreads) attn_step_kernel(const WindowAttn a, int attn_ctas, int per) {
    extern __shared__ __align__(16) float st_smem[];
    __shared__ float run_m[P], run_l[P], corr_s[P];
    __shared__ int s_last;
    if ((int)blockIdx.x >= attn_ctas) {
        pdl_prologue();
        pdl_release();
        ffn_part(a.ffn, 1, attn_ctas);
        return;
    }
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int group = a.heads / a.kv_heads, tiles = (group + P - 1) / P;
    const int range = blockIdx.x % a.ranges, kt = blockIdx.x / a.ranges, tile = kt % tiles, kvh = kt / tiles;
    const int g0 = tile * P, ng = min(P, group - g0), h0 = kvh * group + g0;
    const StepSmem m = step_smem(P, a.dim, a.dim_ld, a.vdim_ld);
    const int n4 = a.dim_ld >> 2, v4 = a.vdim_ld >> 2;
    const int pos = a.span.state[1];
    const int first = max(0, pos - a.window + 1), keys = pos - first + 1;
    const int used = (keys + per - 1) / per;                        // ranges that hold keys
    const int lo = first + range * per, hi = min(pos + 1, lo + per);  // this CTA's keys [lo, hi)
    const bool active = lo < hi, owns_pos = active && hi == pos + 1;
    const float *kb = a.kcache + (size_t)kvh * a.cap * a.dim_ld, *vb = a.vcache + (size_t)kvh * a.cap * a.vdim_ld;
    // keys and values b0 .. b0 + 63 of the range, the current position's excepted
    auto fetch = [&](int b0) {
        const int n = min(kStepKeys, min(hi, pos) - b0), s0 = b0 % a.cap;
        for (int i = tid; i < n * n4; i += kStepThreads) {
            const int r = i / n4, c = i - r * n4;
            int slot = s0 + r;
            if (slot >= a.cap) slot -= a.cap;
            cp_async16_attn(st_smem + m.k + r * m.k_ld + 4 * c, kb + (size_t)slot * a.dim_ld + 4 * c);
        }
        for (int i = tid; i < n * v4; i += kStepThreads) {
            const int r = i / v4, c = i - r * v4;
            int slot = s0 + r;
            if (slot >= a.cap) slot -= a.cap;
            cp_async16_attn(st_smem + m.v + r * a.vdim_ld + 4 * c, vb + (size_t)slot * a.vdim_ld + 4 * c);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    // the channels this CTA convolves: its query heads, then (with the current position) the key and the value
    const int qn = ng * a.dim, total = qn + (owns_pos ? a.dim + a.vdim : 0);
    const int channels = a.heads * a.dim + a.kv_heads * (a.dim + a.vdim);
    auto locate = [&](int i, int &c, int &col) {
        if (i < qn) {
            c = h0 * a.dim + i;
            col = a.c_q + c;
        } else if (i < qn + a.dim) {
            c = (a.heads + kvh) * a.dim + i - qn;
            col = a.c_k + kvh * a.dim + i - qn;
        } else {
            c = (a.heads + a.kv_heads) * a.dim + kvh * a.vdim + i - qn - a.dim;
            col = a.c_v + kvh * a.vdim + i - qn - a.dim;
        }
    };
    float *raw = st_smem + m.raw;
    const int half = a.rot_dims >> 1;
    const float *cs = st_smem + m.trig, *sn = cs + half;
    if (active) {
        fetch(lo);
        for (int i = tid; i < half; i += kStepThreads) {
            st_smem[m.trig + i] = a.cosv[(size_t)pos * half + i];
            st_smem[m.trig + half + i] = a.sinv[(size_t)pos * half + i];
        }
        if (a.taps > 1) {
            for (int i = tid; i < total; i += kStepThreads) {
                int c, col;
                locate(i, c, col);
                float y = 0.0f;
                for (int t = 0; t < a.taps - 1; t++) {
                    const int back = a.taps - 1 - t;
                    const float u = pos >= back ? a.conv_ring[(size_t)((pos - back) % a.taps) * channels + c] : 0.0f;
                    y = fmaf(a.conv[(size_t)c * a.taps + t], u, y);
                }
                raw[(i < qn ? 0 : P * a.dim - qn) + i] = y;   // key and value behind all P query heads' places
            }
        }
    }
    if (tid < P) {
        run_m[tid] = -INFINITY;
        run_l[tid] = 0.0f;
    }
    pdl_prologue();
    pdl_release();
    float acc[P];
#pragma unroll
    for (int p = 0; p < P; p++) acc[p] = 0.0f;
    if (active) {
        for (int i = tid; i < total; i += kStepThreads) {
            int c, col;
            locate(i, c, col);
            const float u = a.ffn.proj[col];
            float &y = raw[(i < qn ? 0 : P * a.dim - qn) + i];
            if (a.taps > 1) {
                y = fmaf(a.conv[(size_t)c * a.taps + a.taps - 1], u, y);
                // this position's slot is read by nobody in this launch (readers look 1 .. taps - 1 back)
                if (i < qn ? range == 0 : tile == 0) a.conv_ring[(size_t)(pos % a.taps) * channels + c] = u;
            } else {
                y = a.taps == 1 ? a.conv[c] * u : u;
            }
        }
        __syncthreads();
        for (int i = tid; i < P * a.dim_ld; i += kStepThreads) {
            const int p = i / a.dim_ld, d = i - p * a.dim_ld;
            st_smem[m.q + i] = p < ng && d < a.dim ? rotated(raw + p * a.dim, d, a.rot_dims, cs, sn) : 0.0f;
        }
        if (owns_pos) {
            // the new key and value: into the cache, and into the shared tile that holds them (the last one)
            const int slot = pos % a.cap, r = (pos - lo) % kStepKeys;
            const bool now = pos - lo < kStepKeys;
            const float *rk = raw + P * a.dim, *rv = rk + a.dim;
            for (int d = tid; d < a.dim_ld; d += kStepThreads) {
                const float k = d < a.dim ? rotated(rk, d, a.rot_dims, cs, sn) : 0.0f;
                if (now) st_smem[m.k + r * m.k_ld + d] = k;
                if (tile == 0) a.kcache[((size_t)kvh * a.cap + slot) * a.dim_ld + d] = k;
            }
            for (int d = tid; d < a.vdim_ld; d += kStepThreads) {
                float v = d < a.vdim ? rv[d] : 0.0f;
                if (d < a.vdim && a.mix_mode == 1 && tile == 0) a.vfirst[kvh * a.vdim + d] = v;
                else if (d < a.vdim && a.mix_mode == 2) v = (1.0f - a.lambda) * v + a.lambda * a.vfirst[kvh * a.vdim + d];
                if (now) st_smem[m.v + r * a.vdim_ld + d] = v;
                if (tile == 0) a.vcache[((size_t)kvh * a.cap + slot) * a.vdim_ld + d] = v;
                if (!now) raw[P * a.dim + a.dim + d] = v;   // (vdim_ld - vdim zeros fit: the area is rounded up)
            }
        }
        for (int b0 = lo; b0 < hi; b0 += kStepKeys) {
            if (b0 > lo) fetch(b0);
            const int n = min(kStepKeys, hi - b0);
            if (b0 > lo && owns_pos && b0 + n == hi) {   // a later tile holds the current position
                const int r = n - 1;
                const float *rk = raw + P * a.dim, *rv = rk + a.dim;
                for (int d = tid; d < a.dim_ld; d += kStepThreads) st_smem[m.k + r * m.k_ld + d] = d < a.dim ? rotated(rk, d, a.rot_dims, cs, sn) : 0.0f;
                for (int d = tid; d < a.vdim_ld; d += kStepThreads) st_smem[m.v + r * a.vdim_ld + d] = d < a.vdim ? rv[d] : 0.0f;
            }
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();
            // scores: warp w takes every eighth group of four dimensions, a lane two keys
            {
                float dot[2][P];
#pragma unroll
                for (int p = 0; p < P; p++) dot[0][p] = dot[1][p] = 0.0f;
                const float *k0 = st_smem + m.k + lane * m.k_ld, *k1 = k0 + 32 * m.k_ld;
                for (int c = warp; c < n4; c += 8) {
                    const float4 x = *reinterpret_cast<const float4 *>(k0 + 4 * c), y = *reinterpret_cast<const float4 *>(k1 + 4 * c);
#pragma unroll
                    for (int p = 0; p < P; p++) {
                        const float4 q = *reinterpret_cast<const float4 *>(st_smem + m.q + p * a.dim_ld + 4 * c);
                        dot[0][p] = fmaf(q.x, x.x, fmaf(q.y, x.y, fmaf(q.z, x.z, fmaf(q.w, x.w, dot[0][p]))));
                        dot[1][p] = fmaf(q.x, y.x, fmaf(q.y, y.y, fmaf(q.z, y.z, fmaf(q.w, y.w, dot[1][p]))));
                    }
                }
#pragma unroll
                for (int p = 0; p < P; p++) {
                    st_smem[m.dots + (warp * P + p) * kStepKeys + lane] = dot[0][p];
                    st_smem[m.dots + (warp * P + p) * kStepKeys + 32 + lane] = dot[1][p];
                }
            }
            __syncthreads();
            if (warp < P) {   // softmax of head `warp` over the tile
                float sc[2];
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    float d = 0.0f;
#pragma unroll
                    for (int w = 0; w < 8; w++) d += st_smem[m.dots + (w * P + warp) * kStepKeys + 32 * e + lane];
                    sc[e] = 32 * e + lane < n ? d * a.scale : -INFINITY;
                }
                const float mo = run_m[warp], mn = fmaxf(mo, warp_max(fmaxf(sc[0], sc[1])));   // finite: the tile holds a key
                const float p0 = expf(sc[0] - mn), p1 = expf(sc[1] - mn), corr = expf(mo - mn);
                const float sum = warp_sum(p0 + p1);
                st_smem[m.probs + lane * P + warp] = p0;
                st_smem[m.probs + (32 + lane) * P + warp] = p1;
                if (lane == 0) {
                    run_m[warp] = mn;
                    run_l[warp] = run_l[warp] * corr + sum;
                    corr_s[warp] = corr;
                }
            }
            __syncthreads();
            // values: a thread per dimension; with at most 128 of them the two halves of the CTA take every other key
            const bool split = a.vdim_ld <= 128;
            const int d0 = split ? tid & 127 : tid, j0 = split ? tid >> 7 : 0, dj = split ? 2 : 1;
#pragma unroll
            for (int p = 0; p < P; p++) acc[p] *= corr_s[p];
            if (d0 < a.vdim_ld) {
#pragma unroll 4
                for (int jj = j0; jj < n; jj += dj) {
                    const float v = st_smem[m.v + jj * a.vdim_ld + d0];
#pragma unroll
                    for (int p = 0; p < P; p++) acc[p] = fmaf(st_smem[m.probs + jj * P + p], v, acc[p]);
                }
            }
            __syncthreads();   // the tile may be overwritten
        }
        if (a.vdim_ld <= 128) {   // the halves meet (in the score area)
            if (tid >= 128 && (tid & 127) < a.vdim_ld)
#pragma unroll
                for (int p = 0; p < P; p++) st_smem[m.dots + p * 128 + (tid & 127)] = acc[p];
            __syncthreads();
            if (tid < a.vdim_ld)
#pragma unroll
                for (int p = 0; p < P; p++) acc[p] += st_smem[m.dots + p * 128 + tid];
        }
        if (tid < a.vdim_ld) {
#pragma unroll
            for (int p = 0; p < P; p++) {
                if (p >= ng) continue;
                if (used == 1) {
                    attn_store(a, 0, h0 + p, tid, acc[p] / run_l[p]);
                } else {
                    float *o = a.part + ((size_t)(kt * a.ranges + range) * P + p) * (a.vdim_ld + 4);   // record: m, l, pad, pad, acc
                    if (tid == 0) {
                        o[0] = run_m[p];
                        o[1] = run_l[p];
                    }
                    o[4 + tid] = acc[p];
                }
            }
        }
    }
    if (used == 1 || !active) return;   // ranges without keys are not counted
    __threadfence();
    __syncthreads();
    unsigned int *cnt = a.arrived + kt;
    if (tid == 0) s_last = atomicAdd(cnt, 1u) == (unsigned)(used - 1);
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    for (int i = tid; i < ng * a.vdim_ld; i += kStepThreads) {
        const int p = i / a.vdim_ld, d = i - p * a.vdim_ld;
        const size_t step = (size_t)P * (a.vdim_ld + 4);
        const float *r0 = a.part + ((size_t)(kt * a.ranges) * P + p) * (a.vdim_ld + 4);
        float M = -INFINITY, L = 0.0f, v = 0.0f;
        for (int s0 = 0; s0 < used; s0 += 8) {
            float2 ml[8];
            float x[8];
#pragma unroll
            for (int s = 0; s < 8; s++) {   // all loads of a pass before the first is used
                ml[s] = s0 + s < used ? __ldcg(reinterpret_cast<const float2 *>(r0 + (s0 + s) * step)) : make_float2(-INFINITY, 0.0f);
                x[s] = s0 + s < used ? __ldcg(r0 + (s0 + s) * step + 4 + d) : 0.0f;
            }
            float mx = M;
#pragma unroll
            for (int s = 0; s < 8; s++) mx = fmaxf(mx, ml[s].x);
            const float c = expf(M - mx);
            L *= c;
            v *= c;
#pragma unroll
            for (int s = 0; s < 8; s++) {
                const float e = expf(ml[s].x - mx);
                L = fmaf(ml[s].y, e, L);
                v = fmaf(x[s], e, v);
            }
            M = mx;
        }
        attn_store(a, 0, h0 + p, d, v / L);
    }
    if (tid == 0) *cnt = 0;   // the next launch starts after this grid has ended
}

// ---- host side ----

static int dec_tile(int group) { return group > 4 ? 8 : (group > 2 ? 4 : (group > 1 ? 2 : 1)); }
static int dec_tiles(int heads, int kv_heads) { return kv_heads * ((heads / kv_heads + dec_tile(heads / kv_heads) - 1) / dec_tile(heads / kv_heads)); }

// Ranges of whole 64-key tiles, as many as leave at most one CTA per SM.
static int step_per(int ranges, int keys) { return ((keys + ranges - 1) / ranges + kStepKeys - 1) / kStepKeys * kStepKeys; }

int attn_step_ranges(int sm_count, int heads, int kv_heads, int window, int max_seq) {
    const int keys = window < max_seq ? window : max_seq;
    int r = sm_count / dec_tiles(heads, kv_heads);
    r = r < 1 ? 1 : (r > kStepMaxRanges ? kStepMaxRanges : r);
    return (keys + step_per(r, keys) - 1) / step_per(r, keys);
}

int attn_step_counters(int heads, int kv_heads) { return dec_tiles(heads, kv_heads); }

size_t attn_step_part_floats(int heads, int kv_heads, int vdim_ld, int ranges) {
    return (size_t)dec_tiles(heads, kv_heads) * ranges * dec_tile(heads / kv_heads) * (vdim_ld + 4);
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

template <int P>
static nnq_status go_step(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const int ctas = dec_tiles(a.heads, a.kv_heads) * a.ranges;
    const size_t smem = (size_t)step_smem(P, a.dim, a.dim_ld, a.vdim_ld).total * sizeof(float);
    nnq_status s = allow_smem(ctx, attn_step_kernel<P>, smem);
    if (s != NNQ_OK) return s;
    launch_pdl_smem(attn_step_kernel<P>, dim3(ctas + ffn_ctas(a.ffn, 1, kStepThreads, ctx->sm_count)), dim3(kStepThreads), smem, st, a, ctas,
                    step_per(a.ranges, a.keys_max));
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "attention step launch");
}

nnq_status launch_attn_step(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    switch (dec_tile(a.heads / a.kv_heads)) {
        case 1: return go_step<1>(ctx, a, st);
        case 2: return go_step<2>(ctx, a, st);
        case 4: return go_step<4>(ctx, a, st);
        default: return go_step<8>(ctx, a, st);
    }
}

}  // namespace nnq
