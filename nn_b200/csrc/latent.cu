// Attention through a latent (LatentAttn in blocks.h): preparation of the latents and the decode step. f32: norms,
// rotation, scores, softmax, sums, the query carried into the latent space and the weighted latents.
//
// Decode step, three launches:
//   absorb  a CTA per (head, 128 latent columns): q_lat = scale * W_uk,h^T q_h, the rotated query part beside it; one
//           more CTA norms and appends the new latent. The weight rows are asked for before the wait.
//   scores  a CTA per (range of keys, 16 heads; f32 decoders: eight): scores, softmax and weighted latents of its range, one
//           record each. With bf16 latents on mma.sync (a few heads per step do not fill tcgen05's 128 rows): queries and
//           weights enter as two bf16 terms (hi + lo, remainder below 2^-16), sums are f32; f32 latents on the FMA units.
//   values  a CTA per (head, 32 value dimensions): merges the records of the head and multiplies with W_uv,h.
#include <math.h>

#include "blocks.cuh"

namespace nnq {

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// ---- preparation ----

template <typename T> struct Four;   // four values at once
template <> struct Four<float> { using type = float4; };
template <> struct Four<__nv_bfloat16> { using type = uint2; };

constexpr int kLpWarps = 4;

// v / rms(v) * w of `n` values to o (zeros up to ld) by one warp. Up to 2048 values in whole groups of four stay in registers.
template <typename T>
__device__ __forceinline__ void warp_rms_row(const float *p, const float *w, int n, int ld, float eps, T *o, T *o2) {
    const int lane = threadIdx.x & 31;
    if ((n & 3) == 0 && n <= 2048) {
        float4 v[16];
        float ss = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; k++) v[k] = 4 * (lane + 32 * k) < n ? *reinterpret_cast<const float4 *>(p + 4 * (lane + 32 * k)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int k = 0; k < 16; k++) ss = fmaf(v[k].x, v[k].x, fmaf(v[k].y, v[k].y, fmaf(v[k].z, v[k].z, fmaf(v[k].w, v[k].w, ss))));
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)n + eps);
#pragma unroll
        for (int k = 0; k < 16; k++) {
            const int i = 4 * (lane + 32 * k);
            if (i >= ld) continue;
            const float4 g = i < n ? *reinterpret_cast<const float4 *>(w + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            const float y[4] = {v[k].x * inv * g.x, v[k].y * inv * g.y, v[k].z * inv * g.z, v[k].w * inv * g.w};
            alignas(16) T t[4];
#pragma unroll
            for (int e = 0; e < 4; e++) t[e] = from_f32<T>(y[e]);
            using V = typename Four<T>::type;
            *reinterpret_cast<V *>(o + i) = *reinterpret_cast<const V *>(t);
            if (o2) *reinterpret_cast<V *>(o2 + i) = *reinterpret_cast<const V *>(t);
        }
        return;
    }
    float ss = 0.0f;
    for (int i = lane; i < n; i += 32) ss = fmaf(p[i], p[i], ss);
    const float rms = sqrtf(warp_sum(ss) / (float)n + eps);
    for (int i = lane; i < ld; i += 32) {
        o[i] = from_f32<T>(i < n ? p[i] / rms * w[i] : 0.0f);
        if (o2) o2[i] = o[i];
    }
}

// A warp per item: n query latents, n key latents, then the older positions in groups of four (copied).
template <typename T>
__global__ void __launch_bounds__(kLpWarps * 32) latent_prep_kernel(const LatentAttn a, int nq, int nk, int copy_end) {
    pdl_prologue();
    pdl_release();
    const int lane = threadIdx.x & 31;
    int item = blockIdx.x * kLpWarps + (threadIdx.x >> 5);
    const int pos0 = span_pos(a.span);
    if (item < nq) {
        warp_rms_row<T>(a.proj + (size_t)item * a.in_cols + a.c_q, a.q_norm, a.q_rank, a.q_ld, a.eps, reinterpret_cast<T *>(a.cq) + (size_t)item * a.q_ld, nullptr);
        return;
    }
    item -= nq;
    if (item < nk) {
        const int pos = pos0 + item, half = a.rot >> 1;
        const float *p = a.proj + (size_t)item * a.in_cols + a.c_kv, *r = p + a.kv_rank;
        T *oc = reinterpret_cast<T *>(a.ring_c) + (size_t)(pos % a.cap) * a.kv_ld, *orr = reinterpret_cast<T *>(a.ring_r) + (size_t)(pos % a.cap) * a.rot_ld;
        T *lc = reinterpret_cast<T *>(a.lin_c) + (size_t)(pos - a.first) * a.kv_ld, *lr = reinterpret_cast<T *>(a.lin_r) + (size_t)(pos - a.first) * a.rot_ld;
        warp_rms_row<T>(p, a.kv_norm, a.kv_rank, a.kv_ld, a.eps, oc, a.linear ? lc : nullptr);
        for (int i = lane; i < a.rot_ld; i += 32) {
            const T v = from_f32<T>(i < a.rot ? rotated(r, i, a.rot, a.cosv + (size_t)pos * half, a.sinv + (size_t)pos * half) : 0.0f);
            orr[i] = v;
            if (a.linear) lr[i] = v;
        }
        return;
    }
    item -= nk;
    constexpr int E = 16 / sizeof(T);
    for (int p = a.first + 4 * item; p < min(a.first + 4 * item + 4, copy_end); p++) {
        const uint4 *sc = reinterpret_cast<const uint4 *>(reinterpret_cast<const T *>(a.ring_c) + (size_t)(p % a.cap) * a.kv_ld);
        const uint4 *sr = reinterpret_cast<const uint4 *>(reinterpret_cast<const T *>(a.ring_r) + (size_t)(p % a.cap) * a.rot_ld);
        uint4 *dc = reinterpret_cast<uint4 *>(reinterpret_cast<T *>(a.lin_c) + (size_t)(p - a.first) * a.kv_ld);
        uint4 *dr = reinterpret_cast<uint4 *>(reinterpret_cast<T *>(a.lin_r) + (size_t)(p - a.first) * a.rot_ld);
        for (int i = lane; i < a.kv_ld / E; i += 32) dc[i] = sc[i];
        for (int i = lane; i < a.rot_ld / E; i += 32) dr[i] = sr[i];
    }
}

nnq_status launch_latent_prep(nnq_ctx *ctx, const LatentAttn &a, int parts, cudaStream_t st) {
    const int n = a.span.n, nq = parts & kLatentQueries ? n : 0, nk = (parts & kLatentKeys) && a.c_kv >= 0 ? n : 0;
    const int copy_end = (parts & kLatentKeys) && a.linear ? (a.c_kv >= 0 ? a.span.pos0 : a.span.pos0 + n) : a.first;
    const int items = nq + nk + (copy_end - a.first + 3) / 4;
    if (items == 0) return NNQ_OK;
    const dim3 grid((items + kLpWarps - 1) / kLpWarps), block(kLpWarps * 32);
    if (a.act_dt == NNQ_F32) launch_pdl(latent_prep_kernel<float>, grid, block, st, a, nq, nk, copy_end);
    else launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, block, st, a, nq, nk, copy_end);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "latent preparation launch");
}

// ---- block of rows on the general attention kernels ----

// f32 queries (rotated), keys and values with the shared key part in every head; zeros in the columns of out behind
// the heads'. Grid: (elements of a row, rows of q / keys / out)
template <typename T>
__global__ void __launch_bounds__(256) latent_assemble_kernel(const LatentAttn a, int dl, int vl) {
    pdl_prologue();
    pdl_release();
    const int row = blockIdx.y, n = a.span.n, i = blockIdx.x * 256 + threadIdx.x, dk = a.dim + a.rot, half = a.rot >> 1;
    if (row < n) {
        const int pos = a.span.pos0 + row;
        const float *cs = a.cosv + (size_t)pos * half, *sn = a.sinv + (size_t)pos * half;
        if (i < a.heads * dl) {
            const int h = i / dl, d = i - h * dl;
            const float *q = a.q + ((size_t)row * a.heads + h) * dk;
            a.qrot[((size_t)row * a.heads + h) * dl + d] = d < a.dim ? q[d] : (d < dk ? rotated(q + a.dim, d - a.dim, a.rot, cs, sn) : 0.0f);
        }
        if (i < a.out_ld - a.heads * a.vdim) store_act(a.out, a.act_dt, (size_t)row * a.out_ld + a.heads * a.vdim + i, 0.0f);
        return;
    }
    const int key = row - n;
    const T *kv = reinterpret_cast<const T *>(a.kv) + (size_t)key * a.heads * (a.dim_ld + a.vdim_ld);
    if (i < a.heads * dl) {
        const int h = i / dl, d = i - h * dl;
        const T *r = reinterpret_cast<const T *>(a.lin_r) + (size_t)key * a.rot_ld;
        a.kfull[((size_t)h * a.keys + key) * dl + d] = d < a.dim ? to_f32(kv[h * a.dim_ld + d]) : (d < dk ? to_f32(r[d - a.dim]) : 0.0f);
    }
    if (i < a.heads * vl) {
        const int h = i / vl, d = i - h * vl;
        a.vfull[((size_t)h * a.keys + key) * vl + d] = d < a.vdim ? to_f32(kv[a.heads * a.dim_ld + h * a.vdim_ld + d]) : 0.0f;
    }
}

nnq_status launch_latent_rows(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) {
    if (latent_tc_supported(a.act_dt, a.dim, a.rot, a.vdim)) return launch_latent_tc(ctx, a, st);
    const int dl = round_up(a.dim + a.rot, 4), vl = round_up(a.vdim, 4);
    int width = a.heads * (dl > vl ? dl : vl);
    if (a.out_ld - a.heads * a.vdim > width) width = a.out_ld - a.heads * a.vdim;
    const dim3 grid((width + 255) / 256, a.span.n + a.keys);
    if (a.act_dt == NNQ_F32) launch_pdl(latent_assemble_kernel<float>, grid, dim3(256), st, a, dl, vl);
    else launch_pdl(latent_assemble_kernel<__nv_bfloat16>, grid, dim3(256), st, a, dl, vl);
    ctx->launches++;
    nnq_status s = check_cuda(ctx, cudaGetLastError(), "latent expansion launch");
    if (s != NNQ_OK) return s;
    WindowAttn w = {};
    w.span = {a.span.n, a.span.pos0 - a.first, nullptr};   // positions count from the first key
    w.heads = w.kv_heads = a.heads;
    w.dim = a.dim + a.rot; w.vdim = a.vdim; w.dim_ld = dl; w.vdim_ld = vl;
    w.scale = a.scale; w.window = a.window;
    w.qrot = a.qrot; w.kcache = a.kfull; w.vcache = a.vfull; w.cap = a.keys;
    w.ffn.act = a.out; w.ffn.act_dt = a.act_dt; w.ffn.out_k = a.out_ld;
    return launch_attn_rows(ctx, w, st);
}

// ---- decode step ----

constexpr int kLsThreads = 256, kLsHeads = 8, kLsMaxRanges = 64;   // kLsHeads: of a CTA with f32 latents
constexpr int kLmHeads = 16, kLmProbLd = 80;                         // heads of a CTA with bf16 latents, bytes of a row of weights

__device__ __forceinline__ float bf_at(uint32_t u, int hi) { return __uint_as_float(hi ? u & 0xFFFF0000u : u << 16); }

// Column c of head h's query in the latent space. f32: qlat[h, c]. bf16: two terms at their places in the operand
// fragments of mma.m16n8k16, [16-head tile][16-column step][lane][a0 .. a3 hi, a0 .. a3 lo]. Called by whole warps of
// neighbouring columns, c even in even lanes: the even lane stores the pair.
template <typename T>
__device__ __forceinline__ void store_query(const LatentAttn &a, int h, int c, int ld, float v) {
    if constexpr (sizeof(T) == 4) {
        a.qlat[(size_t)h * ld + c] = v;
    } else {
        const float w = __shfl_down_sync(__activemask(), v, 1);
        if (c & 1) return;
        const __nv_bfloat162 hi = __floats2bfloat162_rn(v, w);
        const uint32_t hb = *reinterpret_cast<const uint32_t *>(&hi);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(v - bf_at(hb, 0), w - bf_at(hb, 1));
        const int r = h & 15, lane = (r & 7) * 4 + ((c & 7) >> 1), reg = (r >> 3) + 2 * ((c >> 3) & 1);
        uint32_t *f = reinterpret_cast<uint32_t *>(a.qlat) + (((size_t)(h >> 4) * (ld >> 4) + (c >> 4)) * 32 + lane) * 8 + reg;
        f[0] = hb;
        f[4] = *reinterpret_cast<const uint32_t *>(&lo);
    }
}

template <typename T>
__global__ void __launch_bounds__(kLsThreads) latent_absorb_kernel(const LatentAttn a) {
    __shared__ float red[16][132];
    __shared__ float qs[1024 + 32];
    const int tid = threadIdx.x, h = blockIdx.x;
    if (h == a.heads) {   // the new latent
        pdl_prologue();
        pdl_release();
        if (blockIdx.y != 0 || a.c_kv < 0) return;
        const int pos = a.span.state[1], half = a.rot >> 1;
        const float *p = a.proj + a.c_kv, *r = p + a.kv_rank;
        float ss = 0.0f;
        for (int i = tid; i < a.kv_rank; i += kLsThreads) ss = fmaf(p[i], p[i], ss);
        const float rms = sqrtf(block_sum(ss, qs) / (float)a.kv_rank + a.eps);
        T *oc = reinterpret_cast<T *>(a.ring_c) + (size_t)(pos % a.cap) * a.kv_ld, *orr = reinterpret_cast<T *>(a.ring_r) + (size_t)(pos % a.cap) * a.rot_ld;
        for (int i = tid; i < a.kv_ld; i += kLsThreads) oc[i] = from_f32<T>(i < a.kv_rank ? p[i] / rms * a.kv_norm[i] : 0.0f);
        for (int i = tid; i < a.rot_ld; i += kLsThreads)
            orr[i] = from_f32<T>(i < a.rot ? rotated(r, i, a.rot, a.cosv + (size_t)pos * half, a.sinv + (size_t)pos * half) : 0.0f);
        return;
    }
    const int rg = tid >> 4, c0 = blockIdx.y * 128 + 8 * (tid & 15);
    const bool in = c0 < a.kv_ld;
    const __nv_bfloat16 *w = a.ukv + (size_t)h * a.dim_ld * a.kv_ld + c0;
    uint4 wv[8];
#pragma unroll
    for (int i = 0; i < 8; i++) wv[i] = in && rg + 16 * i < a.dim ? *reinterpret_cast<const uint4 *>(w + (size_t)(rg + 16 * i) * a.kv_ld) : make_uint4(0, 0, 0, 0);
    pdl_prologue();
    pdl_release();
    const float *q = a.q + (size_t)h * (a.dim + a.rot);
    const int ld = a.kv_ld + a.rot_ld;
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; e++) acc[e] = 0.0f;
    for (int d0 = 0; d0 < a.dim; d0 += 128) {
        __syncthreads();
        for (int i = tid; i < 128; i += kLsThreads) qs[i] = d0 + i < a.dim ? q[d0 + i] : 0.0f;
        __syncthreads();
        if (d0 > 0)
#pragma unroll
            for (int i = 0; i < 8; i++)
                wv[i] = in && d0 + rg + 16 * i < a.dim ? *reinterpret_cast<const uint4 *>(w + (size_t)(d0 + rg + 16 * i) * a.kv_ld) : make_uint4(0, 0, 0, 0);
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const float x = qs[rg + 16 * i];
            const uint32_t u[4] = {wv[i].x, wv[i].y, wv[i].z, wv[i].w};
#pragma unroll
            for (int e = 0; e < 8; e++) acc[e] = fmaf(bf_at(u[e >> 1], e & 1), x, acc[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < 8; e++) red[rg][8 * (tid & 15) + e] = acc[e];
    __syncthreads();
    if (tid < 128 && blockIdx.y * 128 + tid < a.kv_ld) {
        float v = 0.0f;
#pragma unroll
        for (int g = 0; g < 16; g++) v += red[g][tid];
        store_query<T>(a, h, blockIdx.y * 128 + tid, ld, v * a.scale);
    }
    if (blockIdx.y == 0) {
        const int pos = a.span.state[1], half = a.rot >> 1;
        for (int i = tid; i < a.rot_ld; i += kLsThreads)
            store_query<T>(a, h, a.kv_ld + i, ld,
                           i < a.rot ? rotated(q + a.dim, i, a.rot, a.cosv + (size_t)pos * half, a.sinv + (size_t)pos * half) * a.scale : 0.0f);
    }
}

constexpr int kLsKeys = 32;   // keys of a tile

struct LatentSmem {   // bytes
    int keys, q, dots, probs, total;
    int key_ld;       // bytes of a key row
};
template <typename T>
__host__ __device__ inline LatentSmem latent_smem(int kv_ld, int rot_ld) {
    LatentSmem m;
    m.key_ld = (kv_ld + rot_ld) * (int)sizeof(T) + 16;   // rows four banks apart
    m.keys = 0;
    m.q = m.keys + kLsKeys * m.key_ld;
    if (sizeof(T) == 4) {
        m.dots = m.q + kLsHeads * (kv_ld + rot_ld) * 4;
        m.probs = m.dots + 8 * kLsHeads * kLsKeys * 4;
        m.total = m.probs + kLsKeys * kLsHeads * 4;
    } else {
        m.dots = m.q;                                     // (queries come as fragments from global memory)
        m.probs = m.dots + 8 * kLmHeads * kLsKeys * 4;
        m.total = m.probs + 2 * kLmHeads * kLmProbLd;
    }
    return m;
}

__device__ __forceinline__ void cp_async16_latent(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// f32 latents. NV: 512-wide pieces of the latent
template <int NV>
__global__ void __launch_bounds__(kLsThreads) latent_scores_f32_kernel(const LatentAttn a, int per) {
    using T = float;
    constexpr int KT = kLsKeys, P = kLsHeads, E = 4;
    extern __shared__ __align__(16) uint8_t ls_smem[];
    __shared__ float run_m[P], run_l[P], corr_s[P];
    const LatentSmem m = latent_smem<T>(a.kv_ld, a.rot_ld);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int range = blockIdx.x, h0 = blockIdx.y * P, nh = min(P, a.heads - h0);
    const int ld = a.kv_ld + a.rot_ld, uc = a.kv_ld / E, units = ld / E;
    const int pos = a.span.state[1];
    const int first = max(0, pos - a.window + 1);
    const int lo = first + range * per, hi = min(pos + 1, lo + per);
    float *q_s = reinterpret_cast<float *>(ls_smem + m.q), *dots = reinterpret_cast<float *>(ls_smem + m.dots), *probs = reinterpret_cast<float *>(ls_smem + m.probs);
    auto fetch = [&](int p0, int n) {   // positions p0 .. p0 + n - 1 into the tile, from row 0 on
        for (int i = tid; i < n * units; i += kLsThreads) {
            const int r = i / units, c = i - r * units, slot = (p0 + r) % a.cap;
            const T *src = c < uc ? reinterpret_cast<const T *>(a.ring_c) + (size_t)slot * a.kv_ld + c * E
                                  : reinterpret_cast<const T *>(a.ring_r) + (size_t)slot * a.rot_ld + (c - uc) * E;
            cp_async16_latent(ls_smem + m.keys + r * m.key_ld + 16 * c, src);
        }
    };
    // the older latents do not depend on the kernel in front; the current position's is written by it
    if (lo < hi) fetch(lo, min(KT, min(hi, pos) - lo));
    pdl_prologue();
    pdl_release();
    if (lo >= hi) return;
    for (int i = tid; i < P * ld / 4; i += kLsThreads) {
        const int p = i / (ld / 4);
        reinterpret_cast<float4 *>(q_s)[i] = p < nh ? reinterpret_cast<const float4 *>(a.qlat + (size_t)h0 * ld)[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    if (tid < P) {
        run_m[tid] = -INFINITY;
        run_l[tid] = 0.0f;
    }
    // weighted latents: a thread owns column pairs, groups of threads take every G-th key
    int G = 1;
    while (2 * G * (a.kv_ld / 2) <= kLsThreads && G < 8) G *= 2;
    const int gt = kLsThreads / G, grp = tid / gt, ci = tid - grp * gt;
    float acc[NV][2][P];
#pragma unroll
    for (int v = 0; v < NV; v++)
#pragma unroll
        for (int p = 0; p < P; p++) acc[v][0][p] = acc[v][1][p] = 0.0f;
    for (int b0 = lo; b0 < hi; b0 += KT) {
        const int n = min(KT, hi - b0);
        if (b0 > lo) fetch(b0, n);
        else if (n > min(KT, min(hi, pos) - lo)) {   // the current position is in the first tile
            for (int c = tid; c < units; c += kLsThreads) {
                const T *src = c < uc ? reinterpret_cast<const T *>(a.ring_c) + (size_t)(pos % a.cap) * a.kv_ld + c * E
                                      : reinterpret_cast<const T *>(a.ring_r) + (size_t)(pos % a.cap) * a.rot_ld + (c - uc) * E;
                cp_async16_latent(ls_smem + m.keys + (n - 1) * m.key_ld + 16 * c, src);
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        {
            float dot[P];
#pragma unroll
            for (int p = 0; p < P; p++) dot[p] = 0.0f;
            const uint8_t *krow = ls_smem + m.keys + lane * m.key_ld;
            for (int c = warp; c < units; c += 8) {
                const float4 x = *reinterpret_cast<const float4 *>(krow + 16 * c);
#pragma unroll
                for (int p = 0; p < P; p++) {
                    const float4 q = *reinterpret_cast<const float4 *>(q_s + p * ld + c * E);
                    dot[p] = fmaf(q.x, x.x, fmaf(q.y, x.y, fmaf(q.z, x.z, fmaf(q.w, x.w, dot[p]))));
                }
            }
#pragma unroll
            for (int p = 0; p < P; p++) dots[(warp * P + p) * KT + lane] = dot[p];
        }
        __syncthreads();
        {   // softmax of head `warp` over the tile (eight warps, eight heads)
            float d = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; w++) d += dots[(w * P + warp) * KT + lane];
            const float sc = lane < n ? d : -INFINITY;
            const float mo = run_m[warp], mn = fmaxf(mo, warp_max(sc));   // finite: the tile holds a key
            const float e = expf(sc - mn), sum = warp_sum(e);
            probs[lane * P + warp] = e;
            if (lane == 0) {
                const float corr = expf(mo - mn);
                run_m[warp] = mn;
                run_l[warp] = run_l[warp] * corr + sum;
                corr_s[warp] = corr;
            }
        }
        __syncthreads();
#pragma unroll
        for (int v = 0; v < NV; v++)
#pragma unroll
            for (int p = 0; p < P; p++) {
                acc[v][0][p] *= corr_s[p];
                acc[v][1][p] *= corr_s[p];
            }
#pragma unroll 2
        for (int jj = grp; jj < n; jj += G) {
            float w[P];
            const float4 w0 = *reinterpret_cast<const float4 *>(probs + jj * P), w1 = *reinterpret_cast<const float4 *>(probs + jj * P + 4);
            w[0] = w0.x; w[1] = w0.y; w[2] = w0.z; w[3] = w0.w; w[4] = w1.x; w[5] = w1.y; w[6] = w1.z; w[7] = w1.w;
#pragma unroll
            for (int v = 0; v < NV; v++) {
                const int c = 2 * (ci + gt * v);
                if (c >= a.kv_ld) continue;
                const float2 f = *reinterpret_cast<const float2 *>(ls_smem + m.keys + jj * m.key_ld + 4 * c);
#pragma unroll
                for (int p = 0; p < P; p++) {
                    acc[v][0][p] = fmaf(w[p], f.x, acc[v][0][p]);
                    acc[v][1][p] = fmaf(w[p], f.y, acc[v][1][p]);
                }
            }
        }
        __syncthreads();   // the tile may be overwritten
    }
    // groups meet in the key area ([G][P][kv_ld] floats, kv_ld * G <= 512 for G > 1)
    float *sum = reinterpret_cast<float *>(ls_smem + m.keys);
    if (G > 1) {
        if (2 * ci < a.kv_ld)
#pragma unroll
            for (int p = 0; p < P; p++) *reinterpret_cast<float2 *>(sum + ((size_t)grp * P + p) * a.kv_ld + 2 * ci) = make_float2(acc[0][0][p], acc[0][1][p]);
        __syncthreads();
        for (int i = tid; i < nh * a.kv_ld; i += kLsThreads) {
            float v = 0.0f;
            for (int g = 0; g < G; g++) v += sum[(size_t)g * P * a.kv_ld + i];
            const int p = i / a.kv_ld, c = i - p * a.kv_ld;
            a.part[((size_t)range * a.heads + h0 + p) * (a.kv_ld + 4) + 4 + c] = v;
        }
    } else {
#pragma unroll
        for (int v = 0; v < NV; v++) {
            const int c = 2 * (ci + gt * v);
            if (c >= a.kv_ld) continue;
#pragma unroll
            for (int p = 0; p < P; p++)
                if (p < nh) *reinterpret_cast<float2 *>(a.part + ((size_t)range * a.heads + h0 + p) * (a.kv_ld + 4) + 4 + c) = make_float2(acc[v][0][p], acc[v][1][p]);
        }
    }
    if (tid < nh) {
        float *o = a.part + ((size_t)range * a.heads + h0 + tid) * (a.kv_ld + 4);
        o[0] = run_m[tid];
        o[1] = run_l[tid];
    }
}

// bf16 latents on mma.sync. NB: 16-column blocks of the latent per warp.
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

template <int NB>
__global__ void __launch_bounds__(kLsThreads) latent_scores_mma_kernel(const LatentAttn a, int per) {
    using T = __nv_bfloat16;
    constexpr int KT = kLsKeys, P = kLmHeads;
    extern __shared__ __align__(16) uint8_t ls_smem[];
    __shared__ float run_m[P], run_l[P], corr_s[P];
    const LatentSmem m = latent_smem<T>(a.kv_ld, a.rot_ld);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int range = blockIdx.x, h0 = blockIdx.y * P, nh = min(P, a.heads - h0);
    const int ld = a.kv_ld + a.rot_ld, uc = a.kv_ld >> 3, units = ld >> 3, steps = ld >> 4, blocks = a.kv_ld >> 4;
    const int pos = a.span.state[1];
    const int first = max(0, pos - a.window + 1);
    const int lo = first + range * per, hi = min(pos + 1, lo + per);
    float *dots = reinterpret_cast<float *>(ls_smem + m.dots);
    const uint32_t keys_s = (uint32_t)__cvta_generic_to_shared(ls_smem + m.keys), probs_s = (uint32_t)__cvta_generic_to_shared(ls_smem + m.probs);
    auto fetch = [&](int p0, int r0, int n) {   // positions p0 + r0 .. p0 + n - 1 into rows r0 .. n - 1 of the tile
        for (int i = r0 * units + tid; i < n * units; i += kLsThreads) {
            const int r = i / units, c = i - r * units, slot = (p0 + r) % a.cap;
            const T *src = c < uc ? reinterpret_cast<const T *>(a.ring_c) + (size_t)slot * a.kv_ld + c * 8
                                  : reinterpret_cast<const T *>(a.ring_r) + (size_t)slot * a.rot_ld + (c - uc) * 8;
            cp_async16_latent(ls_smem + m.keys + r * m.key_ld + 16 * c, src);
        }
    };
    // the older latents do not depend on the kernel in front; the current position's is written by it
    const int older = lo < hi ? max(0, min(KT, min(hi, pos) - lo)) : 0;
    fetch(lo, 0, older);
    // rows without a key are multiplied with weights of zero: they must hold numbers
    for (int i = older * units + tid; i < KT * units; i += kLsThreads) {
        const int r = i / units, c = i - r * units;
        *reinterpret_cast<uint4 *>(ls_smem + m.keys + r * m.key_ld + 16 * c) = make_uint4(0, 0, 0, 0);
    }
    if (tid < P) {
        run_m[tid] = -INFINITY;
        run_l[tid] = 0.0f;
    }
    pdl_prologue();
    pdl_release();
    if (lo >= hi) return;
    float acc[NB][2][4];
#pragma unroll
    for (int b = 0; b < NB; b++)
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[b][j][e] = 0.0f;
    const uint4 *qf = reinterpret_cast<const uint4 *>(a.qlat) + (size_t)blockIdx.y * steps * 64 + 2 * lane;
    const int g = lane >> 2, tg = lane & 3;
    for (int b0 = lo; b0 < hi; b0 += KT) {
        const int n = min(KT, hi - b0);
        if (b0 == lo) {
            __syncthreads();   // (the zeros of the current position's row)
            fetch(b0, older, n);
        } else {
            fetch(b0, 0, n);
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        {   // scores: a warp takes every eighth step of 16 columns
            float d[4][4];
#pragma unroll
            for (int j = 0; j < 4; j++)
#pragma unroll
                for (int e = 0; e < 4; e++) d[j][e] = 0.0f;
            for (int s = warp; s < steps; s += 8) {
                const uint4 uh = qf[(size_t)s * 64], ul = qf[(size_t)s * 64 + 1];
                const uint32_t qh[4] = {uh.x, uh.y, uh.z, uh.w}, ql[4] = {ul.x, ul.y, ul.z, ul.w};
#pragma unroll
                for (int j = 0; j < 2; j++) {   // 16 keys: matrices (keys 0-7, columns 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15)
                    uint32_t k[4];
                    ldmatrix4(k, keys_s + (16 * j + (lane & 7) + 8 * (lane >> 4)) * m.key_ld + 32 * s + 16 * ((lane >> 3) & 1));
                    mma16816(d[2 * j], qh, k[0], k[1]);
                    mma16816(d[2 * j + 1], qh, k[2], k[3]);
                    mma16816(d[2 * j], ql, k[0], k[1]);
                    mma16816(d[2 * j + 1], ql, k[2], k[3]);
                }
            }
#pragma unroll
            for (int j = 0; j < 4; j++) {
                *reinterpret_cast<float2 *>(dots + (warp * P + g) * KT + 8 * j + 2 * tg) = make_float2(d[j][0], d[j][1]);
                *reinterpret_cast<float2 *>(dots + (warp * P + g + 8) * KT + 8 * j + 2 * tg) = make_float2(d[j][2], d[j][3]);
            }
        }
        __syncthreads();
        {   // softmax: 16 lanes per head, two keys each
            const int p = tid >> 4, c = 2 * (tid & 15);
            float2 sc = make_float2(0.0f, 0.0f);
#pragma unroll
            for (int w = 0; w < 8; w++) {
                const float2 x = *reinterpret_cast<const float2 *>(dots + (w * P + p) * KT + c);
                sc.x += x.x;
                sc.y += x.y;
            }
            if (c >= n) sc.x = -INFINITY;
            if (c + 1 >= n) sc.y = -INFINITY;
            float mx = fmaxf(sc.x, sc.y);
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xFFFFFFFFu, mx, off));
            const float mo = run_m[p], mn = fmaxf(mo, mx);   // finite: the tile holds a key
            const float e0 = expf(sc.x - mn), e1 = expf(sc.y - mn);
            float sum = e0 + e1;
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xFFFFFFFFu, sum, off);
            const __nv_bfloat162 hi2 = __floats2bfloat162_rn(e0, e1);
            const uint32_t hb = *reinterpret_cast<const uint32_t *>(&hi2);
            const __nv_bfloat162 lo2 = __floats2bfloat162_rn(e0 - bf_at(hb, 0), e1 - bf_at(hb, 1));
            *reinterpret_cast<uint32_t *>(ls_smem + m.probs + p * kLmProbLd + 2 * c) = hb;
            *reinterpret_cast<uint32_t *>(ls_smem + m.probs + (P + p) * kLmProbLd + 2 * c) = *reinterpret_cast<const uint32_t *>(&lo2);
            __syncwarp();   // (run_m is read by all sixteen lanes above)
            if ((tid & 15) == 0) {
                const float corr = expf(mo - mn);
                run_m[p] = mn;
                run_l[p] = run_l[p] * corr + sum;
                corr_s[p] = corr;
            }
        }
        __syncthreads();
        {   // weighted latents: a warp takes every eighth block of 16 columns
            const float c0 = corr_s[g], c1 = corr_s[g + 8];
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int k = 0; k < 2; k++) {   // 16 keys: matrices (heads 0-7, keys 0-7), (8-15, 0-7), (0-7, 8-15), (8-15, 8-15)
                const uint32_t at = probs_s + ((lane & 7) + 8 * ((lane >> 3) & 1)) * kLmProbLd + 32 * k + 16 * (lane >> 4);
                ldmatrix4(ph[k], at);
                ldmatrix4(pl[k], at + P * kLmProbLd);
            }
#pragma unroll
            for (int b = 0; b < NB; b++) {
                const int blk = warp + 8 * b;
                if (blk >= blocks) continue;
#pragma unroll
                for (int j = 0; j < 2; j++) {
                    acc[b][j][0] *= c0; acc[b][j][1] *= c0; acc[b][j][2] *= c1; acc[b][j][3] *= c1;
                }
#pragma unroll
                for (int k = 0; k < 2; k++) {   // transposed: (keys 0-7, columns 0-7), (keys 8-15, columns 0-7), then columns 8-15
                    uint32_t v[4];
                    ldmatrix4_t(v, keys_s + (16 * k + (lane & 7) + 8 * ((lane >> 3) & 1)) * m.key_ld + 32 * blk + 16 * (lane >> 4));
                    mma16816(acc[b][0], ph[k], v[0], v[1]);
                    mma16816(acc[b][1], ph[k], v[2], v[3]);
                    mma16816(acc[b][0], pl[k], v[0], v[1]);
                    mma16816(acc[b][1], pl[k], v[2], v[3]);
                }
            }
        }
        __syncthreads();   // the tile may be overwritten
    }
    float *rec = a.part + ((size_t)range * a.heads + h0) * (a.kv_ld + 4);
#pragma unroll
    for (int b = 0; b < NB; b++) {
        const int blk = warp + 8 * b;
        if (blk >= blocks) continue;
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int c = 4 + 16 * blk + 8 * j + 2 * tg;
            if (g < nh) *reinterpret_cast<float2 *>(rec + (size_t)g * (a.kv_ld + 4) + c) = make_float2(acc[b][j][0], acc[b][j][1]);
            if (g + 8 < nh) *reinterpret_cast<float2 *>(rec + (size_t)(g + 8) * (a.kv_ld + 4) + c) = make_float2(acc[b][j][2], acc[b][j][3]);
        }
    }
    if (tid < nh) *reinterpret_cast<float2 *>(rec + (size_t)tid * (a.kv_ld + 4)) = make_float2(run_m[tid], run_l[tid]);
}

constexpr int kLvRows = 4, kLvGroups = 8;   // value dimensions of a warp; most groups of threads that share the records

// grid (heads, ceil(vdim / 32)). NU: 256-wide pieces of the latent
// (NU = 2: few enough registers for the product behind it to become resident)
template <int NU>
__global__ void __launch_bounds__(kLsThreads, NU <= 2 ? 3 : 1) latent_values_kernel(const LatentAttn a, int per) {
    __shared__ __align__(16) float parts[1024];   // G rows of kv_ld
    __shared__ float wt[8][kLsMaxRanges];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x;
    const int v0 = blockIdx.y * 8 * kLvRows + warp * kLvRows, nu = a.kv_ld >> 3;
    const __nv_bfloat16 *w = a.ukv + ((size_t)a.heads * a.dim_ld + (size_t)h * a.vdim_ld + v0) * a.kv_ld;
    uint4 wv[kLvRows][NU];
#pragma unroll
    for (int r = 0; r < kLvRows; r++)
#pragma unroll
        for (int u = 0; u < NU; u++)
            wv[r][u] = v0 + r < a.vdim && lane + 32 * u < nu ? *reinterpret_cast<const uint4 *>(w + (size_t)r * a.kv_ld + 8 * (lane + 32 * u)) : make_uint4(0, 0, 0, 0);
    pdl_prologue();
    pdl_release();
    const int pos = a.span.state[1], keys = min(pos + 1, a.window), used = (keys + per - 1) / per;
    const size_t step = (size_t)a.heads * (a.kv_ld + 4);
    const float *rec = a.part + (size_t)h * (a.kv_ld + 4);
    // groups of kv_ld / 4 threads take every G-th record; the first batch of records is asked for before their weights
    const int cols = a.kv_ld >> 2, G = min(kLvGroups, kLsThreads / cols), grp = tid / cols, ci = tid - grp * cols;
    float4 x[8];
#pragma unroll
    for (int k = 0; k < 8; k++) {
        const int s = grp + k * G;
        x[k] = grp < G && s < used ? *reinterpret_cast<const float4 *>(rec + s * step + 4 + 4 * ci) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    {   // every warp forms the weights of all records for itself
        float mv[2], lv[2], mx = -INFINITY, sum = 0.0f;
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int s = lane + 32 * k;
            const float2 ml = s < used ? *reinterpret_cast<const float2 *>(rec + s * step) : make_float2(-INFINITY, 0.0f);
            mv[k] = ml.x;
            lv[k] = ml.y;
            mx = fmaxf(mx, mv[k]);
        }
        mx = warp_max(mx);
#pragma unroll
        for (int k = 0; k < 2; k++) {
            mv[k] = expf(mv[k] - mx);
            sum = fmaf(lv[k], mv[k], sum);
        }
        sum = warp_sum(sum);
        wt[warp][lane] = mv[0] / sum;
        wt[warp][lane + 32] = mv[1] / sum;
        __syncwarp();
    }
    float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (grp < G)
        for (int s0 = grp; s0 < used; s0 += 8 * G) {
#pragma unroll
            for (int k = 0; k < 8; k++) {
                const int s = s0 + k * G;
                if (s >= used) continue;
                if (s0 != grp) x[k] = *reinterpret_cast<const float4 *>(rec + s * step + 4 + 4 * ci);
                const float e = wt[warp][s];
                v.x = fmaf(e, x[k].x, v.x); v.y = fmaf(e, x[k].y, v.y); v.z = fmaf(e, x[k].z, v.z); v.w = fmaf(e, x[k].w, v.w);
            }
        }
    if (grp < G) *reinterpret_cast<float4 *>(parts + grp * a.kv_ld + 4 * ci) = v;
    __syncthreads();
    if (G > 1) {
        if (tid < cols) {
            for (int k = 1; k < G; k++) {
                const float4 y = *reinterpret_cast<const float4 *>(parts + k * a.kv_ld + 4 * tid);
                v.x += y.x; v.y += y.y; v.z += y.z; v.w += y.w;
            }
            *reinterpret_cast<float4 *>(parts + 4 * tid) = v;
        }
        __syncthreads();
    }
    const float *lat = parts;
    float acc[kLvRows];
#pragma unroll
    for (int r = 0; r < kLvRows; r++) acc[r] = 0.0f;
#pragma unroll
    for (int u = 0; u < NU; u++) {
        if (lane + 32 * u >= nu) continue;
        const float4 x0 = *reinterpret_cast<const float4 *>(lat + 8 * (lane + 32 * u)), x1 = *reinterpret_cast<const float4 *>(lat + 8 * (lane + 32 * u) + 4);
        const float x[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
        for (int r = 0; r < kLvRows; r++) {
            const uint32_t q[4] = {wv[r][u].x, wv[r][u].y, wv[r][u].z, wv[r][u].w};
#pragma unroll
            for (int e = 0; e < 8; e++) acc[r] = fmaf(bf_at(q[e >> 1], e & 1), x[e], acc[r]);
        }
    }
#pragma unroll
    for (int r = 0; r < kLvRows; r++) {
        const float v = warp_sum(acc[r]);
        if (lane == 0 && v0 + r < a.vdim) store_act(a.out, a.act_dt, h * a.vdim + v0 + r, v);
    }
    if (h == 0 && blockIdx.y == 0)
        for (int i = a.heads * a.vdim + tid; i < a.out_ld; i += kLsThreads) store_act(a.out, a.act_dt, i, 0.0f);
}

// ---- host side ----

static int step_heads(int act_dt) { return act_dt == NNQ_F32 ? kLsHeads : kLmHeads; }
static int range_keys(int ranges, int keys) { return ((keys + ranges - 1) / ranges + kLsKeys - 1) / kLsKeys * kLsKeys; }

int latent_step_ranges(int sm_count, int heads, int window, int max_seq, int act_dt) {
    const int keys = window < max_seq ? window : max_seq, tiles = (heads + step_heads(act_dt) - 1) / step_heads(act_dt);
    int r = sm_count / tiles;
    r = r < 1 ? 1 : (r > kLsMaxRanges ? kLsMaxRanges : r);
    return (keys + range_keys(r, keys) - 1) / range_keys(r, keys);
}

size_t latent_step_query_floats(int heads, int kv_ld, int rot_ld) { return (size_t)round_up(heads, kLmHeads) * (kv_ld + rot_ld); }

bool latent_step_supported(int act_dt, int kv_ld, int rot_ld) {
    const int smem = act_dt == NNQ_F32 ? latent_smem<float>(kv_ld, rot_ld).total : latent_smem<__nv_bfloat16>(kv_ld, rot_ld).total;
    return kv_ld <= 1024 && smem <= 220 * 1024;
}

template <typename K>
static nnq_status go_scores(nnq_ctx *ctx, K kernel, const LatentAttn &a, int per, int smem, cudaStream_t st) {
    nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "latent attention shared memory");
    if (s != NNQ_OK) return s;
    const int heads = step_heads(a.act_dt);
    launch_pdl_smem(kernel, dim3(a.ranges, (a.heads + heads - 1) / heads), dim3(kLsThreads), smem, st, a, per);
    return check_cuda(ctx, cudaGetLastError(), "latent attention launch");
}

nnq_status launch_latent_step(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) {
    const bool f32 = a.act_dt == NNQ_F32;
    const int per = range_keys(a.ranges, a.keys_max);
    const dim3 ag(a.heads + 1, (a.kv_ld + 127) / 128), ab(kLsThreads);
    if (f32) launch_pdl(latent_absorb_kernel<float>, ag, ab, st, a);
    else launch_pdl(latent_absorb_kernel<__nv_bfloat16>, ag, ab, st, a);
    nnq_status s = check_cuda(ctx, cudaGetLastError(), "latent query launch");
    if (s != NNQ_OK) return s;
    if (f32) {
        const int smem = latent_smem<float>(a.kv_ld, a.rot_ld).total;
        s = a.kv_ld <= 512 ? go_scores(ctx, latent_scores_f32_kernel<1>, a, per, smem, st) : go_scores(ctx, latent_scores_f32_kernel<2>, a, per, smem, st);
    } else {
        const int smem = latent_smem<__nv_bfloat16>(a.kv_ld, a.rot_ld).total;
        s = a.kv_ld <= 512 ? go_scores(ctx, latent_scores_mma_kernel<4>, a, per, smem, st) : go_scores(ctx, latent_scores_mma_kernel<8>, a, per, smem, st);
    }
    if (s != NNQ_OK) return s;
    const dim3 vg(a.heads, (a.vdim + 8 * kLvRows - 1) / (8 * kLvRows));
    if (a.kv_ld <= 512) launch_pdl(latent_values_kernel<2>, vg, ab, st, a, per);
    else launch_pdl(latent_values_kernel<4>, vg, ab, st, a, per);
    ctx->launches += 3;
    return check_cuda(ctx, cudaGetLastError(), "latent value launch");
}

}  // namespace nnq
