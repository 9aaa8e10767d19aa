// y[M, N] = x[M, K] W^T (+ bias) for an unquantized bf16 weight and one to four bf16 rows (a decode step).
//
// The work is one pass over the weight, so the kernel is built around keeping enough of it in flight: one CTA
// per SM, sixteen warps (eight for three and four rows), each with a private ring of bulk copies (cp.async.bulk on mbarriers, up to 160 KB in
// flight per SM). A warp owns one chunk of at most 1024 columns for all of its rows: its x values stay in
// registers (a lane's 32 of them as bf16 pairs) and a tile is one row's chunk, 2 KB. KS warps share a row; their
// partial sums meet in shared memory once, at the end. The ring is filled before the kernel waits for its
// predecessor (programmatic dependent launch): the small kernels in front of a product release it early, so the
// weights stream while they run. With GemvNorm.half it takes half of the warps and of the ring, so that two of them, or one
// and a small kernel, fit on an SM. Products bf16 x bf16 in f32, f32 sums. Every wait is bounded.
//
// With NORM the kernel also does what stands in front of a decoder's product: every CTA adds the last block's output
// to the residual row (or reads the embedding row), norms it and keeps the normed row as bf16 in shared memory; CTA 0
// writes the new residual to another buffer (the others may still be reading the old one). Behind a gate / up product
// with interleaved rows the epilogue forms the gated activation. For a mixture of experts the rows (gate / up) or the
// segments of the columns (down) belong to the experts the row is routed to: their addresses are known only behind the
// wait, everything else is the same.
#include <cuda_bf16.h>

#include "block_norm.cuh"
#include "gemm_tc.h"
#include "route.cuh"
#include "sync.cuh"

namespace nnq {

constexpr int kGvChunk = 1024, kGvTileBytes = kGvChunk * 2, kGvTiles = 64, kGvRing = kGvTiles * kGvTileBytes;
// warps of a CTA: three and four rows need the registers of half as many
__host__ __device__ constexpr int gv_warps(int m) { return m <= 2 ? 16 : 8; }

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xFFFF0000u); }

// grid: rows dealt to CTAs in contiguous runs. ks: warps per row (power of two), passes: chunks of a warp.
constexpr int kGvNormMax = 8192;   // width of the normed row: 16 values per thread

enum { kGvPlain = 0, kGvNorm = 1, kGvUp = 2, kGvDown = 3 };

template <int M, int MODE, int W>
__global__ void __launch_bounds__(W * 32, 1)
dense_gemv_kernel(const __nv_bfloat16 *__restrict__ w, const __nv_bfloat16 *__restrict__ x, const float *__restrict__ bias, void *__restrict__ y,
                  int N, int K, int ks, int chunk, int passes, int y_dt, int *status, const GemvNorm nrm, int pair_act, int y_ld, const GemvExperts ex, int stages) {
    constexpr bool NORM = MODE == kGvNorm, PAIRS = MODE == kGvNorm || MODE == kGvUp;
    constexpr int kGvWarps = W, kGvMaxStages = kGvTiles / kGvWarps;
    extern __shared__ __align__(128) uint8_t gv_smem[];
    __shared__ __align__(8) uint64_t bars[kGvWarps * kGvMaxStages];
    const int ring_bytes = kGvWarps * stages * kGvTileBytes;
    float *part = reinterpret_cast<float *>(gv_smem + ring_bytes);   // [rows of this CTA][ks][M]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = PAIRS && pair_act ? 2 : 1;   // rows that stay together
    const int r0 = (int)((long long)(N / unit) * blockIdx.x / gridDim.x) * unit, r1 = (int)((long long)(N / unit) * (blockIdx.x + 1) / gridDim.x) * unit;
    const int groups = kGvWarps / ks, group = warp / ks, kw = warp % ks;
    const int rows = r1 - r0 > group ? (r1 - r0 - group + groups - 1) / groups : 0;   // rows r0 + group, + groups, ...
    const uint32_t bar0 = smem_u32(bars + warp * kGvMaxStages);
    const uint32_t ring = smem_u32(gv_smem) + warp * stages * kGvTileBytes;
    const uint8_t *ring_p = gv_smem + warp * stages * kGvTileBytes;
    if (lane == 0) {
        for (int s = 0; s < stages; s++) mbar_init(bar0 + 8 * s, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    // the columns are `segs` segments of K (one expert each, or a single one), a segment is seg_chunks chunks.
    // tile i of this warp: pass i / rows, row r0 + group + groups * (i % rows); a chunk past the end has no tiles
    __shared__ int slot_e[kMaxTopK];
    __shared__ float slot_w[kMaxTopK];
    const int segs = MODE == kGvDown ? ex.top : 1, seg_chunks = (K + chunk - 1) / chunk;
    const int my_passes = max(0, min(passes, (segs * seg_chunks - kw + ks - 1) / ks));
    const int tiles = rows * my_passes;
    auto issue = [&](int i, int st) {   // lane 0; st = i % stages
        const int pass = i / rows, row = r0 + group + groups * (i - pass * rows);
        const int q = pass * ks + kw, seg = MODE == kGvDown ? q / seg_chunks : 0;
        const int k0 = (q - seg * seg_chunks) * chunk, kc = min(chunk, K - k0);
        size_t wrow = row;
        if constexpr (MODE == kGvDown) wrow += (size_t)slot_e[seg] * N;
        if constexpr (MODE == kGvUp) {
            const int per = N / ex.top, s = row / per;   // rows of an expert, slot
            wrow += ((size_t)slot_e[s] - s) * per;
        }
        const uint32_t bar = bar0 + 8 * st;
        mbar_expect_tx(bar, kc * 2);
        bulk_g2s(ring + st * kGvTileBytes, w + wrow * K + k0, kc * 2, bar);
    };
    auto route = [&]() {   // every CTA for itself
        if (warp == 0) {
            route_token(ex.logits, ex.experts, ex.top, 0, slot_e, slot_w, lane);
        }
        __syncthreads();
    };
    if constexpr (MODE == kGvDown) route();   // the logits are older than the kernel in front
    if (MODE != kGvUp && lane == 0)
        for (int i = 0; i < stages && i < tiles; i++) issue(i, i);
    NormRow row;
    if constexpr (NORM) {
        row.post_w = nrm.post_w;
        row.post_b = nrm.post_b;
        row.in = nrm.in;
        row.hidden = nrm.hidden;
        norm_prefetch<4>(row);
    }
    pdl_prologue();
    pdl_release();   // (the whole grid is resident; the mixer behind it asks for its caches while this kernel streams)
    const __nv_bfloat16 *xrow = x;
    if constexpr (MODE == kGvUp) {
        route();
        if (lane == 0)
            for (int i = 0; i < stages && i < tiles; i++) issue(i, i);
    }
    if constexpr (NORM) {
        __shared__ float red[32];
        __nv_bfloat16 *xn = reinterpret_cast<__nv_bfloat16 *>(gv_smem + ring_bytes + nrm.xn_at);
        row.h_in = nrm.h_in;
        row.delta = nrm.delta;
        row.h_out = blockIdx.x == 0 ? nrm.h_out : nullptr;
        row.e0 = row.e1 = nullptr;
        if (nrm.embed) {
            const int tok = nrm.state[0];
            row.e0 = nrm.embed + (size_t)tok * nrm.embed_ld;
            if (nrm.pairs.table) row.e1 = nrm.pairs.table + pair_row(nrm.pairs, nrm.state[4], tok, nrm.state[1]) * nrm.embed_ld;
        }
        row.alpha = nrm.alpha;
        row.eps = nrm.eps;
        float4 h[4];
        norm_units(row, h, red);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int d = 4 * (threadIdx.x + kGvWarps * 32 * i);
            if (d >= K) continue;   // columns from hidden on are zero
            const __nv_bfloat162 a = __floats2bfloat162_rn(h[i].x, h[i].y), b = __floats2bfloat162_rn(h[i].z, h[i].w);
            const uint2 u = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
            *reinterpret_cast<uint2 *>(xn + d) = u;
            if (nrm.xn_out && blockIdx.x == 0) *reinterpret_cast<uint2 *>(nrm.xn_out + d) = u;
        }
        __syncthreads();
        xrow = xn;
    }
    bool ok = true;
    int stage = 0, issued = min(tiles, stages);
    uint32_t phase = 0;
    for (int pass = 0, i = 0; pass < my_passes && ok; pass++) {
        const int q = pass * ks + kw, seg = MODE == kGvDown ? q / seg_chunks : 0;
        const int k0 = (q - seg * seg_chunks) * chunk, kc = min(chunk, K - k0), x0 = seg * K + k0;
        uint4 xv[M][4];
#pragma unroll
        for (int m = 0; m < M; m++)
#pragma unroll
            for (int j = 0; j < 4; j++)
                xv[m][j] = 8 * (lane + 32 * j) < kc ? *reinterpret_cast<const uint4 *>(xrow + (size_t)m * K + x0 + 8 * (lane + 32 * j)) : make_uint4(0, 0, 0, 0);
        for (int r = 0; r < rows; r++, i++) {
            if (!mbar_wait_fast(bar0 + 8 * stage, phase)) {
                ok = false;
                break;
            }
            const uint4 *tile = reinterpret_cast<const uint4 *>(ring_p + stage * kGvTileBytes);
            float acc[M][2];
#pragma unroll
            for (int m = 0; m < M; m++) acc[m][0] = acc[m][1] = 0.0f;
            uint4 wv[4];
#pragma unroll
            for (int j = 0; j < 4; j++) wv[j] = 8 * (lane + 32 * j) < kc ? tile[lane + 32 * j] : make_uint4(0, 0, 0, 0);
            __syncwarp();
            if (lane == 0 && issued < tiles) issue(issued, stage);   // the tile's values are in registers
            issued++;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const uint32_t wq[4] = {wv[j].x, wv[j].y, wv[j].z, wv[j].w};
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    const float wl = bf_lo(wq[q]), wh = bf_hi(wq[q]);
#pragma unroll
                    for (int m = 0; m < M; m++) {
                        const uint32_t xq = q == 0 ? xv[m][j].x : (q == 1 ? xv[m][j].y : (q == 2 ? xv[m][j].z : xv[m][j].w));
                        acc[m][0] = fmaf(wl, bf_lo(xq), acc[m][0]);
                        acc[m][1] = fmaf(wh, bf_hi(xq), acc[m][1]);
                    }
                }
            }
#pragma unroll
            for (int m = 0; m < M; m++) {
                float v = acc[m][0] + acc[m][1];
#pragma unroll
                for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, off);
                if (lane == 0) {
                    float *p = part + ((size_t)(group + groups * r) * ks + kw) * M + m;
                    *p = pass == 0 ? v : *p + v;
                }
            }
            if (++stage == stages) {
                stage = 0;
                phase ^= 1u;
            }
        }
    }
    if (my_passes == 0)   // fewer chunks than warps per row
        for (int r = lane; r < rows; r += 32)
#pragma unroll
            for (int m = 0; m < M; m++) part[((size_t)(group + groups * r) * ks + kw) * M + m] = 0.0f;
    if (!ok) {
        // give the copies in flight a bounded chance to land before the shared memory goes
        for (int s = 0; s < stages; s++) mbar_wait(bar0 + 8 * s, phase);
        if (lane == 0) atomicExch(status, 1);
    }
    __syncthreads();
    if (PAIRS && pair_act) {
        __nv_bfloat16 *out = reinterpret_cast<__nv_bfloat16 *>(y);
        for (int i = threadIdx.x; i < (r1 - r0) / 2; i += kGvWarps * 32) {
            float g = 0.0f, u = 0.0f;
            for (int q = 0; q < ks; q++) {
                g += part[(size_t)(2 * i) * ks + q];
                u += part[(size_t)(2 * i + 1) * ks + q];
            }
            float v = gate_act(pair_act - 1, g) * u;
            if constexpr (MODE == kGvUp) v *= slot_w[(r0 + 2 * i) / (N / ex.top)];
            out[r0 / 2 + i] = __float2bfloat16_rn(v);
        }
        if (MODE == kGvNorm && blockIdx.x == 0)
            for (int i = N / 2 + threadIdx.x; i < y_ld; i += kGvWarps * 32) out[i] = __float2bfloat16_rn(0.0f);
        return;
    }
    for (int i = threadIdx.x; i < (r1 - r0) * M; i += kGvWarps * 32) {
        const int m = i / (r1 - r0), r = i - m * (r1 - r0);
        float v = 0.0f;
        for (int q = 0; q < ks; q++) v += part[((size_t)r * ks + q) * M + m];
        if (bias) v += __ldg(bias + r0 + r);
        if (y_dt == NNQ_F32) reinterpret_cast<float *>(y)[(size_t)m * N + r0 + r] = v;
        else reinterpret_cast<__nv_bfloat16 *>(y)[(size_t)m * N + r0 + r] = __float2bfloat16_rn(v);
    }
}

bool dense_gemv_supported(const nnq_weight *w, int64_t m, int x_dt) {
    return w && w->fmt == NNQ_BF16_DENSE && w->d_raw && x_dt == NNQ_BF16 && m >= 1 && m <= 4 && w->k >= 64 && w->k % 8 == 0 && w->n >= 1 &&
           w->n < (1ll << 31) && w->k < (1ll << 31) && !((uintptr_t)w->d_raw & 15u);
}

template <int M, int MODE, int W>
static cudaError_t gv_go(const TcArgs &a, int grid, int ks, int chunk, int passes, size_t smem, int *status, const GemvNorm &nrm, int pair_act, int y_ld, cudaStream_t st,
                         int stages, const GemvExperts &ex = {}) {
    cudaError_t e = cudaFuncSetAttribute(dense_gemv_kernel<M, MODE, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    launch_pdl_smem(dense_gemv_kernel<M, MODE, W>, dim3(grid), dim3(W * 32), smem, st, reinterpret_cast<const __nv_bfloat16 *>(a.w),
                    reinterpret_cast<const __nv_bfloat16 *>(a.x), a.bias, a.y, (int)a.n, (int)a.k, ks, chunk, passes, a.y_dt, status, nrm, pair_act, y_ld, ex, stages);
    return cudaGetLastError();
}

bool dense_gemv_norm_supported(const nnq_weight *w, int hidden) {
    return dense_gemv_supported(w, 1, NNQ_BF16) && hidden % 4 == 0 && hidden <= w->k && w->k <= kGvNormMax;
}

static nnq_status gemv(nnq_ctx *ctx, const TcArgs &a, GemvNorm *nrm, int pair_act, int y_ld, cudaStream_t stream) {
    // as few warps per row as keep a warp's columns within one chunk
    const bool half = nrm && nrm->half && a.k <= kGvNormMax / 2;
    const int warps = half ? 8 : gv_warps((int)a.m);
    int ks = 1;
    while (ks < warps && a.k > (int64_t)ks * kGvChunk) ks *= 2;
    int chunk = (int)(((a.k + ks - 1) / ks + 7) / 8 * 8);
    if (chunk > kGvChunk) chunk = kGvChunk;
    const int chunks = (int)((a.k + chunk - 1) / chunk), passes = (chunks + ks - 1) / ks;
    // partial sums of a CTA's rows within 32 KB: more CTAs than SMs for very tall weights
    const int64_t max_rows = (32 << 10) / (4 * ks * a.m);
    const int64_t units = pair_act ? a.n / 2 : a.n, per_unit = pair_act ? 2 : 1;   // runs of rows that stay together
    int64_t grid = units < ctx->sm_count ? units : ctx->sm_count;
    while ((units + grid - 1) / grid * per_unit > max_rows) grid += ctx->sm_count;
    const int stages = half ? kGvTiles / 16 : kGvTiles / warps;
    const size_t ring = (size_t)warps * stages * kGvTileBytes;
    size_t smem = ring + ((size_t)((units + grid - 1) / grid * per_unit) * ks * a.m * 4 + 15) / 16 * 16;
    cudaError_t e;
    const GemvNorm none = {};
    if (nrm) {
        nrm->xn_at = (int)(smem - ring);
        smem += (size_t)a.k * 2;
        e = half ? gv_go<1, kGvNorm, 8>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, *nrm, pair_act, y_ld, stream, stages)
                 : gv_go<1, kGvNorm, 16>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, *nrm, pair_act, y_ld, stream, stages);
    } else {
        switch (a.m) {
            case 1: e = gv_go<1, kGvPlain, 16>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 0, 0, stream, stages); break;
            case 2: e = gv_go<2, kGvPlain, 16>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 0, 0, stream, stages); break;
            case 3: e = gv_go<3, kGvPlain, 8>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 0, 0, stream, stages); break;
            case 4: e = gv_go<4, kGvPlain, 8>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 0, 0, stream, stages); break;
            default: return fail(ctx, NNQ_ERR_UNSUPPORTED, "1 to 4 rows");
        }
    }
    ctx->launches++;
    return check_cuda(ctx, e, "bf16 row product launch");
}

nnq_status launch_dense_gemv_experts(nnq_ctx *ctx, const GemvExperts &g, bool up, cudaStream_t stream) {
    const int64_t n = up ? 2ll * g.inter * g.top : g.hidden, k = up ? g.hidden : g.inter;
    if (g.top < 1 || g.top > kMaxTopK || g.experts < g.top || g.experts > kMaxExperts || k % 8 || k < 8) return fail(ctx, NNQ_ERR_UNSUPPORTED, "bad expert product");
    // chunks of a segment alike, as few warps per row as there are chunks
    const int segs = up ? 1 : g.top, seg_chunks = (int)((k + kGvChunk - 1) / kGvChunk), chunk = (int)((k + seg_chunks - 1) / seg_chunks + 7) / 8 * 8;
    int ks = 1;
    while (ks < gv_warps(1) && ks < segs * seg_chunks) ks *= 2;
    const int passes = (segs * seg_chunks + ks - 1) / ks, per_unit = up ? 2 : 1;
    const int64_t units = n / per_unit, max_rows = (32 << 10) / (4 * ks);
    int64_t grid = units < ctx->sm_count ? units : ctx->sm_count;
    while ((units + grid - 1) / grid * per_unit > max_rows) grid += ctx->sm_count;
    const int stages = kGvTiles / gv_warps(1);
    const size_t smem = kGvRing + ((size_t)((units + grid - 1) / grid * per_unit) * ks * 4 + 15) / 16 * 16;
    const TcArgs a = {(const uint8_t *)g.w, nullptr, g.x, nullptr, g.y, 1, n, k, NNQ_BF16_DENSE, NNQ_BF16, up ? NNQ_BF16 : NNQ_F32};
    const GemvNorm none = {};
    const cudaError_t e = up ? gv_go<1, kGvUp, 16>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 1 + NNQ_ACT_SILU, 0, stream, stages, g)
                             : gv_go<1, kGvDown, 16>(a, (int)grid, ks, chunk, passes, smem, ctx->d_status, none, 0, 0, stream, stages, g);
    ctx->launches++;
    return check_cuda(ctx, e, "expert row product launch");
}

nnq_status launch_dense_gemv(nnq_ctx *ctx, const TcArgs &a, cudaStream_t stream) { return gemv(ctx, a, nullptr, 0, 0, stream); }

nnq_status launch_dense_gemv_norm(nnq_ctx *ctx, const TcArgs &a, const GemvNorm &norm, int pair_act, int y_ld, cudaStream_t stream) {
    GemvNorm n = norm;
    return gemv(ctx, a, &n, pair_act, y_ld, stream);
}

}  // namespace nnq
