// Attention through a latent for a block of rows on the 5th-generation tensor cores (bf16 decoders): per head, keys
// [W_uk,h c | r] with the rotated part r shared by the heads, values W_uv,h c, over a sliding window.
//
// Queries (rotated in f32 here), keys and values are bf16; scores, softmax, weights and sums are f32: the weights
// enter the second product as two bf16 terms (p = hi + lo, remainder below 2^-16 of p), accumulation is f32.
//
// One CTA: 128 query rows of one head, key tiles of KT = 128 (64 where the pieces are many) over the union of the rows'
// windows.
//   warps 0-7: stage the queries, then softmax. Two threads share a row, one per half of a tile's keys (they exchange
//              their maxima) and of the value dimensions: scores of tile t from tensor memory, maximum, sum, weights back
//              into the columns the scores were in; then the weighted values of tile t - 1 from tensor memory into f32
//              accumulators.
//   warp 8:    one thread issues the TMA loads: key tiles (64-wide pieces of the head's part, then the shared part) and
//              value tiles, two stages each, the first ones before the queries are staged.
//   warp 9:    one thread issues the MMAs: S(t + 2) = Q K^T behind O(t) = P V, with P as the operand in tensor memory and
//              the values as the MN-major operand, so that their tiles stay as they lie in memory.
// Scores and weighted values have two buffers each, so the tensor cores work on tile t while the softmax warps are at
// t + 1. The barrier of S(t) also frees the key stage, that of O(t) the value stage. Every wait is bounded.
#include <cuda.h>
#include <math.h>
#include <string.h>

#include "blocks.cuh"
#include "sync.cuh"
#include "tcgen05.cuh"

namespace nnq {

constexpr int kLtRows = 128, kLtSoft = 256, kLtThreads = kLtSoft + 64;
constexpr int kLtQAtom = kLtRows * 128;   // bytes of 128 rows of 64 columns (one swizzle row)
constexpr int kLtMaxAtoms = 4;            // 64-wide pieces of a key

static int lt_smem_bytes(int kt, int atoms, int nv) { return atoms * kLtQAtom + 2 * (atoms + nv) * kt * 128; }

__device__ __forceinline__ void lt_tma_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(dst), "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(bar) : "memory");
}

// MN-major, 128-byte swizzle: 64 columns (128 bytes) by 8 k rows per 1024 bytes, k groups 1024 bytes apart, the next 64
// columns `next` bytes on
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t next) {
    const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((next >> 4) << 16);
    const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
    return ((uint64_t)hi << 32) | lo;
}

// D += A B^T with A in tensor memory (row = lane, a column holds two neighbouring bf16 of k)
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
        " tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n}"
        ::"r"(tmem_d), "r"(tmem_a), "l"(db), "r"(idesc), "r"(accumulate) : "memory");
}

__device__ __forceinline__ void tmem_st16(uint32_t addr, const uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15};"
        ::"r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]),
          "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(addr) : "memory");
}

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// the rotated dimensions j .. j + 3 of a query row (q: where they start); rot a multiple of 8: groups of four stay in one half
__device__ __forceinline__ float4 lt_rotated4(const float *q, int j, int rot, const float *cs, const float *sn) {
    const int half = rot >> 1;
    const bool second = j >= half;
    const int i = second ? j - half : j;
    const float4 x = *reinterpret_cast<const float4 *>(q + j), y = *reinterpret_cast<const float4 *>(q + (second ? j - half : j + half));
    const float4 c = *reinterpret_cast<const float4 *>(cs + i), s = *reinterpret_cast<const float4 *>(sn + i);
    const float g = second ? 1.0f : -1.0f;
    return make_float4(fmaf(x.x, c.x, g * y.x * s.x), fmaf(x.y, c.y, g * y.y * s.y), fmaf(x.z, c.z, g * y.z * s.z), fmaf(x.w, c.w, g * y.w * s.w));
}

template <int KT, int NV>
__global__ void __launch_bounds__(kLtThreads, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap kv_map, const __grid_constant__ CUtensorMap r_map, const LatentAttn a, int *status) {
    constexpr int KH = KT / 2, KAtom = KT * 128;   // keys of a softmax thread; bytes of KT rows of 64 columns
    extern __shared__ __align__(1024) uint8_t lt_smem_raw[];
    uint8_t *smem = lt_smem_raw;
    if (smem_u32(smem) & 1023u) {   // the swizzled tiles start at multiples of 1024 bytes
        if (threadIdx.x == 0) atomicExch(status, 1);
        return;
    }
    __shared__ __align__(8) uint64_t bars[11];   // k_full[2], v_full[2], s_full[2], o_full[2], p_full[2], drain
    __shared__ uint32_t tmem_s;
    __shared__ float half_max[2][2][kLtRows], half_sum[kLtRows];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t kf = smem_u32(bars), vf = kf + 16, sf = kf + 32, of = kf + 48, pf = kf + 64, drain = kf + 80;
    const int h = blockIdx.x, row0 = blockIdx.y * kLtRows, rows = min(kLtRows, a.span.n - row0);
    const int da = a.dim_ld >> 6, ra = a.rot_ld >> 6, atoms = da + ra;
    const int pos_first = a.span.pos0 + row0;                                  // position of the first row
    const int first = max(0, pos_first - a.window + 1), last = pos_first + rows - 1;   // keys some row sees
    const int tiles = (last - first) / KT + 1, key0 = first - a.first;    // key0: row of the expanded keys
    uint8_t *q_s = smem, *k_s = q_s + atoms * kLtQAtom, *v_s = k_s + 2 * atoms * KAtom;

    auto load_k = [&](int t) {
        const uint32_t bar = kf + 8 * (t & 1);
        mbar_expect_tx(bar, atoms * KAtom);
        for (int at = 0; at < atoms; at++) {
            const uint32_t dst = smem_u32(k_s + ((t & 1) * atoms + at) * KAtom);
            if (at < da) lt_tma_2d(dst, &kv_map, h * a.dim_ld + 64 * at, key0 + t * KT, bar);
            else lt_tma_2d(dst, &r_map, 64 * (at - da), key0 + t * KT, bar);
        }
    };
    auto load_v = [&](int t) {
        const uint32_t bar = vf + 8 * (t & 1);
        mbar_expect_tx(bar, NV * KAtom);
        for (int v = 0; v < NV; v++)
            lt_tma_2d(smem_u32(v_s + ((t & 1) * NV + v) * KAtom), &kv_map, a.heads * a.dim_ld + h * a.vdim_ld + 64 * v, key0 + t * KT, bar);
    };
    if (tid == kLtSoft) {   // the loader
        for (int i = 0; i < 8; i++) mbar_init(kf + 8 * i, 1);
        for (int i = 0; i < 2; i++) mbar_init(pf + 8 * i, kLtSoft);
        mbar_init(drain, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        for (int t = 0; t < 2 && t < tiles; t++) {
            load_k(t);
            load_v(t);
        }
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_s)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    // the queries, piece by piece (the rotated part starts a piece of its own): sixteen lanes take the 64 columns of a row,
    // a batch of rows is under way before the first is used
    if (warp < 8) {
        constexpr int QB = 8, step = 16;
        const int e = 4 * (lane & 15), dk = a.dim + a.rot, half = a.rot >> 1, r0 = 2 * warp + (lane >> 4);
        const bool vec = ((a.dim & 3) | (a.rot & 7)) == 0;
        const float *qh = a.q + ((size_t)row0 * a.heads + h) * dk;
        const size_t ld = (size_t)a.heads * dk;
        for (int at = 0; at < atoms; at++) {
            const bool turn = at >= da;
            const int j = turn ? 64 * (at - da) + e : 64 * at + e, width = turn ? a.rot : a.dim;   // column of its part
            float4 v[QB];
#pragma unroll
            for (int i = 0; i < QB; i++) {
                const int r = r0 + i * step;
                v[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (r >= rows || j >= width) continue;
                const float *q = qh + r * ld + (turn ? a.dim : 0);
                const float *cs = a.cosv + (size_t)(pos_first + r) * half, *sn = a.sinv + (size_t)(pos_first + r) * half;
                if (vec) {
                    v[i] = turn ? lt_rotated4(q, j, a.rot, cs, sn) : *reinterpret_cast<const float4 *>(q + j);
                } else {
                    float x[4];
#pragma unroll
                    for (int k = 0; k < 4; k++) x[k] = j + k >= width ? 0.0f : (turn ? rotated(q, j + k, a.rot, cs, sn) : q[j + k]);
                    v[i] = make_float4(x[0], x[1], x[2], x[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < QB; i++)
                *reinterpret_cast<uint2 *>(q_s + at * kLtQAtom + swz(r0 + i * step, e >> 3) + 2 * (e & 7)) = make_uint2(pack_bf16(v[i].x, v[i].y), pack_bf16(v[i].z, v[i].w));
        }
    }
    fence_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_s, o_tmem = tmem + 2 * KT;   // scores: two of KT columns, weighted values: two of 64 NV
    bool ok = true;

    if (warp < 8) {
        // ---------------- softmax ----------------
        const int row = tid & 127, half = tid >> 7;                        // half: keys KH half .. of a tile, value dimensions 32 NV half ..
        const int my_hi = pos_first + row, my_lo = my_hi - a.window + 1;   // keys this row sees (rows past the end are not stored)
        const float c = a.scale * 1.4426950408889634f;
        const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
        float acc[NV * 32];
#pragma unroll
        for (int i = 0; i < NV * 32; i++) acc[i] = 0.0f;
        float m = -INFINITY, l = 0.0f, corr = 1.0f;
        auto add_values = [&](int t) {   // weighted values of tile t, weights relative to the maximum after tile t
            ok = ok && __all_sync(0xFFFFFFFFu, mbar_wait_fast(of + 8 * (t & 1), (t >> 1) & 1));   // (a warp agrees)
            if (!ok) return;
            tc_fence_after();
#pragma unroll
            for (int b = 0; b < NV; b++) {
                uint32_t v[32];
                tmem_ld32(o_tmem + (t & 1) * NV * 64 + half * NV * 32 + lane_base + b * 32, v);
#pragma unroll
                for (int i = 0; i < 32; i++) acc[b * 32 + i] = fmaf(acc[b * 32 + i], corr, __uint_as_float(v[i]));
            }
        };
        // every warp comes to the barrier of every tile, also after a wait that ran out (then without waiting again)
        for (int t = 0; t < tiles; t++) {
            ok = ok && __all_sync(0xFFFFFFFFu, mbar_wait_fast(sf + 8 * (t & 1), (t >> 1) & 1));
            uint32_t s[KH / 32][32];
            float mt = -INFINITY;
            const uint32_t s_tmem = tmem + (t & 1) * KT + lane_base;
            if (ok) {
                tc_fence_after();
                const int k0 = first + t * KT + KH * half;
                const int lo = my_lo - k0, hi = my_hi - k0;   // visible keys of this half
#pragma unroll
                for (int b = 0; b < KH / 32; b++) tmem_ld32(s_tmem + KH * half + 32 * b, s[b]);
                if (__all_sync(0xFFFFFFFFu, lo <= 0 && hi >= KH - 1)) {
#pragma unroll
                    for (int i = 0; i < KH; i++) mt = fmaxf(mt, __uint_as_float(s[i >> 5][i & 31]));
                } else {
#pragma unroll
                    for (int i = 0; i < KH; i++) {
                        const float x = i >= lo && i <= hi ? __uint_as_float(s[i >> 5][i & 31]) : -INFINITY;
                        s[i >> 5][i & 31] = __float_as_uint(x);
                        mt = fmaxf(mt, x);
                    }
                }
                tc_fence_before();   // (the other half's thread overwrites these columns behind the barrier)
            }
            half_max[t & 1][half][row] = mt;
            asm volatile("bar.sync 1, %0;" ::"n"(kLtSoft) : "memory");
            if (!ok) continue;
            mt = fmaxf(mt, half_max[t & 1][half ^ 1][row]);
            mt = mt == -INFINITY ? mt : mt * c;                // (c > 0)
            const float mn = fmaxf(m, mt);
            const float next = m == mn ? 1.0f : ex2(m - mn);   // no key of this row yet: both -inf
            const float base = mn == -INFINITY ? 0.0f : mn;
            float sum = 0.0f;
            tc_fence_after();
#pragma unroll
            for (int b = 0; b < KH / 32; b++) {
                uint32_t hv[16], lv[16];
#pragma unroll
                for (int e = 0; e < 16; e++) {
                    const float p0 = ex2(fmaf(__uint_as_float(s[b][2 * e]), c, -base)), p1 = ex2(fmaf(__uint_as_float(s[b][2 * e + 1]), c, -base));
                    sum += p0 + p1;
                    hv[e] = pack_bf16(p0, p1);
                    lv[e] = pack_bf16(p0 - __uint_as_float(hv[e] << 16), p1 - __uint_as_float(hv[e] & 0xFFFF0000u));
                }
                tmem_st16(s_tmem + KH / 2 * half + 16 * b, hv);            // columns of two keys: hi, then lo
                tmem_st16(s_tmem + KH + KH / 2 * half + 16 * b, lv);
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            tc_fence_before();
            mbar_arrive(pf + 8 * (t & 1));
            if (t > 0) add_values(t - 1);
            l = l * next + sum;
            m = mn;
            corr = next;   // tile t's weighted values join sums that are still relative to the maximum before it
        }
        add_values(tiles - 1);
        if (half) half_sum[row] = l;
        asm volatile("bar.sync 1, %0;" ::"n"(kLtSoft) : "memory");
        if (!half) {
            l += half_sum[row];
            half_max[0][0][row] = l;
        }
        asm volatile("bar.sync 1, %0;" ::"n"(kLtSoft) : "memory");
        if (ok && row < rows) {
            const float inv = 1.0f / half_max[0][0][row];
            const int v0 = half * NV * 32;
            __nv_bfloat16 *o = reinterpret_cast<__nv_bfloat16 *>(a.out) + (size_t)(row0 + row) * a.out_ld + h * a.vdim;
            if ((a.vdim & 7) == 0) {
#pragma unroll
                for (int d = 0; d < NV * 32; d += 8)
                    if (v0 + d < a.vdim)
                        *reinterpret_cast<uint4 *>(o + v0 + d) = make_uint4(pack_bf16(acc[d] * inv, acc[d + 1] * inv), pack_bf16(acc[d + 2] * inv, acc[d + 3] * inv),
                                                                            pack_bf16(acc[d + 4] * inv, acc[d + 5] * inv), pack_bf16(acc[d + 6] * inv, acc[d + 7] * inv));
            } else {
#pragma unroll
                for (int d = 0; d < NV * 32; d++)
                    if (v0 + d < a.vdim) o[v0 + d] = __float2bfloat16_rn(acc[d] * inv);
            }
            if (half && h == a.heads - 1)
                for (int d = a.vdim; d < a.out_ld - h * a.vdim; d++) o[d] = __float2bfloat16_rn(0.0f);
        }
    } else if (warp == 8 && lane == 0) {
        // ---------------- TMA loads ----------------
        int t = min(2, tiles);
        for (; t < tiles; t++) {
            const uint32_t parity = ((t >> 1) - 1) & 1;
            if (!mbar_wait_fast(sf + 8 * (t & 1), parity)) break;
            load_k(t);
            if (!mbar_wait_fast(of + 8 * (t & 1), parity)) {
                mbar_wait(kf + 8 * (t & 1), (t >> 1) & 1);   // the key tile just asked for
                break;
            }
            load_v(t);
        }
        ok = t == tiles;
        for (int k = t - 2; k < t; k++)   // no copy is in flight when the CTA ends
            if (k >= 0) {
                ok = mbar_wait(kf + 8 * (k & 1), (k >> 1) & 1) && ok;
                ok = mbar_wait(vf + 8 * (k & 1), (k >> 1) & 1) && ok;
            }
    } else if (warp == 9 && lane == 0) {
        // ---------------- MMA issuer ----------------
        const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(KT >> 3) << 17) | ((128u >> 4) << 24);
        const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(NV * 64 >> 3) << 17) | ((128u >> 4) << 24);   // B is MN-major
        auto scores = [&](int t) {
            if (!mbar_wait_fast(kf + 8 * (t & 1), (t >> 1) & 1)) return false;
            tc_fence_after();
            bool add = false;
            for (int at = 0; at < atoms; at++) {
                const uint64_t dq = smem_desc(smem_u32(q_s + at * kLtQAtom)), dk = smem_desc(smem_u32(k_s + ((t & 1) * atoms + at) * KAtom));
                const int width = at < da ? min(64, a.dim - 64 * at) : min(64, a.rot - 64 * (at - da));
                for (int k = 0; k < (width + 15) >> 4; k++) {
                    umma_bf16(tmem + (t & 1) * KT, dq + 2 * k, dk + 2 * k, id_s, add);
                    add = true;
                }
            }
            umma_commit(sf + 8 * (t & 1));
            return true;
        };
        ok = scores(0) && (tiles < 2 || scores(1));
        for (int t = 0; t < tiles && ok; t++) {
            if (!mbar_wait_fast(pf + 8 * (t & 1), (t >> 1) & 1) || !mbar_wait_fast(vf + 8 * (t & 1), (t >> 1) & 1)) {
                ok = false;
                break;
            }
            tc_fence_after();
            const uint32_t p = tmem + (t & 1) * KT, o = o_tmem + (t & 1) * NV * 64;
            const uint64_t dv = smem_desc_mn(smem_u32(v_s + (t & 1) * NV * KAtom), KAtom);
#pragma unroll
            for (int x = 0; x < 2; x++)   // hi, lo
#pragma unroll
                for (int k = 0; k < KT / 16; k++) umma_bf16_ts(o, p + x * KH + 8 * k, dv + (2048 >> 4) * k, id_o, (x | k) != 0);
            umma_commit(of + 8 * (t & 1));
            // S(t + 2) overwrites the weights that O(t) reads
            if (t + 2 < tiles) ok = mbar_wait_fast(of + 8 * (t & 1), (t >> 1) & 1) && scores(t + 2);
        }
        if (!ok) {   // MMAs that were issued may still read shared memory and write tensor memory: one more bounded wait
            umma_commit(drain);
            mbar_wait(drain, 0);
        }
    }
    if (!ok) atomicExch(status, 1);
    tc_fence_before();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u) : "memory");
    }
}

// ---- host side ----

typedef CUresult (*LtEncodeFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *,
                               const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

static LtEncodeFn lt_encode_fn() {
    static LtEncodeFn fn = nullptr;
    static bool tried = false;
    if (!tried) {
        tried = true;
        void *p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
            fn = reinterpret_cast<LtEncodeFn>(p);
        cudaGetLastError();
    }
    return fn;
}

// bf16 [rows, cols] row-major (cols a multiple of 64) -> boxes of 64 columns, 128-byte swizzle, zero fill outside
static bool lt_map(const void *base, int64_t rows, int64_t cols, int box_rows, CUtensorMap *map) {
    LtEncodeFn fn = lt_encode_fn();
    memset(map, 0, sizeof(*map));
    if (!fn || ((uintptr_t)base & 15u) || cols % 64) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t)box_rows}, one[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// bf16 decoders, keys of at most four 64-wide pieces (head part and shared part each rounded up), values of two
bool latent_tc_supported(int act_dt, int dim, int rot, int vdim) {
    return act_dt == NNQ_BF16 && (dim + 63) / 64 + (rot + 63) / 64 <= kLtMaxAtoms && vdim <= 128 && lt_encode_fn() != nullptr;
}

template <int KT, int NV>
static nnq_status lt_go(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) {
    CUtensorMap kv_map, r_map;
    if (!lt_map(a.kv, a.keys, (int64_t)a.heads * (a.dim_ld + a.vdim_ld), KT, &kv_map) || (a.rot_ld && !lt_map(a.lin_r, a.keys, a.rot_ld, KT, &r_map)))
        return fail(ctx, NNQ_ERR_DISPATCH_FAILED, "tensor map creation failed");
    if (!a.rot_ld) r_map = kv_map;   // not read
    const int smem = lt_smem_bytes(KT, (a.dim_ld + a.rot_ld) / 64, NV);
    nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(attn_latent_tc_kernel<KT, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "latent attention shared memory");
    if (s != NNQ_OK) return s;
    attn_latent_tc_kernel<KT, NV><<<dim3(a.heads, (a.span.n + kLtRows - 1) / kLtRows), kLtThreads, smem, st>>>(kv_map, r_map, a, ctx->d_status);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "latent attention launch");
}

nnq_status launch_latent_tc(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) {
    const bool wide = lt_smem_bytes(128, (a.dim_ld + a.rot_ld) / 64, a.vdim_ld / 64) <= 216 * 1024;
    if (a.vdim_ld > 64) return wide ? lt_go<128, 2>(ctx, a, st) : lt_go<64, 2>(ctx, a, st);
    return wide ? lt_go<128, 1>(ctx, a, st) : lt_go<64, 1>(ctx, a, st);
}

}  // namespace nnq
