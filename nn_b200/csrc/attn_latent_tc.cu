// Attention through a latent for a block of rows on the 5th-generation tensor cores (bf16 decoders): per head, keys
// [W_uk,h c | r] with the rotated part r shared by the heads, values W_uv,h c, over a sliding window.
//
// Queries (rotated in f32 here), keys and values are bf16; scores, softmax, weights and sums are f32: the weights
// enter the second product as two bf16 terms (p = hi + lo, remainder below 2^-16 of p), accumulation is f32.
//
// One CTA: 128 query rows of one head, key tiles of 64 over the union of the rows' windows.
//   warps 0-7: softmax. Two threads share a row, one per half of a tile's keys (they exchange their maxima) and of the
//              value dimensions: scores of tile t from tensor memory, maximum, sum, weights as two swizzled tiles; then
//              the weighted values of tile t - 1 from tensor memory into f32 accumulators.
//   warp 8:    one thread issues the TMA loads: key tiles (64-wide pieces of the head's part, then the shared part) and
//              value tiles, two stages each.
//   warp 9:    one thread issues the MMAs: S(t + 2) = Q K^T right behind O(t) = P V. Values are the MN-major operand,
//              so their tiles stay as they lie in memory.
// Scores, weights and weighted values have two buffers each, so the tensor cores work on tile t while the softmax
// warps are at t + 1. The barrier of S(t) also frees the key stage, that of O(t) the value stage. Every wait is bounded.
#include <cuda.h>
#include <math.h>
#include <string.h>

#include "blocks.cuh"
#include "sync.cuh"
#include "tcgen05.cuh"

namespace nnq {

constexpr int kLtKeys = 64, kLtRows = 128, kLtSoft = 256, kLtThreads = kLtSoft + 64;
constexpr int kLtQAtom = kLtRows * 128, kLtKAtom = kLtKeys * 128;   // bytes of a tile of 64 columns (one swizzle row)
constexpr int kLtMaxAtoms = 4;                                      // 64-wide pieces of a key

// (the largest case, four pieces and two value pieces, takes all there is beside the static part)
static int lt_smem_bytes(int atoms, int nv) { return atoms * kLtQAtom + 2 * (atoms + nv) * kLtKAtom + 4 * kLtQAtom; }

__device__ __forceinline__ void lt_tma_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(dst), "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(bar) : "memory");
}

// MN-major, 128-byte swizzle: 64 columns (128 bytes) by 8 k rows per 1024 bytes, k groups 1024 bytes apart, the next 64
// columns kLtKAtom bytes on
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr) {
    const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((uint32_t)(kLtKAtom >> 4) << 16);
    const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
    return ((uint64_t)hi << 32) | lo;
}

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// four dimensions d .. d + 3 of a query row: unrotated up to dim, then rotated
__device__ __forceinline__ float4 lt_query4(const LatentAttn &a, const float *q, int d, int pos) {
    float v[4];
    if (d + 4 <= a.dim && ((a.dim | a.rot) & 3) == 0) return *reinterpret_cast<const float4 *>(q + d);
    const int half = a.rot >> 1, j = d - a.dim;
    if (j >= 0 && (a.rot & 7) == 0 && (a.dim & 3) == 0) {   // four dimensions of one half
        if (j >= a.rot) return make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const bool second = j >= half;
        const int i = second ? j - half : j;
        const float4 x = *reinterpret_cast<const float4 *>(q + d), y = *reinterpret_cast<const float4 *>(q + (second ? d - half : d + half));
        const float4 c = *reinterpret_cast<const float4 *>(a.cosv + (size_t)pos * half + i);
        float4 s = *reinterpret_cast<const float4 *>(a.sinv + (size_t)pos * half + i);
        if (!second) s = make_float4(-s.x, -s.y, -s.z, -s.w);
        return make_float4(x.x * c.x + y.x * s.x, x.y * c.y + y.y * s.y, x.z * c.z + y.z * s.z, x.w * c.w + y.w * s.w);
    }
#pragma unroll
    for (int e = 0; e < 4; e++) {
        const int k = d + e;
        v[e] = k < a.dim ? q[k] : (k < a.dim + a.rot ? rotated(q + a.dim, k - a.dim, a.rot, a.cosv + (size_t)pos * half, a.sinv + (size_t)pos * half) : 0.0f);
    }
    return make_float4(v[0], v[1], v[2], v[3]);
}

template <int NV>
__global__ void __launch_bounds__(kLtThreads, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap kv_map, const __grid_constant__ CUtensorMap r_map, const LatentAttn a, int *status) {
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
    const int tiles = (last - first) / kLtKeys + 1, key0 = first - a.first;    // key0: row of the expanded keys
    uint8_t *q_s = smem, *k_s = q_s + atoms * kLtQAtom, *v_s = k_s + 2 * atoms * kLtKAtom, *p_s = v_s + 2 * NV * kLtKAtom;

    if (tid == 0) {
        for (int i = 0; i < 8; i++) mbar_init(kf + 8 * i, 1);
        for (int i = 0; i < 2; i++) mbar_init(pf + 8 * i, kLtSoft);
        mbar_init(drain, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_s)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    // the queries; a piece ends where the unrotated part ends, so the rotated part starts a piece of its own. A batch of
    // loads is under way before the first is used.
    constexpr int QB = 6;
    for (int u0 = tid; u0 < kLtRows * 16 * atoms; u0 += QB * kLtThreads) {
        float4 v[QB];
#pragma unroll
        for (int i = 0; i < QB; i++) {
            const int u = u0 + i * kLtThreads, r = u / (16 * atoms), c = u - r * 16 * atoms, at = c >> 4, e = 4 * (c & 15);
            v[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (r >= rows) continue;
            const int d = at < da ? 64 * at + e : a.dim + 64 * (at - da) + e;
            const float *q = a.q + ((size_t)(row0 + r) * a.heads + h) * (a.dim + a.rot);
            if (at >= da) {
                v[i] = lt_query4(a, q, d, pos_first + r);
            } else if (d < a.dim) {
                if (d + 4 <= a.dim && ((a.dim | a.rot) & 3) == 0) v[i] = *reinterpret_cast<const float4 *>(q + d);
                else v[i] = make_float4(q[d], d + 1 < a.dim ? q[d + 1] : 0.0f, d + 2 < a.dim ? q[d + 2] : 0.0f, d + 3 < a.dim ? q[d + 3] : 0.0f);
            }
        }
#pragma unroll
        for (int i = 0; i < QB; i++) {
            const int u = u0 + i * kLtThreads, r = u / (16 * atoms), c = u - r * 16 * atoms, at = c >> 4, e = 4 * (c & 15);
            if (r < kLtRows)
                *reinterpret_cast<uint2 *>(q_s + at * kLtQAtom + swz(r, e >> 3) + 2 * (e & 7)) = make_uint2(pack_bf16(v[i].x, v[i].y), pack_bf16(v[i].z, v[i].w));
        }
    }
    fence_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_s, o_tmem = tmem + 128;   // scores: two of 64 columns, weighted values: two of 64 NV
    bool ok = true;

    if (warp < 8) {
        // ---------------- softmax ----------------
        const int row = tid & 127, half = tid >> 7;                        // half: keys 32 half .. + 31 of a tile, value dimensions 32 NV half ..
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
            uint32_t s[32];
            float mt = -INFINITY;
            if (ok) {
                tc_fence_after();
                const int k0 = first + t * kLtKeys + 32 * half;
                const int lo = my_lo - k0, hi = my_hi - k0;   // visible keys of this half
                tmem_ld32(tmem + (t & 1) * 64 + 32 * half + lane_base, s);
                if (__all_sync(0xFFFFFFFFu, lo <= 0 && hi >= 31)) {
#pragma unroll
                    for (int i = 0; i < 32; i++) mt = fmaxf(mt, __uint_as_float(s[i]));
                } else {
#pragma unroll
                    for (int i = 0; i < 32; i++) {
                        const float x = i >= lo && i <= hi ? __uint_as_float(s[i]) : -INFINITY;
                        s[i] = __float_as_uint(x);
                        mt = fmaxf(mt, x);
                    }
                }
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
            uint8_t *p_t = p_s + (t & 1) * 2 * kLtQAtom;
#pragma unroll
            for (int ch = 0; ch < 4; ch++) {
                uint4 hv, lv;
                uint32_t *hp = &hv.x, *lp = &lv.x;
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int i = ch * 8 + 2 * e;
                    const float p0 = ex2(fmaf(__uint_as_float(s[i]), c, -base)), p1 = ex2(fmaf(__uint_as_float(s[i + 1]), c, -base));
                    sum += p0 + p1;
                    hp[e] = pack_bf16(p0, p1);
                    lp[e] = pack_bf16(p0 - __uint_as_float(hp[e] << 16), p1 - __uint_as_float(hp[e] & 0xFFFF0000u));
                }
                *reinterpret_cast<uint4 *>(p_t + swz(row, 4 * half + ch)) = hv;
                *reinterpret_cast<uint4 *>(p_t + kLtQAtom + swz(row, 4 * half + ch)) = lv;
            }
            fence_async_smem();
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
        const int vcol = a.heads * a.dim_ld + h * a.vdim_ld;
        int t = 0;
        for (; t < tiles; t++) {
            const int st = t & 1, y = key0 + t * kLtKeys;
            if (t >= 2 && !mbar_wait_fast(sf + 8 * st, ((t >> 1) - 1) & 1)) break;
            mbar_expect_tx(kf + 8 * st, atoms * kLtKAtom);
            for (int at = 0; at < atoms; at++) {
                const uint32_t dst = smem_u32(k_s + (st * atoms + at) * kLtKAtom);
                if (at < da) lt_tma_2d(dst, &kv_map, h * a.dim_ld + 64 * at, y, kf + 8 * st);
                else lt_tma_2d(dst, &r_map, 64 * (at - da), y, kf + 8 * st);
            }
            if (t >= 2 && !mbar_wait_fast(of + 8 * st, ((t >> 1) - 1) & 1)) {
                mbar_wait(kf + 8 * st, (t >> 1) & 1);   // the key tile just asked for
                break;
            }
            mbar_expect_tx(vf + 8 * st, NV * kLtKAtom);
            for (int v = 0; v < NV; v++) lt_tma_2d(smem_u32(v_s + (st * NV + v) * kLtKAtom), &kv_map, vcol + 64 * v, y, vf + 8 * st);
        }
        ok = t == tiles;
        for (int k = t - 2; k < t; k++)   // no copy is in flight when the CTA ends
            if (k >= 0) {
                ok = mbar_wait(kf + 8 * (k & 1), (k >> 1) & 1) && ok;
                ok = mbar_wait(vf + 8 * (k & 1), (k >> 1) & 1) && ok;
            }
    } else if (warp == 9 && lane == 0) {
        // ---------------- MMA issuer ----------------
        const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kLtKeys >> 3) << 17) | ((128u >> 4) << 24);
        const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(NV * 64 >> 3) << 17) | ((128u >> 4) << 24);   // B is MN-major
        auto scores = [&](int t) {
            if (!mbar_wait_fast(kf + 8 * (t & 1), (t >> 1) & 1)) return false;
            tc_fence_after();
            bool add = false;
            for (int at = 0; at < atoms; at++) {
                const uint64_t dq = smem_desc(smem_u32(q_s + at * kLtQAtom)), dk = smem_desc(smem_u32(k_s + ((t & 1) * atoms + at) * kLtKAtom));
                const int width = at < da ? min(64, a.dim - 64 * at) : min(64, a.rot - 64 * (at - da));
                for (int k = 0; k < (width + 15) >> 4; k++) {
                    umma_bf16(tmem + (t & 1) * 64, dq + 2 * k, dk + 2 * k, id_s, add);
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
            const uint32_t pa = smem_u32(p_s + (t & 1) * 2 * kLtQAtom), va = smem_u32(v_s + (t & 1) * NV * kLtKAtom), o = o_tmem + (t & 1) * NV * 64;
#pragma unroll
            for (int x = 0; x < 2; x++) {   // hi, lo
                const uint64_t dp = smem_desc(pa + x * kLtQAtom), dv = smem_desc_mn(va);
#pragma unroll
                for (int k = 0; k < 4; k++) umma_bf16(o, dp + 2 * k, dv + (2048 >> 4) * k, id_o, (x | k) != 0);
            }
            umma_commit(of + 8 * (t & 1));
            if (t + 2 < tiles) ok = scores(t + 2);
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

// bf16 [rows, cols] row-major (cols a multiple of 64) -> boxes of 64 x 64, 128-byte swizzle, zero fill outside
static bool lt_map(const void *base, int64_t rows, int64_t cols, CUtensorMap *map) {
    LtEncodeFn fn = lt_encode_fn();
    memset(map, 0, sizeof(*map));
    if (!fn || ((uintptr_t)base & 15u) || cols % 64) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box[2] = {64, kLtKeys}, one[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, box, one, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// bf16 decoders, keys of at most four 64-wide pieces (head part and shared part each rounded up), values of two
bool latent_tc_supported(int act_dt, int dim, int rot, int vdim) {
    return act_dt == NNQ_BF16 && (dim + 63) / 64 + (rot + 63) / 64 <= kLtMaxAtoms && vdim <= 128 && lt_encode_fn() != nullptr;
}

template <int NV>
static nnq_status lt_go(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) {
    CUtensorMap kv_map, r_map;
    if (!lt_map(a.kv, a.keys, (int64_t)a.heads * (a.dim_ld + a.vdim_ld), &kv_map) || (a.rot_ld && !lt_map(a.lin_r, a.keys, a.rot_ld, &r_map)))
        return fail(ctx, NNQ_ERR_DISPATCH_FAILED, "tensor map creation failed");
    if (!a.rot_ld) r_map = kv_map;   // not read
    const int smem = lt_smem_bytes((a.dim_ld + a.rot_ld) / 64, NV);
    nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(attn_latent_tc_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "latent attention shared memory");
    if (s != NNQ_OK) return s;
    attn_latent_tc_kernel<NV><<<dim3(a.heads, (a.span.n + kLtRows - 1) / kLtRows), kLtThreads, smem, st>>>(kv_map, r_map, a, ctx->d_status);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "latent attention launch");
}

nnq_status launch_latent_tc(nnq_ctx *ctx, const LatentAttn &a, cudaStream_t st) { return a.vdim_ld > 64 ? lt_go<2>(ctx, a, st) : lt_go<1>(ctx, a, st); }

}  // namespace nnq
