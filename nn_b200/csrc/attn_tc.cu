// Sliding-window attention of a block of rows on the 5th-generation tensor cores, with f32-class accuracy.
//
// q, k, v and the softmax weights are f32 and stay so in effect: every operand enters the tensor core as two
// bf16 terms (x = hi + lo, the remainder is below 2^-16 of x), and a product is hi hi + hi lo + lo hi with f32
// accumulation in tensor memory. Scores, maxima, exponentials, sums and the output accumulators are f32.
//
// One CTA: 128 query vectors of one kv head (consecutive (row, query head of the group) pairs), key tiles of
// 64 over the union of the rows' windows.
//   warps 0-3: softmax. Thread r owns query vector r: reads its 64 scores from tensor memory, updates maximum
//              and sum, writes the weights as two swizzled bf16 tiles; adds the previous tile's weighted values
//              from tensor memory to its f32 accumulators.
//   warps 4-6: loaders. Convert the next key / value tile from the f32 ring cache into swizzled bf16 pairs
//              (values transposed), two stages.
//   warp 7:    one thread issues the MMAs: S(t + 1) = Q K^T right behind O(t) = P V.
// A commit after S(t + 1) tells the softmax warps that both are complete. Every wait is bounded.
#include <math.h>

#include "blocks.cuh"
#include "sync.cuh"
#include "tcgen05.cuh"

namespace nnq {

constexpr int kAtKeys = 64, kAtRows = 128;
constexpr int kAtQAtom = kAtRows * 128, kAtKAtom = kAtKeys * 128;   // bytes of a tile of 64 columns (one swizzle row)
constexpr int kAtThreads = 256, kAtLoaders = 3;   // (eight warps: two per scheduler, 255 registers each)
constexpr float kLog2E = 1.4426950408889634f;

// atoms: 64-wide pieces of the query / key dimension; nv: 32-wide pieces of the value dimension
__host__ __device__ constexpr int at_q_bytes(int atoms) { return 2 * atoms * kAtQAtom; }
__host__ __device__ constexpr int at_k_bytes(int atoms) { return 2 * atoms * kAtKAtom; }
__host__ __device__ constexpr int at_v_bytes(int nv) { return 2 * nv * 32 * 128; }
static int at_smem_bytes(int atoms, int nv) { return 1024 + at_q_bytes(atoms) + 2 * (at_k_bytes(atoms) + at_v_bytes(nv)) + 2 * kAtQAtom; }

// x and y as bf16 pairs: the nearest values and the nearest values of what they leave
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    hi = *reinterpret_cast<const uint32_t *>(&h);
    lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}

// byte offset of element e (0 .. 63) of row r inside a swizzled tile of 128-byte rows
__device__ __forceinline__ uint32_t swz_at(int r, int e) { return swz(r, e >> 3) + 2 * (e & 7); }

template <int ATOMS, int NV>
__global__ void __launch_bounds__(kAtThreads, 1) attn_tc_kernel(const WindowAttn a, int *status) {
    extern __shared__ __align__(1024) uint8_t at_smem_raw[];
    uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(at_smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t bars[6];   // kv_full[2], kv_empty[2], s_full, p_full
    __shared__ uint32_t tmem_s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const uint32_t kvf = smem_u32(bars), kve = kvf + 16, sf = kvf + 32, pf = kvf + 40;
    const int kvh = blockIdx.x, group = a.heads / a.kv_heads, pairs = a.span.n * group, t0 = blockIdx.y * kAtRows;
    const int last_pair = min(pairs, t0 + kAtRows) - 1;
    const int pos0 = a.span.pos0;
    const int first = max(0, pos0 + t0 / group - a.window + 1), last = pos0 + last_pair / group;   // keys some row sees
    const int tiles = (last - first) / kAtKeys + 1;
    uint8_t *q_s = smem, *kv_s = q_s + at_q_bytes(ATOMS), *p_s = kv_s + 2 * (at_k_bytes(ATOMS) + at_v_bytes(NV));
    const int kv_stage = at_k_bytes(ATOMS) + at_v_bytes(NV);

    if (tid == 0) {
        for (int i = 0; i < 2; i++) {
            mbar_init(kvf + 8 * i, kAtLoaders * 32);
            mbar_init(kve + 8 * i, 1);
        }
        mbar_init(sf, 1);
        mbar_init(pf, 128);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 7) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_s)), "r"(256u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    {
        // the 128 query vectors: neighbouring lanes take neighbouring dimensions, all loads before the first store
        constexpr int QN = kAtRows * 16 * ATOMS / kAtThreads;
        float4 v[QN];
#pragma unroll
        for (int i = 0; i < QN; i++) {
            const int u = tid + kAtThreads * i, t = t0 + u / (16 * ATOMS), d = 4 * (u % (16 * ATOMS));
            v[i] = t <= last_pair && d < a.dim_ld
                       ? *reinterpret_cast<const float4 *>(a.qrot + ((size_t)(t / group) * a.heads + kvh * group + t % group) * a.dim_ld + d)
                       : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll
        for (int i = 0; i < QN; i++) {
            const int u = tid + kAtThreads * i, r = u / (16 * ATOMS), d = 4 * (u % (16 * ATOMS));
            uint2 hi, lo;
            split2(v[i].x, v[i].y, hi.x, lo.x);
            split2(v[i].z, v[i].w, hi.y, lo.y);
            uint8_t *dst = q_s + (d >> 6) * kAtQAtom + swz_at(r, d & 63);
            *reinterpret_cast<uint2 *>(dst) = hi;
            *reinterpret_cast<uint2 *>(dst + ATOMS * kAtQAtom) = lo;
        }
        fence_async_smem();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_s, o_tmem = tmem + 64;   // scores: 64 columns, weighted values: the next NV * 32
    bool ok = true;

    if (warp < 4) {
        // ---------------- softmax ----------------
        const int row = (t0 + tid) / group;                           // (rows past the end are not stored)
        const int my_hi = pos0 + row, my_lo = my_hi - a.window + 1;   // keys this vector sees
        const float c = a.scale * kLog2E;
        const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
        float acc[NV * 32];
#pragma unroll
        for (int i = 0; i < NV * 32; i++) acc[i] = 0.0f;
        float m = -INFINITY, l = 0.0f, corr = 1.0f;
        for (int t = 0; t <= tiles; t++) {
            if (!mbar_wait_fast(sf, t & 1)) {
                ok = false;
                break;
            }
            tc_fence_after();
            if (t > 0) {
#pragma unroll
                for (int b = 0; b < NV; b++) {
                    uint32_t v[32];
                    tmem_ld32(o_tmem + lane_base + b * 32, v);
#pragma unroll
                    for (int i = 0; i < 32; i++) acc[b * 32 + i] = fmaf(acc[b * 32 + i], corr, __uint_as_float(v[i]));
                }
            }
            if (t == tiles) break;
            const int k0 = first + t * kAtKeys;
            const int lo = max(0, my_lo - k0), hi = min(kAtKeys - 1, my_hi - k0);   // visible keys of the tile
            uint32_t s[2][32];
            tmem_ld32(tmem + lane_base, s[0]);
            tmem_ld32(tmem + lane_base + 32, s[1]);
            float mt = -INFINITY;
#pragma unroll
            for (int i = 0; i < 64; i++) {
                const float x = i >= lo && i <= hi ? __uint_as_float(s[i >> 5][i & 31]) * c : -INFINITY;
                s[i >> 5][i & 31] = __float_as_uint(x);
                mt = fmaxf(mt, x);
            }
            const float mn = fmaxf(m, mt);
            corr = m == mn ? 1.0f : exp2f(m - mn);   // no key of this vector yet: both -inf
            const float base = mn == -INFINITY ? 0.0f : mn;
            float sum = 0.0f;
#pragma unroll
            for (int ch = 0; ch < 8; ch++) {
                uint4 h, lw;
                uint32_t *hp = &h.x, *lp = &lw.x;
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int i = ch * 8 + 2 * e;
                    const float p0 = exp2f(__uint_as_float(s[i >> 5][i & 31]) - base), p1 = exp2f(__uint_as_float(s[i >> 5][(i & 31) + 1]) - base);
                    sum += p0 + p1;
                    split2(p0, p1, hp[e], lp[e]);
                }
                *reinterpret_cast<uint4 *>(p_s + swz(tid, ch)) = h;
                *reinterpret_cast<uint4 *>(p_s + kAtQAtom + swz(tid, ch)) = lw;
            }
            l = l * corr + sum;
            m = mn;
            fence_async_smem();
            tc_fence_before();
            mbar_arrive(pf);
        }
        if (ok && t0 + tid <= last_pair) {
            const int head = kvh * group + (t0 + tid) % group;
            const float inv = 1.0f / l;
            const float *g = a.ffn.proj + (size_t)row * a.ffn.in_cols + a.c_g + head * a.vdim;
            const size_t at = (size_t)row * a.ffn.out_k + head * a.vdim;
            if (a.ffn.act_dt == NNQ_BF16 && (a.vdim & 7) == 0) {
#pragma unroll
                for (int b = 0; b < NV * 32; b += 32) {
                    float4 gv[8];
#pragma unroll
                    for (int i = 0; i < 8; i++)
                        gv[i] = a.gated && b + 4 * i < a.vdim ? *reinterpret_cast<const float4 *>(g + b + 4 * i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                    for (int d = 0; d < 32; d += 8) {
                        if (b + d >= a.vdim) continue;
                        float v[8];
#pragma unroll
                        for (int i = 0; i < 8; i++) v[i] = acc[b + d + i] * inv;
                        if (a.gated) {
                            const float4 g0 = gv[d / 4], g1 = gv[d / 4 + 1];
                            v[0] *= sigmoid_f32(g0.x); v[1] *= sigmoid_f32(g0.y); v[2] *= sigmoid_f32(g0.z); v[3] *= sigmoid_f32(g0.w);
                            v[4] *= sigmoid_f32(g1.x); v[5] *= sigmoid_f32(g1.y); v[6] *= sigmoid_f32(g1.z); v[7] *= sigmoid_f32(g1.w);
                        }
                        *reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(a.ffn.act) + at + b + d) =
                            make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
                    }
                }
            } else {
#pragma unroll
                for (int d = 0; d < NV * 32; d++)
                    if (d < a.vdim) store_act(a.ffn.act, a.ffn.act_dt, at + d, acc[d] * inv * (a.gated ? sigmoid_f32(g[d]) : 1.0f));
            }
        }
    } else if (warp < 4 + kAtLoaders) {
        // ---------------- loaders ----------------
        // The cache is read from L2 in batches held in registers, always one batch ahead of the conversion (the
        // next tile's keys are under way before this tile is handed over).
        constexpr int LT = kAtLoaders * 32;
        constexpr int KU = kAtKeys * 16 * ATOMS, KB = (KU + 2 * LT - 1) / (2 * LT);                // units of four dimensions of a key, two batches
        constexpr int VB = (NV * 8 + 2 * kAtLoaders - 1) / (2 * kAtLoaders);                       // groups of four value dimensions, two batches
        const int w = warp - 4, lt = tid - 128;
        const float *kb = a.kcache + (size_t)kvh * a.cap * a.dim_ld, *vb = a.vcache + (size_t)kvh * a.cap * a.vdim_ld;
        const float4 zero = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        const int j = 2 * lane;   // values: lane = pair of keys, a warp every third group of dimensions
        auto load_k = [&](int t, int b, float4 (&v)[KB]) {   // neighbouring lanes take neighbouring dimensions
            const int k0 = first + t * kAtKeys, have = t < tiles ? min(kAtKeys, last - k0 + 1) : 0, s0 = k0 % a.cap;
#pragma unroll
            for (int i = 0; i < KB; i++) {
                const int u = lt + LT * (b * KB + i), key = u / (16 * ATOMS), d = 4 * (u % (16 * ATOMS));
                int slot = s0 + key;
                if (slot >= a.cap) slot -= a.cap;
                v[i] = key < have && d < a.dim_ld ? *reinterpret_cast<const float4 *>(kb + (size_t)slot * a.dim_ld + d) : zero;
            }
        };
        auto store_k = [&](uint8_t *k_s, int b, const float4 (&v)[KB]) {
#pragma unroll
            for (int i = 0; i < KB; i++) {
                const int u = lt + LT * (b * KB + i), key = u / (16 * ATOMS), d = 4 * (u % (16 * ATOMS));
                if (u >= KU) continue;
                uint2 hi, lo;
                split2(v[i].x, v[i].y, hi.x, lo.x);
                split2(v[i].z, v[i].w, hi.y, lo.y);
                uint8_t *dst = k_s + (d >> 6) * kAtKAtom + swz_at(key, d & 63);
                *reinterpret_cast<uint2 *>(dst) = hi;
                *reinterpret_cast<uint2 *>(dst + ATOMS * kAtKAtom) = lo;
            }
        };
        auto load_v = [&](int t, int b, float4 (&x)[VB], float4 (&y)[VB]) {
            const int k0 = first + t * kAtKeys, have = min(kAtKeys, last - k0 + 1), s0 = k0 % a.cap;
            int sa = s0 + j, sb = s0 + j + 1;
            if (sa >= a.cap) sa -= a.cap;
            if (sb >= a.cap) sb -= a.cap;
            const float *va = vb + (size_t)sa * a.vdim_ld, *vc = vb + (size_t)sb * a.vdim_ld;
#pragma unroll
            for (int i = 0; i < VB; i++) {
                const int d = 4 * (w + kAtLoaders * (b * VB + i));
                x[i] = j < have && d < a.vdim_ld ? *reinterpret_cast<const float4 *>(va + d) : zero;
                y[i] = j + 1 < have && d < a.vdim_ld ? *reinterpret_cast<const float4 *>(vc + d) : zero;
            }
        };
        auto store_v = [&](uint8_t *v_s, int b, const float4 (&x)[VB], const float4 (&y)[VB]) {   // transposed
#pragma unroll
            for (int i = 0; i < VB; i++) {
                const int d = 4 * (w + kAtLoaders * (b * VB + i));
                if (d >= NV * 32) continue;
                const float xv[4] = {x[i].x, x[i].y, x[i].z, x[i].w}, yv[4] = {y[i].x, y[i].y, y[i].z, y[i].w};
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    uint32_t hi, lo;
                    split2(xv[e], yv[e], hi, lo);
                    uint8_t *dst = v_s + swz_at(d + e, j);
                    *reinterpret_cast<uint32_t *>(dst) = hi;
                    *reinterpret_cast<uint32_t *>(dst + NV * 32 * 128) = lo;
                }
            }
        };
        float4 ka[KB], kc[KB], vx[VB], vy[VB];
        load_k(0, 0, ka);
        load_k(0, 1, kc);
        for (int t = 0; t < tiles; t++) {
            const int st = t & 1;
            uint8_t *k_s = kv_s + st * kv_stage, *v_s = k_s + at_k_bytes(ATOMS);
            if (t >= 2 && !mbar_wait_fast(kve + 8 * st, ((t >> 1) - 1) & 1)) {
                ok = false;
                break;
            }
            load_v(t, 0, vx, vy);
            store_k(k_s, 0, ka);
            store_k(k_s, 1, kc);
            load_k(t + 1, 0, ka);
            store_v(v_s, 0, vx, vy);
            load_v(t, 1, vx, vy);
            load_k(t + 1, 1, kc);
            store_v(v_s, 1, vx, vy);
            fence_async_smem();
            mbar_arrive(kvf + 8 * st);
        }
    } else if (lane == 0) {
        // ---------------- MMA issuer ----------------
        const uint32_t id_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kAtKeys >> 3) << 17) | ((128u >> 4) << 24);
        const uint32_t id_o = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(NV * 32 >> 3) << 17) | ((128u >> 4) << 24);
        const uint32_t qa = smem_u32(q_s), pa = smem_u32(p_s);
        auto scores = [&](int t) {
            const uint32_t ka = smem_u32(kv_s + (t & 1) * kv_stage);
            bool add = false;
#pragma unroll 1
            for (int x = 0; x < 3; x++) {   // hi hi, hi lo, lo hi
                const uint32_t qo = qa + (x == 2 ? ATOMS * kAtQAtom : 0), ko = ka + (x == 1 ? ATOMS * kAtKAtom : 0);
                for (int at = 0; at < ATOMS; at++) {
                    const uint64_t dq = smem_desc(qo + at * kAtQAtom), dk = smem_desc(ko + at * kAtKAtom);
#pragma unroll
                    for (int k = 0; k < 4; k++) {
                        umma_bf16(tmem, dq + 2 * k, dk + 2 * k, id_s, add);
                        add = true;
                    }
                }
            }
            umma_commit(sf);
        };
        ok = mbar_wait_fast(kvf, 0);
        tc_fence_after();
        if (ok) scores(0);
        for (int t = 0; t < tiles && ok; t++) {
            if (!mbar_wait_fast(pf, t & 1)) {
                ok = false;
                break;
            }
            tc_fence_after();
            const uint32_t va = smem_u32(kv_s + (t & 1) * kv_stage) + at_k_bytes(ATOMS);
#pragma unroll 1
            for (int x = 0; x < 3; x++) {
                const uint64_t dp = smem_desc(pa + (x == 2 ? kAtQAtom : 0)), dv = smem_desc(va + (x == 1 ? NV * 32 * 128 : 0));
#pragma unroll
                for (int k = 0; k < 4; k++) umma_bf16(o_tmem, dp + 2 * k, dv + 2 * k, id_o, (x | k) != 0);
            }
            umma_commit(kve + 8 * (t & 1));
            if (t + 1 < tiles) {
                if (!mbar_wait_fast(kvf + 8 * ((t + 1) & 1), ((t + 1) >> 1) & 1)) {
                    ok = false;
                    break;
                }
                tc_fence_after();
                scores(t + 1);
            } else {
                umma_commit(sf);   // the last tile's weighted values
            }
        }
        if (!ok) {
            // MMAs that were issued may still read shared memory and write tensor memory: one more bounded wait
            umma_commit(sf);
            for (int i = 0; i < 2; i++) mbar_wait(sf, i);
        }
    }
    if (!ok) atomicExch(status, 1);
    tc_fence_before();
    __syncthreads();
    if (warp == 7) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(256u) : "memory");
    }
}

// Enough query vectors to fill a good part of a tile, heads of at most 128, bf16 decoders (an f32 decoder
// keeps f32 products).
bool attn_tc_supported(const WindowAttn &a) {
    return a.ffn.act_dt == NNQ_BF16 && a.dim <= 128 && a.vdim <= 128 && a.span.n * (a.heads / a.kv_heads) >= 32;
}

template <int ATOMS, int NV>
static nnq_status at_go(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const int smem = at_smem_bytes(ATOMS, NV), pairs = a.span.n * (a.heads / a.kv_heads);
    nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(attn_tc_kernel<ATOMS, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem), "attention shared memory");
    if (s != NNQ_OK) return s;
    attn_tc_kernel<ATOMS, NV><<<dim3(a.kv_heads, (pairs + kAtRows - 1) / kAtRows), kAtThreads, smem, st>>>(a, ctx->d_status);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "tensor-core attention launch");
}

nnq_status launch_attn_tc(nnq_ctx *ctx, const WindowAttn &a, cudaStream_t st) {
    const bool two = a.dim > 64;
    switch ((a.vdim + 31) / 32) {
        case 1: return two ? at_go<2, 1>(ctx, a, st) : at_go<1, 1>(ctx, a, st);
        case 2: return two ? at_go<2, 2>(ctx, a, st) : at_go<1, 2>(ctx, a, st);
        case 3: return two ? at_go<2, 3>(ctx, a, st) : at_go<1, 3>(ctx, a, st);
        default: return two ? at_go<2, 4>(ctx, a, st) : at_go<1, 4>(ctx, a, st);
    }
}

}  // namespace nnq
