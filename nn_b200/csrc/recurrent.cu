// Linear-attention recurrences of a block decoder: S_t = diag(decay_t) S_{t-1} + k_t v_t^T,
// o_t = S_t^T q_t per head, with a fixed decay per head (retention) or a decay per key channel and token
// from a low-rank gate (gated linear attention); optional half-split rotation of q and k; RMS norm of
// each head's o, silu output gate. Everything in f32.
//
// The state of a block of rows is advanced token by token (a warp keeps a [dim, 8] tile of it in registers,
// the prepared q / k / decay rows stream through shared memory), so the result does not depend on how a
// sequence was cut into blocks: a cut only stores and reloads the same f32 state.
#include <math.h>

#include "blocks.cuh"

namespace nnq {

// sigmoid(z)^(1 / tau) without leaving f32 range: exp(-softplus(-z) / tau)
__device__ __forceinline__ float gate_decay(float z, float inv_tau) {
    const float sp = fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z)));
    return expf(-sp * inv_tau);
}

constexpr int kRecPrepWarps = 4, kRecPrepRows = 4;   // rows per warp

// q, k (rotated, scaled) and the decay of a block of rows, padded to dim_ld with zeros. CTA: one head, 16 rows.
__global__ void __launch_bounds__(kRecPrepWarps * 32) rec_prep_kernel(const Recurrence r, int prep_ctas) {
    if ((int)blockIdx.x >= prep_ctas) {
        ffn_part(r.ffn, r.span.n, prep_ctas);
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int head = blockIdx.x % r.heads;
    const int row0 = (blockIdx.x / r.heads) * (kRecPrepWarps * kRecPrepRows) + warp * kRecPrepRows;
    const int rows = min(kRecPrepRows, r.span.n - row0);
    if (rows <= 0) return;
    const int half = r.rot_dims >> 1;
    const size_t hd = (size_t)r.heads * r.dim;
    for (int d = lane; d < r.dim_ld; d += 32) {
        float z[kRecPrepRows];
        if (r.rank > 0 && d < r.dim) {
            const int c = head * r.dim + d;
#pragma unroll
            for (int i = 0; i < kRecPrepRows; i++) z[i] = 0.0f;
            for (int j = 0; j < r.rank; j++) {
                const float w = r.a2t[j * hd + c];
#pragma unroll
                for (int i = 0; i < kRecPrepRows; i++)
                    z[i] = fmaf(r.ffn.proj[(size_t)(row0 + min(i, rows - 1)) * r.ffn.in_cols + r.c_a1 + j], w, z[i]);
            }
            const float b = r.a2b[c];
#pragma unroll
            for (int i = 0; i < kRecPrepRows; i++) z[i] = gate_decay(z[i] + b, r.inv_tau);
        }
        for (int i = 0; i < rows; i++) {
            const int row = row0 + i, pos = r.span.pos0 + row;
            const float *p = r.ffn.proj + (size_t)row * r.ffn.in_cols + head * r.dim;
            const float *cs = r.cosv + (size_t)pos * half, *sn = r.sinv + (size_t)pos * half;
            const size_t at = ((size_t)row * r.heads + head) * r.dim_ld + d;
            const bool in = d < r.dim;
            r.q[at] = in ? rotated(p + r.c_q, d, r.rot_dims, cs, sn) * r.q_scale : 0.0f;
            r.k[at] = in ? rotated(p + r.c_k, d, r.rot_dims, cs, sn) * r.k_scale : 0.0f;
            if (r.rank > 0) {
                float al = 0.0f;
#pragma unroll
                for (int u = 0; u < kRecPrepRows; u++)
                    if (u == i) al = z[u];
                r.a[at] = in ? al : 0.0f;
            }
        }
    }
}

// ---- the scan over a block of rows ----
//
// A warp owns a few columns of the state over all key rows: RL row lanes (32; 16 for heads of at most 64, then two
// column groups) hold rows 4 RL j + 4 rl .. + 3 of C columns each, as packed f32 pairs (two rows of a column), so that
// q, k and the decay come as pairs out of one 16-byte shared-memory read without two lanes reading the same, and the
// three operations of a state element -- k v, s a + (k v), o + s q -- are packed f32x2 instructions. After eight
// tokens the lanes' partial o are reduced across the row lanes by halving exchanges: a lane ends with one token of
// one or two columns. Tokens stream through a three-stage ring of cp.async copies, one barrier per stage.

constexpr int kScanTokens = 8, kScanStages = 3;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
// four bytes, or four zero bytes
__device__ __forceinline__ void cp_async4(uint32_t dst, const void *src, bool real) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(real ? 4 : 0) : "memory");
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float &lo, float &hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// grid (heads, ceil(vdim / columns of a CTA)); NJ = dim_ld / (4 RL)
template <int RL, int NJ, int C, int WARPS, bool FIXED>
__global__ void __launch_bounds__(WARPS * 32) rec_scan_kernel(const Recurrence r) {
    constexpr int NS = FIXED ? 2 : 3;   // streams: q, k (, decay)
    constexpr int RW = 4 * RL, LD = NJ * RW, COLS = WARPS * (32 / RL) * C, T = kScanTokens, THREADS = WARPS * 32;
    constexpr int STAGE = T * (NS * LD + COLS);   // floats
    extern __shared__ __align__(16) float scan_smem[];
    const int tid = threadIdx.x, rl = tid % RL;
    const int wcol = tid / RL * C;
    const int head = blockIdx.x, v0 = blockIdx.y * COLS, n = r.span.n;
    float *state = r.state + (size_t)head * r.dim * r.vdim;
    uint64_t S[NJ][2][C];
#pragma unroll
    for (int j = 0; j < NJ; j++)
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int c = 0; c < C; c++) {
                float s[2];
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int row = RW * j + 4 * rl + 2 * h + e, col = v0 + wcol + c;
                    s[e] = r.span.pos0 > 0 && row < r.dim && col < r.vdim ? state[(size_t)row * r.vdim + col] : 0.0f;
                }
                S[j][h][c] = pack2(s[0], s[1]);
            }
    const float fixed = FIXED ? r.decay[head] : 0.0f;
    const uint64_t fixed2 = pack2(fixed, fixed);
    const size_t row_ld = (size_t)r.heads * LD;
    const float *src[3] = {r.q + (size_t)head * LD, r.k + (size_t)head * LD, r.a + (size_t)head * LD};
    const float *vsrc = r.ffn.proj + r.c_v + head * r.vdim;
    const int chunks = (n + T - 1) / T;
    const uint32_t smem0 = (uint32_t)__cvta_generic_to_shared(scan_smem);
    auto load = [&](int ch) {
        if (ch < chunks) {
            const uint32_t dst = smem0 + 4u * STAGE * (ch % kScanStages);
            const int t0 = ch * T;
#pragma unroll
            for (int s = 0; s < NS; s++)
#pragma unroll
                for (int i = tid; i < T * (LD / 4); i += THREADS) {
                    const int t = i / (LD / 4), c = i % (LD / 4);
                    if (t0 + t < n) cp_async16(dst + 4u * ((s * T + t) * LD + 4 * c), src[s] + (size_t)(t0 + t) * row_ld + 4 * c);
                }
#pragma unroll
            for (int i = tid; i < T * COLS; i += THREADS) {
                const int t = i / COLS, c = i % COLS;
                const bool real = t0 + t < n && v0 + c < r.vdim;
                cp_async4(dst + 4u * (NS * T * LD + i), real ? vsrc + (size_t)(t0 + t) * r.ffn.in_cols + v0 + c : vsrc, real);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");   // (empty past the end: the group count stays in step)
    };
    load(0);
    load(1);
    for (int ch = 0; ch < chunks; ch++) {
        asm volatile("cp.async.wait_group 1;" ::: "memory");   // chunk ch has landed
        __syncthreads();                                       // for everybody, and everybody is done with chunk ch - 1
        load(ch + 2);
        const float *b = scan_smem + STAGE * (ch % kScanStages);
        const int nt = min(T, n - ch * T);
        float po[T * C];
#pragma unroll
        for (int t = 0; t < T; t++) {
            uint64_t o[C];
#pragma unroll
            for (int c = 0; c < C; c++) o[c] = 0;
            if (t < nt) {
                const float *v = b + NS * T * LD + t * COLS + wcol;
                uint64_t vd[C];
#pragma unroll
                for (int c = 0; c < C; c++) vd[c] = pack2(v[c], v[c]);
#pragma unroll
                for (int j = 0; j < NJ; j++) {
                    const int at = RW * j + 4 * rl;
                    const ulonglong2 q = *reinterpret_cast<const ulonglong2 *>(b + t * LD + at);
                    const ulonglong2 k = *reinterpret_cast<const ulonglong2 *>(b + (T + t) * LD + at);
                    const ulonglong2 al = FIXED ? make_ulonglong2(fixed2, fixed2) : *reinterpret_cast<const ulonglong2 *>(b + ((NS - 1) * T + t) * LD + at);
#pragma unroll
                    for (int c = 0; c < C; c++) {
                        S[j][0][c] = fma2(S[j][0][c], al.x, mul2(k.x, vd[c]));
                        o[c] = fma2(S[j][0][c], q.x, o[c]);
                    }
#pragma unroll
                    for (int c = 0; c < C; c++) {
                        S[j][1][c] = fma2(S[j][1][c], al.y, mul2(k.y, vd[c]));
                        o[c] = fma2(S[j][1][c], q.y, o[c]);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < C; c++) {
                float lo, hi;
                unpack2(o[c], lo, hi);
                po[t * C + c] = lo + hi;
            }
        }
        // 8 C sums over RL lanes: the upper three bits of the row lane pick a token, the next ones a column (or a pair)
        constexpr int LR = RL == 32 ? 5 : 4, LC = C == 4 ? 2 : (C == 2 ? 1 : 0);
        constexpr int CB = LC < LR - 3 ? LC : LR - 3, LEFT = C >> CB, SPARE = LR - 3 - CB;
#pragma unroll
        for (int step = 0; step < LR; step++) {
            const int half = (T * C / 2) >> step, bit = (RL / 2) >> step;
            if (step >= 3 + CB) {
#pragma unroll
                for (int i = 0; i < LEFT; i++) po[i] += __shfl_xor_sync(0xFFFFFFFFu, po[i], bit);
            } else {
#pragma unroll
                for (int i = 0; i < half; i++) {
                    const float send = (rl & bit) ? po[i] : po[i + half], keep = (rl & bit) ? po[i + half] : po[i];
                    po[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, bit);
                }
            }
        }
        const int t = ch * T + (rl >> (LR - 3)), col = v0 + wcol + ((rl >> SPARE) & ((1 << CB) - 1)) * LEFT;
        if (t < n && (rl & ((1 << SPARE) - 1)) == 0) {
            float *o = r.o + ((size_t)t * r.heads + head) * r.vdim + col;
#pragma unroll
            for (int i = 0; i < LEFT; i++)
                if (col + i < r.vdim) o[i] = po[i];
        }
    }
#pragma unroll
    for (int j = 0; j < NJ; j++)
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int c = 0; c < C; c++) {
                float s[2];
                unpack2(S[j][h][c], s[0], s[1]);
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int row = RW * j + 4 * rl + 2 * h + e, col = v0 + wcol + c;
                    if (row < r.dim && col < r.vdim) state[(size_t)row * r.vdim + col] = s[e];
                }
            }
}

// act[row, head] = o / rms(o) (* weight) * silu(g): one warp per (row, head)
template <bool VEC>
__global__ void __launch_bounds__(128) rec_finish_kernel(const Recurrence r) {
    const int lane = threadIdx.x & 31;
    const int item = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= r.span.n * r.heads) return;
    const int row = item / r.heads, head = item - row * r.heads;
    const float *o = r.o + (size_t)item * r.vdim;
    const float *g = r.ffn.proj + (size_t)row * r.ffn.in_cols + r.c_g + head * r.vdim;
    const size_t at = (size_t)row * r.ffn.out_k + head * r.vdim;
    float ss = 0.0f;
    if constexpr (VEC) {   // vdim a multiple of 4, at most 512
        float4 ov[4], gv[4];
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int d = 4 * lane + 128 * i;
            ov[i] = d < r.vdim ? *reinterpret_cast<const float4 *>(o + d) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            gv[i] = d < r.vdim ? *reinterpret_cast<const float4 *>(g + d) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            ss = fmaf(ov[i].x, ov[i].x, fmaf(ov[i].y, ov[i].y, fmaf(ov[i].z, ov[i].z, fmaf(ov[i].w, ov[i].w, ss))));
        }
        const float rms = sqrtf(warp_sum(ss) / (float)r.vdim + r.eps);
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int d = 4 * lane + 128 * i;
            if (d >= r.vdim) continue;
            const float4 w = r.head_norm ? *reinterpret_cast<const float4 *>(r.head_norm + d) : make_float4(1.0f, 1.0f, 1.0f, 1.0f);
            const float y0 = ov[i].x / rms * w.x * silu_f32(gv[i].x), y1 = ov[i].y / rms * w.y * silu_f32(gv[i].y);
            const float y2 = ov[i].z / rms * w.z * silu_f32(gv[i].z), y3 = ov[i].w / rms * w.w * silu_f32(gv[i].w);
            if (r.ffn.act_dt == NNQ_F32) {
                *reinterpret_cast<float4 *>(reinterpret_cast<float *>(r.ffn.act) + at + d) = make_float4(y0, y1, y2, y3);
            } else {
                const __nv_bfloat162 a = __floats2bfloat162_rn(y0, y1), b = __floats2bfloat162_rn(y2, y3);
                *reinterpret_cast<uint2 *>(reinterpret_cast<__nv_bfloat16 *>(r.ffn.act) + at + d) =
                    make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
            }
        }
    } else {
        for (int d = lane; d < r.vdim; d += 32) ss = fmaf(o[d], o[d], ss);
        const float rms = sqrtf(warp_sum(ss) / (float)r.vdim + r.eps);
        for (int d = lane; d < r.vdim; d += 32) {
            float v = o[d] / rms;
            if (r.head_norm) v *= r.head_norm[d];
            store_act(r.ffn.act, r.ffn.act_dt, at + d, v * silu_f32(g[d]));
        }
    }
}

// ---- one token ----
//
// Everything between the two products: a cluster of CTAs per head, each with a slice of the value columns (a
// multiple of 32). Every CTA prepares q / k / decay of the head, advances its slice of the state (lanes over
// columns, warps over key rows; the slice's first 32 columns are asked for before the kernel waits for the product
// in front of it), sums o over the warps; the squares of o are summed over the cluster through its shared memory
// for the norm, then the slice is gated and stored. Further CTAs do the feed-forward part.
constexpr int kStepWarps = 8, kStepThreads = kStepWarps * 32, kStepRows = kRecMaxKeyDim / kStepWarps;

__global__ void __launch_bounds__(kStepThreads) rec_step_kernel(const Recurrence r, int cluster, int slice) {
    extern __shared__ float step_smem[];   // q, k, decay [dim], v, o [slice], partial o [warps, 32]
    __shared__ float red[32];
    __shared__ float squares;              // this CTA's sum of o^2
    if ((int)blockIdx.x >= r.heads * cluster) {
        pdl_prologue();
        pdl_release();
        ffn_part(r.ffn, 1, r.heads * cluster);
        return;
    }
    const int head = blockIdx.x / cluster, c0 = (blockIdx.x - head * cluster) * slice, cn = min(slice, r.vdim - c0);   // (cn <= 0: nothing of its own)
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pos = r.span.state[1];
    float *q = step_smem, *k = q + r.dim, *al = k + r.dim, *v = al + r.dim, *o = v + slice, *po = o + slice;
    float *S = r.state + (size_t)head * r.dim * r.vdim + c0;
    float s[kStepRows];
    auto fetch = [&](int c) {
#pragma unroll
        for (int i = 0; i < kStepRows; i++) {
            const int row = warp + i * kStepWarps;
            s[i] = pos > 0 && row < r.dim && c < cn ? S[(size_t)row * r.vdim + c] : 0.0f;
        }
    };
    fetch(lane);
    pdl_prologue();
    pdl_release();
    const float *p = r.ffn.proj;
    const int half = r.rot_dims >> 1;
    const float *cs = r.cosv + (size_t)pos * half, *sn = r.sinv + (size_t)pos * half;
    for (int d = tid; d < r.dim; d += kStepThreads) {
        q[d] = rotated(p + r.c_q + head * r.dim, d, r.rot_dims, cs, sn) * r.q_scale;
        k[d] = rotated(p + r.c_k + head * r.dim, d, r.rot_dims, cs, sn) * r.k_scale;
        if (r.rank > 0) {
            const int c = head * r.dim + d;
            float z = 0.0f;
#pragma unroll 16
            for (int j = 0; j < r.rank; j++) z = fmaf(p[r.c_a1 + j], r.a2t[(size_t)j * r.heads * r.dim + c], z);
            al[d] = gate_decay(z + r.a2b[c], r.inv_tau);
        } else {
            al[d] = r.decay[head];
        }
    }
    for (int d = tid; d < cn; d += kStepThreads) v[d] = p[r.c_v + head * r.vdim + c0 + d];
    __syncthreads();
    float ss = 0.0f;
    for (int b = 0; b < cn; b += 32) {
        const int c = b + lane;
        if (b > 0) fetch(c);
        const float vc = c < cn ? v[c] : 0.0f;
        float acc = 0.0f;
#pragma unroll
        for (int i = 0; i < kStepRows; i++) {
            const int row = warp + i * kStepWarps;
            if (row < r.dim) {
                s[i] = fmaf(s[i], al[row], k[row] * vc);
                acc = fmaf(s[i], q[row], acc);
                if (c < cn) S[(size_t)row * r.vdim + c] = s[i];
            }
        }
        po[warp * 32 + lane] = acc;
        __syncthreads();
        if (warp == 0) {
            float t = 0.0f;
#pragma unroll
            for (int w = 0; w < kStepWarps; w++) t += po[w * 32 + lane];
            if (c < cn) {
                o[c] = t;
                ss = fmaf(t, t, ss);
            }
        }
        __syncthreads();
    }
    ss = block_sum(ss, red);
    if (cluster > 1) {
        if (tid == 0) squares = ss;
        asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
        ss = 0.0f;
        const uint32_t mine = (uint32_t)__cvta_generic_to_shared(&squares);
        for (int i = 0; i < cluster; i++) {   // the same order in every CTA
            uint32_t at;
            float x;
            asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(at) : "r"(mine), "r"(i));
            asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(x) : "r"(at) : "memory");
            ss += x;
        }
    }
    const float rms = sqrtf(ss / (float)r.vdim + r.eps);
    for (int d = tid; d < cn; d += kStepThreads) {
        float x = o[d] / rms;
        if (r.head_norm) x *= r.head_norm[c0 + d];
        const int c = head * r.vdim + c0 + d;
        store_act(r.ffn.act, r.ffn.act_dt, c, x * silu_f32(p[r.c_g + c]));
    }
    // nobody leaves while its sum may still be read
    if (cluster > 1) asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// ---- host side ----

template <int RL, int NJ, int C, int WARPS, bool FIXED>
static nnq_status go_scan(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    constexpr int cols = WARPS * (32 / RL) * C;
    constexpr size_t smem = (size_t)kScanStages * kScanTokens * ((FIXED ? 2 : 3) * NJ * 4 * RL + cols) * sizeof(float);
    auto kernel = rec_scan_kernel<RL, NJ, C, WARPS, FIXED>;
    if (smem > 48 * 1024) {
        nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem), "recurrence shared memory");
        if (s != NNQ_OK) return s;
    }
    kernel<<<dim3(r.heads, (r.vdim + cols - 1) / cols), WARPS * 32, smem, st>>>(r);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "recurrence launch");
}

// Wide tiles amortise the shared-memory reads of q / k / decay over more columns, narrow ones give more warps.
// Measured (us per 1024 rows, all kernels of the mixer, C = 4 / 2 / 1): 16 heads of 128 x 256 254 / 284 / 410,
// 8 heads of 128 x 256 222 / 191 / 244, 8 heads of 64 x 64 141 / 130 / 116.
template <int RL, int NJ>
static nnq_status pick_scan(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    constexpr int W = RL == 32 ? 8 : 4;
    const bool fixed = r.rank == 0;
    auto warps = [&](int c) { return r.heads * ((r.vdim + (32 / RL) * c - 1) / ((32 / RL) * c)); };
    const int enough = 5 * ctx->sm_count;
    const int c = warps(4) >= enough ? 4 : (warps(2) >= enough ? 2 : 1);
    if (c == 4) return fixed ? go_scan<RL, NJ, 4, W, true>(ctx, r, st) : go_scan<RL, NJ, 4, W, false>(ctx, r, st);
    if (c == 2) return fixed ? go_scan<RL, NJ, 2, W, true>(ctx, r, st) : go_scan<RL, NJ, 2, W, false>(ctx, r, st);
    return fixed ? go_scan<RL, NJ, 1, W, true>(ctx, r, st) : go_scan<RL, NJ, 1, W, false>(ctx, r, st);
}

nnq_status launch_rec_rows(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    const int per = kRecPrepWarps * kRecPrepRows;
    const int prep = r.heads * ((r.span.n + per - 1) / per);
    const int ffn = ffn_ctas(r.ffn, r.span.n, kRecPrepWarps * 32, ctx->sm_count);
    rec_prep_kernel<<<prep + ffn, kRecPrepWarps * 32, 0, st>>>(r, prep);
    ctx->launches++;
    nnq_status s = check_cuda(ctx, cudaGetLastError(), "recurrence prologue launch");
    if (s != NNQ_OK) return s;
    switch (r.dim_ld) {
        case 64: s = pick_scan<16, 1>(ctx, r, st); break;
        case 128: s = pick_scan<32, 1>(ctx, r, st); break;
        case 256: s = pick_scan<32, 2>(ctx, r, st); break;
        default: return fail(ctx, NNQ_ERR_UNSUPPORTED, "key dimension %d of a recurrence is above %d", r.dim, kRecMaxKeyDim);
    }
    if (s != NNQ_OK) return s;
    const int ctas = (r.span.n * r.heads + 3) / 4;
    if (r.vdim % 4 == 0 && r.vdim <= 512) rec_finish_kernel<true><<<ctas, 128, 0, st>>>(r);
    else rec_finish_kernel<false><<<ctas, 128, 0, st>>>(r);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "recurrence epilogue launch");
}

nnq_status launch_rec_step(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    // up to eight CTAs per head with at least 32 columns each
    const int want = (r.vdim + 31) / 32 < 8 ? (r.vdim + 31) / 32 : 8;
    const int slice = ((r.vdim + want - 1) / want + 31) / 32 * 32, cluster = (r.vdim + slice - 1) / slice;
    const size_t smem = (size_t)(3 * r.dim + 2 * slice + kStepThreads) * sizeof(float);
    const int ctas = r.heads * cluster + (ffn_ctas(r.ffn, 1, kStepThreads, ctx->sm_count) + cluster - 1) / cluster * cluster;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ctas);
    cfg.blockDim = dim3(kStepThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    attr[1].id = cudaLaunchAttributeClusterDimension;
    attr[1].val.clusterDim.x = cluster;
    attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 2;
    ctx->launches++;
    return check_cuda(ctx, cudaLaunchKernelEx(&cfg, rec_step_kernel, r, cluster, slice), "recurrence step launch");
}

}  // namespace nnq
