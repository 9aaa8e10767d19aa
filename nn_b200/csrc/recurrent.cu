// Linear-attention recurrences of a block decoder: S_t = diag(decay_t) S_{t-1} + k_t v_t^T,
// o_t = S_t^T q_t per head, with a fixed decay per head (retention) or a decay per key channel and token
// from a low-rank gate (gated linear attention); optional half-split rotation of q and k; RMS norm of
// each head's o, silu output gate. Everything in f32.
//
// The state of a block of rows is advanced token by token (each CTA keeps a [dim, 16] tile of it in
// registers and streams the prepared q / k / decay rows through shared memory), so the result does not
// depend on how a sequence was cut into blocks: a cut only stores and reloads the same f32 state.
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

constexpr int kScanCols = 16, kScanThreads = 128;   // 8 threads per column, each every eighth group of four key rows

__device__ __forceinline__ void cp_async16(void *dst, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// grid (heads, ceil(vdim / 16)); NI = dim_ld / 32, TC tokens per stage of the double buffer
template <int NI, int TC, bool FIXED>
__global__ void __launch_bounds__(kScanThreads) rec_scan_kernel(const Recurrence r) {
    constexpr int NS = FIXED ? 2 : 3;   // streams: q, k (, decay)
    constexpr int LD = NI * 32;
    extern __shared__ __align__(16) float scan_smem[];   // [2][NS][TC][LD], then v [2][TC][16]
    float *vbuf = scan_smem + 2 * NS * TC * LD;
    const int tid = threadIdx.x, rg = tid & 7, col = tid >> 3;
    const int head = blockIdx.x, v0 = blockIdx.y * kScanCols;
    const int n = r.span.n;
    const bool live = v0 + col < r.vdim;
    float S[NI * 4];
    float *state = r.state + (size_t)head * r.dim * r.vdim + v0 + col;
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int row = 32 * i + 4 * rg + j;
            S[4 * i + j] = live && r.span.pos0 > 0 && row < r.dim ? state[(size_t)row * r.vdim] : 0.0f;
        }
    const float fixed = FIXED ? r.decay[head] : 0.0f;
    const size_t row_ld = (size_t)r.heads * LD;
    const float *src[3] = {r.q + (size_t)head * LD, r.k + (size_t)head * LD, r.a + (size_t)head * LD};
    const int chunks = (n + TC - 1) / TC;
    auto load = [&](int ch) {
        float *dst = scan_smem + (ch & 1) * NS * TC * LD;
        const int t0 = ch * TC;
#pragma unroll
        for (int s = 0; s < NS; s++)
            for (int i = tid; i < TC * (LD / 4); i += kScanThreads) {
                const int t = i / (LD / 4), c = i % (LD / 4);
                if (t0 + t < n) cp_async16(dst + (s * TC + t) * LD + 4 * c, src[s] + (size_t)(t0 + t) * row_ld + 4 * c);
            }
        for (int i = tid; i < TC * kScanCols; i += kScanThreads) {
            const int t = i / kScanCols, c = i % kScanCols;
            vbuf[(ch & 1) * TC * kScanCols + i] =
                t0 + t < n && v0 + c < r.vdim ? r.ffn.proj[(size_t)(t0 + t) * r.ffn.in_cols + r.c_v + head * r.vdim + v0 + c] : 0.0f;
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0);
    for (int ch = 0; ch < chunks; ch++) {
        if (ch + 1 < chunks) {
            load(ch + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float4 *b4 = reinterpret_cast<const float4 *>(scan_smem + (ch & 1) * NS * TC * LD);
        const float *vb = vbuf + (ch & 1) * TC * kScanCols + col;
        const int nt = min(TC, n - ch * TC);
        float po[TC];
#pragma unroll
        for (int t = 0; t < TC; t++) {
            po[t] = 0.0f;
            if (t < nt) {
                const float v = vb[t * kScanCols];
                float o0 = 0.0f, o1 = 0.0f, o2 = 0.0f, o3 = 0.0f;
#pragma unroll
                for (int i = 0; i < NI; i++) {
                    const float4 q = b4[t * (LD / 4) + rg + 8 * i], k = b4[(TC + t) * (LD / 4) + rg + 8 * i];
                    const float4 a = FIXED ? make_float4(fixed, fixed, fixed, fixed) : b4[((NS - 1) * TC + t) * (LD / 4) + rg + 8 * i];
                    float *s = S + 4 * i;
                    s[0] = fmaf(s[0], a.x, k.x * v);
                    s[1] = fmaf(s[1], a.y, k.y * v);
                    s[2] = fmaf(s[2], a.z, k.z * v);
                    s[3] = fmaf(s[3], a.w, k.w * v);
                    o0 = fmaf(s[0], q.x, o0);
                    o1 = fmaf(s[1], q.y, o1);
                    o2 = fmaf(s[2], q.z, o2);
                    o3 = fmaf(s[3], q.w, o3);
                }
                po[t] = (o0 + o1) + (o2 + o3);
            }
        }
        // sum over the eight threads of a column; thread rg ends up with token rg of the stage
        if (TC == 8) {
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float send = (rg & 4) ? po[i] : po[(i + 4) % TC], keep = (rg & 4) ? po[(i + 4) % TC] : po[i];
                po[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, 4);
            }
        } else {
#pragma unroll
            for (int i = 0; i < 4; i++) po[i] += __shfl_xor_sync(0xFFFFFFFFu, po[i], 4);
        }
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float send = (rg & 2) ? po[i] : po[i + 2], keep = (rg & 2) ? po[i + 2] : po[i];
            po[i] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, 2);
        }
        {
            const float send = (rg & 1) ? po[0] : po[1], keep = (rg & 1) ? po[1] : po[0];
            po[0] = keep + __shfl_xor_sync(0xFFFFFFFFu, send, 1);
        }
        const int t = ch * TC + (rg & (TC - 1));
        if (live && rg < TC && t < n) r.o[(size_t)t * r.heads * r.vdim + head * r.vdim + v0 + col] = po[0];
        __syncthreads();   // this stage's buffer is free for chunk ch + 2
    }
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int row = 32 * i + 4 * rg + j;
            if (live && row < r.dim) state[(size_t)row * r.vdim] = S[4 * i + j];
        }
}

// act[row, head] = o / rms(o) (* weight) * silu(g): one warp per (row, head)
__global__ void __launch_bounds__(128) rec_finish_kernel(const Recurrence r) {
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
    if (item >= (long long)r.span.n * r.heads) return;
    const int row = (int)(item / r.heads), head = (int)(item - (long long)row * r.heads);
    const float *o = r.o + item * r.vdim;
    float ss = 0.0f;
    for (int d = lane; d < r.vdim; d += 32) ss = fmaf(o[d], o[d], ss);
    const float rms = sqrtf(warp_sum(ss) / (float)r.vdim + r.eps);
    const float *g = r.ffn.proj + (size_t)row * r.ffn.in_cols + r.c_g + head * r.vdim;
    for (int d = lane; d < r.vdim; d += 32) {
        float v = o[d] / rms;
        if (r.head_norm) v *= r.head_norm[d];
        store_act(r.ffn.act, r.ffn.act_dt, (size_t)row * r.ffn.out_k + head * r.vdim + d, v * silu_f32(g[d]));
    }
}

constexpr int kStepWarps = 16, kStepBatch = 8;

// One token, everything between the two products: CTA h < heads prepares q / k / decay of its head, advances
// the head's state (read and written once), norms and gates the output; the other CTAs do the feed-forward part.
__global__ void __launch_bounds__(kStepWarps * 32) rec_step_kernel(const Recurrence r) {
    pdl_prologue();
    extern __shared__ float step_smem[];   // q, k, decay [dim], v [vdim], partial o [warps, vdim]
    __shared__ float red[32];
    if ((int)blockIdx.x >= r.heads) {
        ffn_part(r.ffn, 1, r.heads);
        return;
    }
    const int head = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pos = r.span.state[1];
    float *q = step_smem, *k = q + r.dim, *al = k + r.dim, *v = al + r.dim, *po = v + r.vdim;
    const float *p = r.ffn.proj;
    const int half = r.rot_dims >> 1;
    const float *cs = r.cosv + (size_t)pos * half, *sn = r.sinv + (size_t)pos * half;
    for (int d = tid; d < r.dim; d += kStepWarps * 32) {
        q[d] = rotated(p + r.c_q + head * r.dim, d, r.rot_dims, cs, sn) * r.q_scale;
        k[d] = rotated(p + r.c_k + head * r.dim, d, r.rot_dims, cs, sn) * r.k_scale;
        if (r.rank > 0) {
            const int c = head * r.dim + d;
            float z = 0.0f;
#pragma unroll 8
            for (int j = 0; j < r.rank; j++) z = fmaf(p[r.c_a1 + j], r.a2t[(size_t)j * r.heads * r.dim + c], z);
            al[d] = gate_decay(z + r.a2b[c], r.inv_tau);
        } else {
            al[d] = r.decay[head];
        }
    }
    for (int d = tid; d < r.vdim; d += kStepWarps * 32) v[d] = p[r.c_v + head * r.vdim + d];
    __syncthreads();
    float *S = r.state + (size_t)head * r.dim * r.vdim;
    for (int c = lane; c < r.vdim; c += 32) {
        const float vc = v[c];
        float acc = 0.0f;
        for (int r0 = warp; r0 < r.dim; r0 += kStepWarps * kStepBatch) {
            float s[kStepBatch];
#pragma unroll
            for (int i = 0; i < kStepBatch; i++) {
                const int row = r0 + i * kStepWarps;
                s[i] = pos > 0 && row < r.dim ? S[(size_t)row * r.vdim + c] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < kStepBatch; i++) {
                const int row = r0 + i * kStepWarps;
                if (row < r.dim) {
                    s[i] = fmaf(s[i], al[row], k[row] * vc);
                    acc = fmaf(s[i], q[row], acc);
                    S[(size_t)row * r.vdim + c] = s[i];
                }
            }
        }
        po[warp * r.vdim + c] = acc;
    }
    __syncthreads();
    float ss = 0.0f;
    for (int d = tid; d < r.vdim; d += kStepWarps * 32) {
        float o = 0.0f;
#pragma unroll
        for (int w = 0; w < kStepWarps; w++) o += po[w * r.vdim + d];
        v[d] = o;   // the value vector has been used
        ss = fmaf(o, o, ss);
    }
    const float rms = sqrtf(block_sum(ss, red) / (float)r.vdim + r.eps);
    for (int d = tid; d < r.vdim; d += kStepWarps * 32) {
        float o = v[d] / rms;
        if (r.head_norm) o *= r.head_norm[d];
        store_act(r.ffn.act, r.ffn.act_dt, (size_t)head * r.vdim + d, o * silu_f32(p[r.c_g + head * r.vdim + d]));
    }
}

// ---- host side ----

template <int NI>
static nnq_status go_scan(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    constexpr int TC = NI <= 4 ? 8 : 4;
    const bool fixed = r.rank == 0;
    const size_t smem = (size_t)(2 * (fixed ? 2 : 3) * TC * NI * 32 + 2 * TC * kScanCols) * sizeof(float);
    const dim3 grid(r.heads, (r.vdim + kScanCols - 1) / kScanCols);
    if (smem > 48 * 1024) {
        nnq_status s = check_cuda(ctx, fixed ? cudaFuncSetAttribute(rec_scan_kernel<NI, TC, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)
                                             : cudaFuncSetAttribute(rec_scan_kernel<NI, TC, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem),
                                  "recurrence shared memory");
        if (s != NNQ_OK) return s;
    }
    if (fixed) rec_scan_kernel<NI, TC, true><<<grid, kScanThreads, smem, st>>>(r);
    else rec_scan_kernel<NI, TC, false><<<grid, kScanThreads, smem, st>>>(r);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "recurrence launch");
}

nnq_status launch_rec_rows(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    const int per = kRecPrepWarps * kRecPrepRows;
    const int prep = r.heads * ((r.span.n + per - 1) / per);
    const int ffn = ffn_ctas(r.ffn, r.span.n, kRecPrepWarps * 32, ctx->sm_count);
    rec_prep_kernel<<<prep + ffn, kRecPrepWarps * 32, 0, st>>>(r, prep);
    ctx->launches++;
    nnq_status s = check_cuda(ctx, cudaGetLastError(), "recurrence prologue launch");
    if (s != NNQ_OK) return s;
    switch (r.dim_ld / 32) {
        case 1: s = go_scan<1>(ctx, r, st); break;
        case 2: s = go_scan<2>(ctx, r, st); break;
        case 3: s = go_scan<3>(ctx, r, st); break;
        case 4: s = go_scan<4>(ctx, r, st); break;
        case 5: s = go_scan<5>(ctx, r, st); break;
        case 6: s = go_scan<6>(ctx, r, st); break;
        case 7: s = go_scan<7>(ctx, r, st); break;
        case 8: s = go_scan<8>(ctx, r, st); break;
        default: return fail(ctx, NNQ_ERR_UNSUPPORTED, "key dimension %d of a recurrence is above %d", r.dim, kRecMaxKeyDim);
    }
    if (s != NNQ_OK) return s;
    const long long items = (long long)r.span.n * r.heads;
    rec_finish_kernel<<<(unsigned)((items + 3) / 4), 128, 0, st>>>(r);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "recurrence epilogue launch");
}

nnq_status launch_rec_step(nnq_ctx *ctx, const Recurrence &r, cudaStream_t st) {
    const size_t smem = (size_t)(3 * r.dim + (1 + kStepWarps) * r.vdim) * sizeof(float);
    if (smem > 48 * 1024) {
        nnq_status s = check_cuda(ctx, cudaFuncSetAttribute(rec_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem), "recurrence shared memory");
        if (s != NNQ_OK) return s;
    }
    launch_pdl_smem(rec_step_kernel, dim3(r.heads + ffn_ctas(r.ffn, 1, kStepWarps * 32, ctx->sm_count)), dim3(kStepWarps * 32), smem, st, r);
    ctx->launches++;
    return check_cuda(ctx, cudaGetLastError(), "recurrence step launch");
}

}  // namespace nnq
