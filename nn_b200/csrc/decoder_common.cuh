// Device helpers shared by the decoder's own kernels and the block mixers.
#pragma once
#include <cuda_bf16.h>

#include "nnq_internal.h"
#include "pdl.cuh"

namespace nnq {

__device__ __forceinline__ float block_sum(float v, float *red) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, off);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = 0.0f;
    for (int w = 0; w < nw; w++) t += red[w];
    return t;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xFFFFFFFFu, v, off);
    return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v = fmaxf(v, __shfl_xor_sync(0xFFFFFFFFu, v, off));
    return v;
}

__device__ __forceinline__ void store_act(void *dst, int dt, size_t i, float v) {
    if (dt == NNQ_F32) reinterpret_cast<float *>(dst)[i] = v;
    else reinterpret_cast<__nv_bfloat16 *>(dst)[i] = __float2bfloat16_rn(v);
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.0f + expf(-x)); }
// the tanh form of gelu
__device__ __forceinline__ float gelu_tanh_f32(float x) {
    return 0.5f * x * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * x * x, x, x)));
}
// kind: nnq_gate_act
__device__ __forceinline__ float gate_act(int kind, float x) { return kind == NNQ_ACT_GELU_TANH ? gelu_tanh_f32(x) : silu_f32(x); }

}  // namespace nnq
