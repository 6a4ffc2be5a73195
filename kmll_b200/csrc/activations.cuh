// Scalar functions shared by the layered decoders' kernels, all in f32.
#pragma once

#include "internal.cuh"

namespace kmll {

__device__ inline float act_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ inline float act_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ inline float act_gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ inline float apply_act(float z, int act) {
    return act == KMLL_ACT_SILU ? act_silu(z) : act == KMLL_ACT_SIGMOID ? act_sigmoid(z) : act == KMLL_ACT_GELU_TANH ? act_gelu_tanh(z) : z;
}
__device__ inline float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
// 1 / root mean square with eps inside the root
__device__ inline float inv_rms(float sum_sq, int n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }

// count, mean and sum of squared deviations of a set of values; add() merges two disjoint sets
struct Moments {
    float n, mean, dev;
    __device__ inline void add(float n2, float mean2, float dev2) {
        const float total = n + n2, d = mean2 - mean, share = total > 0.0f ? n2 / total : 0.0f;
        mean += d * share;
        dev += dev2 + d * d * n * share;
        n = total;
    }
    __device__ inline void add_warp() {
#pragma unroll
        for (int off = 16; off > 0; off >>= 1)
            add(__shfl_xor_sync(0xffffffffu, n, off), __shfl_xor_sync(0xffffffffu, mean, off), __shfl_xor_sync(0xffffffffu, dev, off));
    }
};
// block-wide moments; every thread gets them (scratch: 96 floats, at most 32 warps)
__device__ inline Moments block_moments(Moments m, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    m.add_warp();
    __syncthreads();
    if (lane == 0) { scratch[warp] = m.n; scratch[32 + warp] = m.mean; scratch[64 + warp] = m.dev; }
    __syncthreads();
    m = lane < nw ? Moments{scratch[lane], scratch[32 + lane], scratch[64 + lane]} : Moments{0.0f, 0.0f, 0.0f};
    m.add_warp();
    return m;
}

}  // namespace kmll
