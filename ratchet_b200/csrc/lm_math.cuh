// Scalar functions of the language-model kernels, in f32 with CUDA's accurate library calls, and the rotation every
// kernel with interleaved pairs shares.
#pragma once
#include "common.cuh"

namespace lm {

__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
// tanh form of gelu
__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// cos and sin of position * frequency, times the table's magnitude.  A frequency is the sum of two floats (its f32
// rounding and the remainder): angles of thousands of radians keep their low bits.
__device__ __forceinline__ float2 rotary_angle(const float* freqs, int pairs, int i, uint32_t position, float magnitude) {
    const double a = (double)position * ((double)freqs[i] + (double)freqs[pairs + i]);
    double s, c;
    sincos(a, &s, &c);
    return make_float2((float)c * magnitude, (float)s * magnitude);
}

// Sum over the block; every thread gets the result.  `scratch` holds 32 floats; barriers before and after its use.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
    __syncthreads();
    const int lane = threadIdx.x & 31;
    return warp_sum(lane < (int)(blockDim.x >> 5) ? scratch[lane] : 0.f);
}

}  // namespace lm
