// What the kernels of the gated delta rule share: activations in float, the decay, the short convolution.
#pragma once
#include "common.cuh"

namespace mdma {

constexpr int kDeltaMaxDim = 256, kDeltaMaxTaps = 16;

__device__ __forceinline__ float delta_silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float delta_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float delta_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// exp(x), x <= 0, rounded once where it lies near one: a slow channel's decays are multiplied over thousands of tokens,
// and an error of a unit in the last place to one side would add up over them
__device__ __forceinline__ float delta_decay(float x) { return x > -0.5f ? 1.0f + expm1f(x) : expf(x); }
__device__ __forceinline__ float delta_weight(const void* w, int dtype, size_t e) {
    return dtype == kF32 ? reinterpret_cast<const float*>(w)[e] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(w)[e]);
}

// silu of the short convolution of channel c at row t (proj rows hold the inputs at column c; rows before the step's
// first row t0 come from the kept inputs)
__device__ __forceinline__ float delta_conv(const float* __restrict__ proj, int stride, const float* __restrict__ kept,
                                            const void* __restrict__ w, int w_dtype, int taps, int channels, int t, int t0, int c) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int src = t - (taps - 1) + j;
        const float x = src >= t0 ? proj[(size_t)src * stride + c] : kept[(size_t)(taps - 1 + (src - t0)) * channels + c];
        acc = fmaf(delta_weight(w, w_dtype, (size_t)c * taps + j), x, acc);
    }
    return delta_silu(acc);
}

}  // namespace mdma
