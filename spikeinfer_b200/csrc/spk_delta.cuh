// Shared by the decode and prefill kernels of the gated delta rule.
#pragma once

#include "spk_dense.cuh"

// exp(-exp(a_log) * softplus(x)): one step's decay, and its logarithm.
__device__ __forceinline__ float spk_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float spk_log_decay(float x, float rate) { return -rate * spk_softplus(x); }

struct SpkDeltaShape {
    int qk, channels;  // channels of q (and of k), and of q, k and v together
};
__device__ __forceinline__ SpkDeltaShape spk_delta_shape(const spk_delta_args& a) {
    return {a.kv_heads * a.dim, 2 * a.kv_heads * a.dim + a.heads * a.vdim};
}

// One channel of the short convolution and its activation.  now: the current token's projection; before(s): the one s tokens earlier.
template <typename F>
__device__ __forceinline__ float spk_conv_silu(const float* taps_of_channel, int taps, float now, F before) {
    float y = now * taps_of_channel[taps - 1];
    for (int s = 1; s < taps; ++s) y = fmaf(before(s), taps_of_channel[taps - 1 - s], y);
    return spk_silu(y);
}
