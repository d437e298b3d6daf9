// Shared by the decode and prefill kernels of the gated delta rule.
#pragma once

#include "spk_dense.cuh"

// exp(-exp(a_log) * softplus(x)): one step's decay, and its logarithm.
__device__ __forceinline__ float spk_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float spk_log_decay(float x, float rate) { return -rate * spk_softplus(x); }

// The decay itself, exp(-rate * softplus(x)), in few instructions.  log(1 + z) = 2 artanh(w), w = z / (2 + z) <= 1/3 for z = exp(-|x|) <= 1: eight
// terms of artanh's series leave a relative error below 3e-8.
__device__ __forceinline__ float spk_decay_series(float x, float rate) {
    constexpr float kLog2e = 1.4426950408889634f;
    float z, r, y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(z) : "f"(-kLog2e * fabsf(x)));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(2.0f + z));
    const float w = z * r, w2 = w * w;
    float s = fmaf(w2, 1.0f / 15.0f, 1.0f / 13.0f);
    s = fmaf(w2, s, 1.0f / 11.0f);
    s = fmaf(w2, s, 1.0f / 9.0f);
    s = fmaf(w2, s, 1.0f / 7.0f);
    s = fmaf(w2, s, 1.0f / 5.0f);
    s = fmaf(w2, s, 1.0f / 3.0f);
    s = fmaf(w2, s, 1.0f);
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(-kLog2e * rate * fmaf(2.0f * w, s, fmaxf(x, 0.0f))));
    return y;
}

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

// One channel's last inputs of a portion into the row's ring.
template <typename T>
__device__ __forceinline__ void spk_commit_conv(const spk_delta_args& a, const int4& po, const SpkDeltaShape& sh, const void* src, int64_t c, int at) {
    float* ring = a.conv_state + static_cast<int64_t>(po.z) * a.taps * sh.channels;
    const int keep = min(a.taps, po.y);
    for (int b = 0; b < keep; ++b) {
        const int64_t t = po.x + po.y - 1 - b;
        ring[((po.w + po.y - 1 - b) % a.taps) * sh.channels + at] = spk_to_float<T>(static_cast<const T*>(src)[t * a.ld + c]);
    }
}

constexpr int kDeltaChunk = 16;  // tokens per chunk of the prefill forms

// 16-bit projections and heads of at most 128 channels run on the tensor cores.
static inline bool spk_delta_tensor_form(int dtype, int dim, int vdim) { return dtype == SPK_BF16 && dim <= 128 && vdim <= 128; }
int64_t spk_delta_mma_bytes(int n_chunks, int heads, int dim, int vdim);
int spk_delta_mma_launch(const spk_delta_args& a, float* outputs, cudaStream_t s);
