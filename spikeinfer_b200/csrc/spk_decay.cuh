// Shared by the 32-bit and the tensor-core forms of the decayed linear attention.
#pragma once

#include "spk_dense.cuh"

constexpr int kDecayChunk = 64;       // tokens of one masked product
constexpr int kDecayMaxSpan = 512;    // most tokens between two stored states (and highest tabulated power)

struct SpkChunk {
    int64_t start;
    int len, seq, index;
};

__device__ __forceinline__ SpkChunk spk_chunk(const spk_decay_attn_args& a, int c) {
    const int4 e = reinterpret_cast<const int4*>(a.chunks)[c];
    return {e.x, e.y, e.z, e.w};
}

// 16-bit projections and heads of at most 128 channels run on the tensor cores.
static inline bool spk_decay_tensor_form(int dtype, int dim, int vdim) { return dtype == SPK_BF16 && dim <= 128 && vdim <= 128; }

int spk_decay_mma_sums(const spk_decay_attn_args& a, cudaStream_t s);
int spk_decay_mma_outputs(const spk_decay_attn_args& a, cudaStream_t s);
