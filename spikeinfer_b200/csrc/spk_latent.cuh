// Shared by the forms of the latent attention: layout of the cache rows and dispatch between the 32-bit and the tensor-core kernels.
#pragma once

#include "spk_dense.cuh"

// A cache row: `rank` latent channels at 0, rot_dim rotated channels at rank_pad; one pool head.  Tiled pages hold eight rows after the other,
// and of eight rows 64 channels after the other: 1 KB atoms of 8 x 128 bytes, the 16-byte group g of row r at group g ^ (r & 7).  So any run
// of whole pages laid end to end is one operand of the tensor core, with all channels, whichever of rows and channels it sums over.
__host__ __device__ __forceinline__ SpkPageLayout spk_latent_layout(int block_size, int rank_pad, int rot_pad, int tiled) {
    return SpkPageLayout{1, block_size, rank_pad + rot_pad, tiled};
}

__device__ __forceinline__ int spk_latent_channel(const SpkPageLayout& p, int r, int d) {
    if (!p.tiled) return r * p.dim_pad + d;
    return (r >> 3) * (p.dim_pad << 3) + ((d >> 6) << 9) + ((r & 7) << 6) + ((((d >> 3) & 7) ^ (r & 7)) << 3) + (d & 7);
}

// Tiled 16-bit pool of at most 512 latent and 64 rotated channels, pages of 16 rows or a larger power of two.
static inline bool spk_latent_tensor_form(int dtype, int rank_pad, int rot_pad, int tiled, int block_size) {
    return dtype == SPK_BF16 && tiled && rank_pad <= 512 && rot_pad == 64 && block_size >= 16 && (block_size & (block_size - 1)) == 0;
}

int spk_latent_decode_splits(int64_t n, int heads, int64_t max_keys);
int spk_latent_decode_launch(const spk_latent_attn_args& a, cudaStream_t s);

// Keys token t of a call sees: position + 1 in a prefill, the row's length in a decode step (0 for rows that sit out).
template <typename Args>
__device__ __forceinline__ int64_t spk_visible_keys(const Args& a, int64_t t, bool prefill) {
    if (prefill) return a.positions[t] + 1;
    return a.active == nullptr || a.active[t] == 1 ? a.seq_lens[t] : 0;
}
