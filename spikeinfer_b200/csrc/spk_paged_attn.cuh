// Internal launchers of the tensor-core forms of the sigmoid-weighted attention (spk_paged_attn.cu dispatches to them).
#pragma once

#include "spk_common.cuh"

// Both pools tiled, 16-bit, at most 128 channels, pages of 16 rows or a larger power of two.
static inline bool spk_attn_tensor_form(int dtype, int k_pad, int v_pad, int k_tiled, int v_tiled, int block_size) {
    return dtype == SPK_BF16 && k_tiled && v_tiled && k_pad <= 128 && v_pad <= 128 && block_size >= 16 && (block_size & (block_size - 1)) == 0;
}

int spk_sigmoid_prefill_launch(const spk_sigmoid_attn_args& a, cudaStream_t s);
int spk_sigmoid_decode_launch(const spk_sigmoid_attn_args& a, cudaStream_t s);
