// Sorted token matrices of the experts: rows grouped by expert, segments starting at multiples of eight rows.
#pragma once

#include "spk_dense.cuh"

constexpr int kExpertAlign = 8;      // rows a segment's start is aligned to: one swizzle atom
constexpr int kExpertTailRows = 256;  // rows a tile may touch beyond the last segment

// Operand tiles of a matrix of `rows` rows: 64-column tiles one after the other, each row of a tile 128 bytes, the 16-byte group g of
// row r at group g ^ (r & 7).  `rows` is a multiple of eight.
__host__ __device__ __forceinline__ int spk_operand_columns(int width) { return (width + 63) & ~63; }
__device__ __forceinline__ int64_t spk_operand_at(int64_t rows, int64_t r, int c) {
    return (static_cast<int64_t>(c >> 6) * rows + r) * 64 + ((((c >> 3) & 7) ^ static_cast<int>(r & 7)) << 3) + (c & 7);
}

// The tile-th run of TN rows over all experts' segments: which expert, its first row and how many rows.  Called by a whole warp;
// false when there are fewer tiles.
template <int TN>
__device__ __forceinline__ bool spk_find_tile(const int32_t* segs, int experts, int tile, int& expert, int64_t& row0, int& rows) {
    const int lane = threadIdx.x & 31;
    int before = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
        const int e = e0 + lane;
        const int2 sg = e < experts ? reinterpret_cast<const int2*>(segs)[e] : make_int2(0, 0);
        const int mine = (sg.y + TN - 1) / TN;
        int upto = mine;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(~0u, upto, o);
            if (lane >= o) upto += up;
        }
        const int first = before + upto - mine;
        const unsigned hit = __ballot_sync(~0u, tile >= first && tile < first + mine);
        if (hit != 0) {
            const int src = __ffs(hit) - 1;
            const int k = tile - __shfl_sync(~0u, first, src);
            expert = e0 + src;
            row0 = static_cast<int64_t>(__shfl_sync(~0u, sg.x, src)) + static_cast<int64_t>(k) * TN;
            rows = min(TN, __shfl_sync(~0u, sg.y, src) - k * TN);
            return true;
        }
        before += __shfl_sync(~0u, upto, 31);
    }
    return false;
}

// Tiles of TN rows that `pairs` rows over `experts` segments can need at most.
static inline int64_t spk_most_tiles(int64_t pairs, int experts, int tn) {
    const int64_t used = pairs < experts ? pairs : experts;
    return used + (pairs - used) / tn;
}

int spk_experts_mma(const spk_experts_args& a, cudaStream_t s);
