// Helpers shared by the dense (non-spiking) decoder kernels: 32-bit arithmetic around 16- or 32-bit storage.
#pragma once

#include "spk_common.cuh"

template <typename T>
__device__ __forceinline__ T spk_from_float(float v);
template <>
__device__ __forceinline__ float spk_from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 spk_from_float<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Four consecutive elements as floats.  VEC: the address is aligned to four elements; otherwise the elements up
// to `left` are read one by one and the rest is zero.
template <typename T, bool VEC>
__device__ __forceinline__ float4 spk_load4(const T* p, int left) {
    float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
    if (VEC) {
        if (left > 0) {
            if (sizeof(T) == 4) {
                r = *reinterpret_cast<const float4*>(p);
            } else {
                const uint2 u = *reinterpret_cast<const uint2*>(p);
                r.x = __uint_as_float(u.x << 16);
                r.y = __uint_as_float(u.x & 0xffff0000u);
                r.z = __uint_as_float(u.y << 16);
                r.w = __uint_as_float(u.y & 0xffff0000u);
            }
        }
    } else {
        if (left > 0) r.x = spk_to_float<T>(p[0]);
        if (left > 1) r.y = spk_to_float<T>(p[1]);
        if (left > 2) r.z = spk_to_float<T>(p[2]);
        if (left > 3) r.w = spk_to_float<T>(p[3]);
    }
    return r;
}

template <typename T, bool VEC>
__device__ __forceinline__ void spk_store4(T* p, float4 v, int left) {
    if (VEC) {
        if (left > 0) {
            if (sizeof(T) == 4) {
                *reinterpret_cast<float4*>(p) = v;
            } else {
                uint2 u;
                __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
                u.x = *reinterpret_cast<uint32_t*>(&a);
                u.y = *reinterpret_cast<uint32_t*>(&b);
                *reinterpret_cast<uint2*>(p) = u;
            }
        }
    } else {
        if (left > 0) p[0] = spk_from_float<T>(v.x);
        if (left > 1) p[1] = spk_from_float<T>(v.y);
        if (left > 2) p[2] = spk_from_float<T>(v.z);
        if (left > 3) p[3] = spk_from_float<T>(v.w);
    }
}

__device__ __forceinline__ float spk_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Sum of N values per thread over the CTA; every thread gets the totals.  `part` holds N * 32 floats.
template <int N>
__device__ __forceinline__ void spk_block_sum(float (&v)[N], float* part) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = spk_warp_sum(v[i]);
    __syncthreads();  // the previous totals have been read
    if (lane == 0) {
#pragma unroll
        for (int i = 0; i < N; ++i) part[i * 32 + warp] = v[i];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = spk_warp_sum(lane < warps ? part[i * 32 + lane] : 0.0f);
}

__device__ __forceinline__ float spk_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float spk_silu(float x) { return x / (1.0f + expf(-x)); }

// A dense K or V pool: pages of `block_size` rows of `dim_pad` channels, [block][kv head][page].  Tiled pages (16-bit
// elements, dim_pad a multiple of 64, block_size a multiple of 8) hold their rows the way the tensor core's
// 128-byte-swizzled shared-memory tiles do: 64-channel column tiles one after the other, each row of a tile 128 bytes,
// the 16-byte group c of row r stored at group c ^ (r & 7).  A page copied as it is becomes part of an operand tile.
struct SpkPageLayout {
    int heads;
    int block_size;
    int dim_pad;
    int tiled;
};

__device__ __forceinline__ int spk_page_channel(const SpkPageLayout& p, int r, int d) {
    if (!p.tiled) return r * p.dim_pad + d;
    return (d >> 6) * (p.block_size << 6) + (r << 6) + ((((d >> 3) & 7) ^ (r & 7)) << 3) + (d & 7);
}

__device__ __forceinline__ int64_t spk_page_base(const SpkPageLayout& p, int64_t block, int head) {
    return (block * p.heads + head) * static_cast<int64_t>(p.block_size) * p.dim_pad;
}

// Keys per range when a row of `len` keys is cut into at most `splits` ranges: whole groups of 64 keys.
__host__ __device__ __forceinline__ int spk_split_keys(int len, int splits) {
    const int per = (len + splits - 1) / splits;
    return per <= 64 ? 64 : (per + 63) & ~63;
}

// Programmatic dependent launch: wait for the launches before this one, and let the launch after this one be placed.  Both
// do nothing in a kernel that was launched plainly.
__device__ __forceinline__ void spk_grid_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void spk_grid_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

template <typename... Params, typename... Args>
static inline int spk_launch(void (*fn)(Params...), dim3 grid, int threads, size_t bytes, cudaStream_t s, bool overlap, const Args&... args) {
    cudaLaunchConfig_t cfg = {};
    cudaLaunchAttribute attr = {};
    attr.id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr.val.programmaticStreamSerializationAllowed = 1;
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = bytes;
    cfg.stream = s;
    cfg.attrs = &attr;
    cfg.numAttrs = overlap ? 1 : 0;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, fn, args...);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    spk_count_launch();
    return SPK_OK;
}

// A row held by a CTA: V groups of four consecutive elements per thread, group v of thread i at element 4 (i + v * threads).
template <int V>
struct SpkRow {
    float4 g[V];
};

// Threads per row and four-element groups per thread for a row of `width` elements; 0 when too wide.
static inline int spk_row_shape(int64_t width, int* v) {
    const int64_t groups = (width + 3) / 4;
    const int threads = groups <= 128 ? (groups <= 32 ? 32 : groups <= 64 ? 64 : 128) : groups <= 256 ? 128 : groups <= 2048 ? 256 : 1024;
    const int64_t need = (groups + threads - 1) / threads;
    if (need > 8) return 0;
    *v = need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : 8;
    return threads;
}
