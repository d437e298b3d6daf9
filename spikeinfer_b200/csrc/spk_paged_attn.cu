// Dense paged attention with element-wise (sigmoid) key weights: the K/V write and the 32-bit form of the product.
//
//  * qk_prepare_kernel: per (token, head) rotary embedding on the first channels, division by the head's root mean square,
//    q to a dense buffer, k and v into the sequence's pages.  One launch for q, k and v.
//  * sigmoid_attn_simt_kernel: out = sum_j sigmoid(scale q.k_j + bias_h) v_j over the visible keys, every product in
//    32 bits; any head sizes, prefill tiles and decode rows alike.
// A weight depends on its own key alone, so there is no running maximum and no denominator, and sums over
// different key ranges simply add up.
#include "spk_paged_attn.cuh"
#include "spk_dense.cuh"

namespace {

constexpr int kWarps = 8;
constexpr int kThreads = 32 * kWarps;

// ---- rotary embedding, unit norm, page write ---------------------------------------------------------------
// One warp per (token, head slot); slots are the query heads, then the key heads, then the value heads.
template <typename T>
__global__ void __launch_bounds__(kThreads)
qk_prepare_kernel(const spk_qk_prepare_args a) {
    extern __shared__ float sm[];
    spk_grid_release();  // a launch that does not need this one's results may be placed beside it
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int slots = a.heads + 2 * a.kv_heads;
    const int64_t item = static_cast<int64_t>(blockIdx.x) * kWarps + warp;
    const int64_t t = item / slots;
    if (t >= a.n) return;
    const int s = static_cast<int>(item % slots);
    const bool is_q = s < a.heads;
    const bool is_v = s >= a.heads + a.kv_heads;
    const int width = is_v ? a.vdim : a.dim;
    const T* src;
    if (is_q) src = static_cast<const T*>(a.q) + t * a.ld + static_cast<int64_t>(s) * a.dim;
    else if (!is_v) src = static_cast<const T*>(a.k) + t * a.ld + static_cast<int64_t>(s - a.heads) * a.dim;
    else src = static_cast<const T*>(a.v) + t * a.ld + static_cast<int64_t>(s - a.heads - a.kv_heads) * a.vdim;

    T* page = nullptr;
    int r = 0;
    SpkPageLayout lay{a.kv_heads, a.block_size, is_v ? a.v_pad : a.k_pad, is_v ? a.v_tiled : a.k_tiled};
    if (!is_q) {
        const int64_t slot = a.slot_mapping[t];
        const int64_t block = slot / a.block_size;
        if (slot < 0 || block >= a.num_blocks) {
            if (lane == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
            return;
        }
        r = static_cast<int>(slot % a.block_size);
        const int g = is_v ? s - a.heads - a.kv_heads : s - a.heads;
        page = static_cast<T*>(is_v ? a.v_pool : a.k_pool) + spk_page_base(lay, block, g);
    }
    if (is_v) {
        for (int c = lane; c < width; c += 32) page[spk_page_channel(lay, r, c)] = src[c];
        return;
    }
    float* x = sm + warp * a.dim;
    for (int c = lane; c < width; c += 32) x[c] = spk_to_float<T>(src[c]);
    __syncwarp();
    const int half = a.rot_table != nullptr ? a.rot_dims / 2 : 0;
    if (half > 0) {
        int64_t pos = a.positions[t];
        if (pos < 0 || pos >= a.rot_positions) {
            if (lane == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
            pos = 0;
        }
        const float2* cs = reinterpret_cast<const float2*>(a.rot_table) + pos * half;
        for (int i = lane; i < half; i += 32) {
            const float2 f = cs[i];
            const float u = x[i], w = x[i + half];
            x[i] = u * f.x - w * f.y;
            x[i + half] = w * f.x + u * f.y;
        }
        __syncwarp();
    }
    float ss = 0.0f;
    for (int c = lane; c < width; c += 32) ss = fmaf(x[c], x[c], ss);
    ss = spk_warp_sum(ss);
    const float inv = a.unit_norm ? 1.0f / sqrtf(ss / static_cast<float>(width) + a.eps) : 1.0f;
    if (is_q) {
        T* o = static_cast<T*>(a.q_out) + (t * a.heads + s) * a.k_pad;
        for (int c = lane; c < a.k_pad; c += 32) o[c] = spk_from_float<T>(c < width ? x[c] * inv : 0.0f);
    } else {
        for (int c = lane; c < width; c += 32) page[spk_page_channel(lay, r, c)] = spk_from_float<T>(x[c] * inv);
    }
}

// The same for bf16 heads of DIM = 64 or 128 channels (q, k and v alike) in tiled pools, eight channels (16 bytes) per lane: a
// rotated pair's channels sit in two lanes of the head.  rot_dims is a multiple of 16.
template <int DIM>
__global__ void __launch_bounds__(kThreads)
qk_prepare_vec_kernel(const spk_qk_prepare_args a) {
    spk_grid_release();
    constexpr int LK = DIM / 8;  // lanes per head: 8 or 16, so a warp holds whole heads
    const int lanes_t = (a.heads + 2 * a.kv_heads) * LK;
    const int64_t item = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x;
    const int64_t t = item / lanes_t;
    const bool in = t < a.n;
    const int l = static_cast<int>(item % lanes_t);
    const int qk_lanes = (a.heads + a.kv_heads) * LK;
    const bool is_v = l >= qk_lanes;
    const int s = (is_v ? l - qk_lanes : l) / LK;  // head slot (q heads, then k heads) or v head
    const int sub = l % LK;
    const bool is_q = !is_v && s < a.heads;
    const __nv_bfloat16* src = is_v ? static_cast<const __nv_bfloat16*>(a.v) + t * a.ld + s * DIM + sub * 8
                             : is_q ? static_cast<const __nv_bfloat16*>(a.q) + t * a.ld + s * DIM + sub * 8
                                    : static_cast<const __nv_bfloat16*>(a.k) + t * a.ld + (s - a.heads) * DIM + sub * 8;
    const uint4 u = in ? *reinterpret_cast<const uint4*>(src) : make_uint4(0u, 0u, 0u, 0u);
    float x[8];
    {
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            x[2 * k] = __uint_as_float(w[k] << 16);
            x[2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
        }
    }
    const int half = a.rot_table != nullptr ? a.rot_dims / 2 : 0;
    const int hl = half / 8;  // lanes of each half of the rotated channels
    const bool low = sub < hl, turn = !is_v && sub < 2 * hl;
    float y[8];
    const int partner = (threadIdx.x & 31) + (turn ? (low ? hl : -hl) : 0);
#pragma unroll
    for (int k = 0; k < 8; ++k) y[k] = __shfl_sync(~0u, x[k], partner);
    if (turn && in) {
        int64_t pos = a.positions[t];
        if (pos < 0 || pos >= a.rot_positions) {
            spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
            pos = 0;
        }
        const float4* cs = reinterpret_cast<const float4*>(reinterpret_cast<const float2*>(a.rot_table) + pos * half + (low ? sub : sub - hl) * 8);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float4 f = cs[k];  // (cos, sin) of two pairs
            const float s0 = low ? -f.y : f.y, s1 = low ? -f.w : f.w;
            x[2 * k] = x[2 * k] * f.x + y[2 * k] * s0;
            x[2 * k + 1] = x[2 * k + 1] * f.z + y[2 * k + 1] * s1;
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < 8; ++k) ss = fmaf(x[k], x[k], ss);
#pragma unroll
    for (int o = LK / 2; o >= 1; o >>= 1) ss += __shfl_xor_sync(~0u, ss, o);
    if (!in) return;
    const float inv = a.unit_norm ? 1.0f / sqrtf(ss / static_cast<float>(DIM) + a.eps) : 1.0f;
    uint4 r = u;
    if (!is_v) {
        uint32_t w[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(x[2 * k] * inv, x[2 * k + 1] * inv);
            w[k] = *reinterpret_cast<const uint32_t*>(&b);
        }
        r = make_uint4(w[0], w[1], w[2], w[3]);
    }
    if (is_q) {
        *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.q_out) + (t * a.heads + s) * DIM + sub * 8) = r;
        return;
    }
    const int64_t slot = a.slot_mapping[t];
    const int64_t block = slot / a.block_size;
    if (slot < 0 || block >= a.num_blocks) {
        spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    const SpkPageLayout lay{a.kv_heads, a.block_size, DIM, 1};
    __nv_bfloat16* page = static_cast<__nv_bfloat16*>(is_v ? a.v_pool : a.k_pool) + spk_page_base(lay, block, is_v ? s : s - a.heads);
    *reinterpret_cast<uint4*>(page + spk_page_channel(lay, static_cast<int>(slot % a.block_size), sub * 8)) = r;
}

template <int DIM>
int launch_prepare_vec(const spk_qk_prepare_args& a, cudaStream_t s) {
    const int64_t items = a.n * (a.heads + 2 * static_cast<int64_t>(a.kv_heads)) * (DIM / 8);
    const int64_t grid = (items + kThreads - 1) / kThreads;
    if (grid > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    qk_prepare_vec_kernel<DIM><<<static_cast<unsigned>(grid), kThreads, 0, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

// ---- attention, 32-bit -----------------------------------------------------------------------------------------
constexpr int kTileQ = 16;
constexpr int kTileK = 32;
constexpr int kMaxCols = 16;  // output columns per thread and query tile: vdim <= 16 * kThreads / kTileQ = 256

template <typename T>
__global__ void __launch_bounds__(kThreads)
sigmoid_attn_simt_kernel(const spk_sigmoid_attn_args a) {
    extern __shared__ float sm[];
    const int h = blockIdx.y;
    const int g = h / (a.heads / a.kv_heads);
    int64_t t0;
    int nq, row;
    int64_t pos0;
    if (a.tiles != nullptr) {
        const int4 e = reinterpret_cast<const int4*>(a.tiles)[blockIdx.x];  // first token, tokens, row, position of the first
        t0 = e.x; nq = e.y; row = e.z; pos0 = e.w;
    } else {
        t0 = row = blockIdx.x;
        nq = 1;
        pos0 = static_cast<int64_t>(a.seq_lens[row]) - 1;
    }
    const int dim = a.dim, vdim = a.vdim;
    T* out = static_cast<T*>(a.out) + t0 * a.out_stride + static_cast<int64_t>(h) * vdim;
    bool live = a.tiles != nullptr || a.active == nullptr || a.active[row] == 1;
    if (live && (pos0 < 0 || pos0 + nq > a.max_blocks * a.block_size || row < 0 || row >= a.table_rows)) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        live = false;
    }
    if (!live) {
        for (int i = threadIdx.x; i < nq * vdim; i += kThreads) out[(i / vdim) * a.out_stride + i % vdim] = spk_from_float<T>(0.0f);
        return;
    }
    float* q = sm;                         // [kTileQ][dim]
    float* k = q + kTileQ * dim;           // [kTileK][dim + 1]
    float* v = k + kTileK * (dim + 1);     // [kTileK][vdim]
    float* p = v + kTileK * vdim;          // [kTileQ][kTileK]
    for (int i = threadIdx.x; i < kTileQ * dim; i += kThreads) {
        const int r = i / dim, c = i % dim;
        q[i] = r < nq ? spk_to_float<T>(static_cast<const T*>(a.q)[((t0 + r) * a.heads + h) * a.k_pad + c]) : 0.0f;
    }
    const SpkPageLayout kl{a.kv_heads, a.block_size, a.k_pad, a.k_tiled}, vl{a.kv_heads, a.block_size, a.v_pad, a.v_tiled};
    const int32_t* table = a.tables + static_cast<int64_t>(row) * a.table_stride;
    const float bias = a.head_bias[h];
    const int cols = kTileQ * vdim;
    float acc[kMaxCols];
#pragma unroll
    for (int i = 0; i < kMaxCols; ++i) acc[i] = 0.0f;
    const int64_t keys = pos0 + nq;
    for (int64_t j0 = 0; j0 < keys; j0 += kTileK) {
        __syncthreads();
        for (int i = threadIdx.x; i < kTileK * (dim + vdim); i += kThreads) {
            const int r = i / (dim + vdim), c = i % (dim + vdim);
            const int64_t j = j0 + r;
            float val = 0.0f;
            if (j < keys) {
                const int64_t block = table[j / a.block_size];
                const int slot = static_cast<int>(j % a.block_size);
                if (block >= 0 && block < a.num_blocks) {
                    val = c < dim ? spk_to_float<T>(static_cast<const T*>(a.k_pool)[spk_page_base(kl, block, g) + spk_page_channel(kl, slot, c)])
                                  : spk_to_float<T>(static_cast<const T*>(a.v_pool)[spk_page_base(vl, block, g) + spk_page_channel(vl, slot, c - dim)]);
                } else if (c == 0) {
                    spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
                }
            }
            if (c < dim) k[r * (dim + 1) + c] = val;
            else v[r * vdim + c - dim] = val;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < kTileQ * kTileK; i += kThreads) {
            const int r = i / kTileK, c = i % kTileK;
            float s = 0.0f;
            for (int d = 0; d < dim; ++d) s = fmaf(q[r * dim + d], k[c * (dim + 1) + d], s);
            p[i] = r < nq && j0 + c <= pos0 + r ? spk_sigmoid(fmaf(s, a.scale, bias)) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kMaxCols; ++i) {
            const int e = threadIdx.x + i * kThreads;
            if (e < cols) {
                const int r = e / vdim, c = e % vdim;
                float s = 0.0f;
                for (int j = 0; j < kTileK; ++j) s = fmaf(p[r * kTileK + j], v[j * vdim + c], s);
                acc[i] += s;
            }
        }
    }
#pragma unroll
    for (int i = 0; i < kMaxCols; ++i) {
        const int e = threadIdx.x + i * kThreads;
        if (e < cols && e / vdim < nq) out[(e / vdim) * a.out_stride + e % vdim] = spk_from_float<T>(acc[i] * a.out_scale);
    }
}

template <typename T>
int launch_simt(const spk_sigmoid_attn_args& a, cudaStream_t s) {
    if (kTileQ * a.vdim > kMaxCols * kThreads) return SPK_ERR_UNSUPPORTED;
    const size_t bytes = sizeof(float) * (static_cast<size_t>(kTileQ) * a.dim + kTileK * (a.dim + 1) + kTileK * a.vdim + kTileQ * kTileK);
    if (bytes > 227 * 1024) return SPK_ERR_UNSUPPORTED;
    if (bytes > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(sigmoid_attn_simt_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
        if (e != cudaSuccess) return spk_set_cuda_error(e);
    }
    const dim3 grid(a.tiles != nullptr ? a.n_tiles : static_cast<int>(a.n), a.heads);
    sigmoid_attn_simt_kernel<T><<<grid, kThreads, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

extern "C" int spk_qk_prepare(const spk_qk_prepare_args* a, void* stream) {
    SpkRange nvtx_range("spk_qk_prepare");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->kv_heads < 1 || a->dim < 1 || a->vdim < 1 || a->block_size < 1 || a->num_blocks < 1 ||
        a->k_pad < a->dim || a->v_pad < a->vdim || a->heads % a->kv_heads != 0)
        return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (((a->k_tiled && (a->k_pad % 64 != 0 || a->block_size % 8 != 0)) || (a->v_tiled && (a->v_pad % 64 != 0 || a->block_size % 8 != 0))))
        return SPK_ERR_UNSUPPORTED;
    if (a->rot_table != nullptr && (a->rot_dims < 2 || a->rot_dims % 2 != 0 || a->rot_dims > a->dim || a->rot_positions < 1 || a->positions == nullptr))
        return SPK_ERR_BAD_SHAPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->k == nullptr || a->v == nullptr || a->q_out == nullptr || a->k_pool == nullptr || a->v_pool == nullptr ||
        a->slot_mapping == nullptr)
        return SPK_ERR_NULL_POINTER;
    auto at16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    if (a->dtype == SPK_BF16 && a->k_tiled && a->v_tiled && a->dim == a->vdim && (a->dim == 64 || a->dim == 128) && a->k_pad == a->dim &&
        a->v_pad == a->vdim && a->ld % 8 == 0 && (a->rot_table == nullptr || (a->rot_dims % 16 == 0 && at16(a->rot_table))) && at16(a->q) &&
        at16(a->k) && at16(a->v) && at16(a->q_out) && at16(a->k_pool) && at16(a->v_pool))
        return a->dim == 64 ? launch_prepare_vec<64>(*a, spk_stream(stream)) : launch_prepare_vec<128>(*a, spk_stream(stream));
    const int64_t items = a->n * (a->heads + 2 * static_cast<int64_t>(a->kv_heads));
    const int64_t grid = (items + kWarps - 1) / kWarps;
    const size_t bytes = sizeof(float) * kWarps * a->dim;
    if (grid > 0x7fffffffLL || bytes > 48 * 1024) return SPK_ERR_TOO_LARGE;
    cudaStream_t s = spk_stream(stream);
    if (a->dtype == SPK_F32) qk_prepare_kernel<float><<<static_cast<unsigned>(grid), kThreads, bytes, s>>>(*a);
    else qk_prepare_kernel<__nv_bfloat16><<<static_cast<unsigned>(grid), kThreads, bytes, s>>>(*a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

extern "C" int spk_sigmoid_attn_tile_tokens(int dtype, int k_pad, int v_pad, int k_tiled, int v_tiled, int block_size) {
    return spk_attn_tensor_form(dtype, k_pad, v_pad, k_tiled, v_tiled, block_size) ? 128 : kTileQ;
}

extern "C" int spk_sigmoid_attn_splits(int dtype, int k_pad, int v_pad, int k_tiled, int v_tiled, int block_size, int64_t n, int heads,
                                       int kv_heads, int64_t max_keys) {
    if (n < 1 || heads < 1 || kv_heads < 1 || max_keys < 1 || !spk_attn_tensor_form(dtype, k_pad, v_pad, k_tiled, v_tiled, block_size)) return 0;
    const int64_t ctas = n * kv_heads * ((heads / kv_heads + 15) / 16);
    const int64_t want = (3 * 148 + ctas - 1) / ctas, most = (max_keys + 255) / 256;
    const int64_t splits = want < most ? want : most;
    return static_cast<int>(splits < 1 ? 1 : splits > 64 ? 64 : splits);
}

extern "C" int spk_sigmoid_attn(const spk_sigmoid_attn_args* a, void* stream) {
    SpkRange nvtx_range("spk_sigmoid_attn");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->kv_heads < 1 || a->dim < 1 || a->vdim < 1 || a->block_size < 1 || a->num_blocks < 1 ||
        a->max_blocks < 1 || a->k_pad < a->dim || a->v_pad < a->vdim || a->heads % a->kv_heads != 0 || a->heads > 65535)
        return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->k_pool == nullptr || a->v_pool == nullptr || a->tables == nullptr || a->head_bias == nullptr ||
        (a->out == nullptr && (a->partials == nullptr || a->tiles != nullptr)))
        return SPK_ERR_NULL_POINTER;
    if (a->tiles == nullptr && a->seq_lens == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->tiles != nullptr && (a->n_tiles < 1 || reinterpret_cast<uintptr_t>(a->tiles) % 16 != 0)) return SPK_ERR_BAD_SHAPE;
    if (a->tiles == nullptr && a->n > a->table_rows) return SPK_ERR_BAD_SHAPE;
    cudaStream_t s = spk_stream(stream);
    if (spk_attn_tensor_form(a->dtype, a->k_pad, a->v_pad, a->k_tiled, a->v_tiled, a->block_size)) {
        // tiles of the tensor-core form's own size; q rows and pages are read 16 bytes at a time
        if (reinterpret_cast<uintptr_t>(a->q) % 16 != 0 || reinterpret_cast<uintptr_t>(a->k_pool) % 16 != 0 ||
            reinterpret_cast<uintptr_t>(a->v_pool) % 16 != 0)
            return SPK_ERR_BAD_STRIDE;
        if (a->tiles != nullptr) return spk_sigmoid_prefill_launch(*a, s);
        if (a->partials != nullptr) return a->splits < 1 ? SPK_ERR_BAD_SHAPE : spk_sigmoid_decode_launch(*a, s);
    } else if (a->partials != nullptr) {
        return SPK_ERR_UNSUPPORTED;
    }
    return a->dtype == SPK_F32 ? launch_simt<float>(*a, s) : launch_simt<__nv_bfloat16>(*a, s);
}
