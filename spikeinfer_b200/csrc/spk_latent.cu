// Attention over a shared latent: what is cached per token is one normalised latent vector and one rotated key part, which all heads
// read.  Keys and values are never spelled out here: queries go through the heads' key matrices instead, sums of latents through
// their value matrices.
//
//  * latent_prepare_kernel: norms of the query latent and of the cached latent, rotation, page write.
//  * latent_query_kernel / _mma_kernel: W_uk^T q and the rotated query part.
//  * latent_attn_simt_kernel: softmax over the cache rows, every product in 32 bits, any sizes (the tensor-core form is
//    spk_latent_decode.cu).  Key ranges leave (sum, max, denominator).
//  * latent_out_kernel / _mma_kernel: ranges and the sink put together, W_uv, output gate.
#include "spk_latent.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kWarps = 8;
constexpr int kThreads = 32 * kWarps;

__device__ __forceinline__ float2 rot_factor(const float* table, int64_t positions, int half, int64_t pos, int i, uint32_t* status) {
    if (pos < 0 || pos >= positions) {
        spk_flag(status, SPK_STATUS_BAD_SEQ_LEN);
        pos = 0;
    }
    return reinterpret_cast<const float2*>(table)[pos * half + i];
}

// ---- norms, rotation, page write -----------------------------------------------------------------------------------
// WPI warps per (token, part): the query latent, the cached latent, the rotated key part.  One warp for many tokens, a CTA for few.
template <typename T, bool VEC, int WPI>
__global__ void __launch_bounds__(kThreads)
latent_prepare_kernel(const spk_latent_prepare_args a) {
    constexpr int L = 32 * WPI;
    static_assert(WPI == 1 || WPI == kWarps, "a warp or a CTA per item");
    __shared__ float sums[32];
    const int lane = threadIdx.x % L;
    const int parts = a.kv != nullptr ? 3 : 1;
    const int64_t item = static_cast<int64_t>(blockIdx.x) * (kWarps / WPI) + threadIdx.x / L;
    const int64_t t = item / parts;
    if (t >= a.n) return;
    const int part = static_cast<int>(item % parts);
    const SpkPageLayout lay = spk_latent_layout(a.block_size, a.rank_pad, a.rot_pad, a.tiled);
    T* page = nullptr;
    int r = 0;
    if (part > 0) {
        const int64_t slot = a.slot_mapping[t], block = slot / a.block_size;
        if (slot < 0 || block >= a.num_blocks) {
            if (lane == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
            return;
        }
        r = static_cast<int>(slot % a.block_size);
        page = static_cast<T*>(a.pool) + spk_page_base(lay, block, 0);
    }
    if (part == 2) {
        const T* src = static_cast<const T*>(a.kv) + t * a.ld + a.rank;
        const int half = a.rot_dim / 2;
        const int64_t pos = a.positions[t];
        for (int i = lane; i < half; i += L) {
            const float2 f = rot_factor(a.rot_table, a.rot_positions, half, pos, i, a.status);
            const float u = spk_to_float<T>(src[i]), v = spk_to_float<T>(src[i + half]);
            page[spk_latent_channel(lay, r, a.rank_pad + i)] = spk_from_float<T>(u * f.x - v * f.y);
            page[spk_latent_channel(lay, r, a.rank_pad + i + half)] = spk_from_float<T>(v * f.x + u * f.y);
        }
        return;
    }
    const int width = part == 0 ? a.q_rank : a.rank;
    const T* src = part == 0 ? static_cast<const T*>(a.cq) + t * a.ld : static_cast<const T*>(a.kv) + t * a.ld;
    const float* w = part == 0 ? a.w_q : a.w_kv;
    float ss[1] = {0.0f};
#pragma unroll 4
    for (int c = 4 * lane; c < width; c += 4 * L) {
        const float4 x = spk_load4<T, VEC>(src + c, width - c);
        ss[0] += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    }
    if (WPI == 1) ss[0] = spk_warp_sum(ss[0]);
    else spk_block_sum<1>(ss, sums);
    const float inv = 1.0f / sqrtf(ss[0] / static_cast<float>(width) + a.eps);
#pragma unroll 4
    for (int c = 4 * lane; c < width; c += 4 * L) {
        const float4 x = spk_load4<T, VEC>(src + c, width - c), m = spk_load4<float, VEC>(w + c, width - c);
        const float4 y = make_float4(x.x * inv * m.x, x.y * inv * m.y, x.z * inv * m.z, x.w * inv * m.w);
        if (part == 0) {
            spk_store4<T, VEC>(static_cast<T*>(a.cq_out) + t * width + c, y, width - c);
        } else if (VEC) {
            spk_store4<T, VEC>(page + spk_latent_channel(lay, r, c), y, width - c);
        } else {
            const float e[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (c + k < width) page[spk_latent_channel(lay, r, c + k)] = spk_from_float<T>(e[k]);
        }
    }
}

// ---- queries ---------------------------------------------------------------------------------------------------------
// The rotated query part of `rows` tokens of a head, and the padding around it.
template <typename T>
__device__ __forceinline__ void rotate_query(const spk_latent_query_args& a, int h, int64_t t0, int rows) {
    const int half = a.rot_dim / 2, W = a.rank_pad + a.rot_pad;
    for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
        const int64_t t = t0 + i / half;
        const int c = i % half;
        const T* q = static_cast<const T*>(a.q) + (t * a.heads + h) * (a.dim + a.rot_dim) + a.dim;
        T* o = static_cast<T*>(a.out) + (t * a.heads + h) * W + a.rank_pad;
        const float2 f = rot_factor(a.rot_table, a.rot_positions, half, a.positions[t], c, a.status);
        const float u = spk_to_float<T>(q[c]), v = spk_to_float<T>(q[c + half]);
        o[c] = spk_from_float<T>(u * f.x - v * f.y);
        o[c + half] = spk_from_float<T>(v * f.x + u * f.y);
    }
    const int p1 = a.rank_pad - a.rank, pads = p1 + a.rot_pad - a.rot_dim;
    for (int i = threadIdx.x; i < rows * pads; i += blockDim.x) {
        const int c = i % pads;
        static_cast<T*>(a.out)[((t0 + i / pads) * a.heads + h) * W + (c < p1 ? a.rank + c : a.rank_pad + a.rot_dim + c - p1)] = spk_from_float<T>(0.0f);
    }
}

constexpr int kQueryRows = 16;

// CTA = (head, 16 tokens): any sizes.
template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_query_kernel(const spk_latent_query_args a) {
    extern __shared__ float sm[];
    const int h = blockIdx.x;
    const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kQueryRows;
    const int rows = static_cast<int>(min(static_cast<int64_t>(kQueryRows), a.n - t0));
    for (int i = threadIdx.x; i < kQueryRows * a.dim; i += kThreads) {
        const int r = i / a.dim, c = i % a.dim;
        sm[i] = r < rows ? spk_to_float<T>(static_cast<const T*>(a.q)[((t0 + r) * a.heads + h) * (a.dim + a.rot_dim) + c]) : 0.0f;
    }
    __syncthreads();
    const T* w = static_cast<const T*>(a.w_uk) + static_cast<int64_t>(h) * a.dim * a.rank;
    for (int c = threadIdx.x; c < a.rank; c += kThreads) {
        float acc[kQueryRows] = {};
        for (int d = 0; d < a.dim; ++d) {
            const float x = spk_to_float<T>(w[static_cast<int64_t>(d) * a.rank + c]);
#pragma unroll
            for (int r = 0; r < kQueryRows; ++r) acc[r] = fmaf(sm[r * a.dim + d], x, acc[r]);
        }
#pragma unroll
        for (int r = 0; r < kQueryRows; ++r)
            if (r < rows) static_cast<T*>(a.out)[((t0 + r) * a.heads + h) * (a.rank_pad + a.rot_pad) + c] = spk_from_float<T>(acc[r]);
    }
    rotate_query<T>(a, h, t0, rows);
}

// bf16 on the tensor cores: CTA = (head, 128 latent channels, 64 tokens), heads of up to 256 channels; warps 4 (tokens) x 2 (channels).
constexpr int kMmaRows = 64, kMmaCols = 128;

// `rows` x `width` elements into a padded tile, zeros beyond; asynchronous where rows are 16-byte aligned.
__device__ __forceinline__ void fetch_tile(__nv_bfloat16* dst, int stride, const __nv_bfloat16* src, int64_t ld, int rows, int live_rows, int width, int live,
                                           bool vec) {
    const int groups = width / 8;
    for (int i = threadIdx.x; i < rows * groups; i += blockDim.x) {
        const int r = i / groups, c = (i % groups) * 8;
        if (vec) {
            const bool in = r < live_rows && c < live;
            cp_async16(smem_u32(dst + r * stride + c), in ? src + r * ld + c : src, in);
        } else {
#pragma unroll
            for (int k = 0; k < 8; ++k)
                dst[r * stride + c + k] = r < live_rows && c + k < live ? src[r * ld + c + k] : __float2bfloat16_rn(0.0f);
        }
    }
}

__global__ void __launch_bounds__(kThreads)
latent_query_mma_kernel(const spk_latent_query_args a, const int dp, const bool vec_q, const bool vec_w) {
    extern __shared__ __align__(16) uint8_t raw[];
    const int SQ = dp + 8;
    constexpr int SW = kMmaCols + 8;
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(raw);  // [64][dp + 8]
    __nv_bfloat16* ws = qs + kMmaRows * SQ;                      // [dp][128 + 8]
    const int h = blockIdx.x, c0 = blockIdx.y * kMmaCols;
    const int64_t t0 = static_cast<int64_t>(blockIdx.z) * kMmaRows;
    const int rows = static_cast<int>(min(static_cast<int64_t>(kMmaRows), a.n - t0));
    const int64_t ld = static_cast<int64_t>(a.heads) * (a.dim + a.rot_dim);
    if (c0 >= a.rank) {  // the last CTA of a head and token block turns the rotated part
        rotate_query<__nv_bfloat16>(a, h, t0, rows);
        return;
    }
    fetch_tile(ws, SW, static_cast<const __nv_bfloat16*>(a.w_uk) + static_cast<int64_t>(h) * a.dim * a.rank + c0, a.rank, dp, a.dim, kMmaCols,
               a.rank - c0, vec_w);
    fetch_tile(qs, SQ, static_cast<const __nv_bfloat16*>(a.q) + t0 * ld + static_cast<int64_t>(h) * (a.dim + a.rot_dim), ld, (rows + 15) & ~15, rows, dp,
               a.dim, vec_q);
    cp_async_commit();
    cp_async_wait_all();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3, m = lane >> 3, mr = lane & 7;
    const int i0 = (warp & 3) * 16, e0 = (warp >> 2) * 64;
    if (i0 >= rows) return;
    float acc[8][4] = {};
    for (int d = 0; d < dp; d += 16) {
        uint32_t x[4];
        ldsm4(x, smem_u32(qs + (i0 + (lane & 15)) * SQ + d + (lane >> 4) * 8));
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
            uint32_t b[4];
            ldsm4t(b, smem_u32(ws + (d + (m & 1) * 8 + mr) * SW + e0 + n * 8 + (m >> 1) * 8));
            mma16816(acc[n], x, b[0], b[1]);
            mma16816(acc[n + 1], x, b[2], b[3]);
        }
    }
    const int W = a.rank_pad + a.rot_pad;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = i0 + gid + 8 * i;
        if (r >= rows) continue;
        __nv_bfloat16* o = static_cast<__nv_bfloat16*>(a.out) + ((t0 + r) * a.heads + h) * W;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const int c = c0 + e0 + n * 8 + tig * 2;
            if (c + 1 < a.rank && (W & 1) == 0) *reinterpret_cast<uint32_t*>(o + c) = pack_bf16(acc[n][2 * i], acc[n][2 * i + 1]);
            else {
                if (c < a.rank) o[c] = __float2bfloat16_rn(acc[n][2 * i]);
                if (c + 1 < a.rank) o[c + 1] = __float2bfloat16_rn(acc[n][2 * i + 1]);
            }
        }
    }
}

// ---- attention, 32-bit ---------------------------------------------------------------------------------------------------
constexpr int kHeadsPer = kWarps;  // heads of a CTA, one warp each for the scores
constexpr int kKeys = 32;
constexpr int kMaxChan = 4;        // output channels per thread: rank <= 4 * kThreads

template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_attn_simt_kernel(const spk_latent_attn_args a) {
    extern __shared__ float sm[];
    const int64_t t = blockIdx.x;
    const int h0 = blockIdx.y * kHeadsPer, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool prefill = a.token_rows != nullptr;
    const int64_t len = spk_visible_keys(a, t, prefill);
    const int64_t row = prefill ? a.token_rows[t] : t;
    if (len < 0 || len > a.max_blocks * a.block_size || row < 0 || row >= a.table_rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        return;
    }
    const int per = spk_split_keys(static_cast<int>(len), a.splits);
    const int64_t lo = static_cast<int64_t>(blockIdx.z) * per, hi = min(lo + per, len);
    if (lo >= len) return;
    const int W = a.rank + a.rot_dim, WP = a.rank_pad + a.rot_pad, KP = W + 1;
    float* q = sm;                        // [8][W]
    float* k = q + kHeadsPer * W;         // [32][KP]
    float* p = k + kKeys * KP;            // [8][32]
    float* corr = p + kHeadsPer * kKeys;  // [8]
    for (int i = threadIdx.x; i < kHeadsPer * W; i += kThreads) {
        const int h = h0 + i / W, c = i % W;
        q[i] = h < a.heads ? spk_to_float<T>(static_cast<const T*>(a.q)[(t * a.heads + h) * WP + (c < a.rank ? c : a.rank_pad + c - a.rank)]) : 0.0f;
    }
    const SpkPageLayout lay = spk_latent_layout(a.block_size, a.rank_pad, a.rot_pad, a.tiled);
    const int32_t* table = a.tables + row * a.table_stride;
    float acc[kMaxChan][kHeadsPer] = {};
    float top = -INFINITY, den = 0.0f;  // of head h0 + warp
    for (int64_t j0 = lo; j0 < hi; j0 += kKeys) {
        __syncthreads();
        for (int i = threadIdx.x; i < kKeys * W; i += kThreads) {
            const int r = i / W, c = i % W;
            const int64_t j = j0 + r;
            float v = 0.0f;
            if (j < hi) {
                const int64_t block = table[j / a.block_size];
                if (block >= 0 && block < a.num_blocks)
                    v = spk_to_float<T>(static_cast<const T*>(a.pool)[spk_page_base(lay, block, 0) +
                                        spk_latent_channel(lay, static_cast<int>(j % a.block_size), c < a.rank ? c : a.rank_pad + c - a.rank)]);
                else if (c == 0)
                    spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
            }
            k[r * KP + c] = v;
        }
        __syncthreads();
        float s = 0.0f;
        for (int c = 0; c < W; ++c) s = fmaf(q[warp * W + c], k[lane * KP + c], s);
        s = j0 + lane < hi ? s * a.scale : -INFINITY;
        float m = s;
#pragma unroll
        for (int o = 16; o >= 1; o >>= 1) m = fmaxf(m, __shfl_xor_sync(~0u, m, o));
        m = fmaxf(m, top);
        const float e = expf(s - m);
        const float fix = expf(top - m);
        den = den * fix + spk_warp_sum(e);
        top = m;
        p[warp * kKeys + lane] = e;
        if (lane == 0) corr[warp] = fix;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < kMaxChan; ++i) {
            const int c = threadIdx.x + i * kThreads;
            if (c < a.rank) {
#pragma unroll
                for (int h = 0; h < kHeadsPer; ++h) acc[i][h] *= corr[h];
                for (int j = 0; j < kKeys; ++j) {
                    const float v = k[j * KP + c];
#pragma unroll
                    for (int h = 0; h < kHeadsPer; ++h) acc[i][h] = fmaf(p[h * kKeys + j], v, acc[i][h]);
                }
            }
        }
    }
    const int64_t rec = (t * a.splits + blockIdx.z) * a.heads;
    if (lane == 0 && h0 + warp < a.heads) {
        a.stats[2 * (rec + h0 + warp)] = top;
        a.stats[2 * (rec + h0 + warp) + 1] = den;
    }
#pragma unroll
    for (int i = 0; i < kMaxChan; ++i) {
        const int c = threadIdx.x + i * kThreads;
        if (c >= a.rank) break;
#pragma unroll
        for (int h = 0; h < kHeadsPer; ++h)
            if (h0 + h < a.heads) a.partials[(rec + h0 + h) * a.rank + c] = acc[i][h];
    }
}

// ---- output ----------------------------------------------------------------------------------------------------------------
constexpr int kOutRows = 16;

// Weight of every (token, key range) of a head: exp(max_s - M) / (sum of denominators and exp(sink), relative to M); 0 where a range has
// no keys.  wts [kOutRows][splits]; half a warp per token, up to 64 ranges.
__device__ __forceinline__ void range_weights(const spk_latent_out_args& a, int h, int64_t t0, int rows, float* wts) {
    static_assert(2 * kWarps == kOutRows, "half a warp per token");
    const int r = threadIdx.x >> 4, l = threadIdx.x & 15;
    const int64_t t = t0 + r;
    const float sink = a.sink[h];
    const int64_t len = r < rows ? spk_visible_keys(a, t, a.seq_lens == nullptr) : 0;
    const int per = spk_split_keys(static_cast<int>(len), a.splits);
    const int valid = static_cast<int>((len + per - 1) / per);
    float2 st[4];
    float m = sink, den = 0.0f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int s = l + 16 * i;
        st[i] = s < valid ? *reinterpret_cast<const float2*>(a.stats + 2 * ((t * a.splits + s) * a.heads + h)) : make_float2(-INFINITY, 0.0f);
        m = fmaxf(m, st[i].x);
    }
#pragma unroll
    for (int o = 8; o >= 1; o >>= 1) m = fmaxf(m, __shfl_xor_sync(~0u, m, o));
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        st[i].x = expf(st[i].x - m);
        den = fmaf(st[i].y, st[i].x, den);
    }
#pragma unroll
    for (int o = 8; o >= 1; o >>= 1) den += __shfl_xor_sync(~0u, den, o);
    den += expf(sink - m);
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (l + 16 * i < a.splits) wts[r * a.splits + l + 16 * i] = st[i].x / den;
}

// 32-bit, CTA = (head, 16 tokens): any sizes.
__global__ void __launch_bounds__(kThreads)
latent_out_kernel(const spk_latent_out_args a) {
    extern __shared__ float sm[];
    const int h = blockIdx.x, lane = threadIdx.x & 31;
    const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kOutRows;
    const int rows = static_cast<int>(min(static_cast<int64_t>(kOutRows), a.n - t0));
    float* wts = sm;                          // [16][splits]
    float* o = wts + kOutRows * a.splits;     // [16][rank]
    range_weights(a, h, t0, rows, wts);
    __syncthreads();
    for (int i = threadIdx.x; i < kOutRows * a.rank; i += kThreads) {
        const int r = i / a.rank, c = i % a.rank;
        float y = 0.0f;
        for (int s = 0; s < a.splits; ++s) {
            const float w = wts[r * a.splits + s];
            if (w != 0.0f) y = fmaf(w, a.partials[(((t0 + r) * a.splits + s) * a.heads + h) * a.rank + c], y);
        }
        o[i] = y;
    }
    __syncthreads();
    for (int e = threadIdx.x >> 5; e < a.vdim; e += kWarps) {
        const float* w = static_cast<const float*>(a.w_uv) + (static_cast<int64_t>(h) * a.vdim + e) * a.rank;
        float acc[kOutRows] = {};
        for (int c = lane; c < a.rank; c += 32) {
            const float x = (w[c]);
#pragma unroll
            for (int r = 0; r < kOutRows; ++r) acc[r] = fmaf(o[r * a.rank + c], x, acc[r]);
        }
        float mine = 0.0f;
#pragma unroll
        for (int r = 0; r < kOutRows; ++r) {
            const float y = spk_warp_sum(acc[r]);
            if (lane == r) mine = y;
        }
        if (lane < rows) {
            const int64_t c = static_cast<int64_t>(h) * a.vdim + e;
            const float g = (static_cast<const float*>(a.gate)[(t0 + lane) * a.gate_stride + c]);
            static_cast<float*>(a.out)[(t0 + lane) * a.out_stride + c] = (mine * spk_sigmoid(g));
        }
    }
}

// bf16 on the tensor cores: CTA = (head, 16 tokens, 64 value channels); warps 4 (sixteen channels each) x 2 (halves of every 128 latent
// channels).  The ranges' sums are put together with all of a thread's loads in flight at once; the value matrix comes through a ring whose
// first stages are on their way before the launch ahead of this one is waited for.
constexpr int kOutStages = 4, kOutCols = 64, kOutK = 128;

template <bool VEC>
__global__ void __launch_bounds__(kThreads)
latent_out_mma_kernel(const spk_latent_out_args a, const bool vec_w) {
    constexpr int S = kOutK + 8;
    extern __shared__ __align__(16) uint8_t raw[];
    const int chunks = (a.rank + kOutK - 1) / kOutK, SO = chunks * kOutK + 8;
    __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(raw);   // stages of [64][136]
    __nv_bfloat16* os = ws + kOutStages * kOutCols * S;           // [16][rank, padded + 8]
    float* wts = reinterpret_cast<float*>(os + kOutRows * SO);   // [16][splits]
    const int h = blockIdx.x, e0 = blockIdx.z * kOutCols;
    const int64_t t0 = static_cast<int64_t>(blockIdx.y) * kOutRows;
    const int rows = static_cast<int>(min(static_cast<int64_t>(kOutRows), a.n - t0));
    const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(a.w_uv) + (static_cast<int64_t>(h) * a.vdim + e0) * a.rank;
    const int live = min(kOutCols, a.vdim - e0), used = (live + 15) & ~15;
    auto fetch = [&](int c) {
        if (c < chunks) fetch_tile(ws + (c % kOutStages) * kOutCols * S, S, w + c * kOutK, a.rank, used, live, kOutK, a.rank - c * kOutK, vec_w);
        cp_async_commit();
    };
    for (int c = 0; c < kOutStages - 1; ++c) fetch(c);
    spk_grid_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3, m = lane >> 3, mr = lane & 7;
    const int cw = (warp & 3) * 16, kw = (warp >> 2) * 64;
    constexpr int U = 8, K = 64;
    const int r = threadIdx.x >> 4, c4 = (threadIdx.x & 15) * 4;
    const float* part = a.partials + ((t0 + r) * a.splits * a.heads + h) * a.rank + c4;
    const int64_t step = static_cast<int64_t>(a.heads) * a.rank;
    auto sums_of = [&](float4 (&x)[U], int s, int g) {  // a range's sums at 8 x 64 latent channels
#pragma unroll
        for (int u = 0; u < U; ++u) x[u] = spk_load4<float, VEC>(part + s * step + (g + u) * K, r < rows ? a.rank - (g + u) * K - c4 : 0);
    };
    float4 head_sums[U];  // of the first range, on their way while the weights are made
    sums_of(head_sums, 0, 0);
    range_weights(a, h, t0, rows, wts);
    __syncthreads();
    for (int g = 0; g < 2 * chunks; g += U) {
        float4 y[U];
#pragma unroll
        for (int u = 0; u < U; ++u) y[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < rows) {
            for (int s = 0; s < a.splits; ++s) {
                const float f = wts[r * a.splits + s];
                if (f == 0.0f) continue;  // a range without keys was never written
                if (s > 0 || g > 0) sums_of(head_sums, s, g);
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const float4 x = head_sums[u];
                    y[u] = make_float4(fmaf(f, x.x, y[u].x), fmaf(f, x.y, y[u].y), fmaf(f, x.z, y[u].z), fmaf(f, x.w, y[u].w));
                }
            }
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (g + u < 2 * chunks)
                *reinterpret_cast<uint2*>(os + r * SO + (g + u) * K + c4) = make_uint2(pack_bf16(y[u].x, y[u].y), pack_bf16(y[u].z, y[u].w));
    }
    float acc[2][4] = {};
    for (int c = 0; c < chunks; ++c) {
        asm volatile("cp.async.wait_group %0;" ::"n"(kOutStages - 2) : "memory");
        __syncthreads();  // this stage is there, the one before has been read
        fetch(c + kOutStages - 1);
        if (cw >= used) continue;
        const __nv_bfloat16 *ob = os + c * kOutK + kw, *wb = ws + (c % kOutStages) * kOutCols * S + kw;
#pragma unroll
        for (int k = 0; k < 64; k += 16) {
            uint32_t x[4], b[4];
            ldsm4(x, smem_u32(ob + (lane & 15) * SO + k + (lane >> 4) * 8));
            ldsm4(b, smem_u32(wb + (cw + (m >> 1) * 8 + mr) * S + k + (m & 1) * 8));
            mma16816(acc[0], x, b[0], b[1]);
            mma16816(acc[1], x, b[2], b[3]);
        }
    }
    __syncthreads();
    float* half = reinterpret_cast<float*>(ws);  // the second halves' sums [64 channels][17]
    if (kw > 0 && cw < used) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) half[(cw + n * 8 + tig * 2 + (i & 1)) * 17 + gid + 8 * (i >> 1)] = acc[n][i];
    }
    __syncthreads();
    if (kw > 0 || cw >= used) return;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int q = gid + 8 * (i >> 1);
        if (q >= rows) continue;
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int e = cw + n * 8 + tig * 2 + (i & 1);
            if (e >= live) continue;
            const int64_t c = static_cast<int64_t>(h) * a.vdim + e0 + e;
            const float g = __bfloat162float(static_cast<const __nv_bfloat16*>(a.gate)[(t0 + q) * a.gate_stride + c]);
            static_cast<__nv_bfloat16*>(a.out)[(t0 + q) * a.out_stride + c] = __float2bfloat16_rn((acc[n][i] + half[e * 17 + q]) * sigmoid_fast(g));
        }
    }
}

int with_smem(const void* fn, size_t bytes) {
    if (bytes > 227 * 1024) return SPK_ERR_TOO_LARGE;
    if (bytes > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
        if (e != cudaSuccess) return spk_set_cuda_error(e);
    }
    return SPK_OK;
}

template <typename T, bool VEC>
int launch_prepare_form(const spk_latent_prepare_args& a, cudaStream_t s) {
    const int64_t items = a.n * (a.kv != nullptr ? 3 : 1);
    const bool few = items <= 4 * 148;
    const int64_t grid = few ? items : (items + kWarps - 1) / kWarps;
    if (grid > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    if (few) latent_prepare_kernel<T, VEC, kWarps><<<static_cast<unsigned>(grid), kThreads, 0, s>>>(a);
    else latent_prepare_kernel<T, VEC, 1><<<static_cast<unsigned>(grid), kThreads, 0, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T>
int launch_prepare(const spk_latent_prepare_args& a, cudaStream_t s) {
    auto at = [](const void* p, size_t b) { return reinterpret_cast<uintptr_t>(p) % b == 0; };
    const bool vec = a.ld % 4 == 0 && a.q_rank % 4 == 0 && a.rank % 4 == 0 && (a.rank_pad + a.rot_pad) % 4 == 0 && at(a.cq, 4 * sizeof(T)) &&
                     at(a.kv, 4 * sizeof(T)) && at(a.cq_out, 4 * sizeof(T)) && at(a.pool, 16) && at(a.w_q, 16) && at(a.w_kv, 16);
    return vec ? launch_prepare_form<T, true>(a, s) : launch_prepare_form<T, false>(a, s);
}

template <typename T>
int launch_query(const spk_latent_query_args& a, cudaStream_t s) {
    const int64_t tiles = (a.n + kQueryRows - 1) / kQueryRows;
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const size_t bytes = sizeof(float) * kQueryRows * a.dim;
    if (const int rc = with_smem(reinterpret_cast<const void*>(latent_query_kernel<T>), bytes)) return rc;
    latent_query_kernel<T><<<dim3(a.heads, static_cast<unsigned>(tiles)), kThreads, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

bool at16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

int launch_query_mma(const spk_latent_query_args& a, cudaStream_t s) {
    const int dp = (a.dim + 15) & ~15;
    const int64_t tiles = (a.n + kMmaRows - 1) / kMmaRows;
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const size_t bytes = 2 * (static_cast<size_t>(kMmaRows) * (dp + 8) + static_cast<size_t>(dp) * (kMmaCols + 8));
    if (const int rc = with_smem(reinterpret_cast<const void*>(latent_query_mma_kernel), bytes)) return rc;
    const bool vq = at16(a.q) && (a.dim + a.rot_dim) % 8 == 0 && a.dim % 8 == 0, vw = at16(a.w_uk) && a.rank % 8 == 0;
    latent_query_mma_kernel<<<dim3(a.heads, (a.rank + kMmaCols - 1) / kMmaCols + 1, static_cast<unsigned>(tiles)), kThreads, bytes, s>>>(a, dp, vq, vw);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

int launch_out_mma(const spk_latent_out_args& a, cudaStream_t s) {
    const int64_t tiles = (a.n + kOutRows - 1) / kOutRows;
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const size_t bytes = 2 * (static_cast<size_t>(kOutStages) * kOutCols * (kOutK + 8) + kOutRows * ((a.rank + kOutK - 1) / kOutK * kOutK + 8)) + sizeof(float) * kOutRows * a.splits;
    const dim3 grid(a.heads, static_cast<unsigned>(tiles), (a.vdim + kOutCols - 1) / kOutCols);
    const bool vec = a.rank % 4 == 0 && at16(a.partials), vw = at16(a.w_uv) && a.rank % 8 == 0;
    auto* fn = vec ? latent_out_mma_kernel<true> : latent_out_mma_kernel<false>;
    if (const int rc = with_smem(reinterpret_cast<const void*>(fn), bytes)) return rc;
    return spk_launch(fn, grid, kThreads, bytes, s, a.overlap != 0, a, vw);
}

template <typename T>
int launch_simt(const spk_latent_attn_args& a, cudaStream_t s) {
    if (a.rank > kMaxChan * kThreads) return SPK_ERR_UNSUPPORTED;
    const size_t W = a.rank + a.rot_dim;
    const size_t bytes = sizeof(float) * (kHeadsPer * W + kKeys * (W + 1) + kHeadsPer * kKeys + kHeadsPer);
    if (const int rc = with_smem(reinterpret_cast<const void*>(latent_attn_simt_kernel<T>), bytes)) return rc;
    const dim3 grid(static_cast<unsigned>(a.n), (a.heads + kHeadsPer - 1) / kHeadsPer, a.splits);
    latent_attn_simt_kernel<T><<<grid, kThreads, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

int launch_out(const spk_latent_out_args& a, cudaStream_t s) {
    const int64_t tiles = (a.n + kOutRows - 1) / kOutRows;
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const size_t bytes = sizeof(float) * kOutRows * (a.splits + static_cast<size_t>(a.rank));
    if (const int rc = with_smem(reinterpret_cast<const void*>(latent_out_kernel), bytes)) return rc;
    latent_out_kernel<<<dim3(a.heads, static_cast<unsigned>(tiles)), kThreads, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

bool bad_dtype(int dtype) { return dtype != SPK_F32 && dtype != SPK_BF16; }

bool bad_row(int rank, int rot_dim, int rank_pad, int rot_pad, int tiled, int block_size) {
    return rank < 1 || rot_dim < 2 || rot_dim % 2 != 0 || rank_pad < rank || rot_pad < rot_dim || block_size < 1 ||
           (tiled ? rank_pad % 64 != 0 || rot_pad % 64 != 0 || block_size % 8 != 0 : rank_pad != rank || rot_pad != rot_dim);
}

}  // namespace

extern "C" int spk_latent_prepare(const spk_latent_prepare_args* a, void* stream) {
    SpkRange nvtx_range("spk_latent_prepare");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->q_rank < 1 || a->ld < a->q_rank) return SPK_ERR_BAD_SHAPE;
    if (bad_dtype(a->dtype)) return SPK_ERR_BAD_DTYPE;
    if (a->kv != nullptr && (a->num_blocks < 1 || a->rot_positions < 1 || bad_row(a->rank, a->rot_dim, a->rank_pad, a->rot_pad, a->tiled, a->block_size)))
        return SPK_ERR_BAD_SHAPE;
    if (a->n == 0) return SPK_OK;
    if (a->cq == nullptr || a->w_q == nullptr || a->cq_out == nullptr ||
        (a->kv != nullptr && (a->w_kv == nullptr || a->pool == nullptr || a->rot_table == nullptr || a->positions == nullptr || a->slot_mapping == nullptr)))
        return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    return a->dtype == SPK_F32 ? launch_prepare<float>(*a, s) : launch_prepare<__nv_bfloat16>(*a, s);
}

extern "C" int spk_latent_query(const spk_latent_query_args* a, void* stream) {
    SpkRange nvtx_range("spk_latent_query");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->dim < 1 || a->rank < 1 || a->rot_dim < 2 || a->rot_dim % 2 != 0 || a->rank_pad < a->rank ||
        a->rot_pad < a->rot_dim || a->rot_positions < 1)
        return SPK_ERR_BAD_SHAPE;
    if (bad_dtype(a->dtype)) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->w_uk == nullptr || a->out == nullptr || a->rot_table == nullptr || a->positions == nullptr) return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    if (a->dtype == SPK_BF16) return a->dim <= 256 ? launch_query_mma(*a, s) : launch_query<__nv_bfloat16>(*a, s);
    return launch_query<float>(*a, s);
}

extern "C" int spk_latent_attn_splits(int dtype, int rank, int rot_dim, int rank_pad, int rot_pad, int tiled, int block_size, int64_t n, int heads,
                                      int64_t max_keys) {
    (void)rank;
    (void)rot_dim;
    if (n < 1 || heads < 1 || max_keys < 1) return 1;
    if (spk_latent_tensor_form(dtype, rank_pad, rot_pad, tiled, block_size)) return spk_latent_decode_splits(n, heads, max_keys);
    const int64_t ctas = n * ((heads + kHeadsPer - 1) / kHeadsPer);
    const int64_t want = (3 * 148 + ctas - 1) / ctas, most = (max_keys + 255) / 256;
    const int64_t splits = want < most ? want : most;
    return static_cast<int>(splits < 1 ? 1 : splits > 64 ? 64 : splits);
}

extern "C" int spk_latent_attn(const spk_latent_attn_args* a, void* stream) {
    SpkRange nvtx_range("spk_latent_attn");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->n > 0x7fffffffLL || a->heads < 1 || a->splits < 1 || a->splits > 64 || a->num_blocks < 1 || a->max_blocks < 1 ||
        bad_row(a->rank, a->rot_dim, a->rank_pad, a->rot_pad, a->tiled, a->block_size))
        return SPK_ERR_BAD_SHAPE;
    if (bad_dtype(a->dtype)) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->pool == nullptr || a->tables == nullptr || a->partials == nullptr || a->stats == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->token_rows != nullptr ? a->positions == nullptr : a->seq_lens == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->token_rows == nullptr && a->n > a->table_rows) return SPK_ERR_BAD_SHAPE;
    cudaStream_t s = spk_stream(stream);
    if (spk_latent_tensor_form(a->dtype, a->rank_pad, a->rot_pad, a->tiled, a->block_size)) {
        // query rows and pages are read 16 bytes at a time
        if (reinterpret_cast<uintptr_t>(a->q) % 16 != 0 || reinterpret_cast<uintptr_t>(a->pool) % 16 != 0) return SPK_ERR_BAD_STRIDE;
        return spk_latent_decode_launch(*a, s);
    }
    return a->dtype == SPK_F32 ? launch_simt<float>(*a, s) : launch_simt<__nv_bfloat16>(*a, s);
}

extern "C" int spk_latent_out(const spk_latent_out_args* a, void* stream) {
    SpkRange nvtx_range("spk_latent_out");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->vdim < 1 || a->rank < 1 || a->splits < 1 || a->splits > 64) return SPK_ERR_BAD_SHAPE;
    if (bad_dtype(a->dtype)) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->partials == nullptr || a->stats == nullptr || a->sink == nullptr || a->w_uv == nullptr || a->gate == nullptr || a->out == nullptr ||
        (a->seq_lens == nullptr && a->positions == nullptr))
        return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    return a->dtype == SPK_F32 ? launch_out(*a, s) : launch_out_mma(*a, s);
}
