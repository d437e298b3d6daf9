// Prefill form of the decayed linear attention with bf16 projections on the tensor cores (heads of up to 128 channels).
//
// A stored state every `span` tokens (64 .. 512, chosen by the host for the call's size) keeps the traffic of the
// states small; inside a span a CTA walks 64-token chunks with the running state in its registers:
//  * decay_span_sum_kernel:  U = sum_j decay^(L-1-j) k_j v_j^T of a span of L tokens;
//  * (the scan of spk_decay.cu turns the U of every span into the state the span starts from);
//  * decay_span_out_kernel:  per chunk o_i = decay^(i+1) S^T q_i + sum_{j<=i} decay^(i-j) (q_i.k_j) v_j, then
//    S <- decay^len S + sum_j decay^(len-1-j) k_j v_j^T.
// q, k and v are bf16 after their activation; everything the recurrence adds to them (decayed keys, decayed scores, states)
// is 32-bit and enters a product as a bf16 pair (hi + lo, 16 significant bits), accumulated in 32 bits.
#include "spk_decay.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int C = kDecayChunk;

// x * sigmoid(x): 1 / (1 + 2^(-x log2 e))
__device__ __forceinline__ float silu_fast(float x) { return x * rcp(1.0f + ex2(-1.4426950408889634f * x)); }

// Rows of one head of a chunk on their way into a shared-memory tile [64][W + 8]; rows and channels beyond the data are zero.
// Asynchronous where the rows are 16-byte aligned.  A thread later transforms the very items it copied, so it needs no
// barrier before that, only its own copies to have landed.
template <int W, int NTH>
__device__ __forceinline__ void fetch(__nv_bfloat16* dst, const __nv_bfloat16* src, int64_t ld, int len, int width, bool vec) {
    constexpr int ST = W + 8;
#pragma unroll
    for (int it = 0; it < C * (W / 8) / NTH; ++it) {
        const int i = threadIdx.x + it * NTH;
        const int r = i / (W / 8), c = (i % (W / 8)) * 8;
        if (vec) {
            const bool live = r < len && c < width;
            cp_async16(smem_u32(dst + r * ST + c), live ? src + r * ld + c : src, live);
        } else {
#pragma unroll
            for (int k = 0; k < 8; ++k)
                dst[r * ST + c + k] = r < len && c + k < width ? src[r * ld + c + k] : __float2bfloat16_rn(0.0f);
        }
    }
}

// Activation of a fetched tile, in place (PLAIN) and, times the row's decay weight pw[top - row], as a bf16 pair (hi != NULL).
template <int W, int NTH, bool PLAIN>
__device__ __forceinline__ void activate(__nv_bfloat16* tile, int len, int silu, __nv_bfloat16* hi, __nv_bfloat16* lo, const float* pw, int top) {
    constexpr int ST = W + 8;
#pragma unroll
    for (int it = 0; it < C * (W / 8) / NTH; ++it) {
        const int i = threadIdx.x + it * NTH;
        const int r = i / (W / 8), c = (i % (W / 8)) * 8;
        const uint4 u = *reinterpret_cast<const uint4*>(tile + r * ST + c);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
        float f[8];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            f[2 * k] = __uint_as_float(w[k] << 16);
            f[2 * k + 1] = __uint_as_float(w[k] & 0xffff0000u);
        }
        if (silu) {
#pragma unroll
            for (int k = 0; k < 8; ++k) f[k] = silu_fast(f[k]);
            if (PLAIN)
                *reinterpret_cast<uint4*>(tile + r * ST + c) =
                    make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
        }
        if (hi != nullptr) {
            const float d = r < len ? pw[top - r] : 0.0f;
            uint4 x, y;
            split_bf16(f[0] * d, f[1] * d, x.x, y.x);
            split_bf16(f[2] * d, f[3] * d, x.y, y.y);
            split_bf16(f[4] * d, f[5] * d, x.z, y.z);
            split_bf16(f[6] * d, f[7] * d, x.w, y.w);
            *reinterpret_cast<uint4*>(hi + r * ST + c) = x;
            *reinterpret_cast<uint4*>(lo + r * ST + c) = y;
        }
    }
}

// A warp's part of the [D][V] state when NW warps share it: 16 rows by COLS columns.
template <int CD, int CV, int NW>
struct StateTile {
    static constexpr int D = CD * 64, V = CV * 64, THREADS = 32 * NW;
    static constexpr int GROUPS = D / 16, COLS = V * GROUPS / NW, NT = COLS / 8;
    static_assert(NT % 2 == 0, "pairs of column tiles");
    __device__ static int row0(int warp) { return (warp % GROUPS) * 16; }
    __device__ static int col0(int warp) { return (warp / GROUPS) * COLS; }
};

// acc += K^T V over the chunk's 64 tokens (K as the pair hi + lo)
template <int CD, int CV, int NW>
__device__ __forceinline__ void add_outer(float (&acc)[StateTile<CD, CV, NW>::NT][4], const __nv_bfloat16* hi, const __nv_bfloat16* lo,
                                          const __nv_bfloat16* v, int warp, int lane) {
    using T = StateTile<CD, CV, NW>;
    constexpr int SK = T::D + 8, SV = T::V + 8;
    const int m = lane >> 3, mr = lane & 7;
#pragma unroll
    for (int k0 = 0; k0 < C; k0 += 16) {
        uint32_t ah[4], al[4];
        const int at = (k0 + (m >> 1) * 8 + mr) * SK + T::row0(warp) + (m & 1) * 8;
        ldsm4t(ah, smem_u32(hi + at));
        ldsm4t(al, smem_u32(lo + at));
#pragma unroll
        for (int n = 0; n < T::NT; n += 2) {
            uint32_t b[4];
            ldsm4t(b, smem_u32(v + (k0 + (m & 1) * 8 + mr) * SV + T::col0(warp) + n * 8 + (m >> 1) * 8));
            mma16816(acc[n], ah, b[0], b[1]);
            mma16816(acc[n], al, b[0], b[1]);
            mma16816(acc[n + 1], ah, b[2], b[3]);
            mma16816(acc[n + 1], al, b[2], b[3]);
        }
    }
}

template <int CD, int CV, int NW>
__global__ void __launch_bounds__(32 * NW, 2)
decay_span_sum_kernel(const spk_decay_attn_args a, const bool vec_k, const bool vec_v) {
    using T = StateTile<CD, CV, NW>;
    constexpr int SK = T::D + 8, SV = T::V + 8;
    extern __shared__ __align__(16) __nv_bfloat16 sm[];
    __nv_bfloat16* hi = sm;
    __nv_bfloat16* lo = hi + C * SK;
    __nv_bfloat16* kb = lo + C * SK;      // two stages each of k and v
    __nv_bfloat16* vb = kb + 2 * C * SK;
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const SpkChunk ci = spk_chunk(a, blockIdx.x);
    const float* pw = a.decay_pow + static_cast<int64_t>(h) * (kDecayMaxSpan + 1);
    const __nv_bfloat16* ks = static_cast<const __nv_bfloat16*>(a.k) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim;
    const __nv_bfloat16* vs = static_cast<const __nv_bfloat16*>(a.v) + ci.start * a.ld + static_cast<int64_t>(h) * a.vdim;
    float acc[T::NT][4] = {};
    auto fetch_chunk = [&](int c0, int buf) {
        const int len = min(C, ci.len - c0);
        fetch<T::D, T::THREADS>(kb + buf * C * SK, ks + c0 * a.ld, a.ld, len, a.dim, vec_k);
        fetch<T::V, T::THREADS>(vb + buf * C * SV, vs + c0 * a.ld, a.ld, len, a.vdim, vec_v);
        cp_async_commit();
    };
    fetch_chunk(0, 0);
    for (int c0 = 0, buf = 0; c0 < ci.len; c0 += C, buf ^= 1) {
        const int len = min(C, ci.len - c0);
        cp_async_wait_all();
        __syncthreads();  // the previous chunk's products have read their operands
        activate<T::D, T::THREADS, false>(kb + buf * C * SK, len, a.silu, hi, lo, pw, ci.len - 1 - c0);
        activate<T::V, T::THREADS, true>(vb + buf * C * SV, len, a.silu, nullptr, nullptr, pw, 0);
        if (c0 + C < ci.len) fetch_chunk(c0 + C, buf ^ 1);
        __syncthreads();
        add_outer<CD, CV, NW>(acc, hi, lo, vb + buf * C * SV, warp, lane);
    }
    float* U = a.workspace + (static_cast<int64_t>(blockIdx.x) * a.heads + h) * a.dim * a.vdim;
    const int gid = lane >> 2, tig = lane & 3;
#pragma unroll
    for (int n = 0; n < T::NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int d = T::row0(warp) + gid + (i >> 1) * 8, e = T::col0(warp) + n * 8 + tig * 2 + (i & 1);
            if (d < a.dim && e < a.vdim) U[static_cast<int64_t>(d) * a.vdim + e] = acc[n][i];
        }
}

template <int CD, int CV, int NW>
__global__ void __launch_bounds__(32 * NW, CD * CV == 1 ? 2 : 1)
decay_span_out_kernel(const spk_decay_attn_args a, const bool vec_k, const bool vec_v) {
    using T = StateTile<CD, CV, NW>;
    constexpr int SK = T::D + 8, SV = T::V + 8;
    extern __shared__ __align__(16) __nv_bfloat16 sm[];
    __nv_bfloat16* qb = sm;               // two stages each of q, k and v
    __nv_bfloat16* kb = qb + 2 * C * SK;
    __nv_bfloat16* vb = kb + 2 * C * SK;
    __nv_bfloat16* hi = vb + 2 * C * SV;  // decayed keys
    __nv_bfloat16* lo = hi + C * SK;
    __nv_bfloat16* sh = lo + C * SK;      // state, hi and lo
    __nv_bfloat16* sl = sh + T::D * SV;
    float* pw = reinterpret_cast<float*>(sl + T::D * SV);  // powers 0 .. 64 of this head's decay
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int m = lane >> 3, mr = lane & 7;
    const SpkChunk ci = spk_chunk(a, blockIdx.x);
    for (int i = threadIdx.x; i <= C; i += T::THREADS) pw[i] = a.decay_pow[static_cast<int64_t>(h) * (kDecayMaxSpan + 1) + i];
    const __nv_bfloat16* qs = static_cast<const __nv_bfloat16*>(a.q) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim;
    const __nv_bfloat16* ks = static_cast<const __nv_bfloat16*>(a.k) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim;
    const __nv_bfloat16* vs = static_cast<const __nv_bfloat16*>(a.v) + ci.start * a.ld + static_cast<int64_t>(h) * a.vdim;
    const float* S0 = a.workspace + (static_cast<int64_t>(blockIdx.x) * a.heads + h) * a.dim * a.vdim;
    float S[T::NT][4];
#pragma unroll
    for (int n = 0; n < T::NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int d = T::row0(warp) + gid + (i >> 1) * 8, e = T::col0(warp) + n * 8 + tig * 2 + (i & 1);
            S[n][i] = d < a.dim && e < a.vdim ? S0[static_cast<int64_t>(d) * a.vdim + e] : 0.0f;
        }
    const int i0 = (warp & 3) * 16;                 // this warp's 16 tokens
    constexpr int OC = T::V / (NW / 4), ON = OC / 8;  // and its share of the output columns
    const int e0 = (warp >> 2) * OC;
    auto fetch_chunk = [&](int c0, int buf) {
        const int len = min(C, ci.len - c0);
        fetch<T::D, T::THREADS>(qb + buf * C * SK, qs + c0 * a.ld, a.ld, len, a.dim, vec_k);
        fetch<T::D, T::THREADS>(kb + buf * C * SK, ks + c0 * a.ld, a.ld, len, a.dim, vec_k);
        fetch<T::V, T::THREADS>(vb + buf * C * SV, vs + c0 * a.ld, a.ld, len, a.vdim, vec_v);
        cp_async_commit();
    };
    fetch_chunk(0, 0);
    for (int c0 = 0, buf = 0; c0 < ci.len; c0 += C, buf ^= 1) {
        const int len = min(C, ci.len - c0);
        const bool more = c0 + C < ci.len;
        __nv_bfloat16 *q = qb + buf * C * SK, *k = kb + buf * C * SK, *v = vb + buf * C * SV;
        cp_async_wait_all();
        __syncthreads();  // the previous chunk's reads are done (and pw is there)
        activate<T::D, T::THREADS, true>(q, len, a.silu, nullptr, nullptr, pw, 0);
        activate<T::D, T::THREADS, true>(k, len, a.silu, more ? hi : nullptr, lo, pw, len - 1);
        activate<T::V, T::THREADS, true>(v, len, a.silu, nullptr, nullptr, pw, 0);
        if (more) fetch_chunk(c0 + C, buf ^ 1);
#pragma unroll
        for (int n = 0; n < T::NT; ++n)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int at = (T::row0(warp) + gid + i * 8) * SV + T::col0(warp) + n * 8 + tig * 2;
                uint32_t x, y;
                split_bf16(S[n][2 * i], S[n][2 * i + 1], x, y);
                *reinterpret_cast<uint32_t*>(sh + at) = x;
                *reinterpret_cast<uint32_t*>(sl + at) = y;
            }
        __syncthreads();
        if (i0 < len) {
            float o[ON][4] = {};
            float sc[8][4] = {};
            // S^T q, and the scores against the chunk's keys up to this warp's rows
#pragma unroll
            for (int d0 = 0; d0 < T::D; d0 += 16) {
                uint32_t aq[4];
                ldsm4(aq, smem_u32(q + (i0 + (lane & 15)) * SK + d0 + (lane >> 4) * 8));
#pragma unroll
                for (int n = 0; n < ON; n += 2) {
                    const int at = (d0 + (m & 1) * 8 + mr) * SV + e0 + n * 8 + (m >> 1) * 8;
                    uint32_t b[4];
                    ldsm4t(b, smem_u32(sh + at));
                    mma16816(o[n], aq, b[0], b[1]);
                    mma16816(o[n + 1], aq, b[2], b[3]);
                    ldsm4t(b, smem_u32(sl + at));
                    mma16816(o[n], aq, b[0], b[1]);
                    mma16816(o[n + 1], aq, b[2], b[3]);
                }
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    if (n * 8 <= i0 + 15) {
                        uint32_t b[4];
                        ldsm4(b, smem_u32(k + (n * 8 + (m >> 1) * 8 + mr) * SK + d0 + (m & 1) * 8));
                        mma16816(sc[n], aq, b[0], b[1]);
                        mma16816(sc[n + 1], aq, b[2], b[3]);
                    }
                }
            }
            const int ra = i0 + gid, rb = ra + 8;
            const float wa = pw[ra + 1], wb = pw[rb + 1];
#pragma unroll
            for (int n = 0; n < ON; ++n) {
                o[n][0] *= wa;
                o[n][1] *= wa;
                o[n][2] *= wb;
                o[n][3] *= wb;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {  // 16 keys each
                if (j * 16 > i0 + 15) break;
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const int key = j * 16 + x * 8 + tig * 2;
                    float(&s)[4] = sc[2 * j + x];
                    auto w = [&](float y, int r, int c) { return c <= r ? y * pw[r - c] : 0.0f; };
                    split_bf16(w(s[0], ra, key), w(s[1], ra, key + 1), ph[2 * x], pl[2 * x]);
                    split_bf16(w(s[2], rb, key), w(s[3], rb, key + 1), ph[2 * x + 1], pl[2 * x + 1]);
                }
#pragma unroll
                for (int n = 0; n < ON; n += 2) {
                    uint32_t b[4];
                    ldsm4t(b, smem_u32(v + (j * 16 + (m & 1) * 8 + mr) * SV + e0 + n * 8 + (m >> 1) * 8));
                    mma16816(o[n], ph, b[0], b[1]);
                    mma16816(o[n], pl, b[0], b[1]);
                    mma16816(o[n + 1], ph, b[2], b[3]);
                    mma16816(o[n + 1], pl, b[2], b[3]);
                }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int r = ra + i * 8;
                if (r >= len) continue;
                float* dst = a.out + ((ci.start + c0 + r) * a.heads + h) * a.vdim;
#pragma unroll
                for (int n = 0; n < ON; ++n) {
                    const int e = e0 + n * 8 + tig * 2;
                    if ((a.vdim & 1) == 0) {
                        if (e < a.vdim) *reinterpret_cast<float2*>(dst + e) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
                    } else {
                        if (e < a.vdim) dst[e] = o[n][2 * i];
                        if (e + 1 < a.vdim) dst[e + 1] = o[n][2 * i + 1];
                    }
                }
            }
        }
        if (more) {  // a whole chunk: len == C
            const float w = pw[C];
#pragma unroll
            for (int n = 0; n < T::NT; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) S[n][i] *= w;
            add_outer<CD, CV, NW>(S, hi, lo, v, warp, lane);
        }
    }
}

template <typename F>
int with_smem(F fn, int threads, size_t bytes, cudaStream_t s, const spk_decay_attn_args& a) {
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    auto aligned = [&](const void* p, int width) { return reinterpret_cast<uintptr_t>(p) % 16 == 0 && a.ld % 8 == 0 && width % 8 == 0; };
    const bool vk = aligned(a.k, a.dim) && (a.q == nullptr || aligned(a.q, a.dim)), vv = aligned(a.v, a.vdim);
    fn<<<dim3(a.n_chunks, a.heads), threads, bytes, s>>>(a, vk, vv);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <int CD, int CV>
int sums(const spk_decay_attn_args& a, cudaStream_t s) {
    constexpr size_t bytes = 2 * C * (4 * (CD * 64 + 8) + 2 * (CV * 64 + 8));
    return with_smem(decay_span_sum_kernel<CD, CV, 8>, 256, bytes, s, a);
}

template <int CD, int CV>
int outputs(const spk_decay_attn_args& a, cudaStream_t s) {
    constexpr size_t bytes = 2 * C * (6 * (CD * 64 + 8) + 2 * (CV * 64 + 8)) + 4 * CD * 64 * (CV * 64 + 8) + 4 * (C + 8);
    static_assert(bytes <= 227 * 1024, "shared memory");
    constexpr int NW = CD * CV == 4 ? 16 : 8;  // one CTA of sixteen warps per SM, or two of eight
    return with_smem(decay_span_out_kernel<CD, CV, NW>, 32 * NW, bytes, s, a);
}

}  // namespace

int spk_decay_mma_sums(const spk_decay_attn_args& a, cudaStream_t s) {
    if (a.dim <= 64) return a.vdim <= 64 ? sums<1, 1>(a, s) : sums<1, 2>(a, s);
    return a.vdim <= 64 ? sums<2, 1>(a, s) : sums<2, 2>(a, s);
}

int spk_decay_mma_outputs(const spk_decay_attn_args& a, cudaStream_t s) {
    if (a.dim <= 64) return a.vdim <= 64 ? outputs<1, 1>(a, s) : outputs<1, 2>(a, s);
    return a.vdim <= 64 ? outputs<2, 1>(a, s) : outputs<2, 2>(a, s);
}
