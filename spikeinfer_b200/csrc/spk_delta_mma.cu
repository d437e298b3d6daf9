// Prefill form of the gated delta rule on the tensor cores: bf16 projections, heads of up to 128 key and 128 value channels.
//
// Over a chunk of 16 tokens, with G_t the product of the decays up to token t and the state S at the chunk's start,
//   A[t, s] = k_t . (k_s * G_t / G_s)  (s < t),   B[t, s] = q_t . (k_s * G_t / G_s)  (s <= t),
//   (1 + beta A) W = beta (k * G),   (1 + beta A) U0 = beta v        (forward substitution, one column per thread)
//   u = U0 - W S,   o = (q * G) S + B u,   S <- G_16 S + (k * G_16 / G)^T u.
// Ratios of G are running products of decays, never quotients: any decay is exact, a vanishing one included.
//  * delta_chunk_kernel, all chunks at once: convolutions, unit vectors, decays, A, B, and the operands W, q G, k G_16 / G, B, U0 of
//    the recurrence, laid out as the shared-memory image they become.
//  * delta_chain_kernel, chunk after chunk: a warp owns sixteen value columns; S^T lives in its registers as the accumulators of the
//    update, which are, as they are, the A operand of the next chunk's products (and u^T that of the update).  One bulk copy brings a
//    chunk's operands.
// 32-bit quantities enter a product as bf16 pairs (hi + lo, three MMAs), sums are 32-bit.
#include "spk_delta.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int C = kDeltaChunk;
constexpr int kThreads = 256;

// A chunk's operands in bytes from the image's start; SD elements per row of W, Q and K.
template <int DP>
struct Image {
    static constexpr int SD = DP + 8, SB = 24, SU = 64 + 4;  // of U0, 64 columns at a time
    static constexpr int kRows = C * SD * 2;                                              // bytes of one of the six matrices
    static constexpr int kWh = 0, kWl = kRows, kQh = 2 * kRows, kQl = 3 * kRows, kKh = 4 * kRows, kKl = 5 * kRows;
    static constexpr int kBh = 6 * kRows, kBl = kBh + C * SB * 2, kE = kBl + C * SB * 2;  // B, then G_16
    static constexpr int kU = kE + DP * 4;                                                // U0 [vdim / 64][C][SU], 32-bit
};

// Lanes L = 0 .. 31 end up with the sum over the warp of v[L].
__device__ __forceinline__ float transpose_sum(float (&v)[32]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int o = 16; o >= 1; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
            v[i] = keep + __shfl_xor_sync(~0u, send, o);
        }
    }
    return v[0];
}

// Channel c of a projection over the chunk's tokens through its convolution and silu into dst[t * stride]; zero beyond the chunk.
template <int TAPS>
__device__ __forceinline__ void conv_channel(const spk_delta_args& a, const int4& po, int64_t t0, int len, const void* src, int64_t c, const float* ring,
                                             int channels, int at, const float* w, float* dst, int stride) {
    const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(src) + t0 * a.ld + c;
    const int taps = TAPS > 0 ? TAPS : a.taps;
    const int before = static_cast<int>(t0 - po.x);  // tokens of the portion ahead of the chunk
    auto raw = [&](int j) {  // projection of token t0 + j, j < 0 reaching back into the portion, then into the ring
        if (j >= 0 || before + j >= 0) return __bfloat162float(p[j * a.ld]);
        const int pos = po.w + before + j;
        return pos >= 0 ? ring[(pos % taps) * channels + at] : 0.0f;
    };
    if (TAPS > 0) {
        float f[TAPS > 0 ? TAPS : 1], win[TAPS > 0 ? TAPS : 1], x[C];
#pragma unroll
        for (int i = 0; i < TAPS; ++i) f[i] = w[c * TAPS + i];
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i) win[i + 1] = raw(i - (TAPS - 1));
#pragma unroll
        for (int t = 0; t < C; ++t) x[t] = t < len ? __bfloat162float(p[t * a.ld]) : 0.0f;
#pragma unroll
        for (int t = 0; t < C; ++t) {
#pragma unroll
            for (int i = 0; i < TAPS - 1; ++i) win[i] = win[i + 1];
            win[TAPS - 1] = x[t];
            float y = 0.0f;
#pragma unroll
            for (int i = 0; i < TAPS; ++i) y = fmaf(win[i], f[i], y);
            dst[t * stride] = t < len ? y * sigmoid_fast(y) : 0.0f;
        }
    } else {
        for (int t = 0; t < C; ++t) {
            float y = 0.0f;
            if (t < len)
                for (int i = 0; i < taps; ++i) y = fmaf(raw(t - (taps - 1 - i)), w[c * taps + i], y);
            dst[t * stride] = t < len ? y * sigmoid_fast(y) : 0.0f;
        }
    }
}

// The same for channels c and c + 1 over half a chunk (eight tokens from `first`), two channels per access; every pair of channels aligned.
template <int TAPS>
__device__ __forceinline__ void conv_pair(const spk_delta_args& a, const int4& po, int64_t t0, int len, int first, const void* src, int64_t c, const float* ring,
                                          int channels, int at, const float* w, float* dst, int stride) {
    if (first >= len) {  // no token of this half, and none between it and the last one to look back at
#pragma unroll
        for (int t = 0; t < C / 2; ++t) *reinterpret_cast<float2*>(dst + (first + t) * stride) = make_float2(0.0f, 0.0f);
        return;
    }
    const __nv_bfloat16* p = static_cast<const __nv_bfloat16*>(src) + (t0 + first) * a.ld + c;
    const int before = static_cast<int>(t0 - po.x) + first;  // tokens of the portion ahead of the half
    uint32_t x[C / 2];
    float f0[TAPS], f1[TAPS], w0[TAPS], w1[TAPS];
#pragma unroll
    for (int t = 0; t < C / 2; ++t) x[t] = first + t < len ? *reinterpret_cast<const uint32_t*>(p + t * a.ld) : 0u;
    if (TAPS == 4) {  // two channels' filters are two 16-byte loads
        const float4 u0 = *reinterpret_cast<const float4*>(w + c * 4), u1 = *reinterpret_cast<const float4*>(w + c * 4 + 4);
        f0[0] = u0.x; f0[1 % TAPS] = u0.y; f0[2 % TAPS] = u0.z; f0[3 % TAPS] = u0.w;
        f1[0] = u1.x; f1[1 % TAPS] = u1.y; f1[2 % TAPS] = u1.z; f1[3 % TAPS] = u1.w;
    } else {
#pragma unroll
        for (int i = 0; i < TAPS; ++i) {
            f0[i] = w[c * TAPS + i];
            f1[i] = w[(c + 1) * TAPS + i];
        }
    }
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
        const int j = i - (TAPS - 1), pos = po.w + before + j;
        float y0 = 0.0f, y1 = 0.0f;
        if (before + j >= 0) {
            const uint32_t u = *reinterpret_cast<const uint32_t*>(p + j * a.ld);
            y0 = __uint_as_float(u << 16);
            y1 = __uint_as_float(u & 0xffff0000u);
        } else if (pos >= 0) {
            y0 = ring[(pos % TAPS) * channels + at];
            y1 = ring[(pos % TAPS) * channels + at + 1];
        }
        w0[i + 1] = y0;
        w1[i + 1] = y1;
    }
#pragma unroll
    for (int t = 0; t < C / 2; ++t) {
        float y0 = 0.0f, y1 = 0.0f;
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i) {
            w0[i] = w0[i + 1];
            w1[i] = w1[i + 1];
            y0 = fmaf(w0[i], f0[i], y0);
            y1 = fmaf(w1[i], f1[i], y1);
        }
        w0[TAPS - 1] = __uint_as_float(x[t] << 16);
        w1[TAPS - 1] = __uint_as_float(x[t] & 0xffff0000u);
        y0 = fmaf(w0[TAPS - 1], f0[TAPS - 1], y0);
        y1 = fmaf(w1[TAPS - 1], f1[TAPS - 1], y1);
        const bool in = first + t < len;
        *reinterpret_cast<float2*>(dst + (first + t) * stride) = make_float2(in ? y0 * sigmoid_fast(y0) : 0.0f, in ? y1 * sigmoid_fast(y1) : 0.0f);
    }
}

// A and B by running products of the decays: warp w of eight walks from tokens w and 15 - w to the chunk's end, fifteen steps in all, and
// sums 32 products over its lanes.
template <int DP>
__device__ __noinline__ void pair_products(const float* q, const float* k, const float* g, const float* qi, const float* ki, float (*A)[C], float (*B)[C],
                                           int warp, int lane) {
    constexpr int SQ = DP + 8, P2 = DP / 64;  // channel pairs per lane
    const int s0 = warp, s1 = C - 1 - warp;
    uint64_t x[P2], y[P2], z[P2];
    float part[32];
    auto load = [&](uint64_t (&r)[P2], const float* m, int t) {
        if (P2 == 2) {
            const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(m + t * SQ + 4 * lane);
            r[0] = f.x;
            r[P2 - 1] = f.y;
        } else {
            r[0] = *reinterpret_cast<const uint64_t*>(m + t * SQ + 2 * lane);
        }
    };
    auto dot = [&](const uint64_t (&p)[P2], const uint64_t (&r)[P2]) {
        uint64_t s = f2_mul(p[0], r[0]);
        if (P2 == 2) s = f2_fma(p[P2 - 1], r[P2 - 1], s);
        float a0, a1;
        f2_unpack(s, a0, a1);
        return a0 + a1;
    };
    load(x, k, s1);
    load(y, q, s1);
    part[31] = dot(x, y);
    load(x, k, s0);
    load(y, q, s0);
    part[30] = dot(x, y);
    const int first = C - 1 - s0;  // steps that start from s0
#pragma unroll
    for (int i = 0; i < C - 1; ++i) {
        if (i == first) load(x, k, s1);
        const int t = i < first ? s0 + 1 + i : s1 + 1 + i - first;
        load(y, g, t);
#pragma unroll
        for (int j = 0; j < P2; ++j) x[j] = f2_mul(x[j], y[j]);
        load(y, k, t);
        load(z, q, t);
        part[i] = dot(x, y);
        part[C - 1 + i] = dot(x, z);
    }
    const float total = transpose_sum(part);
    if (lane < 2 * (C - 1)) {
        const int i = lane < C - 1 ? lane : lane - (C - 1);
        const int s = i < first ? s0 : s1, t = i < first ? s0 + 1 + i : s1 + 1 + i - first;
        if (lane < C - 1) A[t][s] = total * ki[t] * ki[s];
        else B[t][s] = total * qi[t] * ki[s];
    } else {
        const int s = lane == 30 ? s0 : s1;
        B[s][s] = total * qi[s] * ki[s];
    }
}

// CTA = (chunk, head).
template <int DP, int TAPS>
__global__ void __launch_bounds__(kThreads, 4)
delta_chunk_kernel(const spk_delta_args a, const int64_t image_bytes, const int vp, const bool pairs) {
    using I = Image<DP>;
    constexpr int SQ = DP + 8;   // row stride: MMA fragments read without bank conflicts
    constexpr float kSmallest = 1e-30f;
    extern __shared__ __align__(16) float sm[];
    float* q = sm;               // [C][SQ]
    float* k = q + C * SQ;
    float* g = k + C * SQ;       // decays
    float* G = g + C * SQ;       // their products from the chunk's start
    float* v = G + C * SQ;       // [C][vp]
    __shared__ __align__(16) float A[C][C], B[C][C];
    __shared__ float qi[C], ki[C], beta[C];
    const int h = blockIdx.y, grp = h / (a.heads / a.kv_heads), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int4 ch = reinterpret_cast<const int4*>(a.chunks)[blockIdx.x];  // first token, tokens, portion, index
    const int4 po = reinterpret_cast<const int4*>(a.portions)[ch.z];      // first token, tokens, row, tokens before
    if (po.z < 0 || po.z >= a.state_rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    const int64_t t0 = ch.x;
    const int len = ch.y, dim = a.dim, vdim = a.vdim;
    const SpkDeltaShape sh = spk_delta_shape(a);
    const float* ring = a.conv_state + static_cast<int64_t>(po.z) * a.taps * sh.channels;
    // the decays' raw values are on their way while the convolutions run, a channel of k, q or v per thread and turn
    constexpr int RAW = C * DP / kThreads;
    float raw_a[RAW];
#pragma unroll
    for (int j = 0; j < RAW; ++j) {
        const int i = threadIdx.x + j * kThreads, t = i / DP, d = i % DP;
        raw_a[j] = d < dim && t < len ? __bfloat162float(static_cast<const __nv_bfloat16*>(a.a)[(t0 + t) * a.ld2 + static_cast<int64_t>(h) * dim + d]) : 0.0f;
    }
    const int my_d = threadIdx.x % DP;  // kThreads is a multiple of DP: one channel for all of a thread's values
    const float bias = my_d < dim ? a.dt_bias[static_cast<int64_t>(h) * dim + my_d] : 0.0f, rate = expf(a.a_log[h]);
    const bool paired = TAPS > 0 && pairs;
    if constexpr (TAPS > 0) {  // two channels and half the tokens per thread and turn
        for (int i = paired ? threadIdx.x : 2 * DP + vp; i < 2 * DP + vp; i += kThreads) {
            const int kind = i < DP ? 0 : i < 2 * DP ? 1 : 2;  // k, q, v: uniform over a warp
            const int j = i - kind * DP, half = kind == 2 ? vp / 2 : DP / 2, c = 2 * (j % half), first = j / half * (C / 2);
            const int width = kind == 2 ? vdim : dim, stride = kind == 2 ? vp : SQ, head = kind == 2 ? h : grp;
            float* dst = (kind == 0 ? k : kind == 1 ? q : v) + c;
            if (c < width) {
                conv_pair<TAPS>(a, po, t0, len, first, kind == 0 ? a.k : kind == 1 ? a.q : a.v, static_cast<int64_t>(head) * width + c, ring, sh.channels,
                                (kind == 0 ? sh.qk : kind == 1 ? 0 : 2 * sh.qk) + head * width + c, kind == 0 ? a.conv_k : kind == 1 ? a.conv_q : a.conv_v, dst, stride);
            } else {
#pragma unroll
                for (int t = 0; t < C / 2; ++t) *reinterpret_cast<float2*>(dst + (first + t) * stride) = make_float2(0.0f, 0.0f);
            }
        }
    }
    for (int i = paired ? 2 * DP + vp : threadIdx.x; i < 2 * DP + vp; i += kThreads) {
        const int kind = i < DP ? 0 : i < 2 * DP ? 1 : 2;  // k, q, v: uniform over a warp
        const int c = i - kind * DP, width = kind == 2 ? vdim : dim, stride = kind == 2 ? vp : SQ;
        float* dst = (kind == 0 ? k : kind == 1 ? q : v) + c;
        if (c < width) {
            const int head = kind == 2 ? h : grp;
            conv_channel<TAPS>(a, po, t0, len, kind == 0 ? a.k : kind == 1 ? a.q : a.v, static_cast<int64_t>(head) * width + c, ring, sh.channels,
                               (kind == 0 ? sh.qk : kind == 1 ? 0 : 2 * sh.qk) + head * width + c, kind == 0 ? a.conv_k : kind == 1 ? a.conv_q : a.conv_v, dst, stride);
        } else {
#pragma unroll
            for (int t = 0; t < C; ++t) dst[t * stride] = 0.0f;
        }
    }
#pragma unroll
    for (int j = 0; j < RAW; ++j) {
        const int t = (threadIdx.x + j * kThreads) / DP;
        g[t * SQ + my_d] = my_d < dim && t < len ? spk_decay_series(raw_a[j] + bias, rate) : 1.0f;
    }
    if (threadIdx.x < C)
        beta[threadIdx.x] = static_cast<int>(threadIdx.x) < len ? spk_sigmoid(__bfloat162float(static_cast<const __nv_bfloat16*>(a.b)[(t0 + threadIdx.x) * a.ld + h])) : 0.0f;
    __syncthreads();
    float run = 1.0f;
    if (threadIdx.x < DP) {
#pragma unroll
        for (int t = 0; t < C; ++t) {
            run *= g[t * SQ + threadIdx.x];
            G[t * SQ + threadIdx.x] = run;
        }
    }
    // norms: two tokens per warp
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int t = 2 * warp + i;
        float x = 0.0f, y = 0.0f;
#pragma unroll
        for (int j = 0; j < DP / 32; ++j) {
            const float a1 = q[t * SQ + lane + 32 * j], b1 = k[t * SQ + lane + 32 * j];
            x = fmaf(a1, a1, x);
            y = fmaf(b1, b1, y);
        }
        x = spk_warp_sum(x);
        y = spk_warp_sum(y);
        if (lane == 0) {
            qi[t] = 1.0f / (sqrtf(x + 1e-6f) * sqrtf(static_cast<float>(dim)));
            ki[t] = 1.0f / sqrtf(y + 1e-6f);
        }
    }
    const bool steep = __syncthreads_or(run < kSmallest);  // a channel all but forgets within the chunk
    uint8_t* image = static_cast<uint8_t*>(a.workspace) + (static_cast<int64_t>(blockIdx.x) * a.heads + h) * image_bytes;
    // lanes trade tokens in pairs, so that a store carries two channels
    const bool odd = lane & 1;
    auto put = [&](int t, int d, float x0, float x1, int hi_at, int lo_at) {  // column d's values at tokens t and t + 1
        const float got = __shfl_xor_sync(~0u, odd ? x0 : x1, 1);
        uint32_t hi, lo;
        split_bf16(odd ? got : x0, odd ? x1 : got, hi, lo);
        const int at = ((t + (odd ? 1 : 0)) * I::SD + (d & ~1)) * 2;
        *reinterpret_cast<uint32_t*>(image + hi_at + at) = hi;
        *reinterpret_cast<uint32_t*>(image + lo_at + at) = lo;
    };
    // A and B.  Steep chunks: products of running decays by all warps.  Otherwise A = (k G) (k / G)^T and B = (q G) (k / G)^T on the tensor
    // cores, a warp each (nothing below 1e-30 is divided by), beside the other warps' operands.
    if (steep) {
        pair_products<DP>(q, k, g, qi, ki, A, B, warp, lane);
    } else if (warp < 2) {
        const float *left = warp == 0 ? k : q, *li = warp == 0 ? ki : qi;
        const int gid = lane >> 2, tig = lane & 3;
        float acc[2][4] = {}, cross[2][4] = {};
#pragma unroll 2
        for (int d0 = 0; d0 < DP; d0 += 16) {
            uint32_t lh[4], ll[4], rh[4], rl[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {  // left rows gid (+ 8), channels + 8; right: tokens gid (+ 8) of k / G
                const int at = (gid + 8 * (i & 1)) * SQ + d0 + 2 * tig + 8 * (i >> 1);
                const float2 x = *reinterpret_cast<const float2*>(left + at), y = *reinterpret_cast<const float2*>(k + at), z = *reinterpret_cast<const float2*>(G + at);
                split_bf16(x.x * z.x, x.y * z.y, lh[i], ll[i]);
                split_bf16(__fdividef(y.x, z.x), __fdividef(y.y, z.y), rh[i], rl[i]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                mma16816(acc[n], lh, rh[n], rh[2 + n]);
                mma16816(cross[n], lh, rl[n], rl[2 + n]);
                mma16816(cross[n], ll, rh[n], rh[2 + n]);
            }
        }
        float(*M)[C] = warp == 0 ? A : B;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int t = gid + 8 * (i >> 1), s = n * 8 + tig * 2 + (i & 1);
                M[t][s] = s <= t ? (acc[n][i] + cross[n][i]) * li[t] * ki[s] : 0.0f;
            }
    }
    {  // a column of q G or k G_16 / G per thread and turn
        const int skip = steep ? 0 : 64;
        for (int i = static_cast<int>(threadIdx.x) - skip; i < 2 * DP; i += kThreads - skip) {
            if (i < 0) break;  // uniform over a warp
            if (i < DP) {
#pragma unroll
                for (int t = 0; t < C; t += 2)
                    put(t, i, q[t * SQ + i] * qi[t] * G[t * SQ + i], q[(t + 1) * SQ + i] * qi[t + 1] * G[(t + 1) * SQ + i], I::kQh, I::kQl);
                reinterpret_cast<float*>(image + I::kE)[i] = G[(C - 1) * SQ + i];
            } else {
                const int d = i - DP;
                float rest = 1.0f;  // product of the decays behind the token
#pragma unroll
                for (int t = C - 2; t >= 0; t -= 2) {
                    const float y1 = k[(t + 1) * SQ + d] * ki[t + 1] * rest;
                    rest *= g[(t + 1) * SQ + d];
                    const float y0 = k[t * SQ + d] * ki[t] * rest;
                    rest *= g[t * SQ + d];
                    put(t, d, y0, y1, I::kKh, I::kKl);
                }
            }
        }
    }
    __syncthreads();
    if (threadIdx.x < C * C / 2) {
        const int t = threadIdx.x >> 3, s = (threadIdx.x & 7) * 2;
        uint32_t hi, lo;
        split_bf16(s <= t ? B[t][s] : 0.0f, s + 1 <= t ? B[t][s + 1] : 0.0f, hi, lo);
        *reinterpret_cast<uint32_t*>(image + I::kBh + (t * I::SB + s) * 2) = hi;
        *reinterpret_cast<uint32_t*>(image + I::kBl + (t * I::SB + s) * 2) = lo;
    }
    // forward substitution, a column of W or U0 per thread and turn
    for (int i = threadIdx.x; i < DP + vp; i += kThreads) {
        const bool is_w = i < DP;  // uniform over a warp
        const int e = i - DP;
        float w[C];
#pragma unroll
        for (int t = 0; t < C; ++t) {
            float x = is_w ? k[t * SQ + i] * ki[t] * G[t * SQ + i] : v[t * vp + e];
#pragma unroll
            for (int s4 = 0; s4 < t; s4 += 4) {
                const float4 f = *reinterpret_cast<const float4*>(&A[t][s4]);
                x = fmaf(-f.x, w[s4], x);
                if (s4 + 1 < t) x = fmaf(-f.y, w[s4 + 1], x);
                if (s4 + 2 < t) x = fmaf(-f.z, w[s4 + 2], x);
                if (s4 + 3 < t) x = fmaf(-f.w, w[s4 + 3], x);
            }
            w[t] = beta[t] * x;
        }
        if (is_w) {
#pragma unroll
            for (int t = 0; t < C; t += 2) put(t, i, w[t], w[t + 1], I::kWh, I::kWl);
        } else {
            float* u = reinterpret_cast<float*>(image + I::kU) + (e >> 6) * C * I::SU + (e & 63);
#pragma unroll
            for (int t = 0; t < C; ++t) u[t * I::SU] = w[t];
        }
    }
}

// CTA = (NW * 16 value columns of a head, head, portion); warp NW copies.
constexpr int NW = 4;  // a warp per scheduler: the chain is bound by its MMAs

template <int DP>
struct Chain {
    static constexpr int kHead = Image<DP>::kU, kU = C * Image<DP>::SU * 4;
    static constexpr int kStage = (kHead + kU + 127) & ~127;
    static constexpr int NS = DP == 64 ? 4 : 3;
    static constexpr int kBytes = NS * kStage + 128 + 2 * NS * 8;
};

template <int DP>
__global__ void __launch_bounds__(32 * NW + 32, 2)
delta_chain_kernel(const spk_delta_args a, const int64_t image_bytes, float* __restrict__ outputs) {
    using I = Image<DP>;
    using K = Chain<DP>;
    constexpr int NS = K::NS;
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 127) & ~uintptr_t(127));
    uint64_t* full = reinterpret_cast<uint64_t*>(base + NS * K::kStage);
    uint64_t* empty = full + NS;
    __shared__ int abort_flag;
    volatile int* abort = &abort_flag;
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int4 po = reinterpret_cast<const int4*>(a.portions)[blockIdx.z];  // first token, tokens, row, tokens before
    const int4 sq = reinterpret_cast<const int4*>(a.seqs)[blockIdx.z];      // first chunk, chunks, row, tokens before
    if (po.z < 0 || po.z >= a.state_rows) {  // flagged by the chunks
        spk_grid_wait();
        return;
    }
    const int v0 = blockIdx.x * NW * 16;
    const int columns = min(NW * 16, a.vdim - v0);
    if (threadIdx.x == 0) {
        for (int i = 0; i < NS; ++i) {
            mbar_init(smem_u32(full + i), 1);
            mbar_init(smem_u32(empty + i), NW);
        }
        abort_flag = 0;
    }
    fence_async_shared();
    __syncthreads();
    if (warp == NW) {
        spk_grid_wait();  // placed ahead of the chunks' end: their operands are complete from here on
        if (lane == 0) {
            int issued = 0;
            for (int c = 0; c < sq.y; ++c) {
                const int st = c % NS;
                if (c >= NS && !mbar_wait(smem_u32(empty + st), ((c / NS) - 1) & 1, abort)) break;
                const uint8_t* src = static_cast<const uint8_t*>(a.workspace) + (static_cast<int64_t>(sq.x + c) * a.heads + h) * image_bytes;
                const uint32_t bar = smem_u32(full + st), dst = smem_u32(base + st * K::kStage);
                mbar_expect(bar, K::kHead + K::kU);
                bulk_load(dst, src, K::kHead, bar);
                bulk_load(dst + K::kHead, src + I::kU + blockIdx.x * K::kU, K::kU, bar);
                issued = c + 1;
            }
            if (*abort != 0) {  // copies in flight land before the CTA's shared memory is given up
                for (int c = issued > NS ? issued - NS : 0; c < issued; ++c) mbar_wait(smem_u32(full + c % NS), (c / NS) & 1);
                spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
            }
        }
    } else {
        const int gid = lane >> 2, tig = lane & 3, m = lane >> 3, mr = lane & 7;
        constexpr int NT = DP / 8;
        const int dim = a.dim, vdim = a.vdim, v1 = v0 + warp * 16 + gid;
        const bool live = warp * 16 < columns;  // a warp without columns only keeps the ring going
        float* state = a.state + (static_cast<int64_t>(po.z) * a.heads + h) * dim * vdim;
        float S[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int d = n * 8 + tig * 2 + (i & 1), e = v1 + (i >> 1) * 8;
                S[n][i] = live && po.w > 0 && d < dim && e < vdim ? state[static_cast<int64_t>(d) * vdim + e] : 0.0f;
            }
        spk_grid_wait();  // and the convolutions' past has been read
        for (int c = 0; c < sq.y; ++c) {
            const int st = c % NS;
            if (!__all_sync(~0u, mbar_wait(smem_u32(full + st), (c / NS) & 1, abort))) break;
            const uint8_t* im = base + st * K::kStage;
            const uint32_t at = smem_u32(im);
            if (live) {
                // u^T and o^T: columns (tokens) 0-7 and 8-15, main and cross terms apart
                float u[2][4] = {}, uc[2][4] = {}, o[2][4] = {}, oc[2][4] = {};
                const uint32_t row = ((m >> 1) * 8 + mr) * I::SD * 2 + (m & 1) * 16;
#pragma unroll
                for (int j = 0; j < DP / 16; ++j) {
                    uint32_t sh[4], sl[4], bh[4], bl[4];
                    split_bf16(S[2 * j][0], S[2 * j][1], sh[0], sl[0]);
                    split_bf16(S[2 * j][2], S[2 * j][3], sh[1], sl[1]);
                    split_bf16(S[2 * j + 1][0], S[2 * j + 1][1], sh[2], sl[2]);
                    split_bf16(S[2 * j + 1][2], S[2 * j + 1][3], sh[3], sl[3]);
                    ldsm4(bh, at + I::kWh + row + j * 32);
                    ldsm4(bl, at + I::kWl + row + j * 32);
                    mma16816(u[0], sh, bh[0], bh[1]);
                    mma16816(u[1], sh, bh[2], bh[3]);
                    mma16816(uc[0], sh, bl[0], bl[1]);
                    mma16816(uc[1], sh, bl[2], bl[3]);
                    mma16816(uc[0], sl, bh[0], bh[1]);
                    mma16816(uc[1], sl, bh[2], bh[3]);
                    ldsm4(bh, at + I::kQh + row + j * 32);
                    ldsm4(bl, at + I::kQl + row + j * 32);
                    mma16816(o[0], sh, bh[0], bh[1]);
                    mma16816(o[1], sh, bh[2], bh[3]);
                    mma16816(oc[0], sh, bl[0], bl[1]);
                    mma16816(oc[1], sh, bl[2], bl[3]);
                    mma16816(oc[0], sl, bh[0], bh[1]);
                    mma16816(oc[1], sl, bh[2], bh[3]);
                }
                const float* U = reinterpret_cast<const float*>(im + K::kHead) + tig * 2 * I::SU + warp * 16 + gid;
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int i = 0; i < 4; ++i) u[n][i] = U[(n * 8 + (i & 1)) * I::SU + (i >> 1) * 8] - (u[n][i] + uc[n][i]);
                uint32_t uh[4], ul[4];
                split_bf16(u[0][0], u[0][1], uh[0], ul[0]);
                split_bf16(u[0][2], u[0][3], uh[1], ul[1]);
                split_bf16(u[1][0], u[1][1], uh[2], ul[2]);
                split_bf16(u[1][2], u[1][3], uh[3], ul[3]);
                // S^T <- G_16 S^T + u^T K
                const float* E = reinterpret_cast<const float*>(im + I::kE) + tig * 2;
                const uint32_t krow = ((m & 1) * 8 + mr) * I::SD * 2 + (m >> 1) * 16;
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    uint32_t bh[4], bl[4];
                    ldsm4t(bh, at + I::kKh + krow + n * 16);
                    ldsm4t(bl, at + I::kKl + krow + n * 16);
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const float2 f = *reinterpret_cast<const float2*>(E + (n + x) * 8);
                        S[n + x][0] *= f.x;
                        S[n + x][1] *= f.y;
                        S[n + x][2] *= f.x;
                        S[n + x][3] *= f.y;
                        mma16816(S[n + x], uh, bh[2 * x], bh[2 * x + 1]);
                        mma16816(S[n + x], uh, bl[2 * x], bl[2 * x + 1]);
                        mma16816(S[n + x], ul, bh[2 * x], bh[2 * x + 1]);
                    }
                }
                {
                    uint32_t bh[4], bl[4];
                    const uint32_t brow = ((m >> 1) * 8 + mr) * I::SB * 2 + (m & 1) * 16;
                    ldsm4(bh, at + I::kBh + brow);
                    ldsm4(bl, at + I::kBl + brow);
                    mma16816(o[0], uh, bh[0], bh[1]);
                    mma16816(o[1], uh, bh[2], bh[3]);
                    mma16816(oc[0], uh, bl[0], bl[1]);
                    mma16816(oc[1], uh, bl[2], bl[3]);
                    mma16816(oc[0], ul, bh[0], bh[1]);
                    mma16816(oc[1], ul, bh[2], bh[3]);
                }
                const int left = po.y - c * C;
                float* dst = outputs + ((static_cast<int64_t>(po.x) + c * C) * a.heads + h) * vdim;
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int t = n * 8 + tig * 2 + (i & 1), e = v1 + (i >> 1) * 8;
                        if (t < left && e < vdim) dst[static_cast<int64_t>(t) * a.heads * vdim + e] = o[n][i] + oc[n][i];
                    }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(empty + st));
        }
        if (live) {
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int d = n * 8 + tig * 2 + (i & 1), e = v1 + (i >> 1) * 8;
                    if (d < dim && e < vdim) state[static_cast<int64_t>(d) * vdim + e] = S[n][i];
                }
        }
        // the convolution's last inputs, for the next portion or the first decode step
        const SpkDeltaShape shp = spk_delta_shape(a);
        const int rep = a.heads / a.kv_heads, grp = h / rep;
        for (int i = threadIdx.x; i < columns; i += 32 * NW)
            if (v0 + i < vdim) spk_commit_conv<__nv_bfloat16>(a, po, shp, a.v, static_cast<int64_t>(h) * vdim + v0 + i, 2 * shp.qk + h * vdim + v0 + i);
        if (blockIdx.x == 0 && h % rep == 0)
            for (int d = threadIdx.x; d < dim; d += 32 * NW) {
                spk_commit_conv<__nv_bfloat16>(a, po, shp, a.q, static_cast<int64_t>(grp) * dim + d, grp * dim + d);
                spk_commit_conv<__nv_bfloat16>(a, po, shp, a.k, static_cast<int64_t>(grp) * dim + d, shp.qk + grp * dim + d);
            }
    }
    __syncthreads();
}

int padded_v(int vdim) { return (vdim + 63) & ~63; }
int64_t image_size(int dim, int vdim) {
    const int64_t u = static_cast<int64_t>(padded_v(vdim) / 64) * C * Image<64>::SU * 4;
    return (dim <= 64 ? Image<64>::kU : Image<128>::kU) + u;
}

template <int DP>
int launch_chain(const spk_delta_args& a, int64_t image, int vp, float* outputs, cudaStream_t s) {
    constexpr int bytes = Chain<DP>::kBytes;
    const cudaError_t e = cudaFuncSetAttribute(delta_chain_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    return spk_launch(delta_chain_kernel<DP>, dim3((vp + NW * 16 - 1) / (NW * 16), a.heads, a.n_portions), 32 * NW + 32, bytes, s, true, a, image, outputs);
}

template <int DP>
int launch(const spk_delta_args& a, float* outputs, cudaStream_t s) {
    const int vp = padded_v(a.vdim);
    const int64_t image = image_size(a.dim, a.vdim);
    const size_t bytes = sizeof(float) * C * (4 * (DP + 8) + static_cast<size_t>(vp));
    auto* fn = a.taps == 4 ? delta_chunk_kernel<DP, 4> : delta_chunk_kernel<DP, 0>;
    const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    auto even = [&](const void* p) { return reinterpret_cast<uintptr_t>(p) % 4 == 0; };
    auto wide = [&](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool pairs = a.ld % 2 == 0 && a.dim % 2 == 0 && a.vdim % 2 == 0 && even(a.q) && even(a.k) && even(a.v) && wide(a.conv_q) && wide(a.conv_k) && wide(a.conv_v);
    fn<<<dim3(a.n_chunks, a.heads), kThreads, bytes, s>>>(a, image, vp, pairs);
    SPK_CHECK_LAUNCH();
    return launch_chain<DP>(a, image, vp, outputs, s);
}

}  // namespace

int64_t spk_delta_mma_bytes(int n_chunks, int heads, int dim, int vdim) { return static_cast<int64_t>(n_chunks) * heads * image_size(dim, vdim); }

int spk_delta_mma_launch(const spk_delta_args& a, float* outputs, cudaStream_t s) {
    return a.dim <= 64 ? launch<64>(a, outputs, s) : launch<128>(a, outputs, s);
}
