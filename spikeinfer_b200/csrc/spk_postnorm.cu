// Row kernels of a decoder whose residual stream is normalised AFTER each sublayer and kept in 32 bits.
//
//  * residual_norm_kernel: x' = layernorm(alpha * x + delta) * w (mean removed, no bias), or x' = embedding row; then
//    what the next sublayer reads: x' itself, x' mixed per channel with the previous token's x' (token shift), or a second
//    layer norm of x' (the model's last).  One launch per sublayer boundary.
//  * poly_norm_kernel, poly_norm_packed_kernel: a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's root mean square.
//
// The previous token's row is recomputed by the CTA that needs it when it lies in the same launch (it depends on nothing
// but its own x and delta), and read from the sequence's state when the token is the first of its portion.  The
// state is written by the launch that ends the sublayer (it still reads the old x), so no launch reads and
// writes one state row from two CTAs.
#include "spk_dense.cuh"

namespace {

struct ResidualNormParams {
    const float* x;
    float* x_out;
    const void* delta;
    const void* embed;
    const int64_t* ids;
    int64_t vocab;
    const float* w;
    const float* w2;
    float alpha, eps;
    const float* mix;
    const float* prev;
    float* commit;
    int64_t state_stride;
    int64_t state_rows;
    const int64_t* positions;
    const int32_t* token_rows;
    const int32_t* token_edges;
    const int32_t* active;
    int64_t n;
    int width;
    int per_cta;
    uint32_t* status;
};

__device__ __forceinline__ float4 f4_axpy(float a, float4 x, float4 y) {
    return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}

// Layer norm of the row in registers (two passes over them: mean, then squared deviations).
template <int V, bool VEC>
__device__ __forceinline__ void layer_norm_row(SpkRow<V>& y, const float* __restrict__ w, int width, float eps, float* part) {
    float s[1] = {0.0f};
#pragma unroll
    for (int v = 0; v < V; ++v) s[0] += (y.g[v].x + y.g[v].y) + (y.g[v].z + y.g[v].w);
    spk_block_sum<1>(s, part);
    const float mean = s[0] / static_cast<float>(width);
    float q[1] = {0.0f};
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int left = width - 4 * (threadIdx.x + v * blockDim.x);
        float4 d = y.g[v];
        d.x = left > 0 ? d.x - mean : 0.0f;
        d.y = left > 1 ? d.y - mean : 0.0f;
        d.z = left > 2 ? d.z - mean : 0.0f;
        d.w = left > 3 ? d.w - mean : 0.0f;
        q[0] += (d.x * d.x + d.y * d.y) + (d.z * d.z + d.w * d.w);
        y.g[v] = d;
    }
    spk_block_sum<1>(q, part);
    const float inv = 1.0f / sqrtf(q[0] / static_cast<float>(width) + eps);
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        const float4 wv = spk_load4<float, VEC>(w + c, width - c);
        y.g[v] = make_float4(y.g[v].x * inv * wv.x, y.g[v].y * inv * wv.y, y.g[v].z * inv * wv.z, y.g[v].w * inv * wv.w);
    }
}

template <typename T, typename TD, int V, bool VEC>
__device__ __forceinline__ void new_row(const ResidualNormParams& p, int64_t t, int64_t commit_row, SpkRow<V>& y, float* part) {
    if (p.ids != nullptr) {
        const int64_t id = p.ids[t];
        const bool ok = id >= 0 && id < p.vocab;
        if (!ok && threadIdx.x == 0) spk_flag(p.status, SPK_STATUS_BAD_TOKEN);
        const T* e = static_cast<const T*>(p.embed) + (ok ? id : 0) * p.width;
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int c = 4 * (threadIdx.x + v * blockDim.x);
            y.g[v] = spk_load4<T, VEC>(e + c, ok ? p.width - c : 0);
        }
        return;
    }
    const float* xr = p.x + t * p.width;
    const TD* dr = static_cast<const TD*>(p.delta) + t * p.width;
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        const float4 old = spk_load4<float, VEC>(xr + c, p.width - c);
        if (commit_row >= 0) spk_store4<float, VEC>(p.commit + commit_row * p.state_stride + c, old, p.width - c);
        y.g[v] = f4_axpy(p.alpha, old, spk_load4<TD, VEC>(dr + c, p.width - c));
    }
    layer_norm_row<V, VEC>(y, p.w, p.width, p.eps, part);
}

template <typename T, typename TD, int V, bool VEC>
__global__ void __launch_bounds__(1024)
residual_norm_kernel(const ResidualNormParams p, T* __restrict__ out) {
    __shared__ float part[32];
    const int64_t t0 = static_cast<int64_t>(blockIdx.x) * p.per_cta;
    const int64_t t1 = t0 + p.per_cta < p.n ? t0 + p.per_cta : p.n;
    SpkRow<V> before, y;
    for (int64_t t = t0; t < t1; ++t) {
        // decode: token t is row t's only token; prefill: the portion's tables say
        const int32_t edge = p.token_edges != nullptr ? p.token_edges[t] : 3;
        int64_t row = p.token_rows != nullptr ? p.token_rows[t] : t;
        if (p.active != nullptr && p.token_rows == nullptr && p.active[t] != 1) row = -1;
        if (row >= p.state_rows && (p.mix != nullptr || p.commit != nullptr)) {
            if (threadIdx.x == 0) spk_flag(p.status, SPK_STATUS_BAD_SLOT);
            row = -1;
        }
        if (p.mix != nullptr) {
            if (edge & 1) {
                const bool stored = row >= 0 && p.positions[t] > 0;
                const float* s = p.prev + (stored ? row : 0) * p.state_stride;
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    const int c = 4 * (threadIdx.x + v * blockDim.x);
                    before.g[v] = spk_load4<float, VEC>(s + c, stored ? p.width - c : 0);
                }
            } else if (t == t0) {
                new_row<T, TD, V, VEC>(p, t - 1, -1, before, part);
            }
        }
        new_row<T, TD, V, VEC>(p, t, p.commit != nullptr && (edge & 2) ? row : -1, y, part);
        if (p.x_out != nullptr) {
#pragma unroll
            for (int v = 0; v < V; ++v) {
                const int c = 4 * (threadIdx.x + v * blockDim.x);
                spk_store4<float, VEC>(p.x_out + t * p.width + c, y.g[v], p.width - c);
            }
        }
        T* o = out + t * p.width;
        if (p.mix != nullptr) {
#pragma unroll
            for (int v = 0; v < V; ++v) {
                const int c = 4 * (threadIdx.x + v * blockDim.x);
                const float4 m = spk_load4<float, VEC>(p.mix + c, p.width - c);
                const float4 a = y.g[v], b = before.g[v];
                spk_store4<T, VEC>(o + c, make_float4(a.x + (b.x - a.x) * m.x, a.y + (b.y - a.y) * m.y,
                                                      a.z + (b.z - a.z) * m.z, a.w + (b.w - a.w) * m.w), p.width - c);
                before.g[v] = a;
            }
        } else {
            if (p.w2 != nullptr) layer_norm_row<V, VEC>(y, p.w2, p.width, p.eps, part);
#pragma unroll
            for (int v = 0; v < V; ++v) {
                const int c = 4 * (threadIdx.x + v * blockDim.x);
                spk_store4<T, VEC>(o + c, y.g[v], p.width - c);
            }
        }
    }
}

template <typename T, int V, bool VEC>
__global__ void __launch_bounds__(1024)
poly_norm_kernel(const T* __restrict__ z, const float* __restrict__ coef, float eps, T* __restrict__ out, int width) {
    __shared__ float part[3 * 32];
    const T* zr = z + static_cast<int64_t>(blockIdx.x) * width;
    T* o = out + static_cast<int64_t>(blockIdx.x) * width;
    SpkRow<V> y;
    float s[3] = {0.0f, 0.0f, 0.0f};
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        y.g[v] = spk_load4<T, VEC>(zr + c, width - c);
        const float e[4] = {y.g[v].x, y.g[v].y, y.g[v].z, y.g[v].w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float q = e[i] * e[i];
            s[0] += q;
            s[1] = fmaf(q, q, s[1]);
            s[2] = fmaf(q * q, q, s[2]);
        }
    }
    spk_block_sum<3>(s, part);
    const float n = static_cast<float>(width);
    const float k1 = coef[0] / sqrtf(s[0] / n + eps), k2 = coef[1] / sqrtf(s[1] / n + eps);
    const float k3 = coef[2] / sqrtf(s[2] / n + eps), k0 = coef[3];
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        auto f = [&](float x) { return fmaf(x, fmaf(x, fmaf(x, k3, k2), k1), k0); };
        spk_store4<T, VEC>(o + c, make_float4(f(y.g[v].x), f(y.g[v].y), f(y.g[v].z), f(y.g[v].w)), width - c);
    }
}

// bf16 rows in 16-byte groups that stay packed in registers between the two passes: G groups per thread.
template <int G>
__global__ void __launch_bounds__(512)
poly_norm_packed_kernel(const __nv_bfloat16* __restrict__ z, const float* __restrict__ coef, float eps, __nv_bfloat16* __restrict__ out, int width) {
    __shared__ float part[3 * 32];
    const uint4* zr = reinterpret_cast<const uint4*>(z + static_cast<int64_t>(blockIdx.x) * width);
    uint4* o = reinterpret_cast<uint4*>(out + static_cast<int64_t>(blockIdx.x) * width);
    const int groups = width / 8;
    uint4 raw[G];
#pragma unroll
    for (int v = 0; v < G; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        raw[v] = i < groups ? zr[i] : make_uint4(0u, 0u, 0u, 0u);
    }
    float s[3] = {0.0f, 0.0f, 0.0f};
    auto moments = [&](float x) {
        const float q = x * x;
        s[0] += q;
        s[1] = fmaf(q, q, s[1]);
        s[2] = fmaf(q * q, q, s[2]);
    };
#pragma unroll
    for (int v = 0; v < G; ++v) {
        const uint32_t w[4] = {raw[v].x, raw[v].y, raw[v].z, raw[v].w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            moments(__uint_as_float(w[k] << 16));
            moments(__uint_as_float(w[k] & 0xffff0000u));
        }
    }
    spk_block_sum<3>(s, part);
    const float n = static_cast<float>(width);
    const float k1 = coef[0] / sqrtf(s[0] / n + eps), k2 = coef[1] / sqrtf(s[1] / n + eps);
    const float k3 = coef[2] / sqrtf(s[2] / n + eps), k0 = coef[3];
    auto f = [&](float x) { return fmaf(x, fmaf(x, fmaf(x, k3, k2), k1), k0); };
#pragma unroll
    for (int v = 0; v < G; ++v) {
        const int i = threadIdx.x + v * blockDim.x;
        uint32_t w[4] = {raw[v].x, raw[v].y, raw[v].z, raw[v].w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(f(__uint_as_float(w[k] << 16)), f(__uint_as_float(w[k] & 0xffff0000u)));
            w[k] = *reinterpret_cast<const uint32_t*>(&b);
        }
        if (i < groups) o[i] = make_uint4(w[0], w[1], w[2], w[3]);
    }
}

int launch_poly_packed(const void* z, const float* coef, float eps, void* out, int64_t rows, int64_t width, cudaStream_t s) {
    const int groups = static_cast<int>(width / 8);
    int threads = groups <= 512 ? 128 : groups <= 2048 ? 256 : 512;
    if (rows < 2 * 148) threads = groups <= 128 ? 128 : groups <= 256 ? 256 : 512;  // few rows: spread a row wider
    const int g = (groups + threads - 1) / threads;
    const unsigned grid = static_cast<unsigned>(rows);
    const __nv_bfloat16* zi = static_cast<const __nv_bfloat16*>(z);
    __nv_bfloat16* o = static_cast<__nv_bfloat16*>(out);
    const int w = static_cast<int>(width);
#define SPK_PP(G_) poly_norm_packed_kernel<G_><<<grid, threads, 0, s>>>(zi, coef, eps, o, w)
    switch (g) {
        case 1: SPK_PP(1); break;
        case 2: SPK_PP(2); break;
        case 3: SPK_PP(3); break;
        case 4: SPK_PP(4); break;
        case 5: SPK_PP(5); break;
        case 6: SPK_PP(6); break;
        default: SPK_PP(8); break;
    }
#undef SPK_PP
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T, typename TD>
int launch_residual(const ResidualNormParams& p, void* out, cudaStream_t s) {
    int v = 1;
    const int threads = spk_row_shape(p.width, &v);
    if (threads == 0) return SPK_ERR_TOO_LARGE;
    const unsigned grid = static_cast<unsigned>((p.n + p.per_cta - 1) / p.per_cta);
    const bool vec = p.width % 4 == 0;
    T* o = static_cast<T*>(out);
#define SPK_RN(V_)                                                                              \
    do {                                                                                        \
        if (vec) residual_norm_kernel<T, TD, V_, true><<<grid, threads, 0, s>>>(p, o);          \
        else residual_norm_kernel<T, TD, V_, false><<<grid, threads, 0, s>>>(p, o);             \
    } while (0)
    if (v == 1) SPK_RN(1);
    else if (v == 2) SPK_RN(2);
    else if (v == 4) SPK_RN(4);
    else SPK_RN(8);
#undef SPK_RN
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T>
int launch_poly(const void* z, const float* coef, float eps, void* out, int64_t rows, int64_t width, cudaStream_t s) {
    int v = 1;
    const int threads = spk_row_shape(width, &v);
    if (threads == 0) return SPK_ERR_TOO_LARGE;
    const unsigned grid = static_cast<unsigned>(rows);
    const bool vec = width % 4 == 0;
    const T* zi = static_cast<const T*>(z);
    T* o = static_cast<T*>(out);
    const int w = static_cast<int>(width);
#define SPK_PN(V_)                                                                              \
    do {                                                                                        \
        if (vec) poly_norm_kernel<T, V_, true><<<grid, threads, 0, s>>>(zi, coef, eps, o, w);   \
        else poly_norm_kernel<T, V_, false><<<grid, threads, 0, s>>>(zi, coef, eps, o, w);      \
    } while (0)
    if (v == 1) SPK_PN(1);
    else if (v == 2) SPK_PN(2);
    else if (v == 4) SPK_PN(4);
    else SPK_PN(8);
#undef SPK_PN
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

extern "C" int spk_residual_norm(const spk_residual_norm_args* a, void* stream) {
    SpkRange nvtx_range("spk_residual_norm");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->width < 1 || a->width > (1 << 20)) return SPK_ERR_BAD_SHAPE;
    if (a->n == 0) return SPK_OK;
    if (a->n > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    const bool embed = a->ids != nullptr;
    if (a->out == nullptr || (embed && a->embed == nullptr) || (!embed && (a->x == nullptr || a->delta == nullptr || a->w == nullptr)))
        return SPK_ERR_NULL_POINTER;
    if (a->mix != nullptr && (a->prev == nullptr || a->positions == nullptr)) return SPK_ERR_NULL_POINTER;
    if ((a->token_rows == nullptr) != (a->token_edges == nullptr)) return SPK_ERR_NULL_POINTER;
    if ((a->mix != nullptr || a->commit != nullptr) && (a->state_rows < 1 || (a->token_rows == nullptr && a->n > a->state_rows)))
        return SPK_ERR_BAD_SHAPE;
    if (a->mix != nullptr && a->w2 != nullptr) return SPK_ERR_UNSUPPORTED;
    // the row before a CTA's first is recomputed from x, so x may not be overwritten by another CTA meanwhile
    if (a->mix != nullptr && a->token_rows != nullptr && a->x_out != nullptr && a->x_out == a->x) return SPK_ERR_UNSUPPORTED;
    ResidualNormParams p{};
    p.x = a->x; p.x_out = a->x_out; p.delta = a->delta; p.embed = a->embed; p.ids = a->ids; p.vocab = a->vocab;
    p.w = a->w; p.w2 = a->w2; p.alpha = a->alpha; p.eps = a->eps; p.mix = a->mix; p.prev = a->prev; p.commit = a->commit;
    p.state_stride = a->width; p.state_rows = a->state_rows; p.positions = a->positions; p.token_rows = a->token_rows;
    p.token_edges = a->token_edges; p.active = a->active; p.n = a->n; p.width = static_cast<int>(a->width); p.status = a->status;
    // a run of rows per CTA amortises the recomputed predecessor; single rows while there are few
    p.per_cta = (a->mix != nullptr && a->token_rows != nullptr && a->n >= 4 * 148) ? 4 : 1;
    cudaStream_t s = spk_stream(stream);
    if (a->dtype == SPK_F32) {
        if (!embed && a->delta_dtype != SPK_F32) return SPK_ERR_BAD_DTYPE;
        return launch_residual<float, float>(p, a->out, s);
    }
    if (a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (embed || a->delta_dtype == SPK_F32) return launch_residual<__nv_bfloat16, float>(p, a->out, s);
    if (a->delta_dtype == SPK_BF16) return launch_residual<__nv_bfloat16, __nv_bfloat16>(p, a->out, s);
    return SPK_ERR_BAD_DTYPE;
}

extern "C" int spk_poly_norm(const void* z, const float* coef, float eps, void* out, int64_t rows, int64_t width, int dtype,
                             void* stream) {
    SpkRange nvtx_range("spk_poly_norm");
    if (rows < 0 || width < 1 || width > (1 << 20)) return SPK_ERR_BAD_SHAPE;
    if (rows == 0) return SPK_OK;
    if (rows > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    if (z == nullptr || coef == nullptr || out == nullptr) return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    if (dtype == SPK_F32) return launch_poly<float>(z, coef, eps, out, rows, width, s);
    if (dtype == SPK_BF16 && width % 8 == 0 && width <= 8 * 512 * 8 && reinterpret_cast<uintptr_t>(z) % 16 == 0 && reinterpret_cast<uintptr_t>(out) % 16 == 0)
        return launch_poly_packed(z, coef, eps, out, rows, width, s);
    if (dtype == SPK_BF16) return launch_poly<__nv_bfloat16>(z, coef, eps, out, rows, width, s);
    return SPK_ERR_BAD_DTYPE;
}
