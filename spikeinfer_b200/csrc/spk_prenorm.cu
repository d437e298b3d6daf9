// Row kernels of a decoder whose branches read RMS norms of one 32-bit residual stream side by side.
//
//  * rms_residual_kernel: x' = x + delta + the weighted rows of the token's experts (or the scaled embedding row); both norms of x'
//    share one root mean square.  The feed-forward's input can go straight to the rows of the experts' sorted matrix (spk_experts.cuh).
//    One launch per layer boundary.
//  * gelu_kernel: the tanh form of gelu.
#include "spk_experts.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

template <typename T, typename TD, int V, bool VEC>
__global__ void __launch_bounds__(1024)
rms_residual_kernel(const spk_rms_residual_args p) {
    __shared__ float part[32];
    const int64_t t = blockIdx.x;
    const int width = static_cast<int>(p.width);
    SpkRow<V> y;
    if (p.ids != nullptr) {
        const int64_t id = p.ids[t];
        const bool ok = id >= 0 && id < p.vocab;
        if (!ok && threadIdx.x == 0) spk_flag(p.status, SPK_STATUS_BAD_TOKEN);
        const T* e = static_cast<const T*>(p.embed) + (ok ? id : 0) * p.width;
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int c = 4 * (threadIdx.x + v * blockDim.x);
            const float4 f = spk_load4<T, VEC>(e + c, ok ? width - c : 0);
            const float m = p.embed_scale;
            y.g[v] = make_float4(f.x * m, f.y * m, f.z * m, f.w * m);
        }
    } else {
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int c = 4 * (threadIdx.x + v * blockDim.x);
            y.g[v] = spk_load4<float, VEC>(p.x + t * p.width + c, width - c);
        }
        if (p.delta != nullptr) {
            const TD* d = static_cast<const TD*>(p.delta) + t * p.width;
#pragma unroll
            for (int v = 0; v < V; ++v) {
                const int c = 4 * (threadIdx.x + v * blockDim.x);
                const float4 f = spk_load4<TD, VEC>(d + c, width - c);
                y.g[v] = make_float4(y.g[v].x + f.x, y.g[v].y + f.y, y.g[v].z + f.z, y.g[v].w + f.w);
            }
        }
        if (p.pairs != nullptr) {
            SpkRow<V> s;
#pragma unroll
            for (int v = 0; v < V; ++v) s.g[v] = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int j = 0; j < p.pair_top; ++j) {
                const int64_t slot = p.pair_slots[t * p.pair_top + j];
                if (slot < 0) continue;
                if (slot >= p.pair_rows) {
                    if (threadIdx.x == 0) spk_flag(p.status, SPK_STATUS_BAD_SLOT);
                    continue;
                }
                const float* r = p.pairs + slot * p.width;
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    const int c = 4 * (threadIdx.x + v * blockDim.x);
                    const float4 f = spk_load4<float, VEC>(r + c, width - c);
                    s.g[v] = make_float4(s.g[v].x + f.x, s.g[v].y + f.y, s.g[v].z + f.z, s.g[v].w + f.w);
                }
            }
            const float m = p.pair_scale;
#pragma unroll
            for (int v = 0; v < V; ++v)
                y.g[v] = make_float4(fmaf(m, s.g[v].x, y.g[v].x), fmaf(m, s.g[v].y, y.g[v].y), fmaf(m, s.g[v].z, y.g[v].z), fmaf(m, s.g[v].w, y.g[v].w));
        }
    }
    float q[1] = {0.0f};
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        if (p.x_out != nullptr) spk_store4<float, VEC>(p.x_out + t * p.width + c, y.g[v], width - c);
        q[0] += (y.g[v].x * y.g[v].x + y.g[v].y * y.g[v].y) + (y.g[v].z * y.g[v].z + y.g[v].w * y.g[v].w);
    }
    spk_block_sum<1>(q, part);
    const float inv = 1.0f / sqrtf(q[0] / static_cast<float>(width) + p.eps);
    auto normed = [&](int v, int c, const float* w) {
        const float4 f = spk_load4<float, VEC>(w + c, width - c);
        return make_float4(y.g[v].x * inv * f.x, y.g[v].y * inv * f.y, y.g[v].z * inv * f.z, y.g[v].w * inv * f.w);
    };
    if (p.w1 != nullptr) {
        T* o = static_cast<T*>(p.out1) + t * p.width;
#pragma unroll
        for (int v = 0; v < V; ++v) {
            const int c = 4 * (threadIdx.x + v * blockDim.x);
            spk_store4<T, VEC>(o + c, normed(v, c, p.w1), width - c);
        }
    }
    if (p.w2 == nullptr) return;
    T* o2 = static_cast<T*>(p.out2);
#pragma unroll
    for (int v = 0; v < V; ++v) {
        const int c = 4 * (threadIdx.x + v * blockDim.x);
        const float4 f = normed(v, c, p.w2);
        if (p.out2_slots == nullptr) {
            spk_store4<T, VEC>(o2 + t * p.width + c, f, width - c);
            continue;
        }
        for (int j = 0; j < p.out2_top; ++j) {
            const int64_t slot = p.out2_slots[t * p.out2_top + j];
            if (slot < 0) continue;
            if (slot >= p.out2_rows) {
                if (threadIdx.x == 0 && v == 0) spk_flag(p.status, SPK_STATUS_BAD_SLOT);
                continue;
            }
            if (!p.out2_tiled) spk_store4<T, VEC>(o2 + slot * p.width + c, f, width - c);
            else if (c < spk_operand_columns(width)) spk_store4<T, true>(o2 + spk_operand_at(p.out2_rows, slot, c), f, 4);
        }
    }
}

template <typename T, typename TD>
int launch_boundary(const spk_rms_residual_args& p, cudaStream_t s) {
    int v = 1;
    const int threads = spk_row_shape(p.width, &v);
    if (threads == 0) return SPK_ERR_TOO_LARGE;
    const unsigned grid = static_cast<unsigned>(p.n);
    const bool vec = p.width % 4 == 0;
#define SPK_RR(V_)                                                                      \
    do {                                                                                \
        if (vec) rms_residual_kernel<T, TD, V_, true><<<grid, threads, 0, s>>>(p);      \
        else rms_residual_kernel<T, TD, V_, false><<<grid, threads, 0, s>>>(p);         \
    } while (0)
    if (v == 1) SPK_RR(1);
    else if (v == 2) SPK_RR(2);
    else if (v == 4) SPK_RR(4);
    else SPK_RR(8);
#undef SPK_RR
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

// z / 2 (1 + tanh(y)) = z / (1 + exp(-2 y)), y = sqrt(2 / pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh(float z) {
    return z / (1.0f + expf(-1.5957691216057308f * fmaf(0.044715f * z * z, z, z)));
}
__device__ __forceinline__ float gelu_tanh_fast(float z) {  // for 16-bit results
    return z * rcp(1.0f + ex2(-2.302208198f * fmaf(0.044715f * z * z, z, z)));  // 2 sqrt(2 / pi) log2(e)
}

constexpr int kGeluThreads = 256;

// bf16, eight elements per thread; everything aligned to them.
__global__ void __launch_bounds__(kGeluThreads)
gelu_vec_kernel(const __nv_bfloat16* __restrict__ z, __nv_bfloat16* __restrict__ out, int64_t out_stride, int width) {
    const int c = 8 * (blockIdx.x * kGeluThreads + threadIdx.x);
    if (c >= width) return;
    const int64_t t = blockIdx.y;
    const uint4 u = __ldcs(reinterpret_cast<const uint4*>(z + t * width + c));
    uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int k = 0; k < 4; ++k)
        w[k] = pack_bf16(gelu_tanh_fast(__uint_as_float(w[k] << 16)), gelu_tanh_fast(__uint_as_float(w[k] & 0xffff0000u)));
    *reinterpret_cast<uint4*>(out + t * out_stride + c) = make_uint4(w[0], w[1], w[2], w[3]);
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(kGeluThreads)
gelu_kernel(const T* __restrict__ z, T* __restrict__ out, int64_t out_stride, int64_t groups, int per_row, int width) {
    const int64_t i = static_cast<int64_t>(blockIdx.x) * kGeluThreads + threadIdx.x;
    if (i >= groups) return;
    const int64_t t = i / per_row;
    const int c = 4 * static_cast<int>(i % per_row);
    const float4 f = spk_load4<T, VEC>(z + t * width + c, width - c);
    spk_store4<T, VEC>(out + t * out_stride + c, make_float4(gelu_tanh(f.x), gelu_tanh(f.y), gelu_tanh(f.z), gelu_tanh(f.w)), width - c);
}

template <typename T>
int launch_gelu(const void* z, void* out, int64_t out_stride, int64_t n, int64_t width, cudaStream_t s) {
    auto at = [](const void* p, size_t b) { return reinterpret_cast<uintptr_t>(p) % b == 0; };
    if (sizeof(T) == 2 && width % 8 == 0 && out_stride % 8 == 0 && at(z, 16) && at(out, 16) && n <= 65535) {
        const dim3 grid(static_cast<unsigned>((width / 8 + kGeluThreads - 1) / kGeluThreads), static_cast<unsigned>(n));
        gelu_vec_kernel<<<grid, kGeluThreads, 0, s>>>(static_cast<const __nv_bfloat16*>(z), static_cast<__nv_bfloat16*>(out), out_stride, static_cast<int>(width));
        SPK_CHECK_LAUNCH();
        return SPK_OK;
    }
    const int64_t per = (width + 3) / 4, groups = n * per, grid = (groups + kGeluThreads - 1) / kGeluThreads;
    if (grid > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    const bool vec = width % 4 == 0 && out_stride % 4 == 0 && at(z, 4 * sizeof(T)) && at(out, 4 * sizeof(T));
    const T* zi = static_cast<const T*>(z);
    T* o = static_cast<T*>(out);
    const unsigned g = static_cast<unsigned>(grid);
    if (vec) gelu_kernel<T, true><<<g, kGeluThreads, 0, s>>>(zi, o, out_stride, groups, static_cast<int>(per), static_cast<int>(width));
    else gelu_kernel<T, false><<<g, kGeluThreads, 0, s>>>(zi, o, out_stride, groups, static_cast<int>(per), static_cast<int>(width));
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

extern "C" int spk_rms_residual(const spk_rms_residual_args* a, void* stream) {
    SpkRange nvtx_range("spk_rms_residual");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->width < 1 || a->width > (1 << 20)) return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->n > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    const bool embed = a->ids != nullptr;
    if ((embed && a->embed == nullptr) || (!embed && a->x == nullptr)) return SPK_ERR_NULL_POINTER;
    if ((a->w1 != nullptr && a->out1 == nullptr) || (a->w2 != nullptr && a->out2 == nullptr)) return SPK_ERR_NULL_POINTER;
    if (a->pairs != nullptr && (a->pair_slots == nullptr || a->pair_top < 1 || a->pair_rows < 1)) return SPK_ERR_BAD_SHAPE;
    if (a->out2_slots != nullptr && (a->out2_top < 1 || a->out2_rows < 1)) return SPK_ERR_BAD_SHAPE;
    if (a->out2_tiled && (a->dtype != SPK_BF16 || a->out2_slots == nullptr || a->out2_rows % 8 != 0 || reinterpret_cast<uintptr_t>(a->out2) % 16 != 0))
        return SPK_ERR_UNSUPPORTED;
    cudaStream_t s = spk_stream(stream);
    const bool d32 = a->delta == nullptr || a->delta_dtype == SPK_F32;
    if (!d32 && a->delta_dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->dtype == SPK_F32) return d32 ? launch_boundary<float, float>(*a, s) : SPK_ERR_BAD_DTYPE;
    return d32 ? launch_boundary<__nv_bfloat16, float>(*a, s) : launch_boundary<__nv_bfloat16, __nv_bfloat16>(*a, s);
}

extern "C" int spk_gelu_tanh(const void* z, void* out, int64_t out_stride, int64_t n, int64_t width, int dtype, void* stream) {
    SpkRange nvtx_range("spk_gelu_tanh");
    if (n < 0 || width < 1 || width > (1 << 20) || out_stride < width) return SPK_ERR_BAD_SHAPE;
    if (n == 0) return SPK_OK;
    if (z == nullptr || out == nullptr) return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    if (dtype == SPK_F32) return launch_gelu<float>(z, out, out_stride, n, width, s);
    if (dtype == SPK_BF16) return launch_gelu<__nv_bfloat16>(z, out, out_stride, n, width, s);
    return SPK_ERR_BAD_DTYPE;
}
