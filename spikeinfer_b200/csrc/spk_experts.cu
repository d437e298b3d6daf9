// Experts chosen by the token's id: routing for all layers of a step, and the 32-bit form of the experts' products.
//
//  * route_kernel: one CTA per expert layer counts the tokens of every expert, lays the experts' segments out (starts at multiples of
//    eight rows) and hands every (token, choice) pair its row.  Ids are all it reads, so one launch serves the whole step.
//  * experts_simt_kernel: 32-bit products of every expert with its rows; bf16 goes to spk_experts_mma.cu.
#include "spk_experts.cuh"

namespace {

constexpr int kRouteThreads = 1024;

__global__ void __launch_bounds__(kRouteThreads)
route_kernel(const spk_expert_route_args a) {
    extern __shared__ int32_t sm[];
    const int64_t* d = a.layers + 8 * static_cast<int64_t>(blockIdx.x);
    const int32_t* table = reinterpret_cast<const int32_t*>(d[0]);
    const int top = static_cast<int>(d[1]), experts = static_cast<int>(d[2]);
    int32_t* slots = a.slots + d[3] * a.n;
    int32_t* segs = a.segs + d[4];
    int32_t* count = sm;            // [experts]
    int32_t* at = sm + experts;     // [experts] next row of the expert
    for (int e = threadIdx.x; e < experts; e += kRouteThreads) count[e] = 0;
    __syncthreads();
    const int64_t pairs = a.n * top;
    auto expert_of = [&](int64_t i) {
        const int64_t t = i / top;
        if (a.active != nullptr && a.active[t] != 1) return -1;
        const int64_t id = a.ids[t];
        if (id < 0 || id >= a.vocab) return -1;
        const int e = table[id * top + i % top];
        return e >= 0 && e < experts ? e : -1;
    };
    for (int64_t i = threadIdx.x; i < pairs; i += kRouteThreads) {
        const int e = expert_of(i);
        if (e >= 0) atomicAdd(count + e, 1);
    }
    __syncthreads();
    if (threadIdx.x < 32) {
        int before = 0;
        for (int e0 = 0; e0 < experts; e0 += 32) {
            const int e = e0 + threadIdx.x;
            const int c = e < experts ? count[e] : 0;
            const int padded = (c + kExpertAlign - 1) & ~(kExpertAlign - 1);
            int upto = padded;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(~0u, upto, o);
                if (static_cast<int>(threadIdx.x) >= o) upto += up;
            }
            if (e < experts) {
                at[e] = before + upto - padded;
                reinterpret_cast<int2*>(segs)[e] = make_int2(before + upto - padded, c);
            }
            before += __shfl_sync(~0u, upto, 31);
        }
    }
    __syncthreads();
    for (int64_t i = threadIdx.x; i < pairs; i += kRouteThreads) {
        const int e = expert_of(i);
        slots[i] = e >= 0 ? atomicAdd(at + e, 1) : -1;
    }
}

// ---- 32-bit products -------------------------------------------------------------------------------------------
constexpr int kT = 32;          // rows, features and k per step
constexpr int kThreads = 256;

template <bool GATED>
__global__ void __launch_bounds__(kThreads)
experts_simt_kernel(const spk_experts_args a) {
    __shared__ float xs[kT][kT + 1], ws[GATED ? 2 : 1][kT][kT + 1];
    int e, rows;
    int64_t row0;
    if (!spk_find_tile<kT>(a.segs, a.experts, blockIdx.y, e, row0, rows)) return;
    const int f0 = blockIdx.x * kT;
    const float* x = static_cast<const float*>(a.x) + row0 * a.k;
    const float* w = static_cast<const float*>(a.w) + static_cast<int64_t>(e) * (GATED ? 2 : 1) * a.out_features * a.k;
    const int c = threadIdx.x % 32, r0 = threadIdx.x / 32;
    float acc[GATED ? 2 : 1][4] = {};
    for (int k0 = 0; k0 < a.k; k0 += kT) {
        __syncthreads();
        for (int i = r0; i < kT; i += 8) {
            xs[i][c] = i < rows && k0 + c < a.k ? x[static_cast<int64_t>(i) * a.k + k0 + c] : 0.0f;
#pragma unroll
            for (int g = 0; g < (GATED ? 2 : 1); ++g)
                ws[g][i][c] = f0 + i < a.out_features && k0 + c < a.k ? w[(static_cast<int64_t>(g) * a.out_features + f0 + i) * a.k + k0 + c] : 0.0f;
        }
        __syncthreads();
        for (int k = 0; k < kT; ++k)
#pragma unroll
            for (int g = 0; g < (GATED ? 2 : 1); ++g) {
                const float wv = ws[g][c][k];
#pragma unroll
                for (int i = 0; i < 4; ++i) acc[g][i] = fmaf(xs[r0 + 8 * i][k], wv, acc[g][i]);
            }
    }
    if (f0 + c >= a.out_features) return;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = r0 + 8 * i;
        if (r >= rows) break;
        const float y = GATED ? spk_silu(acc[0][i]) * acc[GATED ? 1 : 0][i] : acc[0][i];
        static_cast<float*>(a.out)[(row0 + r) * a.out_features + f0 + c] = y;
    }
}

}  // namespace

extern "C" int64_t spk_expert_rows(int64_t n, int top, int experts) {
    if (n < 1 || top < 1 || experts < 1) return 0;
    const int64_t pairs = n * top, used = pairs < experts ? pairs : experts;
    return ((pairs + used * (kExpertAlign - 1) + kExpertAlign - 1) / kExpertAlign) * kExpertAlign + kExpertTailRows;
}

extern "C" int spk_expert_route(const spk_expert_route_args* a, void* stream) {
    SpkRange nvtx_range("spk_expert_route");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->n_layers < 0 || a->n_layers > 65535 || a->vocab < 1 || a->max_experts < 1 || a->max_experts > 4096) return SPK_ERR_BAD_SHAPE;
    if (a->n == 0 || a->n_layers == 0) return SPK_OK;
    if (a->layers == nullptr || a->ids == nullptr || a->slots == nullptr || a->segs == nullptr) return SPK_ERR_NULL_POINTER;
    route_kernel<<<a->n_layers, kRouteThreads, 2 * sizeof(int32_t) * a->max_experts, spk_stream(stream)>>>(*a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

extern "C" int spk_experts(const spk_experts_args* a, void* stream) {
    SpkRange nvtx_range("spk_experts");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->pairs < 0 || a->experts < 1 || a->k < 1 || a->out_features < 1 || a->rows < 1) return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->pairs == 0) return SPK_OK;
    if (a->x == nullptr || a->w == nullptr || a->out == nullptr || a->segs == nullptr) return SPK_ERR_NULL_POINTER;
    cudaStream_t s = spk_stream(stream);
    if (a->dtype == SPK_BF16) return spk_experts_mma(*a, s);
    const int64_t tiles = spk_most_tiles(a->pairs, a->experts, kT);
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const dim3 grid((a->out_features + kT - 1) / kT, static_cast<unsigned>(tiles));
    if (a->gated) experts_simt_kernel<true><<<grid, kThreads, 0, s>>>(*a);
    else experts_simt_kernel<false><<<grid, kThreads, 0, s>>>(*a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}
