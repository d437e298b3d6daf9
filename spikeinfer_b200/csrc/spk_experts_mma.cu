// The experts' products on the fifth-generation tensor cores (tcgen05), bf16 operands, 32-bit sums.
//
// CTA = (256 weight rows, run of TN tokens of one expert).  The weights are the M operand (two 128-row tiles, an accumulator each), the
// tokens the N operand: a few decoded tokens cost a narrow MMA instead of a padded tile, and every lane of the accumulators is in use.
// Weights and tokens are stored as the swizzled operand tiles they become, so a stage is two plain bulk copies (cp.async.bulk),
// no tensor map and no gather: the launch that normalises the residual has already put every token's row where its experts read it.
//  * gated: the two tiles are gate and up rows of the same 128 features; the epilogue multiplies silu(gate) by up and writes the operand
//    tiles of the next product.
//  * plain: 256 consecutive output features, 32-bit rows.
// Warp 0 copies, warp 1 issues MMAs, warps 2-5 write the results.
#include "spk_experts.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kThreads = 192;
constexpr int kTileW = 128 * 128;  // bytes of a 128-row, 64-column weight tile

template <int TN>
struct Shape {
    static constexpr int kStage = 2 * kTileW + TN * 128;
    static constexpr int NS = TN >= 256 ? 3 : TN >= 128 ? 4 : TN >= 64 ? 5 : 3;  // the narrow form leaves room for a second CTA
    static constexpr int kBytes = NS * kStage + 1024 + 256;
    static constexpr int kColumns = 2 * TN < 32 ? 32 : 2 * TN;
};

struct Bars {
    uint64_t full[8], free[8], done;
    int abort;
    uint32_t tmem;
};

template <int TN, bool GATED>
__global__ void __launch_bounds__(kThreads, TN <= 32 ? 2 : 1)
experts_kernel(const spk_experts_args a, const int blocks, const int ktiles) {
    using Sh = Shape<TN>;
    constexpr int NS = Sh::NS;
    int e, rows;
    int64_t row0;
    // uniform over the CTA: nothing has been set up yet
    if (!spk_find_tile<TN>(a.segs, a.experts, blockIdx.y, e, row0, rows)) return;
    if (row0 + TN > a.rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
    Bars* bars = reinterpret_cast<Bars*>(base + NS * Sh::kStage);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int i = 0; i < NS; ++i) {
            mbar_init(smem_u32(&bars->full[i]), 1);
            mbar_init(smem_u32(&bars->free[i]), 1);
        }
        mbar_init(smem_u32(&bars->done), 1);
        bars->abort = 0;
    }
    if (warp == 0) tmem_alloc(smem_u32(&bars->tmem), Sh::kColumns);
    fence_async_shared();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem;
    volatile int* abort = &bars->abort;
    const int b = blockIdx.x;
    if (warp == 0) {
        if (lane == 0) {
            const uint8_t* w = static_cast<const uint8_t*>(a.w) + (static_cast<int64_t>(e) * blocks + b) * ktiles * (2 * kTileW);
            const uint8_t* x = static_cast<const uint8_t*>(a.x) + row0 * 128;
            int issued = 0;
            for (int k = 0; k < ktiles; ++k) {
                const int s = k % NS;
                if (k >= NS && !mbar_wait(smem_u32(&bars->free[s]), ((k / NS) - 1) & 1, abort)) break;
                const uint32_t bar = smem_u32(&bars->full[s]), dst = smem_u32(base + s * Sh::kStage);
                mbar_expect(bar, Sh::kStage);
                bulk_load(dst, w + static_cast<int64_t>(k) * (2 * kTileW), 2 * kTileW, bar);
                bulk_load(dst + 2 * kTileW, x + static_cast<int64_t>(k) * a.rows * 128, TN * 128, bar);
                issued = k + 1;
            }
            if (*abort != 0)  // copies in flight land before the CTA's shared memory is given up
                for (int k = issued > NS ? issued - NS : 0; k < issued; ++k) mbar_wait(smem_u32(&bars->full[k % NS]), (k / NS) & 1);
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = idesc_bf16(128, TN, false, false);
            for (int k = 0; k < ktiles; ++k) {
                const int s = k % NS;
                if (!mbar_wait(smem_u32(&bars->full[s]), (k / NS) & 1, abort)) break;
                tc_fence_after();
                const uint32_t wa = smem_u32(base + s * Sh::kStage), xa = wa + 2 * kTileW;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const uint64_t xd = desc_sw128(xa + i * 32, 16, 1024);
                    mma_ss(tmem, desc_sw128(wa + i * 32, 16, 1024), xd, idesc, k > 0 || i > 0);
                    mma_ss(tmem + TN, desc_sw128(wa + kTileW + i * 32, 16, 1024), xd, idesc, k > 0 || i > 0);
                }
                mma_commit(smem_u32(&bars->free[s]));
            }
            mma_commit(smem_u32(&bars->done));
            mbar_wait(smem_u32(&bars->done), 0);  // nothing this thread issued is in the tensor pipe any more
        }
    } else {
        const int quad = warp & 3;
        const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
        const bool ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->done), 0, abort)) && *abort == 0;
        tc_fence_after();
        const int f = b * (GATED ? 128 : 256) + quad * 32 + lane;  // this lane's feature (and f + 128)
#pragma unroll 1
        for (int j0 = 0; j0 < TN && j0 < rows; j0 += 32) {
            uint32_t p[32], q[32];
            tmem_ld32(tmem + lanes + j0, p);
            tmem_ld32(tmem + lanes + TN + j0, q);
            tmem_wait_ld(p);
            tmem_wait_ld(q);
            const int n = ok ? min(32, rows - j0) : 0;
            if (GATED) {
                __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out);
                // pairs of lanes trade a token's value, so that a store carries two features
                const bool odd = lane & 1;
                const int fe = f & ~1;
                const bool in = fe < spk_operand_columns(a.out_features);
#pragma unroll
                for (int j = 0; j < 32; j += 2) {
                    const float y0 = __uint_as_float(p[j]) * rcp(1.0f + ex2(-1.4426950408889634f * __uint_as_float(p[j]))) * __uint_as_float(q[j]);
                    const float y1 = __uint_as_float(p[j + 1]) * rcp(1.0f + ex2(-1.4426950408889634f * __uint_as_float(p[j + 1]))) * __uint_as_float(q[j + 1]);
                    const float got = __shfl_xor_sync(~0u, odd ? y0 : y1, 1);
                    const uint32_t v = odd ? pack_bf16(got, y1) : pack_bf16(y0, got);
                    const int jj = j + (odd ? 1 : 0);
                    if (in && jj < n) *reinterpret_cast<uint32_t*>(out + spk_operand_at(a.rows, row0 + j0 + jj, fe)) = v;
                }
            } else {
                float* out = static_cast<float*>(a.out) + (row0 + j0) * a.out_features + f;
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    if (j < n) {
                        if (f < a.out_features) out[static_cast<int64_t>(j) * a.out_features] = __uint_as_float(p[j]);
                        if (f + 128 < a.out_features) out[static_cast<int64_t>(j) * a.out_features + 128] = __uint_as_float(q[j]);
                    }
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (threadIdx.x == 0 && *abort != 0) spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
    if (warp == 0) tmem_dealloc(tmem, Sh::kColumns);
}

template <int TN, bool GATED>
int launch(const spk_experts_args& a, int blocks, int ktiles, cudaStream_t s) {
    constexpr int bytes = Shape<TN>::kBytes;
    static_assert(sizeof(Bars) <= 256 && bytes <= 227 * 1024, "shared memory");
    const int64_t tiles = spk_most_tiles(a.pairs, a.experts, TN);
    if (tiles > 65535) return SPK_ERR_TOO_LARGE;
    const cudaError_t e = cudaFuncSetAttribute(experts_kernel<TN, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    experts_kernel<TN, GATED><<<dim3(blocks, static_cast<unsigned>(tiles)), kThreads, bytes, s>>>(a, blocks, ktiles);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <bool GATED>
int dispatch(const spk_experts_args& a, cudaStream_t s) {
    const int per = GATED ? 128 : 256;
    const int blocks = (a.out_features + per - 1) / per, ktiles = (a.k + 63) / 64;
    const int64_t mean = (a.pairs + a.experts - 1) / a.experts;
    if (mean > 96) return launch<256, GATED>(a, blocks, ktiles, s);
    if (mean > 40) return launch<128, GATED>(a, blocks, ktiles, s);
    if (mean > 16) return launch<64, GATED>(a, blocks, ktiles, s);
    return launch<32, GATED>(a, blocks, ktiles, s);
}

}  // namespace

int spk_experts_mma(const spk_experts_args& a, cudaStream_t s) {
    if (a.rows % kExpertAlign != 0 || reinterpret_cast<uintptr_t>(a.x) % 16 != 0 || reinterpret_cast<uintptr_t>(a.w) % 16 != 0 ||
        reinterpret_cast<uintptr_t>(a.out) % 16 != 0)
        return SPK_ERR_BAD_STRIDE;
    return a.gated ? dispatch<true>(a, s) : dispatch<false>(a, s);
}
