// Attention over a shared latent on the tensor cores (tcgen05): one query token per CTA, up to 512 latent and 64 rotated channels, bf16.
//
// All heads read the same cache rows, so a CTA takes 32 heads of a token at once over a range of its keys, and the cache rows are the M
// operand of both products: S^T = K Q^T (64 keys x 32 heads) and O^T += V^T P^T (128 latent channels x 32 heads per MMA), V being the
// latent part of the very tile K is.  No row of the accumulators is padding, a step reads the cache once and stays bound by that.
//  * warp 4 copies: pages laid end to end are an operand as they are (spk_latent.cuh), so a 64-key stage is one plain bulk copy
//    (cp.async.bulk) per page, all channels at once, whatever pages the block table names;
//  * warp 5 issues S^T into one of two TMEM buffers, warp 6 the weighted sums;
//  * warps 0-3 turn scores into weights, sixteen keys each, in the fragment layout of tcgen05.ld.16x256b: two keys x eight heads per lane.
// Weights are exp2(score - reference), 32-bit, and enter the product as a bf16 pair side by side (columns 0-31 the high, 32-63 the
// low parts, added up at the end).  The reference only moves when a score exceeds it by 2^8, so the accumulators are rarely rescaled.
// A CTA leaves (sum, reference, denominator) of its range; spk_latent_out puts ranges and the sink together.
#include "spk_latent.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kKeys = 64;                  // keys per step
constexpr int kAtom = 1024;                // bytes of eight rows x 64 channels
constexpr int kPTile = kKeys * 128;        // a step's weights: 64 keys x (32 high | 32 low parts)
constexpr int kHeads = 32;                 // heads of a CTA
constexpr int kQTile = kHeads * 128;
constexpr int kSoftThreads = 128;
constexpr int kThreads = kSoftThreads + 128;  // warp 7 only helps to write the sums
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kSlack = 8.0f;             // a score may exceed the reference by 2^8

// CL 64-channel latent tiles and one tile of rotated channels.
template <int CL>
struct Shape {
    static constexpr int CT = CL + 1, MB = (CL + 1) / 2;
    static constexpr int kGroup = CT * kAtom;  // eight rows
    static constexpr int kStage = kKeys / 8 * kGroup;
    static constexpr int NS = CT > 6 ? 2 : CT > 4 ? 3 : 4;
    static constexpr int kBytes = NS * kStage + CT * kQTile + 2 * kPTile + 1024 + 1536;
    static constexpr int kColumns = MB > 2 ? 512 : 256;  // scores 2 x 32, then MB x 64 sums
};
constexpr uint32_t kTmemO = 2 * kHeads;

struct Bars {
    uint64_t full[4], free[4], s_full[2], p_full[2], p_free[2], q_full, o_full, s_done;
    int abort;
    uint32_t tmem;
    float top[2][4][kHeads];  // a step's maxima, per warp
    float fix[kHeads];        // factors of a rescale; totals at the end
};

// 16 lanes x 32 columns in fragment layout: r[4 g + i] = (lane / 4 + 8 (i / 2), 8 g + 2 (lane % 4) + i % 2)
__device__ __forceinline__ void tmem_ld_frag(uint32_t addr, uint32_t (&r)[16]) {
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x4.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : SPK_W8(r, 0), SPK_W8(r, 8) : "r"(addr) : "memory");
    asm volatile("tcgen05.wait::ld.sync.aligned;" : SPK_R8(r, 0), SPK_R8(r, 8) : : "memory");
}
__device__ __forceinline__ void soft_barrier() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

template <int CL>
__global__ void __launch_bounds__(kThreads, 1)
latent_decode_kernel(const spk_latent_attn_args a) {
    using Sh = Shape<CL>;
    constexpr int NS = Sh::NS, CT = Sh::CT, MB = Sh::MB;
    const int64_t t = blockIdx.x;
    const int h0 = blockIdx.y * kHeads, nh = min(kHeads, a.heads - h0);
    const bool prefill = a.token_rows != nullptr;
    const int64_t len = spk_visible_keys(a, t, prefill);
    const int64_t row = prefill ? a.token_rows[t] : t;
    // uniform over the CTA: nothing has been set up yet
    if (len < 0 || len > a.max_blocks * a.block_size || row < 0 || row >= a.table_rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        spk_grid_wait();
        return;
    }
    const int per = spk_split_keys(static_cast<int>(len), a.splits);
    const int lo = blockIdx.z * per, hi = static_cast<int>(min(static_cast<int64_t>(lo) + per, len));
    if (lo >= len) {  // launched to overlap: the launch before this one is complete when this one is
        spk_grid_wait();
        return;
    }
    const int tiles = (hi - lo + kKeys - 1) / kKeys;

    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
    uint8_t* q_s = base + NS * Sh::kStage;
    uint8_t* p_s = q_s + CT * kQTile;
    Bars* bars = reinterpret_cast<Bars*>(p_s + 2 * kPTile);
    const int warp = __shfl_sync(~0u, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int i = 0; i < NS; ++i) {
            mbar_init(smem_u32(&bars->full[i]), 1);
            mbar_init(smem_u32(&bars->free[i]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&bars->s_full[i]), 1);
            mbar_init(smem_u32(&bars->p_full[i]), kSoftThreads);
            mbar_init(smem_u32(&bars->p_free[i]), 1);
        }
        mbar_init(smem_u32(&bars->q_full), kSoftThreads);
        mbar_init(smem_u32(&bars->o_full), 1);
        mbar_init(smem_u32(&bars->s_done), 1);
        bars->abort = 0;
    }
    if (warp == 0) tmem_alloc(smem_u32(&bars->tmem), Sh::kColumns);
    // a step's pages, one block-table entry per lane of the copying warp, the first on its way during the set-up
    const int gran = a.block_size < kKeys ? a.block_size : kKeys;  // rows per copy
    const int pages = kKeys / gran;                                // per step, at most 4
    const int bs_log2 = 31 - __clz(a.block_size);
    const int32_t* table = a.tables + row * a.table_stride;
    auto entry = [&](int s) {
        const int j = lo + s * kKeys + lane * gran;
        return lane < pages && s < tiles && j < hi ? table[j >> bs_log2] : 0;
    };
    int next = warp == 4 ? entry(0) : 0;
    fence_async_shared();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = __shfl_sync(~0u, bars->tmem, 0);
    volatile int* abort = &bars->abort;
    // the rows written and the queries made by the launches ahead are complete from here on; the launch behind may be placed
    spk_grid_wait();
    spk_grid_release();

    if (warp == 4) {  // ---- cache rows
        const SpkPageLayout lay = spk_latent_layout(a.block_size, a.rank_pad, a.rot_pad, 1);
        const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(a.pool);
        int issued = 0;
        for (int s = 0; s < tiles; ++s) {
            const int mine = next;
            next = entry(s + 1);
            const int st = s % NS, j0 = lo + s * kKeys;
            const int n = (min(kKeys, hi - j0) + gran - 1) / gran;
            // waits are made warp-uniform: a vote also brings the lanes back together
            if (s >= NS && !__all_sync(~0u, mbar_wait(smem_u32(&bars->free[st]), ((s / NS) - 1) & 1, abort))) break;
            const uint32_t bar = smem_u32(&bars->full[st]);
            if (lane == 0) mbar_expect(bar, static_cast<uint32_t>(n * gran * CT * 128));
            __syncwarp();
            if (lane < n) {
                int64_t block = mine;
                if (block < 0 || block >= a.num_blocks) {
                    spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
                    block = 0;
                }
                const __nv_bfloat16* src = pool + spk_page_base(lay, block, 0) + ((j0 + lane * gran) & (a.block_size - 1)) * (CT * 64);
                bulk_load(smem_u32(base + st * Sh::kStage) + lane * gran * CT * 128, src, gran * CT * 128, bar);
            }
            issued = s + 1;
        }
        if (*abort != 0)  // copies in flight land before the CTA's shared memory is given up
            for (int s = issued > NS ? issued - NS : 0; s < issued; ++s) mbar_wait(smem_u32(&bars->full[s % NS]), (s / NS) & 1);
    } else if (warp == 5) {  // ---- scores
        constexpr uint32_t idesc = idesc_bf16(kKeys, kHeads, false, false);
        const uint32_t who = elect_one();
        // descriptors of one operand differ in the start address alone
        const uint64_t kd0 = desc_sw128(smem_u32(base), 16, Sh::kGroup), qd = desc_sw128(smem_u32(q_s), 16, 1024);
        bool ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->q_full), 0, abort));
        for (int s = 0; ok && s < tiles; ++s) {
            const int st = s % NS;
            // the buffer's previous scores have been read when that step's weights are complete
            ok = __all_sync(~0u, (s < 2 || mbar_wait(smem_u32(&bars->p_full[s & 1]), ((s >> 1) - 1) & 1, abort)) &&
                                     mbar_wait(smem_u32(&bars->full[st]), (s / NS) & 1, abort));
            if (!ok) break;
            tc_fence_after();
            const uint64_t kd = kd0 + (st * Sh::kStage >> 4);
#pragma unroll
            for (int k = 0; k < CT * 4; ++k)
                mma_ss_by(who, tmem + (s & 1) * kHeads, kd + (((k >> 2) * kAtom + (k & 3) * 32) >> 4), qd + (((k >> 2) * kQTile + (k & 3) * 32) >> 4), idesc, k > 0);
            if (who) mma_commit(smem_u32(&bars->s_full[s & 1]));
            __syncwarp();
        }
        if (who) mma_commit(smem_u32(&bars->s_done));
        mbar_wait(smem_u32(&bars->s_done), 0);  // nothing this warp issued is in the tensor pipe any more
    } else if (warp == 6) {  // ---- weighted sums
        constexpr uint32_t idesc = idesc_bf16(128, 2 * kHeads, true, true);
        const uint32_t who = elect_one();
        const uint64_t vd0 = desc_sw128(smem_u32(base), kAtom, Sh::kGroup), pd0 = desc_sw128(smem_u32(p_s), 16, 1024);
        for (int s = 0; s < tiles; ++s) {
            const int st = s % NS;
            if (!__all_sync(~0u, mbar_wait(smem_u32(&bars->p_full[s & 1]), (s >> 1) & 1, abort))) break;
            tc_fence_after();
            const uint64_t vd = vd0 + (st * Sh::kStage >> 4), pd = pd0 + ((s & 1) * kPTile >> 4);
            const int steps = (min(kKeys, hi - lo - s * kKeys) + 15) >> 4;
#pragma unroll
            for (int k = 0; k < kKeys / 16; ++k) {
                if (k >= steps) break;
#pragma unroll
                for (int b = 0; b < MB; ++b)
                    mma_ss_by(who, tmem + kTmemO + b * 2 * kHeads, vd + ((b * 2 * kAtom + k * 2 * Sh::kGroup) >> 4), pd + (k * 2048 >> 4), idesc, s > 0 || k > 0);
            }
            if (who) {
                mma_commit(smem_u32(&bars->free[st]));
                mma_commit(smem_u32(&bars->p_free[s & 1]));
            }
            __syncwarp();
        }
        if (who) mma_commit(smem_u32(&bars->o_full));
        mbar_wait(smem_u32(&bars->o_full), 0);
    } else if (warp < 4) {  // ---- scores to weights
        // query rows into the operand layout, zeros beyond the heads
        const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + (t * a.heads + h0) * (CT * 64);
#pragma unroll 6
        for (int i = threadIdx.x; i < kHeads * CT * 8; i += kSoftThreads) {
            const int r = i / (CT * 8), c = i % (CT * 8);
            cp_async16(smem_u32(q_s) + (c >> 3) * kQTile + r * 128 + (((c & 7) ^ (r & 7)) << 4), q + (r < nh ? r * (CT * 64) + c * 8 : 0), r < nh);
        }
        cp_async_commit();
        cp_async_wait_all();
        fence_async_shared();
        mbar_arrive(smem_u32(&bars->q_full));
        const uint32_t lanes = static_cast<uint32_t>(warp * 32) << 16;
        const int kr = warp * 16 + (lane >> 2), hc = 2 * (lane & 3);  // this lane's keys kr, kr + 8; heads 8 g + hc, + 1
        const float c1 = a.scale * kLog2e;
        const int groups = (nh + 7) >> 3;
        float ref_own = -INFINITY;  // reference of head `lane`
        float ref[8], den[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) ref[i] = den[i] = 0.0f;
        // a warp that gave up waiting goes on without waiting: the others may stand at a barrier that needs it
        for (int s = 0; s < tiles; ++s) {
            const int buf = s & 1, st = s % NS, valid = min(kKeys, hi - lo - s * kKeys);
            __all_sync(~0u, mbar_wait(smem_u32(&bars->s_full[buf]), (s >> 1) & 1, abort));
            tc_fence_after();
            uint32_t sc[16];
            tmem_ld_frag(tmem + lanes + buf * kHeads, sc);
            float x[4][4];
            float top[8];
            const bool in0 = kr < valid, in1 = kr + 8 < valid;
#pragma unroll
            for (int g = 0; g < 4; ++g) {
#pragma unroll
                for (int i = 0; i < 4; ++i) x[g][i] = (i < 2 ? in0 : in1) ? __uint_as_float(sc[4 * g + i]) * c1 : -INFINITY;
                top[2 * g] = fmaxf(x[g][0], x[g][2]);
                top[2 * g + 1] = fmaxf(x[g][1], x[g][3]);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                if ((i >> 1) < groups) {
                    top[i] = fmaxf(top[i], __shfl_xor_sync(~0u, top[i], 4));
                    top[i] = fmaxf(top[i], __shfl_xor_sync(~0u, top[i], 8));
                    top[i] = fmaxf(top[i], __shfl_xor_sync(~0u, top[i], 16));
                }
            }
            if (lane < 4) {
#pragma unroll
                for (int i = 0; i < 8; ++i) bars->top[buf][warp][8 * (i >> 1) + hc + (i & 1)] = top[i];
            }
            soft_barrier();
            const float most = fmaxf(fmaxf(bars->top[buf][0][lane], bars->top[buf][1][lane]), fmaxf(bars->top[buf][2][lane], bars->top[buf][3][lane]));
            // every warp sees the same maxima and comes to the same decision
            if (__any_sync(~0u, lane < nh && most > ref_own + kSlack)) {
                const float fresh = lane < nh ? fmaxf(most, ref_own) : 0.0f;
                const float fix = s == 0 || lane >= nh ? 0.0f : exp2f(ref_own - fresh);
                ref_own = fresh;
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const int src = 8 * (i >> 1) + hc + (i & 1);
                    ref[i] = __shfl_sync(~0u, fresh, src);
                    den[i] *= __shfl_sync(~0u, fix, src);
                }
                if (s > 0) {
                    if (warp == 0) bars->fix[lane] = fix;
                    __all_sync(~0u, mbar_wait(smem_u32(&bars->p_free[buf ^ 1]), ((s - 1) >> 1) & 1, abort));  // every sum issued so far is in
                    soft_barrier();
                    tc_fence_after();
#pragma unroll 1
                    for (int b = 0; b < 2 * MB; ++b) {
                        uint32_t o[32], lo16[16], hi16[16];
                        const uint32_t at = tmem + lanes + kTmemO + b * kHeads;
                        tmem_ld32(at, o);
                        tmem_wait_ld(o);
#pragma unroll
                        for (int i = 0; i < 16; ++i) {
                            lo16[i] = __float_as_uint(__uint_as_float(o[i]) * bars->fix[i]);
                            hi16[i] = __float_as_uint(__uint_as_float(o[16 + i]) * bars->fix[16 + i]);
                        }
                        tmem_st16(at, lo16);
                        tmem_st16(at + 16, hi16);
                    }
                    tmem_wait_st();
                    soft_barrier();  // the factors have been read
                }
            }
            if (s >= 2) __all_sync(~0u, mbar_wait(smem_u32(&bars->p_free[buf]), ((s >> 1) - 1) & 1, abort));
            uint8_t* p = p_s + buf * kPTile;
#pragma unroll
            for (int g = 0; g < 4; ++g) {
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    uint32_t hi2 = 0u, lo2 = 0u;
                    if (g < groups) {
                        const float p0 = ex2(x[g][2 * r] - ref[2 * g]), p1 = ex2(x[g][2 * r + 1] - ref[2 * g + 1]);
                        den[2 * g] += p0;
                        den[2 * g + 1] += p1;
                        split_bf16(p0, p1, hi2, lo2);
                    }
                    const int key = kr + 8 * r;
                    uint8_t* dst = p + key * 128 + (hc << 1);
                    *reinterpret_cast<uint32_t*>(dst + ((g ^ (key & 7)) << 4)) = hi2;
                    *reinterpret_cast<uint32_t*>(dst + (((g + 4) ^ (key & 7)) << 4)) = lo2;
                }
            }
            if ((valid & 15) != 0 && valid < kKeys) {  // the last step: rows beyond the range may hold anything, and 0 * NaN is NaN
                __all_sync(~0u, mbar_wait(smem_u32(&bars->full[st]), (s / NS) & 1, abort));
                const int end = (valid + 15) & ~15;
                for (int i = threadIdx.x; i < (end - valid) * CL * 8; i += kSoftThreads) {
                    const int c = i / ((end - valid) * 8), rest = i % ((end - valid) * 8), r = valid + (rest >> 3);
                    *reinterpret_cast<uint4*>(base + st * Sh::kStage + (r >> 3) * Sh::kGroup + c * kAtom + (r & 7) * 128 + ((rest & 7) << 4)) =
                        make_uint4(0u, 0u, 0u, 0u);
                }
            }
            fence_async_shared();
            tc_fence_before();
            mbar_arrive(smem_u32(&bars->p_full[buf]));
        }
        // denominators: over this warp's keys, then over the warps
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            den[i] += __shfl_xor_sync(~0u, den[i], 4);
            den[i] += __shfl_xor_sync(~0u, den[i], 8);
            den[i] += __shfl_xor_sync(~0u, den[i], 16);
        }
        soft_barrier();
        if (lane < 4) {
#pragma unroll
            for (int i = 0; i < 8; ++i) bars->top[0][warp][8 * (i >> 1) + hc + (i & 1)] = den[i];
        }
        soft_barrier();
        if (warp == 0 && lane < nh) {
            const float total = (bars->top[0][0][lane] + bars->top[0][1][lane]) + (bars->top[0][2][lane] + bars->top[0][3][lane]);
            *reinterpret_cast<float2*>(a.stats + 2 * ((t * a.splits + blockIdx.z) * a.heads + h0 + lane)) = make_float2(ref_own / kLog2e, total);
        }
    }
    __syncwarp();
    __syncthreads();  // every part has ended; the last one waited for the sums
    {  // ---- all warps write the sums: a warp reaches the lanes of its quarter, the two halves of the CTA take turns at the blocks
        const bool ok = *abort == 0;
        tc_fence_after();
        const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const int64_t rec = (t * a.splits + blockIdx.z) * a.heads + h0;
#pragma unroll 1
        for (int b = warp >> 2; b < MB; b += 2) {
            const int c = b * 128 + (warp & 3) * 32 + lane;
            uint32_t x[32], y[32];
            tmem_ld32(tmem + lanes + kTmemO + b * 2 * kHeads, x);
            tmem_ld32(tmem + lanes + kTmemO + b * 2 * kHeads + kHeads, y);
            tmem_wait_ld(x);
            tmem_wait_ld(y);
            if (c < a.rank) {
                float* dst = a.partials + rec * a.rank + c;
#pragma unroll
                for (int i = 0; i < kHeads; ++i)
                    if (i < nh) dst[static_cast<int64_t>(i) * a.rank] = ok ? __uint_as_float(x[i]) + __uint_as_float(y[i]) : 0.0f;
            }
            __syncwarp();
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (threadIdx.x == 0 && *abort != 0) spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
    if (warp == 0) tmem_dealloc(tmem, Sh::kColumns);
}

template <int CL>
int launch(const spk_latent_attn_args& a, cudaStream_t s) {
    constexpr int bytes = Shape<CL>::kBytes;
    static_assert(sizeof(Bars) <= 1536 && bytes <= 227 * 1024, "shared memory");
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    const dim3 grid(static_cast<unsigned>(a.n), (a.heads + kHeads - 1) / kHeads, a.splits);
    return spk_launch(latent_decode_kernel<CL>, grid, kThreads, bytes, s, a.overlap != 0, a);
}

}  // namespace

int spk_latent_decode_splits(int64_t n, int heads, int64_t max_keys) {
    // ranges whose waves of CTAs take least: a step of 64 keys is one unit, a CTA's set-up and its partial sums about five
    const int64_t ctas = n * ((heads + kHeads - 1) / kHeads);
    int best = 1;
    int64_t least = INT64_MAX;
    for (int s = 1; s <= 64 && (s == 1 || static_cast<int64_t>(s) * 128 <= max_keys); ++s) {
        const int64_t cost = (ctas * s + 147) / 148 * (spk_split_keys(static_cast<int>(max_keys), s) / kKeys + 5);
        if (cost < least) {
            least = cost;
            best = s;
        }
    }
    return best;
}

int spk_latent_decode_launch(const spk_latent_attn_args& a, cudaStream_t s) {
    switch (a.rank_pad / 64) {
        case 1: return launch<1>(a, s);
        case 2: return launch<2>(a, s);
        case 3: return launch<3>(a, s);
        case 4: return launch<4>(a, s);
        case 5: return launch<5>(a, s);
        case 6: return launch<6>(a, s);
        case 7: return launch<7>(a, s);
        default: return launch<8>(a, s);
    }
}
