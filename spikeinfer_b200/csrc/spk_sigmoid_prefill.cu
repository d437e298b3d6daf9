// Prefill attention with sigmoid key weights on the fifth-generation tensor cores (tcgen05), bf16, head sizes up to 128.
//
// CTA = (128 query tokens of one portion, query head).  Twenty warps:
//  * warps 16 and 19 copy K and V: a page of the pool is stored as the swizzled operand tile it becomes, so a 128-key tile is a
//    handful of plain bulk copies (cp.async.bulk), no tensor map, whatever pages the block table names; one copy per lane, the
//    next tile's block-table entries are read ahead;
//  * warp 17 (one thread) issues S = Q K^T into one of two TMEM buffers, warp 18 (one thread) O += P V with P read from TMEM,
//    so that neither kind of MMA waits behind the other's operands;
//  * warps 0-15 turn scores into weights: warpgroups 0 and 2 the two column halves of the even tiles, 1 and 3 those of the odd
//    ones, one thread per query row and half.  The work is latency-bound, hence many warps of few registers.
// A weight is sigmoid(score) of its own key: no running maximum, no rescaling of O, no denominator.  Weights are computed in
// 32 bits and enter the product as a bf16 pair (hi + lo: 16 significant bits), so O is a 32-bit sum of them to 2^-17.
// Visible keys are those up to the query's own position; the last tile's rows of V beyond the portion's end are cleared in
// shared memory (a page's unwritten rows may hold anything, and 0 * NaN is NaN).
#include "spk_paged_attn.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kTile = 128;            // query rows, and keys per step
constexpr int kColTile = kTile * 128; // bytes of a 64-channel column tile
constexpr int kSigmoidThreads = 512;
constexpr int kThreads = kSigmoidThreads + 128;
constexpr uint32_t kTmemS = 0, kTmemLo = 256, kTmemO = 384;  // S/P-hi buffers 2 x 128, P-lo 2 x 64, O up to 128
constexpr float kLog2e = 1.4426950408889634f;

template <int CK, int CV>
struct Shape {
    static constexpr int NS = CK + CV <= 2 ? 4 : 2;  // stages of K and of V
    static constexpr int kK = CK * kColTile, kV = CV * kColTile;
    static constexpr int kBytes = kK + NS * (kK + kV) + 1024 + 256;
};

struct Bars {
    uint64_t k_full[4], k_free[4], v_full[4], v_free[4], s_full[2], p_full[2], p_free[2], o_full, q_full, s_done;
    int abort;
    uint32_t tmem;
};

template <int CK, int CV>
__global__ void __launch_bounds__(kThreads, 1)
sigmoid_prefill_kernel(const spk_sigmoid_attn_args a) {
    using Sh = Shape<CK, CV>;
    constexpr int NS = Sh::NS;
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 1023) & ~uintptr_t(1023));
    uint8_t* q_s = base;
    uint8_t* k_s = q_s + Sh::kK;
    uint8_t* v_s = k_s + NS * Sh::kK;
    Bars* bars = reinterpret_cast<Bars*>(v_s + NS * Sh::kV);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    const int h = blockIdx.x;
    const int g = h / (a.heads / a.kv_heads);
    const int4 tile = reinterpret_cast<const int4*>(a.tiles)[blockIdx.y];
    const int64_t t0 = tile.x;
    const int nq = tile.y, row = tile.z, pos0 = tile.w;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + t0 * a.out_stride + static_cast<int64_t>(h) * a.vdim;
    // uniform over the CTA: nothing has been set up yet
    if (row < 0 || row >= a.table_rows || pos0 < 0 || nq < 1 || nq > kTile ||
        static_cast<int64_t>(pos0) + nq > a.max_blocks * a.block_size) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        for (int i = threadIdx.x; i < nq * a.vdim && nq <= kTile; i += kThreads)
            out[(i / a.vdim) * a.out_stride + i % a.vdim] = __float2bfloat16_rn(0.0f);
        return;
    }
    const int keys = pos0 + nq;
    const int tiles = (keys + kTile - 1) / kTile;

    if (threadIdx.x == 0) {
        for (int i = 0; i < NS; ++i) {
            mbar_init(smem_u32(&bars->k_full[i]), 1);
            mbar_init(smem_u32(&bars->k_free[i]), 1);
            mbar_init(smem_u32(&bars->v_full[i]), 1);
            mbar_init(smem_u32(&bars->v_free[i]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&bars->s_full[i]), 1);
            mbar_init(smem_u32(&bars->p_full[i]), 256);
            mbar_init(smem_u32(&bars->p_free[i]), 1);
        }
        mbar_init(smem_u32(&bars->o_full), 1);
        mbar_init(smem_u32(&bars->s_done), 1);
        mbar_init(smem_u32(&bars->q_full), kSigmoidThreads);
        bars->abort = 0;
    }
    if (warp == 0) tmem_alloc(smem_u32(&bars->tmem), 512);
    fence_async_shared();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem;
    volatile int* abort = &bars->abort;

    if (warp == 16 || warp == 19) {  // ---- K or V copies
        const bool is_k = warp == 16;
        const int cols = is_k ? CK : CV;
        const int gran = a.block_size < kTile ? a.block_size : kTile;  // rows per copy
        const int per = kTile / gran;                                  // copies per column tile, at most 8
        const int p = lane % per, c = lane / per;                      // this lane's copy
        const int bs_log2 = 31 - __clz(a.block_size);
        const int32_t* table = a.tables + static_cast<int64_t>(row) * a.table_stride;
        const SpkPageLayout lay{a.kv_heads, a.block_size, is_k ? a.k_pad : a.v_pad, 1};
        const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(is_k ? a.k_pool : a.v_pool);
        uint8_t* stages = is_k ? k_s : v_s;
        const int stage_bytes = is_k ? Sh::kK : Sh::kV;
        uint64_t* full = is_k ? bars->k_full : bars->v_full;
        uint64_t* free = is_k ? bars->k_free : bars->v_free;
        auto entry = [&](int t) {
            const int j = t * kTile + p * gran;
            return t < tiles && j < keys ? table[j >> bs_log2] : 0;
        };
        int next = entry(0);
        int issued = 0;
        for (int t = 0; t < tiles; ++t) {
            int64_t block = next;
            next = entry(t + 1);
            const int stage = t % NS;
            const int valid = keys - t * kTile < kTile ? keys - t * kTile : kTile;
            const int n = (valid + gran - 1) / gran;
            // waits are made warp-uniform: a vote also brings the lanes back together
            if (t >= NS && !__all_sync(~0u, mbar_wait(smem_u32(free + stage), ((t / NS) - 1) & 1, abort))) break;
            const uint32_t bar = smem_u32(full + stage);
            if (lane == 0) mbar_expect(bar, static_cast<uint32_t>(n * cols * gran * 128));
            __syncwarp();
            if (p < n && c < cols) {
                if (block < 0 || block >= a.num_blocks) {
                    spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
                    block = 0;
                }
                const int j = t * kTile + p * gran;
                const __nv_bfloat16* src = pool + spk_page_base(lay, block, g) + (c << (bs_log2 + 6)) + ((j & (a.block_size - 1)) << 6);
                bulk_load(smem_u32(stages + stage * stage_bytes) + c * kColTile + p * gran * 128, src, gran * 128, bar);
            }
            issued = t + 1;
        }
        if (*abort != 0)  // copies in flight land before the CTA's shared memory is given up
            for (int t = issued > NS ? issued - NS : 0; t < issued; ++t) mbar_wait(smem_u32(full + t % NS), (t / NS) & 1);
    } else if (warp == 17) {  // ---- scores
        if (lane == 0) {
            constexpr uint32_t idesc = idesc_bf16(kTile, kTile, false, false);
            bool ok = mbar_wait(smem_u32(&bars->q_full), 0, abort);
            for (int t = 0; ok && t < tiles; ++t) {
                const int stage = t % NS;
                // the buffer's previous weights (tile t - 2) have been multiplied
                ok = (t < 2 || mbar_wait(smem_u32(&bars->p_free[t & 1]), ((t >> 1) - 1) & 1, abort)) &&
                     mbar_wait(smem_u32(&bars->k_full[stage]), (t / NS) & 1, abort);
                if (!ok) break;
                tc_fence_after();
                const uint32_t qa = smem_u32(q_s), kb = smem_u32(k_s + stage * Sh::kK);
#pragma unroll
                for (int s = 0; s < CK * 4; ++s) {
                    const uint32_t off = (s >> 2) * kColTile + (s & 3) * 32;
                    mma_ss(tmem + kTmemS + (t & 1) * 128, desc_sw128(qa + off, 16, 1024), desc_sw128(kb + off, 16, 1024), idesc, s > 0);
                }
                mma_commit(smem_u32(&bars->k_free[stage]));
                mma_commit(smem_u32(&bars->s_full[t & 1]));
            }
            mma_commit(smem_u32(&bars->s_done));
            mbar_wait(smem_u32(&bars->s_done), 0);  // nothing this thread issued is in the tensor pipe any more
        }
    } else if (warp == 18) {  // ---- weighted sums
        if (lane == 0) {
            constexpr uint32_t idesc = idesc_bf16(kTile, CV * 64, false, true);
            for (int t = 0; t < tiles; ++t) {
                const int stage = t % NS, buf = t & 1;
                if (!mbar_wait(smem_u32(&bars->v_full[stage]), (t / NS) & 1, abort) ||
                    !mbar_wait(smem_u32(&bars->p_full[buf]), (t >> 1) & 1, abort))
                    break;
                tc_fence_after();
                const uint32_t vb = smem_u32(v_s + stage * Sh::kV);
                const int valid = keys - t * kTile < kTile ? keys - t * kTile : kTile;
                const int steps = (valid + 15) >> 4;
                for (int s = 0; s < steps; ++s) {
                    const uint64_t vd = desc_sw128(vb + s * 2048, kColTile, 1024);
                    // a half's weights lie in its own half of the score buffer
                    mma_ts(tmem + kTmemO, tmem + kTmemS + buf * 128 + (s >> 2) * 64 + (s & 3) * 8, vd, idesc, t > 0 || s > 0);
                    mma_ts(tmem + kTmemO, tmem + kTmemLo + buf * 64 + s * 8, vd, idesc, true);
                }
                mma_commit(smem_u32(&bars->p_free[buf]));
                mma_commit(smem_u32(&bars->v_free[stage]));
            }
            mma_commit(smem_u32(&bars->o_full));
            mbar_wait(smem_u32(&bars->o_full), 0);
        }
    } else {  // ---- scores to weights
        // Q rows into the swizzled operand layout, zeros beyond the portion
        for (int i = threadIdx.x; i < kTile * CK * 8; i += kSigmoidThreads) {
            const int r = i / (CK * 8), c = i % (CK * 8);
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (r < nq)
                v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q) + ((t0 + r) * a.heads + h) * a.k_pad + c * 8);
            *reinterpret_cast<uint4*>(q_s + (c >> 3) * kColTile + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
        }
        fence_async_shared();
        mbar_arrive(smem_u32(&bars->q_full));
        const int wg = (warp >> 2) & 1, half = warp >> 3;  // tile parity, column half
        const int r = (warp & 3) * 32 + lane;
        const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const uint64_t c1 = f2_pack(-a.scale * kLog2e, -a.scale * kLog2e), c0 = f2_pack(-a.head_bias[h] * kLog2e, -a.head_bias[h] * kLog2e);
        bool ok = true;
        for (int t = wg; t < tiles; t += 2) {
            const int stage = t % NS;
            ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->s_full[wg]), (t >> 1) & 1, abort));
            if (!ok) break;
            tc_fence_after();
            const int last = pos0 + r - t * kTile;  // last visible column of this row
            const uint32_t sa = tmem + lanes + kTmemS + wg * 128 + half * 64, la = tmem + lanes + kTmemLo + wg * 64 + half * 32;
            // 32 score columns at a time; the hi parts overlay columns of this half that have been read (16 c + 15 < 32 (c + 1))
#pragma unroll 1
            for (int c = 0; c < 2; ++c) {
                uint32_t sc[32];
                tmem_ld32(sa + c * 32, sc);
                tmem_wait_ld(sc);
                uint32_t hi[16], lo[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    float p0, p1;
                    sigmoid2(f2_fma(f2_pack(__uint_as_float(sc[2 * i]), __uint_as_float(sc[2 * i + 1])), c1, c0), p0, p1);
                    split_bf16(p0, p1, hi[i], lo[i]);
                }
                const int seen = last - half * 64 - c * 32;
                if (!__all_sync(~0u, seen >= 31)) {
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const uint32_t m = (2 * i <= seen ? 0xffffu : 0u) | (2 * i + 1 <= seen ? 0xffff0000u : 0u);
                        hi[i] &= m;
                        lo[i] &= m;
                    }
                }
                tmem_st16(sa + c * 16, hi);
                tmem_st16(la + c * 16, lo);
            }
            tmem_wait_st();
            const int valid = keys - t * kTile;
            if (valid < kTile && (valid & 15) != 0) {  // the last tile: clear the V rows its last MMA step reads beyond the end
                ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->v_full[stage]), (t / NS) & 1, abort));
                if (!ok) break;
                const int end = (valid + 15) & ~15;
                for (int i = half * 128 + r; i < (end - valid) * CV * 8; i += 256) {
                    const int c = i / ((end - valid) * 8), rest = i % ((end - valid) * 8);
                    *reinterpret_cast<uint4*>(v_s + stage * Sh::kV + c * kColTile + (valid + (rest >> 3)) * 128 + ((rest & 7) << 4)) =
                        make_uint4(0u, 0u, 0u, 0u);
                }
                fence_async_shared();
            }
            tc_fence_before();
            mbar_arrive(smem_u32(&bars->p_full[wg]));
        }
        ok = __all_sync(~0u, ok && mbar_wait(smem_u32(&bars->o_full), 0, abort) && *abort == 0);
        tc_fence_after();
        const bool vec = a.vdim % 8 == 0 && a.out_stride % 8 == 0 && reinterpret_cast<uintptr_t>(a.out) % 16 == 0;
        if (const int col = (warp >> 2) * 32; col < CV * 64) {  // a warpgroup writes 32 columns of the output
            uint32_t o[32];
            tmem_ld32(tmem + lanes + kTmemO + col, o);
            tmem_wait_ld(o);
            __nv_bfloat16* dst = out + r * a.out_stride + col;
            if (r < nq && vec) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (col + 8 * i >= a.vdim) break;
                    uint4 v;
                    uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        w[k] = ok ? pack_bf16(__uint_as_float(o[8 * i + 2 * k]) * a.out_scale, __uint_as_float(o[8 * i + 2 * k + 1]) * a.out_scale) : 0u;
                    *reinterpret_cast<uint4*>(dst + 8 * i) = v;
                }
            } else if (r < nq) {
#pragma unroll
                for (int i = 0; i < 32; ++i)
                    if (col + i < a.vdim) dst[i] = __float2bfloat16_rn(ok ? __uint_as_float(o[i]) * a.out_scale : 0.0f);
            }
            __syncwarp();
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    if (threadIdx.x == 0 && *abort != 0) spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
    if (warp == 0) tmem_dealloc(tmem, 512);
}

template <int CK, int CV>
int launch(const spk_sigmoid_attn_args& a, cudaStream_t s) {
    constexpr int bytes = Shape<CK, CV>::kBytes;
    static_assert(sizeof(Bars) <= 256 && bytes <= 227 * 1024, "shared memory");
    const cudaError_t e = cudaFuncSetAttribute(sigmoid_prefill_kernel<CK, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    sigmoid_prefill_kernel<CK, CV><<<dim3(a.heads, a.n_tiles), kThreads, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

int spk_sigmoid_prefill_launch(const spk_sigmoid_attn_args& a, cudaStream_t s) {
    if (a.n_tiles > 65535) return SPK_ERR_TOO_LARGE;
    const int ck = a.k_pad / 64, cv = a.v_pad / 64;
    if (ck == 1 && cv == 1) return launch<1, 1>(a, s);
    if (ck == 1 && cv == 2) return launch<1, 2>(a, s);
    if (ck == 2 && cv == 1) return launch<2, 1>(a, s);
    return launch<2, 2>(a, s);
}
