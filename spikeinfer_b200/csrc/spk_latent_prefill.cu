// Prefill attention over a shared latent with keys and values spelled out per head: tcgen05, bf16, softmax with a sink.
//
// For long portions it is cheaper to spell the heads' keys and values out once (one library product over the sequence's latents) than to
// take every query into the latent space.  latent_gather_kernel brings a sequence's cache rows out of its pages; the attention reads
// the product's rows in place through two tensor maps (keys and values | the rotated part all heads share).
//
// CTA = (128 query tokens of one portion, head).  Warps:
//  * warp 12 copies K and V tiles of 128 keys with TMA (cp.async.bulk.tensor);
//  * warp 13 (one thread) issues S = Q K^T into one of three TMEM buffers, warp 14 (one thread) O += P V with P read from TMEM;
//  * warpgroups 0-2 take the key tiles in turn, one thread per query row.  A tile's weights are exp2(score - reference), 32-bit, and enter
//    the product as a bf16 pair (hi + lo).  The row's reference is handed from tile to tile; it only moves when a score exceeds it by
//    2^8, and the warp that moves it rescales O.
// The rotated query part is turned on the way into shared memory; the epilogue adds the sink, divides and applies the output gate.
#include <cuda.h>

#include "spk_latent.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kTile = 128;
constexpr int kColTile = kTile * 128;  // bytes of a 64-channel column tile
constexpr int NB = 3;                  // score buffers and warpgroups
constexpr int kSoftThreads = NB * 128;
constexpr int kThreads = kSoftThreads + 96;
constexpr uint32_t kTmemO = NB * 128;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kSlack = 8.0f;

template <int CK, int CV>  // column tiles of K (the rotated one included) and V
struct Shape {
    static constexpr int kK = CK * kColTile, kV = CV * kColTile;
    static constexpr int NS = CK + CV <= 3 ? 3 : 2;
    static constexpr int kBytes = kK + NS * (kK + kV) + 1024 + 4608;
};

struct Bars {
    uint64_t k_full[3], k_free[3], v_full[3], v_free[3], s_full[NB], p_full[NB], p_free[NB], ref_full[NB], q_full, o_full, s_done;
    int abort;
    uint32_t tmem;
    float ref[NB][kTile];
    float den[NB][kTile];
};

__device__ __forceinline__ void tma_load(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"(dst), "l"(map), "r"(x), "r"(y), "r"(bar) : "memory");
}

template <int CK, int CV>
__global__ void __launch_bounds__(kThreads, 1)
latent_prefill_kernel(const spk_latent_prefill_args a, const __grid_constant__ CUtensorMap kv_map, const __grid_constant__ CUtensorMap kr_map) {
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
    const int4 tile = reinterpret_cast<const int4*>(a.tiles)[blockIdx.y];  // first token, tokens, first context row, position of the first token
    const int64_t t0 = tile.x;
    const int nq = tile.y, row0 = tile.z, pos0 = tile.w;
    // uniform over the CTA: nothing has been set up yet
    if (t0 < 0 || nq < 1 || nq > kTile || t0 + nq > a.n || row0 < 0 || pos0 < 0 || static_cast<int64_t>(row0) + pos0 + nq > a.n_ctx) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
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
        for (int i = 0; i < NB; ++i) {
            mbar_init(smem_u32(&bars->s_full[i]), 1);
            mbar_init(smem_u32(&bars->p_full[i]), 128);
            mbar_init(smem_u32(&bars->p_free[i]), 1);
            mbar_init(smem_u32(&bars->ref_full[i]), 128);
        }
        mbar_init(smem_u32(&bars->q_full), kSoftThreads);
        mbar_init(smem_u32(&bars->o_full), 1);
        mbar_init(smem_u32(&bars->s_done), 1);
        bars->abort = 0;
    }
    if (warp == 0) tmem_alloc(smem_u32(&bars->tmem), 512);
    fence_async_shared();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = bars->tmem;
    volatile int* abort = &bars->abort;

    if (warp == 12) {  // ---- K and V
        if (lane == 0) {
            int ik = 0, iv = 0;
            for (int t = 0; t < tiles; ++t) {
                const int st = t % NS, y = row0 + t * kTile;
                if (t >= NS && !mbar_wait(smem_u32(&bars->k_free[st]), ((t / NS) - 1) & 1, abort)) break;
                uint32_t bar = smem_u32(&bars->k_full[st]), dst = smem_u32(k_s + st * Sh::kK);
                mbar_expect(bar, Sh::kK);
#pragma unroll
                for (int c = 0; c < CK - 1; ++c) tma_load(dst + c * kColTile, &kv_map, h * a.dim_pad + c * 64, y, bar);
                tma_load(dst + (CK - 1) * kColTile, &kr_map, 0, y, bar);
                ik = t + 1;
                if (t >= NS && !mbar_wait(smem_u32(&bars->v_free[st]), ((t / NS) - 1) & 1, abort)) break;
                bar = smem_u32(&bars->v_full[st]);
                dst = smem_u32(v_s + st * Sh::kV);
                mbar_expect(bar, Sh::kV);
#pragma unroll
                for (int c = 0; c < CV; ++c) tma_load(dst + c * kColTile, &kv_map, a.heads * a.dim_pad + h * a.vdim_pad + c * 64, y, bar);
                iv = t + 1;
            }
            if (*abort != 0) {  // copies in flight land before the CTA's shared memory is given up
                for (int t = ik > NS ? ik - NS : 0; t < ik; ++t) mbar_wait(smem_u32(&bars->k_full[t % NS]), (t / NS) & 1);
                for (int t = iv > NS ? iv - NS : 0; t < iv; ++t) mbar_wait(smem_u32(&bars->v_full[t % NS]), (t / NS) & 1);
            }
        }
    } else if (warp == 13) {  // ---- scores
        if (lane == 0) {
            constexpr uint32_t idesc = idesc_bf16(kTile, kTile, false, false);
            bool ok = mbar_wait(smem_u32(&bars->q_full), 0, abort);
            for (int t = 0; ok && t < tiles; ++t) {
                const int st = t % NS, buf = t % NB;
                // the buffer's previous weights have been multiplied
                ok = (t < NB || mbar_wait(smem_u32(&bars->p_free[buf]), ((t / NB) - 1) & 1, abort)) &&
                     mbar_wait(smem_u32(&bars->k_full[st]), (t / NS) & 1, abort);
                if (!ok) break;
                tc_fence_after();
                const uint32_t qa = smem_u32(q_s), kb = smem_u32(k_s + st * Sh::kK);
#pragma unroll
                for (int s = 0; s < CK * 4; ++s) {
                    const uint32_t off = (s >> 2) * kColTile + (s & 3) * 32;
                    mma_ss(tmem + buf * 128, desc_sw128(qa + off, 16, 1024), desc_sw128(kb + off, 16, 1024), idesc, s > 0);
                }
                mma_commit(smem_u32(&bars->k_free[st]));
                mma_commit(smem_u32(&bars->s_full[buf]));
            }
            mma_commit(smem_u32(&bars->s_done));
            mbar_wait(smem_u32(&bars->s_done), 0);  // nothing this thread issued is in the tensor pipe any more
        }
    } else if (warp == 14) {  // ---- weighted sums
        if (lane == 0) {
            constexpr uint32_t idesc = idesc_bf16(kTile, CV * 64, false, true);
            for (int t = 0; t < tiles; ++t) {
                const int st = t % NS, buf = t % NB;
                if (!mbar_wait(smem_u32(&bars->v_full[st]), (t / NS) & 1, abort) || !mbar_wait(smem_u32(&bars->p_full[buf]), (t / NB) & 1, abort)) break;
                tc_fence_after();
                const uint32_t vb = smem_u32(v_s + st * Sh::kV);
                const int steps = (min(kTile, keys - t * kTile) + 15) >> 4;
                for (int s = 0; s < steps; ++s) {
                    const uint64_t vd = desc_sw128(vb + s * 2048, kColTile, 1024);
                    const uint32_t p = tmem + buf * 128 + (s >> 1) * 32 + (s & 1) * 8;  // 32 keys: 16 columns of high, 16 of low parts
                    mma_ts(tmem + kTmemO, p, vd, idesc, t > 0 || s > 0);
                    mma_ts(tmem + kTmemO, p + 16, vd, idesc, true);
                }
                mma_commit(smem_u32(&bars->p_free[buf]));
                mma_commit(smem_u32(&bars->v_free[st]));
            }
            mma_commit(smem_u32(&bars->o_full));
            mbar_wait(smem_u32(&bars->o_full), 0);
        }
    } else {  // ---- scores to weights
        {  // query rows into the operand layout: the unrotated part as it is, the rotated part turned, zeros around
            const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q) + (t0 * a.heads + h) * (a.dim + a.rot_dim);
            const int64_t ld = static_cast<int64_t>(a.heads) * (a.dim + a.rot_dim);
            constexpr int G = (CK - 1) * 8;
            for (int i = threadIdx.x; i < kTile * G; i += kSoftThreads) {
                const int r = i / G, c = i % G;
                uint4 v = make_uint4(0u, 0u, 0u, 0u);
                if (r < nq) {
                    const __nv_bfloat16* src = q + r * ld + c * 8;
                    if (a.vec_q && c * 8 < a.dim) {
                        v = *reinterpret_cast<const uint4*>(src);
                    } else {
                        uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            w[k] = pack_bf16(c * 8 + 2 * k < a.dim ? __bfloat162float(src[2 * k]) : 0.0f, c * 8 + 2 * k + 1 < a.dim ? __bfloat162float(src[2 * k + 1]) : 0.0f);
                    }
                }
                *reinterpret_cast<uint4*>(q_s + (c >> 3) * kColTile + r * 128 + (((c & 7) ^ (r & 7)) << 4)) = v;
            }
            uint8_t* rt = q_s + (CK - 1) * kColTile;
            const int half = a.rot_dim / 2;
            auto at = [&](int r, int c) { return reinterpret_cast<__nv_bfloat16*>(rt + r * 128 + (((c >> 3) ^ (r & 7)) << 4) + (c & 7) * 2); };
            for (int i = threadIdx.x; i < kTile * 32; i += kSoftThreads) {
                const int r = i / 32, c = i % 32;
                if (c < half) {
                    float x = 0.0f, y = 0.0f;
                    if (r < nq) {
                        int64_t pos = static_cast<int64_t>(pos0) + r;
                        if (pos >= a.rot_positions) {
                            spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
                            pos = 0;
                        }
                        const float2 f = reinterpret_cast<const float2*>(a.rot_table)[pos * half + c];
                        const float u = __bfloat162float(q[r * ld + a.dim + c]), w = __bfloat162float(q[r * ld + a.dim + c + half]);
                        x = u * f.x - w * f.y;
                        y = w * f.x + u * f.y;
                    }
                    *at(r, c) = __float2bfloat16_rn(x);
                    *at(r, c + half) = __float2bfloat16_rn(y);
                } else {  // channels 2 half .. 63
                    *at(r, 2 * half + 2 * (c - half)) = __float2bfloat16_rn(0.0f);
                    *at(r, 2 * half + 2 * (c - half) + 1) = __float2bfloat16_rn(0.0f);
                }
            }
        }
        fence_async_shared();
        mbar_arrive(smem_u32(&bars->q_full));
        const int wg = warp >> 2, r = (warp & 3) * 32 + lane;
        const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const float c1 = a.scale * kLog2e;
        float ref = -INFINITY, den = 0.0f;  // the reference this thread's denominator is relative to
        bool ok = true;
        for (int t = wg; t < tiles; t += NB) {
            ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->s_full[wg]), (t / NB) & 1, abort));
            if (!ok) break;
            tc_fence_after();
            const int last = pos0 + r - t * kTile;  // last visible column of this row
            const uint32_t sa = tmem + lanes + wg * 128;
            const bool masked = !__all_sync(~0u, last >= kTile - 1);
            float top = -INFINITY;
#pragma unroll 1
            for (int c = 0; c < 4; ++c) {
                uint32_t sc[32];
                tmem_ld32(sa + c * 32, sc);
                tmem_wait_ld(sc);
                float m0 = -INFINITY, m1 = -INFINITY;
                if (masked) {
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if (c * 32 + i <= last) m0 = fmaxf(m0, __uint_as_float(sc[i]));
                } else {
#pragma unroll
                    for (int i = 0; i < 32; i += 2) {
                        m0 = fmaxf(m0, __uint_as_float(sc[i]));
                        m1 = fmaxf(m1, __uint_as_float(sc[i + 1]));
                    }
                }
                top = fmaxf(top, fmaxf(m0, m1));
            }
            top *= c1;  // the scale is positive
            float fresh = top;
            if (t > 0) {
                ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->ref_full[(t - 1) % NB]), ((t - 1) / NB) & 1, abort));
                if (!ok) break;
                const float before = bars->ref[(t - 1) % NB][r];
                const bool moves = top > before + kSlack;
                fresh = moves ? top : before;
                if (__any_sync(~0u, moves)) {  // every sum issued so far is in, none follows before this tile's weights
                    ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->p_free[(t - 1) % NB]), ((t - 1) / NB) & 1, abort));
                    if (!ok) break;
                    tc_fence_after();
                    const float fix = ex2(before - fresh);
#pragma unroll 1
                    for (int c = 0; c < CV * 4; ++c) {
                        uint32_t o[16];
                        tmem_ld16(tmem + lanes + kTmemO + c * 16, o);
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * fix);
                        tmem_st16(tmem + lanes + kTmemO + c * 16, o);
                    }
                    tmem_wait_st();
                }
            }
            bars->ref[wg][r] = fresh;
            tc_fence_before();
            mbar_arrive(smem_u32(&bars->ref_full[wg]));
            den *= ex2(ref - fresh);
            ref = fresh;
            const uint64_t cc = f2_pack(c1, c1), rr = f2_pack(-fresh, -fresh);
            uint64_t sum = 0;
#pragma unroll 1
            for (int c = 0; c < 4; ++c) {
                uint32_t sc[32];
                tmem_ld32(sa + c * 32, sc);
                tmem_wait_ld(sc);
                uint32_t hi[16], lo[16];
                const int seen = last - c * 32;
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    float u0, u1;
                    f2_unpack(f2_fma(f2_pack(__uint_as_float(sc[2 * i]), __uint_as_float(sc[2 * i + 1])), cc, rr), u0, u1);
                    float p0 = ex2(u0), p1 = ex2(u1);
                    if (masked) {
                        p0 = 2 * i <= seen ? p0 : 0.0f;
                        p1 = 2 * i + 1 <= seen ? p1 : 0.0f;
                    }
                    sum = f2_add(sum, f2_pack(p0, p1));
                    split_bf16(p0, p1, hi[i], lo[i]);
                }
                tmem_st16(sa + c * 32, hi);
                tmem_st16(sa + c * 32 + 16, lo);
            }
            tmem_wait_st();
            float s0, s1;
            f2_unpack(sum, s0, s1);
            den += s0 + s1;
            tc_fence_before();
            mbar_arrive(smem_u32(&bars->p_full[wg]));
        }
        ok = __all_sync(~0u, ok && mbar_wait(smem_u32(&bars->o_full), 0, abort) && *abort == 0);
        tc_fence_after();
        // the last tile's reference holds for O; a group that took no tile contributes nothing
        ok = __all_sync(~0u, mbar_wait(smem_u32(&bars->ref_full[(tiles - 1) % NB]), ((tiles - 1) / NB) & 1, abort)) && ok;
        const float final_ref = bars->ref[(tiles - 1) % NB][r];
        bars->den[wg][r] = ref > -INFINITY ? den * ex2(ref - final_ref) : 0.0f;
        asm volatile("bar.sync 1, %0;" ::"n"(kSoftThreads) : "memory");
        const float total = bars->den[0][r] + bars->den[1][r] + bars->den[2][r] + ex2(a.sink[h] * kLog2e - final_ref);
        const float inv = ok ? 1.0f / total : 0.0f;
        const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(a.gate) + (t0 + r) * a.gate_stride + static_cast<int64_t>(h) * a.vdim;
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (t0 + r) * a.out_stride + static_cast<int64_t>(h) * a.vdim;
#pragma unroll 1
        for (int c = wg; c < CV * 4; c += NB) {  // sixteen columns at a time
            uint32_t o[16];
            tmem_ld16(tmem + lanes + kTmemO + c * 16, o);
            if (r < nq && a.vec_out) {
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int e = c * 16 + i * 8;
                    if (e >= a.vdim) break;
                    const uint4 g = *reinterpret_cast<const uint4*>(gate + e);
                    const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
                    uint4 v;
                    uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        w[k] = pack_bf16(__uint_as_float(o[8 * i + 2 * k]) * inv * sigmoid_fast(__uint_as_float(gw[k] << 16)),
                                         __uint_as_float(o[8 * i + 2 * k + 1]) * inv * sigmoid_fast(__uint_as_float(gw[k] & 0xffff0000u)));
                    *reinterpret_cast<uint4*>(out + e) = v;
                }
            } else if (r < nq) {
#pragma unroll
                for (int i = 0; i < 16; ++i) {
                    const int e = c * 16 + i;
                    if (e < a.vdim) out[e] = __float2bfloat16_rn(__uint_as_float(o[i]) * inv * sigmoid_fast(__bfloat162float(gate[e])));
                }
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

// ---- cache rows of whole sequences ------------------------------------------------------------------------------------
constexpr int kGatherThreads = 256;

// CTA = up to 16 positions of a sequence; 16 bytes per thread and turn.  rows int32 [n][4] = (first destination row, rows, batch row, first
// position); destination: latents [n_ctx][rank], rotated parts [n_ctx][64].
__global__ void __launch_bounds__(kGatherThreads)
latent_gather_kernel(const spk_latent_gather_args a) {
    const int4 e = reinterpret_cast<const int4*>(a.rows)[blockIdx.x];
    const SpkPageLayout lay = spk_latent_layout(a.block_size, a.rank_pad, 64, 1);
    if (e.z < 0 || e.z >= a.table_rows || e.w < 0 || static_cast<int64_t>(e.w) + e.y > a.max_blocks * a.block_size || e.x < 0 ||
        static_cast<int64_t>(e.x) + e.y > a.n_ctx) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        return;
    }
    const int32_t* table = a.tables + e.z * a.table_stride;
    const int groups = (a.rank_pad + 64) / 8, own = a.rank_pad / 8;
    for (int i = threadIdx.x; i < e.y * groups; i += kGatherThreads) {
        const int r = i / groups, g = i % groups, p = e.w + r;
        int64_t block = table[p / a.block_size];
        if (block < 0 || block >= a.num_blocks) {
            spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
            block = a.num_blocks - 1;
        }
        const uint4 v = *reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.pool) + spk_page_base(lay, block, 0) +
                                                         spk_latent_channel(lay, p % a.block_size, g * 8));
        __nv_bfloat16* dst = g < own ? static_cast<__nv_bfloat16*>(a.latents) + static_cast<int64_t>(e.x + r) * a.rank_pad + g * 8
                                     : static_cast<__nv_bfloat16*>(a.rotated) + static_cast<int64_t>(e.x + r) * 64 + (g - own) * 8;
        *reinterpret_cast<uint4*>(dst) = v;
    }
}

typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                                CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encoder() {
    static EncodeTiled fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult found;
        if (cudaGetDriverEntryPointByVersion("cuTensorMapEncodeTiled", &p, 12000, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess)
            p = nullptr;
        return reinterpret_cast<EncodeTiled>(p);
    }();
    return fn;
}

// [rows][columns] bf16, boxes of 128 rows x 64 columns, 128-byte swizzle; rows beyond the end read zero.
bool encode(CUtensorMap* map, const void* p, int64_t rows, int64_t columns) {
    const EncodeTiled fn = encoder();
    if (fn == nullptr) return false;
    const cuuint64_t size[2] = {static_cast<cuuint64_t>(columns), static_cast<cuuint64_t>(rows)}, stride[1] = {static_cast<cuuint64_t>(columns) * 2};
    const cuuint32_t box[2] = {64, kTile}, unit[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), size, stride, box, unit, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int CK, int CV>
int launch(const spk_latent_prefill_args& a, const CUtensorMap& kv, const CUtensorMap& kr, cudaStream_t s) {
    constexpr int bytes = Shape<CK, CV>::kBytes;
    static_assert(sizeof(Bars) <= 4608 && bytes <= 227 * 1024, "shared memory");
    const cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<CK, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    latent_prefill_kernel<CK, CV><<<dim3(a.heads, a.n_tiles), kThreads, bytes, s>>>(a, kv, kr);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

extern "C" int spk_latent_prefill_form(int dtype, int dim, int rot_pad, int vdim, int tiled) {
    return dtype == SPK_BF16 && tiled && dim >= 1 && dim <= 128 && rot_pad == 64 && vdim >= 1 && vdim <= 128;
}

extern "C" int spk_latent_gather(const spk_latent_gather_args* a, void* stream) {
    SpkRange nvtx_range("spk_latent_gather");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n_rows < 0 || a->n_ctx < 0 || a->rank_pad < 64 || a->rank_pad % 64 != 0 || a->block_size < 8 || a->num_blocks < 1 || a->max_blocks < 1 || a->table_rows < 1)
        return SPK_ERR_BAD_SHAPE;
    if (a->n_rows == 0) return SPK_OK;
    if (a->pool == nullptr || a->tables == nullptr || a->rows == nullptr || a->latents == nullptr || a->rotated == nullptr) return SPK_ERR_NULL_POINTER;
    for (const void* p : {a->pool, static_cast<const void*>(a->rows), static_cast<const void*>(a->latents), static_cast<const void*>(a->rotated)})
        if (reinterpret_cast<uintptr_t>(p) % 16 != 0) return SPK_ERR_BAD_STRIDE;
    latent_gather_kernel<<<a->n_rows, kGatherThreads, 0, spk_stream(stream)>>>(*a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

extern "C" int spk_latent_prefill(const spk_latent_prefill_args* args, void* stream) {
    SpkRange nvtx_range("spk_latent_prefill");
    if (args == nullptr) return SPK_ERR_NULL_POINTER;
    spk_latent_prefill_args a = *args;
    if (a.n < 0 || a.heads < 1 || a.heads > 65535 || a.n_tiles < 0 || a.n_ctx < 0 || a.n_ctx > 0x7fffffffLL || a.rot_dim < 2 || a.rot_dim > 64 || a.rot_dim % 2 != 0 ||
        a.dim_pad < a.dim || a.vdim_pad < a.vdim || a.rot_positions < 1 || !(a.scale > 0.0f))
        return SPK_ERR_BAD_SHAPE;
    if (!spk_latent_prefill_form(a.dtype, a.dim, 64, a.vdim, 1) || a.dim_pad % 64 != 0 || a.dim_pad > 128 || a.vdim_pad % 64 != 0 || a.vdim_pad > 128)
        return SPK_ERR_UNSUPPORTED;
    if (a.n == 0 || a.n_tiles == 0) return SPK_OK;
    if (a.n_tiles > 65535) return SPK_ERR_TOO_LARGE;
    if (a.q == nullptr || a.kv == nullptr || a.kr == nullptr || a.tiles == nullptr || a.sink == nullptr || a.gate == nullptr || a.out == nullptr || a.rot_table == nullptr)
        return SPK_ERR_NULL_POINTER;
    auto at16 = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    if (!at16(a.kv) || !at16(a.kr) || !at16(a.tiles)) return SPK_ERR_BAD_STRIDE;
    a.vec_q = at16(a.q) && a.dim % 8 == 0 && (a.dim + a.rot_dim) % 8 == 0;
    a.vec_out = at16(a.out) && at16(a.gate) && a.vdim % 8 == 0 && a.out_stride % 8 == 0 && a.gate_stride % 8 == 0;
    CUtensorMap kv, kr;
    if (!encode(&kv, a.kv, a.n_ctx, static_cast<int64_t>(a.heads) * (a.dim_pad + a.vdim_pad)) || !encode(&kr, a.kr, a.n_ctx, 64)) return SPK_ERR_UNSUPPORTED;
    cudaStream_t s = spk_stream(stream);
    const int ck = a.dim_pad / 64 + 1, cv = a.vdim_pad / 64;
    if (ck == 2 && cv == 1) return launch<2, 1>(a, kv, kr, s);
    if (ck == 2 && cv == 2) return launch<2, 2>(a, kv, kr, s);
    if (ck == 3 && cv == 1) return launch<3, 1>(a, kv, kr, s);
    return launch<3, 2>(a, kv, kr, s);
}
