// Decode attention with sigmoid key weights over the paged pools, bf16, head sizes up to 128: one query token per row.
//
// CTA = (key range, KV head (and block of 16 of its query heads), row), four warps; a warp walks every fourth 16-key step of
// the range on its own.  K and V rows of a step move with bulk copies (2 KB per 64-channel tile) into the warp's ring,
// the step's block-table entries sit in registers 32 steps ahead.  Scores and the weighted sum are warp MMAs with the query
// heads as the sixteen rows: all query heads of a group are served by one read of K and V, and the work is bound by that
// read.  Weights are 32-bit and enter the second product as a bf16 pair (hi + lo).  Key ranges add up without rescaling, so a
// CTA leaves plain 32-bit partial sums; the launch that follows adds them.
#include "spk_paged_attn.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kWarps = 4;
constexpr int kThreads = 32 * kWarps;
constexpr int kStep = 16;
constexpr int kStepTile = kStep * 128;  // bytes of a 64-channel tile of a step
constexpr float kLog2e = 1.4426950408889634f;

template <int CK, int CV>
struct Shape {
    static constexpr int NS = CK + CV <= 2 ? 4 : 3;
    static constexpr int kStage = (CK + CV) * kStepTile;
    static constexpr int kRing = kWarps * NS * kStage;
    static constexpr int kBytes = kRing + 128 + kWarps * NS * 8;
    static_assert(kWarps * 16 * CV * 64 * 4 <= kRing, "the final fold reuses the ring");
};

template <int CK, int CV>
__global__ void __launch_bounds__(kThreads)
sigmoid_decode_kernel(const spk_sigmoid_attn_args a) {
    using Sh = Shape<CK, CV>;
    constexpr int NS = Sh::NS;
    extern __shared__ uint8_t raw[];
    uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(raw) + 127) & ~uintptr_t(127));
    uint64_t* bars_all = reinterpret_cast<uint64_t*>(base + Sh::kRing);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
    const int rep = a.heads / a.kv_heads;
    const int blocks16 = (rep + 15) / 16;
    const int g = blockIdx.y / blocks16, h0 = g * rep + (blockIdx.y % blocks16) * 16;
    const int nh = min(16, (g + 1) * rep - h0);
    const int row = blockIdx.z;
    const int len = (a.active == nullptr || a.active[row] == 1) ? a.seq_lens[row] : 0;
    if (len < 0 || len > a.max_blocks * a.block_size) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SEQ_LEN);
        spk_grid_wait();
        return;
    }
    const int per = spk_split_keys(len, a.splits);
    const int lo = blockIdx.x * per, hi = min(lo + per, len);
    if (lo >= len) {
        spk_grid_wait();
        return;
    }
    const int steps_cta = (hi - lo + kStep - 1) / kStep;
    const int steps = steps_cta > warp ? (steps_cta - warp + kWarps - 1) / kWarps : 0;

    uint8_t* ring = base + warp * NS * Sh::kStage;
    uint64_t* bars = bars_all + warp * NS;
    if (lane == 0)
        for (int i = 0; i < NS; ++i) mbar_init(smem_u32(bars + i), 1);
    fence_async_shared();
    __syncwarp();

    const int32_t* table = a.tables + static_cast<int64_t>(row) * a.table_stride;
    const SpkPageLayout kl{a.kv_heads, a.block_size, a.k_pad, 1}, vl{a.kv_heads, a.block_size, a.v_pad, 1};
    auto key_of = [&](int s) { return lo + (s * kWarps + warp) * kStep; };
    // two windows of 32 block-table entries, one entry per lane: window w holds steps 32 w .. 32 w + 31
    auto entry = [&](int s) { return s < steps ? table[key_of(s) / a.block_size] : 0; };
    int32_t win0 = entry(lane), win1 = entry(32 + lane);
    int win = 0;
    auto issue = [&](int s) {  // s < steps; called in ascending order of s
        if ((s >> 5) > win) {
            win = s >> 5;
            win0 = win1;
            win1 = entry((win + 1) * 32 + lane);
        }
        const uint32_t bar = smem_u32(bars + s % NS);
        int64_t block = __shfl_sync(~0u, win0, s & 31);
        if (block < 0 || block >= a.num_blocks) {
            if (lane == 0) spk_flag(a.status, SPK_STATUS_BAD_BLOCK);
            block = 0;
        }
        const int off = (key_of(s) % a.block_size) << 6;
        if (lane == 0) mbar_expect(bar, Sh::kStage);
        __syncwarp();
        if (lane < CK + CV) {
            const bool is_k = lane < CK;
            const int c = is_k ? lane : lane - CK;
            const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(is_k ? a.k_pool : a.v_pool) +
                                       spk_page_base(is_k ? kl : vl, block, g) + c * (a.block_size << 6) + off;
            bulk_load(smem_u32(ring + (s % NS) * Sh::kStage + lane * kStepTile), src, kStepTile, bar);
        }
    };
    for (int s = 0; s < NS && s < steps; ++s) issue(s);

    // query rows: heads gid and gid + 8 of this block of heads
    uint32_t q[CK * 4][4];
    {
        const __nv_bfloat16* qr = static_cast<const __nv_bfloat16*>(a.q) + (static_cast<int64_t>(row) * a.heads + h0) * a.k_pad;
#pragma unroll
        for (int s = 0; s < CK * 4; ++s)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = gid + (i & 1) * 8, c = s * 16 + tig * 2 + (i >> 1) * 8;
                q[s][i] = r < nh ? *reinterpret_cast<const uint32_t*>(qr + static_cast<int64_t>(r) * a.k_pad + c) : 0u;
            }
    }
    const float c1 = -a.scale * kLog2e;
    const float b0 = gid < nh ? -a.head_bias[h0 + gid] * kLog2e : 0.0f, b1 = gid + 8 < nh ? -a.head_bias[h0 + gid + 8] * kLog2e : 0.0f;
    const bool upper = nh > 8;
    float acc[CV * 8][4];
#pragma unroll
    for (int i = 0; i < CV * 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;

    const int m = lane >> 3, mr = lane & 7;
    bool ok = true;
    for (int s = 0; s < steps; ++s) {
        uint8_t* stage = ring + (s % NS) * Sh::kStage;
        ok = __all_sync(~0u, mbar_wait(smem_u32(bars + s % NS), (s / NS) & 1));
        if (!ok) break;
        const int key0 = key_of(s);
        if (key0 + kStep > hi) {  // rows beyond the sequence may hold anything, and 0 * NaN is NaN
            const int valid = hi - key0;
            for (int i = lane; i < (kStep - valid) * CV * 8; i += 32) {
                const int c = i / ((kStep - valid) * 8), rest = i % ((kStep - valid) * 8);
                *reinterpret_cast<uint4*>(stage + (CK + c) * kStepTile + (valid + (rest >> 3)) * 128 + ((rest & 7) << 4)) = make_uint4(0u, 0u, 0u, 0u);
            }
            __syncwarp();
        }
        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
        const uint32_t ka = smem_u32(stage), va = ka + CK * kStepTile;
        {
            const int r = (m >> 1) * 8 + mr;
#pragma unroll
            for (int k = 0; k < CK * 4; ++k) {
                const int grp = k * 2 + (m & 1);
                uint32_t b[4];
                ldsm4(b, ka + (grp >> 3) * kStepTile + r * 128 + (((grp & 7) ^ (r & 7)) << 4));
                mma16816(s0, q[k], b[0], b[1]);
                mma16816(s1, q[k], b[2], b[3]);
            }
        }
        uint32_t ph[4] = {0u, 0u, 0u, 0u}, pl[4] = {0u, 0u, 0u, 0u};
        {
            const int j0 = key0 + tig * 2;
            auto weigh = [&](float x, float y, float bias, int j, uint32_t& h, uint32_t& l) {
                float p0, p1;
                sigmoid2(f2_fma(f2_pack(x, y), f2_pack(c1, c1), f2_pack(bias, bias)), p0, p1);
                split_bf16(j < hi ? p0 : 0.0f, j + 1 < hi ? p1 : 0.0f, h, l);
            };
            weigh(s0[0], s0[1], b0, j0, ph[0], pl[0]);
            weigh(s1[0], s1[1], b0, j0 + 8, ph[2], pl[2]);
            if (upper) {
                weigh(s0[2], s0[3], b1, j0, ph[1], pl[1]);
                weigh(s1[2], s1[3], b1, j0 + 8, ph[3], pl[3]);
            }
        }
        {
            const int r = (m & 1) * 8 + mr;
#pragma unroll
            for (int v = 0; v < CV * 4; ++v) {
                const int grp = v * 2 + (m >> 1);
                uint32_t b[4];
                ldsm4t(b, va + (grp >> 3) * kStepTile + r * 128 + (((grp & 7) ^ (r & 7)) << 4));
                mma16816(acc[2 * v], ph, b[0], b[1]);
                mma16816(acc[2 * v], pl, b[0], b[1]);
                mma16816(acc[2 * v + 1], ph, b[2], b[3]);
                mma16816(acc[2 * v + 1], pl, b[2], b[3]);
            }
        }
        __syncwarp();
        if (s + NS < steps) issue(s + NS);
    }
    if (!ok && lane == 0) spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
    __syncthreads();
    // fold the warps' sums through shared memory and leave the range's partial sum
    float* red = reinterpret_cast<float*>(base);
    constexpr int RW = CV * 64;
#pragma unroll
    for (int v = 0; v < CV * 8; ++v) {
        *reinterpret_cast<float2*>(red + (warp * 16 + gid) * RW + v * 8 + tig * 2) = make_float2(acc[v][0], acc[v][1]);
        *reinterpret_cast<float2*>(red + (warp * 16 + gid + 8) * RW + v * 8 + tig * 2) = make_float2(acc[v][2], acc[v][3]);
    }
    __syncthreads();
    float* part = a.partials + ((static_cast<int64_t>(row) * a.splits + blockIdx.x) * a.heads + h0) * a.vdim;
    for (int i = threadIdx.x; i < nh * a.vdim; i += kThreads) {
        const int r = i / a.vdim, e = i % a.vdim;
        float sum = 0.0f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) sum += red[(w * 16 + r) * RW + e];
        part[i] = sum;
    }
    // launched to overlap: the launch before this one is complete when this one is
    spk_grid_wait();
}

template <int CK, int CV>
int launch(const spk_sigmoid_attn_args& a, cudaStream_t s) {
    constexpr int bytes = Shape<CK, CV>::kBytes;
    const cudaError_t e = cudaFuncSetAttribute(sigmoid_decode_kernel<CK, CV>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return spk_set_cuda_error(e);
    const int rep = a.heads / a.kv_heads;
    const dim3 grid(a.splits, a.kv_heads * ((rep + 15) / 16), static_cast<unsigned>(a.n));
    return spk_launch(sigmoid_decode_kernel<CK, CV>, grid, kThreads, bytes, s, a.overlap != 0, a);
}

}  // namespace

int spk_sigmoid_decode_launch(const spk_sigmoid_attn_args& a, cudaStream_t s) {
    if (a.n > 65535 || a.kv_heads * ((a.heads / a.kv_heads + 15) / 16) > 65535) return SPK_ERR_TOO_LARGE;
    const int ck = a.k_pad / 64, cv = a.v_pad / 64;
    if (ck == 1 && cv == 1) return launch<1, 1>(a, s);
    if (ck == 1 && cv == 2) return launch<1, 2>(a, s);
    if (ck == 2 && cv == 1) return launch<2, 1>(a, s);
    return launch<2, 2>(a, s);
}
