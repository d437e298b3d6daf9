// Gated delta rule with one decay per head and key channel, and everything around it that enters the recurrence.
//
//   q, k, v <- silu(short causal convolution);  q, k <- unit vectors, q * dim^-1/2
//   S <- g * S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q;  out = o / rms(o) * w * sigmoid(gate)
//
//  * delta_step_kernel: one token per row (decode).  A CTA owns a (head, row): it convolves, normalises, decays, updates and reads the
//    state and writes the gated output; the state crosses the memory bus once each way.
//  * prefill, any sizes, 32-bit: delta_prepare_kernel (convolutions, unit vectors, decays, step sizes), delta_scan_kernel (the
//    recurrence, columns of the state in registers, tokens one after the other); bf16 heads of up to 128 channels take the chunked
//    form of spk_delta_mma.cu instead.  delta_out_kernel (norm and gate) ends both.
// The convolution's past lives in a ring of `taps` slots per row: a step writes its own slot and reads the others, so heads that
// share a key need no order among themselves.
#include "spk_delta.cuh"
#include "spk_tensor.cuh"

namespace {

using namespace spk_tc;

constexpr int kThreads = 256;

// ---- decode ------------------------------------------------------------------------------------------------------------
// CTA (head, row).  W columns per thread (4: 16-byte accesses); threads = (column group, slice of the key channels).  STAGED: the state
// comes into shared memory with one bulk copy while the convolutions run, is updated there and leaves with another; otherwise it is
// read twice from where it is.
template <typename T, int W, bool STAGED, int NT>
__global__ void __launch_bounds__(NT)
delta_step_kernel(const spk_delta_args a) {
    extern __shared__ __align__(128) float sm[];
    __shared__ float part[3 * 32];
    __shared__ uint64_t arrived;
    const int h = blockIdx.x;
    const int64_t row = blockIdx.y;
    const int dim = a.dim, vdim = a.vdim, rep = a.heads / a.kv_heads, g = h / rep;
    T* out = static_cast<T*>(a.out) + row * a.out_stride + static_cast<int64_t>(h) * vdim;
    if (a.active != nullptr && a.active[row] != 1) {
        for (int e = threadIdx.x; e < vdim; e += NT) out[e] = spk_from_float<T>(0.0f);
        return;
    }
    float* S = a.state + (row * a.heads + h) * static_cast<int64_t>(dim) * vdim;
    float* held = sm;                                                        // [dim][vdim] (STAGED)
    float* q = sm + (STAGED ? static_cast<int64_t>(dim) * vdim : 0);         // [dim]
    float* k = q + dim;                                                      // [dim]
    float* dec = k + dim;                                                    // [dim]
    float* v = dec + dim;                                                    // [vdim]; the outputs afterwards
    float* red = v + vdim;                                                   // [slices][vdim]
    const uint32_t state_bytes = static_cast<uint32_t>(dim) * vdim * 4;
    if (STAGED && threadIdx.x == 0) {
        mbar_init(smem_u32(&arrived), 1);
        fence_async_shared();
        mbar_expect(smem_u32(&arrived), state_bytes);
        bulk_load(smem_u32(held), S, state_bytes, smem_u32(&arrived));
    }
    const int cols = vdim / W;
    const int slices = cols < NT ? NT / cols : 1;
    const int slice = slices > 1 ? threadIdx.x / cols : 0;
    const int first = slices > 1 ? threadIdx.x % cols : threadIdx.x;
    const bool mine = slice < slices;
    const SpkDeltaShape sh = spk_delta_shape(a);
    const int64_t pos = a.positions[row];
    const bool fresh = pos == 0;  // whatever the slot holds, a sequence starts from zeros
    float* ring = a.conv_state + row * a.taps * sh.channels;
    const int now_slot = static_cast<int>(static_cast<uint64_t>(pos) % static_cast<uint32_t>(a.taps));
    const int past = pos < a.taps - 1 ? static_cast<int>(pos) : a.taps - 1;  // earlier tokens the convolution sees
    const bool leader = h % rep == 0;
    const T* gate = static_cast<const T*>(a.gate) + row * a.ld2 + static_cast<int64_t>(h) * vdim;
    float sums[3] = {0.0f, 0.0f, 0.0f};
    // one channel of q, k, the decays or v per thread and turn; two turns' loads are in flight together
    struct Item {
        float x, w0, back[3], w[3], bias;
        int kind, local, at;  // 0 q, 1 k, 2 v, 3 decay, -1 none
        const float* taps;
    };
    const int items = 3 * dim + vdim;
    auto fetch = [&](int i) {
        Item it;
        it.kind = i >= items ? -1 : i < dim ? 0 : i < 2 * dim ? 1 : i < 3 * dim ? 3 : 2;
        if (it.kind < 0) return it;
        if (it.kind == 3) {
            it.local = i - 2 * dim;
            const int c = h * dim + it.local;
            it.x = spk_to_float<T>(static_cast<const T*>(a.a)[row * a.ld2 + c]);
            it.bias = a.dt_bias[c];
            it.w0 = a.a_log[h];
            return it;
        }
        it.local = it.kind == 0 ? i : it.kind == 1 ? i - dim : i - 3 * dim;
        const int c = it.kind == 2 ? h * vdim + it.local : g * dim + it.local;  // channel of its projection
        it.at = c + it.kind * sh.qk;                                             // and its place in the ring
        const void* src = it.kind == 0 ? a.q : it.kind == 1 ? a.k : a.v;
        it.taps = (it.kind == 0 ? a.conv_q : it.kind == 1 ? a.conv_k : a.conv_v) + static_cast<int64_t>(c) * a.taps;
        it.x = spk_to_float<T>(static_cast<const T*>(src)[row * a.ld + c]);
        it.w0 = it.taps[a.taps - 1];
#pragma unroll
        for (int b = 1; b <= 3; ++b) {
            const bool in = b <= past;
            const int slot = now_slot >= b ? now_slot - b : now_slot - b + a.taps;
            it.back[b - 1] = in ? ring[slot * sh.channels + it.at] : 0.0f;
            it.w[b - 1] = in ? it.taps[a.taps - 1 - b] : 0.0f;
        }
        return it;
    };
    auto finish = [&](const Item& it) {
        if (it.kind < 0) return;
        if (it.kind == 3) {
            dec[it.local] = expf(spk_log_decay(it.x + it.bias, expf(it.w0)));
            return;
        }
        float y = it.x * it.w0;
#pragma unroll
        for (int b = 0; b < 3; ++b) y = fmaf(it.back[b], it.w[b], y);
        for (int b = 4; b <= past; ++b) {
            const int slot = now_slot >= b ? now_slot - b : now_slot - b + a.taps;
            y = fmaf(ring[slot * sh.channels + it.at], it.taps[a.taps - 1 - b], y);
        }
        y = spk_silu(y);
        if (leader || it.kind == 2) ring[now_slot * sh.channels + it.at] = it.x;
        if (it.kind == 0) {
            q[it.local] = y;
            sums[0] = fmaf(y, y, sums[0]);
        } else if (it.kind == 1) {
            k[it.local] = y;
            sums[1] = fmaf(y, y, sums[1]);
        } else {
            v[it.local] = y;
        }
    };
    const float raw_beta = spk_to_float<T>(static_cast<const T*>(a.b)[row * a.ld + h]);
    for (int i = threadIdx.x; i < items; i += 2 * NT) {
        const Item x = fetch(i), y = fetch(i + NT);
        finish(x);
        finish(y);
    }
    const float gate_mine = static_cast<int>(threadIdx.x) < vdim ? spk_to_float<T>(gate[threadIdx.x]) : 0.0f;
    const float norm_mine = static_cast<int>(threadIdx.x) < vdim ? a.w_norm[threadIdx.x] : 0.0f;
    spk_block_sum<3>(sums, part);  // its barriers also publish q, k, v and the decays
    const float qi = 1.0f / (sqrtf(sums[0] + 1e-6f) * sqrtf(static_cast<float>(dim))), ki = 1.0f / sqrtf(sums[1] + 1e-6f);
    const float beta = spk_sigmoid(raw_beta);
    if (STAGED && !mbar_wait(smem_u32(&arrived), 0) && !mbar_wait(smem_u32(&arrived), 0) && threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_DEVICE_WAIT_EXPIRED);
    const float* from = STAGED ? held : S;
    float* to = STAGED ? held : S;
    auto load = [&](float (&x)[W], int d, int c) {
        const float* p = from + static_cast<int64_t>(d) * vdim + c * W;
        if (W == 4) {
            const float4 f = *reinterpret_cast<const float4*>(p);
            x[0] = f.x; x[1 % W] = f.y; x[2 % W] = f.z; x[3 % W] = f.w;
        } else {
            x[0] = *p;
        }
#pragma unroll
        for (int i = 0; i < W; ++i) x[i] = fresh ? 0.0f : x[i] * dec[d];
    };
    float square[1] = {0.0f};
    for (int c0 = 0; c0 < cols; c0 += NT) {
        const int c = c0 + first;
        const bool in = mine && c < cols;
        float acc[W] = {};
        if (in) {
#pragma unroll 4
            for (int d = slice; d < dim; d += slices) {
                float x[W];
                load(x, d, c);
                const float kd = k[d] * ki;
#pragma unroll
                for (int i = 0; i < W; ++i) acc[i] = fmaf(kd, x[i], acc[i]);
            }
#pragma unroll
            for (int i = 0; i < W; ++i) red[slice * vdim + c * W + i] = acc[i];
        }
        __syncthreads();
        float u[W] = {};
        if (in) {
#pragma unroll
            for (int i = 0; i < W; ++i) {
                float sk = 0.0f;
                for (int z = 0; z < slices; ++z) sk += red[z * vdim + c * W + i];
                u[i] = beta * (v[c * W + i] - sk);
                acc[i] = 0.0f;
            }
        }
        __syncthreads();  // the first product's parts have been read
        if (in) {
#pragma unroll 4
            for (int d = slice; d < dim; d += slices) {
                float x[W];
                load(x, d, c);
                const float kd = k[d] * ki, qd = q[d] * qi;
#pragma unroll
                for (int i = 0; i < W; ++i) {
                    x[i] = fmaf(kd, u[i], x[i]);
                    acc[i] = fmaf(qd, x[i], acc[i]);
                }
                float* dst = to + static_cast<int64_t>(d) * vdim + c * W;
                if (W == 4) *reinterpret_cast<float4*>(dst) = make_float4(x[0], x[1 % W], x[2 % W], x[3 % W]);
                else *dst = x[0];
            }
#pragma unroll
            for (int i = 0; i < W; ++i) red[slice * vdim + c * W + i] = acc[i];
        }
        if (STAGED) fence_async_shared();
        __syncthreads();
        if (STAGED && c0 + NT >= cols && threadIdx.x == 0) {
            asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(__cvta_generic_to_global(S)), "r"(smem_u32(held)), "r"(state_bytes) : "memory");
            asm volatile("cp.async.bulk.commit_group;" ::: "memory");
        }
        if (in && slice == 0) {
#pragma unroll
            for (int i = 0; i < W; ++i) {
                float o = 0.0f;
                for (int z = 0; z < slices; ++z) o += red[z * vdim + c * W + i];
                v[c * W + i] = o;
                square[0] = fmaf(o, o, square[0]);
            }
        }
    }
    spk_block_sum<1>(square, part);
    const float inv = 1.0f / sqrtf(square[0] / static_cast<float>(vdim) + a.eps);
    for (int e = threadIdx.x; e < vdim; e += NT) {
        const bool own = e == static_cast<int>(threadIdx.x);
        out[e] = spk_from_float<T>(v[e] * inv * (own ? norm_mine : a.w_norm[e]) * spk_sigmoid(own ? gate_mine : spk_to_float<T>(gate[e])));
    }
    if (STAGED && threadIdx.x == 0) asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");  // the copy has read shared memory
}

// ---- prefill -----------------------------------------------------------------------------------------------------------

// What the recurrence reads, 32-bit: q [n][kv_heads][dim], k the same, v [n][heads][vdim], decays [n][heads][dim], beta [n][heads],
// outputs [n][heads][vdim].
struct Work {
    float *q, *k, *v, *g, *beta, *o;
};
__host__ __device__ inline int64_t work_floats(int64_t n, int heads, int kv_heads, int dim, int vdim) {
    return n * (2 * static_cast<int64_t>(kv_heads) * dim + static_cast<int64_t>(heads) * (dim + 2 * vdim) + ((heads + 3) & ~3));
}
__host__ __device__ inline Work carve(const spk_delta_args& a) {
    Work w;
    const int64_t qk = a.n * a.kv_heads * a.dim, vv = a.n * a.heads * a.vdim;
    w.q = static_cast<float*>(a.workspace);
    w.k = w.q + qk;
    w.g = w.k + qk;
    w.v = w.g + a.n * a.heads * a.dim;
    w.o = w.v + vv;
    w.beta = w.o + vv;
    return w;
}

// CTA = chunk of up to 16 tokens; a warp per (token, part): the key heads' q, their k, the heads' v, the heads' decays.
template <typename T>
__global__ void __launch_bounds__(kThreads)
delta_prepare_kernel(const spk_delta_args a) {
    const int4 ch = reinterpret_cast<const int4*>(a.chunks)[blockIdx.x];    // first token, tokens, portion, index
    const int4 po = reinterpret_cast<const int4*>(a.portions)[ch.z];        // first token, tokens, row, tokens before
    if (po.z < 0 || po.z >= a.state_rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    const Work w = carve(a);
    const SpkDeltaShape sh = spk_delta_shape(a);
    const int lane = threadIdx.x & 31, parts = 2 * a.kv_heads + 2 * a.heads;
    const float* ring = a.conv_state + static_cast<int64_t>(po.z) * a.taps * sh.channels;
    for (int item = threadIdx.x >> 5; item < ch.y * parts; item += kThreads / 32) {
        const int64_t t = ch.x + item / parts;
        int part = item % parts;
        auto conv = [&](const void* src, int64_t c, int at, const float* taps) {
            const T* p = static_cast<const T*>(src) + t * a.ld + c;
            return spk_conv_silu(taps + c * a.taps, a.taps, spk_to_float<T>(*p), [&](int back) {
                if (t - back >= po.x) return spk_to_float<T>(p[-back * a.ld]);
                const int64_t pos = po.w + (t - po.x) - back;
                return pos >= 0 ? ring[(pos % a.taps) * sh.channels + at] : 0.0f;
            });
        };
        if (part < 2 * a.kv_heads) {
            const bool is_q = part < a.kv_heads;
            const int g = is_q ? part : part - a.kv_heads;
            float* dst = (is_q ? w.q : w.k) + (t * a.kv_heads + g) * a.dim;
            float ss = 0.0f;
            for (int c = lane; c < a.dim; c += 32) {
                const float x = conv(is_q ? a.q : a.k, g * a.dim + c, (is_q ? 0 : sh.qk) + g * a.dim + c, is_q ? a.conv_q : a.conv_k);
                dst[c] = x;
                ss = fmaf(x, x, ss);
            }
            float inv = 1.0f / sqrtf(spk_warp_sum(ss) + 1e-6f);
            if (is_q) inv /= sqrtf(static_cast<float>(a.dim));
            for (int c = lane; c < a.dim; c += 32) dst[c] *= inv;
        } else if (part < 2 * a.kv_heads + a.heads) {
            const int h = part - 2 * a.kv_heads;
            for (int c = lane; c < a.vdim; c += 32)
                w.v[(t * a.heads + h) * a.vdim + c] = conv(a.v, static_cast<int64_t>(h) * a.vdim + c, 2 * sh.qk + h * a.vdim + c, a.conv_v);
        } else {
            const int h = part - 2 * a.kv_heads - a.heads;
            const float rate = expf(a.a_log[h]);
            for (int c = lane; c < a.dim; c += 32) {
                const int64_t i = static_cast<int64_t>(h) * a.dim + c;
                w.g[t * a.heads * a.dim + i] = expf(spk_log_decay(spk_to_float<T>(static_cast<const T*>(a.a)[t * a.ld2 + i]) + a.dt_bias[i], rate));
            }
            if (lane == 0) w.beta[t * a.heads + h] = spk_sigmoid(spk_to_float<T>(static_cast<const T*>(a.b)[t * a.ld + h]));
        }
    }
}

// The recurrence, token by token.  CTA = (32 columns of a head's state, head, portion); four lanes share a column, each with every fourth
// group of four key channels in registers: NR groups, dim <= 16 NR.  Both products are taken of the state before the step:
//   S^T(g k) and S^T(g q) + (q . k) u, so one exchange per token serves them, and the update is off the chain.
constexpr int kScanCols = 32;

template <typename T, int NR>
__global__ void __launch_bounds__(4 * kScanCols)
delta_scan_kernel(const spk_delta_args a) {
    constexpr int D = 16 * NR, kScanTokens = NR > 16 ? 2 : NR > 8 ? 4 : 8;  // tokens staged at a time
    __shared__ __align__(16) float gs[2][kScanTokens][D], ks[2][kScanTokens][D], gk[2][kScanTokens][D], gq[2][kScanTokens][D];
    __shared__ float qk[2][kScanTokens], bs[2][kScanTokens], vs[2][kScanTokens][kScanCols];
    const int4 po = reinterpret_cast<const int4*>(a.portions)[blockIdx.z];
    if (po.z < 0 || po.z >= a.state_rows) {
        if (threadIdx.x == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    const Work w = carve(a);
    const SpkDeltaShape sh = spk_delta_shape(a);
    const int h = blockIdx.y, rep = a.heads / a.kv_heads, g = h / rep;
    const int col = threadIdx.x >> 2, part = threadIdx.x & 3, e = blockIdx.x * kScanCols + col;
    const bool in = e < a.vdim;
    float* S = a.state + (static_cast<int64_t>(po.z) * a.heads + h) * a.dim * a.vdim + e;
    uint64_t s[NR][2];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        float f[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = 16 * i + 4 * part + j;
            f[j] = po.w > 0 && in && d < a.dim ? S[static_cast<int64_t>(d) * a.vdim] : 0.0f;
        }
        s[i][0] = f2_pack(f[0], f[1]);
        s[i][1] = f2_pack(f[2], f[3]);
    }
    auto stage = [&](int buf, int j0) {  // tokens j0 .. of the portion, a warp per token
        const int lane = threadIdx.x & 31;
        for (int j = threadIdx.x >> 5; j < kScanTokens && j0 + j < po.y; j += 4 * kScanCols / 32) {
            const int64_t t = po.x + j0 + j;
            const float *qr = w.q + (t * a.kv_heads + g) * a.dim, *kr = w.k + (t * a.kv_heads + g) * a.dim, *gr = w.g + (t * a.heads + h) * a.dim;
            float dot = 0.0f;
            for (int d = lane; d < D; d += 32) {
                const bool live = d < a.dim;
                const float x = live ? qr[d] : 0.0f, y = live ? kr[d] : 0.0f, z = live ? gr[d] : 0.0f;
                gs[buf][j][d] = z;
                ks[buf][j][d] = y;
                gk[buf][j][d] = z * y;
                gq[buf][j][d] = z * x;
                dot = fmaf(x, y, dot);
            }
            dot = spk_warp_sum(dot);
            if (lane == 0) {
                qk[buf][j] = dot;
                bs[buf][j] = w.beta[t * a.heads + h];
            }
            const int c = blockIdx.x * kScanCols + lane;
            vs[buf][j][lane] = c < a.vdim ? w.v[(t * a.heads + h) * a.vdim + c] : 0.0f;
        }
    };
    stage(0, 0);
    __syncthreads();
    for (int j0 = 0, buf = 0; j0 < po.y; j0 += kScanTokens, buf ^= 1) {
        if (j0 + kScanTokens < po.y) stage(buf ^ 1, j0 + kScanTokens);
        const int n = min(kScanTokens, po.y - j0);
        for (int j = 0; j < n; ++j) {
            uint64_t ak[2] = {0, 0}, aq[2] = {0, 0};
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(&gk[buf][j][16 * i + 4 * part]);
                const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(&gq[buf][j][16 * i + 4 * part]);
                ak[0] = f2_fma(s[i][0], x.x, ak[0]);
                ak[1] = f2_fma(s[i][1], x.y, ak[1]);
                aq[0] = f2_fma(s[i][0], y.x, aq[0]);
                aq[1] = f2_fma(s[i][1], y.y, aq[1]);
            }
            float k0, k1, q0, q1;
            f2_unpack(f2_add(ak[0], ak[1]), k0, k1);
            f2_unpack(f2_add(aq[0], aq[1]), q0, q1);
            float sk = k0 + k1, sq = q0 + q1;
            sk += __shfl_xor_sync(~0u, sk, 1);
            sq += __shfl_xor_sync(~0u, sq, 1);
            sk += __shfl_xor_sync(~0u, sk, 2);
            sq += __shfl_xor_sync(~0u, sq, 2);
            const float u = bs[buf][j] * (vs[buf][j][col] - sk);
            const uint64_t uu = f2_pack(u, u);
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const ulonglong2 z = *reinterpret_cast<const ulonglong2*>(&gs[buf][j][16 * i + 4 * part]);
                const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(&ks[buf][j][16 * i + 4 * part]);
                s[i][0] = f2_fma(s[i][0], z.x, f2_mul(y.x, uu));
                s[i][1] = f2_fma(s[i][1], z.y, f2_mul(y.y, uu));
            }
            if (part == 0 && in) w.o[((static_cast<int64_t>(po.x) + j0 + j) * a.heads + h) * a.vdim + e] = fmaf(qk[buf][j], u, sq);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        float f[4];
        f2_unpack(s[i][0], f[0], f[1]);
        f2_unpack(s[i][1], f[2], f[3]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = 16 * i + 4 * part + j;
            if (in && d < a.dim) S[static_cast<int64_t>(d) * a.vdim] = f[j];
        }
    }
    // the convolution's last inputs, for the next portion or the first decode step
    if (part == 0 && in) spk_commit_conv<T>(a, po, sh, a.v, static_cast<int64_t>(h) * a.vdim + e, 2 * sh.qk + h * a.vdim + e);
    if (blockIdx.x == 0 && h % rep == 0)
        for (int c = threadIdx.x; c < a.dim; c += 4 * kScanCols) {
            spk_commit_conv<T>(a, po, sh, a.q, g * a.dim + c, g * a.dim + c);
            spk_commit_conv<T>(a, po, sh, a.k, g * a.dim + c, sh.qk + g * a.dim + c);
        }
}

// A warp per (token, head): norm over the head's outputs, weight, gate.
template <typename T>
__global__ void __launch_bounds__(kThreads)
delta_out_kernel(const spk_delta_args a, const float* __restrict__ outputs) {
    const int64_t item = static_cast<int64_t>(blockIdx.x) * (kThreads / 32) + (threadIdx.x >> 5);
    if (item >= a.n * a.heads) return;
    const int lane = threadIdx.x & 31;
    const int64_t t = item / a.heads;
    const int h = static_cast<int>(item % a.heads);
    const float* o = outputs + item * a.vdim;
    float ss = 0.0f;
    for (int e = lane; e < a.vdim; e += 32) ss = fmaf(o[e], o[e], ss);
    const float inv = 1.0f / sqrtf(spk_warp_sum(ss) / static_cast<float>(a.vdim) + a.eps);
    const T* gate = static_cast<const T*>(a.gate) + t * a.ld2 + static_cast<int64_t>(h) * a.vdim;
    T* out = static_cast<T*>(a.out) + t * a.out_stride + static_cast<int64_t>(h) * a.vdim;
    for (int e = lane; e < a.vdim; e += 32) out[e] = spk_from_float<T>(o[e] * inv * a.w_norm[e] * spk_sigmoid(spk_to_float<T>(gate[e])));
}

// The same with four channels per lane: V / 4 lanes per head, everything aligned to four elements.
template <typename T, int V>
__global__ void __launch_bounds__(kThreads)
delta_out_vec_kernel(const spk_delta_args a, const float* __restrict__ outputs) {
    constexpr int L = V / 4;
    const int64_t item = static_cast<int64_t>(blockIdx.x) * (kThreads / L) + threadIdx.x / L;
    const bool in = item < a.n * a.heads;
    const int c = 4 * (threadIdx.x % L);
    const int64_t t = item / a.heads;
    const int64_t at = (item % a.heads) * V + c;
    spk_grid_wait();  // launched to overlap the end of the recurrence
    const float4 o = in ? __ldcs(reinterpret_cast<const float4*>(outputs + item * V + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 g = spk_load4<T, true>(static_cast<const T*>(a.gate) + (in ? t * a.ld2 + at : 0), 4);
    const float4 w = *reinterpret_cast<const float4*>(a.w_norm + c);
    float ss = (o.x * o.x + o.y * o.y) + (o.z * o.z + o.w * o.w);
#pragma unroll
    for (int s = L / 2; s >= 1; s >>= 1) ss += __shfl_xor_sync(~0u, ss, s);
    if (!in) return;
    const float inv = 1.0f / sqrtf(ss / static_cast<float>(V) + a.eps);
    auto gated = [&](float x, float m, float y) { return x * inv * m * (sizeof(T) == 2 ? sigmoid_fast(y) : spk_sigmoid(y)); };
    spk_store4<T, true>(static_cast<T*>(a.out) + t * a.out_stride + at, make_float4(gated(o.x, w.x, g.x), gated(o.y, w.y, g.y), gated(o.z, w.z, g.z), gated(o.w, w.w, g.w)), 4);
}

int check(const spk_delta_args* a) {
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->heads > 65535 || a->kv_heads < 1 || a->heads % a->kv_heads != 0 || a->dim < 1 || a->vdim < 1 || a->taps < 1 ||
        a->state_rows < 1)
        return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->k == nullptr || a->v == nullptr || a->b == nullptr || a->a == nullptr || a->gate == nullptr || a->conv_q == nullptr ||
        a->conv_k == nullptr || a->conv_v == nullptr || a->a_log == nullptr || a->dt_bias == nullptr || a->w_norm == nullptr || a->state == nullptr ||
        a->conv_state == nullptr || a->out == nullptr)
        return SPK_ERR_NULL_POINTER;
    return SPK_OK;
}

template <typename T, int W, bool STAGED, int NT>
int launch_step_form(const spk_delta_args& a, cudaStream_t s) {
    const int cols = a.vdim / W, slices = cols < NT ? NT / cols : 1;
    const size_t bytes = sizeof(float) * (3 * static_cast<size_t>(a.dim) + a.vdim + static_cast<size_t>(slices) * a.vdim + (STAGED ? static_cast<size_t>(a.dim) * a.vdim : 0));
    if (bytes > 200 * 1024) return SPK_ERR_TOO_LARGE;
    if (bytes > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(delta_step_kernel<T, W, STAGED, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
        if (e != cudaSuccess) return spk_set_cuda_error(e);
    }
    delta_step_kernel<T, W, STAGED, NT><<<dim3(a.heads, static_cast<unsigned>(a.n)), NT, bytes, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T>
int launch_step(const spk_delta_args& a, cudaStream_t s) {
    const bool vec = a.vdim % 4 == 0 && reinterpret_cast<uintptr_t>(a.state) % 16 == 0;
    const int64_t state = static_cast<int64_t>(a.dim) * a.vdim * 4;
    if (!vec) return launch_step_form<T, 1, false, 256>(a, s);
    if (state <= 20 * 1024) return launch_step_form<T, 4, true, 128>(a, s);
    return state <= 100 * 1024 ? launch_step_form<T, 4, true, 256>(a, s) : launch_step_form<T, 4, false, 256>(a, s);
}

template <typename T>
int launch_out(const spk_delta_args& a, const float* outputs, cudaStream_t s) {
    auto at = [](const void* p, size_t b) { return reinterpret_cast<uintptr_t>(p) % b == 0; };
    if ((a.vdim == 64 || a.vdim == 128) && a.ld2 % 4 == 0 && a.out_stride % 4 == 0 && at(a.gate, 4 * sizeof(T)) && at(a.out, 4 * sizeof(T)) &&
        at(outputs, 16) && at(a.w_norm, 16)) {
        const int per = kThreads / (a.vdim / 4);
        const int64_t grid = (a.n * a.heads + per - 1) / per;
        if (grid > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
        return spk_launch(a.vdim == 64 ? delta_out_vec_kernel<T, 64> : delta_out_vec_kernel<T, 128>, dim3(static_cast<unsigned>(grid)), kThreads, 0, s, true, a,
                          outputs);
    }
    const int64_t grid = (a.n * a.heads + kThreads / 32 - 1) / (kThreads / 32);
    if (grid > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    delta_out_kernel<T><<<static_cast<unsigned>(grid), kThreads, 0, s>>>(a, outputs);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T>
int launch_prefill(const spk_delta_args& a, cudaStream_t s) {
    if (a.dim > 512) return SPK_ERR_UNSUPPORTED;
    delta_prepare_kernel<T><<<a.n_chunks, kThreads, 0, s>>>(a);
    SPK_CHECK_LAUNCH();
    const dim3 grid((a.vdim + kScanCols - 1) / kScanCols, a.heads, a.n_portions);
    const int threads = 4 * kScanCols;
    if (a.dim <= 32) delta_scan_kernel<T, 2><<<grid, threads, 0, s>>>(a);
    else if (a.dim <= 64) delta_scan_kernel<T, 4><<<grid, threads, 0, s>>>(a);
    else if (a.dim <= 128) delta_scan_kernel<T, 8><<<grid, threads, 0, s>>>(a);
    else if (a.dim <= 256) delta_scan_kernel<T, 16><<<grid, threads, 0, s>>>(a);
    else delta_scan_kernel<T, 32><<<grid, threads, 0, s>>>(a);
    SPK_CHECK_LAUNCH();
    return launch_out<T>(a, carve(a).o, s);
}

}  // namespace

extern "C" int spk_delta_step(const spk_delta_args* a, void* stream) {
    SpkRange nvtx_range("spk_delta_step");
    const int rc = check(a);
    if (rc != SPK_OK || a->n == 0) return rc;
    if (a->positions == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n > 65535) return SPK_ERR_TOO_LARGE;
    if (a->n > a->state_rows) return SPK_ERR_BAD_SHAPE;
    cudaStream_t s = spk_stream(stream);
    return a->dtype == SPK_F32 ? launch_step<float>(*a, s) : launch_step<__nv_bfloat16>(*a, s);
}

extern "C" int spk_delta_chunk_tokens(int dtype, int dim, int vdim) {
    (void)dtype;
    (void)dim;
    (void)vdim;
    return kDeltaChunk;
}

extern "C" int64_t spk_delta_workspace_bytes(int dtype, int64_t n, int n_chunks, int heads, int kv_heads, int dim, int vdim) {
    if (n < 1 || n_chunks < 1 || heads < 1 || kv_heads < 1 || dim < 1 || vdim < 1) return 0;
    if (spk_delta_tensor_form(dtype, dim, vdim)) return spk_delta_mma_bytes(n_chunks, heads, dim, vdim) + static_cast<int64_t>(sizeof(float)) * n * heads * vdim;
    return static_cast<int64_t>(sizeof(float)) * work_floats(n, heads, kv_heads, dim, vdim);
}

extern "C" int spk_delta_prefill(const spk_delta_args* a, void* stream) {
    SpkRange nvtx_range("spk_delta_prefill");
    const int rc = check(a);
    if (rc != SPK_OK || a->n == 0) return rc;
    if (a->n_chunks < 1 || a->n_portions < 1 || a->n_portions > 65535) return SPK_ERR_BAD_SHAPE;
    if (a->chunks == nullptr || a->portions == nullptr || a->seqs == nullptr) return SPK_ERR_NULL_POINTER;
    if (reinterpret_cast<uintptr_t>(a->chunks) % 16 != 0 || reinterpret_cast<uintptr_t>(a->portions) % 16 != 0 ||
        reinterpret_cast<uintptr_t>(a->seqs) % 16 != 0 || reinterpret_cast<uintptr_t>(a->workspace) % 16 != 0)
        return SPK_ERR_BAD_STRIDE;
    if (a->workspace == nullptr || a->workspace_bytes < spk_delta_workspace_bytes(a->dtype, a->n, a->n_chunks, a->heads, a->kv_heads, a->dim, a->vdim))
        return SPK_ERR_WORKSPACE_TOO_SMALL;
    cudaStream_t s = spk_stream(stream);
    if (spk_delta_tensor_form(a->dtype, a->dim, a->vdim)) {
        float* outputs = reinterpret_cast<float*>(static_cast<uint8_t*>(a->workspace) + spk_delta_mma_bytes(a->n_chunks, a->heads, a->dim, a->vdim));
        if (const int e = spk_delta_mma_launch(*a, outputs, s)) return e;
        return launch_out<__nv_bfloat16>(*a, outputs, s);
    }
    return a->dtype == SPK_F32 ? launch_prefill<float>(*a, s) : launch_prefill<__nv_bfloat16>(*a, s);
}
