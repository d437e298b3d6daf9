// Linear attention with a per-head decay ("lightning" attention) and its output stage.
//
//   S_t = decay_h S_{t-1} + k_t v_t^T        o_t = S_t^T q_t        (S in 32 bits, one state per sequence and head)
//
//  * decay_step_kernel: one token per row (decode), state read and written once.
//  * prefill cuts a portion into chunks: every chunk's own sum of k v^T (decay_chunk_sum_kernel), a scan over the chunks that
//    leaves each chunk the state it starts from (decay_scan_kernel), and the outputs, a decayed masked product inside the
//    chunk plus the incoming state (decay_chunk_out_kernel).  All chunks of all sequences of the call run at once; only the
//    scan walks them in order.  The two outer kernels here are the 32-bit form (any sizes, chunks of 64 tokens); bf16
//    projections with heads of up to 128 channels take the tensor-core form of spk_decay_mma.cu.
//  * gated_norm_kernel: the heads' outputs under one RMS norm, times sigmoid(gate), scaled into one half of the operand
//    of the output projection; in decode steps it also adds up the attention's partial sums into the other half.
//
// Decay powers come from a host table [head][0 .. 512] (evaluated in double precision), never from repeated products.
#include "spk_decay.cuh"

namespace {

constexpr int kChunk = kDecayChunk;
constexpr int kPow = kDecayMaxSpan + 1;  // tabulated powers per head
constexpr int kThreads = 256;

__device__ __forceinline__ float act(float x, int silu) { return silu ? spk_silu(x) : x; }

// ---- decode ----------------------------------------------------------------------------------------------
// CTA (head, row).  W columns per thread (4: 16-byte accesses); threads = (column group, slice of d).
template <typename T, int W>
__global__ void __launch_bounds__(kThreads)
decay_step_kernel(const spk_decay_attn_args a) {
    extern __shared__ float sm[];
    const int h = blockIdx.x;
    const int64_t row = blockIdx.y;
    const int dim = a.dim, vdim = a.vdim;
    float* out = a.out + (row * a.heads + h) * vdim;
    if (a.active != nullptr && a.active[row] != 1) {
        spk_grid_wait();
        spk_grid_release();
        for (int e = threadIdx.x; e < vdim; e += kThreads) out[e] = 0.0f;
        return;
    }
    float* q = sm;
    float* k = q + dim;
    float* v = k + dim;
    float* red = v + vdim;
    float* S = a.state + row * a.state_stride + static_cast<int64_t>(h) * dim * vdim;
    const int cols = vdim / W;
    const int slices = cols < kThreads ? kThreads / cols : 1;
    const int slice = threadIdx.x / cols;
    constexpr int U = 8;  // state rows in flight per thread
    float s[U][W];
    auto load = [&](int d0, int c) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int d = d0 + u * slices;
            if (d < dim) {
                if (W == 4) {
                    const float4 f = __ldcs(reinterpret_cast<const float4*>(S + static_cast<int64_t>(d) * vdim + c * W));
                    s[u][0] = f.x; s[u][1 % W] = f.y; s[u][2 % W] = f.z; s[u][3 % W] = f.w;
                } else {
                    s[u][0] = S[static_cast<int64_t>(d) * vdim + c];
                }
            }
        }
    };
    // the first rows are on their way before the projections are looked at
    const bool mine = slice < slices;
    const int first = slices > 1 ? threadIdx.x % cols : threadIdx.x;
    if (mine && first < cols) load(slice, first);
    // what was launched before is complete from here on: the launch placed behind this one may rely on that
    spk_grid_wait();
    spk_grid_release();
    const T* qr = static_cast<const T*>(a.q) + row * a.ld + static_cast<int64_t>(h) * dim;
    const T* kr = static_cast<const T*>(a.k) + row * a.ld + static_cast<int64_t>(h) * dim;
    const T* vr = static_cast<const T*>(a.v) + row * a.ld + static_cast<int64_t>(h) * vdim;
    for (int i = threadIdx.x; i < 2 * dim + vdim; i += kThreads) {
        const T* src = i < dim ? qr + i : i < 2 * dim ? kr + (i - dim) : vr + (i - 2 * dim);
        sm[i] = act(spk_to_float<T>(*src), a.silu);
    }
    __syncthreads();
    const float decay = a.decay_pow[h * kPow + 1];
    for (int c0 = 0; c0 < cols; c0 += kThreads) {
        const int c = c0 + first;
        if (!mine || c >= cols) continue;
        float acc[W];
#pragma unroll
        for (int i = 0; i < W; ++i) acc[i] = 0.0f;
        float vv[W];
#pragma unroll
        for (int i = 0; i < W; ++i) vv[i] = v[c * W + i];
        for (int d0 = slice; d0 < dim; d0 += U * slices) {
            if (c0 > 0 || d0 > slice) load(d0, c);
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int d = d0 + u * slices;
                if (d < dim) {
                    const float kd = k[d], qd = q[d];
#pragma unroll
                    for (int i = 0; i < W; ++i) {
                        s[u][i] = fmaf(kd, vv[i], decay * s[u][i]);
                        acc[i] = fmaf(qd, s[u][i], acc[i]);
                    }
                    if (W == 4)
                        __stcs(reinterpret_cast<float4*>(S + static_cast<int64_t>(d) * vdim + c * W),
                               make_float4(s[u][0], s[u][1 % W], s[u][2 % W], s[u][3 % W]));
                    else
                        S[static_cast<int64_t>(d) * vdim + c] = s[u][0];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < W; ++i) red[slice * vdim + c * W + i] = acc[i];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < vdim; e += kThreads) {
        float o = 0.0f;
        for (int s = 0; s < slices; ++s) o += red[s * vdim + e];
        out[e] = o;
    }
}

// ---- prefill, any sizes, 32-bit arithmetic -----------------------------------------------------------------
__host__ __device__ __forceinline__ int pad4(int x) { return (x + 3) & ~3; }

// Rows of one head of a chunk into shared memory [kChunk][pad4(width)], activation applied, zero beyond the data.
template <typename T>
__device__ __forceinline__ void stage_rows(float* dst, const T* src, int64_t ld, int len, int width, int silu) {
    const int wp = pad4(width);
    for (int i = threadIdx.x; i < kChunk * wp; i += kThreads) {
        const int r = i / wp, c = i % wp;
        dst[i] = r < len && c < width ? act(spk_to_float<T>(src[r * ld + c]), silu) : 0.0f;
    }
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
decay_chunk_sum_kernel(const spk_decay_attn_args a) {
    extern __shared__ float sm[];
    const int c = blockIdx.x, h = blockIdx.y;
    const SpkChunk ci = spk_chunk(a, c);
    const int dp = pad4(a.dim), ep = pad4(a.vdim);
    float* k = sm;
    float* v = k + kChunk * dp;
    stage_rows<T>(k, static_cast<const T*>(a.k) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim, a.ld, ci.len, a.dim, a.silu);
    stage_rows<T>(v, static_cast<const T*>(a.v) + ci.start * a.ld + static_cast<int64_t>(h) * a.vdim, a.ld, ci.len, a.vdim, a.silu);
    __syncthreads();
    const float* pw = a.decay_pow + h * kPow;
    float* U = a.workspace + (static_cast<int64_t>(c) * a.heads + h) * a.dim * a.vdim;
    const int te = ep / 4, tiles = (dp / 4) * te;
    for (int t = threadIdx.x; t < tiles; t += kThreads) {
        const int d0 = (t / te) * 4, e0 = (t % te) * 4;
        float acc[4][4] = {};
        for (int j = 0; j < ci.len; ++j) {
            const float w = pw[ci.len - 1 - j];
            const float4 kk = *reinterpret_cast<const float4*>(k + j * dp + d0);
            const float4 vv = *reinterpret_cast<const float4*>(v + j * ep + e0);
            const float kw[4] = {kk.x * w, kk.y * w, kk.z * w, kk.w * w};
            const float vr[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(kw[x], vr[y], acc[x][y]);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y)
                if (d0 + x < a.dim && e0 + y < a.vdim) U[static_cast<int64_t>(d0 + x) * a.vdim + e0 + y] = acc[x][y];
    }
}

// Element (seq, head, d, e): replaces every chunk's own sum by the state the chunk starts from, leaves the sequence's
// final state in its slot.
__global__ void __launch_bounds__(kThreads)
decay_scan_kernel(const spk_decay_attn_args a) {
    const int64_t per_head = static_cast<int64_t>(a.dim) * a.vdim;
    const int64_t per_chunk = per_head * a.heads;
    const int64_t i = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x;
    if (i >= per_chunk) return;
    const int4 sq = reinterpret_cast<const int4*>(a.seqs)[blockIdx.y];  // first chunk, chunks, state row, context
    if (sq.z < 0 || sq.z >= a.state_rows) {
        if (i == 0) spk_flag(a.status, SPK_STATUS_BAD_SLOT);
        return;
    }
    const float* pw = a.decay_pow + (i / per_head) * kPow;
    float* slot = a.state + sq.z * a.state_stride + i;
    float S = sq.w > 0 ? *slot : 0.0f;
    float* w = a.workspace + sq.x * per_chunk + i;
    constexpr int U = 8;  // chunks in flight: only S is a chain, the loads are not
    for (int c0 = 0; c0 < sq.y; c0 += U) {
        float own[U], p[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const bool in = c0 + u < sq.y;
            own[u] = in ? w[(c0 + u) * per_chunk] : 0.0f;
            p[u] = in ? pw[a.chunks[4 * (sq.x + c0 + u) + 1]] : 1.0f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < sq.y) w[(c0 + u) * per_chunk] = S;
            S = fmaf(p[u], S, own[u]);
        }
    }
    *slot = S;
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
decay_chunk_out_kernel(const spk_decay_attn_args a) {
    extern __shared__ float sm[];
    const int c = blockIdx.x, h = blockIdx.y;
    const SpkChunk ci = spk_chunk(a, c);
    const int dp = pad4(a.dim), ep = pad4(a.vdim);
    constexpr int AP = kChunk + 1;
    float* q = sm;
    float* k = q + kChunk * dp;
    float* v = k + kChunk * dp;
    float* A = v + kChunk * ep;
    stage_rows<T>(q, static_cast<const T*>(a.q) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim, a.ld, ci.len, a.dim, a.silu);
    stage_rows<T>(k, static_cast<const T*>(a.k) + ci.start * a.ld + static_cast<int64_t>(h) * a.dim, a.ld, ci.len, a.dim, a.silu);
    stage_rows<T>(v, static_cast<const T*>(a.v) + ci.start * a.ld + static_cast<int64_t>(h) * a.vdim, a.ld, ci.len, a.vdim, a.silu);
    __syncthreads();
    const float* pw = a.decay_pow + h * kPow;
    {
        const int i0 = threadIdx.x / 16, j0 = threadIdx.x % 16;  // rows i0 + 16 x, columns j0 + 16 y
        float acc[4][4] = {};
        for (int d = 0; d < dp; d += 4) {
            float4 qq[4], kk[4];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                qq[x] = *reinterpret_cast<const float4*>(q + (i0 + 16 * x) * dp + d);
                kk[x] = *reinterpret_cast<const float4*>(k + (j0 + 16 * x) * dp + d);
            }
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y)
                    acc[x][y] = fmaf(qq[x].x, kk[y].x, fmaf(qq[x].y, kk[y].y, fmaf(qq[x].z, kk[y].z, fmaf(qq[x].w, kk[y].w, acc[x][y]))));
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y) {
                const int i = i0 + 16 * x, j = j0 + 16 * y;
                A[i * AP + j] = j <= i ? acc[x][y] * pw[i - j] : 0.0f;
            }
    }
    __syncthreads();
    const float* S = a.workspace + (static_cast<int64_t>(c) * a.heads + h) * a.dim * a.vdim;
    const int te = ep / 4, tiles = (kChunk / 4) * te;
    for (int t = threadIdx.x; t < tiles; t += kThreads) {
        const int i0 = (t / te) * 4, e0 = (t % te) * 4;
        if (i0 >= ci.len) continue;
        float in[4][4] = {}, acc[4][4] = {};
        for (int d = 0; d < a.dim; ++d) {
            float s[4];
#pragma unroll
            for (int y = 0; y < 4; ++y) s[y] = e0 + y < a.vdim ? S[static_cast<int64_t>(d) * a.vdim + e0 + y] : 0.0f;
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float qv = q[(i0 + x) * dp + d];
#pragma unroll
                for (int y = 0; y < 4; ++y) in[x][y] = fmaf(qv, s[y], in[x][y]);
            }
        }
        for (int j = 0; j < i0 + 4; ++j) {
            const float4 vv = *reinterpret_cast<const float4*>(v + j * ep + e0);
            const float vr[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float w = A[(i0 + x) * AP + j];
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(w, vr[y], acc[x][y]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            if (i0 + x >= ci.len) break;
            float* o = a.out + ((ci.start + i0 + x) * a.heads + h) * a.vdim;
#pragma unroll
            for (int y = 0; y < 4; ++y)
                if (e0 + y < a.vdim) o[e0 + y] = fmaf(pw[i0 + x + 1], in[x][y], acc[x][y]);
        }
    }
}

// ---- output stage --------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(kThreads)
gated_norm_kernel(const spk_gated_norm_args a) {
    __shared__ float part[32];
    const int64_t t = blockIdx.x;
    T* out = static_cast<T*>(a.out) + t * a.out_stride;
    const bool live = a.active == nullptr || a.active[t] == 1;
    if (a.partials != nullptr) {
        const int len = live ? a.seq_lens[t] : 0;
        const int per = spk_split_keys(len, a.splits);
        const int valid = (len + per - 1) / per;
        const float* p = a.partials + t * a.splits * a.left_width;
        for (int c = threadIdx.x; c < a.left_width; c += kThreads) {
            float s = 0.0f;
            for (int k = 0; k < valid; ++k) s += p[static_cast<int64_t>(k) * a.left_width + c];
            out[c] = spk_from_float<T>(s * a.left_scale);
        }
    }
    const float* x = a.x + t * a.width;
    float ss[1] = {0.0f};
    for (int c = threadIdx.x; c < a.width; c += kThreads) ss[0] = fmaf(x[c], x[c], ss[0]);
    spk_block_sum<1>(ss, part);
    const float inv = 1.0f / sqrtf(ss[0] / static_cast<float>(a.width) + a.eps);
    const T* g = static_cast<const T*>(a.gate) + t * a.gate_stride;
    for (int c = threadIdx.x; c < a.width; c += kThreads) {
        const float y = x[c] * inv * a.w[c] * spk_sigmoid(spk_to_float<T>(g[c]));
        out[a.out_offset + c] = spk_from_float<T>(live ? y * a.scale : 0.0f);
    }
}

// The same with four columns per access: at most 4 * kThreads * V columns, every operand aligned to four elements.
template <typename T, int V>
__global__ void __launch_bounds__(kThreads)
gated_norm_vec_kernel(const spk_gated_norm_args a) {
    __shared__ float part[32];
    const int64_t t = blockIdx.x;
    T* out = static_cast<T*>(a.out) + t * a.out_stride;
    const bool live = a.active == nullptr || a.active[t] == 1;
    const float* x = a.x + t * a.width;
    const T* g = static_cast<const T*>(a.gate) + t * a.gate_stride;
    float4 xv[V], gv[V], wv[V];
    float ss[1] = {0.0f};
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = 4 * (threadIdx.x + i * blockDim.x);
        xv[i] = spk_load4<float, true>(x + c, a.width - c);
        gv[i] = spk_load4<T, true>(g + c, a.width - c);
        wv[i] = spk_load4<float, true>(a.w + c, a.width - c);
    }
    if (a.partials != nullptr) {
        const int len = live ? a.seq_lens[t] : 0;
        const int per = spk_split_keys(len, a.splits);
        const int valid = (len + per - 1) / per;
        const float* p = a.partials + t * a.splits * a.left_width;
        for (int c = 4 * threadIdx.x; c < a.left_width; c += 4 * blockDim.x) {
            float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
            for (int k = 0; k < valid; ++k) {
                const float4 y = spk_load4<float, true>(p + static_cast<int64_t>(k) * a.left_width + c, 4);
                s.x += y.x; s.y += y.y; s.z += y.z; s.w += y.w;
            }
            const float m = a.left_scale;
            spk_store4<T, true>(out + c, make_float4(s.x * m, s.y * m, s.z * m, s.w * m), 4);
        }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) ss[0] += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
    spk_block_sum<1>(ss, part);
    const float inv = a.scale / sqrtf(ss[0] / static_cast<float>(a.width) + a.eps);
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int c = 4 * (threadIdx.x + i * blockDim.x);
        const float4 y = make_float4(xv[i].x * inv * wv[i].x * spk_sigmoid(gv[i].x), xv[i].y * inv * wv[i].y * spk_sigmoid(gv[i].y),
                                     xv[i].z * inv * wv[i].z * spk_sigmoid(gv[i].z), xv[i].w * inv * wv[i].w * spk_sigmoid(gv[i].w));
        spk_store4<T, true>(out + a.out_offset + c, live ? y : make_float4(0.f, 0.f, 0.f, 0.f), a.width - c);
    }
}

template <typename T>
int launch_gated(const spk_gated_norm_args& a, cudaStream_t s) {
    const unsigned grid = static_cast<unsigned>(a.n);
    auto aligned = [](const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; };
    const bool vec = a.width % 4 == 0 && a.width <= 4 * kThreads * 4 && a.out_offset % 4 == 0 && a.out_stride % 4 == 0 && a.gate_stride % 4 == 0 &&
                     aligned(a.x, 16) && aligned(a.w, 16) && aligned(a.gate, 4 * sizeof(T)) && aligned(a.out, 4 * sizeof(T)) &&
                     (a.partials == nullptr || (a.left_width % 4 == 0 && aligned(a.partials, 16)));
    if (!vec) {
        gated_norm_kernel<T><<<grid, kThreads, 0, s>>>(a);
    } else {
        const int groups = a.width / 4;
        const int threads = groups <= 128 && a.partials == nullptr ? 128 : kThreads;
        const int v = (groups + threads - 1) / threads;
        if (v <= 1) gated_norm_vec_kernel<T, 1><<<grid, threads, 0, s>>>(a);
        else if (v <= 2) gated_norm_vec_kernel<T, 2><<<grid, threads, 0, s>>>(a);
        else gated_norm_vec_kernel<T, 4><<<grid, threads, 0, s>>>(a);
    }
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

int check_decay(const spk_decay_attn_args* a) {
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->heads < 1 || a->dim < 1 || a->vdim < 1 || a->state_rows < 1 || a->heads > 65535) return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->q == nullptr || a->k == nullptr || a->v == nullptr || a->state == nullptr || a->decay_pow == nullptr || a->out == nullptr)
        return SPK_ERR_NULL_POINTER;
    if (a->state_stride < static_cast<int64_t>(a->heads) * a->dim * a->vdim) return SPK_ERR_BAD_STRIDE;
    return SPK_OK;
}

int smem_attr(const void* fn, size_t bytes) {
    if (bytes > 227 * 1024) return SPK_ERR_TOO_LARGE;
    if (bytes > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes));
        if (e != cudaSuccess) return spk_set_cuda_error(e);
    }
    return SPK_OK;
}

template <typename T>
int launch_step(const spk_decay_attn_args& a, cudaStream_t s) {
    const bool vec = a.vdim % 4 == 0 && a.state_stride % 4 == 0 && reinterpret_cast<uintptr_t>(a.state) % 16 == 0;
    const int cols = vec ? a.vdim / 4 : a.vdim;
    const int slices = cols < kThreads ? kThreads / cols : 1;
    const size_t bytes = sizeof(float) * (2 * static_cast<size_t>(a.dim) + a.vdim + static_cast<size_t>(slices) * a.vdim);
    const dim3 grid(a.heads, static_cast<unsigned>(a.n));
    const void* fn = vec ? reinterpret_cast<const void*>(decay_step_kernel<T, 4>) : reinterpret_cast<const void*>(decay_step_kernel<T, 1>);
    if (const int rc = smem_attr(fn, bytes)) return rc;
    return spk_launch(vec ? decay_step_kernel<T, 4> : decay_step_kernel<T, 1>, grid, kThreads, bytes, s, a.overlap != 0, a);
}

int launch_scan(const spk_decay_attn_args& a, cudaStream_t s) {
    const int64_t per = static_cast<int64_t>(a.heads) * a.dim * a.vdim;
    decay_scan_kernel<<<dim3(static_cast<unsigned>((per + kThreads - 1) / kThreads), a.n_seqs), kThreads, 0, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

template <typename T>
int launch_chunks(const spk_decay_attn_args& a, cudaStream_t s) {
    const size_t dp = pad4(a.dim), ep = pad4(a.vdim);
    const size_t b1 = sizeof(float) * kChunk * (dp + ep), b3 = sizeof(float) * kChunk * (2 * dp + ep + kChunk + 1);
    if (const int rc = smem_attr(reinterpret_cast<const void*>(decay_chunk_sum_kernel<T>), b1)) return rc;
    if (const int rc = smem_attr(reinterpret_cast<const void*>(decay_chunk_out_kernel<T>), b3)) return rc;
    const dim3 grid(a.n_chunks, a.heads);
    decay_chunk_sum_kernel<T><<<grid, kThreads, b1, s>>>(a);
    SPK_CHECK_LAUNCH();
    if (const int rc = launch_scan(a, s)) return rc;
    decay_chunk_out_kernel<T><<<grid, kThreads, b3, s>>>(a);
    SPK_CHECK_LAUNCH();
    return SPK_OK;
}

}  // namespace

extern "C" int spk_decay_powers(void) { return kPow; }

extern "C" int spk_decay_chunk_tokens(int dtype, int dim, int vdim, int64_t n, int heads) {
    if (!spk_decay_tensor_form(dtype, dim, vdim) || n < 1 || heads < 1) return kChunk;
    // the span whose waves of CTAs take least: a chunk is one unit, a CTA's set-up and its state's traffic one more
    const int64_t slots = 148 * (dim <= 64 && vdim <= 64 ? 2 : 1);
    int span = kChunk;
    int64_t best = INT64_MAX;
    for (int s = kChunk; s <= kDecayMaxSpan; s *= 2) {
        const int64_t ctas = (n + s - 1) / s * heads;
        const int64_t cost = (ctas + slots - 1) / slots * (s / kChunk + 1);
        if (cost <= best) {
            best = cost;
            span = s;
        }
    }
    return span;
}

extern "C" int64_t spk_decay_attn_workspace_bytes(int n_chunks, int heads, int dim, int vdim) {
    if (n_chunks < 1 || heads < 1 || dim < 1 || vdim < 1) return 0;
    return static_cast<int64_t>(n_chunks) * heads * dim * vdim * static_cast<int64_t>(sizeof(float));
}

extern "C" int spk_decay_attn_step(const spk_decay_attn_args* a, void* stream) {
    SpkRange nvtx_range("spk_decay_attn_step");
    const int rc = check_decay(a);
    if (rc != SPK_OK || a->n == 0) return rc;
    if (a->n > 65535) return SPK_ERR_TOO_LARGE;
    if (a->n > a->state_rows) return SPK_ERR_BAD_SHAPE;
    cudaStream_t s = spk_stream(stream);
    return a->dtype == SPK_F32 ? launch_step<float>(*a, s) : launch_step<__nv_bfloat16>(*a, s);
}

extern "C" int spk_decay_attn_chunks(const spk_decay_attn_args* a, void* stream) {
    SpkRange nvtx_range("spk_decay_attn_chunks");
    const int rc = check_decay(a);
    if (rc != SPK_OK || a->n == 0) return rc;
    if (a->n_chunks < 1 || a->n_seqs < 1 || a->n_seqs > 65535) return SPK_ERR_BAD_SHAPE;
    if (a->chunks == nullptr || a->seqs == nullptr) return SPK_ERR_NULL_POINTER;
    if (reinterpret_cast<uintptr_t>(a->chunks) % 16 != 0 || reinterpret_cast<uintptr_t>(a->seqs) % 16 != 0) return SPK_ERR_BAD_STRIDE;
    if (a->workspace == nullptr || a->workspace_bytes < spk_decay_attn_workspace_bytes(a->n_chunks, a->heads, a->dim, a->vdim))
        return SPK_ERR_WORKSPACE_TOO_SMALL;
    cudaStream_t s = spk_stream(stream);
    if (spk_decay_tensor_form(a->dtype, a->dim, a->vdim)) {
        if (const int e = spk_decay_mma_sums(*a, s)) return e;
        if (const int e = launch_scan(*a, s)) return e;
        return spk_decay_mma_outputs(*a, s);
    }
    return a->dtype == SPK_F32 ? launch_chunks<float>(*a, s) : launch_chunks<__nv_bfloat16>(*a, s);
}

extern "C" int spk_gated_norm(const spk_gated_norm_args* a, void* stream) {
    SpkRange nvtx_range("spk_gated_norm");
    if (a == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->n < 0 || a->width < 1 || a->out_offset < 0) return SPK_ERR_BAD_SHAPE;
    if (a->dtype != SPK_F32 && a->dtype != SPK_BF16) return SPK_ERR_BAD_DTYPE;
    if (a->n == 0) return SPK_OK;
    if (a->n > 0x7fffffffLL) return SPK_ERR_TOO_LARGE;
    if (a->x == nullptr || a->w == nullptr || a->gate == nullptr || a->out == nullptr) return SPK_ERR_NULL_POINTER;
    if (a->partials != nullptr && (a->seq_lens == nullptr || a->splits < 1 || a->left_width < 1 ||
                                   a->left_width > a->out_offset))
        return SPK_ERR_BAD_SHAPE;
    cudaStream_t s = spk_stream(stream);
    return a->dtype == SPK_F32 ? launch_gated<float>(*a, s) : launch_gated<__nv_bfloat16>(*a, s);
}
