// Kernels around a residual stream: token rows with a sinusoidal position vector, norms over groups of channels, and
// several residual streams that a sublayer reads one combination of and writes into all of.
//
// The streams are float and so is all arithmetic; the normalised rows that a sublayer's first matrix product reads
// leave in float or bfloat16. Every sum runs in an order fixed by the row's sizes, whatever the number of rows.
#include "common.cuh"

IB_DEFINE_LAST_ERROR()

#define IB_LAUNCH(kernel, grid, block, smem, ...)                                                              \
    do {                                                                                                       \
        const int rc_ = ib::launch(#kernel, kernel, dim3(grid), dim3(block), size_t(smem), stream, 1u, __VA_ARGS__); \
        if (rc_) return rc_;                                                                                   \
    } while (0)

namespace {

using bf16 = __nv_bfloat16;

inline unsigned blocks_for(int64_t n, int threads) { return unsigned((n + threads - 1) / threads); }

// ------------------------------------------------------------------------------------------------
// out[t, c] = table[ids[t], c] * scale + (c even: sin, c odd: cos)(positions[t] * freq[c / 2]). Frequencies are double
// and so is the angle, which is brought into one turn before the float sine and cosine: at a position of hundreds of
// thousands a float product alone would be off by hundredths of a radian. Ids as for the plain embedding kernel (an id
// of -1: the token that the sampler left in feedback[slot of the request]).
template <typename T>
__global__ void embedding_sinusoid_kernel(const T* __restrict__ table, const int* __restrict__ ids, const int* __restrict__ positions,
                                          const double* __restrict__ freq, int64_t n_tokens, int64_t width, int64_t vocab,
                                          float* __restrict__ out, int* status, const int* __restrict__ feedback,
                                          const int* __restrict__ token_seg, const int* __restrict__ seg_slot, float scale) {
    ib::pdl_wait();
    const int64_t pairs = (width + 1) / 2;
    const int64_t i = int64_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= n_tokens * pairs) return;
    const int64_t t = i / pairs, c = (i - t * pairs) * 2;
    int id = ids[t];
    if (id == -1 && feedback) id = feedback[seg_slot[token_seg[t]]];
    float* o = out + t * width + c;
    const bool two = c + 1 < width;
    if (id < 0 || id >= vocab) {
        o[0] = 0.0f;
        if (two) o[1] = 0.0f;
        if (status) atomicExch(status, 1);
        return;
    }
    constexpr double TURN = 6.283185307179586476925;
    const double a = double(positions[t]) * freq[c / 2];
    const float r = float(a - TURN * rint(a / TURN));
    const T* row = table + int64_t(id) * width + c;
    o[0] = fmaf(ib::to_f32(row[0]), scale, sinf(r));
    if (two) o[1] = fmaf(ib::to_f32(row[1]), scale, cosf(r));
}

// ------------------------------------------------------------------------------------------------
// One CTA per row. The row's n streams x_s [width] (x_stream apart; 0: all streams are the same row) first take what the
// last sublayer returned, x_t <- sum_s mix[s, t] x_s + out_w[t] y (y null: they stay), and are stored to x_out (may be x;
// null: not stored); then u = sum_s in_w[s] x_s (in_w null: the plain sum), each of `groups` equal parts of u is divided
// by sqrt(mean(part^2) + eps), and the whole is multiplied by w (w null: u itself) into n_out. `rows` picks input rows.
// The block's warps are shared out among the groups (several warps a group, or several groups a warp, by the number
// of groups alone). V: elements per access (4 where sizes and addresses allow).
constexpr int LINK_THREADS = 256;
constexpr int LINK_WARPS = LINK_THREADS / 32;
constexpr int LINK_MAX_STREAMS = 16;

template <int V> struct Pack;
template <> struct Pack<1> { using type = float; };
template <> struct Pack<4> { using type = float4; };

template <int NS, int V, typename TC>
__global__ void __launch_bounds__(LINK_THREADS)
stream_link_kernel(const float* x, int64_t x_row, int64_t x_stream, const float* __restrict__ y, const float* __restrict__ mix,
                   const float* __restrict__ out_w, const float* __restrict__ in_w, const float* __restrict__ w, float eps, int groups,
                   int64_t width, float* x_out, TC* __restrict__ n_out, const int* __restrict__ rows, int ns) {
    extern __shared__ __align__(16) float u_s[];             // [width]
    __shared__ float M[NS * NS + 2 * NS];                    // mix, out_w, in_w
    __shared__ float red[LINK_WARPS];
    using P = typename Pack<V>::type;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* Bw = M + NS * NS;
    float* Aw = Bw + NS;
    for (int i = tid; i < NS * NS; i += LINK_THREADS) {      // (weights: no predecessor writes them)
        const int s = i / NS, t = i - s * NS;
        M[i] = (mix && s < ns && t < ns) ? mix[s * ns + t] : 0.0f;
    }
    for (int i = tid; i < NS; i += LINK_THREADS) {
        Bw[i] = (out_w && i < ns) ? out_w[i] : 0.0f;
        Aw[i] = i < ns ? (in_w ? in_w[i] : 1.0f) : 0.0f;
    }
    __syncthreads();
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int64_t r_out = blockIdx.x;
    const int64_t r = rows ? rows[r_out] : r_out;
    const float* xr = x + r * x_row;
    const float* yr = y ? y + r * width : nullptr;
    float* xo = x_out ? x_out + r_out * (int64_t(ns) * width) : nullptr;
    const int64_t part = width / groups, part_p = part / V;
    const int per_group = groups <= LINK_WARPS ? LINK_WARPS / groups : 1;      // warps of a group

    auto element = [&](int64_t i) -> float {                 // elements V i .. V i + V - 1; returns their sum of squares of u
        __align__(16) float xs[NS][V], u[V];
#pragma unroll
        for (int s = 0; s < NS; s++) {
            if (s < ns) *reinterpret_cast<P*>(xs[s]) = *reinterpret_cast<const P*>(xr + s * x_stream + i * V);
        }
#pragma unroll
        for (int e = 0; e < V; e++) u[e] = 0.0f;
        if (yr) {
            __align__(16) float ys[V];
            *reinterpret_cast<P*>(ys) = *reinterpret_cast<const P*>(yr + i * V);
#pragma unroll
            for (int t = 0; t < NS; t++) {
                if (t < ns) {
                    __align__(16) float nx[V];
#pragma unroll
                    for (int e = 0; e < V; e++) {
                        nx[e] = Bw[t] * ys[e];
#pragma unroll
                        for (int s = 0; s < NS; s++)
                            if (s < ns) nx[e] = fmaf(M[s * NS + t], xs[s][e], nx[e]);
                        u[e] = fmaf(Aw[t], nx[e], u[e]);
                    }
                    if (xo) *reinterpret_cast<P*>(xo + t * width + i * V) = *reinterpret_cast<P*>(nx);
                }
            }
        } else {
#pragma unroll
            for (int t = 0; t < NS; t++) {
                if (t < ns) {
#pragma unroll
                    for (int e = 0; e < V; e++) u[e] = fmaf(Aw[t], xs[t][e], u[e]);
                    if (xo) *reinterpret_cast<P*>(xo + t * width + i * V) = *reinterpret_cast<P*>(xs[t]);
                }
            }
        }
        *reinterpret_cast<P*>(u_s + i * V) = *reinterpret_cast<P*>(u);
        float ss = 0.0f;
#pragma unroll
        for (int e = 0; e < V; e++) ss = fmaf(u[e], u[e], ss);
        return ss;
    };
    auto emit = [&](int64_t i, float f) {
        __align__(16) float v[V];
        *reinterpret_cast<P*>(v) = *reinterpret_cast<P*>(u_s + i * V);
        if (w) {
            __align__(16) float ws[V];
            *reinterpret_cast<P*>(ws) = *reinterpret_cast<const P*>(w + i * V);
#pragma unroll
            for (int e = 0; e < V; e++) v[e] *= f * ws[e];
        }
        TC* o = n_out + r_out * width + i * V;
        if constexpr (sizeof(TC) == 4) {
            *reinterpret_cast<P*>(o) = *reinterpret_cast<P*>(v);
        } else if constexpr (V == 4) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
            uint2 two;
            two.x = *reinterpret_cast<uint32_t*>(&lo);
            two.y = *reinterpret_cast<uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(o) = two;
        } else {
            *o = ib::from_f32<TC>(v[0]);
        }
    };
    if (groups <= LINK_WARPS) {
        const int g = warp / per_group, wl = warp - g * per_group;
        const int64_t i0 = int64_t(g) * part_p, step = int64_t(per_group) * 32;
        float ss = 0.0f;
        if (g < groups)
            for (int64_t i = wl * 32 + lane; i < part_p; i += step) ss += element(i0 + i);
        ss = ib::warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        if (g < groups) {
            float total = 0.0f;
            for (int i = 0; i < per_group; i++) total += red[g * per_group + i];
            const float f = w ? 1.0f / sqrtf(total / float(part) + eps) : 1.0f;
            for (int64_t i = wl * 32 + lane; i < part_p; i += step) emit(i0 + i, f);     // (a thread's own elements)
        }
    } else {
        for (int g = warp; g < groups; g += LINK_WARPS) {
            const int64_t i0 = int64_t(g) * part_p;
            float ss = 0.0f;
            for (int64_t i = lane; i < part_p; i += 32) ss += element(i0 + i);
            ss = ib::warp_sum(ss);
            const float f = w ? 1.0f / sqrtf(ss / float(part) + eps) : 1.0f;
            for (int64_t i = lane; i < part_p; i += 32) emit(i0 + i, f);
        }
    }
}

template <int NS, int V, typename TC>
int launch_link(unsigned n_rows, size_t smem, cudaStream_t stream, const float* x, int64_t x_row, int64_t x_stream, const float* y,
                const float* mix, const float* out_w, const float* in_w, const float* w, float eps, int groups, int64_t width,
                float* x_out, TC* n_out, const int* rows, int ns) {
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(stream_link_kernel<NS, V, TC>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
        if (e != cudaSuccess) return ib::fail(IB_ERR_CUDA, "ib_stream_link: cannot set shared memory size: %s", cudaGetErrorString(e));
    }
    IB_LAUNCH((stream_link_kernel<NS, V, TC>), n_rows, LINK_THREADS, smem, x, x_row, x_stream, y, mix, out_w, in_w, w, eps, groups, width,
              x_out, n_out, rows, ns);
    return ib::check_launch("ib_stream_link");
}

}  // namespace

// ================================================================================================
// C entry points. dtype arguments: 0 = float, 1 = bfloat16.

IB_EXPORT int ib_embedding_sinusoid(const void* table, int dtype, const int* ids, const int* positions, const double* freq,
                                    int64_t n_tokens, int64_t width, int64_t vocab, float* out, int* status, const int* feedback,
                                    const int* token_seg, const int* seg_slot, float scale, cudaStream_t stream) {
    const int64_t n = n_tokens * ((width + 1) / 2);
    if (n <= 0) return IB_OK;
    if (dtype == IB_F32)
        IB_LAUNCH(embedding_sinusoid_kernel<float>, blocks_for(n, 256), 256, 0, (const float*)table, ids, positions, freq, n_tokens, width,
                  vocab, out, status, feedback, token_seg, seg_slot, scale);
    else if (dtype == IB_BF16)
        IB_LAUNCH(embedding_sinusoid_kernel<bf16>, blocks_for(n, 256), 256, 0, (const bf16*)table, ids, positions, freq, n_tokens, width,
                  vocab, out, status, feedback, token_seg, seg_slot, scale);
    else
        return ib::fail(IB_ERR_ARG, "ib_embedding_sinusoid: unknown dtype %d", dtype);
    return ib::check_launch("ib_embedding_sinusoid");
}

// The most streams that ib_stream_link takes.
IB_EXPORT int ib_stream_link_max_streams() { return LINK_MAX_STREAMS; }

// x: n_streams rows of `width` per token, x_row floats between tokens and x_stream between a token's streams (0: all
// the same row); y [tokens, width] with mix [n_streams (from), n_streams (to)] and out_w [n_streams], or null; in_w
// [n_streams] or null (the plain sum); w [width] or null (no norm); x_out [rows, n_streams, width] or null; n_out
// [rows, width]; rows: which tokens (null: the first n_rows).
IB_EXPORT int ib_stream_link(const float* x, int64_t x_row, int64_t x_stream, const float* y, const float* mix, const float* out_w,
                             const float* in_w, const float* w, float eps, int groups, int64_t width, float* x_out, void* n_out,
                             int n_dtype, const int* rows, int64_t n_rows, int n_streams, cudaStream_t stream) {
    if (n_rows <= 0 || width <= 0) return IB_OK;
    if (!x || !n_out) return ib::fail(IB_ERR_ARG, "ib_stream_link: streams and a result are needed");
    if (n_streams < 1 || n_streams > LINK_MAX_STREAMS) return ib::fail(IB_ERR_ARG, "ib_stream_link: %d streams (up to %d)", n_streams, LINK_MAX_STREAMS);
    if (groups < 1 || width % groups) return ib::fail(IB_ERR_ARG, "ib_stream_link: rows of %lld in %d groups", (long long)width, groups);
    if (y && (!mix || !out_w)) return ib::fail(IB_ERR_ARG, "ib_stream_link: a sublayer's result needs its two matrices");
    if (x_out == x && x_stream == 0 && n_streams > 1) return ib::fail(IB_ERR_ARG, "ib_stream_link: one shared row cannot take several streams");
    if (x_out == x && rows) return ib::fail(IB_ERR_ARG, "ib_stream_link: picked rows go to a buffer of their own");
    if (n_dtype != IB_F32 && n_dtype != IB_BF16) return ib::fail(IB_ERR_ARG, "ib_stream_link: unknown dtype %d", n_dtype);
    const size_t smem = size_t(width) * sizeof(float);
    if (smem > 220 * 1024) return ib::fail(IB_ERR_ARG, "ib_stream_link: rows of %lld do not fit", (long long)width);
    const int64_t part = width / groups;
    const bool vec = part % 4 == 0 && x_row % 4 == 0 && x_stream % 4 == 0 &&
                     !((uintptr_t(x) | uintptr_t(y) | uintptr_t(w) | uintptr_t(x_out) | uintptr_t(n_out)) & 15);
#define IB_LINK(NS)                                                                                                                         \
    do {                                                                                                                                    \
        if (vec && n_dtype == IB_F32) return launch_link<NS, 4, float>(unsigned(n_rows), smem, stream, x, x_row, x_stream, y, mix, out_w,  \
                                                                       in_w, w, eps, groups, width, x_out, (float*)n_out, rows, n_streams); \
        if (vec) return launch_link<NS, 4, bf16>(unsigned(n_rows), smem, stream, x, x_row, x_stream, y, mix, out_w, in_w, w, eps, groups,  \
                                                 width, x_out, (bf16*)n_out, rows, n_streams);                                              \
        if (n_dtype == IB_F32) return launch_link<NS, 1, float>(unsigned(n_rows), smem, stream, x, x_row, x_stream, y, mix, out_w, in_w,   \
                                                                w, eps, groups, width, x_out, (float*)n_out, rows, n_streams);              \
        return launch_link<NS, 1, bf16>(unsigned(n_rows), smem, stream, x, x_row, x_stream, y, mix, out_w, in_w, w, eps, groups, width,     \
                                        x_out, (bf16*)n_out, rows, n_streams);                                                              \
    } while (0)
    switch (n_streams) {
        case 1: IB_LINK(1);
        case 2: IB_LINK(2);
        case 3: IB_LINK(3);
        case 4: IB_LINK(4);
        default: break;
    }
    if (n_streams <= 8) IB_LINK(8);
    IB_LINK(LINK_MAX_STREAMS);
#undef IB_LINK
}
