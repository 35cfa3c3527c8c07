// Kernels for layers whose sublayers' results enter the residual stream through a factor per channel, for state space
// layers (a filter over time in front of a matrix state that fades by one number per head and token) and for matrix
// memories with exponential gates. The recurrences themselves are state_scan mode 5 (mix_ops.cu).
//
// Rows of recurrences, the residual stream and all arithmetic are float; the normalised rows that a layer's first matrix
// products read leave in float or bfloat16. With float storage these kernels are the 32-bit path.
//
// A step's rows are the tokens of several requests ("segments") one after the other: seg_start[s] is the first row
// of segment s, seg_slot[s] the request's state slot. A token's result depends on its own request's earlier tokens
// and state only, and every sum runs in an order fixed by the layer's sizes.
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

__device__ __forceinline__ float silu_(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float log_sigmoid_(float x) { return fminf(x, 0.0f) - log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<unsigned*>(&lo);
    u.y = *reinterpret_cast<unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
}

// ------------------------------------------------------------------------------------------------
// y = x + wa * a + wb * b per row (a, b may be absent; wa, wb: a factor per channel), kept in x with `store`; then
// out = y / sqrt(mean(y^2) + eps) * w, the rows the next sublayers read. `rows` picks and orders input rows (nothing is
// stored then). One CTA per row. VEC: four channels a thread and access.
template <typename TOut, int VEC>
__global__ void __launch_bounds__(256)
scaled_sum_norm_kernel(float* __restrict__ x, const float* __restrict__ a, const float* __restrict__ wa, const float* __restrict__ b,
                       const float* __restrict__ wb, const float* __restrict__ w, float eps, const int* __restrict__ rows, int store,
                       TOut* __restrict__ out, int64_t width) {
    __shared__ float red[32];
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int64_t t = rows ? rows[blockIdx.x] : blockIdx.x;
    float* xr = x + t * width;
    const float* ar = a ? a + t * width : nullptr;
    const float* br = b ? b + t * width : nullptr;
    TOut* o = out + int64_t(blockIdx.x) * width;
    auto sum1 = [&](int64_t i) {
        float y = xr[i];
        if (ar) y = fmaf(wa[i], ar[i], y);
        if (br) y = fmaf(wb[i], br[i], y);
        return y;
    };
    float ss = 0.0f;
    if (VEC == 4) {
        // a thread keeps its first row pieces in registers (rows of up to KEEP * 1024 channels whole)
        constexpr int KEEP = 4;
        float4 kept[KEEP];
        int n = 0;
        auto sum4 = [&](int64_t i) {
            float4 y = load4(xr + i);
            if (ar) {
                const float4 f = load4(wa + i), v = load4(ar + i);
                y.x = fmaf(f.x, v.x, y.x); y.y = fmaf(f.y, v.y, y.y); y.z = fmaf(f.z, v.z, y.z); y.w = fmaf(f.w, v.w, y.w);
            }
            if (br) {
                const float4 f = load4(wb + i), v = load4(br + i);
                y.x = fmaf(f.x, v.x, y.x); y.y = fmaf(f.y, v.y, y.y); y.z = fmaf(f.z, v.z, y.z); y.w = fmaf(f.w, v.w, y.w);
            }
            return y;
        };
#pragma unroll
        for (int k = 0; k < KEEP; k++) {
            const int64_t i = (int64_t(k) * blockDim.x + threadIdx.x) * 4;
            if (i < width) {
                kept[k] = sum4(i);
                n = k + 1;
                ss = fmaf(kept[k].x, kept[k].x, ss); ss = fmaf(kept[k].y, kept[k].y, ss);
                ss = fmaf(kept[k].z, kept[k].z, ss); ss = fmaf(kept[k].w, kept[k].w, ss);
            }
        }
        for (int64_t i = (int64_t(KEEP) * blockDim.x + threadIdx.x) * 4; i < width; i += int64_t(blockDim.x) * 4) {
            const float4 y = sum4(i);
            ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
        }
        ss = ib::block_sum(ss, red);
        const float f = 1.0f / sqrtf(ss / float(width) + eps);
        auto finish = [&](int64_t i, float4 y) {
            if (store && ar) store4(xr + i, y);
            const float4 wv = load4(w + i);
            store4(o + i, make_float4(y.x * f * wv.x, y.y * f * wv.y, y.z * f * wv.z, y.w * f * wv.w));
        };
#pragma unroll
        for (int k = 0; k < KEEP; k++)
            if (k < n) finish((int64_t(k) * blockDim.x + threadIdx.x) * 4, kept[k]);
        for (int64_t i = (int64_t(KEEP) * blockDim.x + threadIdx.x) * 4; i < width; i += int64_t(blockDim.x) * 4) finish(i, sum4(i));
        return;
    }
    for (int64_t i = threadIdx.x; i < width; i += blockDim.x) {
        const float y = sum1(i);
        ss = fmaf(y, y, ss);
    }
    ss = ib::block_sum(ss, red);
    const float f = 1.0f / sqrtf(ss / float(width) + eps);
    for (int64_t i = threadIdx.x; i < width; i += blockDim.x) {
        const float y = sum1(i);
        if (store && ar) xr[i] = y;
        o[i] = ib::from_f32<TOut>(y * f * w[i]);
    }
}

// ------------------------------------------------------------------------------------------------
// What a state space layer's recurrence reads, from the projected rows: columns [col0, col0 + channels) each through a
// causal filter over time, y_t = bias + sum_j w[j][c] u_(t - taps + 1 + j) (u before the segment's first row comes from
// the request's tail, its last taps - 1 inputs, oldest first; zeros for a new request), then silu; and per head, from
// column dt_col, dt = softplus(raw + dt_bias[h]) and g = exp(-exp(a_log[h]) dt).
// out rows (ldo): [channels | up to a multiple of 4 | g (H) | dt (H) | ln g (H)]. Filter weights tap-major [taps, channels].
// inline_tail (steps of one token per request only): the thread that filters a channel, the only reader of its tail, moves it.
// A CTA of 128 threads: VEC channels a thread, grid (tokens, blocks of channels and heads).
template <int VEC>
__global__ void __launch_bounds__(128)
filter_prepare_kernel(const float* __restrict__ rows, int64_t ld, int col0, int channels, const float* __restrict__ filt_w,
                      const float* __restrict__ filt_b, int taps, float* tails, int inline_tail, int dt_col,
                      const float* __restrict__ dt_bias, const float* __restrict__ a_log, int n_heads, const int* __restrict__ token_seg,
                      const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ out, int64_t ldo) {
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int64_t t = blockIdx.x;
    const int u = blockIdx.y * blockDim.x + threadIdx.x;
    const int n_units = (channels + VEC - 1) / VEC;
    if (u >= n_units) {
        const int h = u - n_units;
        if (h >= n_heads) return;
        const float dt = softplus_(rows[t * ld + dt_col + h] + dt_bias[h]);
        float* o = out + t * ldo + (channels + 3) / 4 * 4;
        const float lng = -expf(a_log[h]) * dt;
        o[h] = expf(lng);
        o[n_heads + h] = dt;
        o[2 * n_heads + h] = lng;
        return;
    }
    const int c = u * VEC;
    const int s = token_seg[t];
    const int i_local = int(t - seg_start[s]);
    float* tail = taps > 1 ? tails + int64_t(seg_slot[s]) * (taps - 1) * channels + c : nullptr;
    float y[VEC], newest[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) { y[e] = filt_b[c + e]; newest[e] = 0.0f; }
    for (int j = 0; j < taps; j++) {
        const int back = taps - 1 - j;
        const float* in = i_local >= back ? rows + (t - back) * ld + col0 + c : tail + int64_t(taps - 1 + i_local - back) * channels;
        const float* w = filt_w + int64_t(j) * channels + c;
        if (VEC == 4) {
            const float4 v = load4(in), f = load4(w);
            y[0] = fmaf(f.x, v.x, y[0]); y[1 % VEC] = fmaf(f.y, v.y, y[1 % VEC]);
            y[2 % VEC] = fmaf(f.z, v.z, y[2 % VEC]); y[3 % VEC] = fmaf(f.w, v.w, y[3 % VEC]);
            newest[0] = v.x; newest[1 % VEC] = v.y; newest[2 % VEC] = v.z; newest[3 % VEC] = v.w;
        } else {
            newest[0] = in[0];
            y[0] = fmaf(w[0], newest[0], y[0]);
        }
    }
    if (inline_tail && taps > 1) {
        for (int idx = 0; idx + 1 < taps - 1; idx++)
#pragma unroll
            for (int e = 0; e < VEC; e++) tail[int64_t(idx) * channels + e] = tail[int64_t(idx + 1) * channels + e];
#pragma unroll
        for (int e = 0; e < VEC; e++) tail[int64_t(taps - 2) * channels + e] = newest[e];
    }
    float* o = out + t * ldo + c;
    if (VEC == 4) {
        store4(o, make_float4(silu_(y[0]), silu_(y[1 % VEC]), silu_(y[2 % VEC]), silu_(y[3 % VEC])));
    } else {
        o[0] = silu_(y[0]);
    }
}

// filter_prepare for FT tokens a thread (prompt portions): the inputs that neighbouring tokens share are read once. Tokens
// near their segment's start, or of different segments, take their inputs one by one as above; the sums are the same.
constexpr int FT = 4;

template <int TAPS>
__global__ void __launch_bounds__(128)
filter_prepare_tokens_kernel(const float* __restrict__ rows, int64_t ld, int col0, int channels, const float* __restrict__ filt_w,
                             const float* __restrict__ filt_b, const float* __restrict__ tails, int dt_col, const float* __restrict__ dt_bias,
                             const float* __restrict__ a_log, int n_heads, const int* __restrict__ token_seg,
                             const int* __restrict__ seg_start, const int* __restrict__ seg_slot, float* __restrict__ out, int64_t ldo,
                             int64_t n_tokens) {
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int64_t t0 = int64_t(blockIdx.x) * FT;
    const int nt = int(min(int64_t(FT), n_tokens - t0));
    const int u = blockIdx.y * blockDim.x + threadIdx.x;
    const int n_units = channels / 4;
    if (u >= n_units) {
        const int h = u - n_units;
        if (h >= n_heads) return;
        const float rate = expf(a_log[h]);
        for (int i = 0; i < nt; i++) {
            const float dt = softplus_(rows[(t0 + i) * ld + dt_col + h] + dt_bias[h]);
            float* o = out + (t0 + i) * ldo + channels;
            const float lng = -rate * dt;
            o[h] = expf(lng);
            o[n_heads + h] = dt;
            o[2 * n_heads + h] = lng;
        }
        return;
    }
    const int c = u * 4;
    float4 w[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; j++) w[j] = load4(filt_w + int64_t(j) * channels + c);
    const float4 b = load4(filt_b + c);
    auto finish = [&](int64_t t, float4 y) { store4(out + t * ldo + c, make_float4(silu_(y.x), silu_(y.y), silu_(y.z), silu_(y.w))); };
    const int s = token_seg[t0];
    const int first = int(t0 - seg_start[s]);
    if (nt == FT && first >= TAPS - 1 && token_seg[t0 + FT - 1] == s) {
        float4 in[FT + TAPS - 1];
#pragma unroll
        for (int i = 0; i < FT + TAPS - 1; i++) in[i] = load4(rows + (t0 - (TAPS - 1) + i) * ld + col0 + c);
#pragma unroll
        for (int i = 0; i < FT; i++) {
            float4 y = b;
#pragma unroll
            for (int j = 0; j < TAPS; j++) {
                y.x = fmaf(w[j].x, in[i + j].x, y.x); y.y = fmaf(w[j].y, in[i + j].y, y.y);
                y.z = fmaf(w[j].z, in[i + j].z, y.z); y.w = fmaf(w[j].w, in[i + j].w, y.w);
            }
            finish(t0 + i, y);
        }
        return;
    }
    for (int i = 0; i < nt; i++) {
        const int64_t t = t0 + i;
        const int sg = token_seg[t];
        const int i_local = int(t - seg_start[sg]);
        const float* tail = TAPS > 1 ? tails + int64_t(seg_slot[sg]) * (TAPS - 1) * channels + c : nullptr;
        float4 y = b;
#pragma unroll
        for (int j = 0; j < TAPS; j++) {
            const int back = TAPS - 1 - j;
            const float4 v = load4(i_local >= back ? rows + (t - back) * ld + col0 + c : tail + int64_t(TAPS - 1 + i_local - back) * channels);
            y.x = fmaf(w[j].x, v.x, y.x); y.y = fmaf(w[j].y, v.y, y.y); y.z = fmaf(w[j].z, v.z, y.z); y.w = fmaf(w[j].w, v.w, y.w);
        }
        finish(t, y);
    }
}

// ------------------------------------------------------------------------------------------------
// Gates of a matrix memory over the tokens of every segment in order, one CTA per (segment, head):
//   i = cap tanh((raw[i_col + h] + i_bias[h]) / cap),   f = log sigmoid(cap tanh((raw[f_col + h] + f_bias[h]) / cap))
//   m <- max(f + m, i)   (m kept per request and head in `state` [slots, H], zero for a new request)
//   out rows (ldo): [keep = exp(f + m_before - m) (H) | write = exp(i - m) (H) | floor = exp(-m) (H) | ln keep (H)]
// The gates and the exponentials are computed in parallel over a tile of tokens. The running maximum walks the tile in one
// thread, an addition and a maximum a token, so that it does not depend on where a prompt was cut. With `blocks` (where its
// last bits may) a tile of n tokens is cut into blocks of GATE_BLOCK: what a block makes of the maximum in front of it is
// max(a + m, b), and a thread per block finds a (its sum of f) and b; a walk over the blocks gives the maximum in front of
// each, and the threads walk their blocks again from there.
constexpr int GATE_TILE = 2048, GATE_BLOCK = 32;

__global__ void __launch_bounds__(512)
memory_gates_kernel(const float* __restrict__ rows, int64_t ld, int i_col, int f_col, const float* __restrict__ i_bias,
                    const float* __restrict__ f_bias, float cap, float* __restrict__ state, const int* __restrict__ seg_start,
                    const int* __restrict__ seg_slot, float* __restrict__ out, int64_t ldo, int n_heads, int write_state, int blocks) {
    // (a block's tokens start one place further on than the last block's: threads that walk neighbouring blocks use
    // different banks)
    __shared__ __align__(16) float gi[GATE_TILE + GATE_TILE / GATE_BLOCK + 8], gf[GATE_TILE + GATE_TILE / GATE_BLOCK + 8];
    __shared__ __align__(16) float gm[GATE_TILE + GATE_TILE / GATE_BLOCK + 8];
    __shared__ float ba[GATE_TILE / GATE_BLOCK], bb[GATE_TILE / GATE_BLOCK], bm[GATE_TILE / GATE_BLOCK + 1];
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int64_t t0 = seg_start[s];
    const int len = int(seg_start[s + 1] - t0);
    float* kept = state + int64_t(seg_slot[s]) * n_heads + h;
    const float bi = i_bias[h], bf = f_bias[h];
    float m = *kept;
    const int pad = blocks ? 1 : 0;
    auto at = [&](int c) { return c + pad * (c / GATE_BLOCK); };
    for (int c0 = 0; c0 < len; c0 += GATE_TILE) {
        const int n = min(GATE_TILE, len - c0);
        for (int c = tid; c < n; c += blockDim.x) {
            const float* r = rows + (t0 + c0 + c) * ld;
            gi[at(c)] = cap * tanhf((r[i_col + h] + bi) / cap);
            gf[at(c)] = log_sigmoid_(cap * tanhf((r[f_col + h] + bf) / cap));
        }
        __syncthreads();
        // gm[at(c)] is the maximum before token c; bm[last] the one after the tile
        const int n_blocks = (n + GATE_BLOCK - 1) / GATE_BLOCK;
        if (blocks) {
            if (tid < n_blocks) {
                const int c1 = min(n, (tid + 1) * GATE_BLOCK);
                float a = 0.0f, b = -INFINITY;
                for (int c = tid * GATE_BLOCK; c < c1; c++) {
                    const float f = gf[at(c)];
                    a += f;
                    b = fmaxf(f + b, gi[at(c)]);
                }
                ba[tid] = a;
                bb[tid] = b;
            }
            __syncthreads();
            if (tid == 0) {
                for (int k = 0; k < n_blocks; k++) {
                    bm[k] = m;
                    m = fmaxf(ba[k] + m, bb[k]);
                }
            }
            __syncthreads();
            if (tid < n_blocks) {
                const int c1 = min(n, (tid + 1) * GATE_BLOCK);
                float mm = bm[tid];
                for (int c = tid * GATE_BLOCK; c < c1; c++) {
                    gm[at(c)] = mm;
                    mm = fmaxf(gf[at(c)] + mm, gi[at(c)]);
                }
                if (tid == n_blocks - 1) bm[n_blocks] = mm;
            }
        } else if (tid == 0) {
            int c = 0;
            float4 i_next = load4(gi), f_next = load4(gf);   // (four tokens ahead of the walk)
            for (; c + 4 <= n; c += 4) {
                const float4 i4 = i_next, f4 = f_next;
                i_next = load4(gi + c + 4);
                f_next = load4(gf + c + 4);
                float4 b4;
                b4.x = m;
                m = fmaxf(f4.x + m, i4.x);
                b4.y = m;
                m = fmaxf(f4.y + m, i4.y);
                b4.z = m;
                m = fmaxf(f4.z + m, i4.z);
                b4.w = m;
                m = fmaxf(f4.w + m, i4.w);
                store4(gm + c, b4);
            }
            for (; c < n; c++) {
                gm[c] = m;
                m = fmaxf(gf[c] + m, gi[c]);
            }
            bm[n_blocks] = m;
        }
        __syncthreads();
        for (int c = tid; c < n; c += blockDim.x) {
            float* o = out + (t0 + c0 + c) * ldo;
            const float f = gf[at(c)], i = gi[at(c)], before = gm[at(c)];
            const float now = fmaxf(f + before, i);
            const float lnk = f + before - now;
            o[h] = expf(lnk);
            o[n_heads + h] = expf(i - now);
            o[2 * n_heads + h] = expf(-now);
            o[3 * n_heads + h] = lnk;
        }
        m = bm[n_blocks];
        __syncthreads();
    }
    if (write_state && tid == 0) *kept = m;
}

}  // namespace

// ================================================================================================
// C entry points. dtype arguments: 0 = float, 1 = bfloat16.

IB_EXPORT int ib_scaled_sum_norm(float* x, const float* a, const float* wa, const float* b, const float* wb, const float* w, float eps,
                                 const int* rows, int store, void* out, int out_dtype, int64_t n_rows, int64_t width,
                                 cudaStream_t stream) {
    if (n_rows <= 0 || width <= 0) return IB_OK;
    if (!x || !w || !out || (a && !wa) || (b && (!wb || !a))) return ib::fail(IB_ERR_ARG, "ib_scaled_sum_norm: rows, their factors and a weight are needed");
    if (rows) store = 0;
    const uintptr_t all = uintptr_t(x) | uintptr_t(a) | uintptr_t(wa) | uintptr_t(b) | uintptr_t(wb) | uintptr_t(w) | uintptr_t(out);
    const bool vec = width % 4 == 0 && !(all & 15);           // (by sizes and addresses, never by the number of rows)
#define IB_SSN(TO, VV) IB_LAUNCH((scaled_sum_norm_kernel<TO, VV>), unsigned(n_rows), 256, 0, x, a, wa, b, wb, w, eps, rows, store, (TO*)out, width)
    if (out_dtype == IB_F32) {
        if (vec) IB_SSN(float, 4); else IB_SSN(float, 1);
    } else if (out_dtype == IB_BF16) {
        if (vec) IB_SSN(bf16, 4); else IB_SSN(bf16, 1);
    } else {
        return ib::fail(IB_ERR_ARG, "ib_scaled_sum_norm: unknown dtype %d", out_dtype);
    }
#undef IB_SSN
    return ib::check_launch("ib_scaled_sum_norm");
}

IB_EXPORT int ib_filter_prepare(const float* rows, int64_t ld, int col0, int channels, const float* filt_w, const float* filt_b, int taps,
                                float* tails, int inline_tail, int dt_col, const float* dt_bias, const float* a_log, int n_heads,
                                const int* token_seg, const int* seg_start, const int* seg_slot, float* out, int64_t ldo,
                                int64_t n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return IB_OK;
    if (channels <= 0 || taps <= 0 || n_heads <= 0 || !filt_w || !filt_b) return ib::fail(IB_ERR_ARG, "ib_filter_prepare: bad sizes");
    if (taps > 1 && !tails) return ib::fail(IB_ERR_ARG, "ib_filter_prepare: a filter of %d taps needs tails", taps);
    if (ldo < (channels + 3) / 4 * 4 + 3 * int64_t(n_heads)) return ib::fail(IB_ERR_ARG, "ib_filter_prepare: result rows too short");
    const uintptr_t all = uintptr_t(rows) | uintptr_t(filt_w) | uintptr_t(taps > 1 ? tails : nullptr) | uintptr_t(out);
    const bool vec = channels % 4 == 0 && col0 % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && !(all & 15);
    const int units = (vec ? channels / 4 : channels) + n_heads;
    const dim3 grid{unsigned(n_tokens), blocks_for(units, 128), 1u};
    if (grid.y > 65535) return ib::fail(IB_ERR_ARG, "ib_filter_prepare: too many channels");
    if (vec && !inline_tail && taps <= 4 && n_tokens >= 256) {          // (the same sums for a token, fewer reads)
        const dim3 grid4{blocks_for(n_tokens, FT), grid.y, 1u};
#define IB_FT(TT)                                                                                                                     \
        IB_LAUNCH(filter_prepare_tokens_kernel<TT>, grid4, 128, 0, rows, ld, col0, channels, filt_w, filt_b, tails, dt_col, dt_bias, a_log, \
                  n_heads, token_seg, seg_start, seg_slot, out, ldo, n_tokens)
        if (taps == 1) IB_FT(1); else if (taps == 2) IB_FT(2); else if (taps == 3) IB_FT(3); else IB_FT(4);
#undef IB_FT
        return ib::check_launch("ib_filter_prepare");
    }
    if (vec)
        IB_LAUNCH(filter_prepare_kernel<4>, grid, 128, 0, rows, ld, col0, channels, filt_w, filt_b, taps, tails, inline_tail, dt_col, dt_bias,
                  a_log, n_heads, token_seg, seg_start, seg_slot, out, ldo);
    else
        IB_LAUNCH(filter_prepare_kernel<1>, grid, 128, 0, rows, ld, col0, channels, filt_w, filt_b, taps, tails, inline_tail, dt_col, dt_bias,
                  a_log, n_heads, token_seg, seg_start, seg_slot, out, ldo);
    return ib::check_launch("ib_filter_prepare");
}

IB_EXPORT int ib_memory_gates(const float* rows, int64_t ld, int i_col, int f_col, const float* i_bias, const float* f_bias, float cap,
                              float* state, const int* seg_start, const int* seg_slot, float* out, int64_t ldo, int n_segments,
                              int n_heads, int write_state, int max_len, int blocks, cudaStream_t stream) {
    if (n_segments <= 0) return IB_OK;
    if (n_heads <= 0 || n_heads > 65535 || !(cap > 0.0f) || ldo < 4 * int64_t(n_heads))
        return ib::fail(IB_ERR_ARG, "ib_memory_gates: %d heads, a cap of %f", n_heads, double(cap));
    // (the number of threads changes nothing but how many tokens of a tile are formed at a time)
    IB_LAUNCH(memory_gates_kernel, (dim3{unsigned(n_segments), unsigned(n_heads), 1u}), max_len > 32 ? 512 : 32, 0, rows, ld, i_col, f_col, i_bias, f_bias, cap,
              state, seg_start, seg_slot, out, ldo, n_heads, write_state, blocks && max_len > 2 * GATE_BLOCK);
    return ib::check_launch("ib_memory_gates");
}
