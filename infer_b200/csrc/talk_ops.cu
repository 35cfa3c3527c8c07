// Attention whose heads exchange their scores before the softmax ("talking heads"), over the paged cache:
//
//     s[g, j] = cap * tanh(scale (q_g . k_j) / cap)      (cap 0: scale (q_g . k_j))
//     s'[h, j] = sum_g talk[h, g] s[g, j]                (talk null: s)
//     out_h = softmax over the visible j of s'[h] . v
//
// Query position p sees keys lo..p with lo = the first position of p's own chunk of `chunk` positions (counted from
// position 0; 0: no chunks), and within `window` positions where a window is given. A score of one head needs every
// head's score of the same (query, key) pair, so a CTA works on all heads of its pairs.
//
// Storage is float or bfloat16 (template parameter); scores, the exchange, softmax and sums are float in both.
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

__device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    return lo;
}

// ------------------------------------------------------------------------------------------------
// k and v of projected rows (columns k_col.., v_col.. of rows [tokens, ld]) into their pages. `PT` elements a thread.
template <typename T, int PT>
__global__ void kv_store_kernel(const T* __restrict__ rows, int64_t ld, int k_col, int v_col, const int* __restrict__ positions,
                                const int* __restrict__ token_seg, const int* __restrict__ block_table, int64_t max_blocks,
                                T* __restrict__ k_cache, T* __restrict__ v_cache, int64_t n_tokens, int n_kv, int d, int dv,
                                int page_size, int64_t n_pages, int* status) {
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int nk = n_kv * d / PT, per = nk + n_kv * dv / PT;
    const int64_t i = int64_t(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= n_tokens * per) return;
    const int64_t t = i / per;
    int c = int(i - t * per);
    const bool is_v = c >= nk;
    if (is_v) c -= nk;
    const int size = is_v ? dv : d;
    const int h = c * PT / size, j = c * PT - h * size;
    const int pos = positions[t];
    const int page = block_table[int64_t(token_seg[t]) * max_blocks + pos / page_size];
    if (page < 0 || page >= n_pages) {
        if (status) atomicExch(status, 2);
        return;
    }
    const T* src = rows + t * ld + (is_v ? v_col : k_col) + h * size + j;
    T* dst = (is_v ? v_cache : k_cache) + ((int64_t(page) * n_kv + h) * page_size + pos % page_size) * size + j;
    if constexpr (PT == 1) *dst = *src;
    else *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(src);
}

// ------------------------------------------------------------------------------------------------
// One CTA per token, any sizes: key tiles of KT positions aligned to absolute multiples of KT, online softmax over the
// tiles, so that a token's result depends on (lo, p) only.
constexpr int KT = 64;
constexpr int PLAIN_THREADS = 128;

template <typename T>
__global__ void __launch_bounds__(PLAIN_THREADS)
talk_attention_kernel(const T* __restrict__ q, int64_t ldq, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                      const int* __restrict__ block_table, int64_t max_blocks, const int* __restrict__ token_seg,
                      const int* __restrict__ positions, T* __restrict__ out, int H, int n_kv, int d, int dv, int page_size,
                      int window, int chunk, float scale, float cap, const float* __restrict__ talk, int64_t n_pages, int* status) {
    ib::pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int64_t t = blockIdx.x;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int group = H / n_kv;
    int64_t* rowoff = reinterpret_cast<int64_t*>(sm);        // [KT]; -1: not visible
    float* qs = reinterpret_cast<float*>(rowoff + KT);       // [H][d]
    float* raw = qs + H * d;                                 // [H][KT]
    float* mixed = raw + H * KT;                             // [H][KT]
    float* acc = mixed + H * KT;                             // [H][dv]
    float* ml = acc + H * dv;                                // [H][3] running maximum, sum, correction
    const int pos = positions[t];
    const int lo = first_visible(pos, window, chunk);
    const int* table = block_table + int64_t(token_seg[t]) * max_blocks;
    for (int i = tid; i < H * d; i += PLAIN_THREADS) qs[i] = ib::to_f32(q[t * ldq + i]);
    for (int i = tid; i < H * dv; i += PLAIN_THREADS) acc[i] = 0.0f;
    for (int i = tid; i < H; i += PLAIN_THREADS) { ml[3 * i] = -INFINITY; ml[3 * i + 1] = 0.0f; }
    for (int tile = lo / KT * KT; tile <= pos; tile += KT) {
        __syncthreads();
        for (int j = tid; j < KT; j += PLAIN_THREADS) {
            const int key = tile + j;
            int64_t row = -1;
            if (key >= lo && key <= pos) {
                const int page = table[key / page_size];
                if (page < 0 || page >= n_pages) { if (status) atomicExch(status, 3); }
                else row = int64_t(page) * n_kv * page_size + key % page_size;
            }
            rowoff[j] = row;
        }
        __syncthreads();
        for (int i = tid; i < H * KT; i += PLAIN_THREADS) {
            const int h = i / KT, j = i - h * KT;
            float s = 0.0f;
            if (rowoff[j] >= 0) {
                const T* kr = k_cache + (rowoff[j] + int64_t(h / group) * page_size) * d;
                const float* qh = qs + h * d;
                for (int e = 0; e < d; e++) s = fmaf(qh[e], ib::to_f32(kr[e]), s);
                s *= scale;
                if (cap > 0.0f) s = cap * tanhf(s / cap);
            }
            raw[i] = s;
        }
        __syncthreads();
        for (int i = tid; i < H * KT; i += PLAIN_THREADS) {
            const int h = i / KT, j = i - h * KT;
            float s = raw[i];
            if (talk) {
                s = 0.0f;
                for (int g = 0; g < H; g++) s = fmaf(talk[h * H + g], raw[g * KT + j], s);
            }
            mixed[i] = rowoff[j] >= 0 ? s : -INFINITY;
        }
        __syncthreads();
        for (int h = warp; h < H; h += PLAIN_THREADS / 32) {
            float* row = mixed + h * KT;
            float mx = -INFINITY;
            for (int j = lane; j < KT; j += 32) mx = fmaxf(mx, row[j]);
            mx = ib::warp_max(mx);
            const float m_old = ml[3 * h], m_new = fmaxf(m_old, mx);
            float sum = 0.0f;
            for (int j = lane; j < KT; j += 32) {
                const float pv = row[j] > -INFINITY ? expf(row[j] - m_new) : 0.0f;
                row[j] = pv;
                sum += pv;
            }
            sum = ib::warp_sum(sum);
            const float corr = m_old > -INFINITY ? expf(m_old - m_new) : 0.0f;
            __syncwarp();
            if (lane == 0) {
                ml[3 * h] = m_new;
                ml[3 * h + 1] = ml[3 * h + 1] * corr + sum;
                ml[3 * h + 2] = corr;
            }
        }
        __syncthreads();
        const int j0 = max(lo, tile) - tile, j1 = min(pos, tile + KT - 1) - tile;
        for (int i = tid; i < H * dv; i += PLAIN_THREADS) {
            const int h = i / dv, c = i - h * dv;
            float a = acc[i] * ml[3 * h + 2];
            for (int j = j0; j <= j1; j++) {
                if (rowoff[j] < 0) continue;
                a = fmaf(mixed[h * KT + j], ib::to_f32(v_cache[(rowoff[j] + int64_t(h / group) * page_size) * dv + c]), a);
            }
            acc[i] = a;
        }
    }
    __syncthreads();
    for (int i = tid; i < H * dv; i += PLAIN_THREADS) {
        const float l = ml[3 * (i / dv) + 1];
        out[t * int64_t(H) * dv + i] = ib::from_f32<T>(l > 0.0f ? acc[i] / l : 0.0f);
    }
}

// ------------------------------------------------------------------------------------------------
// Single tokens in bfloat16: one CTA per (token, chunk of KC keys aligned to absolute multiples of KC), all heads. Each
// key and value row is read once for all query heads of its kv head.
//   scores    a warp per (page of 16 keys, kv head): the page's keys are the rows and the group's queries the columns of
//             m16n8k16 tiles. A lane reads 16 bytes of a key row and of a query; which k of the tile an element takes is
//             the same permutation for both operands, so that no operand passes through shared memory
//   exchange  a thread per (key, quarter of the heads)
//   softmax   a warp per head, over the chunk
//   values    a thread per (kv head, 8 channels, share of the keys): its first 8 value rows are requested before the
//             scores are computed; the shares are added through shared memory in ascending order
// A chunk leaves (maximum, sum, unnormalised context) per head; the merge kernel adds a token's chunks in ascending order.
// With `fresh` rows the token's own key and value are taken from them (columns k_col, v_col) and stored to its page, so
// that a step of single tokens needs no store kernel; the chunk that holds the token's position does it.
// `single_only` (a step's seg_start): tokens of longer segments are another kernel's.
constexpr int KC = 64;
constexpr int SPLIT_THREADS = 256;
constexpr int SPLIT_WARPS = SPLIT_THREADS / 32;
constexpr int SST = KC + 8;                  // row stride of the score arrays
constexpr int PAGE = 16;
constexpr int VB = 8;                        // value rows in flight per thread
constexpr int GROUP_MAX = 16;

__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct SplitArgs {
    const bf16* q; int64_t ldq;
    const bf16* k_cache; const bf16* v_cache;
    bf16* k_store; bf16* v_store;            // the same pages, for `fresh`
    const bf16* fresh; int64_t ldf; int k_col, v_col;
    const int* block_table; int64_t max_blocks;
    const int* token_seg; const int* positions; const int* single_only;
    float* parts;
    int H, n_kv, d, dv, window, chunk, n_chunks, n_share;
    float scale, cap;
    const float* talk;
    int64_t n_pages;
    int* status;
};

// GB: the group's size rounded up to 1, 2, 4, 8 or 16.
template <int GB>
__global__ void __launch_bounds__(SPLIT_THREADS)
talk_split_kernel(const SplitArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int H = a.H, group = H / a.n_kv, d = a.d, dv = a.dv;
    float* raw = sm;                                         // [H][SST]
    float* mixed = raw + H * SST;                            // [H][SST]
    float* T_s = mixed + H * SST;                            // [H][H], transposed: T_s[g][h]
    float* red = sm + ((2 * H * SST + H * H + 3) & ~3);      // [n_share - 1][H][dv]
    __shared__ int64_t rowoff[KC];                           // row of a key's kv head 0 in the pages; -1: not visible, -2: fresh
    __shared__ float ml[2 * 128];
    if (a.talk)
        for (int i = tid; i < H * H; i += SPLIT_THREADS) T_s[(i % H) * H + i / H] = a.talk[i];      // (a weight)
    ib::pdl_wait();
    const int64_t t = blockIdx.x;
    const int ci = blockIdx.y;
    const int sg = a.token_seg[t];
    if (a.single_only && a.single_only[sg + 1] - a.single_only[sg] > 1) return;
    const int pos = a.positions[t];
    const int lo = first_visible(pos, a.window, a.chunk);
    const int base = (lo / KC + ci) * KC;
    if (base > pos) return;
    const int* table = a.block_table + int64_t(sg) * a.max_blocks;
    for (int j = tid; j < KC; j += SPLIT_THREADS) {
        const int key = base + j;
        int64_t row = -1;
        if (key >= lo && key <= pos) {
            const int page = table[key / PAGE];
            if (page < 0 || page >= a.n_pages) { if (a.status) atomicExch(a.status, 3); }
            else row = int64_t(page) * a.n_kv * PAGE + key % PAGE;
            if (row >= 0 && a.fresh && key == pos) row = -2 - row;       // (the row itself is -2 - value)
        }
        rowoff[j] = row;
    }
    __syncthreads();
    const bf16* fresh_k = a.fresh ? a.fresh + t * a.ldf + a.k_col : nullptr;
    const bf16* fresh_v = a.fresh ? a.fresh + t * a.ldf + a.v_col : nullptr;
    auto key_row = [&](int j, int g) -> const bf16* {        // null: nothing visible there
        const int64_t r = rowoff[j];
        if (r == -1) return nullptr;
        return r < -1 ? fresh_k + g * d : a.k_cache + (r + int64_t(g) * PAGE) * d;
    };
    auto value_row = [&](int j, int g) -> const bf16* {
        const int64_t r = rowoff[j];
        if (r == -1) return nullptr;
        return r < -1 ? fresh_v + g * dv : a.v_cache + (r + int64_t(g) * PAGE) * dv;
    };
    // values: this thread's place, and its first rows on their way
    const int units = a.n_kv * (dv / 8);
    const int share = tid / units, unit = tid - share * units;
    const bool has_v = share < a.n_share;
    const int vg = unit / (dv / 8), vc = (unit - vg * (dv / 8)) * 8;
    const int per_share = KC / a.n_share, js0 = share * per_share;
    uint4 vrow[VB];
    auto load_values = [&](int j0) {
#pragma unroll
        for (int i = 0; i < VB; i++) {
            vrow[i] = make_uint4(0u, 0u, 0u, 0u);
            if (has_v && i < per_share) {
                const bf16* v = value_row(j0 + i, vg);
                if (v) vrow[i] = *reinterpret_cast<const uint4*>(v + vc);
            }
        }
    };
    load_values(js0);
    // scores
    const int n_units = (KC / PAGE) * a.n_kv, r8 = lane >> 2, c4 = lane & 3;
    for (int u = warp; u < n_units; u += SPLIT_WARPS) {
        const int pg = u / a.n_kv, g = u - pg * a.n_kv;
        const bf16* k0 = key_row(pg * PAGE + r8, g);
        const bf16* k1 = key_row(pg * PAGE + r8 + 8, g);
        float acc[(GB + 7) / 8][4];
#pragma unroll
        for (int n = 0; n < (GB + 7) / 8; n++)
#pragma unroll
            for (int e = 0; e < 4; e++) acc[n][e] = 0.0f;
        for (int kb = 0; kb < d; kb += 64) {
            uint4 x0[2], x1[2], y[(GB + 7) / 8][2];
#pragma unroll
            for (int b = 0; b < 2; b++) {
                const int e = kb + b * 32 + c4 * 8;
                const bool in = kb + b * 32 < d;
                x0[b] = in && k0 ? *reinterpret_cast<const uint4*>(k0 + e) : make_uint4(0u, 0u, 0u, 0u);
                x1[b] = in && k1 ? *reinterpret_cast<const uint4*>(k1 + e) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
                for (int n = 0; n < (GB + 7) / 8; n++) {
                    const int hq = n * 8 + r8;
                    y[n][b] = in && hq < group ? *reinterpret_cast<const uint4*>(a.q + t * a.ldq + (g * group + hq) * d + e)
                                               : make_uint4(0u, 0u, 0u, 0u);
                }
            }
#pragma unroll
            for (int b = 0; b < 2; b++) {
                const uint32_t a0[4] = {x0[b].x, x1[b].x, x0[b].y, x1[b].y}, a1[4] = {x0[b].z, x1[b].z, x0[b].w, x1[b].w};
#pragma unroll
                for (int n = 0; n < (GB + 7) / 8; n++) {
                    mma_16816(acc[n], a0, y[n][b].x, y[n][b].y);
                    mma_16816(acc[n], a1, y[n][b].z, y[n][b].w);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < (GB + 7) / 8; n++) {
#pragma unroll
            for (int e = 0; e < 4; e++) {
                const int hq = n * 8 + c4 * 2 + (e & 1), j = pg * PAGE + r8 + (e >> 1) * 8;
                if (hq < group) {
                    float s = acc[n][e] * a.scale;
                    if (a.cap > 0.0f) s = a.cap * tanhf(s / a.cap);
                    raw[(g * group + hq) * SST + j] = s;
                }
            }
        }
    }
    __syncthreads();
    // the exchange among the heads: four threads a key, each a quarter of the heads
    {
        const int j = tid & (KC - 1), part = tid / KC, per = (H + 3) / 4;
        const int h0 = part * per, h1 = min(H, h0 + per);
        const bool seen = rowoff[j] != -1;
        for (int hb = h0; hb < h1; hb += 8) {
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; e++) o[e] = 0.0f;
            if (a.talk) {
                for (int g = 0; g < H; g++) {
                    const float s = raw[g * SST + j];
#pragma unroll
                    for (int e = 0; e < 8; e++)
                        if (hb + e < h1) o[e] = fmaf(T_s[g * H + hb + e], s, o[e]);
                }
            } else {
#pragma unroll
                for (int e = 0; e < 8; e++)
                    if (hb + e < h1) o[e] = raw[(hb + e) * SST + j];
            }
#pragma unroll
            for (int e = 0; e < 8; e++)
                if (hb + e < h1) mixed[(hb + e) * SST + j] = seen ? o[e] : -INFINITY;
        }
    }
    __syncthreads();
    for (int h = warp; h < H; h += SPLIT_WARPS) {
        float* row = mixed + h * SST;
        const float s0 = row[lane], s1 = row[lane + 32];
        const float m = ib::warp_max(fmaxf(s0, s1));
        const float p0 = s0 > -INFINITY ? expf(s0 - m) : 0.0f, p1 = s1 > -INFINITY ? expf(s1 - m) : 0.0f;
        row[lane] = p0;
        row[lane + 32] = p1;
        const float l = ib::warp_sum(p0 + p1);
        if (lane == 0) { ml[2 * h] = m; ml[2 * h + 1] = l; }
    }
    __syncthreads();
    // values
    float o[GB][8];
#pragma unroll
    for (int q = 0; q < GB; q++)
#pragma unroll
        for (int e = 0; e < 8; e++) o[q][e] = 0.0f;
    if (has_v) {
        for (int jb = 0; jb < per_share; jb += VB) {
            if (jb > 0) load_values(js0 + jb);
#pragma unroll
            for (int i = 0; i < VB; i++) {
                if (i >= per_share) break;
                float v[8];
                const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&vrow[i]);
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float2 f = __bfloat1622float2(h2[e]);
                    v[2 * e] = f.x;
                    v[2 * e + 1] = f.y;
                }
#pragma unroll
                for (int q = 0; q < GB; q++) {
                    if (q < group) {
                        const float p = mixed[(vg * group + q) * SST + js0 + jb + i];
#pragma unroll
                        for (int e = 0; e < 8; e++) o[q][e] = fmaf(p, v[e], o[q][e]);
                    }
                }
            }
        }
        if (share > 0) {
#pragma unroll
            for (int q = 0; q < GB; q++) {
                if (q < group) {
                    float4* dst = reinterpret_cast<float4*>(red + (int64_t(share - 1) * H + vg * group + q) * dv + vc);
                    dst[0] = make_float4(o[q][0], o[q][1], o[q][2], o[q][3]);
                    dst[1] = make_float4(o[q][4], o[q][5], o[q][6], o[q][7]);
                }
            }
        }
    }
    __syncthreads();
    const int64_t stride = dv + 2;
    float* mine = a.parts + (t * H * a.n_chunks + ci) * stride;          // head h: + h * n_chunks * stride
    if (has_v && share == 0) {
#pragma unroll
        for (int q = 0; q < GB; q++) {
            if (q < group) {
                const int h = vg * group + q;
                for (int s = 0; s + 1 < a.n_share; s++) {
                    const float4* src = reinterpret_cast<const float4*>(red + (int64_t(s) * H + h) * dv + vc);
                    const float4 x = src[0], y = src[1];
                    o[q][0] += x.x; o[q][1] += x.y; o[q][2] += x.z; o[q][3] += x.w;
                    o[q][4] += y.x; o[q][5] += y.y; o[q][6] += y.z; o[q][7] += y.w;
                }
                float2* dst = reinterpret_cast<float2*>(mine + int64_t(h) * a.n_chunks * stride + 2 + vc);
#pragma unroll
                for (int e = 0; e < 4; e++) dst[e] = make_float2(o[q][2 * e], o[q][2 * e + 1]);
            }
        }
    }
    for (int h = tid; h < H; h += SPLIT_THREADS) {
        mine[int64_t(h) * a.n_chunks * stride] = ml[2 * h];
        mine[int64_t(h) * a.n_chunks * stride + 1] = ml[2 * h + 1];
    }
    if (a.fresh && pos < base + KC) {                        // this chunk holds the token's own position
        const int64_t r = -2 - rowoff[pos - base];
        if (r >= 0) {
            for (int i = tid; i < a.n_kv * (d / 8); i += SPLIT_THREADS) {
                const int g = i / (d / 8), c = (i - g * (d / 8)) * 8;
                *reinterpret_cast<uint4*>(a.k_store + (r + int64_t(g) * PAGE) * d + c) = *reinterpret_cast<const uint4*>(fresh_k + g * d + c);
            }
            for (int i = tid; i < a.n_kv * (dv / 8); i += SPLIT_THREADS) {
                const int g = i / (dv / 8), c = (i - g * (dv / 8)) * 8;
                *reinterpret_cast<uint4*>(a.v_store + (r + int64_t(g) * PAGE) * dv + c) = *reinterpret_cast<const uint4*>(fresh_v + g * dv + c);
            }
        }
    }
}

// One CTA per (token, head), a thread per channel: the chunks' parts in ascending order, then the division.
constexpr int MERGE_THREADS = 128;
constexpr int MERGE_WEIGHTS = 1024;          // chunks whose weights are kept (65,536 keys; beyond that they are computed again)
__global__ void __launch_bounds__(MERGE_THREADS)
talk_merge_kernel(const float* __restrict__ parts, const int* __restrict__ token_seg, const int* __restrict__ positions,
                  const int* __restrict__ single_only, bf16* __restrict__ out, int H, int dv, int window, int chunk, int n_chunks) {
    ib::pdl_wait();
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int sg = token_seg[t];
    if (single_only && single_only[sg + 1] - single_only[sg] > 1) return;
    const int pos = positions[t];
    const int lo = first_visible(pos, window, chunk);
    const int n = min(n_chunks, pos / KC - lo / KC + 1);
    const int64_t stride = dv + 2;
    const float* mine = parts + (t * H + h) * n_chunks * stride;
    // every warp finds the maximum and the sum for itself; the chunks' weights go through shared memory
    __shared__ float weight[MERGE_WEIGHTS];
    float m = -INFINITY;
    for (int i = lane; i < n; i += 32) m = fmaxf(m, mine[i * stride]);
    m = ib::warp_max(m);
    float l = 0.0f;
    for (int i = lane; i < n; i += 32) {
        const float mi = mine[i * stride], w = mi > -INFINITY ? expf(mi - m) : 0.0f;
        l += mine[i * stride + 1] * w;
        if (tid < 32 && i < MERGE_WEIGHTS) weight[i] = w;
    }
    l = ib::warp_sum(l);
    const float inv = l > 0.0f ? 1.0f / l : 0.0f;
    __syncthreads();
    for (int c = tid; c < dv; c += MERGE_THREADS) {
        float acc = 0.0f;
        const float* col = mine + 2 + c;
        const int n_s = min(n, MERGE_WEIGHTS);
#pragma unroll 16
        for (int i = 0; i < n_s; i++) acc = fmaf(col[i * stride], weight[i], acc);
        for (int i = n_s; i < n; i++) acc = fmaf(col[i * stride], mine[i * stride] > -INFINITY ? expf(mine[i * stride] - m) : 0.0f, acc);
        out[(t * H + h) * dv + c] = __float2bfloat16_rn(acc * inv);
    }
}

// Shares of a chunk's keys among the threads of the value phase: as many as there are threads for, a power of two.
int split_shares(int n_kv, int dv) {
    const int units = n_kv * (dv / 8);
    int n = 1;
    while (n < 8 && 2 * n * units <= SPLIT_THREADS) n *= 2;
    return n;
}
size_t split_smem(int H, int n_kv, int dv) {
    return (size_t((2 * H * SST + H * H + 3) & ~3) + size_t(split_shares(n_kv, dv) - 1) * H * dv) * sizeof(float);
}

size_t plain_smem(int H, int d, int dv) { return KT * sizeof(int64_t) + (size_t(H) * d + 2 * size_t(H) * KT + size_t(H) * dv + 3 * H) * sizeof(float); }

}  // namespace

// ================================================================================================
// C entry points. dtype arguments: 0 = float, 1 = bfloat16.

IB_EXPORT int ib_kv_store(const void* rows, int64_t ld, int k_col, int v_col, const int* positions, const int* token_seg,
                          const int* block_table, int64_t max_blocks, void* k_cache, void* v_cache, int64_t n_tokens, int n_kv, int d,
                          int dv, int page_size, int64_t n_pages, int dtype, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return IB_OK;
    if (n_kv <= 0 || d <= 0 || dv <= 0 || page_size <= 0) return ib::fail(IB_ERR_ARG, "ib_kv_store: bad sizes");
    const int64_t n = n_tokens * n_kv * (d + dv);
#define IB_KV(TT, PT)                                                                                                               \
    IB_LAUNCH((kv_store_kernel<TT, PT>), blocks_for(n / PT, 256), 256, 0, (const TT*)rows, ld, k_col, v_col, positions, token_seg,  \
              block_table, max_blocks, (TT*)k_cache, (TT*)v_cache, n_tokens, n_kv, d, dv, page_size, n_pages, status)
    if (dtype == IB_F32) IB_KV(float, 1);
    else if (dtype == IB_BF16 && d % 8 == 0 && dv % 8 == 0 && ld % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 &&
             !((uintptr_t(rows) | uintptr_t(k_cache) | uintptr_t(v_cache)) & 15)) IB_KV(bf16, 8);
    else if (dtype == IB_BF16) IB_KV(bf16, 1);
    else return ib::fail(IB_ERR_ARG, "ib_kv_store: unknown dtype %d", dtype);
#undef IB_KV
    return ib::check_launch("ib_kv_store");
}

// 1 if the kernels of this library hold all heads of these sizes in a CTA's shared memory.
IB_EXPORT int ib_talk_attention_fits(int n_heads, int d, int dv) { return plain_smem(n_heads, d, dv) <= 220 * 1024; }

// 1 if ib_talk_attention_split takes these sizes (bfloat16, pages of 16 positions).
IB_EXPORT int ib_talk_split_fits(int n_heads, int n_kv, int d, int dv, int page_size) {
    if (n_kv <= 0 || n_heads % n_kv) return 0;
    return page_size == PAGE && d % 32 == 0 && dv % 8 == 0 && n_heads <= 128 && n_heads / n_kv <= GROUP_MAX &&
           n_kv * (dv / 8) <= SPLIT_THREADS && split_smem(n_heads, n_kv, dv) <= 200 * 1024;
}

// Chunks of a token whose queries see up to `visible` keys, and the floats of workspace for n_tokens such tokens.
IB_EXPORT int ib_talk_split_chunks(int visible) { return (visible + KC - 1) / KC + 1; }

// Single tokens (with single_only: only those that are a segment of their own). fresh: rows whose columns k_col and
// v_col hold the tokens' own keys and values, not yet stored (every token must be the last of its request then), or
// null; n_chunks as ib_talk_split_chunks; workspace: n_tokens * n_heads * n_chunks * (dv + 2) floats.
IB_EXPORT int ib_talk_attention_split(const void* q, int64_t ldq, const void* fresh, int64_t ldf, int k_col, int v_col, void* k_cache,
                                      void* v_cache, const int* block_table, int64_t max_blocks, const int* token_seg,
                                      const int* positions, const int* single_only, void* out, float* workspace, int64_t n_tokens,
                                      int n_heads, int n_kv, int d, int dv, int page_size, int window, int chunk, int n_chunks, float scale,
                                      float cap, const float* talk, int64_t n_pages, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return IB_OK;
    if (!ib_talk_split_fits(n_heads, n_kv, d, dv, page_size))
        return ib::fail(IB_ERR_ARG, "ib_talk_attention_split: %d heads on %d kv heads of %d / %d, pages of %d", n_heads, n_kv, d, dv, page_size);
    if (n_chunks < 1 || n_chunks > 65535 || !workspace) return ib::fail(IB_ERR_ARG, "ib_talk_attention_split: %d chunks", n_chunks);
    if (ldq % 8 || (uintptr_t(q) | uintptr_t(k_cache) | uintptr_t(v_cache)) & 15 || (fresh && (ldf % 8 || k_col % 8 || v_col % 8 || uintptr_t(fresh) & 15)))
        return ib::fail(IB_ERR_ARG, "ib_talk_attention_split: rows must be whole 16-byte pieces");
    SplitArgs a = {};
    a.q = (const bf16*)q; a.ldq = ldq;
    a.k_cache = a.k_store = (bf16*)k_cache; a.v_cache = a.v_store = (bf16*)v_cache;
    a.fresh = (const bf16*)fresh; a.ldf = ldf; a.k_col = k_col; a.v_col = v_col;
    a.block_table = block_table; a.max_blocks = max_blocks; a.token_seg = token_seg; a.positions = positions; a.single_only = single_only;
    a.parts = workspace; a.H = n_heads; a.n_kv = n_kv; a.d = d; a.dv = dv; a.window = window; a.chunk = chunk; a.n_chunks = n_chunks;
    a.n_share = split_shares(n_kv, dv); a.scale = scale; a.cap = cap; a.talk = talk; a.n_pages = n_pages; a.status = status;
    const size_t smem = split_smem(n_heads, n_kv, dv);
    const dim3 grid{unsigned(n_tokens), unsigned(n_chunks), 1u};
    const int group = n_heads / n_kv;
#define IB_SPLIT(GG)                                                                                                                          do {                                                                                                                                          if (smem > 40 * 1024) {                                                                                                                       cudaError_t e = cudaFuncSetAttribute(talk_split_kernel<GG>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));                      if (e != cudaSuccess) return ib::fail(IB_ERR_CUDA, "ib_talk_attention_split: cannot set shared memory size: %s", cudaGetErrorString(e));         }                                                                                                                                         IB_LAUNCH(talk_split_kernel<GG>, grid, SPLIT_THREADS, smem, a);                                                                       } while (0)
    if (group <= 1) IB_SPLIT(1);
    else if (group <= 2) IB_SPLIT(2);
    else if (group <= 4) IB_SPLIT(4);
    else if (group <= 8) IB_SPLIT(8);
    else IB_SPLIT(16);
#undef IB_SPLIT
    const dim3 mgrid{unsigned(n_tokens), unsigned(n_heads), 1u};
    IB_LAUNCH(talk_merge_kernel, mgrid, MERGE_THREADS, 0, workspace, token_seg, positions, single_only, (bf16*)out, n_heads, dv, window, chunk,
              n_chunks);
    return ib::check_launch("ib_talk_attention_split");
}

// q: rows of leading dimension ldq, the heads' queries from column 0; out [tokens, heads * dv].
IB_EXPORT int ib_talk_attention(const void* q, int64_t ldq, const void* k_cache, const void* v_cache, const int* block_table,
                                int64_t max_blocks, const int* token_seg, const int* positions, void* out, int64_t n_tokens,
                                int n_heads, int n_kv, int d, int dv, int page_size, int window, int chunk, float scale, float cap,
                                const float* talk, int64_t n_pages, int dtype, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return IB_OK;
    if (n_heads <= 0 || n_kv <= 0 || n_heads % n_kv || d <= 0 || dv <= 0 || page_size <= 0)
        return ib::fail(IB_ERR_ARG, "ib_talk_attention: %d heads on %d kv heads of %d / %d", n_heads, n_kv, d, dv);
    const size_t smem = plain_smem(n_heads, d, dv);
    if (smem > 220 * 1024) return ib::fail(IB_ERR_ARG, "ib_talk_attention: %d heads of %d / %d do not fit", n_heads, d, dv);
#define IB_TALK(TT)                                                                                                                  \
    do {                                                                                                                             \
        if (smem > 48 * 1024) {                                                                                                      \
            cudaError_t e = cudaFuncSetAttribute(talk_attention_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)); \
            if (e != cudaSuccess) return ib::fail(IB_ERR_CUDA, "ib_talk_attention: cannot set shared memory size: %s", cudaGetErrorString(e)); \
        }                                                                                                                            \
        IB_LAUNCH(talk_attention_kernel<TT>, unsigned(n_tokens), PLAIN_THREADS, smem, (const TT*)q, ldq, (const TT*)k_cache,         \
                  (const TT*)v_cache, block_table, max_blocks, token_seg, positions, (TT*)out, n_heads, n_kv, d, dv, page_size,      \
                  window, chunk, scale, cap, talk, n_pages, status);                                                                 \
    } while (0)
    if (dtype == IB_F32) IB_TALK(float);
    else if (dtype == IB_BF16) IB_TALK(bf16);
    else return ib::fail(IB_ERR_ARG, "ib_talk_attention: unknown dtype %d", dtype);
#undef IB_TALK
    return ib::check_launch("ib_talk_attention");
}
