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
