// Attention whose heads exchange their scores before the softmax (talk_ops.cu), for prompt portions on the 5th-generation
// tensor cores over the paged bfloat16 cache. Compiled for one set of sizes: -DIB_HEAD_DIM (keys: 64 or 128),
// -DIB_V_DIM (values: 64 or 128), -DIB_HEADS (up to 32).
//
// A head's score of a (query, key) pair needs every head's score of that pair, and a softmax row needs every key: the two
// do not fit one tile order, so there are two kernels with the exchanged scores (float) in memory between them, a tile
// of 128 queries x 128 keys and a head at a time.
//
// Kernel 1 (scores): one CTA per (query tile, key tile, share of the query tile). The keys of all kv heads are loaded
// once (TMA, a page of 16 keys per lane, 128-byte swizzle) and are the ROWS of the products, S^T = K Q^T; the queries of 16
// positions, all heads, are the columns: 16 columns of tensor memory per head, all heads side by side, so that the
// thread that owns a key reads every head's score of its (query, key) pairs with no exchange between threads:
//   warp 0      TMA producer: the key tile, then the queries through a ring (a kv head's group of heads per stage)
//   warp 1      MMA issuer: the heads of a kv head in one product (a product of few columns costs the tensor core
//               as much as one of a hundred), the blocks of 16 queries in two tensor-memory buffers where they fit
//   the others  thread = (key, share of the block's queries): scale and cap, then score_h = sum_g talk[h, g] score_g for four
//               queries at a time in packed float pairs, and a 16-byte store per head (a warp: 512 bytes)
// Kernel 2 (softmax and values): one CTA per (query tile, head), the softmax and P V of the engine's prompt attention
// (attention_tc.cu) with the scores copied in by bulk copies instead of computed. It masks; kernel 1 writes whatever
// its blocks give (keys that are not visible, rows past the portion), and blocks it skips are masked altogether.
//
// Score tiles: [query / 4 (32)][key (128)][query % 4 (4)] floats. Kernel 2 copies the 32 pieces of 2 KB to rows 16 bytes
// further apart, so that the lanes of a warp (neighbouring queries) read from different banks.
//
// Every mbarrier wait is bounded; one that runs out raises the status word, and the CTA drains its copies, frees its
// tensor memory and returns.
#include <algorithm>

#include "common.cuh"
#include "tc_ops.cuh"
#include "tma_map.cuh"

IB_DEFINE_LAST_ERROR()

#ifndef IB_HEAD_DIM
#define IB_HEAD_DIM 128
#endif
#ifndef IB_V_DIM
#define IB_V_DIM 128
#endif
#ifndef IB_HEADS
#define IB_HEADS 12
#endif

namespace {

using bf16 = __nv_bfloat16;
using namespace ib::tc;
constexpr int D = IB_HEAD_DIM, DV = IB_V_DIM, H = IB_HEADS;
static_assert((D == 64 || D == 128) && (DV == 64 || DV == 128) && H >= 1 && H <= 32, "key and value sizes of 64 or 128, up to 32 heads");
constexpr int DB = D / 64, DVB = DV / 64;   // 64-element (128-byte) blocks
constexpr int PAGE = 16, BN = 128, BM = 128;
constexpr int PAGES_PER_TILE = BN / PAGE;
constexpr int TILE_FLOATS = BM * BN;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int STATUS_TIMEOUT = 107, STATUS_BAD_PAGE = 3;

__device__ __forceinline__ int first_visible(int pos, int window, int chunk) {
    int lo = window > 0 ? max(0, pos - window + 1) : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    return lo;
}
__device__ __forceinline__ float fast_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void tmem_ld4(uint32_t taddr, float* r) {
    uint32_t* u = reinterpret_cast<uint32_t*>(r);
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(u[0]), "=r"(u[1]), "=r"(u[2]), "=r"(u[3]) : "r"(taddr) : "memory");
}
__device__ __forceinline__ uint64_t pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
    return f;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// What a (segment, query tile) of the launch is; false: nothing to do there.
struct Tile {
    int t0, q_len, pos0, q_first, q_last, last_written, kt0, kt1, slot;
};
struct Params {
    const int* block_table; int max_blocks;
    const int* seg_start; const int* seg_pos0;
    int n_kv, window, chunk;
    int64_t n_pages;
    int* status;
    float* scores;                           // [slot = (rank of the long segment, query tile of this launch)][H][max_tiles][TILE_FLOATS]
    int max_tiles, qt0, n_qt;                // key tiles a query tile has room for; this launch's query tiles
    // kernel 1
    float scale, cap;
    const float* talk;                       // [H][H] or null
    int q_col, n_stages, q_split;
    // kernel 2
    bf16* out;                               // [tokens, H * DV]
};

__device__ __forceinline__ bool tile_of(const Params& p, int seg, int qt, Tile& w) {
    w.t0 = p.seg_start[seg];
    w.q_len = p.seg_start[seg + 1] - w.t0;
    if (w.q_len <= 1 || qt * BM >= w.q_len) return false;    // one-token segments belong to another kernel
    w.pos0 = p.seg_pos0[seg];
    w.q_first = w.pos0 + qt * BM;
    w.last_written = w.pos0 + w.q_len - 1;
    w.q_last = min(w.last_written, w.q_first + BM - 1);
    w.kt0 = first_visible(w.q_first, p.window, p.chunk) / BN;
    w.kt1 = w.q_last / BN;
    int before = 0;
    for (int s = 0; s < seg; s++) before += (p.seg_start[s + 1] - p.seg_start[s] > 1) ? 1 : 0;
    w.slot = before * p.n_qt + (qt - p.qt0);
    return w.kt1 - w.kt0 < p.max_tiles;                      // (the host makes room for the most a tile can have)
}

__device__ __forceinline__ int page_at(const Params& p, int seg, int key) {
    const int idx = key / PAGE;
    if (idx >= p.max_blocks) return -1;
    const int page = p.block_table[int64_t(seg) * p.max_blocks + idx];
    return (page < 0 || page >= p.n_pages) ? -1 : page;
}

// ------------------------------------------------------------------------------------------------ kernel 1
constexpr int NQ = 16;                       // queries of a block
constexpr int BLOCKS = BM / NQ;
constexpr int MIX_WARPS = H <= 16 ? 16 : 8;   // (by the registers that H scores of four queries take)
constexpr int Q_SHARES = MIX_WARPS / 4;      // warps that own the same keys share a block's queries
constexpr int PASSES = NQ / 4 / Q_SHARES;    // of four queries each
constexpr int SCORE_THREADS = 64 + MIX_WARPS * 32;
constexpr int S_BUFS = 2 * H * NQ <= 512 ? 2 : 1;
constexpr int s_cols(int need) { return need <= 32 ? 32 : (need <= 64 ? 64 : (need <= 128 ? 128 : (need <= 256 ? 256 : 512))); }
constexpr int S_TMEM = s_cols(S_BUFS * H * NQ);
constexpr int HP = (H + 3) & ~3;             // heads rounded up to a multiple of four
constexpr int MAX_STAGES = 4;
constexpr int K_HEAD_BYTES = DB * BN * 128;  // one kv head's key tile
constexpr int Q_HEAD_BYTES = DB * NQ * 128;  // one head's queries of a block
constexpr int SCORE_FIXED = H * HP * 4 + 1024 + 256;

__global__ void __launch_bounds__(SCORE_THREADS)
talk_scores_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k, const Params p) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
    const int group = H / p.n_kv, stage_bytes = group * Q_HEAD_BYTES;
    const uint32_t k_s = base, q_s = k_s + p.n_kv * K_HEAD_BYTES;
    uint8_t* tail = base_ptr + p.n_kv * K_HEAD_BYTES + p.n_stages * stage_bytes;
    float* T_s = reinterpret_cast<float*>(tail);             // [H][HP] the exchange matrix
    const uint32_t bars = base + uint32_t(tail - base_ptr) + H * HP * 4;
    volatile uint32_t* slots = reinterpret_cast<volatile uint32_t*>(tail + H * HP * 4 + 128);    // [0] TMEM base, [1] abort
    const uint32_t k_full = bars, q_full = bars + 8, q_empty = q_full + 8 * MAX_STAGES, s_full = q_empty + 8 * MAX_STAGES,
                   s_empty = s_full + 16;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seg = blockIdx.z, qt = p.qt0 + int(blockIdx.y) / p.q_split, part = int(blockIdx.y) % p.q_split;
    Tile w;
    if (!tile_of(p, seg, qt, w)) return;
    const int kt = w.kt0 + int(blockIdx.x);
    if (kt > w.kt1) return;
    const int key0 = kt * BN;
    // this CTA's blocks of NQ queries: those of its share that see a key of the tile (a contiguous run)
    int b0 = BLOCKS, b1 = -1;
    for (int b = part * (BLOCKS / p.q_split); b < (part + 1) * (BLOCKS / p.q_split); b++) {
        const int first = w.q_first + b * NQ, last = min(w.last_written, first + NQ - 1);
        if (first <= w.last_written && key0 <= last && key0 + BN - 1 >= first_visible(first, p.window, p.chunk)) {
            b0 = min(b0, b);
            b1 = b;
        }
    }
    if (b1 < b0) return;
    const int lo_key = first_visible(w.q_first, p.window, p.chunk);
    if (p.talk) {
        for (int i = threadIdx.x; i < H * HP; i += SCORE_THREADS) {
            const int h = i / HP, g = i - h * HP;
            T_s[i] = g < H ? p.talk[h * H + g] : 0.0f;
        }
    }
    if (threadIdx.x == 0) {
        mbar_init(k_full, 1);
        for (int i = 0; i < MAX_STAGES; i++) { mbar_init(q_full + 8 * i, 1); mbar_init(q_empty + 8 * i, 1); }
        for (int i = 0; i < 2; i++) { mbar_init(s_full + 8 * i, 1); mbar_init(s_empty + 8 * i, MIX_WARPS); }
        slots[1] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        prefetch_tensormap(&tm_q); prefetch_tensormap(&tm_k);
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(const_cast<uint32_t*>(&slots[0])), S_TMEM);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = slots[0];
    ib::pdl_wait();                                          // the rows and this step's cache rows come from predecessors

    if (warp == 0) {
        // ---------------------------------------------------------------- TMA producer
        int page = -1;
        if (lane < PAGES_PER_TILE) {
            const int key = key0 + lane * PAGE;
            page = key <= w.last_written ? page_at(p, seg, key) : -1;
            if (key <= w.last_written && key + PAGE - 1 >= lo_key && page < 0) atomicExch(p.status, STATUS_BAD_PAGE);
        }
        const int valid = __popc(__ballot_sync(0xffffffffu, page >= 0));
        if (lane == 0) {
            if (valid == 0) mbar_arrive(k_full);
            else mbar_expect_tx(k_full, uint32_t(valid) * p.n_kv * DB * (PAGE * 128));
        }
        __syncwarp();
        if (page >= 0) {
            for (int g = 0; g < p.n_kv; g++)
                for (int db = 0; db < DB; db++)
                    tma_load_2d(k_s + g * K_HEAD_BYTES + db * (BN * 128) + lane * (PAGE * 128), &tm_k, k_full, db * 64, (page * p.n_kv + g) * PAGE);
        }
        bool failed = false;
        int n = 0;
        for (int b = b0; b <= b1 && !failed; b++) {
            for (int g = 0; g < p.n_kv; g++, n++) {
                const int st = n % p.n_stages;
                if (n >= p.n_stages) {
                    int got = 1;
                    if (lane == 0) got = (!slots[1] && mbar_wait(q_empty + 8 * st, (n / p.n_stages - 1) & 1)) ? 1 : 0;
                    if (!__shfl_sync(0xffffffffu, got, 0)) { failed = true; break; }
                }
                if (lane == 0) mbar_expect_tx(q_full + 8 * st, uint32_t(stage_bytes));
                __syncwarp();
                for (int i = lane; i < group * DB; i += 32) {
                    const int hq = i / DB, db = i - hq * DB;
                    tma_load_2d(q_s + st * stage_bytes + (db * group + hq) * (NQ * 128), &tm_q, q_full + 8 * st,
                                p.q_col + (g * group + hq) * D + db * 64, w.t0 + qt * BM + b * NQ);
                }
            }
        }
        if (lane == 0) {
            if (failed && !slots[1]) { atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
            // Whatever happened to the others: no copy may land after the CTA is gone.
            if (valid > 0) mbar_wait(k_full, 0);
            for (int i = max(0, n - p.n_stages); i < n; i++) mbar_wait(q_full + 8 * (i % p.n_stages), (i / p.n_stages) & 1);
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer
        if (lane == 0) {
            const uint32_t idesc = make_idesc(group * NQ, false);
            bool ok = mbar_wait(k_full, 0);
            tc_fence_after();
            int n = 0, nb = 0;
            for (int b = b0; b <= b1 && ok && !slots[1]; b++, nb++) {
                const int buf = nb % S_BUFS;
                if (nb >= S_BUFS) ok = mbar_wait(s_empty + 8 * buf, (nb / S_BUFS - 1) & 1);
                tc_fence_after();
                for (int g = 0; g < p.n_kv && ok; g++, n++) {
                    const int st = n % p.n_stages;
                    ok = mbar_wait(q_full + 8 * st, (n / p.n_stages) & 1);
                    if (!ok) break;
                    tc_fence_after();
                    // one product per 16 channels for all heads of the group: 16 * group columns
                    const uint32_t dst = tmem_base + buf * (H * NQ) + g * group * NQ;
#pragma unroll
                    for (int db = 0; db < DB; db++) {
                        const uint64_t kd = make_desc(k_s + g * K_HEAD_BYTES + db * (BN * 128), 16, 1024);
                        const uint64_t qd = make_desc(q_s + st * stage_bytes + db * group * (NQ * 128), 16, 1024);
#pragma unroll
                        for (int k = 0; k < 4; k++)          // 16 elements of the head per step = 32 bytes = 2 address units
                            umma_f16(dst, kd + uint64_t(2 * k), qd + uint64_t(2 * k), idesc, (db > 0 || k > 0) ? 1u : 0u);
                    }
                    umma_commit(q_empty + 8 * st);
                }
                if (ok) umma_commit(s_full + 8 * buf);
            }
            if (!ok) { if (!slots[1]) atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
        }
    } else {
        // ---------------------------------------------------------------- cap, exchange, store (warps 2 and on)
        const int quad = warp & 3, q_share = (warp - 2) >> 2;
        const int key = quad * 32 + lane;                    // key of the tile = TMEM lane
        const uint32_t lane_addr = tmem_base + (uint32_t(quad * 32) << 16);
        const float two_y = p.cap > 0.0f ? 2.0f * LOG2E * p.scale / p.cap : 0.0f, cap = p.cap, scale = p.scale;
        float* dst0 = p.scores + (int64_t(w.slot) * H * p.max_tiles + (kt - w.kt0)) * TILE_FLOATS + key * 4;
        const int64_t head_stride = int64_t(p.max_tiles) * TILE_FLOATS;
        int nb = 0;
        bool ok = true;
        for (int b = b0; b <= b1; b++, nb++) {
            const int buf = nb % S_BUFS;
            ok = !slots[1] && mbar_wait(s_full + 8 * buf, (nb / S_BUFS) & 1);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
#pragma unroll 1
            for (int pass = 0; pass < PASSES; pass++) {
                const int i0 = (q_share * PASSES + pass) * 4;   // four queries of the block
                uint64_t s2[HP / 2][4];                      // the scores of two neighbouring heads, per query
                {
                    float s[HP][4];
#pragma unroll
                    for (int g = 0; g < H; g++) tmem_ld4(lane_addr + buf * (H * NQ) + g * NQ + i0, s[g]);
                    tmem_ld_wait();
#pragma unroll
                    for (int g = H; g < HP; g++) s[g][0] = s[g][1] = s[g][2] = s[g][3] = 0.0f;
                    if (pass == PASSES - 1) {                // everything this thread reads of the buffer has arrived
                        tc_fence_before();
                        __syncwarp();
                        if (lane == 0) mbar_arrive(s_empty + 8 * buf);
                    }
#pragma unroll
                    for (int g = 0; g < H; g++) {
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            // cap * tanh(y) = cap (1 - 2 / (1 + exp(2 y)))
                            if (cap > 0.0f) s[g][e] = fmaf(-2.0f * cap, fast_rcp(1.0f + fast_exp2(s[g][e] * two_y)), cap);
                            else s[g][e] *= scale;
                        }
                    }
#pragma unroll
                    for (int g = 0; g < HP / 2; g++)
#pragma unroll
                        for (int e = 0; e < 4; e++) s2[g][e] = pack2(s[2 * g][e], s[2 * g + 1][e]);
                }
                float* dst = dst0 + (b * NQ + i0) / 4 * (4 * BN);
                if (p.talk) {
#pragma unroll 2
                    for (int h = 0; h < H; h++) {
                        // even and odd heads are summed in the two halves of a pair
                        uint64_t acc[4] = {0, 0, 0, 0};
                        const ulonglong2* row = reinterpret_cast<const ulonglong2*>(T_s + h * HP);
#pragma unroll
                        for (int g = 0; g < HP / 4; g++) {
                            const ulonglong2 t = row[g];
#pragma unroll
                            for (int e = 0; e < 4; e++) acc[e] = fma2(t.y, s2[2 * g + 1][e], fma2(t.x, s2[2 * g][e], acc[e]));
                        }
                        float o[4];
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const float2 x = unpack2(acc[e]);
                            o[e] = x.x + x.y;
                        }
                        *reinterpret_cast<float4*>(dst + h * head_stride) = make_float4(o[0], o[1], o[2], o[3]);
                    }
                } else {
#pragma unroll
                    for (int h = 0; h < H; h++) {
                        float o[4];
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            const float2 x = unpack2(s2[h / 2][e]);
                            o[e] = h & 1 ? x.y : x.x;
                        }
                        *reinterpret_cast<float4*>(dst + h * head_stride) = make_float4(o[0], o[1], o[2], o[3]);
                    }
                }
            }
        }
        if (!ok && !slots[1]) { atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, S_TMEM);
    }
}

// ------------------------------------------------------------------------------------------------ kernel 2
constexpr int PV_THREADS = 192;
constexpr int PIECES = BM / 4, PIECE_BYTES = 4 * BN * 4, PIECE_ROW = PIECE_BYTES + 16;   // of a score tile
constexpr int V_BYTES = DVB * BN * 128, P_BYTES = (BN / 64) * BM * 128, SC_BYTES = PIECES * PIECE_ROW;
constexpr int PV_SMEM = 2 * V_BYTES + P_BYTES + 2 * SC_BYTES + 1024 + 128;
constexpr float RESCALE_STEP = 8.0f;         // O's reference maximum follows the running maximum in steps of this (log2)

__global__ void __launch_bounds__(PV_THREADS)
talk_pv_kernel(const __grid_constant__ CUtensorMap tm_v, const Params p) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
    const uint32_t v_s = base, p_s = v_s + 2 * V_BYTES, sc_s = p_s + P_BYTES, bars = sc_s + 2 * SC_BYTES;
    uint8_t* v_ptr = base_ptr;
    uint8_t* p_ptr = v_ptr + 2 * V_BYTES;
    const uint8_t* sc_ptr = p_ptr + P_BYTES;
    volatile uint32_t* slots = reinterpret_cast<volatile uint32_t*>(base_ptr + 2 * V_BYTES + P_BYTES + 2 * SC_BYTES + 112);
    const uint32_t s_full = bars, s_empty = bars + 16, v_full = bars + 32, v_empty = bars + 48, p_full = bars + 64, o_full = bars + 72;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // The last query tiles have the most keys: they start first, for every head.
    const int h = blockIdx.x, qt = p.qt0 + int(gridDim.y) - 1 - int(blockIdx.y), seg = blockIdx.z;
    Tile w;
    if (!tile_of(p, seg, qt, w)) return;
    const int kvh = h / (H / p.n_kv);
    const int n_tiles = w.kt1 - w.kt0 + 1;
    const int lo_key = first_visible(w.q_first, p.window, p.chunk);
    if (threadIdx.x == 0) {
        for (int b = 0; b < 2; b++) {
            mbar_init(s_full + 8 * b, 1); mbar_init(s_empty + 8 * b, 4); mbar_init(v_full + 8 * b, 1); mbar_init(v_empty + 8 * b, 1);
        }
        mbar_init(p_full, 4); mbar_init(o_full, 1);
        slots[1] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        prefetch_tensormap(&tm_v);
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(const_cast<uint32_t*>(&slots[0])), DV);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = slots[0];
    ib::pdl_wait();                                          // the scores come from the predecessor

    if (warp == 0) {
        // ---------------------------------------------------------------- producer: score pieces and value pages
        const uint8_t* src = reinterpret_cast<const uint8_t*>(p.scores + (int64_t(w.slot) * H + h) * p.max_tiles * TILE_FLOATS);
        int sent_s = 0, pend_v[2] = {-1, -1};
        auto wait_all = [&](uint32_t bar, uint32_t parity) -> bool {
            int got = 1;
            if (lane == 0) got = (!slots[1] && mbar_wait(bar, parity)) ? 1 : 0;
            return __shfl_sync(0xffffffffu, got, 0) != 0;
        };
        bool failed = false;
        for (int j = 0; j < n_tiles && !failed; j++) {
            const int b = j & 1;
            if (j >= 2 && !wait_all(s_empty + 8 * b, ((j >> 1) - 1) & 1)) { failed = true; break; }
            if (lane == 0) mbar_expect_tx(s_full + 8 * b, uint32_t(PIECES) * PIECE_BYTES);
            __syncwarp();
            bulk_load(sc_s + b * SC_BYTES + lane * PIECE_ROW, src + int64_t(j) * TILE_FLOATS * 4 + lane * PIECE_BYTES, PIECE_BYTES, s_full + 8 * b);
            sent_s = j + 1;
            if (j >= 2 && !wait_all(v_empty + 8 * b, ((j >> 1) - 1) & 1)) { failed = true; break; }
            int page = -1;
            if (lane < PAGES_PER_TILE) {
                const int key = (w.kt0 + j) * BN + lane * PAGE;
                page = key <= w.last_written ? page_at(p, seg, key) : -1;
                if (key <= w.last_written && key + PAGE - 1 >= lo_key && page < 0) atomicExch(p.status, STATUS_BAD_PAGE);
            }
            const int valid = __popc(__ballot_sync(0xffffffffu, page >= 0));
            if (lane == 0) {
                if (valid == 0) mbar_arrive(v_full + 8 * b);
                else mbar_expect_tx(v_full + 8 * b, uint32_t(valid) * DVB * (PAGE * 128));
            }
            __syncwarp();
            if (page >= 0) {
                for (int db = 0; db < DVB; db++)
                    tma_load_2d(v_s + b * V_BYTES + db * (BN * 128) + lane * (PAGE * 128), &tm_v, v_full + 8 * b, db * 64, (page * p.n_kv + kvh) * PAGE);
            }
            if (valid > 0) pend_v[b] = j;
        }
        if (lane == 0) {
            if (failed && !slots[1]) { atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
            for (int j = max(0, sent_s - 2); j < sent_s; j++) mbar_wait(s_full + 8 * (j & 1), (j >> 1) & 1);
            for (int b = 0; b < 2; b++)
                if (pend_v[b] >= 0) mbar_wait(v_full + 8 * b, (pend_v[b] >> 1) & 1);
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer: O += P V
        if (lane == 0) {
            constexpr uint32_t idesc = make_idesc(DV, true);
            bool ok = true;
            for (int j = 0; j < n_tiles && ok && !slots[1]; j++) {
                ok = mbar_wait(p_full, j & 1) && mbar_wait(v_full + 8 * (j & 1), (j >> 1) & 1);
                if (!ok) break;
                tc_fence_after();
#pragma unroll
                for (int k = 0; k < BN / 16; k++) {          // 16 keys per step: 32 bytes along P's rows, 2 groups of 8 rows of V
                    const uint64_t pd = make_desc(p_s + (k / 4) * (BM * 128), 16, 1024) + uint64_t(2 * (k % 4));
                    const uint64_t vd = make_desc(v_s + (j & 1) * V_BYTES + k * (16 * 128), BN * 128, 1024);
                    umma_f16(tmem_base, pd, vd, idesc, (j > 0 || k > 0) ? 1u : 0u);
                }
                umma_commit(o_full);
                umma_commit(v_empty + 8 * (j & 1));
            }
            if (!ok) { if (!slots[1]) atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
        }
    } else {
        // ---------------------------------------------------------------- softmax and epilogue (warps 2..5)
        const int quad = warp & 3;
        const int r = quad * 32 + lane;                      // query row of the tile = TMEM lane
        const uint32_t lane_addr = tmem_base + (uint32_t(quad * 32) << 16);
        const int row_pos = w.q_first + r;
        const int row_lo = first_visible(row_pos, p.window, p.chunk);
        const int tile_lo = first_visible(w.q_first + BM - 1, p.window, p.chunk);    // the last row's (no row's is larger)
        float m_ref = -INFINITY, l = 0.0f;                   // reference maximum of this row's O and P; sum of probabilities
        bool ok = true;
        for (int j = 0; j < n_tiles; j++) {
            const int key0 = (w.kt0 + j) * BN;
            ok = !slots[1] && mbar_wait(s_full + 8 * (j & 1), (j >> 1) & 1);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            float s[BN];
            const float* row = reinterpret_cast<const float*>(sc_ptr + (j & 1) * SC_BYTES + (r >> 2) * PIECE_ROW) + (r & 3);
#pragma unroll
            for (int c = 0; c < BN; c++) s[c] = row[c * 4];
            __syncwarp();
            if (lane == 0) mbar_arrive(s_empty + 8 * (j & 1));
            float mxs[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (key0 + BN - 1 <= w.q_first && key0 >= tile_lo) {
#pragma unroll
                for (int c = 0; c < BN; c++) mxs[c & 3] = fmaxf(mxs[c & 3], s[c]);
            } else {
                const int hi = row_pos - key0, lo = row_lo - key0;       // visible: lo <= c <= hi
#pragma unroll
                for (int c = 0; c < BN; c++) {
                    s[c] = ((c <= hi) & (c >= lo)) ? s[c] : -INFINITY;
                    mxs[c & 3] = fmaxf(mxs[c & 3], s[c]);
                }
            }
            const float mx = fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3])) * LOG2E;
            const bool raise = mx > m_ref + RESCALE_STEP || (m_ref == -INFINITY && mx > -INFINITY);
            const float alpha = raise ? fast_exp2(m_ref - mx) : 1.0f;   // m_ref = -inf gives 0: nothing was summed yet
            if (raise) { m_ref = mx; l *= alpha; }
            // with no visible key so far every score is -inf: subtracting 0 instead of -inf keeps exp2 at 0, not NaN
            const float m_neg = m_ref == -INFINITY ? 0.0f : -m_ref;
            float sums[2] = {0.0f, 0.0f};
            uint32_t pk[BN / 2];                             // the row of P, packed
#pragma unroll
            for (int c = 0; c < BN; c += 2) {
                const float x = fast_exp2(fmaf(s[c], LOG2E, m_neg)), y = fast_exp2(fmaf(s[c + 1], LOG2E, m_neg));
                __nv_bfloat162 two = __floats2bfloat162_rn(x, y);
                pk[c / 2] = *reinterpret_cast<uint32_t*>(&two);
                sums[(c >> 1) & 1] += x + y;
            }
            l += sums[0] + sums[1];
            if (j > 0) {
                // P(j-1) V(j-1) must be complete before P is overwritten and before O is touched
                ok = mbar_wait(o_full, (j - 1) & 1);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                if (__any_sync(0xffffffffu, raise)) {
                    tc_fence_after();
#pragma unroll 1
                    for (int c = 0; c < DV; c += 16) {
                        uint32_t o[16];
                        tmem_ld16(lane_addr + c, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int e = 0; e < 16; e++) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
                        tmem_st16(lane_addr + c, o);
                    }
                    tmem_st_wait();
                }
            }
            uint8_t* prow0 = p_ptr + (r >> 3) * 1024 + (r & 7) * 128;
#pragma unroll
            for (int c8 = 0; c8 < BN / 8; c8++) {
                uint8_t* prow = prow0 + (c8 >> 3) * (BM * 128);
                *reinterpret_cast<uint4*>(prow + (((c8 & 7) ^ (r & 7)) << 4)) = make_uint4(pk[c8 * 4], pk[c8 * 4 + 1], pk[c8 * 4 + 2], pk[c8 * 4 + 3]);
            }
            // Rows of V that hold nothing this step may read (positions after the segment's last token, pages the table
            // does not hold) become zeros, so that 0 x garbage cannot make a NaN.
            if (key0 + BN - 1 > w.last_written || key0 < lo_key) {
                ok = mbar_wait(v_full + 8 * (j & 1), (j >> 1) & 1);
                ok = __all_sync(0xffffffffu, ok);
                if (!ok) break;
                for (int u = r; u < BN * DVB; u += BM) {
                    const int key_row = u % BN, db = u / BN;
                    const int key = key0 + key_row;
                    if (key > w.last_written || page_at(p, seg, key) < 0) {
                        uint4* line = reinterpret_cast<uint4*>(v_ptr + (j & 1) * V_BYTES + db * (BN * 128) + key_row * 128);
#pragma unroll
                        for (int e = 0; e < 8; e++) line[e] = make_uint4(0u, 0u, 0u, 0u);
                    }
                }
            }
            fence_proxy_async();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full);
        }
        if (ok) {
            ok = mbar_wait(o_full, (n_tiles - 1) & 1);
            ok = __all_sync(0xffffffffu, ok);
        }
        if (!ok && !slots[1]) { atomicExch(p.status, STATUS_TIMEOUT); slots[1] = 1; }
        const int qi = qt * BM + r;
        bf16* dst = p.out + (int64_t(w.t0 + qi) * H + h) * DV;
        if (ok) {
            tc_fence_after();
            const float inv = l > 0.0f ? 1.0f / l : 0.0f;
#pragma unroll 1
            for (int c = 0; c < DV; c += 16) {
                uint32_t o[16];
                tmem_ld16(lane_addr + c, o);
                tmem_ld_wait();
                uint32_t two[8];
#pragma unroll
                for (int e = 0; e < 8; e++) {
                    __nv_bfloat162 pair = __floats2bfloat162_rn(__uint_as_float(o[2 * e]) * inv, __uint_as_float(o[2 * e + 1]) * inv);
                    two[e] = *reinterpret_cast<uint32_t*>(&pair);
                }
                if (qi < w.q_len) {
                    *reinterpret_cast<uint4*>(dst + c) = make_uint4(two[0], two[1], two[2], two[3]);
                    *reinterpret_cast<uint4*>(dst + c + 8) = make_uint4(two[4], two[5], two[6], two[7]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, DV);
    }
}

constexpr int SMEM_LIMIT = 227 * 1024;
// Stages of the query ring that fit beside the key tile; 0: the sizes do not fit.
int ring_stages(int n_kv) {
    const int left = SMEM_LIMIT - SCORE_FIXED - n_kv * K_HEAD_BYTES, stage = H / n_kv * Q_HEAD_BYTES;
    return left < 2 * stage ? 0 : std::min(MAX_STAGES, left / stage);
}

}  // namespace

IB_EXPORT int64_t ib_talk_prefill_tile_floats() { return TILE_FLOATS; }

// 1 if this build takes these sizes.
IB_EXPORT int ib_talk_prefill_fits(int n_heads, int n_kv, int d, int dv, int page_size) {
    return n_heads == H && d == D && dv == DV && page_size == PAGE && n_kv > 0 && H % n_kv == 0 && H / n_kv <= 16 && ring_stages(n_kv) > 0;
}

// Attention of the segments with two or more tokens (others are skipped), their query tiles qt0 .. qt0 + n_qt - 1 of 128
// tokens each. q: rows of leading dimension ldq with the heads' queries from column q_col; caches bfloat16 [pages, kv heads,
// 16, D / DV] that hold this step's keys and values already; out [tokens, H * DV]; scores: room for n_long * n_qt * H *
// max_tiles tiles, max_tiles at least the key tiles of 128 that any of these query tiles sees. q_split (1, 2, 4 or 8): CTAs that
// share a (query tile, key tile).
IB_EXPORT int ib_talk_prefill(const void* q, int64_t ldq, int q_col, const void* k_cache, const void* v_cache, void* out,
                              const int* block_table, int max_blocks, const int* seg_start, const int* seg_pos0, int n_segments,
                              int64_t n_tokens, int n_heads, int n_kv, int d, int dv, int page_size, int window, int chunk, float scale,
                              float cap, const float* talk, int64_t n_pages, int qt0, int n_qt, int max_tiles, int q_split, float* scores,
                              int64_t score_floats, int n_long, int* status, cudaStream_t stream) {
    if (n_segments <= 0 || n_qt <= 0) return IB_OK;
    if (!ib_talk_prefill_fits(n_heads, n_kv, d, dv, page_size))
        return ib::fail(IB_ERR_ARG, "ib_talk_prefill: built for %d heads of %d / %d, called with %d on %d kv heads of %d / %d", H, D, DV, n_heads, n_kv, d, dv);
    if (!status || !scores || max_tiles <= 0 || qt0 < 0) return ib::fail(IB_ERR_ARG, "ib_talk_prefill: a status word and room for scores are needed");
    if (q_split < 1 || q_split > BLOCKS || BLOCKS % q_split) return ib::fail(IB_ERR_ARG, "ib_talk_prefill: q_split %d", q_split);
    if (n_long <= 0 || n_long > n_segments || int64_t(n_long) * n_qt * H * max_tiles * TILE_FLOATS > score_floats)
        return ib::fail(IB_ERR_ARG, "ib_talk_prefill: the scores of %d portions do not fit", n_long);
    if (n_segments > 65535 || int64_t(n_qt) * q_split > 65535) return ib::fail(IB_ERR_ARG, "ib_talk_prefill: too many segments or query tiles");
    if (ldq % 8 || q_col % 8 || (uintptr_t(q) | uintptr_t(k_cache) | uintptr_t(v_cache) | uintptr_t(out) | uintptr_t(scores)) & 15)
        return ib::fail(IB_ERR_ARG, "ib_talk_prefill: rows must be whole 16-byte pieces");
    if (n_pages * n_kv * PAGE >= (1LL << 31) || n_tokens >= (1LL << 31)) return ib::fail(IB_ERR_ARG, "ib_talk_prefill: the cache or the step is too large for 32-bit tile coordinates");
    CUtensorMap mq, mk, mv;
    int rc = ib::get_map(q, n_tokens, ldq, NQ, &mq);
    if (rc) return rc;
    rc = ib::get_map(k_cache, n_pages * n_kv * PAGE, D, PAGE, &mk);
    if (rc) return rc;
    rc = ib::get_map(v_cache, n_pages * n_kv * PAGE, DV, PAGE, &mv);
    if (rc) return rc;
    Params p = {};
    p.block_table = block_table; p.max_blocks = max_blocks; p.seg_start = seg_start; p.seg_pos0 = seg_pos0;
    p.n_kv = n_kv; p.window = window; p.chunk = chunk; p.n_pages = n_pages; p.status = status;
    p.scores = scores; p.max_tiles = max_tiles; p.qt0 = qt0; p.n_qt = n_qt;
    p.scale = scale; p.cap = cap; p.talk = talk; p.q_col = q_col; p.n_stages = ring_stages(n_kv); p.q_split = q_split;
    p.out = (bf16*)out;
    const size_t smem = SCORE_FIXED + size_t(n_kv) * K_HEAD_BYTES + size_t(p.n_stages) * (H / n_kv) * Q_HEAD_BYTES;
    static size_t configured = 0;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(talk_scores_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
        if (e == cudaSuccess) e = cudaFuncSetAttribute(talk_pv_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, PV_SMEM);
        if (e != cudaSuccess) return ib::fail(IB_ERR_CUDA, "ib_talk_prefill: cannot set shared memory size: %s", cudaGetErrorString(e));
        configured = smem;
    }
    const dim3 g1{unsigned(max_tiles), unsigned(n_qt * q_split), unsigned(n_segments)};
    rc = ib::launch("talk_scores", talk_scores_kernel, g1, dim3(SCORE_THREADS), smem, stream, 1u, mq, mk, p);
    if (rc) return rc;
    const dim3 g2{unsigned(H), unsigned(n_qt), unsigned(n_segments)};
    return ib::launch("talk_pv", talk_pv_kernel, g2, dim3(PV_THREADS), size_t(PV_SMEM), stream, 1u, mv, p);
}
