// The recurrence S <- g_t S + b_t k_t v_t^T, o_t = S^T q_t + skip v_t (state_scan mode 5, mix_ops.cu) over prompt portions, in
// chunks of L = 64 tokens on the tensor cores. With c_t the sum of ln g over a chunk's tokens up to t, and S the state
// in front of the chunk,
//     o_t = e^(c_t) S^T q_t + sum over s <= t of e^(c_t - c_s) b_s (q_t . k_s) v_s
//     S  <- e^(c_L) S + sum over s of e^(c_L - c_s) b_s k_s v_s^T
// q, k and v (projections behind their filters and activations) are rounded to bfloat16 once. Everything else is float:
// sums of ln g are formed in double and kept as two floats, so that a difference of two of them is exact to float; factors and
// exponentials are float; the state lives in float accumulators from chunk to chunk, and where it, or a product of scores and
// factors, or a weighted value row is an operand, it enters as the sum of two bfloat16 numbers (sixteen bits and more).
//
// One CTA per (segment, head, NB columns of the state) walks over the chunks in order. Its sixteen warps are three groups that
// work side by side on a chunk and meet once per chunk:
//   warps 0..7    (two for 16 tokens: each takes half of the state's rows and every other block of 16 keys) scores, factors,
//                 read-out
//   warps 8..11   (D / 4 rows of the state each) the state's update; leave the two halves of the new state for the next chunk
//   warps 12..15  request the next chunk's q and k (asynchronous copies of bfloat16 rows that pack_qk_kernel has rounded and
//                 padded), and form the sums of ln g and the weighted value rows from what they requested a chunk earlier
#include "common.cuh"

IB_DEFINE_LAST_ERROR()

namespace {

using bf16 = __nv_bfloat16;

constexpr int L = 64;                       // tokens of a chunk
constexpr int THREADS = 512;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float LEAST = -200.0f;            // e^-200 is zero in float: ln g below it (g = 0 too) changes nothing

__device__ __forceinline__ uint32_t smem_at(const void* p) { return uint32_t(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as the sum of two pairs of bfloat16 numbers
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float pow2(float x) {              // (two units in the last place; float's least numbers are zero)
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ uint2 bf16x4(float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    return make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ float4 floats(uint2 u) {
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void group_barrier(int id) { asm volatile("bar.sync %0, 128;" ::"r"(id) : "memory"); }

__device__ __forceinline__ void chunk_barrier() { asm volatile("bar.sync 0;" ::: "memory"); }

template <int D, int NB>
struct Layout {
    static constexpr int DP = D + 8, NP = NB + 8;             // padded rows: eight rows of a fragment on different banks
    bf16 q[2][L][DP], k[2][L][DP];
    bf16 v[2][L][NP], wh[2][L][NP], wl[2][L][NP];             // values; values times e^(c_L - c_s) b_s in two halves
    bf16 sh[2][D][NP], sl[2][D][NP];                          // the state in front of the chunk, in two halves
    float ch[2][L], cl[2][L], b[2][L];                        // sums of log2 g (two floats), strengths
    float part[4][16][NB];                                    // what the second of two read-out warps hands to the first
};

// q and k of every token in bfloat16, heads padded with zeros to D channels: out [tokens, 2 (q, k), heads, D].
__global__ void __launch_bounds__(256)
pack_qk_kernel(const float* __restrict__ rows, int64_t ld, int q_col, int k_col, int n_qk, int d, int D, bf16* __restrict__ out) {
    ib::pdl_launch_dependents();
    ib::pdl_wait();
    const int64_t t = blockIdx.x;
    const int half_width = n_qk * D;
    for (int i = threadIdx.x * 4; i < 2 * half_width; i += blockDim.x * 4) {
        const int side = i >= half_width, j = i - side * half_width, h = j / D, e = j - h * D;
        const float* r = rows + t * ld + (side ? k_col : q_col) + h * d;
        float x[4];
#pragma unroll
        for (int c = 0; c < 4; c++) x[c] = e + c < d ? r[e + c] : 0.0f;
        *reinterpret_cast<uint2*>(out + t * 2 * half_width + i) = bf16x4(make_float4(x[0], x[1], x[2], x[3]));
    }
}

template <int D, int NB>
__global__ void __launch_bounds__(THREADS)
chunk_scan_kernel(const bf16* __restrict__ qk, const float* __restrict__ rows, int64_t ld, int v_col, const float* __restrict__ aux, int64_t lda,
                  int b_col, int lng_col, float* __restrict__ state, float* __restrict__ ones_state, const int* __restrict__ seg_start,
                  const int* __restrict__ seg_slot, float* __restrict__ raw_out, float* __restrict__ ones_out,
                  const float* __restrict__ skip_w, int n_heads, int heads_per_qk, int d, int dv, int write_state, int vec_v) {
    extern __shared__ __align__(16) unsigned char raw_smem[];
    using Lay = Layout<D, NB>;
    Lay& sm = *reinterpret_cast<Lay*>(raw_smem);
    constexpr int NT = NB / 8, KT = D / 16;
    const int seg = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * NB, hq = h / heads_per_qk;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gw = warp & 3;
    const int group = warp < 8 ? 0 : (warp < 12 ? 1 : 2);
    const int fr = lane >> 2, fc = (lane & 3) * 2;             // a fragment's row and first column
    ib::pdl_wait();
    const int64_t t0 = seg_start[seg];
    const int len = int(seg_start[seg + 1] - t0);
    if (len <= 0) return;
    const int n_chunks = (len + L - 1) / L;
    const int64_t slot_head = int64_t(seg_slot[seg]) * n_heads + h;
    float* S_g = state + slot_head * int64_t(d) * dv;
    float* n_g = ones_state ? ones_state + slot_head * d : nullptr;

    // Every group has a loop of its own over the chunks (and so only its own registers); all meet at the chunk's barrier: from
    // there on chunk c and the state in front of it lie in buffer c & 1.
    if (group == 2) {
        // ---- fetching a chunk (warps 12..15)
        const int lt = tid - 384;
        constexpr int PER = L * (D / 8) / 128, PER_V = L * NB / 512;
        const int n_qk = n_heads / heads_per_qk;
        float4 vv[PER_V];                                     // the next chunk's values, ln g and strengths
        float g0, g1, b0, b1;
        auto request_qk = [&](int c) {                        // into the chunk's own buffer
            const int n = min(L, len - c * L), buf = c & 1;
            const bf16* from = qk + ((t0 + int64_t(c) * L) * 2 * n_qk + hq) * D;
#pragma unroll
            for (int j = 0; j < PER; j++) {
                const int i = lt + j * 128, t = i / (D / 8), e = (i % (D / 8)) * 8;
                const int bytes = t < n ? 16 : 0;              // (0: zeros are written)
                const bf16* r = from + (bytes ? int64_t(t) * 2 * n_qk * D + e : 0);
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_at(&sm.q[buf][t][e])), "l"(r), "r"(bytes) : "memory");
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_at(&sm.k[buf][t][e])), "l"(r + n_qk * D), "r"(bytes) : "memory");
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        auto request_v = [&](int c) {                         // into registers
            const int n = min(L, len - c * L);
            const int64_t tc = t0 + int64_t(c) * L;
#pragma unroll
            for (int j = 0; j < PER_V; j++) {
                const int i = lt + j * 128, t = i / (NB / 4), col = col0 + (i % (NB / 4)) * 4;
                const float* r = rows + (tc + t) * ld + v_col + int64_t(h) * dv + col;
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t < n) {
                    if (vec_v && col < dv) {
                        v = *reinterpret_cast<const float4*>(r);
                    } else {
                        const float one = n_g ? 1.0f : 0.0f;  // the column of ones behind the values
                        v.x = col < dv ? r[0] : (col == dv ? one : 0.0f);
                        v.y = col + 1 < dv ? r[1] : (col + 1 == dv ? one : 0.0f);
                        v.z = col + 2 < dv ? r[2] : (col + 2 == dv ? one : 0.0f);
                        v.w = col + 3 < dv ? r[3] : (col + 3 == dv ? one : 0.0f);
                    }
                }
                vv[j] = v;
            }
            g0 = g1 = b0 = b1 = 0.0f;
            if (gw == 0) {                                    // a lane's two neighbouring tokens
                const int i = 2 * lane;
                if (i < n) { g0 = aux[(tc + i) * lda + lng_col + h]; b0 = aux[(tc + i) * lda + b_col + h]; }
                if (i + 1 < n) { g1 = aux[(tc + i + 1) * lda + lng_col + h]; b1 = aux[(tc + i + 1) * lda + b_col + h]; }
            }
        };
        auto form = [&](int c) {                              // sums of ln g, value rows, weighted value rows
            const int buf = c & 1;
            if (gw == 0) {
                const double x0 = double(fmaxf(g0, LEAST) * LOG2E), x1 = double(fmaxf(g1, LEAST) * LOG2E);
                double sum = x0 + x1;                         // inclusive over lanes
#pragma unroll
                for (int o = 1; o < 32; o <<= 1) {
                    const double up = __shfl_up_sync(0xffffffffu, sum, o);
                    if (lane >= o) sum += up;
                }
                const double c0 = sum - x1, c1 = sum;
                const float h0 = float(c0), h1 = float(c1);
                sm.ch[buf][2 * lane] = h0;
                sm.cl[buf][2 * lane] = float(c0 - double(h0));
                sm.ch[buf][2 * lane + 1] = h1;
                sm.cl[buf][2 * lane + 1] = float(c1 - double(h1));
                sm.b[buf][2 * lane] = b0;
                sm.b[buf][2 * lane + 1] = b1;
            }
            group_barrier(1);
            const float eh = sm.ch[buf][L - 1], el = sm.cl[buf][L - 1];
#pragma unroll
            for (int j = 0; j < PER_V; j++) {
                const int i = lt + j * 128, t = i / (NB / 4), e = (i % (NB / 4)) * 4;
                const uint2 v16 = bf16x4(vv[j]);
                const float w = pow2((eh - sm.ch[buf][t]) + (el - sm.cl[buf][t])) * sm.b[buf][t];
                float4 x = floats(v16);
                x.x *= w; x.y *= w; x.z *= w; x.w *= w;
                const uint2 hi = bf16x4(x);
                const float4 f = floats(hi);
                *reinterpret_cast<uint2*>(&sm.v[buf][t][e]) = v16;
                *reinterpret_cast<uint2*>(&sm.wh[buf][t][e]) = hi;
                *reinterpret_cast<uint2*>(&sm.wl[buf][t][e]) = bf16x4(make_float4(x.x - f.x, x.y - f.y, x.z - f.z, x.w - f.w));
            }
            asm volatile("cp.async.wait_all;" ::: "memory");
        };
        request_qk(0);
        request_v(0);
        form(0);
        if (n_chunks > 1) request_v(1);
        for (int c = 0; c < n_chunks; c++) {
            chunk_barrier();
            if (c + 1 < n_chunks) {
                request_qk(c + 1);
                form(c + 1);
            }
            if (c + 2 < n_chunks) request_v(c + 2);
        }
    } else if (group == 1) {
        // ---- the state (warps 8..11): accumulators of MT x NT fragments, rows d0 + 16 m + fr (+ 8), columns 8 n + fc (+ 1)
        constexpr int MT = D / 64;
        const int d0 = gw * (D / 4);
        float S[MT][NT][4];
        auto at_state = [&](int m, int n, int e, bool& there, float*& p) {
            const int r = d0 + 16 * m + fr + (e >> 1) * 8, col = col0 + 8 * n + fc + (e & 1);
            there = r < d && (col < dv || (n_g && col == dv));
            p = col < dv ? S_g + int64_t(r) * dv + col : n_g + r;
        };
        auto leave_state = [&](int buf) {
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int n = 0; n < NT; n++)
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const int r = d0 + 16 * m + fr + half * 8, col = 8 * n + fc;
                        uint32_t hi, lo;
                        split2(S[m][n][2 * half], S[m][n][2 * half + 1], hi, lo);
                        *reinterpret_cast<uint32_t*>(&sm.sh[buf][r][col]) = hi;
                        *reinterpret_cast<uint32_t*>(&sm.sl[buf][r][col]) = lo;
                    }
        };
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int n = 0; n < NT; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    bool there;
                    float* p;
                    at_state(m, n, e, there, p);
                    S[m][n][e] = there ? *p : 0.0f;
                }
        leave_state(0);
        for (int c = 0; c < n_chunks; c++) {
            chunk_barrier();
            const int buf = c & 1, n_tok = min(L, len - c * L);
            const float keep = pow2(sm.ch[buf][L - 1] + sm.cl[buf][L - 1]);
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int n = 0; n < NT; n++)
#pragma unroll
                    for (int e = 0; e < 4; e++) S[m][n][e] *= keep;
#pragma unroll
            for (int kk = 0; kk < L / 16; kk++) {
                if (kk * 16 >= n_tok) break;
                uint32_t a[MT][4];                            // K^T: rows of the state x tokens
#pragma unroll
                for (int m = 0; m < MT; m++)
                    ldm4t(a[m], &sm.k[buf][kk * 16 + (lane >> 4) * 8 + (lane & 7)][d0 + 16 * m + ((lane >> 3) & 1) * 8]);
                uint32_t bh[NT / 2][4], bl[NT / 2][4];        // tokens x two column tiles each
#pragma unroll
                for (int n2 = 0; n2 < NT / 2; n2++) {
                    const int row = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), col = 16 * n2 + (lane >> 4) * 8;
                    ldm4t(bh[n2], &sm.wh[buf][row][col]);
                    ldm4t(bl[n2], &sm.wl[buf][row][col]);
                }
                // (products that add to one fragment stand as far apart as there are fragments)
#pragma unroll
                for (int m = 0; m < MT; m++)
#pragma unroll
                    for (int n = 0; n < NT; n++) mma(S[m][n], a[m], bh[n / 2][(n & 1) * 2], bh[n / 2][(n & 1) * 2 + 1]);
#pragma unroll
                for (int m = 0; m < MT; m++)
#pragma unroll
                    for (int n = 0; n < NT; n++) mma(S[m][n], a[m], bl[n / 2][(n & 1) * 2], bl[n / 2][(n & 1) * 2 + 1]);
            }
            if (c + 1 < n_chunks) {
                leave_state(buf ^ 1);
            } else if (write_state) {
#pragma unroll
                for (int m = 0; m < MT; m++)
#pragma unroll
                    for (int n = 0; n < NT; n++)
#pragma unroll
                        for (int e = 0; e < 4; e++) {
                            bool there;
                            float* p;
                            at_state(m, n, e, there, p);
                            if (there) *p = S[m][n][e];
                        }
            }
        }
    } else {
        const float skip = skip_w ? skip_w[h] : 0.0f;
        // which of the two warps, and which sixteen tokens: later tokens see more keys, so the second warps go the other way round
        // and every scheduler (warps w, w + 4, ..) gets a long and a short one
        const int half = warp >> 2, rg = half ? 3 - gw : gw;
        for (int c = 0; c < n_chunks; c++) {
            chunk_barrier();
            const int buf = c & 1, n_tok = min(L, len - c * L);
            if (rg * 16 >= n_tok) continue;
            const int r0 = rg * 16;                           // this warp's tokens: r0 + fr and r0 + fr + 8
            uint32_t q[KT][4];
#pragma unroll
            for (int kk = 0; kk < KT; kk++)
                ldm4(q[kk], &sm.q[buf][r0 + ((lane >> 3) & 1) * 8 + (lane & 7)][kk * 16 + (lane >> 4) * 8]);
            float o[NT][4];
#pragma unroll
            for (int n = 0; n < NT; n++)
#pragma unroll
                for (int e = 0; e < 4; e++) o[n][e] = 0.0f;
#pragma unroll
            for (int k2 = 0; k2 < KT / 2; k2++) {             // (an even number of steps apart: the registers stay fixed)
                uint32_t bh[NT / 2][4], bl[NT / 2][4], qk[4];
                const int kk = k2 + half * (KT / 2);
#pragma unroll
                for (int i = 0; i < 4; i++) qk[i] = half ? q[k2 + KT / 2][i] : q[k2][i];
#pragma unroll
                for (int n2 = 0; n2 < NT / 2; n2++) {
                    const int row = kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), col = 16 * n2 + (lane >> 4) * 8;
                    ldm4t(bh[n2], &sm.sh[buf][row][col]);
                    ldm4t(bl[n2], &sm.sl[buf][row][col]);
                }
#pragma unroll
                for (int n = 0; n < NT; n++) mma(o[n], qk, bh[n / 2][(n & 1) * 2], bh[n / 2][(n & 1) * 2 + 1]);
#pragma unroll
                for (int n = 0; n < NT; n++) mma(o[n], qk, bl[n / 2][(n & 1) * 2], bl[n / 2][(n & 1) * 2 + 1]);
            }
            const int ra = r0 + fr, rb = ra + 8;
            const float ha = sm.ch[buf][ra], la = sm.cl[buf][ra], hb = sm.ch[buf][rb], lb = sm.cl[buf][rb];
            const float ea = pow2(ha + la), eb = pow2(hb + lb);
#pragma unroll
            for (int n = 0; n < NT; n++) { o[n][0] *= ea; o[n][1] *= ea; o[n][2] *= eb; o[n][3] *= eb; }
            // sixteen keys at a time: scores, factors, their two halves, values
#pragma unroll 1
            for (int j = half; j <= rg; j += 2) {
                float s[2][4], s2[2][4];                      // (even and odd steps over the channels)
#pragma unroll
                for (int i = 0; i < 2; i++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[i][e] = s2[i][e] = 0.0f;
#pragma unroll
                for (int kk = 0; kk < KT; kk++) {
                    uint32_t kb[4];                           // keys 16 j + (0..7 | 8..15), channels in two halves
                    ldm4(kb, &sm.k[buf][16 * j + (lane >> 4) * 8 + (lane & 7)][kk * 16 + ((lane >> 3) & 1) * 8]);
                    mma((kk & 1) ? s2[0] : s[0], q[kk], kb[0], kb[1]);
                    mma((kk & 1) ? s2[1] : s[1], q[kk], kb[2], kb[3]);
                }
#pragma unroll
                for (int i = 0; i < 2; i++)
#pragma unroll
                    for (int e = 0; e < 4; e++) s[i][e] += s2[i][e];
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    const int ka = 16 * j + 8 * i + fc, kb_ = ka + 1;
                    const float h0 = sm.ch[buf][ka], l0 = sm.cl[buf][ka], b0 = sm.b[buf][ka];
                    const float h1 = sm.ch[buf][kb_], l1 = sm.cl[buf][kb_], b1 = sm.b[buf][kb_];
                    const float p0 = ka <= ra ? s[i][0] * pow2((ha - h0) + (la - l0)) * b0 : 0.0f;
                    const float p1 = kb_ <= ra ? s[i][1] * pow2((ha - h1) + (la - l1)) * b1 : 0.0f;
                    const float p2 = ka <= rb ? s[i][2] * pow2((hb - h0) + (lb - l0)) * b0 : 0.0f;
                    const float p3 = kb_ <= rb ? s[i][3] * pow2((hb - h1) + (lb - l1)) * b1 : 0.0f;
                    split2(p0, p1, ph[2 * i], pl[2 * i]);
                    split2(p2, p3, ph[2 * i + 1], pl[2 * i + 1]);
                }
                uint32_t vb[NT / 2][4];
#pragma unroll
                for (int n2 = 0; n2 < NT / 2; n2++)
                    ldm4t(vb[n2], &sm.v[buf][16 * j + ((lane >> 3) & 1) * 8 + (lane & 7)][16 * n2 + (lane >> 4) * 8]);
#pragma unroll
                for (int n = 0; n < NT; n++) mma(o[n], ph, vb[n / 2][(n & 1) * 2], vb[n / 2][(n & 1) * 2 + 1]);
#pragma unroll
                for (int n = 0; n < NT; n++) mma(o[n], pl, vb[n / 2][(n & 1) * 2], vb[n / 2][(n & 1) * 2 + 1]);
            }
            // the second warp's share to the first, which stores
            float(&part)[16][NB] = sm.part[rg];
            if (half == 1) {
#pragma unroll
                for (int n = 0; n < NT; n++) {
                    *reinterpret_cast<float2*>(&part[fr][8 * n + fc]) = make_float2(o[n][0], o[n][1]);
                    *reinterpret_cast<float2*>(&part[fr + 8][8 * n + fc]) = make_float2(o[n][2], o[n][3]);
                }
            }
            asm volatile("bar.sync %0, 64;" ::"r"(2 + rg) : "memory");
            if (half == 0) {
#pragma unroll
                for (int two = 0; two < 2; two++) {
                    const int t = r0 + fr + two * 8;
                    if (t >= n_tok) continue;
                    const int64_t tok = t0 + int64_t(c) * L + t;
                    float* dst = raw_out + (tok * n_heads + h) * int64_t(dv);
#pragma unroll
                    for (int n = 0; n < NT; n++) {
                        const int col = col0 + 8 * n + fc;
                        const float2 other = *reinterpret_cast<const float2*>(&part[fr + two * 8][8 * n + fc]);
                        float y0 = o[n][2 * two] + other.x, y1 = o[n][2 * two + 1] + other.y;
                        if (skip_w) {
                            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&sm.v[buf][t][8 * n + fc]));
                            y0 = fmaf(skip, v.x, y0);
                            y1 = fmaf(skip, v.y, y1);
                        }
                        if (vec_v && col < dv) {
                            *reinterpret_cast<float2*>(dst + col) = make_float2(y0, y1);
                        } else {
                            if (col < dv) dst[col] = y0;
                            else if (n_g && col == dv) ones_out[tok * n_heads + h] = o[n][2 * two] + other.x;
                            if (col + 1 < dv) dst[col + 1] = y1;
                            else if (n_g && col + 1 == dv) ones_out[tok * n_heads + h] = o[n][2 * two + 1] + other.y;
                        }
                    }
                }
            }
        }
    }
}

template <int D, int NB>
int launch_chunk(dim3 grid, cudaStream_t stream, const bf16* qk, const float* rows, int64_t ld, int v_col, const float* aux, int64_t lda,
                 int b_col, int lng_col, float* state, float* ones_state, const int* seg_start, const int* seg_slot, float* raw_out,
                 float* ones_out, const float* skip, int n_heads, int hpq, int d, int dv, int write_state, int vec_v) {
    constexpr size_t smem = sizeof(Layout<D, NB>);
    static bool set = false;
    if (!set) {
        const cudaError_t e = cudaFuncSetAttribute(chunk_scan_kernel<D, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
        if (e != cudaSuccess) return ib::fail(IB_ERR_CUDA, "ib_chunk_scan: %s", cudaGetErrorString(e));
        set = true;
    }
    const int rc = ib::launch("chunk_scan_kernel", chunk_scan_kernel<D, NB>, grid, dim3(THREADS), smem, stream, 1u, qk, rows, ld, v_col,
                              aux, lda, b_col, lng_col, state, ones_state, seg_start, seg_slot, raw_out, ones_out, skip, n_heads, hpq, d, dv,
                              write_state, vec_v);
    return rc ? rc : ib::check_launch("ib_chunk_scan");
}

}  // namespace

// ================================================================================================
// C entry points.

// The largest key size of a head.
IB_EXPORT int ib_chunk_scan_max_dim() { return 128; }

// bfloat16 elements of workspace that ib_chunk_scan needs for n_tokens tokens.
IB_EXPORT int64_t ib_chunk_scan_workspace(int64_t n_tokens, int n_heads, int heads_per_qk, int d) {
    return n_tokens * 2 * (n_heads / heads_per_qk) * (d <= 64 ? 64 : 128);
}

// Float rows: q and k of head h / heads_per_qk at q_col, k_col + that * d, v at v_col + h dv; aux rows: strengths at b_col + h, ln g
// at lng_col + h. state [slots, H, d, dv]; with ones_state [slots, H, d] and ones_out [tokens, H] a column of ones beside
// the values; skip [H] (null: none). raw_out [tokens, H, dv]. qk: workspace as ib_chunk_scan_workspace says.
IB_EXPORT int ib_chunk_scan(const float* rows, int64_t ld, int q_col, int k_col, int v_col, const float* aux, int64_t lda, int b_col,
                            int lng_col, float* state, float* ones_state, const int* seg_start, const int* seg_slot, float* raw_out,
                            float* ones_out, const float* skip, int n_segments, int n_heads, int heads_per_qk, int d, int dv,
                            int write_state, int sm_count, void* qk, int64_t n_tokens, cudaStream_t stream) {
    if (n_segments <= 0) return IB_OK;
    if (n_heads <= 0 || n_heads > 65535 || heads_per_qk <= 0 || n_heads % heads_per_qk || d <= 0 || d > 128 || dv <= 0)
        return ib::fail(IB_ERR_ARG, "ib_chunk_scan: %d heads with a state of %d x %d", n_heads, d, dv);
    if (!qk || (uintptr_t(qk) & 15) || n_tokens <= 0) return ib::fail(IB_ERR_ARG, "ib_chunk_scan: a workspace is needed");
    if (ones_state && !ones_out) return ib::fail(IB_ERR_ARG, "ib_chunk_scan: a column of ones needs a result of its own");
    const int columns = dv + (ones_state ? 1 : 0);
    const int64_t sms = sm_count > 0 ? sm_count : 148;
    const auto ctas = [&](int nb) { return int64_t(n_segments) * n_heads * ((columns + nb - 1) / nb); };
    const int nb = ctas(16) <= sms || columns <= 16 ? 16 : 32;
    const int vec_v = dv % 4 == 0 && ld % 4 == 0 && v_col % 4 == 0 && !((uintptr_t(rows) | uintptr_t(raw_out)) & 15);
    const int D = d <= 64 ? 64 : 128, n_qk = n_heads / heads_per_qk;
    const int prc = ib::launch("pack_qk_kernel", pack_qk_kernel, dim3(unsigned(n_tokens)), dim3(256), 0, stream, 1u, rows, ld, q_col, k_col, n_qk, d, D, (bf16*)qk);
    if (prc) return prc;
    const dim3 grid{unsigned(n_segments), unsigned(n_heads), unsigned((columns + nb - 1) / nb)};
#define IB_CHUNK(DD, NN)                                                                                                             \
    return launch_chunk<DD, NN>(grid, stream, (const bf16*)qk, rows, ld, v_col, aux, lda, b_col, lng_col, state, ones_state, seg_start, \
                                seg_slot, raw_out, ones_out, skip, n_heads, heads_per_qk, d, dv, write_state, vec_v)
    if (d <= 64) {
        if (nb == 16) IB_CHUNK(64, 16);
        IB_CHUNK(64, 32);
    }
    if (nb == 16) IB_CHUNK(128, 16);
    IB_CHUNK(128, 32);
#undef IB_CHUNK
}
