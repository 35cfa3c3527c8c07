// Around the grouped products of routed feed-forwards (gemm_tcgen05.cu, ib_gemm_tc_grouped): the rows of a step that an expert was
// chosen for lie side by side, each expert's padded to whole tiles of TILE rows, so that a prompt's tokens go through the
// chosen experts only.
#include "common.cuh"

IB_DEFINE_LAST_ERROR()

#define IB_LAUNCH(kernel, grid, block, smem, ...)                                                              \
    do {                                                                                                       \
        const int rc_ = ib::launch(#kernel, kernel, dim3(grid), dim3(block), size_t(smem), stream, 1u, __VA_ARGS__); \
        if (rc_) return rc_;                                                                                   \
    } while (0)

namespace {

using bf16 = __nv_bfloat16;
constexpr int TILE = 128;

// chosen [tokens, top] (-1: none), weights [tokens, experts] -> place [tokens * top]: where the (token, choice) pair's row lies;
// row_of [tiles * TILE]: the token of a row, -1 in an expert's padding; scale_of: the token's weight for that expert;
// tiles: [0] the number of tiles in use, [1 + i] the expert of tile i. One CTA. In which order an expert's rows lie does not
// matter: a product's row depends on its own operand row only.
__global__ void __launch_bounds__(1024)
group_rows_kernel(const int* __restrict__ chosen, const float* __restrict__ weights, int n_pairs, int top, int n_experts,
                  int* __restrict__ place, int* __restrict__ row_of, float* __restrict__ scale_of, int* __restrict__ tiles) {
    extern __shared__ int sm[];
    int* count = sm;                         // [experts]
    int* start = sm + n_experts;             // [experts + 1], in tiles
    ib::pdl_wait();
    const int tid = threadIdx.x;
    for (int e = tid; e < n_experts; e += blockDim.x) count[e] = 0;
    __syncthreads();
    for (int i = tid; i < n_pairs; i += blockDim.x) {
        const int e = chosen[i];
        place[i] = e >= 0 ? atomicAdd(&count[e], 1) : -1;
    }
    __syncthreads();
    if (tid == 0) {
        int at = 0;
        for (int e = 0; e < n_experts; e++) {
            start[e] = at;
            at += (count[e] + TILE - 1) / TILE;
        }
        start[n_experts] = at;
        tiles[0] = at;
    }
    __syncthreads();
    for (int e = tid >> 5; e < n_experts; e += blockDim.x >> 5) {           // a warp per expert: its tiles and its padding
        for (int i = start[e] + (tid & 31); i < start[e + 1]; i += 32) tiles[1 + i] = e;
        for (int r = start[e] * TILE + count[e] + (tid & 31); r < start[e + 1] * TILE; r += 32) {
            row_of[r] = -1;
            scale_of[r] = 0.0f;
        }
    }
    for (int i = tid; i < n_pairs; i += blockDim.x) {
        const int e = chosen[i];
        if (e < 0) continue;
        const int r = start[e] * TILE + place[i], t = i / top;
        place[i] = r;
        row_of[r] = t;
        scale_of[r] = weights[int64_t(t) * n_experts + e];
    }
}

// out[r] = x[row_of[r]] for the rows of tiles in use (zeros in the padding); width8: 16-byte pieces of a row.
__global__ void __launch_bounds__(128)
gather_rows_kernel(const uint4* __restrict__ x, const int* __restrict__ row_of, const int* __restrict__ tiles, uint4* __restrict__ out, int width8) {
    ib::pdl_wait();
    const int r = blockIdx.x;
    if (r >= tiles[0] * TILE) return;
    const int t = row_of[r];
    for (int i = threadIdx.x; i < width8; i += blockDim.x)
        out[int64_t(r) * width8 + i] = t >= 0 ? x[int64_t(t) * width8 + i] : make_uint4(0u, 0u, 0u, 0u);
}

// out[t] = (residual[t] +) the sum of the token's rows y[place[t, j]], j ascending; width4: four floats a piece.
__global__ void __launch_bounds__(256)
combine_rows_kernel(const float4* __restrict__ y, const int* __restrict__ place, int top, const float4* residual, float4* out, int width4) {
    ib::pdl_wait();
    const int64_t t = blockIdx.x;
    for (int i = threadIdx.x; i < width4; i += blockDim.x) {
        float4 s = residual ? residual[t * width4 + i] : make_float4(0.f, 0.f, 0.f, 0.f);
        for (int j = 0; j < top; j++) {
            const int r = place[t * top + j];
            if (r < 0) continue;
            const float4 v = y[int64_t(r) * width4 + i];
            s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
        }
        out[t * width4 + i] = s;
    }
}

}  // namespace

// ================================================================================================
// C entry points.

IB_EXPORT int ib_group_tile_rows() { return TILE; }

IB_EXPORT int ib_group_rows(const int* chosen, const float* weights, int64_t n_tokens, int top, int n_experts, int* place, int* row_of,
                            float* scale_of, int* tiles, cudaStream_t stream) {
    if (n_tokens <= 0) return IB_OK;
    if (top <= 0 || n_experts <= 0 || n_experts > 4096 || n_tokens * top > (1LL << 30)) return ib::fail(IB_ERR_ARG, "ib_group_rows: %d of %d experts", top, n_experts);
    IB_LAUNCH(group_rows_kernel, 1u, 1024, size_t(2 * n_experts + 1) * sizeof(int), chosen, weights, int(n_tokens * top), top, n_experts, place,
              row_of, scale_of, tiles);
    return ib::check_launch("ib_group_rows");
}

IB_EXPORT int ib_gather_rows(const void* x, const int* row_of, const int* tiles, void* out, int64_t max_rows, int64_t row_bytes, cudaStream_t stream) {
    if (max_rows <= 0 || row_bytes <= 0) return IB_OK;
    if (row_bytes % 16 || ((uintptr_t(x) | uintptr_t(out)) & 15)) return ib::fail(IB_ERR_ARG, "ib_gather_rows: rows must be whole 16-byte pieces");
    IB_LAUNCH(gather_rows_kernel, unsigned(max_rows), 128, 0, (const uint4*)x, row_of, tiles, (uint4*)out, int(row_bytes / 16));
    return ib::check_launch("ib_gather_rows");
}

IB_EXPORT int ib_combine_rows(const float* y, const int* place, int top, const float* residual, float* out, int64_t n_tokens, int64_t width,
                              cudaStream_t stream) {
    if (n_tokens <= 0 || width <= 0) return IB_OK;
    if (width % 4 || ((uintptr_t(y) | uintptr_t(residual) | uintptr_t(out)) & 15)) return ib::fail(IB_ERR_ARG, "ib_combine_rows: rows must be whole 16-byte pieces");
    IB_LAUNCH(combine_rows_kernel, unsigned(n_tokens), 256, 0, (const float4*)y, place, top, (const float4*)residual, (float4*)out, int(width / 4));
    return ib::check_launch("ib_combine_rows");
}
