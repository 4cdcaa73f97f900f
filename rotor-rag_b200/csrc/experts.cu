// Routing of many tokens to their experts: choice and weights, slots grouped by expert, the table of token
// tiles the expert products walk, and the copy of the rows into their slots.  (Up to DENSE_FEW_ROWS tokens
// need none of this: the matrix-vector products choose for themselves.)
#include "decoder.cuh"

namespace rb {

// One warp per row: choices, weights, and how many rows each expert gets.
__global__ void __launch_bounds__(256) route_choose_kernel(const __grid_constant__ Routing r, int rows) {
    __shared__ int hist[EXPERTS_MAX];
    for (int e = threadIdx.x; e < r.experts; e += blockDim.x) hist[e] = 0;
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const int lane = threadIdx.x & 31, per = blockDim.x >> 5;
    for (int row = blockIdx.x * per + (threadIdx.x >> 5); row < rows; row += gridDim.x * per) {
        int sel;
        float w;
        route_row(r, row, lane, sel, w);
        if (lane < r.top) {
            r.chosen[(size_t)row * r.top + lane] = sel;
            r.weight[(size_t)row * r.top + lane] = w;
            atomicAdd(&hist[sel], 1);
        }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < r.experts; e += blockDim.x)
        if (hist[e]) atomicAdd(&r.counts[e], hist[e]);
}

// One CTA of EXPERTS_MAX threads: first slot of every expert, the tile table; counts are zeroed for the next call.
__global__ void __launch_bounds__(EXPERTS_MAX) route_table_kernel(const __grid_constant__ Routing r, int pairs) {
    __shared__ int2 warp_sums[32];
    pdl_wait();
    pdl_trigger();
    const int e = threadIdx.x, lane = e & 31, warp = e >> 5;
    const int n = e < r.experts ? min(max(r.counts[e], 0), pairs) : 0, tiles = (n + r.tile_rows - 1) / r.tile_rows;
    int2 s = make_int2(n, tiles);  // inclusive sums
    auto scan = [&]() {
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int a = __shfl_up_sync(0xffffffffu, s.x, o), b = __shfl_up_sync(0xffffffffu, s.y, o);
            if (lane >= o) {
                s.x += a;
                s.y += b;
            }
        }
    };
    scan();
    if (lane == 31) warp_sums[warp] = s;
    __syncthreads();
    const int2 own = s;
    if (warp == 0) {
        s = warp_sums[lane];
        scan();
        warp_sums[lane] = s;
    }
    __syncthreads();
    int first = own.x - n, tile = own.y - tiles;
    if (warp > 0) {
        first += warp_sums[warp - 1].x;
        tile += warp_sums[warp - 1].y;
    }
    if (e < r.experts) {
        r.cursor[e] = first;
        r.counts[e] = 0;
        for (int t = 0; t < tiles && tile + t < r.max_tiles && first + t * r.tile_rows < pairs; ++t) {
            int* out = r.table + 1 + 3 * (tile + t);
            out[0] = e;
            out[1] = first + t * r.tile_rows;
            out[2] = min(min(r.tile_rows, n - t * r.tile_rows), pairs - out[1]);
        }
    }
    if (e == 0) r.table[0] = min(warp_sums[31].y, r.max_tiles);
}

// One warp per row: takes the next slot of each of its experts and copies the row there, read once.
__global__ void __launch_bounds__(256) route_scatter_kernel(const __grid_constant__ Routing r, int rows, const uint4* x, int pieces, uint4* permuted) {
    pdl_wait();
    pdl_trigger();
    const int lane = threadIdx.x & 31, per = blockDim.x >> 5, pairs = rows * r.top;
    constexpr int U = 4;  // pieces per lane requested together
    for (int row = blockIdx.x * per + (threadIdx.x >> 5); row < rows; row += gridDim.x * per) {
        const uint4* src = x + (size_t)row * pieces;
        uint4 v[U];
        auto fetch = [&](int c0) {
#pragma unroll
            for (int u = 0; u < U; ++u)
                if (c0 + 32 * u + lane < pieces) v[u] = __ldg(src + c0 + 32 * u + lane);
        };
        fetch(0);
        int slot = 0;
        if (lane < r.top) {
            slot = min(max(atomicAdd(&r.cursor[r.chosen[(size_t)row * r.top + lane]], 1), 0), pairs - 1);
            r.slot_of[(size_t)row * r.top + lane] = slot;
        }
        for (int c0 = 0; c0 < pieces; c0 += 32 * U) {
            if (c0) fetch(c0);
            for (int k = 0; k < r.top; ++k) {
                uint4* dst = permuted + (size_t)__shfl_sync(0xffffffffu, slot, k) * pieces;
#pragma unroll
                for (int u = 0; u < U; ++u)
                    if (c0 + 32 * u + lane < pieces) dst[c0 + 32 * u + lane] = v[u];
            }
        }
    }
}

int launch_route(const Routing& r, int rows, const void* x, size_t row_bytes, void* permuted, cudaStream_t st) {
    RB_REQUIRE(r.logits && r.slot_of && r.weight && r.chosen && r.counts && r.cursor && r.table && x && permuted && rows > 0);
    RB_REQUIRE(r.experts >= 1 && r.experts <= EXPERTS_MAX && r.top >= 1 && r.top <= r.experts && r.top <= EXPERT_TOP_MAX);
    RB_REQUIRE(row_bytes % 16 == 0 && (long long)rows * r.top < 0x7fffffffLL);
    const int pairs = rows * r.top, most = 148 * 8;
    RB_REQUIRE(r.max_tiles >= route_tiles(pairs, r.experts, r.tile_rows));
    int rc = launch_chained(route_choose_kernel, dim3((rows + 7) / 8 < most ? (rows + 7) / 8 : most), dim3(256), 0, st, 1, r, rows);
    if (!rc) rc = launch_chained(route_table_kernel, dim3(1), dim3(EXPERTS_MAX), 0, st, 1, r, pairs);
    if (!rc)
        rc = launch_chained(route_scatter_kernel, dim3((rows + 7) / 8 < most ? (rows + 7) / 8 : most), dim3(256), 0, st, 1, r, rows,
                            static_cast<const uint4*>(x), (int)(row_bytes / 16), static_cast<uint4*>(permuted));
    return rc;
}

}  // namespace rb
