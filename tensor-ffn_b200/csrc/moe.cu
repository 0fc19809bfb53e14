// Mixture-of-experts routing: the router's fp32 logits -> chosen experts and weights per token, then the tokens' rows
// sorted by expert and the tile table of the grouped GEMMs. No host round trip: counts stay on the device and the
// grouped launches are sized for the worst case. The order of rows within an expert follows the arrival of atomics;
// it does not enter any value, since every row of a GEMM is computed independently of its place.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"
#include "route.cuh"

namespace tffn {

namespace {

constexpr int kRouteWarps = 4;

// one warp per token; scores in shared memory
__global__ void __launch_bounds__(kRouteWarps * 32) k_moe_route(const MoeRoute a, int T, unsigned long long* tl) {
    extern __shared__ float route_smem[];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = a.experts + a.identity;
    const int t = blockIdx.x * kRouteWarps + warp;
    if (t < T) {
        float* s = route_smem + (size_t)warp * 2 * n;
        const float* z = a.logits + (size_t)t * a.ld;
        for (int i = lane; i < n; i += 32) s[i] = __ldcg(z + i);
        route_token(a, t, s, s + n, lane);
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

// Block t copies token t's row to its places; the last block writes the tile table. Every block forms the prefix sums
// of the counts itself.
constexpr int kGatherThreads = 128;
template <typename A>
__global__ void __launch_bounds__(kGatherThreads) k_moe_gather(const MoeGather a, int T, unsigned long long* tl) {
    extern __shared__ int gather_smem[];
    int* first = gather_smem;                  // [experts] first sorted row of an expert
    int* tile0 = gather_smem + a.experts;      // [experts + 1] first tile (last block only)
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int tid = threadIdx.x, lane = tid & 31;
    const bool table = (int)blockIdx.x == T;
    int2 mine = make_int2(-1, 0);  // threads from 32 on: the token's pairs, requested before the prefix sums are formed
    const int jj = tid - 32;
    if (!table && jj >= 0 && jj < a.top) mine = __ldcg(a.pair + (size_t)blockIdx.x * a.top + jj);
    if (tid < 32) {
        int rows = 0, tiles = 0;
        for (int e0 = 0; e0 < a.experts; e0 += 32) {
            const int e = e0 + lane, c = e < a.experts ? __ldcg(a.counts + e) : 0;
            const int nt = (c + a.tile_rows - 1) / a.tile_rows;
            int ci = c, ti = nt;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int v = __shfl_up_sync(0xffffffffu, ci, o), w = __shfl_up_sync(0xffffffffu, ti, o);
                if (lane >= o) { ci += v; ti += w; }
            }
            if (e < a.experts) {
                first[e] = rows + ci - c;
                if (table) tile0[e] = tiles + ti - nt;
            }
            rows += __shfl_sync(0xffffffffu, ci, 31);
            tiles += __shfl_sync(0xffffffffu, ti, 31);
        }
        if (table && lane == 0) tile0[a.experts] = tiles;
    }
    __syncthreads();
    if (table) {
        for (int e = tid; e < a.experts; e += kGatherThreads) {
            const int row0 = first[e], end = row0 + __ldcg(a.counts + e);
            for (int i = tile0[e], r = row0; i < tile0[e + 1] && i < a.max_tiles; ++i, r += a.tile_rows)
                a.tiles[i] = GroupTile{e, r, end, 0};
        }
        for (int i = tile0[a.experts] + tid; i < a.max_tiles; i += kGatherThreads) a.tiles[i] = GroupTile{-1, 0, 0, 0};
    } else {
        const int t = blockIdx.x;
        int* dest = tile0;  // [top], at most as many as threads 32 .. 127 (top <= 96)
        if (jj >= 0 && jj < a.top) {
            const int row = mine.x < 0 ? -1 : first[mine.x] + mine.y;
            a.pair_row[(size_t)t * a.top + jj] = row;
            dest[jj] = row;
        }
        const uint4* src = (const uint4*)((const A*)a.x + (size_t)t * a.x_ld);
        const int n16 = (int)(a.x_ld * sizeof(A) / 16);  // rows are padded to 16 bytes
        __syncthreads();
        for (int i = tid; i < n16; i += kGatherThreads) {
            const uint4 v = __ldcg(src + i);
            for (int j = 0; j < a.top; ++j)
                if (dest[j] >= 0) ((uint4*)((A*)a.xg + (size_t)dest[j] * a.x_ld))[i] = v;
        }
    }
    if (tid == 0) tl_mark(tl, 2);
}

}  // namespace

int moe_prepare() {
    cudaError_t e = prefer_max_shared(k_moe_route);
    if (e == cudaSuccess) e = prefer_max_shared(k_moe_gather<bf16>);
    if (e == cudaSuccess) e = prefer_max_shared(k_moe_gather<float>);
    return (int)e;
}

void launch_moe_route(const MoeRoute& a, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const size_t smem = (size_t)kRouteWarps * 2 * (a.experts + a.identity) * 4;
    launch_k(k_moe_route, dim3((T + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32), smem, s, pdl, a, T, tl);
}

void launch_moe_gather(const MoeGather& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const size_t smem = (size_t)(a.experts + (a.experts + 1 > a.top ? a.experts + 1 : a.top)) * 4;
    if (f32) launch_k(k_moe_gather<float>, dim3(T + 1), dim3(kGatherThreads), smem, s, pdl, a, T, tl);
    else launch_k(k_moe_gather<bf16>, dim3(T + 1), dim3(kGatherThreads), smem, s, pdl, a, T, tl);
}

}  // namespace tffn
