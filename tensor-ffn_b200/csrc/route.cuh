// The choice of experts for one token by one warp, shared by the stand-alone router kernel and the row kernel that
// routes in the same pass.
#pragma once
#include "act.cuh"
#include "ptx.cuh"

namespace tffn {

// s[0 .. n): the token's logits in shared memory, n = experts + identity (overwritten with the softmax scores);
// choice[0 .. n): scratch. The lanes own strided entries.
__device__ __forceinline__ void route_token(const MoeRoute& a, int t, float* s, float* choice, int lane) {
    const int n = a.experts + a.identity;
    float mx = -INFINITY;
    for (int i = lane; i < n; i += 32) mx = fmaxf(mx, s[i]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
    for (int i = lane; i < n; i += 32) {
        const float e = expf(s[i] - mx);
        s[i] = e;
        sum += e;
    }
    const float inv = 1.f / warp_sum(sum);
    for (int i = lane; i < n; i += 32) {
        s[i] *= inv;
        choice[i] = s[i] + __ldg(a.correction + i);
    }
    int mine[2] = {-1, -1};  // lane j keeps choices j and 32 + j (top <= 64)
    for (int j = 0; j < a.top; ++j) {
        float best = -INFINITY;
        int bi = 0x7fffffff;
        for (int i = lane; i < n; i += 32)
            if (choice[i] > best) { best = choice[i]; bi = i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        if (bi >= n) bi = j;  // no finite score is left (NaN inputs): stay in range
        if ((bi & 31) == lane) choice[bi] = -INFINITY;
        if ((j & 31) == lane) mine[j >> 5] = bi;
    }
    __syncwarp();  // every lane's scores are visible
    // places within the experts: the choices' atomics in flight together
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int j = k * 32 + lane;
        if (j < a.top) {
            const int bi = mine[k];
            int2 p = make_int2(-1, 0);
            if (bi < a.experts) p = make_int2(bi, atomicAdd(a.counts + bi, 1));
            a.pair[(size_t)t * a.top + j] = p;
            a.pair_w[(size_t)t * a.top + j] = s[bi];
        }
    }
}

}  // namespace tffn
