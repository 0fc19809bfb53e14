// The batched path's matrix products in true fp32: out[t, n] = epilogue(sum_k X[t,k] * W[n,k]) with fp32 activations,
// bf16 weights widened exactly, fp32 FMA on the CUDA cores, the same call structure as the tensor-core GEMM
// (gemm_tc.cu) so that a session that computes in fp32 runs the same sequence of steps. One CTA = 64 tokens x 64
// weight rows, K in slices of 16 through shared memory, 4 x 4 outputs per thread.
#include "kernels.h"
#include "ptx.cuh"
#include "launch.h"
#include <cstring>

namespace tffn {

namespace {

constexpr int TB = kGemmF32Tile, NB = 64, KB = 16;

struct F32Dev {
    const float* X[2];
    const bf16* W[2];
    float* out[2];
    long long ldx[2], ldw[2], ldo;
    int N, T, K, mode;
    float out_scale;
    const GroupTile* grp;
    unsigned long long* tl;
};

__global__ void __launch_bounds__(256) k_gemm_f32(const F32Dev p) {
    __shared__ float sx[KB][TB + 4];
    __shared__ float sw[KB][NB + 4];
    if (threadIdx.x == 0) tl_mark(p.tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(p.tl, 1);
    const int prob = blockIdx.z, n0 = blockIdx.x * NB;
    int t0 = blockIdx.y * TB, t_end = p.T;
    long long w_row0 = 0;
    if (p.grp) {
        const int4 g = __ldcg((const int4*)(p.grp + blockIdx.y));
        if (g.x < 0) return;
        t0 = g.y;
        t_end = min(g.z, g.y + TB);
        w_row0 = (long long)g.x * p.N;
    }
    const float* X = p.X[prob];
    const bf16* W = p.W[prob];
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;  // tx: weight rows, ty: tokens
    const int lk = tid & 15, lr = tid >> 4;                     // copies: k within the slice, first row (then + 16 ...)
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += KB) {
        const int k = k0 + lk;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = t0 + lr + 16 * i, n = n0 + lr + 16 * i;
            sx[lk][lr + 16 * i] = (t < t_end && k < p.K) ? __ldcg(X + (size_t)t * p.ldx[prob] + k) : 0.f;
            sw[lk][lr + 16 * i] = (n < p.N && k < p.K) ? __bfloat162float(W[(size_t)(w_row0 + n) * p.ldw[prob] + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < KB; ++kk) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = sx[kk][ty * 4 + i];
                b[i] = sw[kk][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= t_end) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= p.N) continue;
            float v = acc[i][j] * p.out_scale;
            if (p.mode == GEMM_RELU2) {
                v = fmaxf(v, 0.f);
                v *= v;
            }
            p.out[prob][(size_t)t * p.ldo + n] = v;
        }
    }
    if (tid == 0) tl_mark(p.tl, 2);
}

}  // namespace

int launch_gemm_f32(const GemmCall& c, cudaStream_t stream) {
    if (c.T <= 0 || c.N <= 0 || c.op[0].K <= 0 || !c.out || c.op[1].K > 0) return (int)cudaErrorInvalidValue;
    if (c.mode != GEMM_STORE_F32 && c.mode != GEMM_STORE_BF16 && c.mode != GEMM_RELU2) return (int)cudaErrorInvalidValue;
    if (c.out2 && (c.op2[0].K != c.op[0].K || c.op2[1].K > 0 || c.grp)) return (int)cudaErrorInvalidValue;
    if (c.grp && (c.grp_bn != TB || c.grp_tiles < 1)) return (int)cudaErrorInvalidValue;
    F32Dev p;
    memset(&p, 0, sizeof p);
    p.X[0] = (const float*)c.op[0].X;
    p.W[0] = c.op[0].W;
    p.ldx[0] = c.op[0].ldx;
    p.ldw[0] = c.op[0].ldw;
    p.out[0] = (float*)c.out;
    if (c.out2) {
        p.X[1] = (const float*)c.op2[0].X;
        p.W[1] = c.op2[0].W;
        p.ldx[1] = c.op2[0].ldx;
        p.ldw[1] = c.op2[0].ldw;
        p.out[1] = (float*)c.out2;
    }
    p.ldo = c.ldo;
    p.N = c.N;
    p.T = c.T;
    p.K = c.op[0].K;
    p.mode = c.mode;
    p.out_scale = c.out_scale == 0.f ? 1.f : c.out_scale;
    p.grp = c.grp;
    p.tl = c.tl;
    const dim3 grid((c.N + NB - 1) / NB, c.grp ? c.grp_tiles : (c.T + TB - 1) / TB, c.out2 ? 2 : 1);
    return (int)launch_k(k_gemm_f32, grid, dim3(256), 0, stream, c.pdl, p);
}

}  // namespace tffn
