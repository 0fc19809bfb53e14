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
    int N, T, K[2], mode, batch, x_batch, out_batch;
    float out_scale, alpha;
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
    const int b = p.batch > 1 ? prob : 0;  // batched: the problems share their operands
    if (b > 0) w_row0 = (long long)b * p.N;
    const int op0 = p.batch > 1 ? 0 : prob;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;  // tx: weight rows, ty: tokens
    const int lk = tid & 15, lr = tid >> 4;                     // copies: k within the slice, first row (then + 16 ...)
    float acc[4][4], first[4][4];  // first: the first operand pair's sums while the second one's are formed
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = first[i][j] = 0.f;
    const int pairs = p.K[1] > 0 ? 2 : 1;
    for (int pair = 0; pair < pairs; ++pair) {
        const int op = op0 + pair, K = p.K[pair];
        const float* X = p.X[op] + (size_t)b * p.x_batch;
        const bf16* W = p.W[op];
        const long long ldx = p.ldx[op], ldw = p.ldw[op];
        if (pair == 1) {
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    first[i][j] = acc[i][j];
                    acc[i][j] = 0.f;
                }
        }
        for (int k0 = 0; k0 < K; k0 += KB) {
            const int k = k0 + lk;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int t = t0 + lr + 16 * i, n = n0 + lr + 16 * i;
                sx[lk][lr + 16 * i] = (t < t_end && k < K) ? __ldcg(X + (size_t)t * ldx + k) : 0.f;
                sw[lk][lr + 16 * i] = (n < p.N && k < K) ? __bfloat162float(W[(size_t)(w_row0 + n) * ldw + k]) : 0.f;
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
    }
    float* out = p.batch > 1 ? p.out[0] + (size_t)b * p.out_batch : p.out[prob];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = t0 + ty * 4 + i;
        if (t >= t_end) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= p.N) continue;
            float v = acc[i][j];
            if (pairs == 2) v = p.mode == GEMM_SWIGLU ? first[i][j] / (1.f + expf(-first[i][j])) * v : first[i][j] + p.alpha * v;
            v *= p.out_scale;
            if (p.mode == GEMM_RELU2) {
                v = fmaxf(v, 0.f);
                v *= v;
            }
            out[(size_t)t * p.ldo + n] = v;
        }
    }
    if (tid == 0) tl_mark(p.tl, 2);
}

}  // namespace

int launch_gemm_f32(const GemmCall& c, cudaStream_t stream) {
    if (c.T <= 0 || c.N <= 0 || c.op[0].K <= 0 || !c.out) return (int)cudaErrorInvalidValue;
    if (c.mode != GEMM_STORE_F32 && c.mode != GEMM_STORE_BF16 && c.mode != GEMM_RELU2 && c.mode != GEMM_SWIGLU) return (int)cudaErrorInvalidValue;
    if (c.mode == GEMM_SWIGLU ? c.op[1].K != c.op[0].K : c.mode == GEMM_RELU2 && c.op[1].K > 0) return (int)cudaErrorInvalidValue;
    if (c.op[1].K > 0 && (c.out2 || c.grp || c.batch > 1)) return (int)cudaErrorInvalidValue;
    if (c.batch > 1 && (c.out2 || c.grp || (c.mode != GEMM_STORE_F32 && c.mode != GEMM_STORE_BF16))) return (int)cudaErrorInvalidValue;
    if (c.out2 && (c.op2[0].K != c.op[0].K || c.op2[1].K > 0 || c.grp)) return (int)cudaErrorInvalidValue;
    if (c.grp && (c.grp_bn != TB || c.grp_tiles < 1)) return (int)cudaErrorInvalidValue;
    F32Dev p;
    memset(&p, 0, sizeof p);
    p.X[0] = (const float*)c.op[0].X;
    p.W[0] = c.op[0].W;
    p.ldx[0] = c.op[0].ldx;
    p.ldw[0] = c.op[0].ldw;
    p.out[0] = (float*)c.out;
    if (c.op[1].K > 0) {
        p.X[1] = (const float*)c.op[1].X;
        p.W[1] = c.op[1].W;
        p.ldx[1] = c.op[1].ldx;
        p.ldw[1] = c.op[1].ldw;
    }
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
    p.K[0] = c.op[0].K;
    p.K[1] = c.op[1].K;
    p.alpha = c.alpha;
    p.batch = c.batch > 1 ? c.batch : 1;
    p.x_batch = c.x_batch;
    p.out_batch = c.out_batch;
    p.mode = c.mode;
    p.out_scale = c.out_scale == 0.f ? 1.f : c.out_scale;
    p.grp = c.grp;
    p.tl = c.tl;
    const dim3 grid((c.N + NB - 1) / NB, c.grp ? c.grp_tiles : (c.T + TB - 1) / TB, c.out2 ? 2 : p.batch);
    return (int)launch_k(k_gemm_f32, grid, dim3(256), 0, stream, c.pdl, p);
}

}  // namespace tffn
