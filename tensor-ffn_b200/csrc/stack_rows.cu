// Row kernels of the layers that keep the residual stream in fp32 and norm a sublayer's output before adding it:
// one pass per sublayer does the norm of the output, the residual add and the norm in front of the next sublayer
// (the expert sum of a mixture as well), another one turns a projection's q|k|v rows into rotated queries and
// cache rows.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"

namespace tffn {

namespace {

template <typename A>
__global__ void __launch_bounds__(512) k_residual_rows(const ResidualRows a, unsigned long long* tl) {
    extern __shared__ float rows_smem[];
    __shared__ float red[32];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int H = a.H, r = blockIdx.x, n = blockDim.x, tid = threadIdx.x;
    float* xs = rows_smem;      // [H] the row of the residual stream
    float* ds = rows_smem + H;  // [H] the sublayer's output (ROWS_DELTA, ROWS_MOE)
    const int src = (a.source == ROWS_KEEP && a.row_idx) ? __ldcg(a.row_idx + r) : r;
    float* xr = a.x + (size_t)src * H;
    A* out = (A*)a.out + (size_t)r * a.out_ld;
    float ss = 0.f;
    if (a.source == ROWS_EMBED) {
        int tok = __ldcg(a.tokens + r);
        if (tok < 0 || tok >= a.V) {
            if (tid == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
            tok = 0;
        }
        const bf16* e = a.table + (size_t)tok * a.table_ld;
#pragma unroll 4
        for (int i = tid; i < H; i += n) {
            const float v = __bfloat162float(e[i]);
            xs[i] = v;
            xr[i] = v;
            ss += v * v;
        }
    } else if (a.source == ROWS_KEEP) {
#pragma unroll 4
        for (int i = tid; i < H; i += n) {
            const float v = __ldcg(xr + i);
            xs[i] = v;
            ss += v * v;
        }
    } else {
        float sd = 0.f;
        if (a.source == ROWS_DELTA) {
            const float* d = a.delta + (size_t)r * a.delta_ld;
#pragma unroll 4
            for (int i = tid; i < H; i += n) {
                const float v = __ldcg(d + i);
                xs[i] = __ldcg(xr + i);
                ds[i] = v;
                sd += v * v;
            }
        } else {
            const int* pr = a.pair_row + (size_t)r * a.top;
            const float* pw = a.pair_w + (size_t)r * a.top;
            for (int i = tid; i < H; i += n) {
                xs[i] = __ldcg(xr + i);
                float v = 0.f;
#pragma unroll 4
                for (int j = 0; j < a.top; ++j) {
                    const int row = __ldcg(pr + j);
                    const A* src_row = row < 0 ? out : (const A*)a.y + (size_t)row * a.y_ld;
                    v += __ldcg(pw + j) * act_load(src_row + i);
                }
                ds[i] = v;
                sd += v * v;
            }
        }
        sd = block_sum(sd, red);
        const float dinv = 1.f / sqrtf(sd / (float)H + a.eps);
#pragma unroll 4
        for (int i = tid; i < H; i += n) {  // each thread revisits only what it wrote itself
            const float v = xs[i] + ds[i] * dinv * __ldg(a.post_w + i);
            xs[i] = v;
            xr[i] = v;
            ss += v * v;
        }
    }
    if (a.next_w) {
        ss = block_sum(ss, red);
        const float inv = 1.f / sqrtf(ss / (float)H + a.eps);
#pragma unroll 4
        for (int i = tid; i < H; i += n) act_store(out + i, xs[i] * inv * __ldg(a.next_w + i));
    }
    if (tid == 0) tl_mark(tl, 2);
}

// one warp per (token, head): heads 0 .. nh-1 are queries, then the keys, then the values
constexpr int kQkWarps = 4;
template <typename A>
__global__ void __launch_bounds__(kQkWarps * 32) k_qk_norm_rope(const QkNormRope a, int T, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * kQkWarps + (threadIdx.x >> 5);
    const int nkv = a.kv.nkv, per_tok = a.nh + 2 * nkv;
    if (unit < (long long)T * per_tok) {
        const int t = (int)(unit / per_tok), u = (int)(unit % per_tok);
        const int kind = u < a.nh ? 0 : (u < a.nh + nkv ? 1 : 2);
        const int head = kind == 0 ? u : (kind == 1 ? u - a.nh : u - a.nh - nkv);
        const int dim = kind == 2 ? a.vdim : a.dim;
        const A* src = (const A*)a.qkv + (size_t)t * a.ld + (kind == 0 ? 0 : (kind == 1 ? a.k_off : a.v_off)) + (size_t)head * dim;
        const int pos = __ldcg(a.tok_pos + t), seq = __ldcg(a.tok_seq + t);
        const bool pos_ok = pos >= 0 && pos < a.max_pos;
        const int pg = (kind != 0 && pos_ok) ? __ldcg(a.kv.block_table + (size_t)seq * a.kv.max_pages_per_seq + pos / kPageTokens) : 0;
        if (!pos_ok || (kind != 0 && (pg < 0 || pg >= a.kv.num_pages))) {
            if (lane == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        } else if (kind == 2) {
            A* dst = (A*)a.kv.v_pool + (((size_t)pg * nkv + head) * kPageTokens + pos % kPageTokens) * a.kv.vd;
            for (int i = lane; i < dim; i += 32) act_store(dst + i, act_load(src + i));
        } else {
            // lane = pair (2i, 2i + 1)
            constexpr int MP = 8;  // heads of up to 512
            float u0[MP], u1[MP], ss = 0.f;
#pragma unroll
            for (int j = 0; j < MP; ++j) {
                const int i = 2 * (lane + 32 * j);
                u0[j] = i < dim ? act_load(src + i) : 0.f;
                u1[j] = i + 1 < dim ? act_load(src + i + 1) : 0.f;
                ss += u0[j] * u0[j] + u1[j] * u1[j];
            }
            const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
            const float* w = kind == 0 ? a.q_norm : a.k_norm;
            float* qd = a.q_out + ((size_t)t * a.nh + head) * a.kv.hd;
            A* kdst = (A*)a.kv.k_pool + (((size_t)pg * nkv + head) * kPageTokens + pos % kPageTokens) * a.kv.hd;
#pragma unroll
            for (int j = 0; j < MP; ++j) {
                const int p = lane + 32 * j, i = 2 * p;
                if (i < a.kv.hd) {
                    float x = i < dim ? u0[j] * inv * __ldg(w + i) : 0.f, y = i + 1 < dim ? u1[j] * inv * __ldg(w + i + 1) : 0.f;
                    if (i < a.rope_dims) {
                        const float2 cs = __ldg(a.rope + (size_t)pos * (a.rope_dims / 2) + p);
                        const float xr = x * cs.x - y * cs.y, yr = y * cs.x + x * cs.y;
                        x = xr;
                        y = yr;
                    }
                    if (kind == 0) {
                        *(float2*)(qd + i) = make_float2(x, y);
                    } else {
                        act_store(kdst + i, x);
                        act_store(kdst + i + 1, y);
                    }
                }
            }
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

constexpr int kRowsMaxSmem = 128 * 1024;

}  // namespace

int stack_rows_prepare() {
    cudaError_t e = cudaFuncSetAttribute(k_residual_rows<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRowsMaxSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k_residual_rows<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRowsMaxSmem);
    if (e == cudaSuccess) e = prefer_max_shared(k_residual_rows<bf16>);
    if (e == cudaSuccess) e = prefer_max_shared(k_residual_rows<float>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<bf16>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<float>);
    return (int)e;
}

void launch_residual_rows(const ResidualRows& a, bool f32, int rows, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const int threads = a.H <= 512 ? 128 : (a.H <= 2048 ? 256 : 512);
    const size_t smem = (size_t)a.H * 8;
    if (f32) launch_k(k_residual_rows<float>, dim3(rows), dim3(threads), smem, s, pdl, a, tl);
    else launch_k(k_residual_rows<bf16>, dim3(rows), dim3(threads), smem, s, pdl, a, tl);
}

void launch_qk_norm_rope(const QkNormRope& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const long long units = (long long)T * (a.nh + 2 * a.kv.nkv);
    const dim3 grid((unsigned)((units + kQkWarps - 1) / kQkWarps)), block(kQkWarps * 32);
    if (f32) launch_k(k_qk_norm_rope<float>, grid, block, 0, s, pdl, a, T, tl);
    else launch_k(k_qk_norm_rope<bf16>, grid, block, 0, s, pdl, a, T, tl);
}

}  // namespace tffn
