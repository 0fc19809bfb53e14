// Row kernels of the layers that keep the residual stream in fp32 and norm a sublayer's output before adding it:
// one pass per sublayer does the norm of the output, the residual add and the norm in front of the next sublayer
// (the expert sum of a mixture as well), another one turns a projection's q|k|v rows into rotated queries and
// cache rows.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"
#include "route.cuh"

namespace tffn {

namespace {

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 q = __ldcg((const float4*)p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&v)[4]) {
    const uint2 q = __ldcg((const uint2*)p);
    v[0] = bf16_lo(q.x); v[1] = bf16_hi(q.x); v[2] = bf16_lo(q.y); v[3] = bf16_hi(q.y);
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *(float4*)p = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16* p, const float (&v)[4]) {
    *(uint2*)p = make_uint2((uint32_t)bf16_bits(v[0]) | ((uint32_t)bf16_bits(v[1]) << 16),
                            (uint32_t)bf16_bits(v[2]) | ((uint32_t)bf16_bits(v[3]) << 16));
}
__device__ __forceinline__ float as_stored(float v, const float*) { return v; }
__device__ __forceinline__ float as_stored(float v, const bf16*) { return bf16_round(v); }

// The pass over rows whose width is a multiple of 4: a thread keeps its IT groups of four columns in registers from the
// first load to the last store, all loads of a phase in flight together.
template <typename A, int IT>
__global__ void __launch_bounds__(512) k_residual_rows4(const ResidualRows a, unsigned long long* tl) {
    extern __shared__ float rows4_smem[];  // with a router: the row as stored [H], logits [n], scratch [n]
    __shared__ float red[32];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int H = a.H, r = blockIdx.x, n = blockDim.x, tid = threadIdx.x;
    // norm weights do not depend on earlier kernels
    float pw[IT][4], nw[IT][4];
#pragma unroll
    for (int k = 0; k < IT; ++k) {
        const int i = (tid + k * n) * 4;
        if (i < H && a.post_w) load4(a.post_w + i, pw[k]);
        if (i < H && a.next_w) load4(a.next_w + i, nw[k]);
    }
    pdl_wait();
    if (tid == 0) tl_mark(tl, 1);
    const int src = (a.source == ROWS_KEEP && a.row_idx) ? __ldcg(a.row_idx + r) : r;
    float* xr = a.x + (size_t)src * H;
    A* out = (A*)a.out + (size_t)r * a.out_ld;
    float x[IT][4], ss = 0.f;
    if (a.source == ROWS_EMBED) {
        int tok = __ldcg(a.tokens + r);
        if (tok < 0 || tok >= a.V) {
            if (tid == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
            tok = 0;
        }
        const bf16* e = a.table + (size_t)tok * a.table_ld;
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (tid + k * n) * 4;
            if (i < H) load4(e + i, x[k]);
        }
        if (a.embed_w) {
            float se = 0.f;
#pragma unroll
            for (int k = 0; k < IT; ++k)
                if ((tid + k * n) * 4 < H) se += x[k][0] * x[k][0] + x[k][1] * x[k][1] + x[k][2] * x[k][2] + x[k][3] * x[k][3];
            const float einv = 1.f / sqrtf(block_sum(se, red) / (float)H + a.eps);
#pragma unroll
            for (int k = 0; k < IT; ++k) {
                const int i = (tid + k * n) * 4;
                if (i < H) {
                    float w[4];
                    load4(a.embed_w + i, w);
#pragma unroll
                    for (int c = 0; c < 4; ++c) x[k][c] *= einv * w[c];
                }
            }
        }
    } else {
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (tid + k * n) * 4;
            if (i < H) load4(xr + i, x[k]);
        }
    }
    if (a.source == ROWS_DELTA && !a.post_w) {
        float d[IT][4];
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (tid + k * n) * 4;
            if (i < H) load4(a.delta + (size_t)r * a.delta_ld + i, d[k]);
        }
#pragma unroll
        for (int k = 0; k < IT; ++k)
            if ((tid + k * n) * 4 < H) {
#pragma unroll
                for (int c = 0; c < 4; ++c) x[k][c] += a.delta_mult * d[k][c];
            }
    } else if (a.source >= ROWS_DELTA) {
        float d[IT][4], sd = 0.f;
        if (a.source == ROWS_DELTA) {
#pragma unroll
            for (int k = 0; k < IT; ++k) {
                const int i = (tid + k * n) * 4;
                if (i < H) load4(a.delta + (size_t)r * a.delta_ld + i, d[k]);
            }
        } else {
#pragma unroll
            for (int k = 0; k < IT; ++k) d[k][0] = d[k][1] = d[k][2] = d[k][3] = 0.f;
            for (int j0 = 0; j0 < a.top; j0 += 4) {
                const A* from[4];
                float w[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const bool on = j0 + j < a.top;
                    const int row = on ? __ldcg(a.pair_row + (size_t)r * a.top + j0 + j) : -1;
                    w[j] = on ? __ldcg(a.pair_w + (size_t)r * a.top + j0 + j) : 0.f;
                    from[j] = row < 0 ? out : (const A*)a.y + (size_t)row * a.y_ld;
                }
#pragma unroll
                for (int k = 0; k < IT; ++k) {
                    const int i = (tid + k * n) * 4;
                    if (i < H) {
                        float v[4][4];
#pragma unroll
                        for (int j = 0; j < 4; ++j) load4(from[j] + i, v[j]);
#pragma unroll
                        for (int j = 0; j < 4; ++j)
#pragma unroll
                            for (int c = 0; c < 4; ++c) d[k][c] += w[j] * v[j][c];
                    }
                }
            }
        }
#pragma unroll
        for (int k = 0; k < IT; ++k)
            if ((tid + k * n) * 4 < H) sd += d[k][0] * d[k][0] + d[k][1] * d[k][1] + d[k][2] * d[k][2] + d[k][3] * d[k][3];
        sd = block_sum(sd, red);
        const float dinv = 1.f / sqrtf(sd / (float)H + a.eps);
#pragma unroll
        for (int k = 0; k < IT; ++k)
            if ((tid + k * n) * 4 < H) {
#pragma unroll
                for (int c = 0; c < 4; ++c) x[k][c] += d[k][c] * dinv * pw[k][c];
            }
    }
#pragma unroll
    for (int k = 0; k < IT; ++k) {
        const int i = (tid + k * n) * 4;
        if (i < H) {
            if (a.source != ROWS_KEEP) store4(xr + i, x[k]);
            ss += x[k][0] * x[k][0] + x[k][1] * x[k][1] + x[k][2] * x[k][2] + x[k][3] * x[k][3];
        }
    }
    if (a.next_w) {
        ss = block_sum(ss, red);
        const float inv = 1.f / sqrtf(ss / (float)H + a.eps);
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (tid + k * n) * 4;
            if (i < H) {
                float v[4];
#pragma unroll
                for (int c = 0; c < 4; ++c) v[c] = x[k][c] * inv * nw[k][c];
                store4(out + i, v);
                if (a.next2_w) {
                    float w2[4], v2[4];
                    load4(a.next2_w + i, w2);
#pragma unroll
                    for (int c = 0; c < 4; ++c) v2[c] = x[k][c] * inv * w2[c];
                    store4((A*)a.out2 + (size_t)r * a.out_ld + i, v2);
                }
                if (a.router_w) {
#pragma unroll
                    for (int c = 0; c < 4; ++c) rows4_smem[i + c] = as_stored(v[c], out);
                }
            }
        }
    }
    if (a.router_w) {
        // logits: one warp per output, the row from shared memory, 16 bytes of weights per lane and step (H % 8 == 0)
        const int warp = tid >> 5, lane = tid & 31, outs = a.route.experts + a.route.identity;
        float* z = rows4_smem + H;
        __syncthreads();
        const int warps = n >> 5;
        for (int e0 = warp; e0 < outs; e0 += 2 * warps) {  // two outputs at a time: their loads in flight together
            const int e1 = e0 + warps;
            const bf16 *w0 = a.router_w + (size_t)e0 * a.router_ld, *w1 = a.router_w + (size_t)(e1 < outs ? e1 : e0) * a.router_ld;
            float acc0 = 0.f, acc1 = 0.f;
#pragma unroll 4
            for (int i = lane * 8; i < H; i += 256) {
                const uint4 p = __ldg((const uint4*)(w0 + i)), q = __ldg((const uint4*)(w1 + i));
                const float4 x0 = *(const float4*)(rows4_smem + i), x1 = *(const float4*)(rows4_smem + i + 4);
                acc0 += bf16_lo(p.x) * x0.x + bf16_hi(p.x) * x0.y + bf16_lo(p.y) * x0.z + bf16_hi(p.y) * x0.w;
                acc0 += bf16_lo(p.z) * x1.x + bf16_hi(p.z) * x1.y + bf16_lo(p.w) * x1.z + bf16_hi(p.w) * x1.w;
                acc1 += bf16_lo(q.x) * x0.x + bf16_hi(q.x) * x0.y + bf16_lo(q.y) * x0.z + bf16_hi(q.y) * x0.w;
                acc1 += bf16_lo(q.z) * x1.x + bf16_hi(q.z) * x1.y + bf16_lo(q.w) * x1.z + bf16_hi(q.w) * x1.w;
            }
            acc0 = warp_sum(acc0);
            acc1 = warp_sum(acc1);
            if (lane == 0) {
                z[e0] = acc0;
                if (e1 < outs) z[e1] = acc1;
            }
        }
        __syncthreads();
        if (warp == 0) route_token(a.route, r, z, z + outs, lane);
    }
    if (tid == 0) tl_mark(tl, 2);
}

// the same for any width, one column at a time through shared memory (no router)
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
            if (!a.embed_w) xr[i] = v;
            ss += v * v;
        }
        if (a.embed_w) {
            const float einv = 1.f / sqrtf(block_sum(ss, red) / (float)H + a.eps);
            ss = 0.f;
            for (int i = tid; i < H; i += n) {
                const float v = xs[i] * einv * __ldg(a.embed_w + i);
                xs[i] = v;
                xr[i] = v;
                ss += v * v;
            }
        }
    } else if (a.source == ROWS_DELTA && !a.post_w) {
        const float* d = a.delta + (size_t)r * a.delta_ld;
#pragma unroll 4
        for (int i = tid; i < H; i += n) {
            const float v = __ldcg(xr + i) + a.delta_mult * __ldcg(d + i);
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
        if (a.next2_w)
            for (int i = tid; i < H; i += n) act_store((A*)a.out2 + (size_t)r * a.out_ld + i, xs[i] * inv * __ldg(a.next2_w + i));
    }
    if (tid == 0) tl_mark(tl, 2);
}

__device__ __forceinline__ void load_pair(const float* p, float& x, float& y) {
    const float2 v = __ldcg((const float2*)p);
    x = v.x;
    y = v.y;
}
__device__ __forceinline__ void load_pair(const bf16* p, float& x, float& y) {
    const uint32_t v = __ldcg((const unsigned int*)p);
    x = bf16_lo(v);
    y = bf16_hi(v);
}
__device__ __forceinline__ void store_pair(float* p, float x, float y) { *(float2*)p = make_float2(x, y); }
__device__ __forceinline__ void store_pair(bf16* p, float x, float y) {
    *(uint32_t*)p = (uint32_t)bf16_bits(x) | ((uint32_t)bf16_bits(y) << 16);
}

// one warp per (token, head): heads 0 .. nh-1 are queries, then the keys, then the values
constexpr int kQkWarps = 4;
template <typename A, int MP>  // MP pairs per lane: heads of up to 64 MP
__global__ void __launch_bounds__(kQkWarps * 32) k_qk_norm_rope(const QkNormRope a, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.y, u = blockIdx.x * kQkWarps + (threadIdx.x >> 5);
    const int nkv = a.kv.nkv, per_tok = a.nh + 2 * nkv;
    if (u < per_tok) {
        const int kind = u < a.nh ? 0 : (u < a.nh + nkv ? 1 : 2);
        const int head = kind == 0 ? u : (kind == 1 ? u - a.nh : u - a.nh - nkv);
        const int dim = kind == 2 ? a.vdim : a.dim;
        const float* norm_w = kind == 0 ? a.q_norm : a.k_norm;
        const A* src = (const A*)a.qkv + (size_t)t * a.ld + (kind == 0 ? 0 : (kind == 1 ? a.k_off : a.v_off)) + (size_t)head * dim;
        const int pos = __ldcg(a.tok_pos + t), seq = __ldcg(a.tok_seq + t);
        const bool pos_ok = pos >= 0 && pos < a.max_pos;
        const int pg = (kind != 0 && pos_ok) ? __ldcg(a.kv.block_table + (size_t)seq * a.kv.max_pages_per_seq + pos / kPageTokens) : 0;
        if (!pos_ok || (kind != 0 && (pg < 0 || pg >= a.kv.num_pages))) {
            if (lane == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        } else if (kind == 2) {
            A* dst = (A*)a.kv.v_pool + (((size_t)pg * nkv + head) * kPageTokens + pos % kPageTokens) * a.kv.vd;
            if ((dim & 1) == 0) {
                for (int i = lane * 2; i < dim; i += 64) {
                    float x, y;
                    load_pair(src + i, x, y);
                    store_pair(dst + i, x, y);
                }
            } else {
                for (int i = lane; i < dim; i += 32) act_store(dst + i, act_load(src + i));
            }
        } else {
            // lane = pair (2i, 2i + 1)
            const bool even = (dim & 1) == 0;
            float u0[MP], u1[MP], ss = 0.f;
#pragma unroll
            for (int j = 0; j < MP; ++j) {
                const int i = 2 * (lane + 32 * j);
                u0[j] = u1[j] = 0.f;
                if (i + 1 < dim && even) {
                    load_pair(src + i, u0[j], u1[j]);
                } else {
                    if (i < dim) u0[j] = act_load(src + i);
                    if (i + 1 < dim) u1[j] = act_load(src + i + 1);
                }
                ss += u0[j] * u0[j] + u1[j] * u1[j];
            }
            const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dim + a.eps);
            const float* w = norm_w;
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
                        store_pair(kdst + i, x, y);
                    }
                }
            }
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

constexpr int kRowsMaxSmem = 128 * 1024;

template <typename A, int IT>
cudaError_t rows4_attrs() {
    cudaError_t e = cudaFuncSetAttribute(k_residual_rows4<A, IT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRowsMaxSmem);
    return e == cudaSuccess ? prefer_max_shared(k_residual_rows4<A, IT>) : e;
}
template <typename A>
cudaError_t rows4_attrs_all() {
    cudaError_t e = rows4_attrs<A, 1>();
    if (e == cudaSuccess) e = rows4_attrs<A, 2>();
    if (e == cudaSuccess) e = rows4_attrs<A, 4>();
    if (e == cudaSuccess) e = rows4_attrs<A, 8>();
    return e;
}

}  // namespace

int stack_rows_prepare() {
    cudaError_t e = cudaFuncSetAttribute(k_residual_rows<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRowsMaxSmem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k_residual_rows<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, kRowsMaxSmem);
    if (e == cudaSuccess) e = rows4_attrs_all<bf16>();
    if (e == cudaSuccess) e = rows4_attrs_all<float>();
    if (e == cudaSuccess) e = prefer_max_shared(k_residual_rows<bf16>);
    if (e == cudaSuccess) e = prefer_max_shared(k_residual_rows<float>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<bf16, 2>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<bf16, 8>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<float, 2>);
    if (e == cudaSuccess) e = prefer_max_shared(k_qk_norm_rope<float, 8>);
    return (int)e;
}

template <typename A>
static void launch_rows(const ResidualRows& a, int rows, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (a.H % 4) {
        const int threads = a.H <= 512 ? 128 : (a.H <= 2048 ? 256 : 512);
        launch_k(k_residual_rows<A>, dim3(rows), dim3(threads), (size_t)a.H * 8, s, pdl, a, tl);
        return;
    }
    const int groups = a.H / 4;
    const size_t smem = a.router_w ? (size_t)(a.H + 2 * (a.route.experts + a.route.identity)) * 4 : 0;
    const int per = groups <= 256 ? 1 : groups <= 1024 ? 2 : groups <= 2048 ? 4 : 8;
    const int threads = ((groups + per - 1) / per + 31) / 32 * 32;
    const dim3 grid(rows), block(a.router_w ? 512 : threads);  // routing: as many warps for the router's outputs as fit
    if (per == 1) launch_k(k_residual_rows4<A, 1>, grid, block, smem, s, pdl, a, tl);
    else if (per == 2) launch_k(k_residual_rows4<A, 2>, grid, block, smem, s, pdl, a, tl);
    else if (per == 4) launch_k(k_residual_rows4<A, 4>, grid, block, smem, s, pdl, a, tl);
    else launch_k(k_residual_rows4<A, 8>, grid, block, smem, s, pdl, a, tl);
}
void launch_residual_rows(const ResidualRows& a, bool f32, int rows, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) launch_rows<float>(a, rows, s, pdl, tl);
    else launch_rows<bf16>(a, rows, s, pdl, tl);
}

void launch_qk_norm_rope(const QkNormRope& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const dim3 grid((a.nh + 2 * a.kv.nkv + kQkWarps - 1) / kQkWarps, T), block(kQkWarps * 32);
    const bool narrow = a.dim <= 128 && a.vdim <= 128;
    if (f32) launch_k(narrow ? k_qk_norm_rope<float, 2> : k_qk_norm_rope<float, 8>, grid, block, 0, s, pdl, a, tl);
    else launch_k(narrow ? k_qk_norm_rope<bf16, 2> : k_qk_norm_rope<bf16, 8>, grid, block, 0, s, pdl, a, tl);
}

}  // namespace tffn
