// Latent attention's row kernels: the normed query latent, and the row a token leaves in the cache (normed latent and
// rotated key part, shared by all heads). Norms and rotation in fp32.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"

namespace tffn {

namespace {

constexpr int kPrepThreads = 128;

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

// dst = src / sqrt(mean(src^2) + eps) * w over n columns; src and dst 16-byte aligned, columns past n are left alone. The
// weights of the columns a thread keeps in registers (IT groups of four) are fetched by the constructor, ahead of the wait
// for src.
template <int IT>
struct NormRow {
    static constexpr int kept = kPrepThreads * IT * 4;
    const float* w;
    int n;
    float g[IT][4];
    __device__ __forceinline__ NormRow(const float* w_, int n_) : w(w_), n(n_) {
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (threadIdx.x + k * kPrepThreads) * 4;
            if (i + 3 < n) {
                const float4 q = __ldg((const float4*)(w + i));
                g[k][0] = q.x; g[k][1] = q.y; g[k][2] = q.z; g[k][3] = q.w;
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c) g[k][c] = i + c < n ? __ldg(w + i + c) : 0.f;
            }
        }
    }
    template <typename A>
    __device__ __forceinline__ void run(const A* src, A* dst, float eps, float* red) const {
        float v[IT][4], ss = 0.f;
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (threadIdx.x + k * kPrepThreads) * 4;
#pragma unroll
            for (int c = 0; c < 4; ++c) v[k][c] = 0.f;
            if (i + 3 < n) {
                load4(src + i, v[k]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (i + c < n) v[k][c] = act_load(src + i + c);
            }
        }
#pragma unroll
        for (int k = 0; k < IT; ++k)
#pragma unroll
            for (int c = 0; c < 4; ++c) ss += v[k][c] * v[k][c];
        for (int i = kept + threadIdx.x; i < n; i += kPrepThreads) {
            const float x = act_load(src + i);
            ss += x * x;
        }
        const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            const int i = (threadIdx.x + k * kPrepThreads) * 4;
            const float o[4] = {v[k][0] * inv * g[k][0], v[k][1] * inv * g[k][1], v[k][2] * inv * g[k][2], v[k][3] * inv * g[k][3]};
            if (i + 3 < n) {
                store4(dst + i, o);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (i + c < n) act_store(dst + i + c, o[c]);
            }
        }
        for (int i = kept + threadIdx.x; i < n; i += kPrepThreads) act_store(dst + i, act_load(src + i) * inv * __ldg(w + i));
    }
};

// grid (1 or 2, T): x = 0 the query latent, x = 1 the cached row
template <typename A, int IT>
__global__ void __launch_bounds__(kPrepThreads) k_latent_prep(const LatentPrep a, unsigned long long* tl) {
    __shared__ float red[32];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int t = blockIdx.y;
    const A* row = (const A*)a.proj + (size_t)t * a.ld;
    if (blockIdx.x == 0) {
        const NormRow<IT> norm(a.q_norm, a.q_rank);
        pdl_wait();
        if (threadIdx.x == 0) tl_mark(tl, 1);
        norm.run(row, (A*)a.cq + (size_t)t * a.cq_ld, a.eps, red);
    } else {
        // slots, positions and the block table are older than the step's first kernel
        const NormRow<IT> norm(a.kv_norm, a.rank);
        const int pos = __ldcg(a.tok_pos + t), seq = __ldcg(a.tok_seq + t), half = a.rot / 2, rot_col = (a.rank + 63) / 64 * 64;
        const bool pos_ok = pos >= 0 && pos < a.max_pos;
        const int pg = pos_ok ? __ldcg(a.kv.block_table + (size_t)seq * a.kv.max_pages_per_seq + pos / kPageTokens) : -1;
        float2 cs = make_float2(1.f, 0.f);
        if (pos_ok && (int)threadIdx.x < half) cs = __ldg(a.rope + (size_t)pos * half + threadIdx.x);
        pdl_wait();
        if (threadIdx.x == 0) tl_mark(tl, 1);
        if (pg < 0 || pg >= a.kv.num_pages) {
            if (threadIdx.x == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        } else {
            A* dst = (A*)a.kv.k_pool + ((size_t)pg * kPageTokens + pos % kPageTokens) * a.kv.hd;
            const A* src = row + a.kv_off;
            for (int i = threadIdx.x; i < half; i += kPrepThreads) {
                if (i >= kPrepThreads) cs = __ldg(a.rope + (size_t)pos * half + i);
                const float u = act_load(src + a.rank + i), v = act_load(src + a.rank + half + i);
                act_store(dst + rot_col + i, u * cs.x - v * cs.y);
                act_store(dst + rot_col + half + i, v * cs.x + u * cs.y);
            }
            norm.run(src, dst, a.eps, red);
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

// one warp per (token, head)
constexpr int kRopeWarps = 4;
template <typename A>
__global__ void __launch_bounds__(kRopeWarps * 32) k_latent_rope(const A* __restrict__ q_up, int64_t ld, int off, int heads, int rot,
                                                                 const float2* __restrict__ rope, int max_pos, const int* __restrict__ tok_pos,
                                                                 float* __restrict__ q, int q_cols, int rot_col, int* status,
                                                                 unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int lane = threadIdx.x & 31, h = blockIdx.x * kRopeWarps + (threadIdx.x >> 5), t = blockIdx.y, half = rot / 2;
    const int pos = __ldcg(tok_pos + t);
    if (h < heads) {
        if (pos < 0 || pos >= max_pos) {
            if (lane == 0) dev_fail(status, DEV_ERR_BOUNDS);
        } else {
            const A* src = q_up + (size_t)t * ld + off + (size_t)h * rot;
            float* dst = q + ((size_t)t * heads + h) * q_cols + rot_col;
            for (int i = lane; i < half; i += 32) {
                const float u = act_load(src + i), v = act_load(src + half + i);
                const float2 cs = __ldg(rope + (size_t)pos * half + i);
                dst[i] = u * cs.x - v * cs.y;
                dst[half + i] = v * cs.x + u * cs.y;
            }
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

template <typename A>
cudaError_t prep_attrs() {
    cudaError_t e = prefer_max_shared(k_latent_prep<A, 1>);
    if (e == cudaSuccess) e = prefer_max_shared(k_latent_prep<A, 2>);
    if (e == cudaSuccess) e = prefer_max_shared(k_latent_prep<A, 4>);
    return e;
}
template <typename A>
void prep(const LatentPrep& a, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const dim3 grid(a.own_rows ? 2 : 1, T), block(kPrepThreads);
    const int n = a.q_rank > a.rank ? a.q_rank : a.rank;
    launch_k(n <= 512 ? k_latent_prep<A, 1> : n <= 1024 ? k_latent_prep<A, 2> : k_latent_prep<A, 4>, grid, block, 0, s, pdl, a, tl);
}

}  // namespace

int latent_prepare() {
    cudaError_t e = prep_attrs<bf16>();
    if (e == cudaSuccess) e = prep_attrs<float>();
    if (e == cudaSuccess) e = prefer_max_shared(k_latent_rope<bf16>);
    if (e == cudaSuccess) e = prefer_max_shared(k_latent_rope<float>);
    return (int)e;
}

void launch_latent_prep(const LatentPrep& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) prep<float>(a, T, s, pdl, tl);
    else prep<bf16>(a, T, s, pdl, tl);
}

void launch_latent_rope(const void* q_up, int64_t ld, int off, int heads, int rot, const float2* rope, int max_pos, const int* tok_pos,
                        float* q, int q_cols, int rot_col, bool f32, int T, int* status, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const dim3 grid((heads + kRopeWarps - 1) / kRopeWarps, T), block(kRopeWarps * 32);
    if (f32) launch_k(k_latent_rope<float>, grid, block, 0, s, pdl, (const float*)q_up, ld, off, heads, rot, rope, max_pos, tok_pos, q, q_cols, rot_col, status, tl);
    else launch_k(k_latent_rope<bf16>, grid, block, 0, s, pdl, (const bf16*)q_up, ld, off, heads, rot, rope, max_pos, tok_pos, q, q_cols, rot_col, status, tl);
}

}  // namespace tffn
