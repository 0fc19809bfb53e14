// Real-gated linear recurrence, a recurrent mixer. Two kernels around the gates' block-diagonal product:
//   k_lru_prep  the short causal convolution of every channel (tokens are independent: earlier inputs are rows of this
//               launch or lie in the slot's ring of earlier inputs)
//   k_lru_scan  gates, decays and the recurrence S = a S + b, then the row S * gelu(y). A block takes 32 channels of a
//               sequence; its warps take consecutive pieces of a tile of tokens, scan their pieces from zero at the same
//               time (keeping the running product of a), and fold in what the pieces before left.
// Everything but the projections that come in, u and the mixer's row is fp32.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"

namespace tffn {

namespace {

constexpr int kConvThreads = 128;

// V adjacent channels of a token per thread (V = 4: parts whose length is a multiple of 4)
template <int V>
__device__ __forceinline__ void load_cols(const float* p, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 q = __ldcg((const float4*)p);
        v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
        v[0] = __ldcg(p);
    }
}
template <int V>
__device__ __forceinline__ void load_cols(const bf16* p, float (&v)[V]) {
    if constexpr (V == 4) {
        const uint2 q = __ldcg((const uint2*)p);
        v[0] = bf16_lo(q.x); v[1] = bf16_hi(q.x); v[2] = bf16_lo(q.y); v[3] = bf16_hi(q.y);
    } else {
        v[0] = act_load(p);
    }
}

template <typename A, int V>
__global__ void __launch_bounds__(kConvThreads) k_lru_prep(const RgLru a, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int t = blockIdx.y, ch = (blockIdx.x * kConvThreads + threadIdx.x) * V, R = a.taps - 1;
    // slots and positions are older than the step's first kernel
    const int seq = __ldcg(a.tok_seq + t), pos = __ldcg(a.tok_pos + t);
    // where the input `lag` tokens back lies: bit lag of rows (a row of this launch) or of ring (the slot's ring)
    uint32_t rows, ring;
    {
        const int lag = threadIdx.x & 31;
        const bool in_seq = lag < a.taps && pos - lag >= 0;
        const bool row = in_seq && (lag == 0 || (t >= lag && __ldcg(a.tok_seq + t - lag) == seq && __ldcg(a.tok_pos + t - lag) == pos - lag));
        rows = __ballot_sync(0xffffffffu, row);
        ring = __ballot_sync(0xffffffffu, in_seq && !row);
    }
    // Taps, biases and the ring are older than the step's first kernel as well: only rows of this launch wait. The four
    // youngest inputs have their loads in flight together.
    constexpr int NEAR = 4;
    float xb[V], y[V], w[NEAR][V], x[NEAR][V];
    const bool on = ch < a.width && seq >= 0 && seq < a.max_slots && pos >= 0;
    const float* old = a.ring + (size_t)(on ? seq : 0) * a.ring_stride + ch;
    if (on) {
        load_cols<V>(a.conv_bias + ch, y);
        load_cols<V>(a.x_bias + ch, xb);
#pragma unroll
        for (int lag = 0; lag < NEAR; ++lag) {
#pragma unroll
            for (int v = 0; v < V; ++v) w[lag][v] = x[lag][v] = 0.f;
            if (lag <= R && ((rows | ring) >> lag & 1u)) load_cols<V>(a.conv + (size_t)(R - lag) * a.width + ch, w[lag]);
            if (lag <= R && (ring >> lag & 1u)) load_cols<V>(old + (size_t)((pos - lag) % R) * a.width, x[lag]);
        }
    }
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    if (seq < 0 || seq >= a.max_slots || pos < 0) {
        if (threadIdx.x == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        return;
    }
    if (on) {
        const A* x0 = (const A*)a.proj + (size_t)t * a.proj_ld + a.x_off + ch;
#pragma unroll
        for (int lag = 0; lag < NEAR; ++lag)
            if (rows >> lag & 1u) load_cols<V>(x0 - (ptrdiff_t)lag * a.proj_ld, x[lag]);
        for (int lag = R; lag >= NEAR; --lag) {  // long convolutions: the older inputs
            float xo[V], wo[V];
            if (!((rows | ring) >> lag & 1u)) continue;
            load_cols<V>(a.conv + (size_t)(R - lag) * a.width + ch, wo);
            if (rows >> lag & 1u) load_cols<V>(x0 - (ptrdiff_t)lag * a.proj_ld, xo);
            else load_cols<V>(old + (size_t)((pos - lag) % R) * a.width, xo);
#pragma unroll
            for (int v = 0; v < V; ++v) y[v] += wo[v] * (xo[v] + (rows >> lag & 1u ? xb[v] : 0.f));
        }
#pragma unroll
        for (int lag = NEAR - 1; lag >= 0; --lag)  // oldest first; a projection still lacks its bias, the ring does not
#pragma unroll
            for (int v = 0; v < V; ++v) y[v] += w[lag][v] * (x[lag][v] + (rows >> lag & 1u ? xb[v] : 0.f));
        const int n = a.width / a.blocks;
        A* dst = (A*)a.u + (size_t)t * a.u_ld + (ch / n) * a.u_part + ch % n;
#pragma unroll
        for (int v = 0; v < V; ++v) act_store(dst + v, y[v]);
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

__device__ __forceinline__ float gelu_tanh_f32(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// The inputs of one (token, channel) and what the recurrence makes of them.
struct LruIn {
    float r, i, u, y;
};
template <typename A>
__device__ __forceinline__ LruIn lru_load(const RgLru& a, size_t t, int ch, int col, int ucol) {
    LruIn in;
    const float* z = a.gate_in + t * a.gate_ld + col;
    in.r = __ldcg(z);
    in.i = __ldcg(z + a.width / a.blocks);
    in.u = act_load((const A*)a.u + t * a.u_ld + ucol);
    in.y = act_load((const A*)a.proj + t * a.proj_ld + ch);
    return in;
}

// L tokens per warp and tile, W warps along the tokens, CW along the channels (32 each)
template <typename A, int L, int W, int CW>
__global__ void __launch_bounds__(W * CW * 32) k_lru_scan(const RgLru a, unsigned long long* tl) {
    __shared__ float s_a[CW][W][32], s_s[CW][W][32];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, wt = (threadIdx.x >> 5) % W, wc = (threadIdx.x >> 5) / W;
    const int ch = (blockIdx.x * CW + wc) * 32 + lane;
    const bool on = ch < a.width;
    const int c = on ? ch : 0;
    const int first = __ldcg(a.seg_first + blockIdx.y), count = __ldcg(a.seg_count + blockIdx.y);
    const int slot = __ldcg(a.tok_seq + first), pos0 = __ldcg(a.tok_pos + first);
    const bool ok = slot >= 0 && slot < a.max_slots && pos0 >= 0;
    float* st = a.state + (size_t)(ok ? slot : 0) * a.state_stride + c;
    // state and weights are older than this step's first kernel
    float S = ok && pos0 > 0 ? __ldcg(st) : 0.f;
    const int n = a.width / a.blocks, b = c / n, col = 2 * b * n + c % n, ucol = b * a.u_part + c % n;
    const float decay = -8.f * softplus_f32(__ldg(a.lam + c)), r_bias = __ldg(a.gate_bias + col), i_bias = __ldg(a.gate_bias + col + n);
    const float y_bias = __ldg(a.y_bias + c), x_bias = __ldg(a.x_bias + c);
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    if (!ok) {
        if (threadIdx.x == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        return;
    }
    auto step = [&](const LruIn& in, float& decay_t, float& add) {
        const float log_a = decay * sigmoid_f32(in.r + r_bias);
        decay_t = expf(log_a);
        add = sqrtf(-expm1f(2.f * log_a)) * sigmoid_f32(in.i + i_bias) * in.u;
    };
    for (int t0 = 0; t0 < count; t0 += L * W) {
        const int mine = t0 + wt * L;  // this warp's first token of the tile
        LruIn in[L];
#pragma unroll
        for (int k = 0; k < L; ++k) {
            in[k] = LruIn{0.f, 0.f, 0.f, 0.f};
            if (mine + k < count) in[k] = lru_load<A>(a, (size_t)first + mine + k, c, col, ucol);
        }
        float p[L], s[L];  // product of the decays and the state from zero, up to and with token k
#pragma unroll
        for (int k = 0; k < L; ++k) {
            float g = 1.f, add = 0.f;
            if (mine + k < count) step(in[k], g, add);
            p[k] = k ? p[k - 1] * g : g;
            s[k] = k ? g * s[k - 1] + add : add;
        }
        float carry = S;
        if constexpr (W > 1) {
            s_a[wc][wt][lane] = p[L - 1];
            s_s[wc][wt][lane] = s[L - 1];
            __syncthreads();
#pragma unroll
            for (int w = 0; w < W; ++w) {  // every warp follows the state over the whole tile
                if (w == wt) carry = S;
                S = s_a[wc][w][lane] * S + s_s[wc][w][lane];
            }
            __syncthreads();
        } else {
            S = p[L - 1] * S + s[L - 1];
        }
#pragma unroll
        for (int k = 0; k < L; ++k)
            if (on && mine + k < count)
                act_store((A*)a.out + ((size_t)first + mine + k) * a.out_ld + ch, (s[k] + p[k] * carry) * gelu_tanh_f32(in[k].y + y_bias));
    }
    if (on && count > 0) {
        if (wt == 0) *st = S;
        // the last inputs of the convolution, for the run's continuation (the preparation has finished reading the ring)
        const int R = a.taps - 1;
        for (int i = wt; i < min(R, count); i += W) {
            const int t = first + count - 1 - i, pos = pos0 + count - 1 - i;
            a.ring[(size_t)slot * a.ring_stride + (size_t)(pos % R) * a.width + ch] =
                act_load((const A*)a.proj + (size_t)t * a.proj_ld + a.x_off + ch) + x_bias;
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

template <typename A>
cudaError_t lru_attrs() {
    cudaError_t e = prefer_max_shared(k_lru_prep<A, 1>);
    if (e == cudaSuccess) e = prefer_max_shared(k_lru_prep<A, 4>);
    if (e == cudaSuccess) e = prefer_max_shared(k_lru_scan<A, 1, 1, 4>);
    if (e == cudaSuccess) e = prefer_max_shared(k_lru_scan<A, 8, 8, 1>);
    return e;
}
template <typename A>
void lru_prep(const RgLru& a, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const int v = a.width / a.blocks % 4 ? 1 : 4;
    const dim3 grid((a.width + kConvThreads * v - 1) / (kConvThreads * v), T), block(kConvThreads);
    if (v == 4) launch_k(k_lru_prep<A, 4>, grid, block, 0, s, pdl, a, tl);
    else launch_k(k_lru_prep<A, 1>, grid, block, 0, s, pdl, a, tl);
}
template <typename A>
void lru_scan(const RgLru& a, int n_segs, bool one_each, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (one_each) launch_k(k_lru_scan<A, 1, 1, 4>, dim3((a.width + 127) / 128, n_segs), dim3(128), 0, s, pdl, a, tl);
    else launch_k(k_lru_scan<A, 8, 8, 1>, dim3((a.width + 31) / 32, n_segs), dim3(256), 0, s, pdl, a, tl);
}

}  // namespace

int lru_prepare() {
    cudaError_t e = lru_attrs<bf16>();
    if (e == cudaSuccess) e = lru_attrs<float>();
    return (int)e;
}
void launch_lru_prep(const RgLru& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) lru_prep<float>(a, T, s, pdl, tl);
    else lru_prep<bf16>(a, T, s, pdl, tl);
}
void launch_lru_scan(const RgLru& a, bool f32, int n_segs, bool one_each, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) lru_scan<float>(a, n_segs, one_each, s, pdl, tl);
    else lru_scan<bf16>(a, n_segs, one_each, s, pdl, tl);
}

}  // namespace tffn
