// Gated delta rule with one decay per head and key channel, a recurrent mixer: per head a matrix S (key channels x
// value columns) with, per token,
//     S = g * S (rows), u = beta * (v - S^T k), S = S + k u^T, o = S^T q.
// Two kernels per layer, for prompts and decoding alike:
//   k_delta_prep  one warp per (token, head): the short causal convolutions with SiLU, the unit vectors q and k, beta and
//                 the decays. Tokens are independent here (a convolution reads the projections of earlier rows of the
//                 launch, or the slot's ring of earlier inputs).
//   k_delta_scan  one CTA per (sequence, head): S stays in registers for all tokens of the launch, a value column's key
//                 channels spread over eight lanes; the tokens' vectors pass through a double-buffered shared-memory
//                 stage. The read-out uses o = (g S)^T q + u (k . q), the same sum in one pass over S. The head's norm
//                 and its output gate are applied per stage of tokens before the row is stored.
// Everything is fp32 except the projections that come in and the mixer's output.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"

namespace tffn {

namespace {

constexpr int kPrepWarps = 4;
constexpr int kMaxDimRegs = 8;  // channels per lane: heads of up to 256

template <typename A>
__device__ __forceinline__ void conv_silu(const DeltaRule& a, int t, int seq, int pos, int col, int chan, int dim, int lane,
                                          float (&y)[kMaxDimRegs]) {
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
#pragma unroll
    for (int i = 0; i < kMaxDimRegs; ++i) y[i] = 0.f;
    for (int lag = a.taps - 1; lag >= 0; --lag) {
        if (pos - lag < 0) continue;  // zeros before the sequence
        const bool row = lag == 0 || (t >= lag && __ldcg(a.tok_seq + t - lag) == seq && __ldcg(a.tok_pos + t - lag) == pos - lag);
        const A* src = (const A*)a.proj + (size_t)(row ? t - lag : 0) * a.proj_ld + col;
        const float* old = a.ring + (size_t)seq * a.ring_stride + (size_t)(a.taps > 1 ? (pos - lag) % (a.taps - 1) : 0) * C + chan;
        const float* w = a.conv + (size_t)(a.taps - 1 - lag) * C + chan;
#pragma unroll
        for (int i = 0; i < kMaxDimRegs; ++i) {
            const int d = lane + 32 * i;
            if (d < dim) y[i] += __ldg(w + d) * (row ? act_load(src + d) : __ldcg(old + d));
        }
    }
#pragma unroll
    for (int i = 0; i < kMaxDimRegs; ++i) y[i] *= sigmoid_f32(y[i]);
}

template <typename A>
__global__ void __launch_bounds__(kPrepWarps * 32) k_delta_prep(const DeltaRule a, int T, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int lane = threadIdx.x & 31;
    const long long unit = (long long)blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
    const int G = a.kv_heads, H = a.heads, per_tok = G + H;
    if (unit < (long long)T * per_tok) {
        const int t = (int)(unit / per_tok), u = (int)(unit % per_tok);
        const int seq = __ldcg(a.tok_seq + t), pos = __ldcg(a.tok_pos + t);
        if (seq < 0 || seq >= a.max_slots || pos < 0) {
            if (lane == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        } else if (u < G) {
            float q[kMaxDimRegs], k[kMaxDimRegs];
            conv_silu<A>(a, t, seq, pos, a.q_off + u * a.dim, u * a.dim, a.dim, lane, q);
            conv_silu<A>(a, t, seq, pos, a.k_off + u * a.dim, (G + u) * a.dim, a.dim, lane, k);
            float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
            for (int i = 0; i < kMaxDimRegs; ++i) {  // past dim both are zero
                qq += q[i] * q[i];
                kk += k[i] * k[i];
            }
            const float qs = 1.f / sqrtf(warp_sum(qq) + 1e-6f) / sqrtf((float)a.dim), ks = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
            float* qo = a.qn + ((size_t)t * G + u) * a.dimP;
            float* ko = a.kn + ((size_t)t * G + u) * a.dimP;
#pragma unroll
            for (int i = 0; i < kMaxDimRegs; ++i) {
                const int d = lane + 32 * i;
                if (d < a.dimP) {
                    const float x = q[i] * qs, y = k[i] * ks;
                    qk += x * y;
                    qo[d] = x;
                    ko[d] = y;
                }
            }
            qk = warp_sum(qk);
            const int rep = H / G;
            for (int h = u * rep + lane; h < (u + 1) * rep; h += 32) a.bk[((size_t)t * H + h) * 2 + 1] = qk;
        } else {
            const int h = u - G;
            float v[kMaxDimRegs];
            conv_silu<A>(a, t, seq, pos, a.v_off + h * a.vdim, 2 * G * a.dim + h * a.vdim, a.vdim, lane, v);
            float* vo = a.v + ((size_t)t * H + h) * a.vdimP;
#pragma unroll
            for (int i = 0; i < kMaxDimRegs; ++i)
                if (lane + 32 * i < a.vdimP) vo[lane + 32 * i] = v[i];
            const float rate = -expf(__ldg(a.a_log + h));
            const float* z = a.decay_in + (size_t)t * a.decay_ld + (size_t)h * a.dim;
            float* go = a.g + ((size_t)t * H + h) * a.dimP;
#pragma unroll
            for (int i = 0; i < kMaxDimRegs; ++i) {
                const int d = lane + 32 * i;
                if (d < a.dimP) go[d] = d < a.dim ? expf(rate * softplus_f32(__ldcg(z + d) + __ldg(a.dt_bias + h * a.dim + d))) : 0.f;
            }
            if (lane == 0)
                a.bk[((size_t)t * H + h) * 2] = sigmoid_f32(act_load((const A*)a.proj + (size_t)t * a.proj_ld + a.b_off + h));
        }
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

// pairs of fp32 in a 64-bit register: two adjacent key channels
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 pack2(float x, float y) {
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ float sum2(f32x2 a) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
    return x + y;
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async8(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

constexpr int kScanTokens = 8;  // tokens per stage
__host__ __device__ inline int scan_token_floats(int dimP, int vdimP) { return 3 * dimP + vdimP + 4; }
inline size_t scan_smem(int dimP, int vdimP) { return (size_t)kScanTokens * (2 * scan_token_floats(dimP, vdimP) + vdimP) * 4; }

// J = dimP / 32 float4 of a column per lane; lane r of the eight that share four value columns holds the key channels
// 4 (r + 8 j) + {0..3}
template <typename A, int J, int NT>
__global__ void __launch_bounds__(NT, (NT == 256 && J <= 4) ? 2 : 1) k_delta_scan(const DeltaRule a, unsigned long long* tl) {
    extern __shared__ __align__(16) float scan_buf[];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5;
    const int h = blockIdx.x, H = a.heads, G = a.kv_heads, kvh = h / (H / G);
    const int r = tid & 7, c0 = (tid >> 3) * 4;
    constexpr int dimP = 32 * J;
    const int vdimP = a.vdimP, tokf = scan_token_floats(dimP, vdimP);
    float* o_s = scan_buf + (size_t)2 * kScanTokens * tokf;  // [kScanTokens][vdimP]
    // The token lists and the state are older than this step's first kernel (a full dependency of the stream), so
    // the state is fetched while the preparation is still running.
    const int first = __ldcg(a.seg_first + blockIdx.y), count = __ldcg(a.seg_count + blockIdx.y);
    const int slot = __ldcg(a.tok_seq + first), pos0 = __ldcg(a.tok_pos + first);
    const bool ok = slot >= 0 && slot < a.max_slots && pos0 >= 0;
    const bool mine = ok && c0 < vdimP;
    float* st = a.state + (size_t)(ok ? slot : 0) * a.state_stride + (size_t)h * vdimP * dimP;
    f32x2 S[4][J][2];
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int j = 0; j < J; ++j) {
            ulonglong2 v = make_ulonglong2(0ull, 0ull);
            if (mine && pos0 > 0) v = __ldcg((const ulonglong2*)(st + (size_t)(c0 + c) * dimP + 4 * (r + 8 * j)));
            S[c][j][0] = v.x;
            S[c][j][1] = v.y;
        }
    pdl_wait();
    if (tid == 0) tl_mark(tl, 1);
    if (!ok) {
        if (tid == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        return;
    }
    auto fetch = [&](int tile) {  // tokens [tile * kScanTokens, ...) of the run into buffer tile & 1
        float* buf = scan_buf + (size_t)(tile & 1) * kScanTokens * tokf;
        const int n = min(kScanTokens, count - tile * kScanTokens);
        const int per = (3 * dimP + vdimP) / 4;  // 16-byte pieces of a token
        for (int i = tid; i < n * per; i += blockDim.x) {
            const int k = i / per, p = (i % per) * 4;
            const size_t t = (size_t)first + tile * kScanTokens + k;
            const float* src = p < dimP ? a.qn + (t * G + kvh) * dimP + p
                               : p < 2 * dimP ? a.kn + (t * G + kvh) * dimP + (p - dimP)
                               : p < 3 * dimP ? a.g + (t * H + h) * dimP + (p - 2 * dimP)
                                              : a.v + (t * H + h) * vdimP + (p - 3 * dimP);
            cp_async16(buf + (size_t)k * tokf + p, src);
        }
        if (tid < n) {
            const size_t t = (size_t)first + tile * kScanTokens + tid;
            cp_async8(buf + (size_t)tid * tokf + 3 * dimP + vdimP, a.bk + (t * H + h) * 2);
        }
    };
    const int tiles = (count + kScanTokens - 1) / kScanTokens;
    if (tiles > 0) fetch(0);
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int tile = 0; tile < tiles; ++tile) {
        if (tile + 1 < tiles) fetch(tile + 1);  // its buffer was last read before the barrier that ended tile - 1
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const float* buf = scan_buf + (size_t)(tile & 1) * kScanTokens * tokf;
        const int n = min(kScanTokens, count - tile * kScanTokens);
        for (int k = 0; k < n; ++k) {
            const float* tok = buf + (size_t)k * tokf;
            f32x2 t2[4], w2[4], kk[J][2];
#pragma unroll
            for (int c = 0; c < 4; ++c) t2[c] = w2[c] = 0ull;
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const int d = 4 * (r + 8 * j);
                const ulonglong2 q4 = *(const ulonglong2*)(tok + d);
                const ulonglong2 k4 = *(const ulonglong2*)(tok + dimP + d);
                const ulonglong2 g4 = *(const ulonglong2*)(tok + 2 * dimP + d);
                kk[j][0] = k4.x;
                kk[j][1] = k4.y;
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    S[c][j][0] = mul2(S[c][j][0], g4.x);
                    S[c][j][1] = mul2(S[c][j][1], g4.y);
                    t2[c] = fma2(S[c][j][0], k4.x, t2[c]);
                    t2[c] = fma2(S[c][j][1], k4.y, t2[c]);
                    w2[c] = fma2(S[c][j][0], q4.x, w2[c]);
                    w2[c] = fma2(S[c][j][1], q4.y, w2[c]);
                }
            }
            // eight sums over eight lanes: halving exchange, lane r ends with S^T k of column r (r < 4) or S^T q of
            // column r - 4
            float x4[4], x2[2];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const float tt = sum2(t2[c]), ww = sum2(w2[c]);
                const float got = __shfl_xor_sync(0xffffffffu, (r & 4) ? tt : ww, 4);
                x4[c] = ((r & 4) ? ww : tt) + got;
            }
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const float got = __shfl_xor_sync(0xffffffffu, (r & 2) ? x4[c] : x4[c + 2], 2);
                x2[c] = ((r & 2) ? x4[c + 2] : x4[c]) + got;
            }
            const float got = __shfl_xor_sync(0xffffffffu, (r & 1) ? x2[0] : x2[1], 1);
            const float x = ((r & 1) ? x2[1] : x2[0]) + got;
            const float2 bk = *(const float2*)(tok + 3 * dimP + vdimP);
            const int col = c0 + (r & 3);
            const float v = col < vdimP ? tok[3 * dimP + col] : 0.f;
            const float u = bk.x * (v - x);  // meaningful in lanes r < 4
            float uc[4];
#pragma unroll
            for (int c = 0; c < 4; ++c) uc[c] = __shfl_sync(0xffffffffu, u, (lane & ~7) | c);
            const float mine_u = (r & 2) ? ((r & 1) ? uc[3] : uc[2]) : ((r & 1) ? uc[1] : uc[0]);
            if (r >= 4 && col < vdimP) o_s[k * vdimP + col] = x + mine_u * bk.y;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const f32x2 uu = pack2(uc[c], uc[c]);
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    S[c][j][0] = fma2(kk[j][0], uu, S[c][j][0]);
                    S[c][j][1] = fma2(kk[j][1], uu, S[c][j][1]);
                }
            }
        }
        __syncthreads();
        // the head's norm and gate, one warp per token of the stage
        for (int k = warp; k < n; k += nwarps) {
            const size_t t = (size_t)first + tile * kScanTokens + k;
            const float* o = o_s + k * vdimP;
            float ss = 0.f;
            for (int d = lane; d < a.vdim; d += 32) ss += o[d] * o[d];
            const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
            const float* gate = a.gate_in + t * a.gate_ld + (size_t)h * a.vdim;
            A* out = (A*)a.out + t * a.out_ld + (size_t)h * a.vdim;
            for (int d = lane; d < a.vdim; d += 32) act_store(out + d, o[d] * inv * __ldg(a.out_norm + d) * sigmoid_f32(__ldcg(gate + d)));
        }
    }
    if (mine && count > 0) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
            for (int j = 0; j < J; ++j)
                *(ulonglong2*)(st + (size_t)(c0 + c) * dimP + 4 * (r + 8 * j)) = make_ulonglong2(S[c][j][0], S[c][j][1]);
    }
    // The last inputs of the convolutions, for the run's continuation. The preparation of this launch has finished
    // reading the ring. A head keeps its value channels, the first head of a group the shared query and key channels.
    const int R = a.taps - 1, C = 2 * G * a.dim + H * a.vdim;
    for (int i = 0; i < min(R, count); ++i) {
        const int t = first + count - 1 - i, pos = pos0 + count - 1 - i;
        const A* row = (const A*)a.proj + (size_t)t * a.proj_ld;
        float* ring = a.ring + (size_t)slot * a.ring_stride + (size_t)(pos % R) * C;
        for (int d = tid; d < a.vdim; d += blockDim.x) ring[2 * G * a.dim + h * a.vdim + d] = act_load(row + a.v_off + h * a.vdim + d);
        if (h % (H / G) == 0)
            for (int d = tid; d < a.dim; d += blockDim.x) {
                ring[kvh * a.dim + d] = act_load(row + a.q_off + kvh * a.dim + d);
                ring[(G + kvh) * a.dim + d] = act_load(row + a.k_off + kvh * a.dim + d);
            }
    }
    if (tid == 0) tl_mark(tl, 2);
}

template <typename A, int J, int NT>
cudaError_t scan_attrs() {
    cudaError_t e = cudaFuncSetAttribute(k_delta_scan<A, J, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan_smem(256, 256));
    return e == cudaSuccess ? prefer_max_shared(k_delta_scan<A, J, NT>) : e;
}
template <typename A>
cudaError_t scan_attrs_all() {
    cudaError_t e = scan_attrs<A, 1, 256>();
    if (e == cudaSuccess) e = scan_attrs<A, 2, 256>();
    if (e == cudaSuccess) e = scan_attrs<A, 3, 256>();
    if (e == cudaSuccess) e = scan_attrs<A, 4, 256>();
    if (e == cudaSuccess) e = scan_attrs<A, 8, 256>();
    if (e == cudaSuccess) e = scan_attrs<A, 1, 512>();
    if (e == cudaSuccess) e = scan_attrs<A, 2, 512>();
    if (e == cudaSuccess) e = scan_attrs<A, 3, 512>();
    if (e == cudaSuccess) e = scan_attrs<A, 4, 512>();
    if (e == cudaSuccess) e = scan_attrs<A, 8, 512>();
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_prep<A>);
    return e;
}

template <typename A, int J>
void launch_scan(const DeltaRule& a, int n_segs, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const int threads = (a.vdimP / 4 * 8 + 31) / 32 * 32;
    const dim3 grid(a.heads, n_segs);
    const size_t smem = scan_smem(a.dimP, a.vdimP);
    if (threads <= 256) launch_k(k_delta_scan<A, J, 256>, grid, dim3(threads), smem, s, pdl, a, tl);
    else launch_k(k_delta_scan<A, J, 512>, grid, dim3(threads), smem, s, pdl, a, tl);
}
template <typename A>
void launch_scan_j(const DeltaRule& a, int n_segs, cudaStream_t s, bool pdl, unsigned long long* tl) {
    switch (a.dimP) {
        case 32: return launch_scan<A, 1>(a, n_segs, s, pdl, tl);
        case 64: return launch_scan<A, 2>(a, n_segs, s, pdl, tl);
        case 96: return launch_scan<A, 3>(a, n_segs, s, pdl, tl);
        case 128: return launch_scan<A, 4>(a, n_segs, s, pdl, tl);
        default: return launch_scan<A, 8>(a, n_segs, s, pdl, tl);
    }
}

}  // namespace

int delta_prepare() {
    cudaError_t e = scan_attrs_all<bf16>();
    if (e == cudaSuccess) e = scan_attrs_all<float>();
    return (int)e;
}
int delta_padded_dim(int dim) { return dim <= 128 ? (dim + 31) / 32 * 32 : 256; }

void launch_delta_prep(const DeltaRule& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const long long units = (long long)T * (a.kv_heads + a.heads);
    const dim3 grid((unsigned)((units + kPrepWarps - 1) / kPrepWarps)), block(kPrepWarps * 32);
    if (f32) launch_k(k_delta_prep<float>, grid, block, 0, s, pdl, a, T, tl);
    else launch_k(k_delta_prep<bf16>, grid, block, 0, s, pdl, a, T, tl);
}
void launch_delta_scan(const DeltaRule& a, bool f32, int n_segs, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) launch_scan_j<float>(a, n_segs, s, pdl, tl);
    else launch_scan_j<bf16>(a, n_segs, s, pdl, tl);
}

}  // namespace tffn
