// Gated delta rule with one decay per head and key channel or (HEAD_DECAY) per head, a recurrent mixer: per head a matrix
// S (key channels x value columns) with, per token,
//     S = g * S (rows), u = beta * (v - S^T k), S = S + k u^T, o = S^T q.
// Two kernels per layer, for prompts and decoding alike:
//   k_delta_prep  one warp per (token, head): the short causal convolutions with SiLU, the unit vectors q and k, beta and
//                 the decays. Tokens are independent here (a convolution reads the projections of earlier rows of the
//                 launch, or the slot's ring of earlier inputs).
//   k_delta_scan  one CTA per (sequence, head, slice of value columns): S stays in registers for all tokens of the
//                 launch, a value column's key channels spread over eight lanes; the tokens' vectors pass through a
//                 double-buffered shared-memory stage. The read-out uses o = (g S)^T q + u (k . q), the same sum in one
//                 pass over S. In a decode step the head's norm and its output gate are applied here,
//   k_delta_out   for prompts in a kernel of their own, off the sequential path.
// Everything is fp32 except the projections that come in and the mixer's output.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"

namespace tffn {

namespace {

constexpr int kPrepWarps = 4;

// V adjacent values of an activation or fp32 row; V = 2 needs 4- / 8-byte aligned rows (even head sizes)
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&x)[V]) {
    if constexpr (V == 2) {
        const float2 v = __ldcg((const float2*)p);
        x[0] = v.x;
        x[1] = v.y;
    } else {
        x[0] = __ldcg(p);
    }
}
template <int V>
__device__ __forceinline__ void load_v(const bf16* p, float (&x)[V]) {
    if constexpr (V == 2) {
        const uint32_t v = __ldcg((const unsigned int*)p);
        x[0] = bf16_lo(v);
        x[1] = bf16_hi(v);
    } else {
        x[0] = act_load(p);
    }
}

// Where the inputs of a token's convolutions lie: the projections of earlier rows of this launch, the slot's ring, or
// nowhere (before the sequence). Bit lag of the masks; every lane of the warp calls it.
struct ConvSource {
    uint32_t rows, ring;
    bool inside;  // all of them rows
    int place;    // this lane's lag: its place in the ring
};
__device__ __forceinline__ ConvSource conv_source(const DeltaRule& a, int t, int seq, int pos, int lane) {
    const int lag = lane;
    const bool in_seq = lag < a.taps && pos - lag >= 0;
    const bool row = in_seq && (lag == 0 || (t >= lag && __ldcg(a.tok_seq + t - lag) == seq && __ldcg(a.tok_pos + t - lag) == pos - lag));
    ConvSource s;
    s.rows = __ballot_sync(0xffffffffu, row);
    s.ring = __ballot_sync(0xffffffffu, in_seq && !row);
    s.inside = __popc(s.rows) == a.taps;
    s.place = in_seq && !row ? (pos - lag) % (a.taps - 1) : 0;  // lag 0 is always a row, so taps > 1 here
    return s;
}

// channels [chan, chan + dim) of the convolution of token t, SiLU included: lane holds channels (lane + 32 i) * V + v.
// The loads of four taps are in flight together.
template <typename A, int V, int NI>
__device__ __forceinline__ void conv_silu(const DeltaRule& a, const ConvSource& cs, int t, int seq, int pos, int col, int chan, int dim,
                                          int lane, float (&y)[NI][V]) {
    const int C = 2 * a.kv_heads * a.dim + a.heads * a.vdim, R = a.taps - 1;
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) y[i][v] = 0.f;
    const A* row0 = (const A*)a.proj + (size_t)t * a.proj_ld + col;
    const float* w0 = a.conv + chan;
    if (cs.inside) {  // every input is a row of this launch
        for (int l0 = R; l0 >= 0; l0 -= 4) {  // oldest tap first
            float x[4][NI][V], w[4][NI][V];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int lag = l0 - j;
                const A* src = row0 - (ptrdiff_t)lag * a.proj_ld;
                const float* wt = w0 + (ptrdiff_t)(R - lag) * C;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int d = (lane + 32 * i) * V;
#pragma unroll
                    for (int v = 0; v < V; ++v) x[j][i][v] = w[j][i][v] = 0.f;
                    if (lag >= 0 && d < dim) {
                        load_v<V>(src + d, x[j][i]);
                        load_v<V>(wt + d, w[j][i]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int v = 0; v < V; ++v) y[i][v] += w[j][i][v] * x[j][i][v];
        }
    } else {
        for (int l0 = R; l0 >= 0; l0 -= 4) {
            float x[4][NI][V], w[4][NI][V];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int lag = l0 - j;
                const bool row = lag >= 0 && ((cs.rows >> lag) & 1u), ring = lag >= 0 && ((cs.ring >> lag) & 1u);
                const A* src = row0 - (ptrdiff_t)(row ? lag : 0) * a.proj_ld;
                const float* old = a.ring + (size_t)seq * a.ring_stride + (size_t)__shfl_sync(0xffffffffu, cs.place, lag & 31) * C + chan;
                const float* wt = w0 + (ptrdiff_t)(lag >= 0 ? R - lag : 0) * C;
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const int d = (lane + 32 * i) * V;
#pragma unroll
                    for (int v = 0; v < V; ++v) x[j][i][v] = w[j][i][v] = 0.f;
                    if (d < dim) {
                        if (row) load_v<V>(src + d, x[j][i]);
                        else if (ring) load_v<V>(old + d, x[j][i]);
                        if (row || ring) load_v<V>(wt + d, w[j][i]);
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int i = 0; i < NI; ++i)
#pragma unroll
                    for (int v = 0; v < V; ++v) y[i][v] += w[j][i][v] * x[j][i][v];
        }
    }
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int v = 0; v < V; ++v) y[i][v] *= sigmoid_f32(y[i][v]);
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&x)[V]) {
    if constexpr (V == 2) *(float2*)p = make_float2(x[0], x[1]);
    else *p = x[0];
}

template <typename A, int V, int NI>
__global__ void __launch_bounds__(kPrepWarps * 32) k_delta_prep(const DeltaRule a, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int G = a.kv_heads, H = a.heads;
    const int t = blockIdx.y, u = blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
    const bool on = u < G + H;
    // slots and positions are older than the step's first kernel
    const int seq = __ldcg(a.tok_seq + t), pos = __ldcg(a.tok_pos + t);
    const ConvSource cs = conv_source(a, t, seq, pos, lane);
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    if (on) {
        if (seq < 0 || seq >= a.max_slots || pos < 0) {
            if (lane == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        } else if (u < G) {
            float q[NI][V], k[NI][V];
            conv_silu<A, V, NI>(a, cs, t, seq, pos, a.q_off + u * a.dim, u * a.dim, a.dim, lane, q);
            conv_silu<A, V, NI>(a, cs, t, seq, pos, a.k_off + u * a.dim, (G + u) * a.dim, a.dim, lane, k);
            float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int v = 0; v < V; ++v) {  // past dim both are zero
                    qq += q[i][v] * q[i][v];
                    kk += k[i][v] * k[i][v];
                    qk += q[i][v] * k[i][v];
                }
            qq = warp_sum(qq);
            kk = warp_sum(kk);
            qk = warp_sum(qk);
            const float qs = 1.f / sqrtf(qq + 1e-6f) / sqrtf((float)a.dim), ks = 1.f / sqrtf(kk + 1e-6f);
            float* qo = a.qn + ((size_t)t * G + u) * a.dimP;
            float* ko = a.kn + ((size_t)t * G + u) * a.dimP;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int d = (lane + 32 * i) * V;
#pragma unroll
                for (int v = 0; v < V; ++v) {
                    q[i][v] *= qs;
                    k[i][v] *= ks;
                }
                if (d < a.dimP) {
                    store_v<V>(qo + d, q[i]);
                    store_v<V>(ko + d, k[i]);
                }
            }
            const int rep = H / G;
            for (int h = u * rep + lane; h < (u + 1) * rep; h += 32) a.bk[((size_t)t * H + h) * (a.head_decay ? 4 : 2) + 1] = qk * qs * ks;
        } else {
            const int h = u - G;
            const float rate = -expf(__ldg(a.a_log + h));
            const float* z = a.decay_in + (size_t)t * a.decay_ld + (size_t)h * a.dim;
            float zz[NI][V], dt[NI][V];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int d = (lane + 32 * i) * V;
#pragma unroll
                for (int v = 0; v < V; ++v) zz[i][v] = dt[i][v] = 0.f;
                if (d < a.dim && !a.head_decay) {
                    load_v<V>(z + d, zz[i]);
                    load_v<V>(a.dt_bias + h * a.dim + d, dt[i]);
                }
            }
            float v[NI][V];
            conv_silu<A, V, NI>(a, cs, t, seq, pos, a.v_off + h * a.vdim, 2 * G * a.dim + h * a.vdim, a.vdim, lane, v);
            float* vo = a.v + ((size_t)t * H + h) * a.vdimP;
            float* go = a.g + ((size_t)t * H + h) * a.dimP;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const int d = (lane + 32 * i) * V;
                if (d < a.vdimP) store_v<V>(vo + d, v[i]);
                if (d < a.dimP && !a.head_decay) {
                    float g[V];
#pragma unroll
                    for (int c = 0; c < V; ++c) g[c] = d < a.dim ? expf(rate * softplus_f32(zz[i][c] + dt[i][c])) : 0.f;
                    store_v<V>(go + d, g);
                }
            }
            if (lane == 0) {
                const A* row = (const A*)a.proj + (size_t)t * a.proj_ld;
                float* bk = a.bk + ((size_t)t * H + h) * (a.head_decay ? 4 : 2);
                bk[0] = sigmoid_f32(act_load(row + a.b_off + h));
                if (a.head_decay) bk[2] = expf(rate * softplus_f32(act_load(row + a.a_off + h) + __ldg(a.dt_bias + h)));
            }
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

// one output row of a head: o / rms(o) * weight * sigmoid(gate) or silu(gate). One warp; `at(d)` gives the raw value.
template <typename A, typename At>
__device__ __forceinline__ void delta_out_row(const DeltaRule& a, size_t t, int h, int lane, At at) {
    constexpr int NI = 8;  // vdim <= 256
    float o[NI], gate[NI], ss = 0.f;
    const float* g = a.gate_in ? a.gate_in + t * a.gate_ld + (size_t)h * a.vdim : nullptr;
    const A* gp = (const A*)a.proj + t * a.proj_ld + a.gate_off + (size_t)h * a.vdim;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int d = lane + 32 * i;
        o[i] = d < a.vdim ? at(d) : 0.f;
        gate[i] = d < a.vdim ? (g ? __ldcg(g + d) : act_load(gp + d)) : 0.f;
        ss += o[i] * o[i];
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
    A* out = (A*)a.out + t * a.out_ld + (size_t)h * a.vdim;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int d = lane + 32 * i;
        if (d < a.vdim) act_store(out + d, o[i] * inv * __ldg(a.out_norm + d) * sigmoid_f32(gate[i]) * (a.gate_silu ? gate[i] : 1.f));
    }
}

constexpr int kScanTokens = 8;  // tokens per stage
// of a token: q | k | decays (one per key channel) | v | beta, k . q (and the head's decay)
__host__ __device__ inline int scan_token_floats(int dimP, int cols, bool head_decay) { return (head_decay ? 2 : 3) * dimP + cols + 4; }
inline size_t scan_smem(int dimP, int cols, bool fused, bool head_decay) {
    return (size_t)kScanTokens * 2 * scan_token_floats(dimP, cols, head_decay) * 4 + (fused ? (size_t)kScanTokens * cols * 4 : 0);
}

// J = dimP / 32, C = value columns per lane: lane r of the eight that share C columns holds the key channels
// 4 (r + 8 j) + {0..3} of each. Blocks take `cols` columns of a head (grid z covers the head). Whatever C and cols
// are, a column's sums are formed in the same order. FUSED (one block per head): norm and gate of the output row here,
// else the raw row goes to `o` for k_delta_out.
template <typename A, int J, int C, bool FUSED, int NT, bool HEAD_DECAY>
__global__ void __launch_bounds__(NT) k_delta_scan(const DeltaRule a, int cols, unsigned long long* tl) {
    extern __shared__ __align__(16) float scan_buf[];
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5;
    const int h = blockIdx.x, H = a.heads, G = a.kv_heads, kvh = h / (H / G);
    const int r = tid & 7, cb = blockIdx.z * cols, c0 = cb + (tid >> 3) * C;  // the block's and this lane's first column
    constexpr int dimP = 32 * J;
    const int vdimP = a.vdimP, tokf = scan_token_floats(dimP, cols, HEAD_DECAY);
    constexpr int vOff = (HEAD_DECAY ? 2 : 3) * dimP;  // within a token's floats
    const int ncols = min(cols, vdimP - cb);  // columns of this block that exist (a multiple of 4)
    float* o_s = scan_buf + (size_t)2 * kScanTokens * tokf;  // FUSED: [kScanTokens][cols]
    // The token lists and the state are older than this step's first kernel (a full dependency of the stream), so
    // the state is fetched while the preparation is still running.
    const int first = __ldcg(a.seg_first + blockIdx.y), count = __ldcg(a.seg_count + blockIdx.y);
    const int slot = __ldcg(a.tok_seq + first), pos0 = __ldcg(a.tok_pos + first);
    const bool ok = slot >= 0 && slot < a.max_slots && pos0 >= 0;
    float* st = a.state + (size_t)(ok ? slot : 0) * a.state_stride + (size_t)h * vdimP * dimP;
    f32x2 S[C][J][2];
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
        for (int j = 0; j < J; ++j) {
            ulonglong2 v = make_ulonglong2(0ull, 0ull);
            if (ok && pos0 > 0 && c0 + c < vdimP) v = __ldcg((const ulonglong2*)(st + (size_t)(c0 + c) * dimP + 4 * (r + 8 * j)));
            S[c][j][0] = v.x;
            S[c][j][1] = v.y;
        }
    pdl_wait();
    if (tid == 0) tl_mark(tl, 1);
    if (!ok) {
        if (tid == 0) dev_fail(a.status, DEV_ERR_BOUNDS);
        return;
    }
    auto fetch = [&](int tile) {  // tokens [tile * kScanTokens, ...) of the run into buffer tile & 1; warp = token
        float* buf = scan_buf + (size_t)(tile & 1) * kScanTokens * tokf;
        const int n = min(kScanTokens, count - tile * kScanTokens);
        for (int k = warp; k < n; k += nwarps) {
            const size_t t = (size_t)first + tile * kScanTokens + k;
            float* dst = buf + (size_t)k * tokf;
            const float *q = a.qn + (t * G + kvh) * dimP, *kk = a.kn + (t * G + kvh) * dimP, *g = HEAD_DECAY ? nullptr : a.g + (t * H + h) * dimP;
            const float* v = a.v + (t * H + h) * vdimP + cb;
            for (int p = lane * 4; p < dimP; p += 128) {
                cp_async16(dst + p, q + p);
                cp_async16(dst + dimP + p, kk + p);
                if constexpr (!HEAD_DECAY) cp_async16(dst + 2 * dimP + p, g + p);
            }
            for (int p = lane * 4; p < ncols; p += 128) cp_async16(dst + vOff + p, v + p);
            if (lane == 0) {
                if constexpr (HEAD_DECAY) cp_async16(dst + vOff + cols, a.bk + (t * H + h) * 4);
                else cp_async8(dst + vOff + cols, a.bk + (t * H + h) * 2);
            }
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
        // The token's vectors in registers; with room for them, the next token's are requested before this token's sums
        // are exchanged, so that the exchange hides the shared-memory latency.
        constexpr bool AHEAD = !FUSED && J <= 2;
        ulonglong2 q4[J], k4[J], g4[J];
        auto vectors = [&](int k) {
            const float* tok = buf + (size_t)k * tokf;
#pragma unroll
            for (int j = 0; j < J; ++j) {
                const int d = 4 * (r + 8 * j);
                q4[j] = *(const ulonglong2*)(tok + d);
                k4[j] = *(const ulonglong2*)(tok + dimP + d);
                if constexpr (!HEAD_DECAY) g4[j] = *(const ulonglong2*)(tok + 2 * dimP + d);
            }
        };
        if (AHEAD) vectors(0);
        for (int k = 0; k < n; ++k) {
            const float* tok = buf + (size_t)k * tokf;
            if (!AHEAD) vectors(k);
            f32x2 t2[C], w2[C];
#pragma unroll
            for (int c = 0; c < C; ++c) t2[c] = w2[c] = 0ull;
            f32x2 gh = 0ull;
            if constexpr (HEAD_DECAY) {
                const float g = tok[vOff + cols + 2];
                gh = pack2(g, g);
            }
#pragma unroll
            for (int j = 0; j < J; ++j) {
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    S[c][j][0] = mul2(S[c][j][0], HEAD_DECAY ? gh : g4[j].x);
                    S[c][j][1] = mul2(S[c][j][1], HEAD_DECAY ? gh : g4[j].y);
                    t2[c] = fma2(S[c][j][0], k4[j].x, t2[c]);
                    w2[c] = fma2(S[c][j][0], q4[j].x, w2[c]);
                    t2[c] = fma2(S[c][j][1], k4[j].y, t2[c]);
                    w2[c] = fma2(S[c][j][1], q4[j].y, w2[c]);
                }
            }
            ulonglong2 kk[J];  // this token's key for the update
            if (AHEAD) {
#pragma unroll
                for (int j = 0; j < J; ++j) kk[j] = k4[j];
                vectors(min(k + 1, n - 1));
            }
            const float2 bk = *(const float2*)(tok + vOff + cols);
            // Sums over the eight lanes by halving exchange (partners 4, 2, 1 lanes away): lane r ends with S^T k and
            // S^T q of column r (C = 8), or of column r & 3 with S^T k in lanes 0-3 and S^T q in lanes 4-7 (C = 4).
            float uc[C];
            if constexpr (C == 8) {
                float tx[4], wx[4], ty[2], wy[2];
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float t0 = sum2(t2[c]), t1 = sum2(t2[c + 4]), w0 = sum2(w2[c]), w1 = sum2(w2[c + 4]);
                    tx[c] = ((r & 4) ? t1 : t0) + __shfl_xor_sync(0xffffffffu, (r & 4) ? t0 : t1, 4);
                    wx[c] = ((r & 4) ? w1 : w0) + __shfl_xor_sync(0xffffffffu, (r & 4) ? w0 : w1, 4);
                }
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    ty[c] = ((r & 2) ? tx[c + 2] : tx[c]) + __shfl_xor_sync(0xffffffffu, (r & 2) ? tx[c] : tx[c + 2], 2);
                    wy[c] = ((r & 2) ? wx[c + 2] : wx[c]) + __shfl_xor_sync(0xffffffffu, (r & 2) ? wx[c] : wx[c + 2], 2);
                }
                const float ts = ((r & 1) ? ty[1] : ty[0]) + __shfl_xor_sync(0xffffffffu, (r & 1) ? ty[0] : ty[1], 1);
                const float ws = ((r & 1) ? wy[1] : wy[0]) + __shfl_xor_sync(0xffffffffu, (r & 1) ? wy[0] : wy[1], 1);
                const int col = c0 + r;
                const float v = col - cb < ncols ? tok[vOff + (col - cb)] : 0.f;
                const float u = bk.x * (v - ts);
#pragma unroll
                for (int c = 0; c < 8; ++c) uc[c] = __shfl_sync(0xffffffffu, u, (lane & ~7) | c);
                if (col - cb < ncols) {
                    const float o = ws + u * bk.y;
                    if constexpr (FUSED) o_s[k * cols + (col - cb)] = o;
                    else a.o[((size_t)(first + tile * kScanTokens + k) * H + h) * vdimP + col] = o;
                }
            } else {
                static_assert(C == 4, "");
                float x4[4], x2[2];
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const float tt = sum2(t2[c]), ww = sum2(w2[c]);
                    x4[c] = ((r & 4) ? ww : tt) + __shfl_xor_sync(0xffffffffu, (r & 4) ? tt : ww, 4);
                }
#pragma unroll
                for (int c = 0; c < 2; ++c) x2[c] = ((r & 2) ? x4[c + 2] : x4[c]) + __shfl_xor_sync(0xffffffffu, (r & 2) ? x4[c] : x4[c + 2], 2);
                const float x = ((r & 1) ? x2[1] : x2[0]) + __shfl_xor_sync(0xffffffffu, (r & 1) ? x2[0] : x2[1], 1);
                const int col = c0 + (r & 3);
                const float v = col - cb < ncols ? tok[vOff + (col - cb)] : 0.f;
                const float u = bk.x * (v - x);  // meaningful in lanes r < 4
#pragma unroll
                for (int c = 0; c < 4; ++c) uc[c] = __shfl_sync(0xffffffffu, u, (lane & ~7) | c);
                const float mine = (r & 2) ? ((r & 1) ? uc[3] : uc[2]) : ((r & 1) ? uc[1] : uc[0]);
                if (r >= 4 && col - cb < ncols) {
                    const float o = x + mine * bk.y;
                    if constexpr (FUSED) o_s[k * cols + (col - cb)] = o;
                    else a.o[((size_t)(first + tile * kScanTokens + k) * H + h) * vdimP + col] = o;
                }
            }
#pragma unroll
            for (int j = 0; j < J; ++j) {
                if (!AHEAD) kk[j] = *(const ulonglong2*)(tok + dimP + 4 * (r + 8 * j));
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    const f32x2 uu = pack2(uc[c], uc[c]);
                    S[c][j][0] = fma2(kk[j].x, uu, S[c][j][0]);
                    S[c][j][1] = fma2(kk[j].y, uu, S[c][j][1]);
                }
            }
        }
        __syncthreads();
        if constexpr (FUSED) {  // the head's norm and gate, one warp per token of the stage
            for (int k = warp; k < n; k += nwarps) {
                const size_t t = (size_t)first + tile * kScanTokens + k;
                delta_out_row<A>(a, t, h, lane, [&](int d) { return o_s[k * cols + d]; });
            }
        }
    }
    if (count > 0) {
#pragma unroll
        for (int c = 0; c < C; ++c)
#pragma unroll
            for (int j = 0; j < J; ++j)
                if (c0 + c < vdimP)
                    *(ulonglong2*)(st + (size_t)(c0 + c) * dimP + 4 * (r + 8 * j)) = make_ulonglong2(S[c][j][0], S[c][j][1]);
    }
    // The last inputs of the convolutions, for the run's continuation. The preparation of this launch has finished
    // reading the ring. A head keeps its value channels, the first head of a group the shared query and key channels.
    const int R = a.taps - 1, chans = 2 * G * a.dim + H * a.vdim;
    for (int i = 0; i < min(R, count); ++i) {
        const int t = first + count - 1 - i, pos = pos0 + count - 1 - i;
        const A* row = (const A*)a.proj + (size_t)t * a.proj_ld;
        float* ring = a.ring + (size_t)slot * a.ring_stride + (size_t)(pos % R) * chans;
        for (int d = cb + tid; d < min(a.vdim, cb + cols); d += blockDim.x)
            ring[2 * G * a.dim + h * a.vdim + d] = act_load(row + a.v_off + h * a.vdim + d);
        if (h % (H / G) == 0 && blockIdx.z == 0)
            for (int d = tid; d < a.dim; d += blockDim.x) {
                ring[kvh * a.dim + d] = act_load(row + a.q_off + kvh * a.dim + d);
                ring[(G + kvh) * a.dim + d] = act_load(row + a.k_off + kvh * a.dim + d);
            }
    }
    if (tid == 0) tl_mark(tl, 2);
}

// prompts: norm and gate of the raw output rows, one warp per (token, head)
template <typename A>
__global__ void __launch_bounds__(kPrepWarps * 32) k_delta_out(const DeltaRule a, unsigned long long* tl) {
    if (threadIdx.x == 0) tl_mark(tl, 0);
    pdl_launch_dependents();
    pdl_wait();
    if (threadIdx.x == 0) tl_mark(tl, 1);
    const int h = blockIdx.x * kPrepWarps + (threadIdx.x >> 5);
    if (h < a.heads) {
        const size_t t = blockIdx.y;
        const float* o = a.o + (t * a.heads + h) * a.vdimP;
        delta_out_row<A>(a, t, h, threadIdx.x & 31, [&](int d) { return __ldcg(o + d); });
    }
    if (threadIdx.x == 0) tl_mark(tl, 2);
}

template <typename A, int J, int C, bool FUSED, int NT, bool HD>
cudaError_t scan_attr() {
    cudaError_t e = cudaFuncSetAttribute(k_delta_scan<A, J, C, FUSED, NT, HD>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)scan_smem(32 * J, 256, true, HD));
    return e == cudaSuccess ? prefer_max_shared(k_delta_scan<A, J, C, FUSED, NT, HD>) : e;
}
// FUSED blocks hold a whole head of up to 256 columns; the others 128 threads, 128 columns (C = 8) or 64 (C = 4). Eight
// columns of more than 128 key channels do not fit a lane's registers, and heads that wide are not fused.
template <typename A, int J, bool HD>
cudaError_t scan_attrs_hd() {
    cudaError_t e = cudaSuccess;
    if constexpr (J <= 4) {
        e = scan_attr<A, J, 8, true, 256, HD>();
        if (e == cudaSuccess) e = scan_attr<A, J, 4, true, 256, HD>();
        if (e == cudaSuccess) e = scan_attr<A, J, 8, false, 128, HD>();
    }
    if (e == cudaSuccess) e = scan_attr<A, J, 4, false, 128, HD>();
    return e;
}
template <typename A, int J>
cudaError_t scan_attrs() {
    const cudaError_t e = scan_attrs_hd<A, J, false>();
    return e == cudaSuccess ? scan_attrs_hd<A, J, true>() : e;
}
template <typename A>
cudaError_t delta_attrs() {
    cudaError_t e = scan_attrs<A, 1>();
    if (e == cudaSuccess) e = scan_attrs<A, 2>();
    if (e == cudaSuccess) e = scan_attrs<A, 3>();
    if (e == cudaSuccess) e = scan_attrs<A, 4>();
    if (e == cudaSuccess) e = scan_attrs<A, 8>();
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_out<A>);
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_prep<A, 1, 8>);
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_prep<A, 2, 1>);
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_prep<A, 2, 2>);
    if (e == cudaSuccess) e = prefer_max_shared(k_delta_prep<A, 2, 4>);
    return e;
}

template <typename A, int J, bool HD>
void launch_scan_hd(const DeltaRule& a, int n_segs, bool fused, int num_sms, cudaStream_t s, bool pdl, unsigned long long* tl) {
    auto go = [&](auto kernel, int C, int cols, bool f) {
        const int threads = (cols / C * 8 + 31) / 32 * 32;
        launch_k(kernel, dim3(a.heads, n_segs, (a.vdimP + cols - 1) / cols), dim3(threads), scan_smem(32 * J, cols, f, HD), s, pdl, a, cols, tl);
    };
    const int whole = (a.vdimP + 7) / 8 * 8;
    if constexpr (J <= 4) {
        if (fused && a.heads * n_segs < num_sms && whole <= 128) return go(k_delta_scan<A, J, 4, true, 256, HD>, 4, whole, true);
        if (fused) return go(k_delta_scan<A, J, 8, true, 256, HD>, 8, whole, true);
        // eight columns per lane need the fewest shared-memory reads; with few sequences half as many columns per lane
        // and twice the warps make a token's chain of steps shorter
        const long long warps = (long long)a.heads * n_segs * ((a.vdimP + 31) / 32);
        if (warps >= 3ll * num_sms) return go(k_delta_scan<A, J, 8, false, 128, HD>, 8, whole < 128 ? whole : 128, false);
    }
    go(k_delta_scan<A, J, 4, false, 128, HD>, 4, whole < 64 ? whole : 64, false);
}
template <typename A, int J>
void launch_scan(const DeltaRule& a, int n_segs, bool fused, int num_sms, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (a.head_decay) launch_scan_hd<A, J, true>(a, n_segs, fused, num_sms, s, pdl, tl);
    else launch_scan_hd<A, J, false>(a, n_segs, fused, num_sms, s, pdl, tl);
}
template <typename A>
void launch_scan_j(const DeltaRule& a, int n_segs, bool fused, int num_sms, cudaStream_t s, bool pdl, unsigned long long* tl) {
    switch (a.dimP) {
        case 32: return launch_scan<A, 1>(a, n_segs, fused, num_sms, s, pdl, tl);
        case 64: return launch_scan<A, 2>(a, n_segs, fused, num_sms, s, pdl, tl);
        case 96: return launch_scan<A, 3>(a, n_segs, fused, num_sms, s, pdl, tl);
        case 128: return launch_scan<A, 4>(a, n_segs, fused, num_sms, s, pdl, tl);
        default: return launch_scan<A, 8>(a, n_segs, fused, num_sms, s, pdl, tl);
    }
}
template <typename A>
void launch_prep(const DeltaRule& a, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const dim3 grid((a.kv_heads + a.heads + kPrepWarps - 1) / kPrepWarps, T), block(kPrepWarps * 32);
    const int wide = a.dimP > a.vdimP ? a.dimP : a.vdimP;
    if (a.dim % 2 || a.vdim % 2) launch_k(k_delta_prep<A, 1, 8>, grid, block, 0, s, pdl, a, tl);
    else if (wide <= 64) launch_k(k_delta_prep<A, 2, 1>, grid, block, 0, s, pdl, a, tl);
    else if (wide <= 128) launch_k(k_delta_prep<A, 2, 2>, grid, block, 0, s, pdl, a, tl);
    else launch_k(k_delta_prep<A, 2, 4>, grid, block, 0, s, pdl, a, tl);
}

}  // namespace

int delta_prepare() {
    cudaError_t e = delta_attrs<bf16>();
    if (e == cudaSuccess) e = delta_attrs<float>();
    return (int)e;
}
int delta_padded_dim(int dim) { return dim <= 128 ? (dim + 31) / 32 * 32 : 256; }

void launch_delta_prep(const DeltaRule& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) launch_prep<float>(a, T, s, pdl, tl);
    else launch_prep<bf16>(a, T, s, pdl, tl);
}
void launch_delta_scan(const DeltaRule& a, bool f32, int n_segs, bool fused, int num_sms, cudaStream_t s, bool pdl, unsigned long long* tl) {
    if (f32) launch_scan_j<float>(a, n_segs, fused, num_sms, s, pdl, tl);
    else launch_scan_j<bf16>(a, n_segs, fused, num_sms, s, pdl, tl);
}
void launch_delta_out(const DeltaRule& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl) {
    const dim3 grid((a.heads + kPrepWarps - 1) / kPrepWarps, T), block(kPrepWarps * 32);
    if (f32) launch_k(k_delta_out<float>, grid, block, 0, s, pdl, a, tl);
    else launch_k(k_delta_out<bf16>, grid, block, 0, s, pdl, a, tl);
}

}  // namespace tffn
