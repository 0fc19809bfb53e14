// Latent attention on the tensor cores, prompts and decoding alike. A cached row is the key of every head (the heads' key
// projections are folded into the queries) and its first `rank` columns are the value, so the heads of up to eight tokens of
// a sequence are the 128 rows of one tile:
//   S[row, key] = Q[row, :] . K[key, :]      tcgen05.mma, Q and K in shared memory (both K-major)
//   O[row, :]  += P[row, :] . K[:, columns]  tcgen05.mma, P in tensor memory, K read the other way round (N-major)
// One CTA = the rows of one tile x at most 256 value columns x one context split, 6 warps:
//   warps 0-3  thread = row: S out of tensor memory, online softmax in fp32, P back as a bf16 pair (hi + lo, 16 mantissa
//              bits), the rotated part of Q at the start, and the output rows at the end
//   warp 4     TMA producer: Q, then 64 keys (two pages) per stage, 64 columns per box with the 128-byte swizzle
//   warp 5     tensor memory, MMA issue
// The reference maximum of a row moves only when it would be exceeded by more than 2^8, so O is rarely rescaled. Splits
// leave partial rows and the last one to finish (a ticket, no waiting) adds them up in split order.
// Rows of a page past the end of a sequence are finite (zeros or an earlier request's normed latents) and weigh zero.
#include "act.cuh"
#include "launch.h"
#include "ptx.cuh"
#include <algorithm>
#include <cstring>

namespace tffn {

namespace {

constexpr int TK = 64;                     // keys per stage
constexpr int kRowsMax = 128;              // rows of a tile
constexpr int kSliceCols = 256;            // value columns of a CTA
constexpr int kThreads = 192;
constexpr int kMaxStages = 4;
constexpr int kBlockBytes = TK * 128;      // 64 keys x 64 columns
constexpr int kSmemLimit = 227 * 1024;
constexpr uint32_t kTmemCols = 512, kColS = 0, kColP = 2 * TK, kColO = 3 * TK;  // S twice, P hi | lo, O
constexpr float kNeg = -1e30f;

struct LatentDev {
    CUtensorMap tmQ;  // [T * heads][rank], box 64 x q_rows
    CUtensorMap tmK;  // [pages * kPageTokens][row], box 64 x kPageTokens
    const bf16* q_up; // rotated parts: [T][q_up_ld], `rot` columns per head from column rot_off
    long long q_up_ld;
    int rot_off, rot;
    const float2* rope;
    int max_pos;
    const int* block_table;
    int max_pages_per_seq, num_pages;
    const int *tok_seq, *tok_pos;
    const int *grp_first, *grp_count;  // nullptr: every row is a group of its own
    int heads, part_heads, parts;      // heads of a tile; parts of at most kRowsMax heads
    int tile_tokens, subs;             // tokens of a tile; tiles a group may need
    int q_rows;                        // rows of the Q box
    int rank, slices, slice_cols;
    int stages, splits, early;
    float scale_log2;
    const bf16* gate;                  // [T][gate_ld]
    long long gate_ld;
    bf16* out;                         // [T][heads][head_ld]
    int head_ld;
    float* ws;
    int* counters;
    int* status;
    unsigned long long* tl;
};

// shared-memory descriptor of an operand whose rows are its K extent: 64 columns (128 swizzled bytes) per row, groups of 64
// columns kBlockBytes apart (leading byte offset), groups of 8 rows 1024 bytes apart (stride byte offset)
__device__ __forceinline__ uint64_t desc_n128(uint32_t smem_addr) {
    return (uint64_t)((smem_addr & 0x3FFFFu) >> 4) | ((uint64_t)(kBlockBytes >> 4) << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
// D[tmem] (+)= A[tmem] * B[smem]
__device__ __forceinline__ void umma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d_tmem),
        "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15};" ::"r"(v[0]),
        "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]),
        "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__global__ void __launch_bounds__(kThreads, 1) k_attn_latent(const __grid_constant__ LatentDev p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t k_full[kMaxStages], k_empty[kMaxStages], s_full[2], q_full, p_full, pv_done;
    __shared__ uint32_t tmem_slot;
    __shared__ int s_last;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

    // unit = ((group * subs + sub) * parts + part) * slices + slice
    const int unit = blockIdx.x, slice = unit % p.slices, part = unit / p.slices % p.parts;
    const int sub = unit / p.slices / p.parts % p.subs, group = unit / p.slices / p.parts / p.subs;
    const int g_first = p.grp_first ? __ldcg(p.grp_first + group) : group, g_count = p.grp_first ? __ldcg(p.grp_count + group) : 1;
    const int t0 = g_first + sub * p.tile_tokens, ntok = min(p.tile_tokens, g_count - sub * p.tile_tokens);
    const int head0 = part * p.part_heads, nheads = min(p.part_heads, p.heads - head0);
    const int seq = __ldcg(p.tok_seq + (ntok > 0 ? t0 : g_first));
    const int len = ntok > 0 ? __ldcg(p.tok_pos + t0 + ntok - 1) + 1 : 0;  // positions ascend within a group
    int per_split = (len + p.splits - 1) / p.splits;
    per_split = (per_split + TK - 1) / TK * TK;
    const int k_begin = blockIdx.y * per_split, k_end = min(len, k_begin + per_split);
    const int n_tiles = k_end > k_begin ? (k_end - k_begin + TK - 1) / TK : 0;
    const bool len_ok = len <= p.max_pos && (len + kPageTokens - 1) / kPageTokens <= p.max_pages_per_seq;

    const int rank_blocks = (p.rank + 63) / 64, rot_blocks = (p.rot + 63) / 64, blocks = rank_blocks + rot_blocks;
    const int q_block = p.q_rows * 128, stage_bytes = blocks * kBlockBytes;
    uint8_t* const q_s = smem;
    uint8_t* const k_s = smem + blocks * q_block;

    if (tid == 0) {
        tl_mark(p.tl, 0);
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
        }
        mbar_init(&s_full[0], 1);
        mbar_init(&s_full[1], 1);
        mbar_init(&q_full, 1 + kRowsMax);
        mbar_init(&p_full, kRowsMax);
        mbar_init(&pv_done, 1);
        fence_mbar_init();
    }
    if (warp == 5) {
        tmem_alloc(&tmem_slot, kTmemCols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_launch_dependents();
    if (!len_ok && tid == 0) dev_fail(p.status, DEV_ERR_BOUNDS);
    const int tiles = len_ok ? n_tiles : 0;

    // this thread's row
    const int row_tok = tid / p.part_heads, row_head = tid % p.part_heads;
    const bool active = tid < kRowsMax && row_tok < ntok && row_head < nheads;
    const int row_t = t0 + (active ? row_tok : 0);
    float m_ref = kNeg, l_sum = 0.f;

    if (warp == 4) {
        if (lane == 0) {
            prefetch_tmap(&p.tmQ);
            prefetch_tmap(&p.tmK);
            const int* bt = p.block_table + (size_t)seq * p.max_pages_per_seq;
            const int last_page = (len - 1) / kPageTokens;
            auto load_tile = [&](int j) {
                const int st = j % p.stages;
                uint8_t* dst = k_s + st * stage_bytes;
                mbar_arrive_expect_tx(&k_full[st], stage_bytes);
                for (int h = 0; h < TK / kPageTokens; ++h) {
                    // a page past the end is replaced by the last one; its keys are masked
                    int pg = __ldg(bt + min((k_begin + j * TK) / kPageTokens + h, last_page));
                    if (pg < 0 || pg >= p.num_pages) {
                        dev_fail(p.status, DEV_ERR_BOUNDS);
                        pg = 0;
                    }
                    for (int b = 0; b < blocks; ++b)
                        tma_load_2d(dst + b * kBlockBytes + h * kPageTokens * 128, &p.tmK, b * 64, pg * kPageTokens, &k_full[st]);
                }
            };
            // In decode everything but the newest row is older than the step's first kernel
            int next = 0;
            if (p.early)
                while (next < min(p.stages, tiles) && k_begin + (next + 1) * TK <= last_page * kPageTokens) load_tile(next++);
            pdl_wait();
            tl_mark(p.tl, 1);
            if (tiles > 0) mbar_arrive_expect_tx(&q_full, rank_blocks * q_block);  // no copy that nobody waits for
            for (int b = 0; b < rank_blocks && tiles > 0; ++b) tma_load_2d(q_s + b * q_block, &p.tmQ, b * 64, t0 * p.heads + head0, &q_full);
            for (; next < tiles; ++next) {
                if (next >= p.stages && !mbar_wait(&k_empty[next % p.stages], (uint32_t)(next / p.stages - 1) & 1u, p.status, DEV_ERR_EMPTY_WAIT)) break;
                load_tile(next);
            }
        }
    } else if (warp == 5) {
        if (lane == 0 && tiles > 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(kRowsMax, TK);
            const int ncols = min(p.slice_cols, (p.rank - slice * p.slice_cols + 15) / 16 * 16);
            const uint32_t idesc_o = umma_idesc_bf16(kRowsMax, ncols) | (1u << 16);  // B is N-major
            const uint32_t q_a = smem_u32(q_s), k_a = smem_u32(k_s);
            const int rank_steps = (p.rank + 15) / 16, rot_steps = (p.rot + 15) / 16;
            auto scores = [&](int j) {
                const int st = j % p.stages;
                if (!mbar_wait(&k_full[st], (uint32_t)(j / p.stages) & 1u, p.status, DEV_ERR_FULL_WAIT)) return false;
                tc_fence_after();
                const uint32_t kb = k_a + st * stage_bytes, d = tmem + kColS + (j & 1) * TK;
                for (int i = 0; i < rank_steps + rot_steps; ++i) {
                    const int i2 = i < rank_steps ? i : rank_blocks * 4 + (i - rank_steps);
                    const uint32_t in = (uint32_t)(i2 & 3) * 32;
                    umma_bf16(d, umma_desc_k128(q_a + (i2 >> 2) * q_block + in), umma_desc_k128(kb + (i2 >> 2) * kBlockBytes + in), idesc_s, i > 0);
                }
                umma_commit(&s_full[j & 1]);
                return true;
            };
            const bool ahead = p.stages > 1;  // the scores of the next tile run while this tile's softmax does
            bool ok = mbar_wait(&q_full, 0, p.status, DEV_ERR_FULL_WAIT) && scores(0);
            for (int j = 0; j < tiles && ok; ++j) {
                if (ahead && j + 1 < tiles) ok = scores(j + 1);
                if (!ok || !mbar_wait(&p_full, (uint32_t)j & 1u, p.status, DEV_ERR_ACC_WAIT)) break;
                tc_fence_after();
                const uint32_t v = k_a + (j % p.stages) * stage_bytes + slice * (p.slice_cols / 64) * kBlockBytes;
#pragma unroll
                for (int half = 0; half < 2; ++half)  // P hi, P lo
#pragma unroll
                    for (int kk = 0; kk < TK / 16; ++kk)
                        umma_bf16_ts(tmem + kColO, tmem + kColP + half * (TK / 2) + kk * 8, desc_n128(v + kk * 2048), idesc_o, j > 0 || half > 0 || kk > 0);
                umma_commit(&k_empty[j % p.stages]);
                umma_commit(&pv_done);
                if (!ahead && j + 1 < tiles) ok = scores(j + 1);
            }
        }
    } else {
        pdl_wait();
        // the rotated part of Q: block rank_blocks and on, columns past `rot` zero
        {
            const int half = p.rot / 2, zero_to = (p.rot + 15) / 16 * 16;
            auto put = [&](int r, int col, float v) {
                uint8_t* blk = q_s + (rank_blocks + col / 64) * q_block;
                const int c = col % 64;
                *(bf16*)(blk + r * 128 + (((c >> 3) ^ (r & 7)) << 4) + (c & 7) * 2) = __float2bfloat16_rn(v);
            };
            const int rows = ntok * p.part_heads;
            for (int i = tid; i < rows * half; i += kRowsMax) {
                const int r = i / half, c = i % half, h = r % p.part_heads, t = t0 + r / p.part_heads;
                if (h >= nheads) continue;
                const bf16* src = p.q_up + (size_t)t * p.q_up_ld + p.rot_off + (size_t)(head0 + h) * p.rot;
                const float u = act_load(src + c), v = act_load(src + half + c);
                const int pos = __ldcg(p.tok_pos + t);
                const float2 cs = __ldg(p.rope + (size_t)(pos >= 0 && pos < p.max_pos ? pos : 0) * half + c);
                put(r, c, u * cs.x - v * cs.y);
                put(r, half + c, v * cs.x + u * cs.y);
            }
            for (int i = tid; i < rows * (zero_to - p.rot); i += kRowsMax) put(i / (zero_to - p.rot), p.rot + i % (zero_to - p.rot), 0.f);
            fence_proxy_async_smem();
            mbar_arrive(&q_full);
        }
        const int my_end = active ? min(k_end, __ldcg(p.tok_pos + row_t) + 1) : 0;
        const uint32_t lane_addr = tmem + ((uint32_t)(warp * 32) << 16);
        const int ncols16 = (min(p.slice_cols, p.rank - slice * p.slice_cols) + 15) / 16;
        bool ok = true;
        for (int j = 0; j < tiles && ok; ++j) {
            ok = __all_sync(0xffffffffu, mbar_wait(&s_full[j & 1], (uint32_t)(j >> 1) & 1u, p.status, DEV_ERR_ACC_WAIT));
            if (!ok) break;
            tc_fence_after();
            uint32_t s[TK / 16][16];
#pragma unroll
            for (int c = 0; c < TK / 16; ++c) tmem_ld16(lane_addr + kColS + (j & 1) * TK + c * 16, s[c]);
            tc_wait_ld();
            const int live = my_end - (k_begin + j * TK);  // visible keys of this tile
            float mx = kNeg;
#pragma unroll
            for (int i = 0; i < TK; ++i) {
                const float v = i < live ? __uint_as_float(s[i >> 4][i & 15]) * p.scale_log2 : kNeg;
                s[i >> 4][i & 15] = __float_as_uint(v);
                mx = fmaxf(mx, v);
            }
            float corr = 1.f;
            bool moved = false;
            if (j == 0) {
                m_ref = mx;
            } else if (mx > m_ref + 8.f) {
                corr = exp2_fast(m_ref - mx);
                m_ref = mx;
                moved = true;
            }
            l_sum *= corr;
            uint32_t hi[TK / 32][16], lo[TK / 32][16];
#pragma unroll
            for (int i = 0; i < TK; i += 2) {
                const float a = i < live ? exp2_fast(__uint_as_float(s[i >> 4][i & 15]) - m_ref) : 0.f;
                const float b = i + 1 < live ? exp2_fast(__uint_as_float(s[i >> 4][(i & 15) + 1]) - m_ref) : 0.f;
                l_sum += a + b;
                const __nv_bfloat162 h2 = __floats2bfloat162_rn(a, b);
                const uint32_t h = *(const uint32_t*)&h2;
                const __nv_bfloat162 l2 = __floats2bfloat162_rn(a - bf16_lo(h), b - bf16_hi(h));
                hi[i >> 5][(i & 31) >> 1] = h;
                lo[i >> 5][(i & 31) >> 1] = *(const uint32_t*)&l2;
            }
            if (j > 0) {  // P and O are free again once the previous tile's product is done
                ok = __all_sync(0xffffffffu, mbar_wait(&pv_done, (uint32_t)(j - 1) & 1u, p.status, DEV_ERR_ACC_WAIT));
                if (!ok) break;
                tc_fence_after();
                if (__any_sync(0xffffffffu, moved)) {
                    for (int c = 0; c < ncols16; ++c) {
                        uint32_t o[16];
                        tmem_ld16(lane_addr + kColO + c * 16, o);
                        tc_wait_ld();
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                        tmem_st16(lane_addr + kColO + c * 16, o);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < TK / 32; ++c) {
                tmem_st16(lane_addr + kColP + c * 16, hi[c]);
                tmem_st16(lane_addr + kColP + TK / 2 + c * 16, lo[c]);
            }
            tc_wait_st();
            tc_fence_before();
            mbar_arrive(&p_full);
        }
        if (tiles > 0 && ok) ok = __all_sync(0xffffffffu, mbar_wait(&pv_done, (uint32_t)(tiles - 1) & 1u, p.status, DEV_ERR_ACC_WAIT));
        tc_fence_after();
        // ---- this slice's columns of the row
        const int col0 = slice * p.slice_cols;
        float mult = 0.f;
        if (active && l_sum > 0.f && p.splits == 1) {
            const float z = act_load(p.gate + (size_t)row_t * p.gate_ld + head0 + row_head);
            mult = sigmoid_f32(z) / l_sum;
        }
        bf16* dst = p.out + ((size_t)row_t * p.heads + head0 + row_head) * p.head_ld + col0;
        // partial rows: [unit][split][row][slice_cols + 2], the last two: maximum, sum
        float* part_row = p.ws + (((size_t)unit * p.splits + blockIdx.y) * p.part_heads + row_head) * (p.slice_cols + 2);
        if (tiles > 0 && ok) {
            for (int c = 0; c < ncols16; ++c) {
                uint32_t o[16];
                tmem_ld16(lane_addr + kColO + c * 16, o);
                tc_wait_ld();
                if (active && p.splits == 1) {
#pragma unroll
                    for (int i = 0; i < 16; i += 8) {
                        uint32_t w[4];
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            w[k] = (uint32_t)bf16_bits(__uint_as_float(o[i + 2 * k]) * mult) | ((uint32_t)bf16_bits(__uint_as_float(o[i + 2 * k + 1]) * mult) << 16);
                        if (col0 + c * 16 + i < p.rank) *(uint4*)(dst + c * 16 + i) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                } else if (active) {
#pragma unroll
                    for (int i = 0; i < 16; i += 2) *(uint2*)(part_row + c * 16 + i) = make_uint2(o[i], o[i + 1]);
                }
                __syncwarp();
            }
        }
        if (p.splits > 1 && active) {
            part_row[p.slice_cols] = m_ref;
            part_row[p.slice_cols + 1] = l_sum;
        }
    }
    tc_fence_before();
    if (p.splits > 1) __threadfence();
    __syncthreads();
    if (warp == 5) tmem_dealloc(tmem, kTmemCols);
    if (p.splits > 1) {
        if (tid == 0) {
            const int old = atomicAdd(&p.counters[unit], 1);
            s_last = old == p.splits - 1;
            if (s_last) p.counters[unit] = 0;
        }
        __syncthreads();
        if (s_last && ntok > 0) {
            __threadfence();
            const int cols = min(p.slice_cols, p.rank - slice * p.slice_cols), ld = p.slice_cols + 2, pad_cols = (cols + 7) / 8 * 8;
            const float* parts = p.ws + (size_t)unit * p.splits * p.part_heads * ld;
            for (int h = warp; h < nheads; h += kThreads / 32) {
                const float* row = parts + (size_t)h * ld;
                const size_t step = (size_t)p.part_heads * ld;
                float M = kNeg, L = 0.f;
                for (int z = 0; z < p.splits; ++z) M = fmaxf(M, __ldcg(row + z * step + p.slice_cols));
                for (int z = 0; z < p.splits; ++z) L += __ldcg(row + z * step + p.slice_cols + 1) * exp2_fast(__ldcg(row + z * step + p.slice_cols) - M);
                const float mult = sigmoid_f32(act_load(p.gate + (size_t)t0 * p.gate_ld + head0 + h)) / L;
                bf16* dst = p.out + ((size_t)t0 * p.heads + head0 + h) * p.head_ld + slice * p.slice_cols;
                for (int c = lane * 4; c < pad_cols; c += 128) {
                    float a[4] = {0.f, 0.f, 0.f, 0.f};
                    for (int z = 0; z < p.splits; ++z) {
                        const float w = exp2_fast(__ldcg(row + z * step + p.slice_cols) - M);
                        if (__ldcg(row + z * step + p.slice_cols + 1) <= 0.f) continue;  // a split without keys wrote no columns
                        const float2 x = __ldcg((const float2*)(row + z * step + c)), y = __ldcg((const float2*)(row + z * step + c + 2));
                        a[0] += w * x.x; a[1] += w * x.y; a[2] += w * y.x; a[3] += w * y.y;
                    }
                    *(uint2*)(dst + c) = make_uint2((uint32_t)bf16_bits(a[0] * mult) | ((uint32_t)bf16_bits(a[1] * mult) << 16),
                                                    (uint32_t)bf16_bits(a[2] * mult) | ((uint32_t)bf16_bits(a[3] * mult) << 16));
                }
            }
        }
    }
    if (tid == 0) tl_mark(p.tl, 2);
}

// how a launch is cut into tiles; stages == 0: does not fit
struct LatentPlan {
    int part_heads, parts, tile_tokens, q_rows, slices, slice_cols, stages, smem;
};
LatentPlan plan(int rank, int rot, int heads, bool prompt) {
    LatentPlan l;
    const int blocks = (rank + 63) / 64 + (rot + 63) / 64;
    l.parts = (heads + kRowsMax - 1) / kRowsMax;
    l.part_heads = (heads + l.parts - 1) / l.parts;
    l.tile_tokens = prompt ? std::max(1, std::min(8, kRowsMax / l.part_heads)) : 1;
    l.slices = (rank + kSliceCols - 1) / kSliceCols;
    l.slice_cols = ((rank + l.slices - 1) / l.slices + 63) / 64 * 64;
    l.slices = (rank + l.slice_cols - 1) / l.slice_cols;
    const int fixed = 1024 + 512;  // alignment, static shared memory
    for (;; l.tile_tokens = (l.tile_tokens + 1) / 2) {
        l.q_rows = (l.tile_tokens * l.part_heads + 7) / 8 * 8;
        const int q = blocks * l.q_rows * 128;
        l.stages = std::min(kMaxStages, (kSmemLimit - fixed - q) / (blocks * kBlockBytes));
        // an operand tile is always read as 128 rows: what follows the last block of Q has to exist
        l.smem = 1024 + q + std::max(l.stages * blocks * kBlockBytes, (kRowsMax - l.q_rows) * 128);
        if (l.stages >= 1 && l.smem <= kSmemLimit - 512) return l;
        l.stages = 0;
        if (l.tile_tokens == 1) return l;
    }
}

}  // namespace

bool attention_latent_supported(int rank, int rot, int heads) {
    return heads >= 1 && plan(rank, rot, heads, false).stages >= 1 && plan(rank, rot, heads, true).stages >= 1;
}

int attention_latent_splits(int rows, int rank, int rot, int heads, int max_ctx, const AttnWorkspace& ws, int num_sms) {
    const LatentPlan l = plan(rank, rot, heads, false);
    const int units = rows * l.parts * l.slices;
    int splits = 1;
    if (units * 2 <= num_sms) {
        splits = std::min(num_sms / units, (max_ctx + kLatentSplitKeys - 1) / kLatentSplitKeys);
        splits = std::max(1, std::min(splits, 64));
        while (splits > 1 && ((size_t)units * splits * l.part_heads * (l.slice_cols + 2) > ws.partial_floats || units > ws.num_counters)) --splits;
    }
    return splits;
}

int launch_attention_latent(const LatentAttn& a, int T, int n_groups, int max_ctx, const AttnWorkspace& ws, int num_sms, TmapCache* tmaps,
                            cudaStream_t s, bool pdl, unsigned long long* tl) {
    const bool prompt = n_groups > 0;
    const LatentPlan l = plan(a.rank, a.rot, a.heads, prompt);
    if (l.stages < 1 || a.head_ld % 8 || a.kv.hd != latent_row_cols(a.rank, a.rot)) return (int)cudaErrorInvalidValue;
    LatentDev p;
    memset(&p, 0, sizeof p);
    if (!make_tmap_2d(tmaps, &p.tmQ, a.q_lat, (uint64_t)a.rows_alloc * a.heads, a.rank, a.head_ld, l.q_rows)) return -1000;
    if (!make_tmap_2d(tmaps, &p.tmK, a.kv.k_pool, (uint64_t)a.kv.num_pages * kPageTokens, a.kv.hd, a.kv.hd, kPageTokens)) return -1000;
    p.q_up = a.q_up;
    p.q_up_ld = a.q_up_ld;
    p.rot_off = a.rot_off;
    p.rot = a.rot;
    p.rope = a.rope;
    p.max_pos = a.max_pos;
    p.block_table = a.kv.block_table;
    p.max_pages_per_seq = a.kv.max_pages_per_seq;
    p.num_pages = a.kv.num_pages;
    p.tok_seq = a.tok_seq;
    p.tok_pos = a.tok_pos;
    p.grp_first = prompt ? a.grp_first : nullptr;
    p.grp_count = a.grp_count;
    p.heads = a.heads;
    p.part_heads = l.part_heads;
    p.parts = l.parts;
    p.tile_tokens = l.tile_tokens;
    p.subs = prompt ? (8 + l.tile_tokens - 1) / l.tile_tokens : 1;
    p.q_rows = l.q_rows;
    p.rank = a.rank;
    p.slices = l.slices;
    p.slice_cols = l.slice_cols;
    p.stages = l.stages;
    p.splits = prompt ? 1 : attention_latent_splits(T, a.rank, a.rot, a.heads, max_ctx, ws, num_sms);
    p.early = pdl && a.only_newest_row_fresh;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.gate = a.gate;
    p.gate_ld = a.gate_ld;
    p.out = a.out;
    p.head_ld = a.head_ld;
    p.ws = ws.partials;
    p.counters = ws.counters;
    p.status = a.status;
    p.tl = tl;
    const int units = (prompt ? n_groups * p.subs : T) * l.parts * l.slices;
    return (int)launch_k(k_attn_latent, dim3(units, p.splits), dim3(kThreads), (size_t)l.smem, s, pdl, p);
}

int attention_latent_prepare() {
    cudaError_t e = cudaFuncSetAttribute(k_attn_latent, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - 512);
    return (int)(e == cudaSuccess ? prefer_max_shared(k_attn_latent) : e);
}

}  // namespace tffn
