// Latent attention on the tensor cores. A cached row is the key of every head (the heads' key projections are folded into
// the queries) and its first `rank` columns are the value.
//
// Prompts (k_attn_latent): the heads of up to eight tokens of a sequence are the 128 rows of one tile:
//   S[row, key] = Q[row, :] . K[key, :]      tcgen05.mma, Q and K in shared memory (both K-major)
//   O[row, :]  += P[row, :] . K[:, columns]  tcgen05.mma, P in tensor memory, K read the other way round (N-major)
// One CTA = the rows of one tile x at most 256 value columns, 7 warps:
//   warps 0-3  thread = row: S out of tensor memory, online softmax in fp32, P back as a bf16 pair (hi + lo, 16 mantissa
//              bits), the rotated part of Q at the start, and the output rows at the end
//   warp 4     TMA producer: Q, then 64 keys (two pages) per stage, 64 columns per box with the 128-byte swizzle
//   warp 5     tensor memory, issue of S (two tiles ahead of the softmax where the ring is deep enough)
//   warp 6     issue of O
// The reference maximum of a row moves only when it would be exceeded by more than 2^8, so O is rarely rescaled.
//
// Decoding (k_attn_latent_decode): one token's heads would leave most of those rows empty, so keys and value columns take
// the long side instead, S^T[key, head] = K . Q^T and O^T[column, head] += K^T . P^T: all value columns in one CTA. P^T is
// written to shared memory next to its lo part (twice the columns of one product). One CTA = 16 or 32 heads of a token x
// one context split, the same seven warps (thread = key). Up to eight splits are a thread-block cluster and add up their rows through
// distributed shared memory; more leave partial rows and the last one to finish (a ticket, no waiting) adds them up. Both in
// split order.
//
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
constexpr int kThreads = 224;
constexpr int kMaxStages = 6;
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
    int stages;
    int splits, cluster, early;        // decoding only; cluster: the splits are one thread-block cluster
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
// columns block_bytes apart (leading byte offset), groups of 8 rows 1024 bytes apart (stride byte offset)
__device__ __forceinline__ uint64_t desc_n128(uint32_t smem_addr, int block_bytes) {
    return (uint64_t)((smem_addr & 0x3FFFFu) >> 4) | ((uint64_t)(block_bytes >> 4) << 16) | (64ull << 32) | (1ull << 46) | (2ull << 61);
}
// D[tmem] (+)= A[tmem] * B[smem]
__device__ __forceinline__ void umma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "elect.sync _|q, 0xffffffff;\n\t"
        "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(d_tmem),
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

// every lane of an issuing warp waits (acquire), the outcome is made uniform
__device__ __forceinline__ bool mma_wait(uint64_t* bar, uint32_t parity, int* status, int code) {
    return __all_sync(0xffffffffu, mbar_wait(bar, parity, status, code));
}

// The producer warp's view of a sequence's pages: KEYS keys (whole pages) per tile, page ids fetched 32 at a time (lane = page).
template <int KEYS>
struct PageLoader {
    const LatentDev& p;
    const int* bt;
    int page0, last_page, blocks, lane;  // first page of tile 0; last page of the sequence
    uint32_t ring, full;                 // shared memory: stages, their barriers
    int ids;

    __device__ __forceinline__ PageLoader(const LatentDev& p_, int seq, int len, int key0, int blocks_, void* ring_, uint64_t* full_, int lane_)
        : p(p_), bt(p_.block_table + (size_t)seq * p_.max_pages_per_seq), page0(key0 / kPageTokens), last_page((len - 1) / kPageTokens),
          blocks(blocks_), lane(lane_), ring(smem_u32(ring_)), full(smem_u32(full_)), ids(0) {}
    // the whole warp. Pages past the end are replaced by the last one; their keys are masked.
    __device__ __forceinline__ void load(int tile) {
        constexpr int PAGES = KEYS / kPageTokens;
        const int st = tile % p.stages;
        const uint32_t bar = full + st * 8, dst = ring + st * (blocks * KEYS * 128);
        if ((tile * PAGES) % 32 == 0) {
            ids = __ldg(bt + min(page0 + tile * PAGES + lane, last_page));
            if (ids < 0 || ids >= p.num_pages) {
                dev_fail(p.status, DEV_ERR_BOUNDS);
                ids = 0;
            }
        }
        mbar_arrive_expect_tx_elect(bar, blocks * KEYS * 128);
#pragma unroll
        for (int h = 0; h < PAGES; ++h) {
            const int row = __shfl_sync(0xffffffffu, ids, (tile * PAGES + h) % 32) * kPageTokens;
            const uint32_t to = dst + h * kPageTokens * 128;
#pragma unroll 4
            for (int b = 0; b < blocks; ++b) tma_load_2d_elect(to + b * (KEYS * 128), &p.tmK, b * 64, row, bar);
        }
    }
};

// The rotated parts of Q, rows 0 .. rows - 1 of the tile (row = token * part_heads + head), into the blocks behind the latent
// ones; columns past `rot` are zero, and so are rows of heads that do not exist. The 128 softmax threads call it. Angles are
// older than the previous kernel (they are read by the constructor), the parts themselves are not.
// B: pieces of 8 pairs with their loads in flight together
template <int B>
struct QueryRotation {
    const LatentDev& p;
    int t0, head0, nheads, rows, half, q_block;
    uint8_t* q_rot;
    float4 cs[B][4];

    // `i`-th piece of the first batch and of the ones that follow it: row, first pair
    __device__ __forceinline__ void load_angles(int i0) {
        const int pieces = half / 8;
#pragma unroll
        for (int k = 0; k < B; ++k) {
            const int i = i0 + k * kRowsMax;
            if (i < rows * pieces) {
                const int pos = min(max(__ldcg(p.tok_pos + t0 + i / pieces / p.part_heads), 0), p.max_pos - 1);
                const float4* f = (const float4*)(p.rope + (size_t)pos * half + i % pieces * 8);
#pragma unroll
                for (int q = 0; q < 4; ++q) cs[k][q] = __ldg(f + q);
            }
        }
    }
    __device__ __forceinline__ QueryRotation(const LatentDev& p_, int t0_, int head0_, int nheads_, int rows_, uint8_t* q_rot_, int q_block_)
        : p(p_), t0(t0_), head0(head0_), nheads(nheads_), rows(rows_), half(p_.rot / 2), q_block(q_block_), q_rot(q_rot_) {
        if (half % 8 == 0) load_angles(threadIdx.x);
    }
    __device__ __forceinline__ uint8_t* at(int r, int col) const {  // the 8 columns from `col` (a multiple of 8) of row r
        return q_rot + (col >> 6) * q_block + r * 128 + ((((col & 63) >> 3) ^ (r & 7)) << 4);
    }
    __device__ __forceinline__ void put(int r, int col, float x) const { *(bf16*)(at(r, col & ~7) + (col & 7) * 2) = __float2bfloat16_rn(x); }

    __device__ __forceinline__ void store() {
        const int tid = threadIdx.x;
        if (half % 8 == 0) {  // rot is a multiple of 16: no columns to clear
            const int pieces = half / 8, n = rows * pieces;
            for (int i0 = tid; i0 < n; i0 += B * kRowsMax) {
                if (i0 != tid) load_angles(i0);
                uint4 u[B], v[B];
#pragma unroll
                for (int k = 0; k < B; ++k) {
                    const int i = i0 + k * kRowsMax, r = i / pieces, h = r % p.part_heads;
                    u[k] = v[k] = make_uint4(0u, 0u, 0u, 0u);
                    if (i < n && h < nheads) {
                        const bf16* src = p.q_up + (size_t)(t0 + r / p.part_heads) * p.q_up_ld + p.rot_off + (size_t)(head0 + h) * p.rot + i % pieces * 8;
                        u[k] = __ldcg((const uint4*)src);
                        v[k] = __ldcg((const uint4*)(src + half));
                    }
                }
#pragma unroll
                for (int k = 0; k < B; ++k) {
                    const int i = i0 + k * kRowsMax, r = i / pieces, c = i % pieces * 8;
                    if (i >= n) break;
                    const uint32_t uu[4] = {u[k].x, u[k].y, u[k].z, u[k].w}, vv[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
                    uint32_t a[4], b[4];
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        const float4 f = cs[k][q];
                        const float u0 = bf16_lo(uu[q]), u1 = bf16_hi(uu[q]), v0 = bf16_lo(vv[q]), v1 = bf16_hi(vv[q]);
                        a[q] = (uint32_t)bf16_bits(u0 * f.x - v0 * f.y) | ((uint32_t)bf16_bits(u1 * f.z - v1 * f.w) << 16);
                        b[q] = (uint32_t)bf16_bits(v0 * f.x + u0 * f.y) | ((uint32_t)bf16_bits(v1 * f.z + u1 * f.w) << 16);
                    }
                    *(uint4*)at(r, c) = make_uint4(a[0], a[1], a[2], a[3]);
                    *(uint4*)at(r, half + c) = make_uint4(b[0], b[1], b[2], b[3]);
                }
            }
            return;
        }
        const int zero_to = (p.rot + 15) / 16 * 16;
        for (int i = tid; i < rows * half; i += kRowsMax) {
            const int r = i / half, c = i % half, h = r % p.part_heads, t = t0 + r / p.part_heads;
            const int pos = min(max(__ldcg(p.tok_pos + t), 0), p.max_pos - 1);
            const float2 f = __ldg(p.rope + (size_t)pos * half + c);
            const bf16* src = p.q_up + (size_t)t * p.q_up_ld + p.rot_off + (size_t)(head0 + h) * p.rot + c;
            const float u = h < nheads ? act_load(src) : 0.f, v = h < nheads ? act_load(src + half) : 0.f;
            put(r, c, u * f.x - v * f.y);
            put(r, half + c, v * f.x + u * f.y);
        }
        for (int i = tid; i < rows * (zero_to - p.rot); i += kRowsMax) put(i / (zero_to - p.rot), p.rot + i % (zero_to - p.rot), 0.f);
    }
};

__global__ void __launch_bounds__(kThreads, 1) k_attn_latent(const __grid_constant__ LatentDev p) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t k_full[kMaxStages], k_empty[kMaxStages], s_full[2], p_full[2], q_full, pv_done;
    __shared__ uint32_t tmem_slot;
    const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;

    // unit = ((group * subs + sub) * parts + part) * slices + slice
    const int unit = blockIdx.x, slice = unit % p.slices, part = unit / p.slices % p.parts;
    const int sub = unit / p.slices / p.parts % p.subs;
    const int group = gridDim.x / (p.slices * p.parts * p.subs) - 1 - unit / p.slices / p.parts / p.subs;  // later groups see more keys: first
    const int g_first = p.grp_first ? __ldcg(p.grp_first + group) : group, g_count = p.grp_first ? __ldcg(p.grp_count + group) : 1;
    const int t0 = g_first + sub * p.tile_tokens, ntok = min(p.tile_tokens, g_count - sub * p.tile_tokens);
    const int head0 = part * p.part_heads, nheads = min(p.part_heads, p.heads - head0);
    const int seq = __ldcg(p.tok_seq + (ntok > 0 ? t0 : g_first));
    const int len = ntok > 0 ? __ldcg(p.tok_pos + t0 + ntok - 1) + 1 : 0;  // positions ascend within a group
    const int n_tiles = (len + TK - 1) / TK;
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
        mbar_init(&p_full[0], kRowsMax);
        mbar_init(&p_full[1], kRowsMax);
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
        }
        __syncwarp();
        pdl_wait();
        if (lane == 0) tl_mark(p.tl, 1);
        if (tiles > 0) {  // no copy that nobody waits for
            PageLoader<TK> pages(p, seq, len, 0, blocks, k_s, k_full, lane);
            mbar_arrive_expect_tx_elect(smem_u32(&q_full), rank_blocks * q_block);
            for (int b = 0; b < rank_blocks; ++b) tma_load_2d_elect(smem_u32(q_s + b * q_block), &p.tmQ, b * 64, t0 * p.heads + head0, smem_u32(&q_full));
            bool ok = true;
            for (int j = 0; j < tiles && ok; ++j) {
                if (j >= p.stages) ok = __all_sync(0xffffffffu, mbar_wait(&k_empty[j % p.stages], (uint32_t)(j / p.stages - 1) & 1u, p.status, DEV_ERR_EMPTY_WAIT));
                if (ok) pages.load(j);
            }
        }
    } else if (warp == 5) {
        if (tiles > 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(kRowsMax, TK);
            const uint32_t q_a = smem_u32(q_s), k_a = smem_u32(k_s);
            const int last_steps = ((p.rot - 1) % 64 + 16) / 16;
            bool ok = mma_wait(&q_full, 0, p.status, DEV_ERR_FULL_WAIT);
            for (int j = 0; j < tiles && ok; ++j) {
                const int st = j % p.stages;
                // the softmax has read S of tile j - 2 (it says so with its P)
                if (j > 1) ok = mma_wait(&p_full[j & 1], (uint32_t)((j - 2) >> 1) & 1u, p.status, DEV_ERR_ACC_WAIT);
                ok = ok && mma_wait(&k_full[st], (uint32_t)(j / p.stages) & 1u, p.status, DEV_ERR_FULL_WAIT);
                if (!ok) break;
                tc_fence_after();
                const uint32_t d = tmem + kColS + (j & 1) * TK;
                // descriptors advance by constants: address / 16
                uint64_t qd = umma_desc_k128(q_a), kd = umma_desc_k128(k_a + st * stage_bytes);
#pragma unroll
                for (int i = 0; i < 4; ++i) umma_bf16_elect(d, qd + 2 * i, kd + 2 * i, idesc_s, i > 0);  // the latent has a block at least
#pragma unroll 2
                for (int blk = 2; blk < blocks; ++blk) {
                    qd += q_block >> 4;
                    kd += kBlockBytes >> 4;
#pragma unroll
                    for (int i = 0; i < 4; ++i) umma_bf16_elect(d, qd + 2 * i, kd + 2 * i, idesc_s, 1);
                }
                qd += q_block >> 4;
                kd += kBlockBytes >> 4;
                for (int i = 0; i < last_steps; ++i) umma_bf16_elect(d, qd + 2 * i, kd + 2 * i, idesc_s, 1);  // Q is not defined past these steps
                umma_commit_elect(&s_full[j & 1]);
            }
        }
    } else if (warp == 6) {
        const int ncols = min(p.slice_cols, (p.rank - slice * p.slice_cols + 15) / 16 * 16);
        const uint32_t idesc_o = umma_idesc_bf16(kRowsMax, ncols) | (1u << 16);  // B has its K extent in rows
        const uint32_t v_a = smem_u32(k_s) + slice * (p.slice_cols / 64) * kBlockBytes;
        for (int j = 0; j < tiles; ++j) {
            if (!mma_wait(&p_full[j & 1], (uint32_t)(j >> 1) & 1u, p.status, DEV_ERR_ACC_WAIT)) break;
            tc_fence_after();
            const uint64_t vd = desc_n128(v_a + (j % p.stages) * stage_bytes, kBlockBytes);
#pragma unroll
            for (int half = 0; half < 2; ++half)  // P hi, P lo
#pragma unroll
                for (int kk = 0; kk < TK / 16; ++kk)
                    umma_bf16_ts(tmem + kColO, tmem + kColP + half * (TK / 2) + kk * 8, vd + kk * 128, idesc_o, j > 0 || half > 0 || kk > 0);
            umma_commit_elect(&k_empty[j % p.stages]);
            umma_commit_elect(&pv_done);
        }
    } else {
        QueryRotation<4> rotation(p, t0, head0, nheads, max(ntok, 0) * p.part_heads, q_s + rank_blocks * q_block, q_block);
        pdl_wait();
        rotation.store();
        fence_proxy_async_smem();
        mbar_arrive(&q_full);
        const int my_end = active ? __ldcg(p.tok_pos + row_t) + 1 : 0;
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
            const int live = my_end - j * TK;  // visible keys of this tile
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
            mbar_arrive(&p_full[j & 1]);
        }
        if (tiles > 0 && ok) ok = __all_sync(0xffffffffu, mbar_wait(&pv_done, (uint32_t)(tiles - 1) & 1u, p.status, DEV_ERR_ACC_WAIT));
        tc_fence_after();
        // ---- this slice's columns of the row
        const int col0 = slice * p.slice_cols;
        float mult = 0.f;
        if (active && l_sum > 0.f) mult = sigmoid_f32(act_load(p.gate + (size_t)row_t * p.gate_ld + head0 + row_head)) / l_sum;
        bf16* dst = p.out + ((size_t)row_t * p.heads + head0 + row_head) * p.head_ld + col0;
        if (tiles > 0 && ok) {
            for (int c = 0; c < ncols16; ++c) {
                uint32_t o[16];
                tmem_ld16(lane_addr + kColO + c * 16, o);
                tc_wait_ld();
                if (active) {
#pragma unroll
                    for (int i = 0; i < 16; i += 8) {
                        uint32_t w[4];
#pragma unroll
                        for (int k = 0; k < 4; ++k)
                            w[k] = (uint32_t)bf16_bits(__uint_as_float(o[i + 2 * k]) * mult) | ((uint32_t)bf16_bits(__uint_as_float(o[i + 2 * k + 1]) * mult) << 16);
                        if (col0 + c * 16 + i < p.rank) *(uint4*)(dst + c * 16 + i) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                }
                __syncwarp();
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) tmem_dealloc(tmem, kTmemCols);
    if (tid == 0) tl_mark(p.tl, 2);
}

// ---------------------------------------------------------------------------------------------- decoding
constexpr int kDecSoftmax = 128;           // threads of the softmax warps
constexpr int kDecMaxSplits = 64, kClusterSplits = 8;
__host__ __device__ inline int partial_ld(int rank) { return (rank + 3) / 4 * 4 + 4; }  // floats of a split's partial row
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool softmax_any(bool x) {
    int r;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.b32 p, %1, 0;\n\t"
        "bar.red.or.pred q, 1, 128, p;\n\t"
        "selp.b32 %0, 1, 0, q;\n\t}"
        : "=r"(r)
        : "r"((int)x)
        : "memory");
    return r != 0;
}

// HP: heads of a tile (16 or 32). KEYS: keys of a tile, 64, or 32 (one page; half of the rows of S^T are not used) where rows
// are so wide that the ring would hold too few tiles of 64.
template <int HP, int KEYS>
__global__ void __launch_bounds__(kThreads, 1) k_attn_latent_decode(const __grid_constant__ LatentDev p, uint32_t tmem_cols) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t k_full[kMaxStages], k_empty[kMaxStages], s_full[2], p_full[2], pv_done[2], q_full;
    __shared__ uint32_t tmem_slot;
    __shared__ int s_last;
    __shared__ float s_max[4][HP], s_sum[4][HP], s_mult[HP], s_rehearsal[128];
    __shared__ float2 s_ml[HP];  // cluster: this split's maximum and sum per head
    const int tid = threadIdx.x, warp = __shfl_sync(0xffffffffu, tid >> 5, 0), lane = tid & 31;

    const int unit = blockIdx.x, t = unit / p.parts, part = unit % p.parts;
    const int head0 = part * p.part_heads, nheads = min(p.part_heads, p.heads - head0);
    const int seq = __ldcg(p.tok_seq + t), len = __ldcg(p.tok_pos + t) + 1;
    int per_split = (len + p.splits - 1) / p.splits;
    per_split = (per_split + KEYS - 1) / KEYS * KEYS;
    const int k_begin = blockIdx.y * per_split, k_end = min(len, k_begin + per_split);
    const bool len_ok = len <= p.max_pos && (len + kPageTokens - 1) / kPageTokens <= p.max_pages_per_seq;
    const int tiles = len_ok && k_end > k_begin ? (k_end - k_begin + KEYS - 1) / KEYS : 0;

    const int rank_blocks = (p.rank + 63) / 64, rot_blocks = (p.rot + 63) / 64, blocks = rank_blocks + rot_blocks;
    const int mblocks = (p.rank + 127) / 128;
    constexpr int q_block = HP * 128, k_block = KEYS * 128, p_buf = KEYS * 128;  // a P^T buffer: rows of 128 bytes, (hi | lo) heads of a key
    const int stage_bytes = blocks * k_block;
    uint8_t* const q_s = smem;
    uint8_t* const p_s = smem + blocks * q_block;
    uint8_t* const k_s = p_s + 2 * p_buf;
    constexpr uint32_t colO = 2 * HP;
    const int o_ld = (p.rank + 127) / 128 * 128 + 4;  // floats of a row of O on its way out

    if (tid == 0) {
        tl_mark(p.tl, 0);
        for (int i = 0; i < p.stages; ++i) {
            mbar_init(&k_full[i], 1);
            mbar_init(&k_empty[i], 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&s_full[i], 1);
            mbar_init(&p_full[i], kDecSoftmax);  // two: the softmax may be a tile ahead of the product
            mbar_init(&pv_done[i], 1);
        }
        mbar_init(&q_full, 1 + kDecSoftmax);
        fence_mbar_init();
    }
    if (warp == 5) {
        tmem_alloc(&tmem_slot, tmem_cols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;
    pdl_launch_dependents();
    if (!len_ok && tid == 0) dev_fail(p.status, DEV_ERR_BOUNDS);
    // Everything but the newest row is older than the step's first kernel, so the first tiles are requested before the
    // wait for the previous kernel. With the first one there, the time until then goes into a rehearsal: one tile whose
    // keys all weigh zero passes through every warp, so that their instructions are at hand when the queries arrive.
    const int old_keys = (len - 1) / kPageTokens * kPageTokens;
    const int warm = p.early && tiles > 0 && k_begin + KEYS <= old_keys ? 1 : 0;

    if (warp == 4) {
        if (lane == 0) {
            prefetch_tmap(&p.tmQ);
            prefetch_tmap(&p.tmK);
        }
        __syncwarp();
        PageLoader<KEYS> pages(p, seq, max(len, 1), k_begin, blocks, k_s, k_full, lane);
        int next = 0;
        if (p.early)
            for (; next < min(p.stages, tiles) && k_begin + (next + 1) * KEYS <= old_keys; ++next) pages.load(next);
        pdl_wait();
        if (lane == 0) tl_mark(p.tl, 1);
        if (tiles > 0) {  // no copy that nobody waits for
            mbar_arrive_expect_tx_elect(smem_u32(&q_full), rank_blocks * q_block);
            for (int b = 0; b < rank_blocks; ++b) tma_load_2d_elect(smem_u32(q_s + b * q_block), &p.tmQ, b * 64, t * p.heads + head0, smem_u32(&q_full));
        }
        bool ok = true;
        for (; next < tiles && ok; ++next) {
            if (next >= p.stages) ok = __all_sync(0xffffffffu, mbar_wait(&k_empty[next % p.stages], (uint32_t)(next / p.stages - 1) & 1u, p.status, DEV_ERR_EMPTY_WAIT));
            if (ok) pages.load(next);
        }
    } else if (warp == 5) {
        if (tiles > 0) {
            constexpr uint32_t idesc_s = umma_idesc_bf16(64, HP);
            const uint32_t q_a = smem_u32(q_s), k_a = smem_u32(k_s);
            const int last_steps = ((p.rot - 1) % 64 + 16) / 16;
            bool ok = true;
            for (int it = 0; it < tiles + warm && ok; ++it) {
                const int j = max(it - warm, 0), st = j % p.stages;
                if (it == warm) ok = mma_wait(&q_full, 0, p.status, DEV_ERR_FULL_WAIT);
                // the softmax has read S of the tile before the previous one (it says so with its P)
                if (it > 1) ok = ok && mma_wait(&p_full[it & 1], (uint32_t)((it - 2) >> 1) & 1u, p.status, DEV_ERR_ACC_WAIT);
                ok = ok && mma_wait(&k_full[st], (uint32_t)(j / p.stages) & 1u, p.status, DEV_ERR_FULL_WAIT);
                if (!ok) break;
                tc_fence_after();
                const uint32_t d = tmem + (it & 1) * HP;
                // descriptors advance by constants: address / 16
                uint64_t qd = umma_desc_k128(q_a), kd = umma_desc_k128(k_a + st * stage_bytes);
#pragma unroll
                for (int i = 0; i < 4; ++i) umma_bf16_elect(d, kd + 2 * i, qd + 2 * i, idesc_s, i > 0);  // the latent has a block at least
#pragma unroll 2
                for (int blk = 2; blk < blocks; ++blk) {
                    qd += q_block >> 4;
                    kd += k_block >> 4;
#pragma unroll
                    for (int i = 0; i < 4; ++i) umma_bf16_elect(d, kd + 2 * i, qd + 2 * i, idesc_s, 1);
                }
                qd += q_block >> 4;
                kd += k_block >> 4;
                for (int i = 0; i < last_steps; ++i) umma_bf16_elect(d, kd + 2 * i, qd + 2 * i, idesc_s, 1);  // Q is not defined past these steps
                umma_commit_elect(&s_full[it & 1]);
            }
        }
    } else if (warp == 6) {
        constexpr uint32_t idesc_o = umma_idesc_bf16(128, 2 * HP) | (1u << 15) | (1u << 16);  // A and B with their K extent in rows
        const uint32_t k_a = smem_u32(k_s), p_a = smem_u32(p_s);
        for (int it = 0; it < tiles + warm; ++it) {
            const int j = max(it - warm, 0);
            if (!mma_wait(&p_full[it & 1], (uint32_t)(it >> 1) & 1u, p.status, DEV_ERR_ACC_WAIT)) break;
            tc_fence_after();
            uint64_t vd = desc_n128(k_a + (j % p.stages) * stage_bytes, k_block);
            const uint64_t pd = desc_n128(p_a + (it & 1) * p_buf, p_buf);
            const uint32_t again = it > 0;
            uint32_t d = tmem + colO;
#pragma unroll 2
            for (int mb = 0; mb < mblocks; ++mb) {
                umma_bf16_elect(d, vd, pd, idesc_o, again);
#pragma unroll
                for (int kk = 1; kk < KEYS / 16; ++kk) umma_bf16_elect(d, vd + kk * 128, pd + kk * 128, idesc_o, 1);
                vd += 2 * k_block >> 4;
                d += 2 * HP;
            }
            if (it >= warm) umma_commit_elect(&k_empty[j % p.stages]);
            umma_commit_elect(&pv_done[it & 1]);
        }
    } else {
        float gate = 0.f;
        QueryRotation<1> rotation(p, t, head0, nheads, p.part_heads, q_s + rank_blocks * q_block, q_block);
        // rows of S^T: key 16 w + l of the tile is lane l < 16 of warp w
        const uint32_t lane_addr = tmem + ((uint32_t)(warp * 32) << 16);
        const int row = warp * 16 + (lane & 15);
        bool ok = true;  // after a wait has run out the warp goes through the motions, so that the others' barriers complete
        auto wait = [&](uint64_t* bar, uint32_t parity) {
            if (ok) ok = __all_sync(0xffffffffu, mbar_wait(bar, parity, p.status, DEV_ERR_ACC_WAIT));
        };
        int it = 0;  // tiles so far, the rehearsal's included
        for (int pass = 1 - warm; pass < 2; ++pass) {
            const bool real = pass == 1;
            const int n = real ? tiles : 1;
            float m_ref[HP], l_sum[HP];
#pragma unroll
            for (int h = 0; h < HP; ++h) {
                m_ref[h] = kNeg;
                l_sum[h] = 0.f;
            }
            if (real) pdl_wait();
            if (tid < nheads) gate = act_load(p.gate + (size_t)t * p.gate_ld + head0 + tid);
            rotation.store();
            for (int i = tid; i < (HP - p.part_heads) * rot_blocks * 8; i += kDecSoftmax)  // rows without a head
                *(uint4*)(q_s + (rank_blocks + i / 8 % rot_blocks) * q_block + (p.part_heads + i / 8 / rot_blocks) * 128 + i % 8 * 16) = make_uint4(0u, 0u, 0u, 0u);
            fence_proxy_async_smem();
            if (real) mbar_arrive(&q_full);
            for (int j = 0; j < n; ++j, ++it) {
                wait(&s_full[it & 1], (uint32_t)(it >> 1) & 1u);
                tc_fence_after();
                float s[HP];
#pragma unroll
                for (int c = 0; c < HP / 16; ++c) {
                    uint32_t v[16];
                    tmem_ld16(lane_addr + (it & 1) * HP + c * 16, v);
                    tc_wait_ld();
#pragma unroll
                    for (int i = 0; i < 16; ++i) s[c * 16 + i] = __uint_as_float(v[i]) * p.scale_log2;
                }
                const bool live = real && lane < 16 && row < KEYS && k_begin + j * KEYS + row < k_end;
                if (j == 0) {  // the first key's scores are the first reference
                    if (tid == 0) {
#pragma unroll
                        for (int h = 0; h < HP; ++h) s_max[0][h] = s[h];
                    }
                    softmax_sync();
#pragma unroll
                    for (int h = 0; h < HP; ++h) m_ref[h] = s_max[0][h];
                }
                bool up = false;
#pragma unroll
                for (int h = 0; h < HP; ++h) {
                    if (!live) s[h] = kNeg;
                    up = up || (h < nheads && s[h] > m_ref[h] + 8.f);
                }
                if (softmax_any(up)) {  // rare: the reference maxima move to the running maxima
#pragma unroll
                    for (int h = 0; h < HP; ++h) {
                        float m = s[h];
#pragma unroll
                        for (int o = 8; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
                        if (lane == 0) s_max[warp][h] = m;
                    }
                    softmax_sync();
                    if (j > 0) {
                        wait(&pv_done[(it - 1) & 1], (uint32_t)((it - 1) >> 1) & 1u);
                        tc_fence_after();
                    }
                    float corr[HP];
#pragma unroll
                    for (int h = 0; h < HP; ++h) {
                        const float m = fmaxf(fmaxf(fmaxf(s_max[0][h], s_max[1][h]), fmaxf(s_max[2][h], s_max[3][h])), m_ref[h]);
                        corr[h] = exp2_fast(m_ref[h] - m);
                        m_ref[h] = m;
                        l_sum[h] *= corr[h];
                    }
                    if (j > 0) {
                        for (int c = 0; c < mblocks * 2; ++c) {
#pragma unroll
                            for (int q = 0; q < HP / 16; ++q) {
                                uint32_t o[16];
                                tmem_ld16(lane_addr + colO + c * HP + q * 16, o);
                                tc_wait_ld();
#pragma unroll
                                for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr[q * 16 + i]);
                                tmem_st16(lane_addr + colO + c * HP + q * 16, o);
                            }
                        }
                        tc_wait_st();
                    }
                    softmax_sync();  // s_max may be written again
                }
                uint32_t hi[HP / 2], lo[HP / 2];
#pragma unroll
                for (int h = 0; h < HP; h += 2) {
                    const float a = live ? exp2_fast(s[h] - m_ref[h]) : 0.f, b = live ? exp2_fast(s[h + 1] - m_ref[h + 1]) : 0.f;
                    l_sum[h] += a;
                    l_sum[h + 1] += b;
                    const __nv_bfloat162 h2 = __floats2bfloat162_rn(a, b);
                    hi[h / 2] = *(const uint32_t*)&h2;
                    const __nv_bfloat162 l2 = __floats2bfloat162_rn(a - bf16_lo(hi[h / 2]), b - bf16_hi(hi[h / 2]));
                    lo[h / 2] = *(const uint32_t*)&l2;
                }
                if (it > 1) wait(&pv_done[it & 1], (uint32_t)((it - 2) >> 1) & 1u);  // the buffer's last product is done
                if (lane < 16 && row < KEYS) {
                    uint8_t* dst = p_s + (it & 1) * p_buf + row * 128;
#pragma unroll
                    for (int c = 0; c < HP / 8; ++c) {
                        *(uint4*)(dst + ((c ^ (row & 7)) << 4)) = make_uint4(hi[4 * c], hi[4 * c + 1], hi[4 * c + 2], hi[4 * c + 3]);
                        *(uint4*)(dst + (((c + HP / 8) ^ (row & 7)) << 4)) = make_uint4(lo[4 * c], lo[4 * c + 1], lo[4 * c + 2], lo[4 * c + 3]);
                    }
                }
                fence_proxy_async_smem();
                tc_fence_before();
                mbar_arrive(&p_full[it & 1]);
            }
            if (n > 0) wait(&pv_done[(it - 1) & 1], (uint32_t)((it - 1) >> 1) & 1u);
            tc_fence_after();
            // ---- sums over the keys
#pragma unroll
            for (int h = 0; h < HP; ++h) {
                float l = l_sum[h];
#pragma unroll
                for (int o = 8; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);  // lanes 16 and on hold nothing
                if (lane == 0) s_sum[warp][h] = l;
            }
            softmax_sync();
            const int row_ld = partial_ld(p.rank);  // partial rows: [unit][split][part_heads][row_ld], at their end: maximum, sum
            float* parts = p.ws + ((size_t)unit * p.splits + blockIdx.y) * p.part_heads * row_ld;
            if (tid < nheads) {
                const float l = s_sum[0][tid] + s_sum[1][tid] + s_sum[2][tid] + s_sum[3][tid];
                s_mult[tid] = sigmoid_f32(gate) / (p.splits == 1 ? l : 1.f);
                if (p.splits > 1) {
                    float m = kNeg;
#pragma unroll
                    for (int h = 0; h < HP; ++h) m = h == tid ? m_ref[h] : m;
                    s_ml[tid] = make_float2(m, l);
                    if (real && !p.cluster) *(float2*)(parts + tid * row_ld + row_ld - 4) = make_float2(m, l);
                }
            }
            softmax_sync();
            // ---- O^T (lane = column of a group of 128) through the idle ring, rows of ld_s floats, then row by row
            if (n > 0) {
                const int ld_s = real ? o_ld : 0, mb_s = real ? 128 : 0;
                float* const o_s = real ? (float*)k_s : s_rehearsal;
                for (int mb = 0; mb < mblocks; ++mb) {
#pragma unroll
                    for (int g = 0; g < HP / 16; ++g) {
                        uint32_t a[16], b[16];
                        tmem_ld16(lane_addr + colO + mb * 2 * HP + g * 16, a);
                        tmem_ld16(lane_addr + colO + mb * 2 * HP + HP + g * 16, b);
                        tc_wait_ld();
#pragma unroll
                        for (int i = 0; i < 16; ++i)  // P_hi V + P_lo V
                            o_s[(g * 16 + i) * ld_s + mb * mb_s + warp * 32 + lane] = __uint_as_float(a[i]) + __uint_as_float(b[i]);
                    }
                }
                softmax_sync();
                const int per_head = (p.rank + 3) / 4;
                for (int h = warp; h < nheads && real && !p.cluster; h += 4) {
                    const float mult = s_mult[h];
                    const float4* src = (const float4*)(o_s + h * ld_s);
                    bf16* dst = p.out + ((size_t)t * p.heads + head0 + h) * p.head_ld;
#pragma unroll 4
                    for (int c = lane; c < per_head; c += 32) {
                        const float4 o = src[c];
                        if (p.splits == 1)  // columns of the padding are zero in the cache, so they are here
                            *(uint2*)(dst + c * 4) = make_uint2((uint32_t)bf16_bits(o.x * mult) | ((uint32_t)bf16_bits(o.y * mult) << 16),
                                                                (uint32_t)bf16_bits(o.z * mult) | ((uint32_t)bf16_bits(o.w * mult) << 16));
                        else *(float4*)(parts + (size_t)h * row_ld + c * 4) = o;
                    }
                }
            }
        }
        if (p.splits > 1 && !p.cluster) __threadfence();
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) tmem_dealloc(tmem, tmem_cols);
    if (p.cluster) {
        // The splits are a thread-block cluster: each rank adds up the heads that are its own, in split order, out of the
        // shared memory of all.
        cluster_sync_all();
        const int rank = (int)cluster_ctarank(), per_head = (p.rank + 3) / 4, own = (nheads - rank + p.splits - 1) / p.splits;
        float* wgt = (float*)p_s;  // [own head][split], in the idle buffers of P
        if (tid < own) {
            const uint32_t ml = smem_u32(s_ml) + (rank + tid * p.splits) * 8;
            float m[kClusterSplits], l[kClusterSplits], M = kNeg, L = 0.f;
#pragma unroll
            for (int z = 0; z < kClusterSplits; ++z) {
                const uint32_t from = map_shared_rank(ml, z < p.splits ? z : 0);
                m[z] = ld_shared_cluster_f32(from);
                l[z] = z < p.splits ? ld_shared_cluster_f32(from + 4) : 0.f;
            }
#pragma unroll
            for (int z = 0; z < kClusterSplits; ++z) M = fmaxf(M, m[z]);
#pragma unroll
            for (int z = 0; z < kClusterSplits; ++z) {
                m[z] = l[z] > 0.f ? exp2_fast(m[z] - M) : 0.f;  // a split without keys has no rows
                L += l[z] * m[z];
            }
            const float mult = s_mult[rank + tid * p.splits] / L;
#pragma unroll
            for (int z = 0; z < kClusterSplits; ++z) wgt[tid * kClusterSplits + z] = m[z] * mult;
        }
        __syncthreads();
        // a piece = four columns of a head; two pieces and two splits with their loads in flight together
        const uint32_t o_s = smem_u32(k_s);
        const int n = own * per_head;
        for (int i0 = tid; i0 < n; i0 += 2 * kThreads) {
            float o[2][4];
#pragma unroll
            for (int k = 0; k < 2; ++k) o[k][0] = o[k][1] = o[k][2] = o[k][3] = 0.f;
            for (int z0 = 0; z0 < p.splits; z0 += 2) {
                float x[2][2][4], w[2][2];
#pragma unroll
                for (int k = 0; k < 2; ++k)
#pragma unroll
                    for (int q = 0; q < 2; ++q) {
                        const int i = min(i0 + k * kThreads, n - 1), h = i / per_head, c = i % per_head;
                        w[k][q] = wgt[h * kClusterSplits + z0 + q];
                        const uint32_t from = map_shared_rank(o_s + (uint32_t)((rank + h * p.splits) * o_ld + c * 4) * 4, z0 + q);
                        asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(x[k][q][0]), "=f"(x[k][q][1]), "=f"(x[k][q][2]), "=f"(x[k][q][3])
                                     : "r"(from) : "memory");
                    }
#pragma unroll
                for (int k = 0; k < 2; ++k)
#pragma unroll
                    for (int q = 0; q < 2; ++q)
#pragma unroll
                        for (int c = 0; c < 4; ++c) o[k][c] += w[k][q] > 0.f ? w[k][q] * x[k][q][c] : 0.f;
            }
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int i = i0 + k * kThreads, h = rank + i / per_head * p.splits;
                if (i < n)
                    *(uint2*)(p.out + ((size_t)t * p.heads + head0 + h) * p.head_ld + i % per_head * 4) =
                        make_uint2((uint32_t)bf16_bits(o[k][0]) | ((uint32_t)bf16_bits(o[k][1]) << 16), (uint32_t)bf16_bits(o[k][2]) | ((uint32_t)bf16_bits(o[k][3]) << 16));
            }
        }
        cluster_sync_all();  // no rank leaves while its rows are read
    } else if (p.splits > 1) {
        if (tid == 0) {
            __threadfence();
            const int old = atomicAdd(&p.counters[unit], 1);
            s_last = old == p.splits - 1;
            if (s_last) p.counters[unit] = 0;
        }
        __syncthreads();
        if (s_last) {
            __threadfence();
            // weight of split z for head h: 2^(m_z - M) gate / sum; in the idle buffers of P
            const size_t row_ld = partial_ld(p.rank), step = p.part_heads * row_ld;
            const float* parts = p.ws + (size_t)unit * p.splits * step;
            float* wgt = (float*)p_s;  // [HP][splits]
            static_assert(HP * kDecMaxSplits * 4 <= 2 * p_buf, "");
            for (int h = warp; h < nheads; h += kThreads / 32) {
                const float* ml = parts + h * row_ld + row_ld - 4;
                float m[2], l[2], M = kNeg, L = 0.f;
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int z = lane + 32 * i;
                    m[i] = z < p.splits ? __ldcg(ml + z * step) : kNeg;
                    l[i] = z < p.splits ? __ldcg(ml + z * step + 1) : 0.f;
                    M = fmaxf(M, m[i]);
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
#pragma unroll
                for (int i = 0; i < 2; ++i) L += l[i] * exp2_fast(m[i] - M);
                L = warp_sum(L);
                const float mult = sigmoid_f32(act_load(p.gate + (size_t)t * p.gate_ld + head0 + h)) / L;
#pragma unroll
                for (int i = 0; i < 2; ++i)
                    if (lane + 32 * i < p.splits) wgt[h * p.splits + lane + 32 * i] = l[i] > 0.f ? exp2_fast(m[i] - M) * mult : 0.f;
            }
            __syncthreads();
            // a piece = four columns of a head; the loads of four pieces and two splits in flight together
            const int per_head = (p.rank + 3) / 4, n = nheads * per_head;
            for (int i0 = tid; i0 < n; i0 += 4 * kThreads) {
                float o[4][4];
#pragma unroll
                for (int k = 0; k < 4; ++k) o[k][0] = o[k][1] = o[k][2] = o[k][3] = 0.f;
                for (int z0 = 0; z0 < p.splits; z0 += 2) {
                    float4 x[4][2];
                    float w[4][2];
#pragma unroll
                    for (int k = 0; k < 4; ++k)
#pragma unroll
                        for (int q = 0; q < 2; ++q) {
                            const int i = min(i0 + k * kThreads, n - 1), h = i / per_head, z = z0 + q;
                            w[k][q] = z < p.splits ? wgt[h * p.splits + z] : 0.f;
                            x[k][q] = make_float4(0.f, 0.f, 0.f, 0.f);
                            if (w[k][q] > 0.f) x[k][q] = __ldcg((const float4*)(parts + z * step + h * row_ld) + i % per_head);
                        }
#pragma unroll
                    for (int k = 0; k < 4; ++k)
#pragma unroll
                        for (int q = 0; q < 2; ++q) {
                            o[k][0] += w[k][q] * x[k][q].x;
                            o[k][1] += w[k][q] * x[k][q].y;
                            o[k][2] += w[k][q] * x[k][q].z;
                            o[k][3] += w[k][q] * x[k][q].w;
                        }
                }
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const int i = i0 + k * kThreads, h = i / per_head, c = i % per_head * 4;
                    if (i >= n) break;
                    bf16* dst = p.out + ((size_t)t * p.heads + head0 + h) * p.head_ld + c;  // rows padded to 8 columns
#pragma unroll
                    for (int q = 0; q < 4; ++q) o[k][q] = c + q < p.rank ? o[k][q] : 0.f;
                    *(uint2*)dst = make_uint2((uint32_t)bf16_bits(o[k][0]) | ((uint32_t)bf16_bits(o[k][1]) << 16),
                                              (uint32_t)bf16_bits(o[k][2]) | ((uint32_t)bf16_bits(o[k][3]) << 16));
                }
            }
        }
    }
    if (tid == 0) tl_mark(p.tl, 2);
}

// how a launch is cut into tiles; stages == 0: does not fit
struct LatentPlan {
    int part_heads, parts, tile_tokens, q_rows, slices, slice_cols, stages, smem, tmem_cols, keys;
};
constexpr int kStaticSmem = 3072;  // room for the kernels' static shared memory

LatentPlan plan_prompt(int rank, int rot, int heads) {
    LatentPlan l;
    const int blocks = (rank + 63) / 64 + (rot + 63) / 64;
    l.parts = (heads + kRowsMax - 1) / kRowsMax;
    l.part_heads = (heads + l.parts - 1) / l.parts;
    l.tile_tokens = std::max(1, std::min(8, kRowsMax / l.part_heads));
    l.keys = TK;
    l.slices = (rank + kSliceCols - 1) / kSliceCols;
    l.slice_cols = ((rank + l.slices - 1) / l.slices + 63) / 64 * 64;
    l.slices = (rank + l.slice_cols - 1) / l.slice_cols;
    l.tmem_cols = kTmemCols;
    for (;; l.tile_tokens = (l.tile_tokens + 1) / 2) {
        l.q_rows = (l.tile_tokens * l.part_heads + 7) / 8 * 8;
        const int q = blocks * l.q_rows * 128;
        l.stages = std::min(kMaxStages, (kSmemLimit - kStaticSmem - 1024 - q) / (blocks * kBlockBytes));
        // an operand tile is always read as 128 rows: what follows the last block of Q has to exist
        l.smem = 1024 + q + std::max(l.stages * blocks * kBlockBytes, (kRowsMax - l.q_rows) * 128);
        if (l.stages >= 1 && l.smem <= kSmemLimit - kStaticSmem) return l;
        l.stages = 0;
        if (l.tile_tokens == 1) return l;
    }
}

LatentPlan plan_decode(int rank, int rot, int heads) {
    LatentPlan l;
    memset(&l, 0, sizeof l);
    const int blocks = (rank + 63) / 64 + (rot + 63) / 64, mblocks = (rank + 127) / 128;
    for (int hp = heads > 16 ? 32 : 16; hp >= 16; hp /= 2) {
        l.parts = (heads + hp - 1) / hp;
        l.part_heads = (heads + l.parts - 1) / l.parts;
        l.q_rows = hp;
        const int cols = 2 * hp + mblocks * 2 * hp;
        l.tmem_cols = 32;
        while (l.tmem_cols < cols) l.tmem_cols *= 2;
        if (l.tmem_cols > 512) continue;
        for (l.keys = TK; l.keys >= kPageTokens; l.keys /= 2) {
            // S^T always has 64 rows: with 32 keys its operand reaches a block past its own
            const int stage = blocks * l.keys * 128, fixed = 1024 + blocks * hp * 128 + 2 * l.keys * 128 + (TK - l.keys) * 128;
            l.stages = std::min(kMaxStages, (kSmemLimit - kStaticSmem - fixed) / stage);
            const int out = hp * ((rank + 127) / 128 * 128 + 4) * 4;  // O^T passes through the ring
            l.smem = fixed + std::max(l.stages * stage, out);
            if (l.stages >= (l.keys == TK ? 3 : 1) && l.smem <= kSmemLimit - kStaticSmem) return l;
        }
    }
    l.stages = 0;
    return l;
}

}  // namespace

bool attention_latent_supported(int rank, int rot, int heads) {
    return heads >= 1 && plan_decode(rank, rot, heads).stages >= 1 && plan_prompt(rank, rot, heads).stages >= 1;
}

int attention_latent_splits(int rows, int rank, int rot, int heads, int max_ctx, const AttnWorkspace& ws, int num_sms) {
    const LatentPlan l = plan_decode(rank, rot, heads);
    const int units = rows * l.parts;
    int splits = 1;
    if (units * 2 <= num_sms) {
        const int room = num_sms / units, many = std::min(std::min(room, max_ctx / kLatentSplitKeys), kDecMaxSplits);
        if (many > kClusterSplits) {
            splits = many;
            while (splits > kClusterSplits && ((size_t)units * splits * l.part_heads * partial_ld(rank) > ws.partial_floats || units > ws.num_counters)) --splits;
        } else {
            while (splits < kClusterSplits && splits * 2 <= room && max_ctx / (splits * 2) >= kLatentClusterKeys) splits *= 2;
        }
    }
    return splits;
}

int launch_attention_latent(const LatentAttn& a, int T, int n_groups, int max_ctx, const AttnWorkspace& ws, int num_sms, TmapCache* tmaps,
                            cudaStream_t s, bool pdl, unsigned long long* tl) {
    const bool prompt = n_groups > 0;
    const LatentPlan l = prompt ? plan_prompt(a.rank, a.rot, a.heads) : plan_decode(a.rank, a.rot, a.heads);
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
    p.grp_first = a.grp_first;
    p.grp_count = a.grp_count;
    p.heads = a.heads;
    p.part_heads = l.part_heads;
    p.parts = l.parts;
    p.tile_tokens = l.tile_tokens;
    p.q_rows = l.q_rows;
    p.rank = a.rank;
    p.slices = l.slices;
    p.slice_cols = l.slice_cols;
    p.stages = l.stages;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.gate = a.gate;
    p.gate_ld = a.gate_ld;
    p.out = a.out;
    p.head_ld = a.head_ld;
    p.ws = ws.partials;
    p.counters = ws.counters;
    p.status = a.status;
    p.tl = tl;
    if (prompt) {
        p.subs = (8 + l.tile_tokens - 1) / l.tile_tokens;
        return (int)launch_k(k_attn_latent, dim3(n_groups * p.subs * l.parts * l.slices), dim3(kThreads), (size_t)l.smem, s, pdl, p);
    }
    p.splits = attention_latent_splits(T, a.rank, a.rot, a.heads, max_ctx, ws, num_sms);
    p.early = pdl && a.only_newest_row_fresh;
    p.cluster = p.splits > 1 && p.splits <= kClusterSplits;
    const dim3 grid(T * l.parts, p.splits);
    const auto kernel = l.q_rows == 16 ? (l.keys == TK ? k_attn_latent_decode<16, TK> : k_attn_latent_decode<16, kPageTokens>)
                                       : (l.keys == TK ? k_attn_latent_decode<32, TK> : k_attn_latent_decode<32, kPageTokens>);
    return (int)launch_k_cluster(kernel, grid, dim3(kThreads), dim3(1, p.cluster ? p.splits : 1), (size_t)l.smem, s, pdl, p, (uint32_t)l.tmem_cols);
}

template <typename Kern>
static cudaError_t latent_attr(Kern k) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit - kStaticSmem);
    return e == cudaSuccess ? prefer_max_shared(k) : e;
}
int attention_latent_prepare() {
    cudaError_t e = latent_attr(k_attn_latent);
    if (e == cudaSuccess) e = latent_attr(k_attn_latent_decode<16, TK>);
    if (e == cudaSuccess) e = latent_attr(k_attn_latent_decode<16, kPageTokens>);
    if (e == cudaSuccess) e = latent_attr(k_attn_latent_decode<32, TK>);
    if (e == cudaSuccess) e = latent_attr(k_attn_latent_decode<32, kPageTokens>);
    return (int)e;
}

}  // namespace tffn
