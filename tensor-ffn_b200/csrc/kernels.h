// Launchers of the device kernels. Host code (model.cu / session.cu) calls only these.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <cstdint>

namespace tffn {

typedef __nv_bfloat16 bf16;

constexpr int kPageTokens = 32;  // tokens per KV page

// ------------------------------------------------------------------ paged KV cache view
// K rows may differ from V rows in width (kv.vd); with uniform layers one pool holds all of them (layer_stride),
// with listed layers every attention layer has a view of its own (layer 0 of it).
struct KvView {
    bf16* k_pool;            // [L][pages][nkv][kPageTokens][hd]; fp32 rows instead in a session that computes in fp32
    bf16* v_pool;            // [L][pages][nkv][kPageTokens][vd]
    const int* block_table;  // [max_batch][max_pages_per_seq]
    int max_pages_per_seq;
    int num_pages;           // pages per layer
    size_t layer_stride;     // elements between layers of a pool
    int nkv, hd;
    int vd;                  // width of a V row (= hd for the uniform layers); hd and vd are multiples of 8
};

// ------------------------------------------------------------------ tensor-core GEMM (batched path)
// out[t, n] = epilogue( sum_k X0[t,k] W0[n,k] , sum_k X1[t,k] W1[n,k] )
enum GemmMode : int {
    GEMM_STORE_F32 = 0,   // out fp32  = a0 (+ alpha * a1)
    GEMM_STORE_BF16 = 1,  // out bf16  = bf16(a0 (+ alpha * a1))
    GEMM_RESIDUAL = 2,    // out bf16 += a0 (+ alpha * a1), i.e. out = bf16(float(out) + sum)
    GEMM_SWIGLU = 3,      // out bf16  = bf16(silu(bf16(a0)) * bf16(a1))   (a0 gate rows, a1 up rows)
    GEMM_RELU2 = 5,       // out bf16  = bf16(max(a0, 0)^2)
    GEMM_QKV = 4,         // q|k|v rows: bias + RoPE + page writes in the epilogue (GemmCall::qkv), no `out`
};
struct GemmQkvEpilogue {
    const bf16* bias;               // [(nh+2nkv)*hd] or null
    const float *rope_cos, *rope_sin;
    const int *tok_seq, *tok_pos;   // per token: sequence slot and position
    float* q_out;                   // fp32 [T, nh*hd]
    KvView kv;
    int layer, nh, max_pos;
};
struct GemmOperand {
    const bf16* W;  // [N, K] row-major, row stride ldw elements
    int64_t ldw;
    const bf16* X;  // [T, K] row-major, row stride ldx elements
    int64_t ldx;
    int K;          // 0 = operand unused
};
constexpr int kTpMaxRanks = 8;  // ranks of a tensor-parallel group

struct GemmCall {
    GemmOperand op[2];
    int N, T;
    int mode;
    float alpha;
    void* out;
    int64_t ldo;
    int x_rows_alloc;  // rows that exist in the X buffers (>= T); the tensor map covers them
    // optional second, independent problem of the same shape in the same launch (e.g. the expert's
    // gate/up next to the base's): its operands and its output; out2 == nullptr means none
    GemmOperand op2[2];
    void* out2;
    float out_scale;  // GEMM_STORE_F32: the stored value is out_scale * sum (0 means 1)
    const GemmQkvEpilogue* qkv;  // GEMM_QKV only
    // GEMM_STORE_F32 only, optional: greedy pick fused into the epilogue. Every CTA leaves, per token, the
    // maximum of its 128 output rows and its index (lowest index among equal maxima) in
    // amax_val / amax_idx [t * ceil(N / 128) + tile]; launch_argmax_tiles combines them. With it `out` may
    // be nullptr: the values themselves are then not stored.
    float* amax_val;
    int* amax_idx;
    // optional device buffer of 64 u64 per CTA: globaltimer (ns) at 0 start, 1 weight boxes requested,
    // 2 dependency wait over, 3 last MMA issued, 4 accumulator complete, 5 epilogue/park done,
    // 6 cluster barrier passed, 7 reduction done, 8 end, 16+i stage i arrived (i < 40)
    unsigned long long* trace;
    int trace_ctas;          // CTAs the trace buffer holds; a larger grid is not traced
    unsigned long long* tl;  // optional 6 u64 of the step timeline (see tl_mark)
    bool pdl;          // launch with programmatic dependent launch (the kernel waits before touching X / out)
    // Grouped launch (the experts of a mixture): the rows of X are sorted by group, W holds the groups' matrices back
    // to back (N rows each) and grp[0 .. grp_tiles) says which group and rows each token tile of grp_bn rows covers
    // (written by an earlier kernel, see GroupTile). op[1], op2 and GEMM_QKV are not available with it.
    const struct GroupTile* grp;
    int grp_tiles, grp_bn, grp_count;  // grp_count: groups in W
    int grp_rows_hint;                 // tiles that will be in use, about (0: all)
    // Batched launch (the heads of a per-head projection, the parts of a block-diagonal matrix): `batch` > 1 products of
    // N rows of W each (back to back in W), problem b reading columns [b * x_batch, b * x_batch + K) of X and writing
    // columns [b * out_batch, b * out_batch + N) of out. Modes STORE_F32 and STORE_BF16, op[0] only; x_batch a multiple of 8.
    int batch, x_batch, out_batch;
};
struct GroupTile {
    int group;           // -1: this tile and all later ones are unused
    int row0, row_end;   // rows [row0, min(row0 + grp_bn, row_end)) of X and out belong to it
    int pad;
};
// token tile (16 .. 256) of a grouped launch whose groups hold `rows` rows on average
int gemm_group_tile(int rows);
// The same products in true fp32 (fp32 X and out, fp32 FMA, weights still bf16): modes STORE_F32, STORE_BF16, RELU2 and
// SWIGLU (which then store fp32), grouped and batched launches included; two operand pairs only in a plain launch. The operands' X pointers
// are fp32 arrays behind the bf16 type.
int launch_gemm_f32(const GemmCall& c, cudaStream_t stream);
constexpr int kGemmF32Tile = 64;  // its token tile (grp_bn)
// Encoded tensor maps of the (buffer, shape, box) combinations a caller keeps launching with: encoding one costs
// microseconds of host time and a decode step needs about 200. Owned by whoever owns the buffers (a session keeps
// one for its lifetime), so entries die with the buffers they describe.
struct TmapCache;
TmapCache* tmap_cache_create();
void tmap_cache_free(TmapCache* c);
// bf16 tensor [rows, cols] with a row stride of ld elements, boxes of box_rows x 64 columns with the 128-byte swizzle
bool make_tmap_2d(TmapCache* cache, CUtensorMap* tm, const bf16* ptr, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows);

struct GemmWorkspace {
    int* status;  // device status word
    int num_sms;
    TmapCache* tmaps = nullptr;  // optional; without it every launch encodes its maps
};
// opt the kernels into their dynamic shared memory sizes (once per device, outside stream capture)
int gemm_prepare();
// returns cudaError (launch) or -1000 if the tensor maps could not be encoded
int launch_gemm(const GemmCall& c, const GemmWorkspace& ws, cudaStream_t stream, int force_splits = 0);

// ------------------------------------------------------------------ row kernels of the batched path
// (pdl: launch with programmatic dependent launch; every kernel here waits before reading its inputs)
// tl: optional 6 u64 of the step timeline (see tl_mark): min / max over the CTAs of entry, grid-wait return, exit
// the row kernels share the step's shared-memory carveout with the large kernels (see prefer_max_shared)
int rows_prepare();
void launch_embed(const int* tokens, const bf16* table, bf16* h, int T, int H, int V, int* status, cudaStream_t s,
                  bool pdl = false, unsigned long long* tl = nullptr);
void launch_rmsnorm(const bf16* x, const bf16* w, bf16* out, int T, int H, float eps, const int* row_idx, cudaStream_t s,
                    bool pdl = false, unsigned long long* tl = nullptr);
// temperature sampling (inference/src/main.cpp:52-63) of R rows of fp32 logits on the device;
// u[step * R + row] = canonical uniform draws in [0, 1), step = *step_counter (0 if nullptr)
void launch_sample(const float* logits, int R, int V, float temperature, const double* u, const int* step_counter, int* out,
                   cudaStream_t s, bool pdl = false, unsigned long long* tl = nullptr);
// Tensor parallel over peer memory (decode-sized launches). Every rank owns an exchange window that the
// other ranks of the group have mapped; kTpFlagBlocks = the largest grid of a kernel that hand-shakes. Block b
// waits for block b of every peer, so all blocks of such a grid have to be resident at once on every rank
// whatever order the hardware starts them in: 128 blocks of 1 024 threads fit the 148 SMs of a B200.
constexpr int kTpFlagBlocks = 128;
struct TpPeerSync {
    unsigned* flags_local;              // this rank's window: [size][kTpFlagBlocks] counters, written by the peers
    unsigned* flags_peer[kTpMaxRanks];  // the same array inside every peer's window
    unsigned* calls;                    // this rank only: [kTpFlagBlocks] calls made so far, per block
    int rank, size;
    unsigned long long wait_ns;         // how long a block waits for its peers before it gives up
};
// the ranks' pick candidates: part[p] = rank p's {maximum, global index} per row as mapped into this process
struct TpPickParts {
    const float2* part[kTpMaxRanks];
};
// per-tile maxima left by the GEMM (GemmCall::amax_val / amax_idx, `tiles` per row) -> argmax per row
// pack (optional, 8 bytes per row): {the row's maximum, idx_offset + its index} for the exchange between
// tensor-parallel ranks, which launch_tp_pick resolves (cand = `ranks` such arrays of R rows back to back)
void launch_argmax_tiles(const float* amax_val, const int* amax_idx, int R, int tiles, int* out, cudaStream_t s,
                         bool pdl = false, unsigned long long* tl = nullptr, void* pack = nullptr, int idx_offset = 0);
// the ranks' partial sums of one exchange: part[p] = rank p's fp32 [rows][H] buffer as mapped into this process
struct TpParts {
    const float* part[kTpMaxRanks];
};
// h += sum over ranks p (in rank order) of part[p][row * H ...], then out = RMSNorm(h) * w (w == nullptr: no
// norm). T <= kTpFlagBlocks rows, H a multiple of 4.
void launch_tp_reduce_residual_norm(bf16* h, const TpParts& parts, const TpPeerSync& sync, const bf16* w, bf16* out, int T, int H,
                                    float eps, int* status, cudaStream_t s, bool pdl = false, unsigned long long* tl = nullptr);
// launch_tp_pick over the candidates every rank left in its own window (launch_argmax_tiles' pack), loaded over
// NVLink after a hand-shake with the peers; R <= 128 * kTpFlagBlocks rows
void launch_tp_pick_peer(const TpPickParts& parts, const TpPeerSync& sync, int R, int* out, int* status, cudaStream_t s,
                         bool pdl = false);
void launch_tp_pick(const void* cand, int ranks, int R, int* out, cudaStream_t s, bool pdl = false);
// tensor parallel: h = bf16(h + delta) and, if w != null, out = rmsnorm(h) * w, per row
void launch_residual_norm(bf16* h, const float* delta, const bf16* w, bf16* out, int T, int H, float eps, cudaStream_t s,
                          bool pdl = false);
// logits fp32 [R, V] -> argmax (lowest index among maxima). scratch (>= 2 * R * 64 floats) and
// counters (>= R ints, zero, left zero) let several blocks share a row; without them one block per row.
void launch_argmax(const float* logits, int R, int V, int* out, float* scratch, size_t scratch_floats, int* counters,
                   int num_counters, int num_sms, cudaStream_t s, bool pdl = false, unsigned long long* tl = nullptr);

// ------------------------------------------------------------------ attention over the paged cache
struct AttnWorkspace {
    float* partials;  // [T*nkv][splits][G*(hd+2)]
    size_t partial_floats;
    int* counters;    // [T*nkv]
    int num_counters;
};
// Which keys a query sees and how the scores are scaled, when it differs from the uniform layers' causal attention
// over 1 / sqrt(hd).
struct AttnOptions {
    float scale = 0.f;  // 0: 1 / sqrt(hd)
    int chunk = 0;      // > 0: only the keys of the query's own chunk of `chunk` positions, counted from position 0
    int vdim = 0;       // > 0: columns of an output head (kv.vd is the padded row); 0: kv.vd
    int64_t ctx_ld = 0; // row stride of ctx (0: nh * vdim)
    int head_ld = 0;    // (launch_attention_simt) columns between the heads of a ctx row (0: vdim)
    const void* gate = nullptr;  // (launch_attention_simt) optional [T][gate_ld], stored like activations: head h's output times sigmoid(gate[t][h])
    int64_t gate_ld = 0;
};
// opt the attention kernels into their dynamic shared memory (once per device, outside stream capture)
int attn_prepare();
// context splits launch_attention will use (a CUDA-graph key: the grid depends on it)
int attention_splits(int T, int nh, int nkv, int hd, int max_ctx, const AttnWorkspace& ws, int num_sms);
// whether the tensor-core kernels take this head geometry (else launch_attention_simt)
inline bool attention_tc_supported(int hd, int vd) { return hd <= 128 && vd <= 128; }
// One warp-per-key-group attention without tensor cores: any key size up to 2048 and value size up to 1024, bf16 or (f32) fp32 cache and
// output, prompt and decode rows alike.
void launch_attention_simt(const float* q, KvView kv, bool f32, const int* tok_seq, const int* tok_pos, void* ctx, int T, int nh,
                           const AttnOptions& opt, int* status, cudaStream_t s, bool pdl = false, unsigned long long* tl = nullptr);
// one query token per (t): context = tok_pos[t] + 1 cached tokens of sequence tok_seq[t].
// only_newest_row_fresh (decode): of everything the kernel reads, only q and the cached row at
// tok_pos[t] were written since the last kernel of the stream that was launched WITHOUT programmatic
// dependent launch; the rest may then be fetched before the previous kernel has finished.
void launch_attention(const float* q, KvView kv, int layer, const int* tok_seq, const int* tok_pos, bf16* ctx, int T,
                      int nh, int max_ctx, AttnWorkspace ws, int num_sms, int* status, cudaStream_t s, bool pdl = false,
                      bool only_newest_row_fresh = false, unsigned long long* tl = nullptr,
                      unsigned long long* trace = nullptr, int trace_ctas = 0,  // trace: 16 u64 per CTA, see attn.cu
                      const AttnOptions& opt = AttnOptions());

// Prompt tokens: rows grp_first[g] .. grp_first[g] + grp_count[g] - 1 (at most 8, consecutive positions of
// one sequence) share one pass over that sequence's cache; n_groups groups cover the T rows of the call.
void launch_attention_prefill(const float* q, KvView kv, int layer, const int* tok_seq, const int* tok_pos, const int* grp_first,
                              const int* grp_count, int n_groups, bf16* ctx, int nh, int* status, cudaStream_t s,
                              bool pdl = false, unsigned long long* tl = nullptr, const AttnOptions& opt = AttnOptions());

// ------------------------------------------------------------------ layers with an fp32 residual stream
// "f32" below selects the storage type of activations and cache: fp32 in a session that computes in fp32, else bf16.
// A router's scores: softmax of fp32 logits over experts and identity outputs; the `top` largest of score + correction
// are chosen, lowest index first among equals
struct MoeRoute {
    const float* logits;      // [T][ld], experts + identity columns
    int64_t ld;
    const float* correction;  // [experts + identity]
    int experts, identity, top;
    int* counts;              // [experts], zero before the launch
    int2* pair;               // [T][top]: expert (-1: identity) and the pair's place within it
    float* pair_w;            // [T][top] softmax score (without the correction)
};
enum RowSource : int { ROWS_KEEP = 0, ROWS_EMBED, ROWS_DELTA, ROWS_MOE };
// One pass over the residual stream per sublayer: x = table[token] (or its norm * embed_w) | x + norm(delta) * post_w, or
// x + delta_mult * delta without post_w | x + norm(sum of the chosen experts' outputs) * post_w; then out = norm(x) * next_w
// and, for a second sublayer that reads the same x, out2 = norm(x) * next2_w. Norm: v / sqrt(mean(v^2) + eps). All in fp32.
struct ResidualRows {
    float* x;                 // [T][H]
    int H;
    float eps;
    int source;               // RowSource
    const int* tokens;        // ROWS_EMBED
    const bf16* table;
    int64_t table_ld;
    int V;
    int* status;
    const float* delta;       // ROWS_DELTA: [T][delta_ld]
    int64_t delta_ld;
    const void* y;            // ROWS_MOE: expert outputs, rows in expert order [.][y_ld]
    int64_t y_ld;
    const int* pair_row;      // [T][top] row of y, or -1: the pair's output is the sublayer's input itself (`out` before this call)
    const float* pair_w;      // [T][top]
    int top;
    const float* embed_w;     // ROWS_EMBED, optional
    const float* post_w;      // norm of the sublayer's output
    float delta_mult;         // ROWS_DELTA without post_w
    const float* next_w;      // nullptr: no `out`
    void* out;                // [.][out_ld]
    const float* next2_w;     // nullptr: no `out2`; only with next_w and without a router
    void* out2;               // [.][out_ld]
    int64_t out_ld;
    const int* row_idx;       // with ROWS_KEEP: out row r = norm of x row row_idx[r]
    // Optional (rows_can_route): the router of the mixture that reads `out`, in the same pass. route.logits is not used.
    const bf16* router_w;     // [experts + identity][router_ld]
    int64_t router_ld;
    MoeRoute route;
};
int stack_rows_prepare();
// few rows and a router small enough to be read once per row
inline bool rows_can_route(int rows, int H, int outs) { return rows <= 128 && H % 8 == 0 && (size_t)H * outs * 2 <= (256u << 10); }
void launch_residual_rows(const ResidualRows& a, bool f32, int rows, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);

// ------------------------------------------------------------------ latent attention
// A cached row holds the normed latent at [0, rank), zeros up to a multiple of 64, then the rotated key part; it is the key
// of every head (whose key projection is folded into the query) and its first `rank` columns are the value.
constexpr int kLatentMaxRank = 1024;
inline int latent_rot_col(int rank) { return (rank + 63) / 64 * 64; }
inline int latent_row_cols(int rank, int rot) { return latent_rot_col(rank) + (rot + 7) / 8 * 8; }
// Rows of the input projection -> normed query latent and, for a layer with rows of its own, the cached row.
struct LatentPrep {
    const void* proj;         // [T][ld]: query latent at 0, latent and unrotated key part at kv_off
    int64_t ld;
    int kv_off, q_rank, rank, rot;
    bool own_rows;
    const float *q_norm, *kv_norm;
    float eps;
    const float2* rope;       // [max_pos][rot / 2] (cos, sin); pairs (i, i + rot / 2)
    int max_pos;
    const int *tok_seq, *tok_pos;
    void* cq;                 // [T][cq_ld]
    int64_t cq_ld;
    KvView kv;
    int* status;
};
void launch_latent_prep(const LatentPrep& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
// the heads' rotated query parts [T][ld] at column `off`, `rot` columns each -> fp32 columns [rot_col, rot_col + rot) of
// q [T][heads][q_cols]
void launch_latent_rope(const void* q_up, int64_t ld, int off, int heads, int rot, const float2* rope, int max_pos, const int* tok_pos,
                        float* q, int q_cols, int rot_col, bool f32, int T, int* status, cudaStream_t s, bool pdl,
                        unsigned long long* tl = nullptr);
int latent_prepare();
// The attention itself on the tensor cores (bf16 sessions): the unrotated queries come with the key projections folded in,
// the rotated parts as projected. Groups as in launch_attention_prefill; n_groups = 0: every row is a token of its own
// (decode), its context possibly in splits (see launch_attention for only_newest_row_fresh).
struct LatentAttn {
    const bf16* q_lat;        // [rows_alloc][heads][head_ld]
    int rows_alloc;
    const bf16* q_up;         // rotated parts, before the rotation: [T][q_up_ld], `rot` columns per head from rot_off
    int64_t q_up_ld;
    int rot_off, rot, rank, heads;
    const float2* rope;
    int max_pos;
    float scale;
    KvView kv;
    const int *tok_seq, *tok_pos, *grp_first, *grp_count;
    const bf16* gate;         // [T][gate_ld]: head h's output times sigmoid(gate[t][h])
    int64_t gate_ld;
    bf16* out;                // [T][heads][head_ld] weighted latents
    int head_ld;              // rank padded to 8
    bool only_newest_row_fresh;
    int* status;
};
// fewest keys of a context split: of those that add up within a cluster, and of more than eight
constexpr int kLatentClusterKeys = 128, kLatentSplitKeys = 512;
bool attention_latent_supported(int rank, int rot, int heads);  // otherwise launch_attention_simt
int attention_latent_splits(int rows, int rank, int rot, int heads, int max_ctx, const AttnWorkspace& ws, int num_sms);
// returns cudaError (launch) or -1000 if the tensor maps could not be encoded
int launch_attention_latent(const LatentAttn& a, int T, int n_groups, int max_ctx, const AttnWorkspace& ws, int num_sms, TmapCache* tmaps,
                            cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
int attention_latent_prepare();

// q|k|v rows of one projection -> per-head norm of q and k (weights shared by the heads), rotation of neighbouring
// pairs, q in fp32 for the attention kernels, k and v into the sequence's page.
struct QkNormRope {
    const void* qkv;          // [T][ld]: q at 0, k at k_off, v at v_off
    int64_t ld;
    int k_off, v_off;
    const float *q_norm, *k_norm;
    float eps;
    int nh, dim, vdim, rope_dims;
    const float2* rope;       // [max_pos][rope_dims / 2] (cos, sin)
    int max_pos;
    const int *tok_seq, *tok_pos;
    float* q_out;             // [T][nh][kv.hd], zeros past dim
    KvView kv;
    int* status;
};
void launch_qk_norm_rope(const QkNormRope& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);

// ------------------------------------------------------------------ gated delta rule, one decay per key channel or per head
// Recurrent state of a slot: S [heads][vdimP][dimP] fp32 (transposed: a value column's keys are contiguous; dimP a
// multiple of 32, vdimP of 4, the padding stays zero) and the last taps - 1 inputs of the convolution as a ring
// [taps - 1][channels] fp32 addressed by position. A sequence that starts at position 0 starts from zeros whatever
// the slot held before.
struct DeltaRule {
    int heads, kv_heads, dim, vdim, dimP, vdimP, taps;
    float eps;
    const void* proj;         // [T][proj_ld]: q at q_off, k at k_off, v at v_off, beta logits at b_off
    int64_t proj_ld;
    int q_off, k_off, v_off, b_off;
    const float* conv;        // [taps][channels], channels = q | k | v
    const float* a_log;       // [heads]
    bool head_decay;          // one decay per head instead of one per key channel
    const float* dt_bias;     // [heads * dim], head_decay: [heads]
    const float* decay_in;    // [T][decay_ld] decay logits; head_decay: in proj at a_off
    int64_t decay_ld;
    int a_off;
    const float* gate_in;     // [T][gate_ld] gate logits, or nullptr: in proj at gate_off
    int64_t gate_ld;
    int gate_off;
    bool gate_silu;           // the output gate is silu(logit), otherwise sigmoid(logit)
    const float* out_norm;    // [vdim]
    float *state, *ring;      // of slot 0
    size_t state_stride, ring_stride;  // floats between slots
    // per token, from the preparation to the scan
    float *qn, *kn;           // [T][kv_heads][dimP] unit vectors, q scaled
    float *v;                 // [T][heads][vdimP]
    float *g;                 // [T][heads][dimP] decays (not with head_decay)
    float *bk;                // [T][heads][2]: beta, k . q; head_decay: [T][heads][4]: beta, k . q, decay, unused
    float* o;                 // [T][heads][vdimP] raw output rows
    void* out;                // [T][out_ld]
    int64_t out_ld;
    const int *tok_seq, *tok_pos;
    const int *seg_first, *seg_count;  // runs of consecutive positions of one sequence among the T rows
    int max_slots;
    int* status;
};
void launch_delta_prep(const DeltaRule& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
// fused (decode; heads of up to 128 key channels): the scan writes the normed and gated rows; otherwise raw rows to
// `o`, then launch_delta_out
void launch_delta_scan(const DeltaRule& a, bool f32, int n_segs, bool fused, int num_sms, cudaStream_t s, bool pdl,
                       unsigned long long* tl = nullptr);
void launch_delta_out(const DeltaRule& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
int delta_prepare();
int delta_padded_dim(int dim);  // dimP
inline bool delta_supported(int dim, int vdim) { return dim <= 256 && vdim <= 256; }

// ------------------------------------------------------------------ real-gated linear recurrence
// Per channel, behind a short causal convolution u: S = a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), the gates
// r and i sigmoids of block-diagonal products of u; the mixer's row is S * gelu(y). State of a slot: S [width] and the
// convolution's last inputs as a ring [taps - 1][width] addressed by position, fp32; a sequence starts from zeros.
struct RgLru {
    int width, blocks, taps;
    const void* proj;         // [T][proj_ld]: y at 0, the convolution's input at x_off, both without their biases
    int64_t proj_ld;
    int x_off;
    const float *x_bias, *y_bias, *conv_bias, *lam;  // [width]
    const float* conv;        // [taps][width]
    const float* gate_bias;   // [blocks][2][width / blocks]: r, i
    void* u;                  // [T][u_ld], each part's channels padded to u_part, from the preparation to the gates' product and the scan
    int64_t u_ld;
    int u_part;
    const float* gate_in;     // [T][gate_ld]: products, laid out like gate_bias
    int64_t gate_ld;
    float *state, *ring;      // of slot 0
    size_t state_stride, ring_stride;  // floats between slots
    void* out;                // [T][out_ld]
    int64_t out_ld;
    const int *tok_seq, *tok_pos;
    const int *seg_first, *seg_count;  // runs of consecutive positions of one sequence among the T rows
    int max_slots;
    int* status;
};
void launch_lru_prep(const RgLru& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
// one_each: every run is a single token (decode)
void launch_lru_scan(const RgLru& a, bool f32, int n_segs, bool one_each, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
int lru_prepare();

// ------------------------------------------------------------------ mixture of experts
int moe_prepare();
void launch_moe_route(const MoeRoute& a, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);
struct MoeGather {
    const void* x;            // [T][x_ld]
    int64_t x_ld;
    int H, experts, top;
    const int* counts;
    const int2* pair;
    void* xg;                 // [T * top][x_ld] rows sorted by expert
    int* pair_row;            // [T][top] row of xg, -1 for identity
    GroupTile* tiles;         // [max_tiles]
    int max_tiles, tile_rows;
};
void launch_moe_gather(const MoeGather& a, bool f32, int T, cudaStream_t s, bool pdl, unsigned long long* tl = nullptr);

// ------------------------------------------------------------------ batch-1 fused decode kernels
struct Bs1Layer {
    const bf16 *wqkv, *bqkv;  // [(nh+2nkv)*hd, H] rows q|k|v ; bias or null
    const bf16 *wo;           // [H, nh*hd]
    const bf16 *attn_norm, *ffn_norm;
    const bf16 *ffn_base;     // [I][3][H]: gate row, up row, down column (= row of down^T) per intermediate index
    const bf16 *ffn_expert;   // same layout or null
};
struct Bs1Ctx {
    int H, I, nh, nkv, hd, V;
    float eps, expert_scale;
    const float *rope_cos, *rope_sin;
    int max_pos;
    bf16* h;          // [H] residual stream of this layer: published by the q|k|v kernel, updated by o_proj, read by the FFN
    const bf16* h_in; // [H] residual stream the q|k|v kernel (or the LM head) starts from: the previous layer's `h`
    // The FFN leaves its output as fixed-point sums (see bs1_acc_words): acc_out is where this layer's FFN
    // adds, acc_in what the previous layer's FFN left (null: nothing to fold in). The consumer of the
    // residual stream forms h = bf16(h_in + acc_in) itself; the q|k|v kernel also clears acc_out.
    const long long* acc_in;
    long long* acc_out;
    float* q;         // [nh*hd]
    bf16* ctx;        // [nh*hd]
    int* token;       // device: current input token (slot 0)
    int* seq_len;     // device: cached tokens of the slot = position of the new token
    int slot;
    int* tickets;     // zeroed tickets (LM head)
    float* lm_val;    // [lm_grid] candidates
    int* lm_idx;
    float* logits;    // optional fp32 [V] or null
    int* out_tokens;  // device ring of picks, or null
    int* step_counter;
    int* status;
    int num_sms;
    // optional profiling aid for k_bs1_ffn: 16 u64 per CTA, globaltimer ns at 0 start, 1 rmsnorm done,
    // 2 first record arrived, 3 last record consumed, 4 this CTA's sums added to acc_out
    unsigned long long* trace;
    unsigned long long* tl;  // optional 6 u64 of the step timeline for this launch (see tl_mark)
};
bool bs1_supported(int H, int I, int hd, int nh, int nkv);
// 64-bit words of one FFN accumulator: a few replicas (CTAs spread over them to thin out same-address
// atomics) of H fixed-point sums, value * 2^32 as int64. Integer addition is associative, so the sum of
// the CTAs' contributions does not depend on the order in which the atomics land: results stay
// bit-reproducible although no CTA waits for another.
size_t bs1_acc_words(int H);
// h[i] = bf16(h[i] + acc[i]) and acc cleared: closes a stand-alone launch_bs1_ffn (inside a decode step
// the next kernel folds the sums in instead)
void launch_bs1_ffn_finalize(bf16* h, long long* acc, int H, cudaStream_t s);
int bs1_prepare(int H, bool expert);  // dynamic shared memory opt-in for this shape (outside stream capture)
void launch_bs1_qkv(const Bs1Ctx& c, const Bs1Layer& ly, const bf16* embed, KvView kv, int layer, bool first, cudaStream_t s,
                    bool pdl);
void launch_bs1_oproj(const Bs1Ctx& c, const Bs1Layer& ly, cudaStream_t s, bool pdl);
void launch_bs1_ffn(const Bs1Ctx& c, const Bs1Layer& ly, cudaStream_t s, bool pdl);
void launch_bs1_lmhead(const Bs1Ctx& c, const bf16* final_norm, const bf16* lm_head, cudaStream_t s, bool pdl);

// fp32 -> bf16 (RNE) on device, used by the expert loader (inference/src/io/checkpoint.cpp:33-62)
void launch_cast_f32_bf16(const float* src, bf16* dst, size_t n, cudaStream_t s);
// pack gate/up/down^T rows into the [I][3][H] record layout of the batch-1 FFN kernel
void launch_pack_ffn(const bf16* gate, const bf16* up, const bf16* down, bf16* packed, int I, int H, cudaStream_t s);

// a kernel whose only job is to wait on an mbarrier nothing signals, for the bounded-wait test
void launch_wait_selftest(int* status, cudaStream_t s);

}  // namespace tffn
