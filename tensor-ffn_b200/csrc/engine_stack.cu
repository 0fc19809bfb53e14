// Models that list their layers (Config::layers): weight loading, what a session keeps for them, and the step. The step
// runs under the same prefill / forward / decode calls, page allocator, slots, graphs and pick as the uniform stack
// (engine.cu); every layer is described by its LayerSpec, so a family that combines the same mechanisms differently
// needs a reader in host_io.cpp and nothing here.
#include "engine.h"
#include "launch.h"
#include "upload.h"
#include <cmath>

namespace tffn {

namespace {

int64_t pad4(int64_t n) { return (n + 3) & ~(int64_t)3; }

// bf16 matrix of the file -> device rows of `ld` elements (the padding was zeroed when the slab was made)
void put_matrix(Stager& up, bf16* dst, const uint16_t* src, size_t rows, size_t cols, size_t ld) {
    if (ld == cols) return up.copy(dst, src, rows * cols * 2);
    std::vector<uint16_t> wide(rows * ld, 0);
    for (size_t r = 0; r < rows; ++r) memcpy(wide.data() + r * ld, src + r * cols, cols * 2);
    up.copy(dst, wide.data(), wide.size() * 2);
}
void put_vector(Stager& up, const DeviceBuffer& dst, const uint16_t* src, size_t n) {
    std::vector<float> wide(n);
    for (size_t i = 0; i < n; ++i) wide[i] = bf16_to_f32(src[i]);
    up.copy(dst.p, wide.data(), n * 4);
}

// every weight buffer of a layer with its size, in slab order
template <typename Take>
void layout_layer(StackLayer& l, const Config& c, Take take) {
    const LayerSpec& s = l.spec;
    const size_t H = c.hidden_size, ld = pad8(H), nv = (size_t)s.out_cols(), W = (size_t)s.lru_width;
    take(l.w_in, (size_t)l.in_rows * ld * 2);
    take(l.wo, H * pad8(nv) * 2);
    take(l.norm1, H * 4);
    if (c.block == Block::PostNorm) take(l.norm1b, H * 4);
    switch (s.mixer) {
        case Mixer::Attention:
            take(l.q_norm, (size_t)s.dim * 4);
            take(l.k_norm, (size_t)s.dim * 4);
            break;
        case Mixer::ChannelDelta:
        case Mixer::Delta:
            take(l.conv, (2 * (size_t)s.kv_heads * s.dim + nv) * s.conv * 4);
            take(l.a_log, (size_t)s.heads * 4);
            take(l.out_norm, (size_t)s.vdim * 4);
            if (s.mixer == Mixer::Delta) {
                take(l.dt_bias, (size_t)s.heads * 4);
            } else {
                take(l.dt_bias, (size_t)s.heads * s.dim * 4);
                take(l.a2, (size_t)s.heads * s.dim * pad8(l.a_rank) * 2);
                take(l.g2, nv * pad8(l.g_rank) * 2);
            }
            break;
        case Mixer::LatentAttention:
            take(l.dq_norm, (size_t)s.q_rank * 4);
            take(l.uq, (size_t)l.q_rows * pad8(s.q_rank) * 2);
            take(l.uk, (size_t)s.heads * s.kv_rank * pad8(s.dim) * 2);
            take(l.uv, nv * pad8(s.kv_rank) * 2);
            if (s.kv_from < 0) take(l.dkv_norm, (size_t)s.kv_rank * 4);
            break;
        case Mixer::Rglru:
            take(l.conv, W * s.conv * 4);
            take(l.lru_gates, 2 * W * pad8(W / s.lru_blocks) * 2);
            take(l.lru_gate_bias, 2 * W * 4);
            for (DeviceBuffer* v : {&l.conv_bias, &l.x_bias, &l.y_bias, &l.lru_lam}) take(*v, W * 4);
            break;
    }
    if (s.ff > 0) {
        const size_t n = (size_t)std::max(s.experts, 1);
        take(l.norm2, H * 4);
        if (c.block == Block::PostNorm) take(l.norm2b, H * 4);
        if (s.experts > 0) {
            take(l.router, (size_t)(s.experts + s.identity) * ld * 2);
            take(l.correction, (size_t)(s.experts + s.identity) * 4);
        } else {
            take(l.gate, (size_t)s.ff * ld * 2);
        }
        take(l.up, n * s.ff * ld * 2);
        take(l.down, n * H * pad8(s.ff) * 2);
    }
}

__global__ void k_copy_rows_f32(const float* __restrict__ src, float* __restrict__ dst, size_t n) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) dst[i] = src[i];
}

}  // namespace

void Model::load_stack(const std::string& dir) {
    const Config& c = cfg;
    const size_t H = c.hidden_size, vocab = c.vocab_size, ld = pad8(H);
    V = c.vocab_size;
    if (H > 16384) throw Error(kErrUnsupported, "the residual stream is wider than 16384");
    SafeTensorsDir st(dir);
    stack.resize(c.layers.size());
    size_t total = (c.tie_embeddings ? 1 : 2) * Slab::padded(vocab * ld * 2) + 2 * Slab::padded(H * 4);
    auto name = [](size_t i) { return "l" + std::to_string(i) + "."; };
    for (size_t i = 0; i < stack.size(); ++i) {
        StackLayer& l = stack[i];
        LayerSpec& s = l.spec = c.layers[i];
        const std::string p = name(i) + "mix.";
        const int nq = s.kv_heads * s.dim, nv = s.heads * s.vdim;
        auto rank = [&](const char* t) {  // rows of a [rank, width] tensor
            const TensorInfo& ti = st.get(p + t);
            if (ti.shape.size() != 2 || ti.shape[0] < 1) throw Error(kErrShape, "Tensor " + p + t + " is not a matrix");
            return (int)ti.shape[0];
        };
        if (s.dim > 512 || s.vdim > 512) throw Error(kErrUnsupported, "heads wider than 512 are not supported");
        if (s.conv > 32) throw Error(kErrUnsupported, "short convolutions of more than 32 taps are not supported");
        switch (s.mixer) {
            case Mixer::Attention:
                l.k_off = (int)pad8((int64_t)s.heads * s.dim);
                l.v_off = l.k_off + (int)pad8(nq);
                l.in_rows = l.v_off + (int)pad8((int64_t)s.kv_heads * s.vdim);
                break;
            case Mixer::ChannelDelta:
            case Mixer::Delta:
                if (!delta_supported(s.dim, s.vdim)) throw Error(kErrUnsupported, "delta-rule heads wider than 256 are not supported");
                l.a_rank = s.mixer == Mixer::Delta ? s.heads : rank("a1");
                l.g_rank = s.mixer == Mixer::Delta ? nv : rank("g1");
                l.k_off = (int)pad8(nq);
                l.v_off = 2 * l.k_off;
                l.b_off = l.v_off + (int)pad8(nv);
                l.a1_off = l.b_off + (int)pad8(s.heads);
                l.g1_off = l.a1_off + (int)pad8(l.a_rank);
                l.in_rows = l.g1_off + (int)pad8(l.g_rank);
                break;
            case Mixer::LatentAttention:
                if (s.q_rank == 0) s.q_rank = rank("dq");
                if (s.kv_rank > kLatentMaxRank || s.rot_dim > 512) throw Error(kErrUnsupported, "latent attention: rows this wide are not supported");
                l.a1_off = (int)pad8(s.q_rank);
                l.g1_off = l.a1_off + (s.kv_from < 0 ? (int)pad8(s.kv_rank + s.rot_dim) : 0);
                l.in_rows = l.g1_off + (int)pad8(s.heads);
                l.q_rows = s.heads * ((int)pad8(s.dim) + s.rot_dim);
                break;
            case Mixer::Rglru:
                l.a1_off = (int)pad8(s.lru_width);
                l.in_rows = 2 * l.a1_off;
                break;
        }
        if (s.top > 64) throw Error(kErrUnsupported, "more than 64 experts per token");
        if (s.experts + s.identity > 1024) throw Error(kErrUnsupported, "more than 1024 experts in a layer");
        if (c.block == Block::Parallel && s.experts > 0)
            throw Error(kErrUnsupported, "mixtures of experts beside the mixer are not supported");
        layout_layer(l, c, [&](DeviceBuffer&, size_t bytes) { total += Slab::padded(bytes); });
    }
    slab.alloc(total + 256);  // zero-filled: the padding of rows is never written again
    Slab carve{&slab};
    Stager up;
    carve.take(embed, vocab * ld * 2);
    put_matrix(up, embed.as<bf16>(), st.bf16("embed", {(int64_t)vocab, (int64_t)H}), vocab, H, ld);
    embed_ld = (int64_t)ld;
    lm_head = embed.as<bf16>();
    if (!c.tie_embeddings) {
        carve.take(lm_head_own, vocab * ld * 2);
        put_matrix(up, lm_head_own.as<bf16>(), st.bf16("head", {(int64_t)vocab, (int64_t)H}), vocab, H, ld);
        lm_head = lm_head_own.as<bf16>();
    }
    if (c.embed_norm) {
        carve.take(embed_norm_f32, H * 4);
        put_vector(up, embed_norm_f32, st.bf16("embed.norm", {(int64_t)H}), H);
    }
    carve.take(final_norm_f32, H * 4);
    put_vector(up, final_norm_f32, st.bf16("final.norm", {(int64_t)H}), H);
    uint64_t weights = vocab * H * 2;
    for (size_t i = 0; i < stack.size(); ++i) {
        StackLayer& l = stack[i];
        const LayerSpec& s = l.spec;
        layout_layer(l, c, [&](DeviceBuffer& b, size_t bytes) { carve.take(b, bytes); });
        const std::string n = name(i), p = n + "mix.", f = n + "mlp.";
        const int64_t W = (int64_t)H, nq = (int64_t)s.kv_heads * s.dim, nv = (int64_t)s.out_cols();
        auto in_block = [&](const char* t, int row, int64_t rows) {  // rows of the stacked input projection
            put_matrix(up, l.w_in.as<bf16>() + (size_t)row * ld, st.bf16(p + t, {rows, W}), rows, H, ld);
            weights += (uint64_t)rows * H * 2;
        };
        auto vec = [&](const DeviceBuffer& b, const std::string& t, int64_t len) { put_vector(up, b, st.bf16(t, {len}), len); };
        auto mat = [&](bf16* dst, const std::string& t, int64_t rows, int64_t cols) {
            put_matrix(up, dst, st.bf16(t, {rows, cols}), rows, cols, pad8(cols));
            weights += (uint64_t)rows * cols * 2;
        };
        auto conv = [&](std::initializer_list<std::pair<const char*, int64_t>> parts) {  // [taps][channels of all parts]
            int64_t C = 0;
            for (const auto& part : parts) C += part.second;
            std::vector<float> taps((size_t)C * s.conv);
            size_t ch = 0;
            for (const auto& part : parts) {
                const uint16_t* w = st.bf16(p + part.first, {part.second, (int64_t)s.conv});
                for (int64_t r = 0; r < part.second; ++r, ++ch)
                    for (int j = 0; j < s.conv; ++j) taps[(size_t)j * C + ch] = bf16_to_f32(w[r * s.conv + j]);
            }
            up.copy(l.conv.p, taps.data(), taps.size() * 4);
        };
        switch (s.mixer) {
            case Mixer::Attention:
                in_block("q", 0, (int64_t)s.heads * s.dim);
                in_block("k", l.k_off, nq);
                in_block("v", l.v_off, (int64_t)s.kv_heads * s.vdim);
                vec(l.q_norm, p + "q.norm", s.dim);
                vec(l.k_norm, p + "k.norm", s.dim);
                break;
            case Mixer::ChannelDelta:
            case Mixer::Delta:
                in_block("q", 0, nq);
                in_block("k", l.k_off, nq);
                in_block("v", l.v_off, nv);
                in_block("b", l.b_off, s.heads);
                vec(l.a_log, p + "A_log", s.heads);
                vec(l.out_norm, p + "norm", s.vdim);
                if (s.mixer == Mixer::Delta) {
                    in_block("a", l.a1_off, s.heads);
                    in_block("g", l.g1_off, nv);
                    vec(l.dt_bias, p + "dt_bias", s.heads);
                } else {
                    in_block("a1", l.a1_off, l.a_rank);
                    in_block("g1", l.g1_off, l.g_rank);
                    mat(l.a2.as<bf16>(), p + "a2", (int64_t)s.heads * s.dim, l.a_rank);
                    mat(l.g2.as<bf16>(), p + "g2", nv, l.g_rank);
                    vec(l.dt_bias, p + "dt_bias", (int64_t)s.heads * s.dim);
                }
                conv({{"q.conv", nq}, {"k.conv", nq}, {"v.conv", nv}});
                break;
            case Mixer::LatentAttention: {
                const int64_t nh = s.heads, dim = s.dim, dim8 = pad8(dim), rd = s.rot_dim, R = s.kv_rank, Q = s.q_rank, q_ld = pad8(Q);
                in_block("dq", 0, Q);
                vec(l.dq_norm, p + "dq.norm", Q);
                if (s.kv_from < 0) {
                    in_block("dkv", l.a1_off, R + rd);
                    vec(l.dkv_norm, p + "dkv.norm", R);
                }
                in_block("g", l.g1_off, nh);
                const uint16_t* q = st.bf16(p + "uq", {nh * (dim + rd), Q});
                for (int64_t h = 0; h < nh; ++h) {
                    put_matrix(up, l.uq.as<bf16>() + h * dim8 * q_ld, q + h * (dim + rd) * Q, dim, Q, q_ld);
                    put_matrix(up, l.uq.as<bf16>() + (nh * dim8 + h * rd) * q_ld, q + (h * (dim + rd) + dim) * Q, rd, Q, q_ld);
                }
                const uint16_t* k = st.bf16(p + "uk", {nh * dim, R});
                std::vector<uint16_t> kt((size_t)(nh * R * dim8), 0);
                for (int64_t h = 0; h < nh; ++h)
                    for (int64_t d = 0; d < dim; ++d)
                        for (int64_t c0 = 0; c0 < R; ++c0) kt[(size_t)((h * R + c0) * dim8 + d)] = k[(h * dim + d) * R + c0];
                up.copy(l.uk.p, kt.data(), kt.size() * 2);
                mat(l.uv.as<bf16>(), p + "uv", nv, R);
                weights += (uint64_t)(nh * (dim + rd) * Q + nh * dim * R) * 2;
                break;
            }
            case Mixer::Rglru: {
                const int64_t Wd = s.lru_width, B = s.lru_blocks, n = Wd / B, g_ld = pad8(n);
                in_block("y", 0, Wd);
                in_block("x", l.a1_off, Wd);
                vec(l.y_bias, p + "y.b", Wd);
                vec(l.x_bias, p + "x.b", Wd);
                conv({{"conv", Wd}});
                vec(l.conv_bias, p + "conv.b", Wd);
                vec(l.lru_lam, p + "lam", Wd);
                const uint16_t *ra = st.bf16(p + "ra", {B, n, n}), *ri = st.bf16(p + "ri", {B, n, n});
                const uint16_t *rab = st.bf16(p + "ra.b", {B, n}), *rib = st.bf16(p + "ri.b", {B, n});
                std::vector<float> bias((size_t)(2 * Wd));
                for (int64_t b = 0; b < B; ++b) {
                    put_matrix(up, l.lru_gates.as<bf16>() + 2 * b * n * g_ld, ra + b * n * n, n, n, g_ld);
                    put_matrix(up, l.lru_gates.as<bf16>() + (2 * b + 1) * n * g_ld, ri + b * n * n, n, n, g_ld);
                    for (int64_t j = 0; j < n; ++j) {
                        bias[(size_t)(2 * b * n + j)] = bf16_to_f32(rab[b * n + j]);
                        bias[(size_t)((2 * b + 1) * n + j)] = bf16_to_f32(rib[b * n + j]);
                    }
                }
                up.copy(l.lru_gate_bias.p, bias.data(), bias.size() * 4);
                weights += (uint64_t)(2 * Wd * n) * 2;
                break;
            }
        }
        mat(l.wo.as<bf16>(), p + "o", W, nv);
        vec(l.norm1, n + "norm1", W);
        if (c.block == Block::PostNorm) vec(l.norm1b, n + "norm1b", W);
        if (s.ff > 0) {
            vec(l.norm2, n + "norm2", W);
            if (c.block == Block::PostNorm) vec(l.norm2b, n + "norm2b", W);
        }
        if (s.experts > 0) {
            mat(l.router.as<bf16>(), f + "router", s.experts + s.identity, W);
            vec(l.correction, f + "correction", s.experts + s.identity);
            for (int e = 0; e < s.experts; ++e) {
                const std::string en = f + "e" + std::to_string(e) + ".";
                mat(l.up.as<bf16>() + (size_t)e * s.ff * ld, en + "up", s.ff, W);
                mat(l.down.as<bf16>() + (size_t)e * H * pad8(s.ff), en + "down", W, s.ff);
            }
        } else if (s.ff > 0) {
            mat(l.gate.as<bf16>(), f + "gate", s.ff, W);
            mat(l.up.as<bf16>(), f + "up", s.ff, W);
            mat(l.down.as<bf16>(), f + "down", W, s.ff);
        }
    }
    up.finish();
    weight_bytes_base = weights;
}

void Session::alloc_stack(bool f32) {
    if (e_) throw Error(kErrUnsupported, "expert deltas belong to the Qwen2 family");
    const Model* m = m_;
    const size_t T = cap_tokens_, H = m->cfg.hidden_size;
    st_.reset(new StackState());
    StackState& s = *st_;
    s.f32 = f32;
    s.act = f32 ? 4 : 2;
    s.h_ld = pad8((int64_t)H);
    s.delta_ld = pad4((int64_t)H);
    s.layers.resize(m->stack.size());
    size_t q_cols = 0, qn = 0, vn = 0, gn = 0, heads = 0, pairs = 0;
    bool dense = false;
    size_t q_lat_cols = 0;
    for (size_t i = 0; i < m->stack.size(); ++i) {
        const StackLayer& l = m->stack[i];
        const LayerSpec& sp = l.spec;
        StackState::LayerCache& c = s.layers[i];
        s.proj_ld = std::max<int64_t>(s.proj_ld, l.in_rows);
        s.ctx_ld = std::max<int64_t>(s.ctx_ld, pad8(sp.out_cols()));
        if (sp.rope.dims > 0 || sp.mixer == Mixer::Attention) c.rope = rope_table(sp.rope);
        if (sp.mixer == Mixer::Attention) {
            KvView& kv = c.kv;
            kv.nkv = sp.kv_heads;
            kv.hd = (int)pad8(sp.dim);
            kv.vd = (int)pad8(sp.vdim);
            kv.num_pages = num_pages_;
            kv.max_pages_per_seq = max_pages_per_seq_;
            kv.block_table = block_table_.as<int>();
            kv.layer_stride = 0;
            c.k.alloc((size_t)num_pages_ * kv.nkv * kPageTokens * kv.hd * s.act);  // zeros: padding columns stay zero
            c.v.alloc((size_t)num_pages_ * kv.nkv * kPageTokens * kv.vd * s.act);
            kv.k_pool = c.k.as<bf16>();
            kv.v_pool = c.v.as<bf16>();
            q_cols = std::max<size_t>(q_cols, (size_t)sp.heads * kv.hd);
        } else if (sp.mixer == Mixer::LatentAttention) {
            KvView& kv = c.kv;
            if (sp.kv_from >= 0) {
                kv = s.layers[sp.kv_from].kv;
            } else {
                kv.nkv = 1;
                kv.hd = kv.vd = latent_row_cols(sp.kv_rank, sp.rot_dim);
                kv.num_pages = num_pages_;
                kv.max_pages_per_seq = max_pages_per_seq_;
                kv.block_table = block_table_.as<int>();
                kv.layer_stride = 0;
                c.k.alloc((size_t)num_pages_ * kPageTokens * kv.hd * s.act);  // zeros: padding columns stay zero
                kv.k_pool = kv.v_pool = c.k.as<bf16>();
            }
            s.cq_ld = std::max<int64_t>(s.cq_ld, pad8(sp.q_rank));
            s.q_up_ld = std::max<int64_t>(s.q_up_ld, pad8(l.q_rows));
            c.tc = !f32 && attention_latent_supported(sp.kv_rank, sp.rot_dim, sp.heads);
            if (c.tc) q_lat_cols = std::max<size_t>(q_lat_cols, (size_t)sp.heads * pad8(sp.kv_rank));
            else q_cols = std::max<size_t>(q_cols, (size_t)sp.heads * kv.hd);
            s.o_lat_cols = std::max<size_t>(s.o_lat_cols, (size_t)sp.heads * pad8(sp.kv_rank));
        } else if (sp.mixer == Mixer::Rglru) {
            c.state_stride = (size_t)sp.lru_width;
            c.ring_stride = (size_t)(sp.conv - 1) * sp.lru_width;
            c.state.alloc((size_t)max_batch_ * c.state_stride * 4);
            c.ring.alloc(std::max<size_t>(4, (size_t)max_batch_ * c.ring_stride * 4));
            s.u_ld = std::max<int64_t>(s.u_ld, sp.lru_blocks * pad8(sp.lru_width / sp.lru_blocks));
            s.lru_gate_ld = std::max<int64_t>(s.lru_gate_ld, pad4(2 * sp.lru_width));
        } else {
            c.dimP = delta_padded_dim(sp.dim);
            c.vdimP = (int)pad4(sp.vdim);
            c.state_stride = (size_t)sp.heads * c.dimP * c.vdimP;
            c.ring_stride = (size_t)(sp.conv - 1) * (2 * sp.kv_heads * sp.dim + sp.heads * sp.vdim);
            c.state.alloc((size_t)max_batch_ * c.state_stride * 4);
            c.ring.alloc(std::max<size_t>(4, (size_t)max_batch_ * c.ring_stride * 4));
            if (sp.mixer == Mixer::ChannelDelta) {
                s.decay_ld = std::max<int64_t>(s.decay_ld, pad4((int64_t)sp.heads * sp.dim));
                s.gate_ld = std::max<int64_t>(s.gate_ld, pad4((int64_t)sp.heads * sp.vdim));
                gn = std::max<size_t>(gn, (size_t)sp.heads * c.dimP);
            }
            qn = std::max<size_t>(qn, (size_t)sp.kv_heads * c.dimP);
            vn = std::max<size_t>(vn, (size_t)sp.heads * c.vdimP);
            heads = std::max<size_t>(heads, sp.heads);
        }
        if (sp.ff > 0 && sp.experts == 0) {
            dense = true;
            s.act_ld = std::max<int64_t>(s.act_ld, pad8(sp.ff));
        }
        if (sp.experts > 0) {
            c.moe = s.moe_layers++;
            s.max_top = std::max(s.max_top, sp.top);
            s.max_experts = std::max(s.max_experts, sp.experts);
            s.router_ld = std::max<int64_t>(s.router_ld, pad4(sp.experts + sp.identity));
            s.act_ld = std::max<int64_t>(s.act_ld, pad8(sp.ff));
            // tiles of the finest kind: one partly filled tile per expert and the full ones
            s.max_tiles = std::max<int>(s.max_tiles, sp.experts + (int)(T * sp.top / 16) + 1);
        }
    }
    pairs = T * s.max_top;
    h_.alloc(T * H * 4);
    xn_.alloc(T * s.h_ld * s.act);
    xn_last_.alloc(T * s.h_ld * s.act);
    s.proj.alloc(T * s.proj_ld * s.act);
    ctx_.alloc(T * s.ctx_ld * s.act);
    s.delta.alloc(T * s.delta_ld * 4);
    if (q_cols) q_.alloc(T * q_cols * 4);
    if (dense) s.ff_act.alloc(T * s.act_ld * s.act);
    if (dense && m->cfg.block == Block::Parallel) s.xn2.alloc(T * s.h_ld * s.act);
    if (s.cq_ld) {
        s.cq.alloc(T * s.cq_ld * s.act);
        s.q_up.alloc(T * s.q_up_ld * s.act);
        s.o_lat.alloc(T * s.o_lat_cols * s.act);
        if (q_lat_cols) s.q_lat.alloc(T * q_lat_cols * s.act);
    }
    if (s.u_ld) {
        s.u.alloc(T * s.u_ld * s.act);
        s.lru_gate.alloc(T * s.lru_gate_ld * 4);
    }
    if (heads) {
        s.qn.alloc(T * qn * 4);
        s.kn.alloc(T * qn * 4);
        if (gn) s.g.alloc(T * gn * 4);
        s.v.alloc(T * vn * 4);
        s.o.alloc(T * vn * 4);
        s.bk.alloc(T * heads * 16);
        if (s.decay_ld) s.decay.alloc(T * s.decay_ld * 4);
        if (s.gate_ld) s.gate.alloc(T * s.gate_ld * 4);
    }
    if (pairs) {
        s.router.alloc(T * s.router_ld * 4);
        s.counts.alloc((size_t)s.moe_layers * s.max_experts * 4);
        s.pair.alloc(pairs * 8);
        s.pair_w.alloc(pairs * 4);
        s.pair_row.alloc(pairs * 4);
        s.xg.alloc(pairs * s.h_ld * s.act);
        s.act_e.alloc(pairs * s.act_ld * s.act);
        s.y.alloc(pairs * s.h_ld * s.act);
        s.tiles.alloc((size_t)s.max_tiles * sizeof(GroupTile));
    }
    s.seg_first.alloc(T * 4);
    s.seg_count.alloc(T * 4);
    std::vector<int> ones(T, 1);
    upload(s.ones, ones.data(), T * 4);
    cuda_check((cudaError_t)stack_rows_prepare(), "stack_rows_prepare", __FILE__, __LINE__);
    cuda_check((cudaError_t)delta_prepare(), "delta_prepare", __FILE__, __LINE__);
    cuda_check((cudaError_t)moe_prepare(), "moe_prepare", __FILE__, __LINE__);
    cuda_check((cudaError_t)latent_prepare(), "latent_prepare", __FILE__, __LINE__);
    cuda_check((cudaError_t)attention_latent_prepare(), "attention_latent_prepare", __FILE__, __LINE__);
    cuda_check((cudaError_t)lru_prepare(), "lru_prepare", __FILE__, __LINE__);
}

// index of the (cos, sin) table of a rotation
int Session::rope_table(const RopeSpec& spec) {
    StackState& s = *st_;
    for (size_t r = 0; r < s.rope_specs.size(); ++r)
        if (s.rope_specs[r] == spec) return (int)r;
    s.rope_specs.push_back(spec);
    const int half = spec.dims / 2;
    std::vector<float> cs((size_t)max_seq_ * half * 2 + 2);
    for (int j = 0; j < half; ++j) {
        const double f = rope_frequency(spec, j);
        for (int pos = 0; pos < max_seq_; ++pos) {
            cs[((size_t)pos * half + j) * 2] = (float)std::cos(pos * f);
            cs[((size_t)pos * half + j) * 2 + 1] = (float)std::sin(pos * f);
        }
    }
    s.rope.emplace_back();
    upload(s.rope.back(), cs.data(), cs.size() * 4);
    return (int)s.rope.size() - 1;
}

AttnOptions Session::attn_options(const LayerSpec& l) const {
    AttnOptions o;
    o.scale = l.scale;
    o.chunk = l.chunk;
    o.vdim = l.vdim;
    o.ctx_ld = pad8((int64_t)l.heads * l.vdim);
    return o;
}

int Session::decode_graph_key(int n_seqs, int max_ctx) const {
    if (!st_) {
        const Config& c = m_->cfg;
        return attention_splits(n_seqs, c.num_heads, c.num_kv_heads, c.head_dim, max_ctx, attn_ws(), m_->num_sms);
    }
    int key = 0;  // at most 64 splits per layer; layers that see the same context agree, so one digit per distinct choice
    std::vector<int> seen;
    for (size_t i = 0; i < m_->stack.size(); ++i) {
        const LayerSpec& l = m_->stack[i].spec;
        if (l.mixer == Mixer::Attention)
            seen.push_back(attention_splits(n_seqs, l.heads, l.kv_heads, (int)pad8(std::max(l.dim, l.vdim)), attn_ctx(l, max_ctx), attn_ws(), m_->num_sms));
        else if (l.mixer == Mixer::LatentAttention && st_->layers[i].tc)
            seen.push_back(attention_latent_splits(n_seqs, l.kv_rank, l.rot_dim, l.heads, max_ctx, attn_ws(), m_->num_sms));
    }
    for (int sp : seen) key = (int)(((uint32_t)key * 257u + (uint32_t)sp) & 0x3fffffffu);
    return key;
}

void Session::run_stack(int T, int n_logit_rows, bool logit_rows_are_all, bool decode, int max_ctx, int n_groups, int n_segs) {
    StackState& s = *st_;
    const Config& c = m_->cfg;
    const int H = c.hidden_size;
    const bool f32 = s.f32, pdl = launch_mode_ >= 1 && !profile_;
    const int* tok_seq = decode ? identity_.as<int>() : tok_seq_.as<int>();
    const int* tok_pos = decode ? seq_len_dev_.as<int>() : tok_pos_.as<int>();
    const int* seg_first = decode ? identity_.as<int>() : s.seg_first.as<int>();
    const int* seg_count = decode ? s.ones.as<int>() : s.seg_count.as<int>();
    if (decode) n_segs = T;
    int* status = status_.as<int>();
    auto live = [&](int cls) { return !ablated(cls); };
    auto step = [&](int cls, auto&& launch) {  // one kernel that is not a GEMM
        prof_begin(cls);
        if (live(cls)) launch(tl_next(cls));
        prof_end();
        launches_++;
    };
    const bf16* xn = xn_.as<bf16>();
    // out[., n] = rows of X . W, activations out of and into the step's buffers
    auto product = [&](const bf16* W, int64_t ldw, const void* X, int64_t ldx, int K, int N, int mode, void* out, int64_t ldo) {
        GemmCall g;
        memset(&g, 0, sizeof g);
        g.x_rows_alloc = cap_tokens_;
        g.T = T;
        g.alpha = 1.f;
        g.op[0] = {W, ldw, (const bf16*)X, ldx, K};
        g.N = N;
        g.mode = mode;
        g.out = out;
        g.ldo = ldo;
        return g;
    };
    auto run_product = [&](int cls, const bf16* W, int64_t ldw, const void* X, int64_t ldx, int K, int N, int mode, void* out, int64_t ldo) {
        GemmCall g = product(W, ldw, X, ldx, K, N, mode, out, ldo);
        gemm(g, cls, pdl);
    };
    auto act_at = [&](const DeviceBuffer& b, int64_t col) { return (const void*)((const char*)b.p + col * s.act); };

    ResidualRows rows;
    memset(&rows, 0, sizeof rows);
    rows.x = h_.as<float>();
    rows.H = H;
    rows.eps = c.rms_norm_eps;
    rows.status = status;
    rows.out = xn_.p;
    rows.out_ld = s.h_ld;

    if (s.moe_layers) TFFN_CUDA(cudaMemsetAsync(s.counts.p, 0, s.counts.bytes, stream_));
    // the step's first kernel is a full dependency: all that earlier steps wrote is complete for every kernel of this one
    rows.source = ROWS_EMBED;
    rows.tokens = decode ? dec_tokens_.as<int>() : tokens_.as<int>();
    rows.table = m_->embed.as<bf16>();
    rows.table_ld = m_->embed_ld;
    rows.V = c.vocab_size;
    rows.embed_w = m_->embed_norm_f32.as<float>();
    rows.delta_mult = c.residual_mult;
    rows.out2 = s.xn2.p;
    // the norms in front of a layer (Parallel: the feed-forward's as well)
    auto before_layer = [&](const StackLayer& l) {
        rows.next_w = l.norm1.as<float>();
        rows.next2_w = c.block == Block::Parallel ? l.norm2.as<float>() : nullptr;
    };
    before_layer(m_->stack[0]);
    step(KC_EMBED, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, T, stream_, false, tl); });

    auto keep_hidden = [&](size_t li) {
        if (hidden_rows_cap_ <= 0) return;
        const int n = std::min(T, hidden_rows_cap_);
        const size_t elems = (size_t)n * H;
        k_copy_rows_f32<<<(unsigned)((elems + 255) / 256), 256, 0, stream_>>>(h_.as<float>(), hidden_.as<float>() + li * (size_t)hidden_rows_cap_ * H,
                                                                              elems);
        hidden_rows_ = n;
        launches_++;
    };
    for (size_t li = 0; li < m_->stack.size(); ++li) {
        const StackLayer& l = m_->stack[li];
        const LayerSpec& sp = l.spec;
        StackState::LayerCache& cache = s.layers[li];
        const bool last = li + 1 == m_->stack.size();
        // the norm behind this layer: the next layer's, or the model's own when every row gets logits
        auto after_layer = [&] {
            if (!last) return before_layer(m_->stack[li + 1]);
            rows.next_w = n_logit_rows == T && logit_rows_are_all ? m_->final_norm_f32.as<float>() : nullptr;
            rows.next2_w = nullptr;
        };
        const int64_t nv = sp.out_cols(), ctx_ld = pad8(nv);
        const bool dense = sp.ff > 0 && sp.experts == 0;
        const int64_t ffp = pad8(sp.ff);
        auto gate_up = [&](const void* x) {  // the dense feed-forward's gated activations
            GemmCall g = product(l.gate.as<bf16>(), s.h_ld, x, s.h_ld, H, sp.ff, GEMM_SWIGLU, s.ff_act.p, ffp);
            g.op[1] = {l.up.as<bf16>(), s.h_ld, (const bf16*)x, s.h_ld, H};
            gemm(g, KC_GEMM_GATEUP, pdl);
        };
        auto batched = [&](int cls, int batch, const bf16* W, int64_t ldw, const void* X, int64_t ldx, int x_batch, int K, int N, int mode, void* out,
                           int64_t ldo, int out_batch) {
            GemmCall g = product(W, ldw, X, ldx, K, N, mode, out, ldo);
            g.batch = batch;
            g.x_batch = x_batch;
            g.out_batch = out_batch;
            gemm(g, cls, pdl);
        };

        run_product(KC_GEMM_IN, l.w_in.as<bf16>(), s.h_ld, xn, s.h_ld, H, l.in_rows, GEMM_STORE_BF16, s.proj.p, l.in_rows);
        if (sp.mixer == Mixer::Attention) {
            QkNormRope q;
            memset(&q, 0, sizeof q);
            q.qkv = s.proj.p;
            q.ld = l.in_rows;
            q.k_off = l.k_off;
            q.v_off = l.v_off;
            q.q_norm = l.q_norm.as<float>();
            q.k_norm = l.k_norm.as<float>();
            q.eps = c.rms_norm_eps;
            q.nh = sp.heads;
            q.dim = sp.dim;
            q.vdim = sp.vdim;
            q.rope_dims = sp.rope.dims;
            q.rope = s.rope[cache.rope].as<float2>();
            q.max_pos = max_seq_;
            q.tok_seq = tok_seq;
            q.tok_pos = tok_pos;
            q.q_out = q_.as<float>();
            q.kv = cache.kv;
            q.status = status;
            step(KC_QK_ROPE, [&](unsigned long long* tl) { launch_qk_norm_rope(q, f32, T, stream_, pdl, tl); });
            const AttnOptions opt = attn_options(sp);
            step(KC_ATTENTION, [&](unsigned long long* tl) {
                if (f32 || !attention_tc_supported(cache.kv.hd, cache.kv.vd))
                    launch_attention_simt(q_.as<float>(), cache.kv, f32, tok_seq, tok_pos, ctx_.p, T, sp.heads, opt, status, stream_, pdl, tl);
                else if (n_groups > 0)
                    launch_attention_prefill(q_.as<float>(), cache.kv, 0, tok_seq, tok_pos, grp_first_.as<int>(), grp_count_.as<int>(),
                                             n_groups, ctx_.as<bf16>(), sp.heads, status, stream_, pdl, tl, opt);
                else
                    launch_attention(q_.as<float>(), cache.kv, 0, tok_seq, tok_pos, ctx_.as<bf16>(), T, sp.heads, attn_ctx(sp, max_ctx),
                                     attn_ws(), m_->num_sms, status, stream_, pdl, decode, tl, nullptr, 0, opt);
            });
        } else if (sp.mixer == Mixer::LatentAttention) {
            const int kd = cache.kv.hd, rot_col = latent_rot_col(sp.kv_rank), dim8 = (int)pad8(sp.dim), rank8 = (int)pad8(sp.kv_rank);
            LatentPrep p;
            memset(&p, 0, sizeof p);
            p.proj = s.proj.p;
            p.ld = l.in_rows;
            p.kv_off = l.a1_off;
            p.q_rank = sp.q_rank;
            p.rank = sp.kv_rank;
            p.rot = sp.rot_dim;
            p.own_rows = sp.kv_from < 0;
            p.q_norm = l.dq_norm.as<float>();
            p.kv_norm = l.dkv_norm.as<float>();
            p.eps = c.rms_norm_eps;
            p.rope = s.rope[cache.rope].as<float2>();
            p.max_pos = max_seq_;
            p.tok_seq = tok_seq;
            p.tok_pos = tok_pos;
            p.cq = s.cq.p;
            p.cq_ld = s.cq_ld;
            p.kv = cache.kv;
            p.status = status;
            step(KC_LATENT_PREP, [&](unsigned long long* tl) { launch_latent_prep(p, f32, T, stream_, pdl, tl); });
            run_product(KC_GEMM_UQ, l.uq.as<bf16>(), pad8(sp.q_rank), s.cq.p, s.cq_ld, sp.q_rank, l.q_rows, GEMM_STORE_BF16, s.q_up.p, s.q_up_ld);
            // a head's key projection folded into its query: q . (W_uk c) = (W_uk^T q) . c
            if (cache.tc) {
                batched(KC_GEMM_UK, sp.heads, l.uk.as<bf16>(), dim8, s.q_up.p, s.q_up_ld, dim8, sp.dim, sp.kv_rank, GEMM_STORE_BF16, s.q_lat.p,
                        (int64_t)sp.heads * rank8, rank8);
                LatentAttn at;
                memset(&at, 0, sizeof at);
                at.q_lat = s.q_lat.as<bf16>();
                at.rows_alloc = cap_tokens_;
                at.q_up = s.q_up.as<bf16>();
                at.q_up_ld = s.q_up_ld;
                at.rot_off = sp.heads * dim8;
                at.rot = sp.rot_dim;
                at.rank = sp.kv_rank;
                at.heads = sp.heads;
                at.rope = p.rope;
                at.max_pos = max_seq_;
                at.scale = sp.scale;
                at.kv = cache.kv;
                at.tok_seq = tok_seq;
                at.tok_pos = tok_pos;
                at.grp_first = grp_first_.as<int>();
                at.grp_count = grp_count_.as<int>();
                at.gate = (const bf16*)act_at(s.proj, l.g1_off);
                at.gate_ld = l.in_rows;
                at.out = s.o_lat.as<bf16>();
                at.head_ld = rank8;
                at.only_newest_row_fresh = decode;
                at.status = status;
                step(KC_ATTENTION, [&](unsigned long long* tl) {
                    const int rc = launch_attention_latent(at, T, n_groups, max_ctx, attn_ws(), m_->num_sms, tmaps_, stream_, pdl, tl);
                    if (rc == -1000) throw Error(kErrCuda, "cuTensorMapEncodeTiled failed or is unavailable");
                    if (rc != 0) cuda_check((cudaError_t)rc, "latent attention launch", __FILE__, __LINE__);
                });
            } else {
                batched(KC_GEMM_UK, sp.heads, l.uk.as<bf16>(), dim8, s.q_up.p, s.q_up_ld, dim8, sp.dim, sp.kv_rank, GEMM_STORE_F32, q_.p,
                        (int64_t)sp.heads * kd, kd);
                step(KC_LATENT_ROPE, [&](unsigned long long* tl) {
                    launch_latent_rope(s.q_up.p, s.q_up_ld, sp.heads * dim8, sp.heads, sp.rot_dim, p.rope, max_seq_, tok_pos, q_.as<float>(), kd, rot_col,
                                       f32, T, status, stream_, pdl, tl);
                });
                AttnOptions opt;
                opt.scale = sp.scale;
                opt.vdim = sp.kv_rank;
                opt.ctx_ld = (int64_t)sp.heads * rank8;
                opt.head_ld = rank8;
                opt.gate = act_at(s.proj, l.g1_off);
                opt.gate_ld = l.in_rows;
                step(KC_ATTENTION, [&](unsigned long long* tl) {
                    launch_attention_simt(q_.as<float>(), cache.kv, f32, tok_seq, tok_pos, s.o_lat.p, T, sp.heads, opt, status, stream_, pdl, tl);
                });
            }
            batched(KC_GEMM_UV, sp.heads, l.uv.as<bf16>(), rank8, s.o_lat.p, (int64_t)sp.heads * rank8, rank8, sp.kv_rank, sp.vdim, GEMM_STORE_BF16,
                    ctx_.p, ctx_ld, sp.vdim);
        } else if (sp.mixer == Mixer::Rglru) {
            RgLru u;
            memset(&u, 0, sizeof u);
            u.width = sp.lru_width;
            u.blocks = sp.lru_blocks;
            u.taps = sp.conv;
            u.proj = s.proj.p;
            u.proj_ld = l.in_rows;
            u.x_off = l.a1_off;
            u.x_bias = l.x_bias.as<float>();
            u.y_bias = l.y_bias.as<float>();
            u.conv_bias = l.conv_bias.as<float>();
            u.lam = l.lru_lam.as<float>();
            u.conv = l.conv.as<float>();
            u.gate_bias = l.lru_gate_bias.as<float>();
            u.u = s.u.p;
            u.u_ld = s.u_ld;
            u.gate_in = s.lru_gate.as<float>();
            u.gate_ld = s.lru_gate_ld;
            u.state = cache.state.as<float>();
            u.ring = cache.ring.as<float>();
            u.state_stride = cache.state_stride;
            u.ring_stride = cache.ring_stride;
            u.out = ctx_.p;
            u.out_ld = ctx_ld;
            u.tok_seq = tok_seq;
            u.tok_pos = tok_pos;
            u.seg_first = seg_first;
            u.seg_count = seg_count;
            u.max_slots = max_batch_;
            u.status = status;
            const int n = sp.lru_width / sp.lru_blocks;
            u.u_part = (int)pad8(n);
            step(KC_LRU_PREP, [&](unsigned long long* tl) { launch_lru_prep(u, f32, T, stream_, pdl, tl); });
            batched(KC_GEMM_LRU, sp.lru_blocks, l.lru_gates.as<bf16>(), pad8(n), s.u.p, s.u_ld, u.u_part, n, 2 * n, GEMM_STORE_F32,
                    s.lru_gate.p, s.lru_gate_ld, 2 * n);
            step(KC_LRU_SCAN, [&](unsigned long long* tl) { launch_lru_scan(u, f32, n_segs, decode, stream_, pdl, tl); });
        } else {
            const bool per_head = sp.mixer == Mixer::Delta;  // decay and gate logits are part of the input projection
            if (!per_head) {
                // the second halves of the two low-rank projections; one launch when they have the same shape
                const int na = sp.heads * sp.dim;
                GemmCall a = product(l.a2.as<bf16>(), pad8(l.a_rank), act_at(s.proj, l.a1_off), l.in_rows, l.a_rank, na,
                                     GEMM_STORE_F32, s.decay.p, s.decay_ld);
                if (na == nv && l.a_rank == l.g_rank && s.decay_ld == s.gate_ld) {
                    a.op2[0] = {l.g2.as<bf16>(), pad8(l.g_rank), (const bf16*)act_at(s.proj, l.g1_off), l.in_rows, l.g_rank};
                    a.out2 = s.gate.p;
                    gemm(a, KC_GEMM_LOWRANK, pdl);
                } else {
                    gemm(a, KC_GEMM_LOWRANK, pdl);
                    run_product(KC_GEMM_LOWRANK, l.g2.as<bf16>(), pad8(l.g_rank), act_at(s.proj, l.g1_off), l.in_rows, l.g_rank, (int)nv,
                                GEMM_STORE_F32, s.gate.p, s.gate_ld);
                }
            }
            DeltaRule d;
            memset(&d, 0, sizeof d);
            d.heads = sp.heads;
            d.kv_heads = sp.kv_heads;
            d.dim = sp.dim;
            d.vdim = sp.vdim;
            d.dimP = cache.dimP;
            d.vdimP = cache.vdimP;
            d.taps = sp.conv;
            d.eps = c.rms_norm_eps;
            d.proj = s.proj.p;
            d.proj_ld = l.in_rows;
            d.k_off = l.k_off;
            d.v_off = l.v_off;
            d.b_off = l.b_off;
            d.conv = l.conv.as<float>();
            d.a_log = l.a_log.as<float>();
            d.dt_bias = l.dt_bias.as<float>();
            d.head_decay = d.gate_silu = per_head;
            d.decay_in = per_head ? nullptr : s.decay.as<float>();
            d.decay_ld = s.decay_ld;
            d.a_off = l.a1_off;
            d.gate_in = per_head ? nullptr : s.gate.as<float>();
            d.gate_ld = s.gate_ld;
            d.gate_off = l.g1_off;
            d.out_norm = l.out_norm.as<float>();
            d.state = cache.state.as<float>();
            d.ring = cache.ring.as<float>();
            d.state_stride = cache.state_stride;
            d.ring_stride = cache.ring_stride;
            d.qn = s.qn.as<float>();
            d.kn = s.kn.as<float>();
            d.v = s.v.as<float>();
            d.g = s.g.as<float>();
            d.bk = s.bk.as<float>();
            d.o = s.o.as<float>();
            d.out = ctx_.p;
            d.out_ld = ctx_ld;
            d.tok_seq = tok_seq;
            d.tok_pos = tok_pos;
            d.seg_first = seg_first;
            d.seg_count = seg_count;
            d.max_slots = max_batch_;
            d.status = status;
            const bool fuse_out = decode && cache.dimP <= 128;
            step(KC_DELTA_PREP, [&](unsigned long long* tl) { launch_delta_prep(d, f32, T, stream_, pdl, tl); });
            step(KC_DELTA_SCAN, [&](unsigned long long* tl) { launch_delta_scan(d, f32, n_segs, fuse_out, m_->num_sms, stream_, pdl, tl); });
            if (!fuse_out) step(KC_DELTA_OUT, [&](unsigned long long* tl) { launch_delta_out(d, f32, T, stream_, pdl, tl); });
        }
        rows.source = ROWS_DELTA;
        rows.delta = s.delta.as<float>();
        rows.delta_ld = s.delta_ld;
        GemmCall o = product(l.wo.as<bf16>(), ctx_ld, ctx_.p, ctx_ld, (int)nv, H, GEMM_STORE_F32, s.delta.p, s.delta_ld);
        if (c.block == Block::Parallel) {
            // both sublayers' outputs are sums of one launch
            if (dense) {
                gate_up(s.xn2.p);
                o.op[1] = {l.down.as<bf16>(), ffp, s.ff_act.as<bf16>(), ffp, sp.ff};
            }
            gemm(o, dense ? KC_GEMM_OUT_DOWN : KC_GEMM_OPROJ, pdl);
            after_layer();
            step(KC_ROWS, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, T, stream_, pdl, tl); });
            keep_hidden(li);
            continue;
        }
        gemm(o, KC_GEMM_OPROJ, pdl);
        rows.post_w = l.norm1b.as<float>();
        if (sp.ff > 0) rows.next_w = l.norm2.as<float>();
        else after_layer();
        const int outs = sp.experts + sp.identity;
        MoeRoute r;
        r.logits = s.router.as<float>();
        r.ld = s.router_ld;
        r.correction = l.correction.as<float>();
        r.experts = sp.experts;
        r.identity = sp.identity;
        r.top = sp.top;
        r.counts = s.counts.as<int>() + (size_t)std::max(cache.moe, 0) * s.max_experts;
        r.pair = s.pair.as<int2>();
        r.pair_w = s.pair_w.as<float>();
        // few rows: the row kernel routes as well
        const bool routed = sp.experts > 0 && rows_can_route(T, H, outs);
        if (routed) {
            rows.router_w = l.router.as<bf16>();
            rows.router_ld = s.h_ld;
            rows.route = r;
        }
        step(KC_ROWS, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, T, stream_, pdl, tl); });
        rows.router_w = nullptr;
        if (dense) {
            gate_up(xn);
            run_product(KC_GEMM_DOWN, l.down.as<bf16>(), ffp, s.ff_act.p, ffp, sp.ff, H, GEMM_STORE_F32, s.delta.p, s.delta_ld);
            rows.post_w = l.norm2b.as<float>();
            after_layer();
            step(KC_ROWS, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, T, stream_, pdl, tl); });
        }

        if (sp.experts > 0) {
            const int pairs = T * sp.top;
            const int tile = f32 ? kGemmF32Tile : gemm_group_tile((pairs + outs - 1) / outs);
            const int tiles = std::min(sp.experts, pairs) + pairs / tile;
            if (!routed) {
                run_product(KC_GEMM_ROUTER, l.router.as<bf16>(), s.h_ld, xn, s.h_ld, H, outs, GEMM_STORE_F32, s.router.p, s.router_ld);
                step(KC_ROUTE, [&](unsigned long long* tl) { launch_moe_route(r, T, stream_, pdl, tl); });
            }
            MoeGather g;
            g.x = xn_.p;
            g.x_ld = s.h_ld;
            g.H = H;
            g.experts = sp.experts;
            g.top = sp.top;
            g.counts = r.counts;
            g.pair = r.pair;
            g.xg = s.xg.p;
            g.pair_row = s.pair_row.as<int>();
            g.tiles = s.tiles.as<GroupTile>();
            g.max_tiles = tiles;
            g.tile_rows = tile;
            step(KC_GATHER, [&](unsigned long long* tl) { launch_moe_gather(g, f32, T, stream_, pdl, tl); });
            auto grouped = [&](int cls, const bf16* W, int64_t ldw, const void* X, int64_t ldx, int K, int N, int mode, void* out, int64_t ldo) {
                GemmCall e = product(W, ldw, X, ldx, K, N, mode, out, ldo);
                e.x_rows_alloc = cap_tokens_ * s.max_top;
                e.T = pairs;
                e.grp = g.tiles;
                e.grp_tiles = tiles;
                e.grp_bn = tile;
                e.grp_count = sp.experts;
                e.grp_rows_hint = std::min(tiles, std::max(std::min(sp.experts, pairs), pairs / tile));
                gemm(e, cls, pdl);
            };
            grouped(KC_GEMM_UP, l.up.as<bf16>(), s.h_ld, s.xg.p, s.h_ld, H, sp.ff, GEMM_RELU2, s.act_e.p, ffp);
            grouped(KC_GEMM_EXPERT_DOWN, l.down.as<bf16>(), ffp, s.act_e.p, ffp, sp.ff, H, GEMM_STORE_BF16, s.y.p, s.h_ld);
            rows.source = ROWS_MOE;
            rows.y = s.y.p;
            rows.y_ld = s.h_ld;
            rows.pair_row = s.pair_row.as<int>();
            rows.pair_w = s.pair_w.as<float>();
            rows.top = sp.top;
            rows.post_w = l.norm2b.as<float>();
            after_layer();
            step(KC_ROWS, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, T, stream_, pdl, tl); });
        }
        keep_hidden(li);
    }
    if (n_logit_rows > 0) {
        const void* x = xn_.p;
        if (!(n_logit_rows == T && logit_rows_are_all)) {
            rows.source = ROWS_KEEP;
            rows.next2_w = nullptr;
            rows.next_w = m_->final_norm_f32.as<float>();
            rows.row_idx = logit_rows_are_all ? nullptr : row_idx_.as<int>();
            rows.out = xn_last_.p;
            step(KC_RMSNORM, [&](unsigned long long* tl) { launch_residual_rows(rows, f32, n_logit_rows, stream_, pdl, tl); });
            x = xn_last_.p;
        }
        lm_head(x, s.h_ld, n_logit_rows, decode, pdl);
    }
    TFFN_CUDA(cudaGetLastError());
}

}  // namespace tffn
