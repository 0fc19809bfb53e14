"""CPU: the Razesun family's configuration reader and registry, and the plain restatement the GPU tests compare with: each
mechanism's mistakes must move the logits by far more than those tests allow."""
import copy
import json

import numpy as np
import pytest

import razesun_plain as plain
from razesun_cases import DELTA, LATENT, LIMIT, RGLRU, Case, error, mixed_config, plant_key
from synth import dense_mlp, latent_layer, razesun_config, rglru_layer


def write_cfg(tmp_path, cfg):
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return str(tmp_path)


def test_registry_and_config_fields(tmp_path):
    import tffn
    d = write_cfg(tmp_path, mixed_config())
    assert tffn.model_family(d) == "Razesun"
    c = tffn.qwen_config_from_json(d)
    assert (c.hidden_size, c.vocab_size, c.num_layers, c.eos_token_id, c.tie_embeddings) == (72, 211, 9, -1, 0)
    assert (c.num_heads, c.num_kv_heads, c.head_dim, c.intermediate_size) == (1, 1, 96, 136)
    assert abs(c.rms_norm_eps - 2e-5) < 1e-11 and c.rope_theta == 3000.0
    cfg = mixed_config()
    cfg["layers"] = cfg["layers"][1:3]
    c = tffn.qwen_config_from_json(write_cfg(tmp_path, cfg))
    assert (c.num_heads, c.num_kv_heads, c.head_dim, c.num_layers) == (6, 1, 48, 2)


@pytest.mark.parametrize("path,value,code", [
    (("width",), None, -3), (("vocab",), 0, -3), (("norm",), {}, -3), (("layers",), [], -3), (("residual_mult",), None, -3),
    (("logit_scale",), "x", -3), (("layers", 0, "type"), "channel_delta", -7), (("layers", 0, "mlp", "kind"), "moe", -7),
    (("layers", 0, "mixer", "blocks"), 7, -3), (("layers", 0, "mixer", "conv"), None, -3), (("layers", 0, "mlp", "ff"), 0, -3),
    (("layers", 1, "mixer", "rot", "dims"), 14, -3), (("layers", 1, "mixer", "kv_rank"), None, -3), (("layers", 1, "mixer", "scale"), None, -3),
    (("layers", 2, "mixer", "kv_heads"), 3, -3), (("layers", 3, "mixer", "kv_from"), 3, -3), (("layers", 3, "mixer", "kv_from"), 2, -3),
    (("layers", 3, "mixer", "kv_from"), 4, -3), (("layers", 5, "mixer", "kv_from"), 3, -3), (("layers", 5, "mixer", "kv_rank"), 88, -3),
    (("layers", 5, "mixer", "rot", "base"), 3001.0, -3),
])
def test_config_errors(tmp_path, path, value, code):
    """a missing or impossible entry is an error that names it, never a default"""
    import tffn
    cfg = copy.deepcopy(mixed_config())
    at = cfg
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(tffn.TffnError) as e:
        tffn.model_family(write_cfg(tmp_path, cfg))
    assert e.value.code == code


def test_plain_prefix(tmp_path):
    """causal: the logits of a prefix do not change when tokens follow"""
    c = Case(tmp_path, mixed_config(), sharp=2.0)
    t = c.tokens(60)
    whole, _ = c.expect(t)
    part, _ = c.expect(t[:37])
    assert np.abs(whole[:37] - part).max() < 1e-9


def test_planted_key_decides(tmp_path):
    """the key the GPU tests plant shows at the query that asks for it, and hardly anywhere else"""
    c, key, ask, other = plant_key(tmp_path)
    t = c.tokens(200, seed=5)
    t[np.isin(t, [key, ask])] = other
    t[40], t[199] = key, ask
    without = t.copy()
    without[40] = other
    moved = error(c.expect(without)[0], c.expect(t)[0])
    assert moved[199] > 0.3 and moved[100:199].max() < 0.2 * moved[199]


def mutate(monkeypatch, what):
    """plant one mistake in the restatement"""
    set_ = lambda name, fn: monkeypatch.setattr(plain, name, fn)
    if what == "neighbour_rotation":
        def rotate(x, pos, rot):
            y = x.copy()
            for i in range(rot["dims"] // 2):
                a = pos * rot["base"] ** (-2.0 * i / rot["dims"])
                u, v = x[..., 2 * i], x[..., 2 * i + 1]
                y[..., 2 * i], y[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
            return y
        set_("rotate_halves", rotate)
    elif what == "unnormed_latent":
        real = plain.latent_rows
        set_("latent_rows", lambda h, w, p, m, eps: ((h @ w[p + "dkv"].T)[:, :m["kv_rank"]], real(h, w, p, m, eps)[1]))
    elif what == "key_unrotated":
        real = plain.latent_rows
        set_("latent_rows", lambda h, w, p, m, eps: (real(h, w, p, m, eps)[0], (h @ w[p + "dkv"].T)[:, m["kv_rank"]:]))
    elif what == "no_gate":
        real = plain.latent_attention
        set_("latent_attention", lambda h, w, p, m, eps, rows: real(h, {**w, p + "g": w[p + "g"] * 0}, p, m, eps, rows) * 2)
    elif what == "conv_order":
        real = plain.short_conv
        set_("short_conv", lambda x, taps: real(x, taps[:, ::-1]))
    elif what == "lru_conv_order":
        real = plain.plain_conv
        set_("plain_conv", lambda x, taps, b: real(x, taps[:, ::-1], b))
    elif what == "old_state_read":
        def scan(q, k, v, g, beta):
            T, H, dim = q.shape
            S, o = np.zeros((H, dim, v.shape[2])), np.zeros_like(v)
            for t in range(T):
                for h in range(H):
                    S[h] *= g[t, h]
                    o[t, h] = S[h].T @ q[t, h]
                    S[h] += np.outer(k[t, h], beta[t, h] * (v[t, h] - S[h].T @ k[t, h]))
            return o
        set_("delta_scan", scan)
    elif what == "lost_state":
        real = plain.delta_scan
        set_("delta_scan", lambda *a: np.concatenate([real(*(x[:40] for x in a)), real(*(x[40:] for x in a))]))
    elif what == "lost_lru_state":
        real = plain.rglru_scan
        set_("rglru_scan", lambda u, r, i, lam: np.concatenate([real(u[:40], r[:40], i[:40], lam), real(u[40:], r[40:], i[40:], lam)]))
    elif what == "gates_swapped":
        real = plain.rglru_scan
        set_("rglru_scan", lambda u, r, i, lam: real(u, i, r, lam))
    elif what == "plain_first_input":  # no sqrt(1 - a^2) for the first token
        real = plain.rglru_scan

        def scan(u, r, i, lam):
            v = u.copy()
            v[0] = u[0] / np.sqrt(-np.expm1(-16.0 * r[0] * plain.softplus(lam)))
            return real(v, r, i, lam)
        set_("rglru_scan", scan)
    elif what == "transposed_gates":
        real = plain.block_linear
        set_("block_linear", lambda u, m, b: real(u, m.transpose(0, 2, 1), b))
    elif what == "exact_gelu":
        from math import erf
        set_("gelu_tanh", np.vectorize(lambda z: 0.5 * z * (1 + erf(z / 2 ** 0.5))))
    else:
        raise ValueError(what)


@pytest.mark.parametrize("what,model", [
    ("neighbour_rotation", "plain"), ("unnormed_latent", "plain"), ("key_unrotated", "unaligned"), ("no_gate", "plain"),
    ("conv_order", "shared_qk"), ("old_state_read", "shared_qk"), ("lost_state", "shared_qk"), ("lru_conv_order", "one_part"),
    ("lost_lru_state", "one_part"), ("gates_swapped", "many_parts"), ("plain_first_input", "one_part"), ("transposed_gates", "many_parts"),
    ("exact_gelu", "one_part")])
def test_mistakes_would_show(tmp_path, monkeypatch, what, model):
    """where a planted mistake acts, the logits leave the fp32 limit of the GPU tests many times over"""
    width, layer, *sharp = {**LATENT, **{k: v for k, v in DELTA.items() if k == "shared_qk"},
                            **{k: v for k, v in RGLRU.items() if k in ("one_part", "many_parts")}}[model]
    c = Case(tmp_path, razesun_config(width, 97, [layer]), sharp=sharp[0] if sharp else 1.0)
    t = c.tokens(80)
    good, _ = c.expect(t)
    mutate(monkeypatch, what)
    e = error(c.expect(t)[0], good)
    assert e.max() > (3 if what == "exact_gelu" else 100) * LIMIT["float32"], e.max()
    if what in ("lost_state", "lost_lru_state"):
        assert e[40:48].max() > 100 * LIMIT["float32"] and e[:40].max() == 0.0
    if what == "plain_first_input":
        assert e[0] > 100 * LIMIT["float32"]


@pytest.mark.parametrize("edit", ["sequential", "one_norm", "no_mult", "no_scale", "no_embed_norm", "own_rows"])
def test_block_mistakes_would_show(tmp_path, edit):
    """mistakes of the block and of the model around it, made by changing the weights or the configuration alike"""
    layers = [latent_layer(2, 16, 8, 16, 40, 24, mlp=dense_mlp(48)), rglru_layer(32, 2, mlp=dense_mlp(40)),
              latent_layer(3, 16, 8, 16, 40, 24, kv_from=0, mlp=dense_mlp(32))]
    c = Case(tmp_path, razesun_config(48, 97, layers, residual_mult=0.4, logit_scale=0.3), sharp=2.0)
    t = c.tokens(40)
    good, _ = c.expect(t)
    cfg, w = copy.deepcopy(c.plain_cfg), dict(c.w)
    if edit == "sequential":  # the feed-forward of the first layer reads what the mixer has added: as layers of their own
        cfg["layers"] = [dict(cfg["layers"][0], mlp=None)] + cfg["layers"][1:]
    elif edit == "one_norm":
        w["l1.norm2"] = w["l1.norm1"]
    elif edit == "no_mult":
        cfg["residual_mult"] = 1.0
    elif edit == "no_scale":
        cfg["logit_scale"] = 1.0
    elif edit == "no_embed_norm":
        w["embed.norm"] = np.ones_like(w["embed.norm"])
    else:
        w["l2.mix.dkv"], w["l2.mix.dkv.norm"] = w["l0.mix.dkv"], w["l0.mix.dkv.norm"]
        del cfg["layers"][2]["mixer"]["kv_from"]
    assert error(plain.forward(cfg, w, t)[0], good).max() > 100 * LIMIT["float32"]
