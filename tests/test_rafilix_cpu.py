"""CPU: the Rafilix family's configuration reader and registry, and the plain restatement the GPU tests compare with:
each mechanism's mistakes must move the logits by far more than those tests allow."""
import copy
import json

import numpy as np
import pytest

import rafilix_plain as plain
import synth
from rafilix_cases import ATTENTION, DELTA, LIMIT, SCALING, Case, error, mixed_config, moe_model
from synth import attention_layer, rafilix_config


def write_cfg(tmp_path, cfg):
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return str(tmp_path)


def test_registry_and_config_fields(tmp_path):
    import tffn
    d = write_cfg(tmp_path, mixed_config())
    assert tffn.model_family(d) == "Rafilix"
    c = tffn.qwen_config_from_json(d)
    assert (c.hidden_size, c.vocab_size, c.num_layers, c.eos_token_id, c.tie_embeddings) == (72, 211, 6, -1, 1)
    assert (c.num_heads, c.num_kv_heads, c.head_dim, c.intermediate_size) == (4, 2, 40, 72)
    assert abs(c.rms_norm_eps - 2e-5) < 1e-11
    write_cfg(tmp_path, {"hidden_size": 64, "num_attention_heads": 4, "num_key_value_heads": 2})
    assert tffn.model_family(d) == "Qwen2"
    write_cfg(tmp_path, {"architecture": "Nothing", "width": 8})
    with pytest.raises(tffn.TffnError) as e:
        tffn.model_family(d)
    assert e.value.code == -7 and "Nothing" in e.value.msg


@pytest.mark.parametrize("path,value,code", [
    (("width",), None, -3), (("vocab",), 0, -3), (("norm",), {}, -3), (("layers",), [], -3),
    (("layers", 0, "type"), "lstm", -7), (("layers", 0, "mixer", "conv"), None, -3),
    (("layers", 0, "mixer", "kv_heads"), 3, -3), (("layers", 1, "mixer", "scale"), "x", -3),
    (("layers", 1, "mixer", "rot", "dims"), 33, -3), (("layers", 1, "mixer", "rot", "scaling", "low"), None, -3),
    (("layers", 1, "mixer", "mask", "size"), 2.5, -3), (("layers", 0, "mlp", "kind"), "glu", -7),
    (("layers", 0, "mlp", "router", "top"), 9, -3),
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


def test_no_tensor_parallel_split(tmp_path):
    import tffn
    if tffn.device_count() > 0:
        pytest.skip("a GPU is present")
    d = str(tmp_path)
    synth.write_rafilix(d, mixed_config())
    with pytest.raises(tffn.TffnError) as e:
        tffn.load_model(d)  # no GPU, no CPU path
    assert e.value.code == -5


def test_plain_prefix_and_stepwise(tmp_path):
    """causal: the logits of a prefix do not change when tokens follow"""
    c = Case(tmp_path, mixed_config(), qk_norm=2.0)
    t = c.tokens(90)
    whole, _ = c.expect(t)
    part, _ = c.expect(t[:57])
    assert np.abs(whole[:57] - part).max() < 1e-9


def mutate(monkeypatch, what):
    """plant one mistake in the restatement"""
    if what == "chunk_edge":
        monkeypatch.setattr(plain, "visible_keys", lambda i, m: range(max(0, (i // m["size"]) * m["size"] - 1), i + 1))
    elif what == "chunk_short":
        monkeypatch.setattr(plain, "visible_keys",
                            lambda i, m: range(min(i, (i // m["size"]) * m["size"] + 1), i + 1))
    elif what == "half_rotation":
        def rotate(x, pos, rot):
            y, n = x.copy(), rot["dims"] // 2
            for i, f in enumerate(plain.rotary_frequencies(rot)):
                c, s = np.cos(pos * f), np.sin(pos * f)
                y[:, i], y[:, i + n] = x[:, i] * c - x[:, i + n] * s, x[:, i + n] * c + x[:, i] * s
            return y
        monkeypatch.setattr(plain, "rotate", rotate)
    elif what == "no_scaling":
        real = plain.rotary_frequencies
        monkeypatch.setattr(plain, "rotary_frequencies", lambda rot: real({k: v for k, v in rot.items() if k != "scaling"}))
    elif what == "conv_order":
        real = plain.short_conv
        monkeypatch.setattr(plain, "short_conv", lambda x, taps: real(x, taps[:, ::-1]))
    elif what == "old_state_read":
        def scan(q, k, v, g, beta, state=None):
            T, H, dim = q.shape
            S, o = np.zeros((H, dim, v.shape[2])), np.zeros_like(v)
            for t in range(T):
                for h in range(H):
                    S[h] = g[t, h][:, None] * S[h]
                    o[t, h] = S[h].T @ q[t, h]
                    S[h] += np.outer(k[t, h], beta[t, h] * (v[t, h] - S[h].T @ k[t, h]))
            return o
        monkeypatch.setattr(plain, "channel_delta_scan", scan)
    elif what == "lost_state":
        real = plain.channel_delta_scan
        monkeypatch.setattr(plain, "channel_delta_scan", lambda q, k, v, g, b, state=None: np.concatenate(
            [real(q[:40], k[:40], v[:40], g[:40], b[:40]), real(q[40:], k[40:], v[40:], g[40:], b[40:])]))
    elif what == "weights_with_correction":
        def route(h, w, p, r):
            z = h @ w[p + "router"].T
            s = np.exp(z - z.max(-1, keepdims=True))
            s = s / s.sum(-1, keepdims=True) + w[p + "correction"]
            idx = np.argsort(-s, axis=-1, kind="stable")[:, :r["top"]]
            return idx, np.take_along_axis(s, idx, axis=-1)
        monkeypatch.setattr(plain, "route", route)
    elif what == "choice_without_correction":
        def route(h, w, p, r):
            z = h @ w[p + "router"].T
            s = np.exp(z - z.max(-1, keepdims=True))
            s = s / s.sum(-1, keepdims=True)
            idx = np.argsort(-s, axis=-1, kind="stable")[:, :r["top"]]
            return idx, np.take_along_axis(s, idx, axis=-1)
        monkeypatch.setattr(plain, "route", route)
    elif what == "relu_not_squared":
        monkeypatch.setattr(plain, "expert", lambda h, w, p, e: np.maximum(h @ w[f"{p}e{e}.up"].T, 0) @ w[f"{p}e{e}.down"].T)
    else:
        raise ValueError(what)


@pytest.mark.parametrize("what,model", [
    ("chunk_edge", "odd_chunk"), ("chunk_short", "odd_chunk"), ("chunk_edge", "page_chunk"), ("half_rotation", "plain"),
    ("no_scaling", "odd_chunk"), ("conv_order", "delta"), ("old_state_read", "delta"), ("lost_state", "delta"),
    ("weights_with_correction", "moe"), ("choice_without_correction", "moe"), ("relu_not_squared", "moe")])
def test_mistakes_would_show(tmp_path, monkeypatch, what, model):
    """at the positions where a planted mistake acts, the logits leave the fp32 limit of the GPU tests many times over"""
    if model == "delta":
        width, layer = DELTA["shared_qk"]
        c = Case(tmp_path, rafilix_config(width, 97, [layer]))
    elif model == "moe":
        c = Case(tmp_path, moe_model("top3_identity"))
    else:
        width, layer, sharp = ATTENTION[model]
        c = Case(tmp_path, rafilix_config(width, 97, [layer]), qk_norm=sharp)
    t = c.tokens(80)
    good, _ = c.expect(t)
    mutate(monkeypatch, what)
    bad, _ = c.expect(t)
    e = error(bad, good)
    assert e.max() > 100 * LIMIT["float32"], e.max()
    if what in ("chunk_edge", "chunk_short", "lost_state"):  # also right behind the edge, not only on average
        first = {"lost_state": 40}.get(what, c.cfg["layers"][0]["mixer"].get("mask", {}).get("size", 0) + (what == "chunk_short"))
        assert e[first:first + 8].max() > 100 * LIMIT["float32"]


def test_frequency_scaling_has_three_ranges():
    """the test configurations exercise all three cases of the frequency scaling"""
    rot = {"base": 10000.0, "dims": 24, "scaling": SCALING}
    f, raw = plain.rotary_frequencies(rot), plain.rotary_frequencies({"base": 10000.0, "dims": 24})
    r = f / raw
    assert (r == 1.0).any() and np.isclose(r, 1 / SCALING["factor"]).any()
    assert ((r < 1.0) & (r > 1.001 / SCALING["factor"])).any()
