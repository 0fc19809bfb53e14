"""-m gpu: the Rafilix family on the CUDA path against the plain 64-bit restatement (oracle/rafilix_plain.py): every
mechanism alone, then whole models under every way of cutting, batching and re-using slots. fp32 sessions are held to a
tight limit; bf16 sessions to one that leaves room for the rounding of products and activations."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import synth
from rafilix_cases import ATTENTION, DELTA, LIMIT, MOE, Case, error, mixed_config, moe_model
from synth import attention_layer, channel_delta_layer, moe_mlp, rafilix_config

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def check(got, want, compute, what=""):
    e = error(got, want)
    if compute == "float32":
        assert e.max() <= LIMIT[compute], (what, int(e.argmax()), float(e.max()))
    else:  # a choice of experts that is a near tie may fall the other way at a few positions
        assert (e > LIMIT[compute]).mean() <= 0.05, (what, float(np.quantile(e, 0.9)), float(e.max()))
    return e


def in_portions(sess, tokens, sizes, slot=0):
    """logits of all positions, the tokens cut into portions of the given sizes (cycled); single tokens decode"""
    out, i, k = [], 0, 0
    while i < len(tokens):
        n = min(sizes[k % len(sizes)], len(tokens) - i)
        part = tokens[i:i + n]
        if n == 1 and slot == 0 and i > 0:
            out.append(sess.decode_step(part, want_logits=True)[1])
        else:
            out.append(sess.qwen_forward(part, slot=slot))
        i, k = i + n, k + 1
    return np.concatenate(out)


@pytest.fixture(scope="module")
def mixed(tmp_path_factory):
    return Case(tmp_path_factory.mktemp("rafilix_mixed"), mixed_config(), seed=3, qk_norm=1.5)


@pytest.fixture(scope="module")
def settled(tmp_path_factory):
    """the same layers with mild scores and corrections that settle every choice of experts: random routers have near
    ties, which bf16 rounding decides differently and which then mask everything behind them"""
    def edit(name, x):
        if name.endswith("correction"):
            return np.random.default_rng(len(name) + x.size).permutation(x.size) * 1.5
    return Case(tmp_path_factory.mktemp("rafilix_settled"), mixed_config(), seed=4, edit=edit)


@pytest.fixture(scope="module")
def model_for(mixed, settled):
    return {"float32": mixed, "bfloat16": settled}


# ------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ATTENTION))
def test_attention_alone(tmp_path, name, compute):
    """chunks, rotation, per-head norms and scaling for many head geometries: a prompt at once, then the same tokens as a
    prompt part and decoded one by one; every position is compared, so every chunk's edge is"""
    width, layer, sharp = ATTENTION[name]
    c = Case(tmp_path, rafilix_config(width, 97, [layer]), qk_norm=sharp if compute == "float32" else 1.0)
    t = c.tokens(170)
    want, after = c.expect(t)
    s = c.session(compute, max_seq=200)
    s.capture_hidden(200)
    check(s.qwen_forward(t), want, compute, "prompt")
    if compute == "float32":
        assert np.abs(s.get_hidden_f32(0, 200) - after[0]).max() <= 1e-4 * np.abs(after).max()
    s.capture_hidden(0)
    s.qwen_reset()
    check(in_portions(s, t, [61] + [1] * 75 + [34]), want, compute, "decoded")
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(DELTA))
def test_channel_delta_alone(tmp_path, name, compute):
    width, layer = DELTA[name]
    c = Case(tmp_path, rafilix_config(width, 97, [layer]), rank=10)
    t = c.tokens(90)
    want, after = c.expect(t)
    s = c.session(compute, max_seq=128)
    s.capture_hidden(128)
    check(s.qwen_forward(t), want, compute, "prompt")
    if compute == "float32":
        assert np.abs(s.get_hidden_f32(0, 128) - after[0]).max() <= 1e-4 * np.abs(after).max()
    s.capture_hidden(0)
    s.qwen_reset()
    check(in_portions(s, t, [2, 3, 1, 1, 20, 1, 7, 1]), want, compute, "portions")
    s.free()


def test_delta_rule_keeps_and_forgets(tmp_path):
    """decays of nearly one (a state that a lost carry would change for good) and of nearly zero, beta near one"""
    def edit(name, x):
        if name.endswith("A_log"):
            return np.linspace(-9.0, 3.0, x.size).reshape(x.shape)
        if name.endswith("mix.b"):
            return x * 6.0
    c = Case(tmp_path, rafilix_config(48, 97, [channel_delta_layer(6, 3, 32, 32)]), edit=edit)
    t = c.tokens(200)
    want, _ = c.expect(t)
    s = c.session(max_seq=256)
    check(in_portions(s, t, [60, 1, 1, 30]), want, "float32")
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MOE))
def test_experts(tmp_path, name, compute):
    c = Case(tmp_path, moe_model(name))
    t = c.tokens(150)
    want, after = c.expect(t)
    s = c.session(compute, max_seq=256)
    s.capture_hidden(256)
    check(s.qwen_forward(t), want, compute, "prompt")
    if compute == "float32":
        assert np.abs(s.get_hidden_f32(0, 256) - after[0]).max() <= 1e-4 * np.abs(after).max()
    s.capture_hidden(0)
    s.qwen_reset()
    check(in_portions(s, t, [100, 1, 1, 1, 5]), want, compute, "decoded")
    s.free()


def test_all_rows_choose_one_expert(tmp_path):
    """the worst case of the grouped launches: every token at the same expert (several tiles), the others empty; and
    the choice made by the correction alone while the weights ignore it"""
    def edit(name, x):
        if name.endswith("correction"):
            y = np.zeros_like(x)
            y[2], y[5] = 8.0, 4.0  # expert 2 and the identity expert 5 for everybody
            return y
    c = Case(tmp_path, rafilix_config(64, 97, [attention_layer(2, 1, 16, 16, chunk=20, mlp=moe_mlp(5, 2, 40, identity=1))]), edit=edit)
    t = c.tokens(300)
    want, _ = c.expect(t)
    for compute in ("float32", "bfloat16"):
        s = c.session(compute, max_seq=320)
        check(in_portions(s, t, [280, 1, 1, 18]), want, compute)
        s.free()


@pytest.mark.parametrize("decoded", [False, True])
def test_one_key_inside_and_outside_a_chunk(tmp_path, decoded):
    """a planted key that one later query asks for: it decides the logits at every distance inside the chunk, and is
    invisible from the first position of the next chunk on"""
    width, chunk, key, ask, other = 48, 45, 11, 12, 13

    def edit(name, x):
        if name == "embed":
            x[:, :4] = 0.0
            x[key] = x[ask] = 0.0
            x[key, 0], x[ask, 1] = 6.0, 6.0
            x[key, 4:] = np.linspace(-1, 1, width - 4)
            return x
        if name.endswith(("mix.q", "mix.k")):  # query of `ask` and key of `key` share one direction
            x *= 0.05
            x[:, 0 if name.endswith("k") else 1] = np.linspace(1, 2, x.shape[0])
            return x
    layer = attention_layer(1, 1, 16, 32, chunk=chunk, rot_dims=0, scale=2.0)
    c = Case(tmp_path, rafilix_config(width, 64, [layer]), edit=edit, qk_norm=1.0)
    filler = c.tokens(200, seed=5)
    filler[np.isin(filler, [key, ask])] = other
    s = c.session(max_seq=256)
    for kpos, apos in [(45, 46), (45, 89), (45, 90), (44, 45), (31, 32), (31, 44), (64, 89), (90, 134), (90, 135), (0, 44)]:
        t = filler[:apos + 1].copy()
        t[kpos], t[apos] = key, ask
        want, _ = c.expect(t)
        without = t.copy()
        without[kpos] = other
        moved = error(c.expect(without)[0], want)[apos]
        if kpos // chunk == apos // chunk:
            assert moved > 1000 * LIMIT["float32"], (kpos, apos)  # the plant is seen
        else:
            assert moved == 0.0
        s.qwen_reset()
        got = in_portions(s, t, [max(1, apos)] + [1] * 3 if decoded else [len(t)])
        check(got, want, "float32", (kpos, apos))
    s.free()


# ------------------------------------------------------------------------------------------- schedules
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2], [2, 37, 5], [64], [33, 1, 1], [129, 1, 1, 1, 8]])
def test_portions(model_for, sizes, compute):
    mixed = model_for[compute]
    t = mixed.tokens(150)
    want, _ = mixed.expect(t)
    s = mixed.session(compute, max_seq=160)
    check(in_portions(s, t, sizes), want, compute)
    assert s.status() == 0
    s.free()


@pytest.mark.parametrize("mode", [0, 1, 2])
def test_launch_modes_agree(mixed, mode):
    """plain launches, dependent launches and graph replay run the same kernels: bit-equal logits"""
    t = mixed.tokens(60, seed=9)
    runs = []
    for m in (0, mode):
        s = mixed.session("bfloat16", max_seq=96, mode=m)
        runs.append(in_portions(s, t, [25] + [1] * 35))
        s.free()
    assert np.array_equal(runs[0], runs[1])


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_batch_of_unequal_requests(model_for, compute):
    """prompts of 1 to 130 tokens prefilled together and decoded together give what each gives alone, and what the
    restatement gives; a second prefill appends unequal pieces to all of them"""
    mixed = model_for[compute]
    lens, more, steps = [37, 1, 130, 64, 5], [3, 20, 1, 2, 33], 12
    seqs = [mixed.tokens(n + m + steps, seed=20 + i) for i, (n, m) in enumerate(zip(lens, more))]
    s = mixed.session(compute, max_batch=5, max_seq=256)
    first = s.prefill([q[:n] for q, n in zip(seqs, lens)], want_logits=True)[1].copy()
    second = s.prefill([q[n:n + m] for q, n, m in zip(seqs, lens, more)], want_logits=True)[1].copy()
    rows = []
    for k in range(steps):
        rows.append(s.decode_step([q[n + m + k] for q, n, m in zip(seqs, lens, more)], want_logits=True)[1].copy())
    one = mixed.session(compute, max_seq=256)
    for i, (q, n, m) in enumerate(zip(seqs, lens, more)):
        want, _ = mixed.expect(q)
        got = np.stack([first[i], second[i]] + [r[i] for r in rows])
        at = [n - 1, n + m - 1] + list(range(n + m, n + m + steps))
        assert error(got, want[at]).max() <= LIMIT[compute], i
        one.qwen_reset()
        alone = in_portions(one, q, [n, m] + [1] * steps)[at]
        assert error(got, alone).max() <= LIMIT[compute], i
    s.free()
    one.free()


def test_slots_and_pages_are_reused(mixed):
    """requests that come and go through the same slots: recurrent state, convolution inputs and pages of an earlier
    request never reach a later one, whatever pages it gets; neighbours in other slots are not disturbed"""
    s = mixed.session(max_batch=3, max_seq=160)
    keep = mixed.tokens(140, seed=40)
    want_keep, _ = mixed.expect(keep)
    at = 30
    check(s.qwen_forward(keep[:at], slot=1), want_keep[:at], "float32")
    for r, n in enumerate([100, 1, 33, 2, 64, 7]):
        q = mixed.tokens(n, seed=50 + r)
        want, _ = mixed.expect(q)
        slot = 0 if r % 2 == 0 else 2
        check(in_portions(s, q, [40, 2, 1], slot=slot), want, "float32", r)
        part = keep[at:at + 15]
        check(s.qwen_forward(part, slot=1), want_keep[at:at + 15], "float32", ("kept", r))
        at += 15
        s.qwen_reset(slot)
        assert s.seq_len(slot) == 0 and s.seq_len(1) == at
    s.qwen_reset()
    # scattered pages: slots filled in turn, one freed, its pages taken over by a longer request
    a, b = mixed.tokens(70, seed=60), mixed.tokens(150, seed=61)
    for i in range(0, 64, 16):
        for slot in (0, 1, 2):
            s.qwen_forward(a[i:i + 16], slot=slot, want_logits=False)
    s.qwen_reset(1)
    want, _ = mixed.expect(b)
    check(s.qwen_forward(b, slot=1), want, "float32")
    want, _ = mixed.expect(a)
    check(s.qwen_forward(a[64:], slot=2), want[64:], "float32")
    s.free()


def test_first_tokens(mixed):
    """sequences of one to five tokens, shorter than any convolution, chunk or page, as prompts and decoded"""
    s = mixed.session(max_batch=2, max_seq=64)
    for n in range(1, 6):
        t = mixed.tokens(n, seed=70 + n)
        want, _ = mixed.expect(t)
        s.qwen_reset()
        check(s.qwen_forward(t), want, "float32", n)
        s.qwen_reset()
        rows = [s.decode_step([int(x), int(x)], want_logits=True)[1].copy() for x in t]  # two slots from nothing
        for b in range(2):
            check(np.stack([r[b] for r in rows]), want, "float32", (n, b))
    s.free()


def test_launch_row_limit_is_no_boundary(tmp_path):
    """a prefill of more rows than one launch takes: a sequence continues across launches inside a chunk"""
    c = Case(tmp_path, rafilix_config(32, 64, [channel_delta_layer(2, 1, 16, 16, mlp=moe_mlp(3, 2, 16, identity=1)),
                                               attention_layer(2, 1, 16, 16, chunk=300)]))
    n = [1500, 2000, 1000]
    seqs = [c.tokens(k, seed=80 + i) for i, k in enumerate(n)]
    s = c.session(max_batch=3, max_seq=2048)
    got = s.prefill(seqs, want_logits=True)[1]
    for i, q in enumerate(seqs):
        want, _ = c.expect(q)
        check(got[i:i + 1], want[-1:], "float32", i)
    s.free()


# ------------------------------------------------------------------------------------------- generation
def test_long_greedy_decoding(mixed):
    """device-resident greedy decoding over many chunk, page and state updates, several sequences at once: every token is
    the restatement's own pick after the same history (or within rounding of it)"""
    lens, steps = [3, 40, 71], 180
    s = mixed.session(max_batch=3, max_seq=300)
    prompts = [mixed.tokens(n, seed=90 + i) for i, n in enumerate(lens)]
    nxt, _ = s.prefill(prompts)
    toks = s.decode_run(3, steps)
    for i, p in enumerate(prompts):
        gen = np.concatenate([[nxt[i]], toks[:, i]])
        want, _ = mixed.expect(np.concatenate([p, gen]))
        w = want[len(p) - 1:len(p) + steps]
        gap = w.max(axis=1) - w[np.arange(steps + 1), gen]
        assert (gap <= 1e-3 * w.std()).all(), (i, int(gap.argmax()), float(gap.max()))
    s.free()


def test_sampling_follows_the_logits(mixed):
    """the session's sampler runs on this family's logits: a tiny temperature gives the greedy tokens, a seed repeats"""
    p = mixed.tokens(30, seed=100)
    out = {}
    for key, temp, seed in [("greedy", 0.0, 1), ("cold", 1e-4, 1), ("hot", 3.0, 5), ("again", 3.0, 5), ("other", 3.0, 6)]:
        s = mixed.session(max_seq=96)
        if temp > 0:
            s.set_sampling(temp, seed)
        nxt, _ = s.prefill([p])
        out[key] = [int(nxt[0])] + [int(x) for x in s.decode_run(1, 24)[:, 0]]
        s.free()
    assert out["cold"] == out["greedy"] and out["hot"] == out["again"] != out["other"]


def test_command_line_generates(mixed, tmp_path):
    """tensor-ffn-inference --prompt-ids on a folder without a tokenizer prints the ids the library generates"""
    p = mixed.tokens(33, seed=110)
    p.tofile(tmp_path / "ids.i32")
    cli = os.path.join(ROOT, "tensor-ffn_b200", "tensor-ffn-inference")
    for compute in ("float32", "bfloat16"):
        r = subprocess.run([cli, "--model", mixed.dir, "--prompt-ids", str(tmp_path / "ids.i32"), "--dtype", compute, "--max-tokens", "20",
                            "--max-seq", "96", "--device", "0"], capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        ids = [int(x) for x in r.stdout.split("Generating:")[1].split()]
        s = mixed.session(compute, max_seq=96, mode=1)
        nxt, _ = s.prefill([p])
        assert ids == [int(nxt[0])] + [int(x) for x in s.decode_run(1, 19)[:, 0]]
        s.free()


def test_trace_replay(mixed, tmp_path):
    """bin/trace_run: portions of interleaved requests, wanted places only, slots given back"""
    a, b = mixed.tokens(60, seed=120), mixed.tokens(41, seed=121)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50].tolist(), "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:40].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[50:].tolist(), "want": [3]}, {"id": "b", "tokens": b[40:].tolist(), "want": [0]}],
              "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:20].tolist(), "want": [19]}], "end": []},
             {"step": 4, "entries": [{"id": "c", "tokens": b[20:21].tolist(), "want": [0]}], "end": ["c"]}]
    wa, wb = mixed.expect(a)[0], mixed.expect(b)[0]
    want = {0: wa[[0, 49]], 2: np.stack([wa[53], wb[40]]), 3: wb[19:20], 4: wb[20:21]}
    for compute in ("float32", "bfloat16"):
        out = tmp_path / compute
        out.mkdir()
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", mixed.dir, "--dtype", compute, "--out", str(out),
                            "--max-tokens", "160"], input="\n".join(json.dumps(x) for x in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(5)]
        assert not (out / "1.f32").exists()
        for k, w in want.items():
            got = np.fromfile(out / f"{k}.f32", np.float32).reshape(w.shape)
            e = error(got, w)
            assert e.max() <= (LIMIT[compute] if compute == "float32" else 3 * LIMIT[compute])


# ------------------------------------------------------------------------------------------- limits
def test_refusals(mixed, model_dirs, tmp_path):
    """what the family does not have is an error that says so"""
    import tffn
    d, ep, _ = model_dirs["tiny"]
    qwen = tffn.load_model(d)
    assert (qwen.family, mixed.model.family) == ("Qwen2", "Rafilix")
    with pytest.raises(tffn.TffnError) as e:
        tffn.Session(qwen, compute="float32")
    assert e.value.code == -7
    with pytest.raises(tffn.TffnError):
        tffn.load_model(mixed.dir, tp_rank=0, tp_size=2)
    with pytest.raises(tffn.TffnError):
        tffn.checkpoint_load(ep, mixed.model)
    s = mixed.session(max_seq=40)
    with pytest.raises(tffn.TffnError) as e:
        s.qwen_forward(mixed.tokens(41))
    assert e.value.code == -6
    with pytest.raises(tffn.TffnError):
        s.qwen_forward([mixed.cfg["vocab"]])
    want, _ = mixed.expect(mixed.tokens(20))
    check(s.qwen_forward(mixed.tokens(20)), want, "float32")  # a refused call left nothing behind
    s.free()
    # a tensor of the wrong shape, and one that is missing
    for edit_name in ("l0.mix.a2", "l1.mix.q.norm"):
        bad = tmp_path / edit_name
        synth.write_rafilix(str(bad), mixed.cfg, rank=12, edit=lambda n, x, m=edit_name: None)
        specs = [x for x in synth.rafilix_specs(mixed.cfg, 12)]
        tensors = []
        for n, shape, _, _ in specs:
            if n == edit_name and n.endswith("norm"):
                continue
            shape = tuple(reversed(shape)) if n == edit_name else shape
            tensors.append((n, shape, np.zeros(int(np.prod(shape)), np.uint16)))
        synth.write_safetensors(str(bad / "model.safetensors"), tensors)
        with pytest.raises(tffn.TffnError) as e:
            tffn.load_model(str(bad))
        assert e.value.code in (-3, -4) and edit_name in e.value.msg
