"""-m gpu: the Razesun family on the CUDA path against the plain 64-bit restatement (oracle/razesun_plain.py): every
mechanism alone, then whole models under every way of cutting, batching and re-using slots. fp32 sessions are held to a
tight limit; bf16 sessions to one that leaves room for the rounding of products and activations."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import synth
from razesun_cases import DELTA, DENSE, LATENT, LIMIT, RGLRU, Case, error, mixed_config, plant_key
from synth import delta_layer, dense_mlp, latent_layer, razesun_config, rglru_layer

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def check(got, want, compute, what=""):
    e = error(got, want)
    assert e.max() <= LIMIT[compute], (what, int(e.argmax()), float(e.max()))


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
    return Case(tmp_path_factory.mktemp("razesun_mixed"), mixed_config(), seed=3, sharp=1.5)


# ------------------------------------------------------------------------------------------- mechanisms alone
def alone(path, cfg, compute, sharp=1.0, n=170, sizes=None, edit=None):
    """a prompt at once with the residual stream behind every layer, then the same tokens partly decoded one by one"""
    c = Case(path, cfg, sharp=sharp, edit=edit)
    t = c.tokens(n)
    want, after = c.expect(t)
    s = c.session(compute, max_seq=n + 30)
    s.capture_hidden(n)
    check(s.qwen_forward(t), want, compute, "prompt")
    for i in range(len(after)):
        tol = 1e-5 if compute == "float32" else 3e-2
        assert np.abs(s.get_hidden_f32(i, n) - after[i]).max() <= tol * np.abs(after[i]).max()
    s.capture_hidden(0)
    s.qwen_reset()
    check(in_portions(s, t, sizes or [61] + [1] * 75 + [34]), want, compute, "decoded")
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(LATENT))
def test_latent_attention_alone(tmp_path, name, compute):
    width, layer, sharp = LATENT[name]
    alone(tmp_path, razesun_config(width, 97, [layer]), compute, sharp=sharp if compute == "float32" else 1.0)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_rows_of_another_layer(tmp_path, compute):
    """layers that read the rows an earlier layer cached: other heads and sizes, own queries, not only the next layer"""
    a = latent_layer(3, 24, 16, 20, 72, 40)
    layers = [a, latent_layer(5, 16, 16, 32, 72, 24, kv_from=0, scale=0.4), latent_layer(2, 32, 8, 16, 40, 32, base=99.0),
              latent_layer(1, 40, 16, 8, 72, 56, kv_from=0), latent_layer(4, 8, 8, 24, 40, 16, base=99.0, kv_from=2)]
    alone(tmp_path, razesun_config(56, 97, layers), compute, sharp=2.0 if compute == "float32" else 1.0)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(DELTA))
def test_delta_rule_alone(tmp_path, name, compute):
    width, layer = DELTA[name]
    alone(tmp_path, razesun_config(width, 97, [layer]), compute, n=90, sizes=[2, 3, 1, 1, 20, 1, 7, 1])


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(RGLRU))
def test_real_gated_recurrence_alone(tmp_path, name, compute):
    width, layer = RGLRU[name]
    alone(tmp_path, razesun_config(width, 97, [layer]), compute, sizes=[2, 3, 1, 1, 65, 1, 7, 1])


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(DENSE))
def test_parallel_block(tmp_path, name, compute):
    """both sublayers read the same stream through norms of their own; constants that are not one"""
    width, mlp = DENSE[name]
    alone(tmp_path, razesun_config(width, 97, [rglru_layer(16, 2, mlp=mlp), rglru_layer(24, 1, mlp=None)], eps=3e-2, residual_mult=-1.7,
                                   logit_scale=0.05), compute)


def test_delta_rule_keeps_and_forgets(tmp_path):
    """decays of nearly one (a state that a lost carry would change for good) and of nearly zero, beta near one"""
    def edit(name, x):
        if name.endswith("A_log"):
            return np.linspace(-9.0, 3.0, x.size).reshape(x.shape)
        if name.endswith("mix.b"):
            return x * 6.0
    c = Case(tmp_path, razesun_config(48, 97, [delta_layer(6, 3, 32, 32)]), edit=edit)
    t = c.tokens(200)
    want, _ = c.expect(t)
    s = c.session(max_seq=256)
    check(in_portions(s, t, [60, 1, 1, 30]), want, "float32")
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_real_gated_recurrence_remembers(tmp_path, compute):
    """decays from almost one to almost zero; the first token still shows hundreds of tokens later"""
    def edit(name, x):
        if name.endswith("lam"):
            return np.linspace(-14.0, 3.0, x.size).reshape(x.shape)
    c = Case(tmp_path, razesun_config(48, 97, [rglru_layer(40, 5)], residual_mult=2.0), edit=edit)
    t = c.tokens(420)
    want, _ = c.expect(t)
    other = t.copy()
    other[0] = (t[0] + 1) % 97
    assert error(c.expect(other)[0], want)[-1] > 10 * LIMIT["float32"]
    s = c.session(compute, max_seq=440)
    check(s.qwen_forward(t), want, compute)
    s.qwen_reset()
    check(in_portions(s, t, [64, 65, 1, 128, 63, 1, 1]), want, compute)
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("decoded", [False, True])
def test_one_far_key(tmp_path, decoded, compute):
    """one key that one later query asks for decides that query's row at every distance: the first token, borders of pages,
    of key tiles and of context splits, the query's own predecessor; in the layer that cached it and in one that borrows"""
    c, key, ask, other = plant_key(tmp_path)
    filler = c.tokens(1300, seed=5)
    filler[np.isin(filler, [key, ask])] = other
    s = c.session(compute, max_seq=1400)
    for kpos, apos in [(0, 1), (0, 63), (31, 64), (32, 65), (63, 64), (64, 127), (10, 300), (5, 511), (511, 512), (512, 640), (0, 1099), (383, 1099), (384, 1150),
                       (575, 1151), (576, 1200), (1098, 1099), (1023, 1024)]:
        t = filler[:apos + 1].copy()
        t[kpos], t[apos] = key, ask
        want = c.expect(t)[0][apos]
        without = t.copy()
        without[kpos] = other
        assert error(c.expect(without)[0][apos:], want[None])[0] > 3 * LIMIT["bfloat16"], (kpos, apos)  # the plant is seen
        s.qwen_reset()
        if decoded:
            s.qwen_forward(t[:apos], want_logits=False)
            got = s.decode_step(t[apos:], want_logits=True)[1]
        else:
            got = s.qwen_forward(t)[apos:]
        check(got, want[None], compute, (kpos, apos))
    s.free()


def test_one_key_among_thousands(tmp_path):
    """a context of more splits than a cluster holds: their rows go through the workspace; a key in the first, in the middle
    and in the last of them"""
    c, key, ask, other = plant_key(tmp_path)
    filler = c.tokens(4750, seed=6)
    filler[np.isin(filler, [key, ask])] = other
    s = c.session("bfloat16", max_seq=4800)
    for kpos in (3, 2304, 4700):
        t = filler.copy()
        t[kpos], t[-1] = key, ask
        want = c.expect(t, last=1)[0]
        s.qwen_reset()
        s.prefill([t[:-1]])
        check(s.decode_step(t[-1:], want_logits=True)[1], want, "bfloat16", kpos)
        t[kpos] = other
        assert error(c.expect(t, last=1)[0], want)[0] > 3 * LIMIT["bfloat16"]  # the plant is seen
    s.free()


# ------------------------------------------------------------------------------------------- schedules
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2], [2, 37, 5], [64], [33, 1, 1], [129, 1, 1, 1, 8]])
def test_portions(mixed, sizes, compute):
    t = mixed.tokens(150)
    want, _ = mixed.expect(t)
    s = mixed.session(compute, max_seq=160)
    check(in_portions(s, t, sizes), want, compute)
    assert s.status() == 0
    s.free()


@pytest.mark.parametrize("mode", [1, 2])
def test_launch_modes_agree(mixed, mode):
    """plain launches, dependent launches and graph replay run the same kernels: bit-equal logits"""
    t = mixed.tokens(100, seed=9)
    runs = []
    for m in (0, mode):
        s = mixed.session("bfloat16", max_seq=128, mode=m)
        runs.append(in_portions(s, t, [25] + [1] * 75))
        s.free()
    assert np.array_equal(runs[0], runs[1])


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_batch_of_unequal_requests(mixed, compute):
    """prompts of 1 to 130 tokens prefilled together and decoded together give what each gives alone, and what the
    restatement gives; a second prefill appends unequal pieces to all of them"""
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


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_large_batch(mixed, compute):
    """more sequences than fill the GPU: one context split, several token tiles per product"""
    n, steps = 150, 4
    lens = [1 + (7 * i) % 40 for i in range(n)]
    seqs = [mixed.tokens(k + steps, seed=200 + i) for i, k in enumerate(lens)]
    s = mixed.session(compute, max_batch=n, max_seq=64)
    first = s.prefill([q[:k] for q, k in zip(seqs, lens)], want_logits=True)[1].copy()
    rows = [s.decode_step([q[k + j] for q, k in zip(seqs, lens)], want_logits=True)[1].copy() for j in range(steps)]
    for i in (0, 1, 63, 64, 77, 127, 128, 149):
        want, _ = mixed.expect(seqs[i])
        got = np.stack([first[i]] + [r[i] for r in rows])
        assert error(got, want[lens[i] - 1:]).max() <= LIMIT[compute], i
    s.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_slots_and_pages_are_reused(mixed, compute):
    """requests that come and go through the same slots: recurrent state, convolution inputs and pages of an earlier
    request never reach a later one, whatever pages it gets; neighbours in other slots are not disturbed"""
    s = mixed.session(compute, max_batch=3, max_seq=160)
    keep = mixed.tokens(140, seed=40)
    want_keep, _ = mixed.expect(keep)
    at = 30
    check(s.qwen_forward(keep[:at], slot=1), want_keep[:at], compute)
    for r, n in enumerate([100, 1, 33, 2, 64, 7]):
        q = mixed.tokens(n, seed=50 + r)
        want, _ = mixed.expect(q)
        slot = 0 if r % 2 == 0 else 2
        check(in_portions(s, q, [40, 2, 1], slot=slot), want, compute, r)
        part = keep[at:at + 15]
        check(s.qwen_forward(part, slot=1), want_keep[at:at + 15], compute, ("kept", r))
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
    check(s.qwen_forward(b, slot=1), want, compute)
    want, _ = mixed.expect(a)
    check(s.qwen_forward(a[64:], slot=2), want[64:], compute)
    s.free()


def test_first_tokens(mixed):
    """sequences of one to five tokens, shorter than any convolution or page, as prompts and decoded"""
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


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_launch_row_limit_is_no_boundary(tmp_path, compute):
    """a prefill of more rows than one launch takes: a sequence continues across launches"""
    c = Case(tmp_path, razesun_config(32, 64, [delta_layer(2, 1, 16, 16, mlp=dense_mlp(16)), latent_layer(1, 16, 8, 16, 24, 16),
                                               rglru_layer(16, 2)]))
    n = [1500, 2000, 1000]
    seqs = [c.tokens(k, seed=80 + i) for i, k in enumerate(n)]
    s = c.session(compute, max_batch=3, max_seq=2048)
    got = s.prefill(seqs, want_logits=True)[1]
    for i, q in enumerate(seqs):
        want, _ = c.expect(q)
        check(got[i:i + 1], want[-1:], compute, i)
    s.free()


# ------------------------------------------------------------------------------------------- generation
def test_long_greedy_decoding(mixed):
    """device-resident greedy decoding over many page and state updates, several sequences at once: every token is the
    restatement's own pick after the same history (or within rounding of it)"""
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


@pytest.mark.parametrize("scale", [0.02, -0.5])
def test_greedy_pick_follows_the_scaled_logits(tmp_path, scale):
    """the pick is the largest of head x * logit_scale, whatever the scale's size or sign"""
    c = Case(tmp_path, razesun_config(48, 300, [rglru_layer(32, 2, mlp=dense_mlp(40))], logit_scale=scale))
    p = c.tokens(20)
    want, _ = c.expect(p)
    for compute in ("float32", "bfloat16"):
        s = c.session(compute, max_seq=64)
        nxt, lg = s.prefill([p], want_logits=True)
        check(lg, want[-1:], compute)
        assert int(nxt[0]) == int(lg[0].argmax())
        step, lg = s.decode_step([int(nxt[0])], want_logits=True)
        assert int(step[0]) == int(lg[0].argmax())
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
            check(np.fromfile(out / f"{k}.f32", np.float32).reshape(w.shape), w, compute, k)


# ------------------------------------------------------------------------------------------- limits
def test_refusals(mixed, tmp_path):
    """what the family does not have is an error that says so, and leaves the session usable"""
    import tffn
    assert mixed.model.family == "Razesun"
    with pytest.raises(tffn.TffnError):
        tffn.load_model(mixed.dir, tp_rank=0, tp_size=2)
    s = mixed.session(max_seq=40)
    with pytest.raises(tffn.TffnError) as e:
        s.qwen_forward(mixed.tokens(41))
    assert e.value.code == -6
    with pytest.raises(tffn.TffnError):
        s.qwen_forward([mixed.cfg["vocab"]])
    want, _ = mixed.expect(mixed.tokens(20))
    check(s.qwen_forward(mixed.tokens(20)), want, "float32")
    s.free()
    # a tensor of the wrong shape, and one that is missing
    for i, (edit_name, drop) in enumerate([("l1.mix.uk", False), ("l0.mix.ra", False), ("l2.mix.a", False), ("embed.norm", True), ("head", True),
                                           ("l1.mix.dkv", True)]):
        bad = tmp_path / str(i)
        synth.write_razesun(str(bad), mixed.cfg)
        tensors = []
        for n, shape, _, _ in synth.razesun_specs(mixed.cfg):
            if n == edit_name and drop:
                continue
            shape = tuple(shape[:-1]) + (shape[-1] + 1,) if n == edit_name else shape
            tensors.append((n, shape, np.zeros(int(np.prod(shape)), np.uint16)))
        synth.write_safetensors(str(bad / "model.safetensors"), tensors)
        with pytest.raises(tffn.TffnError) as e:
            tffn.load_model(str(bad))
        assert e.value.code in (-3, -4) and edit_name in e.value.msg
