"""Small configurations of the Rafilix family for the tests, and helpers that run them through the library and through
the plain restatement."""
import os

import numpy as np

import rafilix_plain as plain
import synth
from synth import attention_layer, channel_delta_layer, moe_mlp, rafilix_config

SCALING = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}

# One mechanism per model: a single layer without (or with only) a feed-forward. Sharp scores (large norm weights of q
# and k) make nearly every query depend on one key, so that a key too many or too few at an edge shows.
ATTENTION = {
    # name: (width, layer, norm weight of q and k)
    "plain": (64, attention_layer(4, 2, 32, 32, chunk=50), 3.0),
    "page_chunk": (64, attention_layer(2, 2, 64, 64, chunk=32), 2.0),
    "page_chunk_plus": (64, attention_layer(2, 1, 64, 32, chunk=33), 2.0),
    "odd_chunk": (48, attention_layer(3, 1, 40, 24, chunk=17, rot_dims=24, scaling=SCALING), 3.0),
    "tiny_chunk": (48, attention_layer(3, 3, 16, 48, chunk=3, base=500.0), 2.0),
    "chunk_of_one": (40, attention_layer(2, 1, 16, 16, chunk=1), 1.0),
    "wide_value": (64, attention_layer(4, 4, 48, 112, chunk=70, scaling=SCALING), 3.0),
    "many_queries": (64, attention_layer(20, 2, 32, 32, chunk=45, rot_dims=8), 3.0),
    "one_key_head": (72, attention_layer(12, 1, 80, 80, chunk=90, scale=0.2), 1.5),
    "wide_head": (64, attention_layer(2, 1, 160, 144, chunk=41, scaling=dict(SCALING, factor=8.0, high=3.0)), 1.5),
    "unaligned": (52, attention_layer(3, 1, 18, 10, chunk=29, rot_dims=6), 2.0),
    "no_rotation": (48, attention_layer(2, 2, 24, 24, chunk=37, rot_dims=0), 2.0),
}
DELTA = {
    "plain": (64, channel_delta_layer(4, 4, 32, 32)),
    "shared_qk": (64, channel_delta_layer(6, 2, 32, 48, conv=3)),
    "one_group": (48, channel_delta_layer(4, 1, 64, 16, conv=2)),
    "no_conv": (48, channel_delta_layer(3, 3, 24, 40, conv=1)),
    "long_conv": (64, channel_delta_layer(2, 1, 96, 64, conv=7)),
    "wide": (64, channel_delta_layer(2, 2, 128, 128)),
    "very_wide": (64, channel_delta_layer(2, 1, 200, 160)),
    "widest_value": (40, channel_delta_layer(1, 1, 40, 250)),
    "unaligned": (52, channel_delta_layer(3, 1, 18, 10, conv=4)),
}
# the layer in front is a small attention so that the rows differ by position
MOE = {
    "top1": (64, moe_mlp(4, 1, 32)),
    "top3_identity": (64, moe_mlp(5, 3, 48, identity=3)),
    "all": (48, moe_mlp(3, 4, 40, identity=1)),
    "many": (96, moe_mlp(70, 8, 24, identity=6)),
    "mostly_identity": (48, moe_mlp(1, 2, 136, identity=4)),
    "unaligned": (52, moe_mlp(6, 2, 30, identity=1)),
    "wide": (160, moe_mlp(3, 2, 300)),
}


def moe_model(name, vocab=97):
    width, mlp = MOE[name]
    return rafilix_config(width, vocab, [attention_layer(2, 1, 16, 16, chunk=20, mlp=mlp)])


def mixed_config(width=72, vocab=211):
    """every mechanism and both kinds of layers in an order of their own, sizes that differ from each other"""
    return rafilix_config(width, vocab, [
        channel_delta_layer(4, 2, 40, 24, conv=3, mlp=moe_mlp(6, 3, 40, identity=2)),
        attention_layer(6, 2, 32, 48, chunk=40, rot_dims=16, scaling=SCALING, base=3000.0, mlp=moe_mlp(4, 1, 56)),
        attention_layer(4, 4, 24, 24, chunk=75, base=20000.0, mlp=None),
        channel_delta_layer(3, 3, 64, 64, conv=4, mlp=None),
        channel_delta_layer(2, 1, 16, 96, conv=1, mlp=moe_mlp(9, 2, 24, identity=1)),
        attention_layer(8, 1, 56, 40, chunk=33, mlp=moe_mlp(5, 2, 72, identity=3)),
    ], eps=2e-5)


class Case:
    """a model folder with its library model and its plain weights"""

    def __init__(self, path, cfg, seed=1, rank=12, qk_norm=1.0, edit=None):
        self.dir, self.cfg = str(path), cfg
        synth.write_rafilix(self.dir, cfg, seed=seed, rank=rank, qk_norm=qk_norm, edit=edit)
        self.plain_cfg, self.w = plain.load_dir(self.dir)
        self._model = None

    @property
    def model(self):
        import tffn
        if self._model is None:
            self._model = tffn.load_model(self.dir)
        return self._model

    def session(self, compute="float32", max_batch=1, max_seq=512, mode=2):
        import tffn
        s = tffn.Session(self.model, max_batch=max_batch, max_seq=max_seq, compute=compute)
        s.set_launch_mode(mode)
        return s

    def expect(self, tokens):
        return plain.forward(self.plain_cfg, self.w, tokens)

    def tokens(self, n, seed=0):
        return np.random.default_rng([7, seed]).integers(0, self.cfg["vocab"], n).astype(np.int32)


def error(got, want):
    """per position: rms difference over the vocabulary (mean removed), relative to the logits' own spread"""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()


# fp32 against the 64-bit restatement, and bf16 products and activations against it
LIMIT = {"float32": 1e-4, "bfloat16": 6e-2}
