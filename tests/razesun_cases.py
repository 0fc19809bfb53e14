"""Small configurations of the Razesun family for the tests, and the model folders made of them."""
import numpy as np

import razesun_plain as plain
import synth
from rafilix_cases import error  # noqa: F401
from synth import delta_layer, dense_mlp, latent_layer, razesun_config, rglru_layer

# One mechanism per model: a single layer without a feed-forward.
LATENT = {
    # name: (width, layer, weight of the query latent's norm: large values make nearly every query depend on few keys)
    "plain": (64, latent_layer(4, 32, 16, 32, 64, 48), 3.0),
    "one_head": (48, latent_layer(1, 24, 8, 40, 40, 24), 4.0),
    "wide_rank": (64, latent_layer(3, 32, 32, 16, 320, 40, scale=0.2), 2.0),
    "widest_rank": (64, latent_layer(2, 48, 64, 64, 512, 64), 3.0),
    "very_wide_rank": (48, latent_layer(2, 16, 16, 24, 712, 32), 2.0),
    "wide_rotation": (72, latent_layer(5, 16, 80, 24, 96, 56, base=500.0), 3.0),
    "many_heads": (64, latent_layer(20, 16, 8, 16, 48, 32), 3.0),
    "parts_of_heads": (40, latent_layer(130, 8, 8, 8, 32, 24), 3.0),
    "unaligned": (52, latent_layer(3, 18, 6, 10, 44, 30), 3.0),
    "narrow": (40, latent_layer(2, 6, 2, 3, 12, 10, base=50.0), 3.0),
    "wide_heads": (64, latent_layer(2, 160, 32, 144, 128, 72), 2.0),
}
DELTA = {
    "plain": (64, delta_layer(4, 4, 32, 32)),
    "shared_qk": (64, delta_layer(6, 2, 32, 48, conv=3)),
    "one_group": (48, delta_layer(4, 1, 64, 16, conv=2)),
    "no_conv": (48, delta_layer(3, 3, 24, 40, conv=1)),
    "long_conv": (64, delta_layer(2, 1, 96, 64, conv=7)),
    "wide": (64, delta_layer(2, 2, 128, 128)),
    "very_wide": (64, delta_layer(2, 1, 200, 160)),
    "unaligned": (52, delta_layer(3, 1, 18, 10, conv=4)),
    "one_head": (40, delta_layer(1, 1, 16, 24, conv=5)),
}
RGLRU = {
    "plain": (64, rglru_layer(64, 4)),
    "one_part": (48, rglru_layer(72, 1, conv=3)),
    "many_parts": (64, rglru_layer(160, 20, conv=2)),
    "parts_of_one": (40, rglru_layer(24, 24, conv=5)),
    "no_conv": (48, rglru_layer(96, 3, conv=1)),
    "long_conv": (64, rglru_layer(128, 2, conv=9)),
    "unaligned": (52, rglru_layer(90, 6, conv=4)),
    "wide": (72, rglru_layer(768, 3, conv=4)),
}
DENSE = {
    "plain": (64, dense_mlp(96)),
    "wide": (48, dense_mlp(600)),
    "unaligned": (52, dense_mlp(30)),
}


def mixed_config(width=72, vocab=211):
    """every mechanism, rows of another layer, layers without a feed-forward, sizes that differ from each other"""
    return razesun_config(width, vocab, [
        rglru_layer(96, 4, conv=3, mlp=dense_mlp(104)),
        latent_layer(6, 32, 16, 24, 80, 56, base=3000.0, mlp=dense_mlp(72)),
        delta_layer(4, 2, 40, 24, conv=4, mlp=None),
        latent_layer(9, 24, 16, 40, 80, 40, base=3000.0, scale=0.3, kv_from=1, mlp=None),
        latent_layer(3, 16, 24, 48, 136, 64, base=20000.0, mlp=dense_mlp(136)),
        latent_layer(6, 40, 16, 16, 80, 48, base=3000.0, kv_from=1, mlp=dense_mlp(56)),
        delta_layer(3, 3, 64, 64, conv=2, mlp=dense_mlp(88)),
        latent_layer(2, 8, 24, 32, 136, 32, base=20000.0, kv_from=4, mlp=dense_mlp(40)),
        rglru_layer(60, 5, conv=5, mlp=dense_mlp(64)),
    ], eps=2e-5, residual_mult=0.6, logit_scale=1.3)


class Case:
    """a model folder with its library model and its plain weights"""

    def __init__(self, path, cfg, seed=1, sharp=1.0, edit=None):
        self.dir, self.cfg = str(path), cfg
        synth.write_razesun(self.dir, cfg, seed=seed, sharp=sharp, edit=edit)
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

    def expect(self, tokens, last=None):
        """last: logits of that many positions at the end only"""
        return plain.forward(self.plain_cfg, self.w, tokens, last)

    def tokens(self, n, seed=0):
        return np.random.default_rng([11, seed]).integers(0, self.cfg["vocab"], n).astype(np.int32)




def plant_key(path, width=48, key=11, ask=12, other=13):
    """-> (case, key, ask, other): two latent-attention layers, the second on the first one's rows, in which the query of
    token `ask` prefers the key of token `key` to every other one by far, wherever they stand, and nobody else asks for it"""
    def edit(name, x):
        if name == "embed":
            x[:, :2] = 0.0
            x[key], x[ask] = 0.0, 0.0
            x[key, 0], x[ask, 1] = 3.0, 3.0
            return x
        if name.endswith(("dkv", "dq")):  # the first latent reads feature 0 (keys) or 1 (queries), the others neither
            f = 0 if name.endswith("dkv") else 1
            x[:, :2] = 0.0
            x[1:, :] *= 0.3
            x[0, :], x[0, f] = 0.0, 2.0
            return x
        if name.endswith(("uq", "uk")):  # unrotated score: the product of the two first latents
            x *= 0.03 if name.endswith("uq") else 0.3
            x[:, 0] = 0.8
            return x
        if name.endswith("mix.o"):  # the two features stay as the embedding left them
            x[:2] = 0.0
            return x
        if name.endswith("mix.uv"):
            return x * 2.0
    layers = [latent_layer(2, 16, 8, 32, 40, 24, scale=0.5), latent_layer(1, 24, 8, 24, 40, 32, scale=0.4, kv_from=0)]
    return Case(path, razesun_config(width, 64, layers, residual_mult=1.0), edit=edit), key, ask, other


# fp32 against the 64-bit restatement, and bf16 products and activations against it
LIMIT = {"float32": 1e-5, "bfloat16": 3e-2}
