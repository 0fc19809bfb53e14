"""Plain, slow restatement of the Rafilix decoder in numpy (64-bit), one function per mechanism.

TEST INFRASTRUCTURE: the tests compare the CUDA path with it; nothing of the product imports it and it
imports nothing of the product. A whole sequence is computed at once, every mechanism token by token or
key by key where its definition is sequential.

Model = (config dict as in config.json, {tensor name: float array}).
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np

F = np.float64


# ------------------------------------------------------------------------------------------- files
def bf16_to_float(bits: np.ndarray) -> np.ndarray:
    return (bits.astype(np.uint32) << 16).view(np.float32).astype(F)


def float_to_bf16_bits(x: np.ndarray) -> np.ndarray:
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def load_dir(path: str):
    """(config, weights) of a model folder with one model.safetensors"""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    w = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        raw = data[a:b]
        if t["dtype"] == "BF16":
            v = bf16_to_float(np.frombuffer(raw, dtype=np.uint16))
        elif t["dtype"] == "I32":
            v = np.frombuffer(raw, dtype=np.int32)
        else:
            raise ValueError(t["dtype"])
        w[name] = v.reshape(t["shape"])
    return cfg, w


# ------------------------------------------------------------------------------------------- small functions
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=F)))


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, dtype=F))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def unit_vector(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ------------------------------------------------------------------------------------------- rotary positions
def rotary_frequencies(rot):
    """one frequency per rotated pair, with the wavelength-dependent scaling if the config has one"""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        if sc:
            wl = 2.0 * math.pi / f
            if wl < sc["original"] / sc["high"]:
                pass
            elif wl > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wl - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.array(out, dtype=F)


def rotate(x, pos, rot):
    """x [heads, dim] at one position: neighbours (2i, 2i+1) of the first rot['dims'] are a pair"""
    y = x.copy()
    for i, f in enumerate(rotary_frequencies(rot)):
        c, s = math.cos(pos * f), math.sin(pos * f)
        u, v = x[:, 2 * i].copy(), x[:, 2 * i + 1].copy()
        y[:, 2 * i] = u * c - v * s
        y[:, 2 * i + 1] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------- mixers
def visible_keys(i, mask):
    """keys position i may see: its own chunk up to itself"""
    first = (i // mask["size"]) * mask["size"] if mask else 0
    return range(first, i + 1)


def attention(h, w, p, m, eps):
    """h [T, width] -> [T, width]; p = tensor prefix, m = the layer's 'mixer' entry"""
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim)
    k = (h @ w[p + "k"].T).reshape(T, G, dim)
    v = (h @ w[p + "v"].T).reshape(T, G, vdim)
    q = rms_norm(q, w[p + "q.norm"], eps)
    k = rms_norm(k, w[p + "k.norm"], eps)
    q = np.stack([rotate(q[t], t, m["rot"]) for t in range(T)])
    k = np.stack([rotate(k[t], t, m["rot"]) for t in range(T)])
    out = np.zeros((T, H, vdim), dtype=F)
    for i in range(T):
        keys = visible_keys(i, m.get("mask"))
        sl = slice(keys.start, keys.stop)
        for hd in range(H):
            g = hd // (H // G)
            s = k[sl, g] @ q[i, hd] * m["scale"]
            e = np.exp(s - s.max())
            out[i, hd] = (e / e.sum()) @ v[sl, g]
    return out.reshape(T, H * vdim) @ w[p + "o"].T


def short_conv(x, taps):
    """x [T, channels], taps [channels, n]: causal, the last column weighs the current token; then silu"""
    T, n = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1 - j)
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return silu(y)


def channel_delta_scan(q, k, v, g, beta, state=None):
    """q, k [T, heads, dim], v [T, heads, vdim], g [T, heads, dim], beta [T, heads] -> o [T, heads, vdim]"""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]), dtype=F) if state is None else state
    o = np.zeros_like(v)
    for t in range(T):
        for hd in range(H):
            S[hd] = g[t, hd][:, None] * S[hd]
            u = beta[t, hd] * (v[t, hd] - S[hd].T @ k[t, hd])
            S[hd] = S[hd] + np.outer(k[t, hd], u)
            o[t, hd] = S[hd].T @ q[t, hd]
    return o


def channel_delta(h, w, p, m, eps):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, G, dim)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, G, dim)
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, H, vdim)
    q = unit_vector(q) * dim ** -0.5
    k = unit_vector(k)
    rep = H // G
    q, k = np.repeat(q, rep, axis=1), np.repeat(k, rep, axis=1)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(T, H, dim))
    o = channel_delta_scan(q, k, v, g, beta)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, vdim)
    o = rms_norm(o, w[p + "norm"], eps) * gate
    return o.reshape(T, H * vdim) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------- feed-forward
def route(h, w, p, r):
    """-> (chosen indices [T, top], weights [T, top])"""
    z = h @ w[p + "router"].T
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    idx = np.argsort(-(s + w[p + "correction"]), axis=-1, kind="stable")[:, :r["top"]]
    return idx, np.take_along_axis(s, idx, axis=-1)


def expert(h, w, p, e):
    a = np.maximum(h @ w[f"{p}e{e}.up"].T, 0.0)
    return (a * a) @ w[f"{p}e{e}.down"].T


def moe(h, w, p, mlp):
    r = mlp["router"]
    idx, wt = route(h, w, p, r)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(idx[t], wt[t]):
            out[t] += c * (h[t] if e >= r["experts"] else expert(h[t:t + 1], w, p, e)[0])
    return out


# ------------------------------------------------------------------------------------------- model
MIXERS = {"attention": attention, "channel_delta": channel_delta}


def forward(cfg, w, tokens):
    """-> (logits [T, vocab], residual stream after every layer [layers, T, width])"""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)].astype(F)
    after = []
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        y = MIXERS[layer["type"]](rms_norm(x, w[n + "norm1"], eps), w, n + "mix.", layer["mixer"], eps)
        x = x + rms_norm(y, w[n + "norm1b"], eps)
        if layer.get("mlp"):
            y = moe(rms_norm(x, w[n + "norm2"], eps), w, n + "mlp.", layer["mlp"])
            x = x + rms_norm(y, w[n + "norm2b"], eps)
        after.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T, np.stack(after)
