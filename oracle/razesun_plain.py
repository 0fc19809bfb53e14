"""Plain, slow restatement of the Razesun decoder in numpy (64-bit), one function per mechanism.

TEST INFRASTRUCTURE: the tests compare the CUDA path with it; nothing of the product imports it and it
imports nothing of the product. A whole sequence is computed at once, every mechanism token by token or
key by key where its definition is sequential. Keys and values of the latent attention are expanded per
head (nothing is folded into the queries).

Model = (config dict as in config.json, {tensor name: float array}).
"""
from __future__ import annotations

import math

import numpy as np

from rafilix_plain import load_dir, rms_norm, short_conv, sigmoid, silu, softplus, unit_vector  # noqa: F401

F = np.float64


# ------------------------------------------------------------------------------------------- small functions
def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_halves(x, pos, rot):
    """x [..., n] at one position: dimension i and i + dims/2 of the first rot['dims'] are a pair"""
    y, half = x.copy(), rot["dims"] // 2
    for i in range(half):
        a = pos * float(rot["base"]) ** (-2.0 * i / rot["dims"])
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------- latent attention
def latent_rows(h, w, p, m, eps):
    """what a layer with its own down-projection keeps per token: (normed latent [T, kv_rank], rotated key part [T, rot_dim])"""
    r = m["kv_rank"]
    z = h @ w[p + "dkv"].T
    c = rms_norm(z[:, :r], w[p + "dkv.norm"], eps)
    k = np.stack([rotate_halves(z[t, r:], t, m["rot"]) for t in range(len(z))])
    return c, k


def latent_attention(h, w, p, m, eps, rows):
    T, H, dim, rd, vdim = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = rows
    cq = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).reshape(T, H, dim + rd)
    k = (c @ w[p + "uk"].T).reshape(T, H, dim)
    v = (c @ w[p + "uv"].T).reshape(T, H, vdim)
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, vdim), dtype=F)
    for i in range(T):
        qr = rotate_halves(q[i, :, dim:], i, m["rot"])
        for hd in range(H):
            s = (k[:i + 1, hd] @ q[i, hd, :dim] + k_rot[:i + 1] @ qr[hd]) * m["scale"]
            e = np.exp(s - s.max())
            out[i, hd] = gate[i, hd] * ((e / e.sum()) @ v[:i + 1, hd])
    return out.reshape(T, H * vdim) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------- delta rule, one decay per head
def delta_scan(q, k, v, g, beta):
    """q, k [T, heads, dim], v [T, heads, vdim], g and beta [T, heads] -> o [T, heads, vdim]"""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]), dtype=F)
    o = np.zeros_like(v)
    for t in range(T):
        for hd in range(H):
            S[hd] = g[t, hd] * S[hd]
            u = beta[t, hd] * (v[t, hd] - S[hd].T @ k[t, hd])
            S[hd] = S[hd] + np.outer(k[t, hd], u)
            o[t, hd] = S[hd].T @ q[t, hd]
    return o


def delta(h, w, p, m, eps):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(T, G, dim)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(T, G, dim)
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(T, H, vdim)
    q = np.repeat(unit_vector(q) * dim ** -0.5, H // G, axis=1)
    k = np.repeat(unit_vector(k), H // G, axis=1)
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms_norm(delta_scan(q, k, v, g, beta), w[p + "norm"], eps)
    o = o * silu(h @ w[p + "g"].T).reshape(T, H, vdim)
    return o.reshape(T, H * vdim) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------- real-gated linear recurrence
def plain_conv(x, taps, bias):
    T, n = x.shape[0], taps.shape[1]
    y = np.tile(np.asarray(bias, dtype=F), (T, 1))
    for t in range(T):
        for j in range(n):
            s = t - (n - 1 - j)
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def block_linear(u, mats, bias):
    """u [T, width], mats [blocks, n, n], bias [blocks, n]"""
    B, n = bias.shape
    return np.concatenate([u[:, b * n:(b + 1) * n] @ mats[b].T + bias[b] for b in range(B)], axis=1)


def rglru_scan(u, r, i, lam):
    S, out = np.zeros(u.shape[1], dtype=F), np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out


def rglru(h, w, p, m, eps):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = plain_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = sigmoid(block_linear(u, w[p + "ra"], w[p + "ra.b"]))
    i = sigmoid(block_linear(u, w[p + "ri"], w[p + "ri.b"]))
    return (rglru_scan(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------- feed-forward, model
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, tokens, last=None):
    """-> (logits [T, vocab], residual stream after every layer [layers, T, width]); last: the logits of so many last tokens"""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = rms_norm(w["embed"][np.asarray(tokens)].astype(F), w["embed.norm"], eps)
    after, kept = [], {}
    for i, layer in enumerate(cfg["layers"]):
        n, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[n + "norm1"], eps)
        if layer["type"] == "latent_attention":
            if "kv_from" in m:
                rows = kept[m["kv_from"]]
            else:
                rows = kept[i] = latent_rows(h, w, n + "mix.", m, eps)
            y = latent_attention(h, w, n + "mix.", m, eps, rows)
        else:
            y = {"delta": delta, "rglru": rglru}[layer["type"]](h, w, n + "mix.", m, eps)
        if layer.get("mlp"):
            y = y + dense(rms_norm(x, w[n + "norm2"], eps), w, n + "mlp.")
        x = x + mult * y
        after.append(x.copy())
    x = x if last is None else x[-last:]
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"], np.stack(after)
