"""The plain Dipivik: every mechanism as a slow function of its own, in 64-bit numpy, over one whole sequence.

It shares nothing with the engine: it reads a configuration dictionary (the keys of config.json) and a dictionary of
arrays by tensor name, and runs the sequence position by position where a mechanism is recurrent and as dense
[T, T] tables where it is attention. The tests hold the engine's parts and whole models to it.

Notation: n is a normed row, W is stored [out, in] and applied as W n, T tokens at positions 0..T-1.
"""

from __future__ import annotations

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x * x * x)))


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def plain_norm(x, w, eps):
    return unit_rms(x, eps) * w


# ---- the embedding ----

def bigram_rows(tokens, b):
    """[T]: the row of the table of pairs every token reads; the first token has no token before it and reads the last row."""
    buckets, mp, mc = int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])
    return np.array([buckets if t == 0 else (int(tokens[t - 1]) * mp + int(tokens[t]) * mc) % buckets for t in range(len(tokens))],
                    dtype=np.int64)


def embedding(tokens, config, w):
    x = w["embed"][np.asarray(tokens)]
    b = (config.get("embedding") or {}).get("bigram")
    return x if b is None else x + w["bigram"][bigram_rows(tokens, b)]


# ---- rotation ----

def rotate_halves(x, positions, base, dims):
    """x [T, heads, D]: entries i and i + dims / 2 (i < dims / 2) are a pair that turns by p base^(-2i / dims); the rest pass."""
    if dims == 0:
        return x
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    a = positions[:, None, None].astype(np.float64) * f
    c, s = np.cos(a), np.sin(a)
    out = x.copy()
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    out[..., :dims // 2] = u * c - v * s
    out[..., dims // 2:dims] = v * c + u * s
    return out


# ---- latent attention ----

def window_mask(T, size):
    """[T, T]: row i sees j with 0 <= i - j < size (None: every j <= i)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size is not None else True)


def latent_queries(n, m, w, pre, eps):
    """(unrotated [T, H, dim], rotated [T, H, rot_dim])."""
    T, H, D, R = n.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"])
    q = (plain_norm(n @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).reshape(T, H, D + R)
    rot = m.get("rot")
    qr = rotate_halves(q[..., D:], np.arange(T), float(rot["base"]), int(rot["dims"])) if rot else q[..., D:]
    return q[..., :D], qr


def latent_keys(n, m, w, pre, eps):
    """(the latent [T, kv_rank], the shared rotated key part [T, rot_dim])."""
    L, T = int(m["kv_rank"]), n.shape[0]
    kv = n @ w[pre + "dkv"].T
    rot = m.get("rot")
    kr = kv[:, None, L:]
    if rot:
        kr = rotate_halves(kr, np.arange(T), float(rot["base"]), int(rot["dims"]))
    return plain_norm(kv[:, :L], w[pre + "dkv.norm"], eps), kr[:, 0]


def mixer_latent_attention(n, m, w, pre, eps):
    T, H, D, VD = n.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    qu, qr = latent_queries(n, m, w, pre, eps)
    c, kr = latent_keys(n, m, w, pre, eps)
    ku = (c @ w[pre + "uk"].T).reshape(T, H, D)
    v = (c @ w[pre + "uv"].T).reshape(T, H, VD)
    seen = window_mask(T, int(m["mask"]["size"]) if m.get("mask") else None)
    gate = sigmoid(n @ w[pre + "g"].T)                      # one number a head
    out = np.zeros((T, H, VD))
    for h in range(H):
        s = np.where(seen, (qu[:, h] @ ku[:, h].T + qr[:, h] @ kr.T) * float(m["scale"]), -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = gate[:, h:h + 1] * ((e / e.sum(-1, keepdims=True)) @ v[:, h])
    return out.reshape(T, H * VD) @ w[pre + "o"].T


# ---- retention ----

def retention_inputs(n, m, w, pre):
    """(q, k [T, H, dim], turned, k with its factor; v [T, H, vdim])."""
    T, H, D, VD = n.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k = ((n @ w[pre + x].T).reshape(T, H, D) for x in ("q", "k"))
    rot = m.get("rot")
    if rot:
        q, k = (rotate_halves(x, np.arange(T), float(rot["base"]), int(rot["dims"])) for x in (q, k))
    return q, k * D ** -0.5, (n @ w[pre + "v"].T).reshape(T, H, VD)


def retention_scan(q, k, v, decay, state=None):
    """Per head: S <- decay S + k v^T, o = S^T q. Returns (o [T, H, vdim], S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1])) if state is None else state.copy()
    c = np.asarray(decay, dtype=np.float64)[:, None, None]
    o = np.zeros_like(v)
    for t in range(T):
        S = c * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def mixer_retention(n, m, w, pre, eps, return_state=False):
    T = n.shape[0]
    o, S = retention_scan(*retention_inputs(n, m, w, pre), m["decay"])
    o = unit_rms(o, eps).reshape(T, -1)
    out = (o * silu(n @ w[pre + "g"].T)) @ w[pre + "o"].T
    return (out, S) if return_state else out


# ---- feed-forwards ----

def dense_gated(n, w, pre):
    g = gelu_tanh(n @ w[pre + "gate"].T + w[pre + "gate.b"])
    return (g * (n @ w[pre + "up"].T + w[pre + "up.b"])) @ w[pre + "down"].T + w[pre + "down.b"]


def expert(n, w, pre):
    return (silu(n @ w[pre + "gate"].T) * (n @ w[pre + "up"].T)) @ w[pre + "down"].T


def routed_experts(n, mlp, w, pre, scores=None):
    """The `top` experts with the largest scores, each of its row times its own score. `scores`: the router's, where its rows
    are not the experts'."""
    top = int(mlp["router"]["top"])
    s = sigmoid(n @ w[pre + "router"].T) if scores is None else scores
    out = np.zeros((n.shape[0], w[pre + "e0.down"].shape[0]))
    for t in range(n.shape[0]):
        for e in np.argsort(-s[t], kind="stable")[:top]:
            out[t] += expert(s[t, e] * n[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


def feed_forward(n, mlp, w, pre):
    if mlp["kind"] == "dense":
        return dense_gated(n, w, pre)
    out = routed_experts(n, mlp, w, pre)
    return out + expert(n, w, pre + "shared.") if mlp.get("shared") else out


# ---- the model ----

MIXERS = {"latent_attention": mixer_latent_attention, "retention": mixer_retention}


def choice_margin(z, top):
    """[T]: how far the last chosen logit is above the first one left out."""
    s = np.sort(z, axis=-1)[:, ::-1]
    return s[:, top - 1] - s[:, top] if top < z.shape[1] else np.full(len(z), np.inf)


def head(x, config, w):
    logits = plain_norm(x, w["final.norm"], float(config["norm"]["eps"])) @ w["embed"].T
    cap = config.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits


def forward(config, weights, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence; with `return_layers` also the residual stream after every layer. A list given as
    `margins` receives every routed layer's `choice_margin`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = embedding(tokens, config, w)
    layers = []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        n = plain_norm(x, w[pre + "norm1"], eps)
        y = MIXERS[layer["type"]](n, layer["mixer"], w, pre + "mix.", eps)
        if layer.get("mlp"):
            y = y + feed_forward(n, layer["mlp"], w, pre + "mlp.")
            if margins is not None and layer["mlp"]["kind"] == "moe":
                margins.append(choice_margin(n @ w[pre + "mlp.router"].T, int(layer["mlp"]["router"]["top"])))
        x = x + y
        layers.append(x.copy())
    logits = head(x, config, w)
    return (logits, np.stack(layers)) if return_layers else logits
