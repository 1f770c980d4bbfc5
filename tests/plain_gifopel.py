"""The plain Gifopel: every mechanism as a slow function of its own, in 64-bit numpy, over one whole sequence.

It shares nothing with the engine: it reads a configuration dictionary (the keys of config.json) and a dictionary of
arrays by tensor name, and runs the sequence position by position where a mechanism is recurrent and as dense
[T, T] tables where it is attention. The tests hold the engine's parts and whole models to it.

Notation: n is a normed row, W is stored [out, in] and applied as W n, T tokens at positions 0..T-1.
"""

from __future__ import annotations

import numpy as np

UNIT_EPS = 1e-6          # inside the root of a key's (and a query's) length
READ_FLOOR = 1e-6        # added to the normaliser of the exponentially gated memory


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.maximum(x, 0.0) + np.log1p(np.exp(-np.abs(x)))


def log_sigmoid(x):
    return -softplus(-x)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def plain_norm(x, w, eps):
    return unit_rms(x, eps) * w


def unit_vector(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + UNIT_EPS)


def softmax(z):
    e = np.exp(z - z.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


# ---- the convolution over time ----

def causal_conv(u, taps):
    """u [T, C], taps [C, K]: out[t] = sum_j taps[:, j] u[t - (K - 1) + j], zeros before the first token."""
    T, K = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, u.shape[1])), u])
    return sum(taps[:, j] * padded[j:j + T] for j in range(K))


# ---- the gated delta rule ----

def delta_inputs(n, m, w, pre):
    """(q, k [T, heads, dim] unit vectors, q with its factor; v [T, heads, vdim]; beta [T, heads])."""
    T = n.shape[0]
    H, G, D, VD = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (silu(causal_conv(n @ w[pre + x].T, w[pre + x + ".conv"])) for x in ("q", "k", "v"))
    q, k = unit_vector(q.reshape(T, G, D)) * D ** -0.5, unit_vector(k.reshape(T, G, D))
    of_head = np.arange(H) // (H // G)
    return q[:, of_head], k[:, of_head], v.reshape(T, H, VD), sigmoid(n @ w[pre + "b"].T)


def channel_decay(n, m, w, pre):
    """[T, heads, dim]: one decay a head and key channel, its logits through a narrow product."""
    T, H, D = n.shape[0], int(m["heads"]), int(m["dim"])
    z = (n @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]
    return np.exp(-np.exp(w[pre + "A_log"])[None, :, None] * softplus(z).reshape(T, H, D))


def head_decay(n, m, w, pre):
    """[T, heads, 1]: one decay a head."""
    z = n @ w[pre + "a"].T + w[pre + "dt_bias"]
    return np.exp(-np.exp(w[pre + "A_log"]) * softplus(z))[:, :, None]


def delta_scan(q, k, v, beta, g, state=None):
    """Per head: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q. Returns (o [T, heads, vdim], S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[-1])) if state is None else state.copy()
    o = np.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def mixer_channel_delta(n, m, w, pre, eps, return_state=False):
    T = n.shape[0]
    o, S = delta_scan(*delta_inputs(n, m, w, pre), channel_decay(n, m, w, pre))
    o = plain_norm(o, w[pre + "norm"], eps).reshape(T, -1)
    out = (o * sigmoid((n @ w[pre + "g1"].T) @ w[pre + "g2"].T)) @ w[pre + "o"].T
    return (out, S) if return_state else out


def mixer_head_delta(n, m, w, pre, eps, return_state=False):
    """The right one of two mixers side by side."""
    T = n.shape[0]
    o, S = delta_scan(*delta_inputs(n, m, w, pre), head_decay(n, m, w, pre))
    o = plain_norm(o, w[pre + "norm"], eps).reshape(T, -1)
    out = (o * silu(n @ w[pre + "g"].T)) @ w[pre + "o"].T
    return (out, S) if return_state else out


# ---- the exponentially gated matrix memory ----

def memory_gates(n, m, w, pre):
    """Log input and log forget gates [T, heads]."""
    cap = float(m["gate_cap"])
    i = cap * np.tanh((n @ w[pre + "i"].T + w[pre + "i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((n @ w[pre + "f"].T + w[pre + "f.b"]) / cap))
    return i, f


def mixer_mlstm(n, m, w, pre, eps, return_state=False):
    T = n.shape[0]
    H, D, VD = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (n @ w[pre + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (n @ w[pre + "k"].T).reshape(T, H, D)
    v = (n @ w[pre + "v"].T).reshape(T, H, VD)
    i, f = memory_gates(n, m, w, pre)
    S, nn, mx = np.zeros((H, D, VD)), np.zeros((H, D)), np.zeros(H)
    o = np.zeros((T, H, VD))
    for t in range(T):
        new = np.maximum(f[t] + mx, i[t])
        keep, add = np.exp(f[t] + mx - new), np.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nn = keep[:, None] * nn + add[:, None] * k[t]
        mx = new
        den = np.maximum(np.abs((nn * q[t]).sum(-1)), np.exp(-mx)) + READ_FLOOR
        o[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    o = unit_rms(o, eps).reshape(T, H * VD) * w[pre + "norm"]
    out = (o * sigmoid(n @ w[pre + "g"].T)) @ w[pre + "o"].T
    return (out, (S, nn, mx)) if return_state else out


# ---- chunked attention ----

def rotate_neighbours(x, positions, base, dims):
    """x [T, heads, D]: entries 2i and 2i + 1 (i < dims / 2) are a pair that turns by p base^(-2i / dims); the rest pass."""
    if dims == 0:
        return x
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    a = positions[:, None, None].astype(np.float64) * f
    c, s = np.cos(a), np.sin(a)
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def chunk_mask(T, size):
    """[T, T]: row i sees j <= i of its own chunk of `size` positions (None: every j <= i)."""
    i = np.arange(T)
    seen = i[None, :] <= i[:, None]
    return seen if size is None else seen & (i[None, :] // size == i[:, None] // size)


def mixer_chunked_attention(n, m, w, pre, eps):
    """The left one of two mixers side by side."""
    T = n.shape[0]
    H, G, D, VD = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = np.arange(T)
    q = plain_norm((n @ w[pre + "q"].T).reshape(T, H, D), w[pre + "q.norm"], eps)
    k = plain_norm((n @ w[pre + "k"].T).reshape(T, G, D), w[pre + "k.norm"], eps)
    v = (n @ w[pre + "v"].T).reshape(T, G, VD)
    rot = m.get("rot")
    if rot:
        q = rotate_neighbours(q, pos, float(rot["base"]), int(rot["dims"]))
        k = rotate_neighbours(k, pos, float(rot["base"]), int(rot["dims"]))
    seen = chunk_mask(T, int(m["mask"]["size"]) if m.get("mask") else None)
    gate = sigmoid(n @ w[pre + "g"].T)
    out = np.zeros((T, H, VD))
    for h in range(H):
        s = np.where(seen, (q[:, h] @ k[:, h // (H // G)].T) * float(m["scale"]), -np.inf)
        sink = float(w[pre + "sink"][h])
        top = np.maximum(s.max(-1, keepdims=True), sink)
        e = np.exp(s - top)
        p = e / (e.sum(-1, keepdims=True) + np.exp(sink - top))      # the sink counts once, has no key and no value
        out[:, h] = (p @ v[:, h // (H // G)]) * gate[:, h:h + 1]
    return out.reshape(T, H * VD) @ w[pre + "o"].T


def mixer_parallel(n, m, w, pre, eps):
    left = mixer_chunked_attention(n, m["left"], w, pre + "left.", eps)
    right = mixer_head_delta(n, m["right"], w, pre + "right.", eps)
    return 0.5 * (plain_norm(left, w[pre + "left.out"], eps) + plain_norm(right, w[pre + "right.out"], eps))


# ---- feed-forwards ----

def dense_gated(n, w, pre):
    return (silu(n @ w[pre + "gate"].T) * (n @ w[pre + "up"].T)) @ w[pre + "down"].T


def squared_relu_expert(n, w, pre):
    return (np.maximum(n @ w[pre + "up"].T, 0.0) ** 2) @ w[pre + "down"].T


def router_logits(n, w, pre):
    return n @ w[pre + "router"].T + w[pre + "router.b"]


def routed_experts(n, mlp, w, pre, logits=None):
    """The `top` experts with the largest logits, weighed by the softmax over those logits only. `logits`: the router's, where
    its rows are not the experts'."""
    top = int(mlp["router"]["top"])
    z = router_logits(n, w, pre) if logits is None else logits
    out = np.zeros((n.shape[0], w[pre + "e0.down"].shape[0]))
    for t in range(n.shape[0]):
        chosen = np.argsort(-z[t], kind="stable")[:top]
        for p, e in zip(softmax(z[t, chosen]), chosen):
            out[t] += p * squared_relu_expert(n[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


def feed_forward(n, mlp, w, pre):
    return dense_gated(n, w, pre) if mlp["kind"] == "dense" else routed_experts(n, mlp, w, pre)


# ---- the model ----

MIXERS = {"channel_delta": mixer_channel_delta, "mlstm": mixer_mlstm, "parallel": mixer_parallel}


def choice_margin(z, top):
    """[T]: how far the last chosen logit is above the first one left out."""
    s = np.sort(z, axis=-1)[:, ::-1]
    return s[:, top - 1] - s[:, top] if top < z.shape[1] else np.full(len(z), np.inf)


def forward(config, weights, tokens, return_layers=False, margins=None):
    """Logits [T, vocab] of one whole sequence; with `return_layers` also the residual stream after every layer. A list given as
    `margins` receives every routed layer's `choice_margin`."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)]
    layers = []
    for i, layer in enumerate(config["layers"]):
        owner = i
        while config["layers"][owner].get("weights_of") is not None:
            owner = int(config["layers"][owner]["weights_of"])
        pre = f"l{owner}."
        y = MIXERS[layer["type"]](plain_norm(x, w[pre + "norm1"], eps), layer["mixer"], w, pre + "mix.", eps)
        if layer.get("mlp"):
            n = plain_norm(x, w[pre + "norm2"], eps)
            y = y + feed_forward(n, layer["mlp"], w, pre + "mlp.")
            if margins is not None and layer["mlp"]["kind"] == "moe":
                margins.append(choice_margin(router_logits(n, w, pre + "mlp."), int(layer["mlp"]["router"]["top"])))
        x = x + y
        layers.append(x.copy())
    logits = plain_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, np.stack(layers)) if return_layers else logits
