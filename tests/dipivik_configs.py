"""Tiny Dipivik configurations of the tests (config.json dictionaries), their random weights and prompts.

d1: sizes no kernel is tuned for (an odd vocabulary, a width that is no multiple of 8): retention with part of a head turned and
    values narrower than keys, a latent of 20 with a window of 19, experts top 2 of 5 with a shared one, layers without a
    feed-forward.
d2: sizes the tensor-core kernels take (heads of 64, a width of 128), a window of 40 that no page divides, experts top 3 of 8, one
    layer of them without a shared expert.
d3: what another model makes equal, 1 or absent: one head, a window of one position, no rotation, one expert, every expert chosen, no
    table of token pairs, no cap on the logits, a decay of one.
d4: large heads: keys of 130 and of 40 in retention (filled up to the next power of two), a latent of 160, values of 72, top 4 of 20
    experts, a table of pairs with one bucket.
"""

from __future__ import annotations

import json
import os
import random

import torch


def mlp(ff):
    """None; a width (dense); (experts, top, ff, shared ff or None)."""
    if ff is None:
        return None
    if isinstance(ff, tuple):
        d = {"kind": "moe", "router": {"experts": ff[0], "top": ff[1]}, "expert": {"ff": ff[2]}}
        if ff[3]:
            d["shared"] = {"ff": ff[3]}
        return d
    return {"kind": "dense", "ff": ff}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, window, ff=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if base:
        m["rot"] = {"base": base, "dims": rot_dim}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp(ff)}


def retention(heads, dim, vdim, rot, decay=None, ff=None):
    """`rot` = (base, dims) or None; the decays run from 0.9 to close to one."""
    decay = decay or [1.0 - 0.1 * 0.4 ** h for h in range(heads)]
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return {"type": "retention", "mixer": m, "mlp": mlp(ff)}


def model(vocab, width, eps, layers, bigram=None, cap=None):
    cfg = {"architecture": "Dipivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}
    if bigram:
        cfg["embedding"] = {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


D1 = model(97, 44, 1e-4, [retention(3, 8, 6, (500.0, 6), ff=(5, 2, 24, 20)), latent(4, 12, 6, 10, 20, 14, 0.3, 700.0, 19, ff=52),
                          retention(2, 10, 12, (90.0, 10), ff=None), latent(3, 8, 4, 6, 9, 11, 0.4, 50.0, 33, ff=(5, 2, 24, 20)),
                          latent(2, 6, 2, 14, 12, 7, 0.5, 50.0, 27, ff=None)], bigram=(61, 5, 3), cap=9.0)
D2 = model(320, 128, 1e-6, [latent(2, 64, 32, 64, 64, 64, 0.11, 10000.0, 40, ff=(8, 3, 64, 128)),
                            retention(4, 64, 64, (100000.0, 64), ff=256), latent(4, 32, 16, 64, 128, 32, 0.15, 10000.0, 100, ff=192),
                            retention(2, 32, 64, (10000.0, 32), ff=(8, 3, 64, None))], bigram=(257, 1001, 77), cap=20.0)
D3 = model(130, 64, 1e-5, [latent(1, 16, 8, 16, 16, 16, 0.25, None, None, ff=(1, 1, 24, 16)), retention(1, 8, 8, None, decay=[1.0], ff=40),
                           latent(2, 8, 2, 8, 8, 8, 0.3, 30.0, 1, ff=(3, 3, 16, None))])
D4 = model(211, 96, 3e-6, [retention(2, 130, 20, (3000.0, 128), ff=(20, 4, 40, 72)), latent(3, 40, 10, 72, 160, 48, 0.12, 3000.0, 64, ff=88),
                           retention(3, 40, 72, (3000.0, 4), ff=None)], bigram=(1, 7, 7), cap=30.0)
CONFIGS = {"d1": D1, "d2": D2, "d3": D3, "d4": D4}
SEEDS = {"d1": 51, "d2": 52, "d3": 53, "d4": 54}


def tensor_shapes(cfg: dict) -> dict[str, tuple]:
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        out["bigram"] = (b["buckets"] + 1, W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        out[f"l{i}.norm1"] = (W,)
        H = m["heads"]
        if layer["type"] == "retention":
            out[p + "q"] = out[p + "k"] = (H * m["dim"], W)
            out[p + "v"] = out[p + "g"] = (H * m["vdim"], W)
        else:
            Q, L, R = m["q_rank"], m["kv_rank"], m["rot_dim"]
            out[p + "dq"], out[p + "dq.norm"], out[p + "uq"] = (Q, W), (Q,), (H * (m["dim"] + R), Q)
            out[p + "dkv"], out[p + "dkv.norm"] = (L + R, W), (L,)
            out[p + "uk"], out[p + "uv"], out[p + "g"] = (H * m["dim"], L), (H * m["vdim"], L), (H, W)
        out[p + "o"] = (W, H * m["vdim"])
        ff, q = layer["mlp"], f"l{i}.mlp."
        if ff is None:
            continue

        def gated(pre, n, biases):
            out[pre + "gate"] = out[pre + "up"] = (n, W)
            out[pre + "down"] = (W, n)
            if biases:
                out[pre + "gate.b"] = out[pre + "up.b"] = (n,)
                out[pre + "down.b"] = (W,)

        if ff["kind"] == "dense":
            gated(q, ff["ff"], True)
        else:
            out[q + "router"] = (ff["router"]["experts"], W)
            for e in range(ff["router"]["experts"]):
                gated(f"{q}e{e}.", ff["expert"]["ff"], False)
            if ff.get("shared"):
                gated(q + "shared.", ff["shared"]["ff"], False)
    return out


def random_weights(cfg: dict, seed: int, bf16_exact: bool = True) -> dict[str, torch.Tensor]:
    """32-bit random weights by stored name; with `bf16_exact` every value is a bfloat16 value, so that the engine in
    either precision and the plain model read the same numbers."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for key, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = key.rsplit(".", 1)[-1]
        if key in ("embed", "bigram"):
            t = t * 0.8
        elif last in ("norm", "norm1"):
            t = 1.0 + 0.2 * t
        elif last == "b":
            t = 0.4 * t
        elif last == "router":
            t = t * (1.5 * shape[1] ** -0.5)
        else:
            t = t * (shape[1] ** -0.5)
        out[key] = t.to(torch.bfloat16).float() if bf16_exact else t
    return out


def weights(name: str, bf16_exact: bool = True) -> dict[str, torch.Tensor]:
    return random_weights(CONFIGS[name], SEEDS[name], bf16_exact)


def tokens(name: str, n: int, seed: int = 0) -> list[int]:
    g = torch.Generator().manual_seed(seed * 7919 + n)
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist()


def write_folder(folder: str, name: str) -> str:
    """config.json and model.safetensors (bfloat16, as the design stores them) of the tiny model `name`."""
    from tandemllm_b200.weights.safetensors_io import write_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(CONFIGS[name], f)
    write_file(os.path.join(folder, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in weights(name).items()})
    return folder


def random_config(seed: int) -> dict:
    """A model drawn at random: layer order, small sizes and large (a normed head of one or two entries is little more than signs,
    which rounding can turn, so values begin at 6), windows, rotations, decays, feed-forwards, the table of pairs, the cap."""
    r = random.Random(seed)
    layers = []
    for _ in range(r.randint(2, 5)):
        ff = r.choice([None, 16, 40, 64, (r.choice([1, 2, 3, 6]), 1, 16, r.choice([None, 24])), (4, r.choice([2, 4]), 24, 40), (18, 3, 8, 16)])
        if r.random() < 0.5:
            heads, dim = r.choice([1, 2, 3, 6]), r.choice([8, 10, 16, 24, 64])
            dims = r.choice([d for d in (2, 4, 8, 10, 16, 24, 64) if d <= dim])
            layers.append(retention(heads, dim, r.choice([6, 8, 16, 40, 64]), r.choice([None, (r.choice([100.0, 1e6]), dims)]),
                                    decay=[r.choice([0.5, 0.9, 0.97, 0.995, 1.0]) for _ in range(heads)], ff=ff))
        else:
            layers.append(latent(r.choice([1, 2, 4, 5]), r.choice([8, 10, 16, 64]), r.choice([2, 6, 16, 32]), r.choice([4, 8, 16, 48, 64]),
                                 r.choice([8, 12, 24, 64]), r.choice([8, 10, 24, 64]), r.uniform(0.1, 0.4), r.choice([None, 100.0, 10000.0]),
                                 r.choice([None, 1, 9, 16, 33, 64]), ff=ff))
    return model(r.choice([50, 131, 256]), r.choice([24, 36, 40, 50, 64, 72, 100]), r.choice([1e-6, 1e-4]), layers,
                 bigram=r.choice([None, (1, 3, 5), (37, 11, 4), (400, 90001, 7)]), cap=r.choice([None, 5.0, 25.0]))
