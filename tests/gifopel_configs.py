"""Tiny Gifopel configurations of the tests (config.json dictionaries), their random weights and prompts.

f1: sizes no kernel is tuned for (an odd vocabulary, a width that is no multiple of 8): a parallel layer with values narrower than
    its keys, half a head rotated and chunks of 24, routed experts top 2 of 5, a channel delta with three key heads under six heads
    and a dense feed-forward, a matrix memory without a feed-forward, and the parallel layer's tensors run a second time.
f2: sizes the tensor-core kernels take (heads of 64, a width of 128), chunks of 40 that no page divides, experts top 3 of 8, a matrix
    memory and a channel delta of 64 x 64, the memory's tensors run again, dense feed-forward last.
f3: what another model makes equal, 1 or absent: one head, a convolution of one tap, no rotation, no chunks, one expert, keys of
    size 1 in the memory, a layer that borrows the tensors of a layer that borrows.
f4: large heads: keys of 128 over values of 64 with all entries rotated, chunks of 64, a delta rule of 40 keys and 72 values, a memory
    of 130 keys (filled up to the next power of two), five taps, top 4 of 20 experts.
The inner sizes of the narrow products are no keys of the configuration: the stored tensors say them (RANKS).
"""

from __future__ import annotations

import copy
import json
import os
import random

import torch


def mlp(ff):
    if ff is None:
        return None
    if isinstance(ff, tuple):
        return {"kind": "moe", "router": {"experts": ff[0], "top": ff[1]}, "expert": {"ff": ff[2]}}
    return {"kind": "dense", "ff": ff}


def delta_sizes(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def left_sizes(heads, kv, dim, vdim, scale, rot, chunk):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if chunk:
        m["mask"] = {"size": chunk}
    return m


def delta(heads, kv, dim, vdim, conv, ff=None):
    return {"type": "channel_delta", "mixer": delta_sizes(heads, kv, dim, vdim, conv), "mlp": mlp(ff)}


def memory(heads, dim, vdim, cap, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp(ff)}


def parallel(left, right, ff=None):
    return {"type": "parallel", "mixer": {"left": left_sizes(*left), "right": delta_sizes(*right)}, "mlp": mlp(ff)}


def again(layers, j):
    return dict(copy.deepcopy(layers[j]), weights_of=j)


F1 = {"architecture": "Gifopel", "vocab": 97, "width": 44, "norm": {"eps": 1e-4},
      "layers": [parallel((4, 2, 12, 10, 0.3, (500.0, 6), 24), (4, 2, 6, 10, 3), ff=(5, 2, 24)),
                 delta(6, 3, 8, 6, 4, ff=52),
                 memory(3, 8, 12, 5.0, ff=None)]}
F1["layers"].append(again(F1["layers"], 0))
F2 = {"architecture": "Gifopel", "vocab": 320, "width": 128, "norm": {"eps": 1e-6},
      "layers": [memory(2, 64, 64, 15.0, ff=(8, 3, 64)),
                 parallel((8, 2, 64, 64, 0.14, (100000.0, 32), 40), (4, 4, 32, 64, 4), ff=(8, 3, 64)),
                 delta(4, 2, 64, 64, 2, ff=(8, 3, 64))]}
F2["layers"] += [again(F2["layers"], 0), delta(2, 1, 32, 32, 3, ff=256)]
F3 = {"architecture": "Gifopel", "vocab": 130, "width": 64, "norm": {"eps": 1e-5},
      "layers": [parallel((1, 1, 16, 16, 0.25, None, None), (1, 1, 8, 8, 1), ff=40),
                 memory(1, 1, 16, 2.0, ff=(1, 1, 24)),
                 delta(2, 2, 5, 8, 1, ff=(3, 3, 16))]}
F3["layers"] += [again(F3["layers"], 1), dict(copy.deepcopy(F3["layers"][1]), weights_of=3)]
F4 = {"architecture": "Gifopel", "vocab": 211, "width": 96, "norm": {"eps": 3e-6},
      "layers": [delta(3, 1, 40, 72, 5, ff=(20, 4, 40)),
                 parallel((2, 1, 128, 64, 0.09, (3000.0, 128), 64), (2, 1, 24, 40, 2), ff=None),
                 memory(2, 130, 20, 30.0, ff=(20, 4, 40)),
                 parallel((3, 3, 20, 128, 0.2, (3000.0, 20), 17), (3, 3, 33, 5, 5), ff=88)]}
CONFIGS = {"f1": F1, "f2": F2, "f3": F3, "f4": F4}
SEEDS = {"f1": 41, "f2": 42, "f3": 43, "f4": 44}
RANKS = {"f1": (5, 7), "f2": (16, 8), "f3": (1, 3), "f4": (12, 20)}       # of the decay's and the gate's narrow products


def _delta_shapes(out, p, m, W, ranks):
    H, D, VD, G, K = m["heads"], m["dim"], m["vdim"], m["kv_heads"], m["conv"]
    for x, n in (("q", G * D), ("k", G * D), ("v", H * VD)):
        out[p + x], out[p + x + ".conv"] = (n, W), (n, K)
    out[p + "b"], out[p + "A_log"], out[p + "norm"], out[p + "o"] = (H, W), (H,), (VD,), (W, H * VD)
    if ranks:
        out[p + "a1"], out[p + "a2"], out[p + "dt_bias"] = (ranks[0], W), (H * D, ranks[0]), (H * D,)
        out[p + "g1"], out[p + "g2"] = (ranks[1], W), (H * VD, ranks[1])
    else:
        out[p + "a"], out[p + "dt_bias"], out[p + "g"] = (H, W), (H,), (H * VD, W)


def tensor_shapes(cfg: dict, ranks: tuple) -> dict[str, tuple]:
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}.mix."
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "channel_delta":
            _delta_shapes(out, p, m, W, ranks)
        elif layer["type"] == "mlstm":
            H, D, VD = m["heads"], m["dim"], m["vdim"]
            out[p + "q"] = out[p + "k"] = (H * D, W)
            out[p + "v"] = out[p + "g"] = (H * VD, W)
            out[p + "o"], out[p + "norm"] = (W, H * VD), (H * VD,)
            for x in ("i", "f"):
                out[p + x], out[p + x + ".b"] = (H, W), (H,)
        else:
            a, q = m["left"], p + "left."
            out[q + "q"], out[q + "k"] = (a["heads"] * a["dim"], W), (a["kv_heads"] * a["dim"], W)
            out[q + "v"], out[q + "o"] = (a["kv_heads"] * a["vdim"], W), (W, a["heads"] * a["vdim"])
            out[q + "q.norm"] = out[q + "k.norm"] = (a["dim"],)
            out[q + "sink"], out[q + "g"] = (a["heads"],), (a["heads"], W)
            _delta_shapes(out, p + "right.", m["right"], W, None)
            out[p + "left.out"] = out[p + "right.out"] = (W,)
        ff = layer["mlp"]
        if ff is not None:
            out[f"l{i}.norm2"] = (W,)
            q = f"l{i}.mlp."
            if ff["kind"] == "dense":
                out[q + "gate"] = out[q + "up"] = (ff["ff"], W)
                out[q + "down"] = (W, ff["ff"])
            else:
                E = ff["router"]["experts"]
                out[q + "router"], out[q + "router.b"] = (E, W), (E,)
                for e in range(E):
                    out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = (ff["expert"]["ff"], W), (W, ff["expert"]["ff"])
    return out


def random_weights(cfg: dict, ranks: tuple, seed: int, bf16_exact: bool = True) -> dict[str, torch.Tensor]:
    """32-bit random weights by stored name; with `bf16_exact` every value is a bfloat16 value, so that the engine in
    either precision and the plain model read the same numbers."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for key, shape in tensor_shapes(cfg, ranks).items():
        t = torch.randn(shape, generator=g)
        last = key.rsplit(".", 1)[-1]
        if key == "embed":
            t = t * 0.8
        elif last in ("norm", "norm1", "norm2", "out"):
            t = 1.0 + 0.2 * t
        elif last == "sink":
            t = 1.5 * t
        elif last == "A_log":
            t = 0.5 * t - 1.0
        elif last == "dt_bias":
            t = t - 1.5                             # decays mostly near one, some far from it
        elif key.endswith(".f.b"):
            t = t + 3.0
        elif last == "b" and len(shape) == 1:
            t = 0.7 * t
        elif last == "conv":
            t = t * 0.5
            t[:, -1] += 0.7
        elif last == "router":
            t = t * (1.5 * shape[1] ** -0.5)
        else:
            t = t * (shape[1] ** -0.5)
        out[key] = t.to(torch.bfloat16).float() if bf16_exact else t
    return out


def weights(name: str, bf16_exact: bool = True) -> dict[str, torch.Tensor]:
    return random_weights(CONFIGS[name], RANKS[name], SEEDS[name], bf16_exact)


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


def random_config(seed: int) -> tuple[dict, tuple]:
    """A model drawn at random: layer order, small sizes and large (unit keys and normed heads of one or two entries are
    little more than signs, which rounding can turn, so those begin at 4 and 3), chunks, rotations, taps, borrowed tensors, feed-forwards. Returns
    (config, the narrow products' inner sizes)."""
    r = random.Random(seed)

    def dsizes():
        kv = r.choice([1, 2, 3])
        return (kv * r.choice([1, 1, 2, 3]), kv, r.choice([4, 7, 16, 24, 40, 64]), r.choice([3, 6, 8, 16, 40, 64]), r.choice([1, 2, 3, 4, 6]))

    layers = []
    for _ in range(r.randint(2, 5)):
        kind = r.choice(["channel_delta", "mlstm", "parallel", "parallel"])
        ff = r.choice([None, 16, 40, 64, (r.choice([1, 2, 3, 6]), 1, 16), (4, r.choice([2, 4]), 24), (18, 3, 8)])
        if kind == "channel_delta":
            layers.append(delta(*dsizes(), ff=ff))
        elif kind == "mlstm":
            layers.append(memory(r.choice([1, 2, 4]), r.choice([1, 4, 16, 24, 64]), r.choice([3, 8, 16, 40]), r.choice([1.5, 8.0, 20.0]), ff=ff))
        else:
            kv, dim = r.choice([1, 2, 3]), r.choice([8, 10, 16, 24, 64])
            dims = r.choice([d for d in (2, 4, 8, 10, 16, 24, 64) if d <= dim])
            layers.append(parallel((kv * r.choice([1, 2, 4]), kv, dim, r.choice([4, 8, 16, 48, 64]), r.uniform(0.1, 0.5),
                                    r.choice([None, (r.choice([100.0, 10000.0]), dims), (r.choice([100.0, 10000.0]), dims)]),
                                    r.choice([None, 1, 9, 16, 33, 64])), dsizes(), ff=ff))
        if layers[:-1] and r.random() < 0.3:
            layers.append(again([dict(l) for l in layers], r.choice([i for i, l in enumerate(layers) if "weights_of" not in l])))
    return {"architecture": "Gifopel", "vocab": r.choice([50, 131, 256]), "width": r.choice([24, 36, 40, 50, 64, 72, 100]),
            "norm": {"eps": r.choice([1e-6, 1e-4])}, "layers": layers}, (r.choice([1, 3, 8, 16]), r.choice([2, 8, 11]))
