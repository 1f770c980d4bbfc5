"""The Dipivik configuration (`"architecture": "Dipivik"`), typed.

A decoder whose layers are listed one by one in config.json; an entry names its mixer's type, the mixer's sizes and constants and
its feed-forward (or none). Everything that can differ between models of the design is read here and nowhere else; `to_spec()`
turns it into the architecture-neutral `ModelSpec`. A key this reader does not know stops the load with its name.

  config.json       vocab, width, norm: {eps}, logit_softcap, embedding: {bigram: {buckets, mul_prev, mul_cur}}, layers: [{type, mixer,
                    mlp | null}, ...]
  embedding         embed[token] + bigram[(token before * mul_prev + token * mul_cur) mod buckets], a sequence's first token with the
                    last row of `bigram`; the head is `embed` again, its logits softly capped at logit_softcap
  layer             mixer and feed-forward read one norm of the same residual, x <- x + (mixer(n) + ff(n)) with n = norm1 x; plain RMS
                    norms l<i>.norm1, final.norm
  latent_attention  mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot: {base, dims}, mask: {size}}: attention over a cached
                    latent with a sliding window, rotary halves on the rot_dim part, a sigmoid gate a head; tensors
                    l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}
  retention         mixer {heads, dim, vdim, decay: [a number a head], rot: {base, dims}}: linear attention with a fixed decay a head,
                    rotary halves on q and k, k times dim^(-1/2), every head's output at unit root mean square, a silu gate; tensors
                    l<i>.mix.{q,k,v,g,o}
  mlp               {kind: dense, ff}: down(gelu(gate n + b) * (up n + b)) + b, gelu in its tanh form, tensors
                    l<i>.mlp.{gate,up,down}, each with .b;
                    {kind: moe, router: {experts, top}, expert: {ff}, shared: {ff}}: the `top` experts with the largest
                    s = sigmoid(router n), the sum of down(silu(gate s n) * (up s n)) over them, and the same form with s = 1 for a
                    shared expert (optional) of every row; tensors l<i>.mlp.{router,e<j>.{gate,up,down},shared.{gate,up,down}}
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .spec import LayerSpec, ModelSpec, PartSpec, TokenPairs, plain_schedule

ARCHITECTURES = ("Dipivik",)
MODEL_TYPES = ("dipivik",)

TOP_KEYS = {"architecture", "architectures", "model_type", "embedding", "layers", "logit_softcap", "norm", "vocab", "width"}
LAYER_KEYS = {"type", "mixer", "mlp"}
BIGRAM_KEYS = {"buckets", "mul_prev", "mul_cur"}
LATENT_KEYS = {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot", "mask"}
RETENTION_KEYS = {"heads", "dim", "vdim", "decay", "rot"}
MLP_KEYS = {"kind", "ff", "router", "expert", "shared"}


def _only(d: dict, known: set, where: str) -> None:
    unknown = sorted(set(d) - known)
    if unknown:
        raise ValueError(f"Dipivik config: {where} has key(s) this engine does not know: {', '.join(unknown)}")


def _need(d: dict, keys, where: str) -> None:
    for k in keys:
        if k not in d:
            raise ValueError(f"Dipivik config: {where} lacks the required key {k!r}")


def _positive(d: dict, keys, where: str) -> None:
    for k in keys:
        if int(d[k]) <= 0:
            raise ValueError(f"Dipivik config: {where}.{k} {d[k]}: a positive number")


def _check_rot(rot: dict | None, dim: int, where: str) -> None:
    if rot is None:
        return
    _only(rot, {"base", "dims"}, where)
    _need(rot, ("base", "dims"), where)
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= dim:
        raise ValueError(f"Dipivik config: {where}: {rot['dims']} rotated entries of {dim}")


def _check_mixer(kind: str, m: dict, at: str) -> None:
    if kind == "latent_attention":
        _only(m, LATENT_KEYS, at)
        _need(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale"), at)
        _positive(m, ("heads", "vdim", "kv_rank", "q_rank"), at)
        _check_rot(m.get("rot"), int(m["rot_dim"]), at + ".rot")
        if m.get("mask") is not None:
            _only(m["mask"], {"size"}, at + ".mask")
            _need(m["mask"], ("size",), at + ".mask")
            _positive(m["mask"], ("size",), at + ".mask")
    elif kind == "retention":
        _only(m, RETENTION_KEYS, at)
        _need(m, ("heads", "dim", "vdim", "decay"), at)
        _positive(m, ("heads", "dim", "vdim"), at)
        _check_rot(m.get("rot"), int(m["dim"]), at + ".rot")
        if len(m["decay"]) != int(m["heads"]):
            raise ValueError(f"Dipivik config: {at}: {len(m['decay'])} decays for {m['heads']} heads")
    else:
        raise ValueError(f"Dipivik config: {at}: type {kind!r}: latent_attention and retention are implemented")


def _check_mlp(mlp: dict, at: str) -> None:
    _only(mlp, MLP_KEYS, at)
    _need(mlp, ("kind",), at)
    if mlp["kind"] == "dense":
        _need(mlp, ("ff",), at)
        _positive(mlp, ("ff",), at)
    elif mlp["kind"] == "moe":
        _need(mlp, ("router", "expert"), at)
        _only(mlp["router"], {"experts", "top"}, at + ".router")
        _need(mlp["router"], ("experts", "top"), at + ".router")
        for part in ("expert", "shared"):
            if mlp.get(part) is not None:
                _only(mlp[part], {"ff"}, f"{at}.{part}")
                _need(mlp[part], ("ff",), f"{at}.{part}")
                _positive(mlp[part], ("ff",), f"{at}.{part}")
        if not 0 < int(mlp["router"]["top"]) <= int(mlp["router"]["experts"]):
            raise ValueError(f"Dipivik config: {at}: top {mlp['router']['top']} of {mlp['router']['experts']} experts")
    else:
        raise ValueError(f"Dipivik config: {at}.kind {mlp['kind']!r}: dense and moe are implemented")


@dataclass
class DipivikLayer:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class DipivikConfig:
    vocab: int
    width: int
    norm_eps: float
    bigram: dict | None = None
    logit_softcap: float | None = None
    layers: list[DipivikLayer] = field(default_factory=list)
    path: str = ""

    @classmethod
    def from_dict(cls, raw: dict, path: str = "", generation: dict | None = None) -> "DipivikConfig":
        _only(raw, TOP_KEYS, "the top level")
        _need(raw, ("layers", "norm", "vocab", "width"), "the top level")
        _only(raw["norm"], {"eps"}, "norm")
        _need(raw["norm"], ("eps",), "norm")
        emb = raw.get("embedding") or {}
        _only(emb, {"bigram"}, "embedding")
        bigram = emb.get("bigram")
        if bigram is not None:
            bigram = dict(bigram)
            _only(bigram, BIGRAM_KEYS, "embedding.bigram")
            _need(bigram, sorted(BIGRAM_KEYS), "embedding.bigram")
            _positive(bigram, ("buckets",), "embedding.bigram")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _only(entry, LAYER_KEYS, where)
            _need(entry, ("type", "mixer"), where)
            kind, m = str(entry["type"]), dict(entry["mixer"])
            _check_mixer(kind, m, where + ".mixer")
            mlp = entry.get("mlp")
            if mlp is not None:
                mlp = dict(mlp)
                _check_mlp(mlp, where + ".mlp")
            layers.append(DipivikLayer(kind, m, mlp))
        cap = raw.get("logit_softcap")
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]), bigram=bigram,
                  logit_softcap=float(cap) if cap else None, layers=layers, path=path)
        if cfg.vocab <= 0 or cfg.width <= 0 or not layers:
            raise ValueError("Dipivik config: vocab, width and the number of layers must be positive")
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": ARCHITECTURES[0], "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": [{"type": l.type, "mixer": l.mixer, "mlp": l.mlp} for l in self.layers]}
        if self.bigram is not None:
            out["embedding"] = {"bigram": self.bigram}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out

    def to_spec(self) -> ModelSpec:
        eps = self.norm_eps

        def norm(tensor: str) -> PartSpec:
            return PartSpec("rmsnorm", {"eps": eps, "tensor": tensor})

        def position(rot: dict | None) -> PartSpec:
            if not rot or int(rot["dims"]) == 0:
                return PartSpec("none", {})
            return PartSpec("rope_neox", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "precise": True})

        def gated(ff: int, activation: str, at: str, biases: bool) -> PartSpec:
            names = {k: at + k for k in ("gate", "up", "down")}
            return PartSpec("swiglu", {"intermediate_size": ff, "activation": activation, "weight_suffix": "", "names": names,
                                       "biases": {k: v + ".b" for k, v in names.items()} if biases else None})

        layers = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if layer.type == "latent_attention":
                mixer = PartSpec("latent_attention", {
                    "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
                    "value_dim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]),
                    "scale": float(m["scale"]), "window": int(m["mask"]["size"]) if m.get("mask") else None, "eps": eps,
                    "position": position(m.get("rot")), "gate_heads": True,
                    "names": {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq", "dkv": "mix.dkv",
                              "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv", "gate": "mix.g", "out": "mix.o"}})
            else:
                mixer = PartSpec("decayed_linear_attention", {
                    "heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]),
                    "decay": tuple(float(d) for d in m["decay"]), "activation": "identity", "eps": eps,
                    "position": position(m.get("rot")), "key_scale": int(m["dim"]) ** -0.5, "norm_each": True,
                    "gate_activation": "silu",
                    "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "gate": "mix.g", "out": "mix.o"}})
            mlp = layer.mlp
            if mlp is None:
                ff = PartSpec("none", {})
            elif mlp["kind"] == "dense":
                ff = gated(int(mlp["ff"]), "gelu_tanh", "mlp.", biases=True)
            else:
                ff = PartSpec("sigmoid_topk_experts", {
                    "num_experts": int(mlp["router"]["experts"]), "top_k": int(mlp["router"]["top"]),
                    "intermediate_size": int(mlp["expert"]["ff"]), "expert_bias": False, "normalize": False, "scale": 1.0,
                    "scoring": "sigmoid", "activation": "silu", "weigh": "input", "weight_suffix": "", "expert_separator": "",
                    "names": {"router": "mlp.router", "experts": "mlp.e", "gate": "gate", "up": "up", "down": "down"}})
                if mlp.get("shared"):
                    ff = PartSpec("shared_and_routed", {
                        "routed": ff, "shared": gated(int(mlp["shared"]["ff"]), "silu", "mlp.shared.", biases=False),
                        "shared_gate": None})
            layers.append(LayerSpec(prefix=f"l{i}.", mixer=mixer, feed_forward=ff, mixer_norm=norm("norm1"), feed_forward_norm=None,
                                    arrangement="parallel_residual"))
        b = self.bigram
        pairs = TokenPairs("bigram", int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None
        return ModelSpec(
            architecture=ARCHITECTURES[0], hidden_size=self.width, vocab_size=self.vocab, layers=tuple(layers),
            schedule=plain_schedule(len(layers)), final_norm=norm("norm"), embedding_name="embed", final_norm_prefix="final.",
            head_name=None, token_pairs=pairs, logit_softcap=self.logit_softcap, name_prefixes=())
