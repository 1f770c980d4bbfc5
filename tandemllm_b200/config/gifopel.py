"""The Gifopel configuration (`"architecture": "Gifopel"`), typed.

A decoder whose layers are listed one by one in config.json; an entry names its mixer's type, the mixer's sizes and constants and
its feed-forward (or none). Everything that can differ between models of the design is read here and nowhere else; `to_spec()`
turns it into the architecture-neutral `ModelSpec`. A key this reader does not know stops the load with its name.

  config.json       vocab, width, norm: {eps}, layers: [{type, mixer, mlp | null, weights_of}, ...]
  layer             mixer and feed-forward read two norms of the same residual, x <- x + (mixer(norm1 x) + ff(norm2 x)); plain RMS
                    norms l<i>.norm1, l<i>.norm2, final.norm. With `weights_of`: j the layer runs layer j's tensors and has none of
                    its own, with a cache and state of its own
  channel_delta     mixer {heads, kv_heads, dim, vdim, conv}: the gated delta rule with a decay a head and key channel and a narrow
                    sigmoid gate; tensors l<i>.mix.{q,k,v}, .{q,k,v}.conv, .b, .A_log, .dt_bias, .a1, .a2, .norm, .g1, .g2, .o
  mlstm             mixer {heads, dim, vdim, gate_cap}: the gated matrix memory; tensors l<i>.mix.{q,k,v,g,o,norm,i,i.b,f,f.b}
  parallel          mixer {left, right}: half the sum of two mixers' outputs, each normed over the width (.left.out, .right.out)
    left            {heads, kv_heads, dim, vdim, scale, rot: {base, dims}, mask: {size}}: grouped-query attention within chunks of
                    `mask.size` positions, q and k normed a head (.q.norm, .k.norm), interleaved rotary pairs, a sink a head in
                    the softmax, a sigmoid gate a head; tensors l<i>.mix.left.{q,k,v,q.norm,k.norm,sink,g,o}
    right           {heads, kv_heads, dim, vdim, conv}: the gated delta rule with one decay a head and a silu gate; tensors
                    l<i>.mix.right.{q,k,v}, .{q,k,v}.conv, .b, .A_log, .dt_bias, .a, .norm, .g, .o
  mlp               {kind: dense, ff}: down(silu(gate n) * up n), tensors l<i>.mlp.{gate,up,down};
                    {kind: moe, router: {experts, top}, expert: {ff}}: ungated experts down(relu(up n)^2), the `top` with the largest
                    logits (router n + router.b), weighed by the softmax over those; tensors l<i>.mlp.{router,router.b,e<j>.{up,down}}
  head              the embedding table `embed`
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .spec import LayerSpec, ModelSpec, PartSpec, Site

ARCHITECTURES = ("Gifopel",)
MODEL_TYPES = ("gifopel",)

UNIT_EPS = 1e-6         # inside the root of q's and k's length in the delta rule
READ_FLOOR = 1e-6       # added to the matrix memory's normaliser
AVERAGE_SCALE = 0.5     # two mixers side by side: half the sum of their normed outputs

TOP_KEYS = {"architecture", "architectures", "model_type", "layers", "norm", "vocab", "width"}
LAYER_KEYS = {"type", "mixer", "mlp", "weights_of"}
DELTA_KEYS = {"heads", "kv_heads", "dim", "vdim", "conv"}
MEMORY_KEYS = {"heads", "dim", "vdim", "gate_cap"}
ATTENTION_KEYS = {"heads", "kv_heads", "dim", "vdim", "scale", "rot", "mask"}
MLP_KEYS = {"kind", "ff", "router", "expert"}


def _only(d: dict, known: set, where: str) -> None:
    unknown = sorted(set(d) - known)
    if unknown:
        raise ValueError(f"Gifopel config: {where} has key(s) this engine does not know: {', '.join(unknown)}")


def _need(d: dict, keys, where: str) -> None:
    for k in keys:
        if k not in d:
            raise ValueError(f"Gifopel config: {where} lacks the required key {k!r}")


def _check_heads(m: dict, where: str) -> None:
    H, G = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
    if H <= 0 or G <= 0 or H % G or int(m["dim"]) <= 0 or int(m["vdim"]) <= 0:
        raise ValueError(f"Gifopel config: {where}: {H} heads over {G} kv_heads of sizes {m['dim']} and {m['vdim']}")


def _check_delta(m: dict, where: str) -> None:
    _only(m, DELTA_KEYS, where)
    _need(m, ("heads", "dim", "vdim", "conv"), where)
    _check_heads(m, where)
    if int(m["conv"]) < 1:
        raise ValueError(f"Gifopel config: {where}.conv {m['conv']}: a positive number of taps")


def _check_attention(m: dict, where: str) -> None:
    _only(m, ATTENTION_KEYS, where)
    _need(m, ("heads", "kv_heads", "dim", "vdim", "scale"), where)
    _check_heads(m, where)
    rot = m.get("rot")
    if rot is not None:
        _only(rot, {"base", "dims"}, where + ".rot")
        _need(rot, ("base", "dims"), where + ".rot")
        if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= int(m["dim"]):
            raise ValueError(f"Gifopel config: {where}: {rot['dims']} rotated entries of a head of {m['dim']}")
    mask = m.get("mask")
    if mask is not None:
        _only(mask, {"size"}, where + ".mask")
        _need(mask, ("size",), where + ".mask")
        if int(mask["size"]) <= 0:
            raise ValueError(f"Gifopel config: {where}.mask.size {mask['size']}: a positive number of positions")


@dataclass
class GifopelLayer:
    type: str
    mixer: dict
    mlp: dict | None
    weights_of: int | None = None


@dataclass
class GifopelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: list[GifopelLayer] = field(default_factory=list)
    path: str = ""

    @classmethod
    def from_dict(cls, raw: dict, path: str = "", generation: dict | None = None) -> "GifopelConfig":
        _only(raw, TOP_KEYS, "the top level")
        _need(raw, ("layers", "norm", "vocab", "width"), "the top level")
        _only(raw["norm"], {"eps"}, "norm")
        _need(raw["norm"], ("eps",), "norm")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _only(entry, LAYER_KEYS, where)
            _need(entry, ("type", "mixer"), where)
            kind, m, at = str(entry["type"]), dict(entry["mixer"]), where + ".mixer"
            if kind == "channel_delta":
                _check_delta(m, at)
            elif kind == "mlstm":
                _only(m, MEMORY_KEYS, at)
                _need(m, ("heads", "dim", "vdim", "gate_cap"), at)
                _check_heads(m, at)
                if not float(m["gate_cap"]) > 0.0:
                    raise ValueError(f"Gifopel config: {at}.gate_cap must be positive")
            elif kind == "parallel":
                _only(m, {"left", "right"}, at)
                _need(m, ("left", "right"), at)
                _check_attention(m["left"], at + ".left")
                _check_delta(m["right"], at + ".right")
            else:
                raise ValueError(f"Gifopel config: {where}.type {kind!r}: channel_delta, mlstm and parallel are implemented")
            mlp = entry.get("mlp")
            if mlp is not None:
                mlp, at = dict(mlp), where + ".mlp"
                _only(mlp, MLP_KEYS, at)
                _need(mlp, ("kind",), at)
                if mlp["kind"] == "dense":
                    _need(mlp, ("ff",), at)
                    if int(mlp["ff"]) <= 0:
                        raise ValueError(f"Gifopel config: {at}.ff must be positive")
                elif mlp["kind"] == "moe":
                    _need(mlp, ("router", "expert"), at)
                    _only(mlp["router"], {"experts", "top"}, at + ".router")
                    _need(mlp["router"], ("experts", "top"), at + ".router")
                    _only(mlp["expert"], {"ff"}, at + ".expert")
                    _need(mlp["expert"], ("ff",), at + ".expert")
                    E, k = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
                    if not 0 < k <= E or int(mlp["expert"]["ff"]) <= 0:
                        raise ValueError(f"Gifopel config: {at}: top {k} of {E} experts of {mlp['expert']['ff']}")
                else:
                    raise ValueError(f"Gifopel config: {at}.kind {mlp['kind']!r}: dense and moe are implemented")
            of = entry.get("weights_of")
            layers.append(GifopelLayer(kind, m, mlp, int(of) if of is not None else None))
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]), layers=layers, path=path)
        cfg.validate()
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            j = self.layers[i].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ValueError(f"Gifopel config: layers[{i}].weights_of {j} names no layer with tensors of its own")
            seen.add(j)
            i = j
        return i

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ValueError("Gifopel config: vocab, width and the number of layers must be positive")
        for i, layer in enumerate(self.layers):
            own = self.layers[self.owner(i)]
            if (own.type, own.mixer, own.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ValueError(f"Gifopel config: layers[{i}] runs layer {self.owner(i)}'s tensors and differs from it")

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            d = {"type": l.type, "mixer": l.mixer, "mlp": l.mlp}
            if l.weights_of is not None:
                d["weights_of"] = l.weights_of
            layers.append(d)
        return {"architecture": ARCHITECTURES[0], "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": layers}

    def to_spec(self) -> ModelSpec:
        eps = self.norm_eps

        def norm(tensor: str) -> PartSpec:
            return PartSpec("rmsnorm", {"eps": eps, "tensor": tensor})

        def delta(m: dict, at: str, channel: bool) -> PartSpec:
            names = {"q": "q", "k": "k", "v": "v", "b": "b", "a_log": "A_log", "dt_bias": "dt_bias", "norm": "norm", "out": "o"}
            names.update({"a1": "a1", "a2": "a2", "g1": "g1", "g2": "g2"} if channel else {"a": "a", "gate": "g"})
            return PartSpec("gated_delta_rule", {
                "heads": int(m["heads"]), "groups": int(m.get("kv_heads", m["heads"])), "head_dim": int(m["dim"]),
                "value_dim": int(m["vdim"]), "taps": int(m["conv"]), "eps": eps, "unit_eps": UNIT_EPS,
                "decay": "channel" if channel else "head", "gate": "narrow_sigmoid" if channel else "silu",
                "names": {k: at + v for k, v in names.items()}})

        def attention(m: dict, at: str) -> PartSpec:
            rot = m.get("rot")
            if rot and int(rot["dims"]) > 0:
                position = PartSpec("rope_pairs", {"theta": float(rot["base"]), "rotary_dim": int(rot["dims"])})
            else:
                position = PartSpec("none", {})
            return PartSpec("attention", {
                "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]), "head_dim": int(m["dim"]),
                "value_dim": int(m["vdim"]), "qk_norm": norm("norm"), "position": position, "scale": float(m["scale"]),
                "chunk": int(m["mask"]["size"]) if m.get("mask") else None, "sinks": at + "sink", "gate": at + "g",
                "weight_suffix": "", "names": {"q": at + "q", "k": at + "k", "v": at + "v", "q_norm": at + "q", "k_norm": at + "k",
                                               "out": at + "o"}})

        layers, place, ignored = [], {}, []
        for i, layer in enumerate(self.layers):
            if layer.weights_of is not None:
                continue
            m = layer.mixer
            if layer.type == "channel_delta":
                mixer = delta(m, "mix.", True)
            elif layer.type == "mlstm":
                mixer = PartSpec("matrix_memory", {
                    "heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "gate_cap": float(m["gate_cap"]),
                    "eps": eps, "read_floor": READ_FLOOR,
                    "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "gate": "mix.g", "i": "mix.i", "i_bias": "mix.i.b",
                              "f": "mix.f", "f_bias": "mix.f.b", "norm": "mix.norm", "out": "mix.o"}})
            else:
                mixer = PartSpec("normed_average", {
                    "mixers": (attention(m["left"], "mix.left."), delta(m["right"], "mix.right.", False)),
                    "norms": ("mix.left.out", "mix.right.out"), "eps": eps, "scale": AVERAGE_SCALE})
            mlp = layer.mlp
            if mlp is None:
                ff = PartSpec("none", {})
                ignored.append(f"l{i}.norm2")       # what a folder may still hold for the feed-forward that is not there
            elif mlp["kind"] == "dense":
                ff = PartSpec("swiglu", {"intermediate_size": int(mlp["ff"]), "activation": "silu", "weight_suffix": "",
                                         "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
            else:
                ff = PartSpec("sigmoid_topk_experts", {
                    "num_experts": int(mlp["router"]["experts"]), "top_k": int(mlp["router"]["top"]),
                    "intermediate_size": int(mlp["expert"]["ff"]), "expert_bias": True, "normalize": True, "norm_floor": 0.0,
                    "scale": 1.0, "scoring": "chosen_softmax", "gated": False, "activation": "relu2", "weight_suffix": "",
                    "expert_separator": "",
                    "names": {"router": "mlp.router", "bias": "mlp.router.b", "experts": "mlp.e", "up": "up", "down": "down"}})
            place[i] = len(layers)
            layers.append(LayerSpec(prefix=f"l{i}.", mixer=mixer, feed_forward=ff, mixer_norm=norm("norm1"),
                                    feed_forward_norm=norm("norm2") if mlp is not None else None, arrangement="parallel_residual"))
        schedule = tuple(Site(place[self.owner(i)]) for i in range(len(self.layers)))
        return ModelSpec(
            architecture=ARCHITECTURES[0], hidden_size=self.width, vocab_size=self.vocab, layers=tuple(layers), schedule=schedule,
            final_norm=norm("norm"), embedding_name="embed", final_norm_prefix="final.", head_name=None,
            ignored_names=tuple(ignored), name_prefixes=())
