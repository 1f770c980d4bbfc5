"""The decoder built from a `ModelSpec`: embedding, the scheduled layers, final norm, head.

  h = embed[tokens] (times the spec's embedding scale); for each site of the schedule: run its layer on its cache; h = final_norm(h);
  logits = h @ head^T in 32-bit, head = the embedding when tied   (engine/models/lfm2_moe/ref.py:218-241)
  with `token_pairs` in the spec the embedded row is the sum of two: the token's own and the one of (token before, token)
  with a soft cap c in the spec: logits <- c tanh(logits / c); with a logit scale: logits <- logits * scale
  with `streams` in the spec the residual is [streams, rows, hidden], every stream starts as the embedded row, the layers'
  arrangement rewrites them, and the last norm reads their sum

The model owns no cache: `cache_needs()` tells the cache manager what every site needs (and, behind the sites, what the embedding
does: a request's last token) and `forward` is given the per-site caches it made. It computes the final norm and the head for the wanted rows only.
"""

from __future__ import annotations

import torch

from ..config.spec import ModelSpec
from ..kernels import ops
from ..settings import SETTINGS
from ..weights.loader import TensorSpec
from .base import Runtime, SlotNeed, StepContext, make_part
from .block import Layer
from .linear import linear


class DecoderModel:
    def __init__(self, spec: ModelSpec):
        self.spec = spec
        self.hidden_size, self.vocab_size = spec.hidden_size, spec.vocab_size
        self.layers = [Layer(ls, spec.hidden_size) for ls in spec.layers]
        self.final_norm = make_part("norm", spec.final_norm, prefix=spec.final_norm_prefix, size=spec.hidden_size)
        self.runtime: Runtime | None = None
        self.embedding = self.head = self.pair_embedding = None

    # ---- weights ----
    def weight_specs(self, present: set[str] | None = None) -> list[TensorSpec]:
        s = self.spec
        out = [TensorSpec(s.embedding_name, (s.vocab_size, s.hidden_size))]
        if s.token_pairs:
            out.append(TensorSpec(s.token_pairs.tensor, (s.token_pairs.buckets + 1, s.hidden_size)))
        out += self.final_norm.weight_specs(present)
        if s.head_name:
            out.append(TensorSpec(s.head_name, (s.vocab_size, s.hidden_size)))
        for layer in self.layers:
            out += layer.weight_specs(present)
        seen = set()
        for site in s.schedule:             # vectors the run order adds to the stream between layers
            if site.add is not None and site.add.tensor not in seen:
                seen.add(site.add.tensor)
                out.append(TensorSpec(site.add.tensor, (site.add.rows, s.hidden_size), role="vector", init="bias"))
        return out

    def load(self, weights, runtime: Runtime) -> "DecoderModel":
        """Check `weights` (a FolderWeights or DictWeights) against what the parts read, then bind every part."""
        s = self.spec
        present = weights.present()
        for layer in self.layers:           # a size that only a stored tensor's shape gives is read before the check
            for part in layer.parts:
                if hasattr(part, "shapes_from"):
                    part.shapes_from(weights.shape_of)
        specs = self.weight_specs(present)
        ignored = set(s.ignored_names)
        weights.check(specs, ignore=(lambda n: n in ignored) if ignored else None)
        self.runtime = runtime
        self.embedding = runtime.matrix(weights.read(s.embedding_name))
        if s.token_pairs:
            self.pair_embedding = runtime.matrix(weights.read(s.token_pairs.tensor))
        self.head = runtime.matrix(weights.read(s.head_name)) if s.head_name else self.embedding
        self.final_norm.bind(weights.read, runtime)
        for layer in self.layers:
            layer.bind(weights.read, runtime)
        self.stream_adds = {}
        for site in s.schedule:
            if site.add is not None and site.add.tensor not in self.stream_adds:
                self.stream_adds[site.add.tensor] = runtime.vector(weights.read(site.add.tensor))
        return self

    def weight_bytes(self) -> int:
        seen, total = set(), 0
        for obj in [self, self.final_norm] + [p for layer in self.layers for p in layer.parts]:
            stack = [obj]
            while stack:
                o = stack.pop()
                for v in vars(o).values():
                    if isinstance(v, torch.Tensor) and v.is_cuda and v.data_ptr() not in seen:
                        seen.add(v.data_ptr())
                        total += v.numel() * v.element_size()
                    elif hasattr(v, "weight_specs") and v is not o:
                        stack.append(v)
        return total

    def decode_bytes(self, batch: int, experts_read: list[float] | None = None) -> dict:
        """Bytes of weights one decode step of `batch` rows reads, every weight it uses once (the reference accounts a
        token the same way, engine/models/lfm2_moe/pack.py:292-315): per site of the run order its norms', mixer's and
        feed-forward's weights as the parts themselves count them (`Part.step_bytes`), the last norm, the head, and
        `batch` rows of the embedding. `experts_read[i]`: the experts the i-th routed site of the run order really
        read (default: what uniform routing of `batch` rows would). The cache's bytes are the engine's to add."""
        elem = torch.empty(0, dtype=self.runtime.dtype).element_size() if self.runtime else 2
        it = iter(experts_read) if experts_read is not None else None
        dense = experts = 0
        for site in self.spec.schedule:
            layer = self.layers[site.layer]
            for part in layer.parts:
                if hasattr(part, "expected_experts_read"):
                    n = next(it) if it is not None else None
                    whole = part.step_bytes(elem, experts_read=n, rows=batch)
                    fixed = part.step_bytes(elem, experts_read=0)
                    dense += fixed
                    experts += whole - fixed
                else:
                    dense += part.step_bytes(elem)
        dense += self.final_norm.step_bytes(elem)
        head = self.vocab_size * self.hidden_size * elem
        embed = batch * self.hidden_size * elem * (2 if self.spec.token_pairs else 1)
        return {"dense": dense, "experts": experts, "head": head, "embedding_rows": embed,
                "total": dense + experts + head + embed}

    @property
    def graph_safe(self) -> bool:
        """Every part of every layer says its forward may be captured in a CUDA graph."""
        return all(getattr(p, "graph_safe", False) for layer in self.layers for p in layer.parts) and \
            getattr(self.final_norm, "graph_safe", False)

    # ---- caches ----
    def cache_needs(self) -> list:
        """Per site of the schedule: the need of its mixer, or None when the site reads another site's cache; last, with a table of
        token pairs, the embedding's: a request's last token (-1: it has none yet)."""
        needs = [None if site.cache_of is not None else self.layers[site.layer].mixer.cache_need()
                 for site in self.spec.schedule]
        return needs + [SlotNeed((1,), torch.int32, init=-1)] if self.spec.token_pairs else needs

    # ---- the forward pass of one batch ----
    def forward(self, step: StepContext, site_caches: list) -> torch.Tensor:
        rt = self.runtime
        shape = (step.n_rows, self.hidden_size)
        residual = torch.empty((self.spec.streams,) + shape if self.spec.streams else shape, dtype=torch.float32, device=rt.device)
        pairs = self.spec.token_pairs
        if pairs is None:
            ops.embed_rows(self.embedding, step.token_ids, residual, rt.status, self.spec.embedding_scale)
        else:
            if self.spec.streams:
                raise NotImplementedError("a second embedding over a residual of several streams")
            ops.embed_token_pairs(self.embedding, self.pair_embedding, step, site_caches[len(self.spec.schedule)].state, residual,
                                  rt.status, pairs.mul_prev, pairs.mul_cur, self.spec.embedding_scale)
        pending = None
        ranges = SETTINGS.is_set("NVTX")             # named ranges for profilers: the step, and each layer in run order
        if ranges:
            torch.cuda.nvtx.range_push(f"step rows={step.n_rows} requests={step.n_requests}")
        try:
            for i, site in enumerate(self.spec.schedule):
                own = site.cache_of is None
                cache = site_caches[i if own else site.cache_of]
                if ranges:
                    layer = self.layers[site.layer]
                    torch.cuda.nvtx.range_push(f"site {i} layer {site.layer} {type(layer.mixer).__name__} + "
                                               f"{type(layer.feed_forward).__name__}")
                if site.add is not None:
                    # (what is pending is added by the layer's first norm; the order of the two additions is free)
                    if self.spec.streams:
                        raise NotImplementedError("a vector added between layers to a residual of several streams")
                    ops.add_vector(residual, self.stream_adds[site.add.tensor][site.add.row])
                pending = self.layers[site.layer].run(residual, pending, step, cache, writes_cache=own)
                if ranges:
                    torch.cuda.nvtx.range_pop()
            if step.n_out == 0:
                return torch.empty(0, self.vocab_size, dtype=torch.float32, device=rt.device)
            if ranges:
                torch.cuda.nvtx.range_push("final norm + head")
            if self.spec.streams:       # the last sublayer's output goes into the streams, whose plain sum is normed
                pending = (pending or ops.StreamUpdate(None, None, None)).reading(None)
            n = self.final_norm.add_norm(residual, pending, gather=step.out_rows, n_out=step.n_out)
            out = linear(rt, n, self.head, out_dtype=torch.float32)
            if self.spec.logit_scale != 1.0:
                ops.activation(out, out, ops.ACTIVATIONS["scale"], float(self.spec.logit_scale))
            if self.spec.logit_softcap:
                ops.softcap(out, float(self.spec.logit_softcap))
            if ranges:
                torch.cuda.nvtx.range_pop()
            return out
        finally:
            if ranges:
                torch.cuda.nvtx.range_pop()
