"""Mixers over a matrix state whose writes depend on what the state holds or on a running maximum, and the mixer that averages two
mixers' normed outputs.

`gated_delta_rule`: q, k (`groups` heads of `head_dim`) and v (`heads` of `value_dim`) are projections that each pass a causal
    convolution over the last `taps` tokens a channel and silu; q and k are brought to unit length, x / sqrt(sum x^2 + unit_eps), and
    q is multiplied by head_dim^(-1/2); a head uses the q and k of group h // (heads / groups). beta = sigmoid(W_b n) a head;
    a decay exp(-exp(a_log_h) softplus(z + dt_bias)), z = W_a n one a head (`decay` "head") or z = W_a2 (W_a1 n) one a head and key
    channel (`decay` "channel", the inner size from the stored `a1`). Per head
        S <- decay S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
    Every head's o is brought to unit root mean square, times the weight `norm` (one head's size, shared by the heads), times the
    gate, and projected by W_o. The gate is silu(W_g n) (`gate` "silu") or sigmoid(W_g2 (W_g1 n)) (`gate` "narrow_sigmoid").

`matrix_memory`: q = W_q n head_dim^(-1/2), k = W_k n (`heads` x `head_dim`), v = W_v n (`heads` x `value_dim`). A log input gate
    i = cap tanh((W_i n + i_bias) / cap) and a log forget gate f = log sigmoid(cap tanh((W_f n + f_bias) / cap)) a head. With the running
    maximum m_t = max(f + m, i), which starts at 0:
        S <- exp(f + m_(t-1) - m_t) S + exp(i - m_t) k v^T, the keys' sum n likewise;  o = S^T q / (max(|n . q|, exp(-m_t)) + read_floor).
    Every head's o is brought to unit root mean square, times `norm` (all heads' size), times sigmoid(W_g n), and projected by W_o.

`normed_average`: out = scale * sum_i norm_i * mixer_i(n) / rms(mixer_i(n)) of two mixers on the same rows, each norm over the
    model width with a weight of its own. Each mixer keeps what it needs (pages, a slot) for itself.

What enters a recurrence is 32-bit in both precisions, and so are the in-projections' results (csrc/recurrence_write.cu). A request's
slot holds the convolution's last inputs (or the running maxima) and behind them the state, [heads, values, keys]; a new request's
slot is zero.
"""

from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import Part, SlotNeed, make_part, register_part
from .linear import linear
from .linear_recurrence import _stack


def _round4(n: int) -> int:
    return -(-n // 4) * 4


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Part):
    graph_safe = True

    def __init__(self, spec, prefix: str = "", hidden_size: int = 0, **_):
        super().__init__(spec, prefix, hidden_size)
        self.heads, self.head_dim = int(spec["heads"]), int(spec["head_dim"])
        self.groups = int(spec.get("groups") or self.heads)
        self.value_dim = int(spec.get("value_dim") or self.head_dim)
        self.taps = int(spec["taps"])
        if self.heads <= 0 or self.groups <= 0 or self.heads % self.groups:
            raise ValueError(f"{self.heads} heads over {self.groups} key heads")
        if not 1 <= self.head_dim <= 512:
            raise ValueError(f"a state of {self.head_dim} keys a head: 1 to 512 are implemented")
        if not 1 <= self.taps <= 64:
            raise ValueError(f"a convolution of {self.taps} taps: 1 to 64 are implemented")
        self.eps, self.unit_eps = float(spec["eps"]), float(spec["unit_eps"])
        self.decay, self.gate = str(spec["decay"]), str(spec["gate"])
        if self.decay not in ("head", "channel") or self.gate not in ("silu", "narrow_sigmoid"):
            raise ValueError(f"decay {self.decay!r} (head or channel), gate {self.gate!r} (silu or narrow_sigmoid)")
        self.n = {k: prefix + v for k, v in spec["names"].items()}
        self.conv_suffix = str(spec.get("conv_suffix", ".conv"))
        self.ranks = {"a1": None, "g1": None}       # inner sizes: the stored tensors' shapes say them
        # the convolved columns of the in-projection: q, k, v, each beginning at a multiple of 8
        self.conv_widths = {"q": self.groups * self.head_dim, "k": self.groups * self.head_dim, "v": self.heads * self.value_dim}
        self.conv_cols = sum(-(-w // 8) * 8 for w in self.conv_widths.values())
        self.conv_floats = (self.taps - 1) * self.conv_cols
        self.state_at = _round4(self.conv_floats)

    @property
    def out_dim(self) -> int:
        return self.heads * self.value_dim

    @property
    def inner(self) -> list[tuple[str, str, int]]:
        """The products that go through an inner size: (first matrix, second matrix, outputs)."""
        return ([("a1", "a2", self.heads * self.head_dim)] if self.decay == "channel" else []) + \
               ([("g1", "g2", self.out_dim)] if self.gate == "narrow_sigmoid" else [])

    def weight_specs(self, present=None):
        n, W = self.n, self.hidden_size
        out = []
        for x, width in self.conv_widths.items():
            out += [TensorSpec(n[x], (width, W)), TensorSpec(n[x] + self.conv_suffix, (width, self.taps), "vector", "normal")]
        out += [TensorSpec(n["b"], (self.heads, W)), TensorSpec(n["a_log"], (self.heads,), "vector", "bias"),
                TensorSpec(n["norm"], (self.value_dim,), "vector", "ones")]
        if self.decay == "head":
            out += [TensorSpec(n["a"], (self.heads, W)), TensorSpec(n["dt_bias"], (self.heads,), "vector", "bias")]
        else:
            out.append(TensorSpec(n["dt_bias"], (self.heads * self.head_dim,), "vector", "bias"))
        for first, second, outputs in self.inner:
            rank = self.ranks[first] if self.ranks[first] is not None else max(8, outputs // 16)
            out += [TensorSpec(n[first], (rank, W)), TensorSpec(n[second], (outputs, rank))]
        if self.gate == "silu":
            out.append(TensorSpec(n["gate"], (self.out_dim, W)))
        out.append(TensorSpec(n["out"], (W, self.out_dim)))
        return out

    def shapes_from(self, shape_of) -> None:
        for first, _, _ in self.inner:
            shape = shape_of(self.n[first])
            if shape is not None:
                self.ranks[first] = int(shape[0])

    def bind(self, read, runtime):
        self.runtime = runtime
        n = self.n
        # everything that reads the normed row is one product whose result stays 32-bit: q, k, v, the write strengths, then one
        # decay a head and the gate where they are plain projections
        names = ["q", "k", "v", "b"] + (["a"] if self.decay == "head" else []) + (["gate"] if self.gate == "silu" else [])
        self.w_in, self.col = _stack([(x, runtime.matrix(read(n[x]))) for x in names])
        taps = torch.zeros(self.conv_cols, self.taps, dtype=torch.float32, device=runtime.device)
        for x, width in self.conv_widths.items():
            taps[self.col[x]:self.col[x] + width] = runtime.vector(read(n[x] + self.conv_suffix))
        self.w_conv = taps.contiguous()
        self.a_log, self.dt_bias = runtime.vector(read(n["a_log"])), runtime.vector(read(n["dt_bias"]))
        self.w_norm = runtime.vector(read(n["norm"]))
        self.w_out = runtime.matrix(read(n["out"]))
        # the products through an inner size run together: the first matrices stacked, the second ones as blocks of one matrix
        self.w_inner = self.w_outer = None
        if self.inner:
            firsts, self.inner_col = _stack([(a, runtime.matrix(read(n[a]))) for a, _, _ in self.inner])
            self.w_inner, rows, at, self.outer_col = firsts, [], 0, {}
            for a, b, outputs in self.inner:
                m = runtime.matrix(read(n[b]))
                block = torch.zeros(-(-outputs // 8) * 8, firsts.shape[0], dtype=m.dtype, device=m.device)
                block[:outputs, self.inner_col[a]:self.inner_col[a] + m.shape[1]] = m
                self.outer_col[b] = at
                at += block.shape[0]
                rows.append(block)
            self.w_outer = torch.cat(rows).contiguous()

    def cache_need(self):
        return SlotNeed((_round4(self.state_at + self.heads * self.value_dim * self.head_dim),), torch.float32)

    def forward_inner(self, x, step, cache, writes_cache: bool, out: torch.Tensor, out_scale: float = 1.0) -> torch.Tensor:
        R, dev = x.shape[0], x.device
        proj = linear(self.runtime, x, self.w_in, out_dtype=torch.float32)
        outer = None
        if self.w_inner is not None:
            outer = linear(self.runtime, linear(self.runtime, x, self.w_inner), self.w_outer, out_dtype=torch.float32)
        y = torch.empty(R, self.out_dim, dtype=torch.float32, device=dev)
        ops.gated_delta_scan(proj, self.col, self.w_conv, self.conv_cols, cache.state, self.state_at, step, y, self.heads, self.groups,
                             self.head_dim, self.value_dim, self.a_log, self.dt_bias, unit_eps=self.unit_eps,
                             q_scale=self.head_dim ** -0.5,
                             decay_logits=outer[:, self.outer_col["a2"]:] if self.decay == "channel" else None,
                             write_state=writes_cache)
        if writes_cache:
            ops.conv_state(proj, self.conv_cols, self.taps, cache.state, step.state_slot, step.row_start, step.n_requests)
        gate = proj[:, self.col["gate"]:] if self.gate == "silu" else outer[:, self.outer_col["g2"]:]
        return ops.group_norm_gate(y, gate, gate.stride(0), self.w_norm, self.eps, self.heads, out_scale, out,
                                   gate_activation="silu" if self.gate == "silu" else "sigmoid")

    def forward(self, x, step, cache, writes_cache: bool = True):
        o = torch.empty(x.shape[0], self.out_dim, dtype=x.dtype, device=x.device)
        self.forward_inner(x, step, cache, writes_cache, o)
        return linear(self.runtime, o, self.w_out, out_dtype=torch.float32, defer=True)


@register_part("mixer", "matrix_memory")
class MatrixMemory(Part):
    graph_safe = True

    def __init__(self, spec, prefix: str = "", hidden_size: int = 0, **_):
        super().__init__(spec, prefix, hidden_size)
        self.heads, self.head_dim = int(spec["heads"]), int(spec["head_dim"])
        self.value_dim = int(spec.get("value_dim") or self.head_dim)
        if self.heads <= 0 or not 1 <= self.head_dim <= 512:
            raise ValueError(f"{self.heads} heads with a state of {self.head_dim} keys: 1 to 512 are implemented")
        self.cap = float(spec["gate_cap"])
        if not self.cap > 0.0:
            raise ValueError(f"gates capped at {self.cap}: a positive number")
        self.eps, self.read_floor = float(spec["eps"]), float(spec["read_floor"])
        self.n = {k: prefix + v for k, v in spec["names"].items()}
        self.state_at = _round4(self.heads)

    @property
    def out_dim(self) -> int:
        return self.heads * self.value_dim

    def weight_specs(self, present=None):
        n, W, H = self.n, self.hidden_size, self.heads
        return [TensorSpec(n["q"], (H * self.head_dim, W)), TensorSpec(n["k"], (H * self.head_dim, W)),
                TensorSpec(n["v"], (self.out_dim, W)), TensorSpec(n["gate"], (self.out_dim, W)),
                TensorSpec(n["i"], (H, W)), TensorSpec(n["i_bias"], (H,), "vector", "bias"),
                TensorSpec(n["f"], (H, W)), TensorSpec(n["f_bias"], (H,), "vector", "bias"),
                TensorSpec(n["norm"], (self.out_dim,), "vector", "ones"), TensorSpec(n["out"], (W, self.out_dim))]

    def bind(self, read, runtime):
        self.runtime = runtime
        n = self.n
        self.w_in, self.col = _stack([(x, runtime.matrix(read(n[x]))) for x in ("q", "k", "v", "gate", "i", "f")])
        self.i_bias, self.f_bias = runtime.vector(read(n["i_bias"])), runtime.vector(read(n["f_bias"]))
        self.w_norm = runtime.vector(read(n["norm"]))
        self.w_out = runtime.matrix(read(n["out"]))

    def cache_need(self):
        return SlotNeed((_round4(self.state_at + self.heads * (self.value_dim + 1) * self.head_dim),), torch.float32)

    def forward(self, x, step, cache, writes_cache: bool = True):
        R, dev, H, VD = x.shape[0], x.device, self.heads, self.value_dim
        proj = linear(self.runtime, x, self.w_in, out_dtype=torch.float32)
        y = torch.empty(R, H * (VD + 1), dtype=torch.float32, device=dev)
        maxima = torch.empty(R, H, dtype=torch.float32, device=dev)
        ops.matrix_memory_scan(proj, self.col, self.i_bias, self.f_bias, self.cap, cache.state, self.state_at, step, y, maxima, H,
                               self.head_dim, VD, q_scale=self.head_dim ** -0.5, write_state=writes_cache)
        o = torch.empty(R, self.out_dim, dtype=x.dtype, device=dev)
        ops.memory_norm_gate(y, maxima, proj[:, self.col["gate"]:], self.w_norm, self.eps, self.read_floor, o, H, VD)
        return linear(self.runtime, o, self.w_out, out_dtype=torch.float32, defer=True)


@register_part("mixer", "normed_average")
class NormedAverageMixer(Part):
    """See the module's text. `mixers`: two specs; `norms`: the names of their outputs' norm weights; `scale`; `eps`. The site's
    cache is the tuple of what the mixers need."""

    def __init__(self, spec, prefix: str = "", hidden_size: int = 0, **_):
        super().__init__(spec, prefix, hidden_size)
        self.mixers = [make_part("mixer", ps, prefix=prefix, hidden_size=hidden_size) for ps in spec["mixers"]]
        self.norm_names = [prefix + name for name in spec["norms"]]
        if len(self.mixers) != 2 or len(self.norm_names) != 2:
            raise ValueError(f"{len(self.mixers)} mixers with {len(self.norm_names)} norms: two of each are implemented")
        self.eps, self.scale = float(spec["eps"]), float(spec["scale"])

    @property
    def graph_safe(self) -> bool:
        return all(m.graph_safe for m in self.mixers)

    def weight_specs(self, present=None):
        return [s for m in self.mixers for s in m.weight_specs(present)] + \
               [TensorSpec(n, (self.hidden_size,), "vector", "ones") for n in self.norm_names]

    def shapes_from(self, shape_of) -> None:
        for m in self.mixers:
            if hasattr(m, "shapes_from"):
                m.shapes_from(shape_of)

    def bind(self, read, runtime):
        self.runtime = runtime
        for m in self.mixers:
            m.bind(read, runtime)
        self.w_norms = [runtime.vector(read(n)) for n in self.norm_names]

    def cache_need(self):
        return tuple(m.cache_need() for m in self.mixers)

    def forward(self, x, step, cache, writes_cache: bool = True):
        first = self.mixers[0].forward(x, step, cache[0], writes_cache)
        with self.runtime.branch(2):        # both may still be partial sums when they are normed
            second = self.mixers[1].forward(x, step, cache[1], writes_cache)
        out = torch.empty(x.shape[0], self.hidden_size, dtype=torch.float32, device=x.device)
        return ops.normed_sum(first, second, *self.w_norms, self.eps, self.scale, out)
