"""Gifopel on the GPU against the plain implementation (`tests/plain_gifopel.py`): every mechanism alone as a part with a
cache of its own, then whole models through the step function, the scheduler and the replay program.

The tiny models (`tests/gifopel_configs.py`) differ from one another in every size and constant. Where random weights would
hide a fault (a key at a chunk's edge, a first token whose trace must last, the maximum's start at zero), weights or inputs are
set so that it shows, and the test first says so with the plain functions.

Tolerances as for the engine's other models: 32-bit within 1e-4 of a row's largest magnitude, bfloat16 within 3e-2.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import gifopel_configs as C
from tests import plain_gifopel as P
from tests.test_gpu_niralix import DEV, DT, ROOT, TOL, cuts, in_portions, rel, rt_of, run_schedule
from tests.test_gpu_parts import plain, reader, stepper

pytestmark = pytest.mark.gpu


def one_model(layers, width, eps=1e-5, ranks=(8, 8), seed=0):
    from tandemllm_b200.config import GifopelConfig
    cfg = {"architecture": "Gifopel", "vocab": 11, "width": width, "norm": {"eps": eps}, "layers": list(layers)}
    return GifopelConfig.from_dict(cfg).to_spec(), C.random_weights(cfg, ranks, seed)


def bound(part_spec, W, rt, width, prefix="l0.", family="mixer"):
    from tandemllm_b200.parts import make_part
    part = make_part(family, part_spec, prefix=prefix, hidden_size=width)
    if hasattr(part, "shapes_from"):
        part.shapes_from(lambda n: tuple(W[n].shape) if n in W else None)
    part.bind(reader(W), rt)
    return part


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width,E", [(9, 44, 0), (3, 328, 20), (300, 1000, 6), (9, 2052, 20), (1500, 256, 40), (70, 2048, 32), (5, 4100, 3)])
def test_the_norm_kernel_adds_two_branches_and_writes_two_norms(dtype, rows, width, E):
    from tandemllm_b200.kernels import ops
    g = torch.Generator().manual_seed(width + rows)
    x, a, b = (torch.randn(rows, width, generator=g) for _ in range(3))
    w1, w2 = (1 + 0.2 * torch.randn(width, generator=g) for _ in range(2))
    tol = 2e-5 if dtype == "float32" else 1e-2
    k = 3
    # the second branch as a routed layer left it: three rows a token in some order, weighed
    pos = torch.randperm(rows * k, generator=g).to(torch.int32)
    wts, rows_e = torch.rand(rows, k, generator=g), torch.randn(rows * k, width, generator=g)
    ids = torch.stack([torch.randperm(8, generator=g)[:k] for _ in range(rows)]).to(torch.int32)
    routed = (wts[:, :, None] * rows_e[pos.long()].view(rows, k, width)).sum(1)
    experts = ops.ExpertRows(rows_e.to(DEV), pos.to(DEV), ids.to(DEV), wts.to(DEV))
    parts_a = ops.PartialSums(torch.stack([0.25 * a, 0.75 * a]).to(DEV).contiguous(), 2, rows, width)
    parts_b = ops.PartialSums(torch.stack([0.5 * b, 0.125 * b, 0.375 * b]).to(DEV).contiguous(), 3, rows, width)
    router = 0.3 * torch.randn(E, width, generator=g) if E else None
    bias = torch.randn(E, generator=g) if E else None
    for first, second, added in ((a.to(DEV), b.to(DEV), a + b), (parts_a, parts_b, a + b), (parts_a, experts, a + routed),
                                 (a.to(DEV), None, a), (None, None, 0 * a), (None, experts, routed)):
        res = x.to(DEV)
        out, out2 = (torch.full((rows, width), 9.0, dtype=DT[dtype], device=DEV) for _ in range(2))
        route = None
        if E:
            top = min(3, E)
            route = {"weight": router.to(DEV), "bias": bias.to(DEV), "k": top, "normalize": True, "scoring": "chosen_softmax",
                     "floor": 0.0, "scale": 1.0, "ids": torch.empty(rows, top, dtype=torch.int32, device=DEV),
                     "wts": torch.empty(rows, top, device=DEV)}
        delta = ops.BranchSum(first, second) if second is not None or first is None else first
        ops.add_rmsnorm_pair(res, delta, w1.to(DEV), 1e-5, out, w2.to(DEV), out2, None, route)
        new = (x + added).double().numpy()
        n2 = P.plain_norm(new, w2.double().numpy(), 1e-5)
        assert rel(res, new) < 2e-6
        assert rel(out.float(), P.plain_norm(new, w1.double().numpy(), 1e-5)) < tol and rel(out2.float(), n2) < tol
        if E:
            # the router reads the second norm's unrounded rows; the bias is part of the logits
            z = n2 @ router.double().numpy().T + bias.double().numpy()
            order = np.argsort(-z, axis=-1, kind="stable")[:, :top]
            srt = np.sort(z, axis=-1)[:, ::-1]
            clear = (srt[:, top - 1] - srt[:, top] > 1e-4) if top < E else np.ones(rows, bool)
            got = route["ids"].cpu().numpy()
            assert clear.mean() > 0.9 and (np.sort(got, -1) == np.sort(order, -1))[clear].all()
            want = P.softmax(np.take_along_axis(z, got.astype(np.int64), -1))
            assert np.abs(route["wts"].cpu().numpy() - want)[clear].max() < 1e-4
    # the model's last norm: some rows of the sum, the residual left as it was
    res, gather = x.to(DEV), torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
    out = torch.empty(2, width, dtype=DT[dtype], device=DEV)
    ops.add_rmsnorm(res, ops.BranchSum(parts_a, experts), w1.to(DEV), 1e-5, out, gather)
    assert torch.equal(res.cpu(), x)
    assert rel(out.float(), P.plain_norm((x + a + routed).double().numpy(), w1.double().numpy(), 1e-5)[[rows - 1, 0]]) < tol


@pytest.mark.parametrize("rows,width", [(1, 44), (37, 1000), (9, 4096), (5, 2052)])
def test_two_branches_are_normed_each_on_its_own_and_averaged(rows, width):
    from tandemllm_b200.kernels import ops
    g = torch.Generator().manual_seed(width)
    a, b = torch.randn(rows, width, generator=g), 30 * torch.randn(rows, width, generator=g)
    wa, wb = (1 + 0.2 * torch.randn(width, generator=g) for _ in range(2))
    want = 0.5 * (P.plain_norm(a.double().numpy(), wa.double().numpy(), 1e-3) + P.plain_norm(b.double().numpy(), wb.double().numpy(), 1e-3))
    parts = ops.PartialSums(torch.stack([0.5 * b, 0.25 * b, 0.25 * b]).to(DEV).contiguous(), 3, rows, width)
    for second in (b.to(DEV), parts):
        out = torch.empty(rows, width, device=DEV)
        ops.normed_sum(a.to(DEV), second, wa.to(DEV), wb.to(DEV), 1e-3, 0.5, out)
        assert rel(out, want) < 1e-5


def two_requests_and_a_reused_slot(part, xa, xb, want_a, want_b, state_of_b, rt, dtype, tol):
    """Request a in portions down to single tokens, b beside it whole in one of them; then a newcomer in b's old slot; then a
    whole, and token by token."""
    T = xa.shape[0]
    cache, step = stepper([part.cache_need()], rt, requests=2)
    got_a, at = [], 0
    for i, n in enumerate(cuts(T, [1, 2, 9, 1, 17, 3, 64, 2])):
        ctx = step([("a", n)] + ([("b", xb.shape[0])] if i == 2 else []))
        rows = torch.cat([xa[at:at + n]] + ([xb] if i == 2 else [])).to(DT[dtype]).to(DEV)
        out = plain(part.forward(rows, ctx, cache.site_cache[0]))
        got_a.append(out[:n])
        if i == 2:
            assert rel(out[n:], want_b) < tol
            state_of_b(cache.site_cache[0].state[cache._slot_of["b"]])
            cache.free("b")
        at += n
    assert rel(torch.cat(got_a), want_a) < tol
    ctx = step([("c", xb.shape[0])])         # a newcomer in b's old slot starts from zero
    assert rel(plain(part.forward(xb.to(DT[dtype]).to(DEV), ctx, cache.site_cache[0])), want_b) < tol
    cache, step = stepper([part.cache_need()], rt, requests=2)
    assert rel(in_portions(part, xa.to(DT[dtype]), cache, step, [T]), want_a) < tol
    cache, step = stepper([part.cache_need()], rt, requests=2)
    assert rel(in_portions(part, xa[:40].to(DT[dtype]), cache, step, [1] * 40), want_a[:40]) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("channel", [True, False])
@pytest.mark.parametrize("heads,kv,dim,vdim,taps,ranks", [(4, 2, 6, 10, 3, (5, 7)), (2, 2, 64, 64, 4, (16, 16)), (6, 2, 40, 72, 2, (12, 8)),
                                                          (1, 1, 2, 3, 1, (1, 1)), (2, 1, 128, 128, 5, (24, 8)), (3, 1, 130, 20, 4, (8, 40))])
def test_the_gated_delta_rule_in_portions_in_slots_used_again_and_a_first_token_that_lasts(dtype, channel, heads, kv, dim, vdim, taps, ranks):
    width, T = 40, 220
    sizes = (heads, kv, dim, vdim, taps)
    layer = C.delta(*sizes) if channel else C.parallel((1, 1, 16, 16, 0.2, None, None), sizes)
    m = layer["mixer"] if channel else layer["mixer"]["right"]
    pre = "l0.mix." if channel else "l0.mix.right."
    spec, W = one_model([layer], width, eps=3e-5, ranks=ranks, seed=dim + vdim)
    W[pre + "dt_bias"] = (W[pre + "dt_bias"] - 4.0).to(torch.bfloat16).float()        # decays of 0.98 to 0.9999
    W[pre + "b"] = W[pre + "b"] * 0.2
    w64 = {k: v.double().numpy() for k, v in W.items()}
    fn = P.mixer_channel_delta if channel else P.mixer_head_delta
    g = torch.Generator().manual_seed(3)
    xa = (torch.randn(T, width, generator=g) * 0.7).to(DT[dtype]).float()
    xb = torch.randn(33, width, generator=g).to(DT[dtype]).float()
    want_a = fn(xa.double().numpy(), m, w64, pre, 3e-5)
    want_b, S_b = fn(xb.double().numpy(), m, w64, pre, 3e-5, return_state=True)
    x2 = xa.clone()
    x2[0] = -xa[0] * 3
    changed = fn(x2.double().numpy(), m, w64, pre, 3e-5)
    if dim >= 6:
        assert rel(changed[taps + 20:taps + 60], want_a[taps + 20:taps + 60]) > 1e-3, \
            "the first token must still show long after the convolution for this test to say anything"
    rt = rt_of(dtype)
    part_spec = spec.layers[0].mixer if channel else spec.layers[0].mixer["mixers"][1]
    part = bound(part_spec, W, rt, width)
    tol = TOL[dtype] * (4 if dtype == "bfloat16" else 1)

    def state_of_b(slot):
        got = slot[part.state_at:part.state_at + heads * vdim * dim].view(heads, vdim, dim).transpose(1, 2)
        assert rel(got.reshape(heads, -1), S_b.reshape(heads, -1)) < (1e-4 if dtype == "float32" else 4e-2)

    two_requests_and_a_reused_slot(part, xa, xb, want_a, want_b, state_of_b, rt, dtype, tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim,cap,i_shift", [(3, 8, 12, 5.0, 0.0), (2, 64, 64, 15.0, -6.0), (1, 1, 1, 2.0, 0.0), (2, 130, 20, 30.0, 8.0),
                                                        (5, 24, 96, 8.0, -3.0), (4, 128, 127, 12.0, 0.0)])
def test_the_matrix_memory_in_portions_in_slots_used_again_and_its_maximum_from_zero(dtype, heads, dim, vdim, cap, i_shift):
    width, T = 40, 220
    layer = C.memory(heads, dim, vdim, cap)
    spec, W = one_model([layer], width, eps=3e-5, seed=dim + vdim)
    m, pre = layer["mixer"], "l0.mix."
    W[pre + "i.b"] = (W[pre + "i.b"] + i_shift).to(torch.bfloat16).float()
    W[pre + "i"] = W[pre + "i"] * 2
    W[pre + "f.b"] = (W[pre + "f.b"] + 2.0).to(torch.bfloat16).float()
    w64 = {k: v.double().numpy() for k, v in W.items()}
    g = torch.Generator().manual_seed(4)
    xa = (torch.randn(T, width, generator=g) * 0.7).to(DT[dtype]).float()
    xb = torch.randn(33, width, generator=g).to(DT[dtype]).float()
    want_a = P.mixer_mlstm(xa.double().numpy(), m, w64, pre, 3e-5)
    want_b, (S_b, n_b, m_b) = P.mixer_mlstm(xb.double().numpy(), m, w64, pre, 3e-5, return_state=True)
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer, W, rt, width)
    tol = TOL[dtype] * (4 if dtype == "bfloat16" else 1)

    def state_of_b(slot):
        exact = 1e-4 if dtype == "float32" else 4e-2
        assert rel(slot[:heads].view(1, -1), m_b.reshape(1, -1)) < exact
        got = slot[part.state_at:part.state_at + heads * (vdim + 1) * dim].view(heads, vdim + 1, dim)
        assert rel(got[:, :vdim].transpose(1, 2).reshape(heads, -1), S_b.reshape(heads, -1)) < exact
        assert rel(got[:, vdim], n_b) < exact

    if dim == 1 and dtype == "bfloat16":
        tol *= 3            # a head of one value is normed to +-1 and its numerator may be tiny
    two_requests_and_a_reused_slot(part, xa, xb, want_a, want_b, state_of_b, rt, dtype, tol)
    if i_shift < -4:
        # with tiny input gates the floor exp(-m) of a maximum that starts at zero decides: one that starts at minus infinity
        # would give another answer
        i, f = P.memory_gates(xa.double().numpy(), m, w64, pre)
        assert (np.cumsum(f, 0)[:5] > i[:5]).all()


def spiked(x, W, pre, m, pairs, strength):
    """x and W changed so that in every head row r's score with key j stands out for each (r, j) of `pairs`: input columns are set
    aside, one a pair drives the last entry of every query head from r, and of every key head from j."""
    x, W = x.clone(), {k: v.clone() for k, v in W.items()}
    D = m["dim"]
    x[:, 0] = 0
    x[:, 1] = 0
    for name, col, heads in ((pre + "q", 0, m["heads"]), (pre + "k", 1, m["kv_heads"])):
        W[name][:, [0, 1]] = 0
        for h in range(heads):
            W[name][h * D + D - 1, col] = 1.0
    for r, j in pairs:
        x[r, 0] = strength
        x[j, 1] = strength
    for w in ("q.norm", "k.norm"):
        W[pre + w][D - 1] = 2.0
    return x, W


LEFT_CASES = {
    # heads, kv, dim, vdim, scale, rot, chunk
    "narrow values, half a head turned": ((4, 2, 12, 10, 0.4, (500.0, 6), 24)),
    "tensor-core sizes": ((8, 2, 64, 64, 0.14, (100000.0, 32), 100)),
    "tensor-core sizes, chunks of pages": ((4, 1, 64, 128, 0.125, (10000.0, 64), 128)),
    "keys of 128, all turned": ((2, 1, 128, 64, 0.09, (1e6, 128), 75)),
    "heads of 128 both": ((6, 2, 128, 128, 0.09, (10000.0, 64), 64)),
    "one head, chunks of 7": ((1, 1, 8, 24, 0.5, (100.0, 2), 7)),
    "no rotation, no chunks": ((3, 3, 33, 5, 0.2, None, None)),
    "chunks of one": ((2, 1, 64, 64, 0.2, (100.0, 8), 1)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(LEFT_CASES))
def test_attention_within_chunks_reaches_their_first_key_and_no_further(case, dtype):
    """Rows late in a chunk whose scores stand out with the chunk's first key (just inside) and with the last key of the chunk
    before (just outside). In portions across pages' and chunks' edges and token by token; with sinks that matter."""
    sizes = LEFT_CASES[case]
    m = C.left_sizes(*sizes)
    chunk = sizes[6] or 1000
    width, T = 48, 230
    spec, W = one_model([C.parallel(sizes, (1, 1, 4, 4, 2))], width, seed=sizes[2] + sizes[3])
    pre = "l0.mix.left."
    g = torch.Generator().manual_seed(5)
    x = torch.randn(T, width, generator=g).to(DT[dtype]).float()
    # row `inside` with its chunk's first key; row `outside` with the key just before its chunk
    start = chunk * ((T - 3) // chunk)
    inside = min(T - 1, start + chunk - 1)
    s2 = max(0, start - chunk)
    pairs = [(inside, start)]
    outside = None
    if chunk > 1 and s2 > 0:
        outside = start - 1
        pairs.append((outside, s2 - 1))
    x, W = spiked(x, W, pre, m, pairs, 8.0)
    W[pre + "sink"] = torch.linspace(-2.0, 3.0, sizes[0]) if sizes[0] > 1 else torch.tensor([1.0])
    w64 = {k: v.double().numpy() for k, v in W.items()}
    n64 = x.double().numpy()
    want = P.mixer_chunked_attention(n64, m, w64, pre, 1e-5)
    if chunk > 1:       # a chunk one shorter or one longer, or no sink, is another answer
        short = P.mixer_chunked_attention(n64[start + 1:], dict(m, mask=None), w64, pre, 1e-5)
        assert m.get("mask") is None or rel(short[inside - start - 1:inside - start], want[inside:inside + 1]) > 0.05
        if outside is not None:
            longer = P.mixer_chunked_attention(n64[s2 - 1:start], dict(m, mask=None), w64, pre, 1e-5)
            assert rel(longer[-1:], want[outside:outside + 1]) > 0.05
    no_sink = dict(w64)
    no_sink[pre + "sink"] = np.full(sizes[0], -1e9)
    assert rel(P.mixer_chunked_attention(n64, m, no_sink, pre, 1e-5), want) > 0.05
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer["mixers"][0], W, rt, width)
    assert part.chunk == sizes[6] and part.gate_heads and part.flex
    tol = TOL[dtype] * (2 if dtype == "bfloat16" else 1)
    for cut in ([T], [7, 2, 33, 3, 16, 5], [180] + [1] * 50):
        cache, step = stepper([part.cache_need()], rt, requests=2)
        assert rel(in_portions(part, x.to(DT[dtype]), cache, step, cuts(T, cut)), want) < tol, cut
        if sizes[6] and sizes[6] < 100:
            assert any(p < 0 for p in cache.table(0, "r"))          # pages of chunks that are over went back


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,k,ff,rows,width", [(5, 2, 24, 37, 72), (8, 3, 64, 300, 128), (1, 1, 40, 5, 72), (4, 4, 16, 1, 72), (24, 5, 48, 20, 72),
                                               (16, 4, 64, 8, 256), (16, 4, 128, 40, 256), (16, 4, 128, 700, 256), (32, 2, 64, 3000, 64)])
def test_ungated_experts_are_weighed_by_the_softmax_over_the_chosen(dtype, E, k, ff, rows, width):
    spec, W = one_model([C.memory(1, 8, 8, 2.0, ff=(E, k, ff))], width, seed=E + k)
    rt = rt_of(dtype)
    ffp = bound(spec.layers[0].feed_forward, W, rt, width, family="feed_forward")
    from tandemllm_b200.parts import make_part
    n1 = make_part("norm", spec.layers[0].mixer_norm, prefix="l0.", size=width)
    n2 = make_part("norm", spec.layers[0].feed_forward_norm, prefix="l0.", size=width)
    n1.bind(reader(W), rt)
    n2.bind(reader(W), rt)
    g = torch.Generator().manual_seed(8)
    x = torch.randn(rows, width, generator=g)
    w64 = {k_: v.double().numpy() for k_, v in W.items()}
    route = ffp.router_args(rows, torch.device(DEV))
    _, fed_rows = n1.add_two_norms(x.to(DEV), None, n2, route)
    out = plain(ffp.forward(fed_rows, None, routing=(route["ids"], route["wts"])))
    n = P.plain_norm(x.double().numpy(), w64["l0.norm2"], 1e-5)
    z = P.router_logits(n, w64, "l0.mlp.")
    fed = torch.from_numpy(n).to(DT[dtype]).double().numpy()
    want = P.routed_experts(fed, spec_mlp(E, k, ff), w64, "l0.mlp.", logits=z)
    srt = np.sort(z, axis=-1)[:, ::-1]
    clear = (srt[:, k - 1] - srt[:, k] > 1e-4) if k < E else np.ones(rows, bool)
    assert clear.sum() >= max(1, int(0.9 * rows))
    assert rel(out[torch.from_numpy(clear)], want[clear]) < TOL[dtype] * (3 if dtype == "bfloat16" else 1)


def spec_mlp(E, k, ff):
    return {"kind": "moe", "router": {"experts": E, "top": k}, "expert": {"ff": ff}}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_chosen_share_the_weight_even_where_all_logits_are_far_apart(dtype):
    """Logits hundreds apart: the second chosen expert's weight is 0 to 32-bit, the choice still goes by the logits."""
    from tandemllm_b200.kernels import ops
    E, k = 40, 3
    z = torch.stack([torch.linspace(-900, 0, E), torch.linspace(0, -900, E), torch.full((E,), -500.0)])
    z[2, 7], z[2, 30] = -499.0, -498.0
    ids = torch.empty(3, k, dtype=torch.int32, device=DEV)
    wts = torch.empty(3, k, device=DEV)
    ops.router_topk(z.to(DEV), None, k, True, 0.0, 1.0, ids, wts, "chosen_softmax")
    assert ids.cpu().tolist() == [[39, 38, 37], [0, 1, 2], [30, 7, 0]]
    want = P.softmax(np.take_along_axis(z.double().numpy(), ids.cpu().long().numpy(), -1))
    assert np.allclose(wts.cpu().numpy(), want, atol=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("left,right", [((4, 2, 12, 10, 0.4, (500.0, 6), 24), (4, 2, 6, 10, 3)), ((8, 4, 64, 64, 0.14, (1e5, 32), 40), (4, 4, 64, 64, 4))])
def test_two_mixers_side_by_side_averaged_behind_their_norms(dtype, left, right):
    width, T = 96, 130
    spec, W = one_model([C.parallel(left, right)], width, seed=left[2])
    w64 = {k: v.double().numpy() for k, v in W.items()}
    x = torch.randn(T, width, generator=torch.Generator().manual_seed(6)).to(DT[dtype]).float()
    want = P.mixer_parallel(x.double().numpy(), {"left": C.left_sizes(*left), "right": C.delta_sizes(*right)}, w64, "l0.mix.", 1e-5)
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer, W, rt, width)
    for cut in ([T], [7, 2, 33, 3], [90] + [1] * 40):
        cache, step = stepper([part.cache_need()], rt, requests=2)
        assert rel(in_portions(part, x.to(DT[dtype]), cache, step, cuts(T, cut)), want) < TOL[dtype] * (2 if dtype == "bfloat16" else 1), cut


# ------------------------------------------------------------------------------------------ whole models
def engine_of(name, dtype, pages=64, parallel=4, cfg=None, W=None, **kw):
    from tandemllm_b200.config import GifopelConfig
    from tandemllm_b200.engine import Engine, EngineArgs
    from tandemllm_b200.weights.loader import DictWeights
    cfg = cfg or C.CONFIGS[name]
    W = W or C.weights(name, bf16_exact=True)
    spec = GifopelConfig.from_dict(cfg).to_spec()
    args = EngineArgs(dtype=dtype, max_len=4096, parallel=parallel, block_size=16, kv_blocks=pages, graph=False, **kw)
    return Engine._build(None, spec, DictWeights({k: v.clone() for k, v in W.items()}), args), cfg, W


def held_to_the_plain_model(engine, cfg, W, requests, schedule, dtype, what="", slack=1.0, outliers=0.0):
    """32-bit: every row within the tolerance. bfloat16: nine rows in ten (of all requests together) within the tolerance and every
    row within four times that (where a normed part of a dozen numbers happens to be small, its norm multiplies the rounding of
    what went in), but for rows one of whose routed layers chooses between two logits that rounding can exchange,
    and but for the share `outliers` of the others (a memory of one key divides by a sum that may all but cancel). A fault moves a
    row by its own size."""
    got = run_schedule(engine, requests, schedule)
    rows, clear = [], []
    for r, toks in requests.items():
        margins = []
        want = torch.from_numpy(P.forward(cfg, W, toks, margins=margins))
        rows.append(((got[r].double() - want).abs() / want.abs().amax(dim=-1, keepdim=True).clamp_min(1e-30)).amax(dim=-1))
        clear.append(torch.from_numpy(np.min(margins, axis=0) > 0.06 * slack) if margins else torch.ones(len(toks), dtype=torch.bool))
        if dtype == "float32":
            assert float(rows[-1].max()) < slack * TOL[dtype], (what, r, float(rows[-1].max()))
    if dtype == "bfloat16":
        rows, clear = torch.cat(rows), torch.cat(clear)
        worst = float(rows[clear].quantile(1.0 - outliers)) if bool(clear.any()) else 0.0
        assert float(rows.quantile(0.9)) < slack * TOL[dtype] and worst < 4 * slack * TOL[dtype], \
            (what, float(rows.quantile(0.9)), worst, float(rows.max()), float(clear.double().mean()))
    return got


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["f1", "f2", "f3", "f4"])
def test_whole_prompts_decoding_and_portions_agree_with_the_plain_model(name, dtype):
    engine, cfg, W = engine_of(name, dtype)
    odd = 0.02 if name == "f3" else 0.0
    toks = C.tokens(name, 150, seed=3)
    reqs = {"a": toks}
    whole = held_to_the_plain_model(engine, cfg, W, reqs, [[("a", len(toks))]], dtype, "whole", outliers=odd)["a"]
    # the first tokens of a sequence alone
    held_to_the_plain_model(engine, cfg, W, {"a": toks[:3]}, [[("a", 1)], [("a", 1)], [("a", 1)]], dtype, "first tokens")
    # most of it at once, then token by token across pages' and chunks' edges
    held_to_the_plain_model(engine, cfg, W, reqs, [[("a", 60)]] + [[("a", 1)]] * 90, dtype, "decode", outliers=odd)
    # token by token from the very first
    held_to_the_plain_model(engine, cfg, W, {"a": toks[:70]}, [[("a", 1)]] * 70, dtype, "every token alone", outliers=odd)
    # portions of changing size, down to two tokens
    for sizes in ([2], [7, 2, 33, 3, 16, 5], [64, 2, 31]):
        got = held_to_the_plain_model(engine, cfg, W, reqs, [[("a", c)] for c in cuts(len(toks), sizes)], dtype,
                                      f"portions {sizes}", outliers=odd)["a"]
        if dtype == "float32":          # how the prompt was cut changes nothing beyond rounding
            assert rel(got, whole) < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["f1", "f4"])
def test_layer_by_layer(name, dtype):
    """The models cut off behind their first, second, ... layer: a fault shows at the first layer that has it."""
    full, W = C.CONFIGS[name], C.weights(name)
    toks = C.tokens(name, 40, seed=9)
    for n in range(1, len(full["layers"]) + 1):
        cfg = dict(full, layers=full["layers"][:n])
        keep = {k: v for k, v in W.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}
        engine, _, _ = engine_of(None, dtype, cfg=cfg, W=keep)
        held_to_the_plain_model(engine, cfg, keep, {"a": toks}, [[("a", 33)], [("a", 2)]] + [[("a", 1)]] * 5, dtype, f"{n} layers")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["f1", "f2", "f4"])
def test_unequal_requests_in_one_batch_on_pages_and_slots_that_are_used_again(name, dtype):
    """Seven requests of unequal length through four slots and a pool too small for all of them: portions beside single
    tokens, requests that pause, pages and state slots that come back and are taken again."""
    lengths = [90, 5, 47, 130, 1, 33, 64]
    reqs = {f"q{i}": C.tokens(name, n, seed=10 + i) for i, n in enumerate(lengths)}
    engine, cfg, W = engine_of(name, dtype, pages=24, parallel=4)
    rng = np.random.default_rng(0)
    at = {r: 0 for r in reqs}
    waiting, live, schedule = list(reqs), [], []
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for r in list(live):
            if len(live) > 1 and rng.random() < 0.2:
                continue                                    # left out of this step
            n = min(len(reqs[r]) - at[r], int(rng.choice([1, 1, 2, 3, 16, 29])))
            step.append((r, n))
            at[r] += n
            if at[r] == len(reqs[r]):
                live.remove(r)
        if step:
            schedule.append(step)
    got = held_to_the_plain_model(engine, cfg, W, reqs, schedule, dtype, "mixed")
    if dtype == "float32":
        # each request alone, whole: what else was in the batch changes nothing beyond rounding
        for r, toks in reqs.items():
            assert rel(got[r], run_schedule(engine, {r: toks}, [[(r, len(toks))]])[r]) < 4e-5, r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype):
    engine, cfg, W = engine_of("f2", dtype, pages=28)
    toks = C.tokens("f2", 330, seed=8)
    held_to_the_plain_model(engine, cfg, W, {"a": toks}, [[("a", 9)]] + [[("a", 1)]] * 321, dtype, "long decoding")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype, tmp_path):
    """A folder on disk (config.json chooses the architecture), `Engine.generate`, several requests at once, decode steps
    from CUDA graphs where the engine takes them."""
    from tandemllm_b200.engine import Engine, EngineArgs
    from tandemllm_b200.sampling import SamplingParams
    name = "f2"
    folder = C.write_folder(str(tmp_path / "m"), name)
    engine = Engine.from_folder(folder, EngineArgs(dtype=dtype, max_len=256, parallel=3, chunk_size=32, max_batched_tokens=64))
    assert engine.model.spec.architecture == "Gifopel" and engine.model.graph_safe
    prompts = [C.tokens(name, n, seed=40 + n) for n in (70, 3, 21, 45)]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    cfg, W = C.CONFIGS[name], C.weights(name, bf16_exact=True)
    for prompt, out in zip(prompts, outs):
        assert len(out) == 12
        text = list(prompt)
        for t in out:
            row = P.forward(cfg, W, text)[-1]
            assert float(row.max() - row[t]) <= (2e-3 if dtype == "float32" else 0.12) * float(np.abs(row).max())
            text.append(t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_folder(dtype, tmp_path):
    name = "f3"
    folder = C.write_folder(str(tmp_path / "m"), name)
    toks = {"x": C.tokens(name, 40, seed=1), "y": C.tokens(name, 19, seed=2)}
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks["x"][:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks["x"][25:], "want": [14]},
                                     {"id": "y", "tokens": toks["y"], "want": [18]}], "end": ["x", "y"]},
             {"step": 2, "entries": [{"id": "z", "tokens": toks["y"][:2], "want": []}], "end": ["z"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out",
                        str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    V = C.CONFIGS[name]["vocab"]
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(-1, V)
    b = np.fromfile(out / "1.f32", dtype="<f4").reshape(-1, V)
    cfg, W = C.CONFIGS[name], C.weights(name)
    wx, wy = P.forward(cfg, W, toks["x"]), P.forward(cfg, W, toks["y"])
    assert rel(a, wx[[0, 24]]) < TOL[dtype]
    assert rel(b, np.stack([wx[39], wy[18]])) < TOL[dtype]
    assert not (out / "2.f32").exists()


@pytest.mark.parametrize("seed", range(10))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_models_drawn_at_random(seed, dtype):
    cfg, ranks = C.random_config(seed)
    W = C.random_weights(cfg, ranks, 100 + seed)
    engine, cfg, W = engine_of(None, dtype, cfg=cfg, W=W, pages=32)
    g = torch.Generator().manual_seed(seed)
    toks = {r: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for r, n in (("a", 97), ("b", 30), ("c", 2))}
    schedule = [[("a", 40), ("b", 1)], [("a", 2), ("b", 17), ("c", 2)], [("a", 1), ("b", 1)], [("a", 31), ("b", 11)],
                [("a", 23)]]
    held_to_the_plain_model(engine, cfg, W, toks, schedule, dtype, f"random {seed}", slack=3.0 if dtype == "bfloat16" else 1.0,
                            outliers=0.015)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_command_line_writes_a_random_model_and_generates_from_it(dtype, tmp_path):
    """`random-weights` from a config.json of this design (a layer that runs another's tensors has none in the folder), then
    `generate` on the folder: greedy tokens that the plain model agrees with."""
    from tandemllm_b200.weights.safetensors_io import index_file, read_tensor
    cfg_path, folder, out = tmp_path / "config.json", tmp_path / "m", tmp_path / "out.json"
    cfg_path.write_text(json.dumps(C.F1))
    base = [sys.executable, "-m", "tandemllm_b200"]
    r = subprocess.run(base + ["random-weights", "--config", str(cfg_path), "--seed", "5", "--out", str(folder)], cwd=ROOT,
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    prompt = C.tokens("f1", 19, seed=6)
    r = subprocess.run(base + ["generate", "--model", str(folder), "--dtype", dtype, "--prompt-ids", ",".join(map(str, prompt)),
                               "--tokens", "8", "--json", str(out)], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = json.loads(out.read_text())["outputs"][0]
    assert len(got) == 8
    W = {k: read_tensor(v).double().numpy() for k, v in index_file(str(folder / "model.safetensors")).items()}
    assert not any(k.startswith("l3.") for k in W)
    text = list(prompt)
    for t in got:
        row = P.forward(C.F1, W, text)[-1]
        assert float(row.max() - row[t]) <= (2e-3 if dtype == "float32" else 0.12) * float(np.abs(row).max())
        text.append(t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_of_real_layer_widths(dtype):
    """Layer sizes of a model that would be served (width 1024, heads of 64 and 128, 16 experts), few layers and a small vocabulary:
    the products, attentions and scans run the forms they take at such sizes. A prompt in two portions, then decoding beside a
    second request."""
    cfg = {"architecture": "Gifopel", "vocab": 1000, "width": 1024, "norm": {"eps": 1e-6},
           "layers": [C.parallel((16, 4, 64, 64, 0.125, (500000.0, 64), 112), (16, 8, 64, 64, 4), ff=(16, 4, 256)),
                      C.delta(8, 4, 128, 128, 4, ff=1024), C.memory(8, 64, 128, 15.0, ff=(16, 4, 256))]}
    cfg["layers"].append(C.again(cfg["layers"], 1))
    W = C.random_weights(cfg, (64, 32), 77)
    engine, cfg, W = engine_of(None, dtype, cfg=cfg, W=W, pages=32)
    g = torch.Generator().manual_seed(9)
    toks = {r: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for r, n in (("a", 200), ("b", 70))}
    schedule = [[("a", 150)], [("a", 40), ("b", 64)]] + [[("a", 1), ("b", 1)]] * 6 + [[("a", 4)]]
    held_to_the_plain_model(engine, cfg, W, toks, schedule, dtype, "real widths")
