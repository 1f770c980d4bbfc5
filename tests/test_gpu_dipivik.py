"""Dipivik on the GPU against the plain implementation (`tests/plain_dipivik.py`): every mechanism alone as a part with a
cache of its own, then whole models through the step function, the scheduler and the replay program.

The tiny models (`tests/dipivik_configs.py`) differ from one another in every size and constant. Where random weights would
hide a fault (a key at a window's edge, a first token whose trace must last, a token pair), weights or inputs are set so that
it shows, and the test first says so with the plain functions.

Tolerances as for the engine's other models: 32-bit within 1e-4 of a row's largest magnitude, bfloat16 within 3e-2.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import dipivik_configs as C
from tests import plain_dipivik as P
from tests.test_gpu_niralix import DEV, DT, ROOT, TOL, cuts, in_portions, rel, rt_of, run_schedule
from tests.test_gpu_parts import plain, reader, stepper

pytestmark = pytest.mark.gpu


def one_model(layers, width, eps=1e-5, seed=0, **kw):
    from tandemllm_b200.config import DipivikConfig
    cfg = C.model(11, width, eps, layers, **kw)
    return DipivikConfig.from_dict(cfg).to_spec(), C.random_weights(cfg, seed)


def bound(part_spec, W, rt, width, prefix="l0.", family="mixer"):
    from tandemllm_b200.parts import make_part
    part = make_part(family, part_spec, prefix=prefix, hidden_size=width)
    part.bind(reader(W), rt)
    return part


def w64_of(W):
    return {k: v.double().numpy() for k, v in W.items()}


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("vocab,width,bigram", [(97, 44, (61, 5, 3)), (50, 1032, (1, 7, 7)), (300, 128, (4001, 1000003, 999)), (20, 8, (7, 0, 1))])
def test_token_pairs_across_portions_slots_and_first_tokens(dtype, vocab, width, bigram):
    """Exact in both precisions: two rows of the tables, added in 32-bit. Portions of one and two tokens beside longer ones, a slot
    that another request had before, and a request that is left out of steps in between."""
    from tandemllm_b200.kernels import ops
    from tandemllm_b200.parts.base import SlotNeed
    cfg = C.model(vocab, width, 1e-5, [], bigram=bigram)
    W = {k: v.to(torch.bfloat16) for k, v in C.random_weights(cfg, 1).items()}
    table, pairs = (W[k].to(DT[dtype]).to(DEV) for k in ("embed", "bigram"))
    rt = rt_of(dtype)
    cache, step = stepper([SlotNeed((1,), torch.int32, init=-1)], rt, requests=3)
    texts = {r: torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(n)).tolist() for r, n in
             (("a", 41), ("b", 9), ("c", 3), ("d", 12), ("e", 1))}
    b = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    want = {r: (W["embed"].float()[t] + W["bigram"].float()[P.bigram_rows(t, b)]) for r, t in texts.items()}
    at = {r: 0 for r in texts}
    for batch, gone in (([("a", 1), ("b", 2)], ""), ([("a", 2)], ""), ([("b", 1), ("c", 3), ("a", 17)], "c"), ([("d", 1), ("a", 1)], ""),
                        ([("b", 6), ("d", 11)], "bd"), ([("e", 1), ("a", 20)], "ea")):
        ctx = step(batch)
        toks = [t for r, n in batch for t in texts[r][at[r]:at[r] + n]]
        ctx.token_ids.copy_(torch.tensor(toks, dtype=torch.int32))
        out = torch.empty(len(toks), width, dtype=torch.float32, device=DEV)
        ops.embed_token_pairs(table, pairs, ctx, cache.site_cache[0].state, out, rt.status, bigram[1], bigram[2], 1.0)
        o = 0
        for r, n in batch:
            assert torch.equal(out[o:o + n].cpu(), want[r][at[r]:at[r] + n]), (r, at[r], n)
            o, at[r] = o + n, at[r] + n
        for r in gone:
            assert at[r] == len(texts[r])
            cache.free(r)
    assert int(rt.status.item()) == 0


RETENTION_CASES = [(3, 8, 6, (500.0, 6)), (2, 64, 64, (1e6, 64)), (3, 40, 72, (300.0, 4)), (1, 16, 16, None), (2, 128, 128, (1e4, 128)),
                   (2, 130, 20, (3000.0, 128)), (5, 32, 96, (1e6, 32)), (6, 2, 8, (10.0, 2)), (16, 64, 64, (1e6, 64))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,vdim,rot", RETENTION_CASES)
def test_retention_in_portions_in_slots_used_again_and_a_first_token_that_lasts(dtype, heads, dim, vdim, rot):
    """Two requests side by side, one whole and one in portions down to single tokens; a third request takes a slot that was
    given back and must find it zero; with decays near one the first token still shows hundreds of tokens later."""
    width, T = 40, 300
    layer = C.retention(heads, dim, vdim, rot, decay=[1.0 - 0.005 * 0.5 ** h for h in range(heads)])
    spec, W = one_model([layer], width, eps=3e-5, seed=dim + vdim)
    m, pre, w64 = layer["mixer"], "l0.mix.", w64_of(W)
    g = torch.Generator().manual_seed(3)
    xa = (torch.randn(T, width, generator=g) * 0.7).to(DT[dtype]).float()
    xa[0] *= 8
    xb = torch.randn(33, width, generator=g).to(DT[dtype]).float()
    want_a = P.mixer_retention(xa.double().numpy(), m, w64, pre, 3e-5)
    want_b, S_b = P.mixer_retention(xb.double().numpy(), m, w64, pre, 3e-5, return_state=True)
    x2 = xa.clone()
    x2[0] = xa[0].roll(1)
    assert rel(P.mixer_retention(x2.double().numpy(), m, w64, pre, 3e-5)[-1:], want_a[-1:]) > 1e-3, \
        "the first token must still show at the end for this test to say anything"
    if rot:
        assert rel(P.mixer_retention(xa.double().numpy(), {k: v for k, v in m.items() if k != "rot"}, w64, pre, 3e-5), want_a) > 0.05
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer, W, rt, width)
    tol = TOL[dtype]
    cache, step = stepper([part.cache_need()], rt, requests=2)
    got_a, at = [], 0
    for i, n in enumerate(cuts(T, [1, 2, 9, 1, 17, 3, 64, 2])):
        batch = [("a", n)] + ([("b", 33)] if i == 2 else [])
        ctx = step(batch)
        rows = torch.cat([xa[at:at + n]] + ([xb] if i == 2 else [])).to(DT[dtype]).to(DEV)
        out = plain(part.forward(rows, ctx, cache.site_cache[0]))
        got_a.append(out[:n])
        if i == 2:
            assert rel(out[n:], want_b) < tol
            slot = cache._slot_of["b"]
            assert rel(cache.site_cache[0].state[slot].reshape(heads, -1), S_b.reshape(heads, -1)) < 1e-4
            cache.free("b")
        at += n
    assert rel(torch.cat(got_a), want_a) < tol
    # a newcomer in b's old slot starts from zero
    ctx = step([("c", 33)])
    assert rel(plain(part.forward(xb.to(DT[dtype]).to(DEV), ctx, cache.site_cache[0])), want_b) < tol
    # the whole text at once, and token by token from the start
    cache, step = stepper([part.cache_need()], rt, requests=2)
    assert rel(in_portions(part, xa.to(DT[dtype]), cache, step, [T]), want_a) < tol
    cache, step = stepper([part.cache_need()], rt, requests=2)
    assert rel(in_portions(part, xa[:40].to(DT[dtype]), cache, step, [1] * 40), want_a[:40]) < tol


LATENT_CASES = {
    # heads, dim, rot_dim, vdim, kv_rank, q_rank, base, window
    "odd sizes": (3, 12, 6, 10, 20, 14, 700.0, 19),
    "tensor-core sizes": (4, 64, 32, 64, 64, 48, 1e4, 40),
    "a window of pages": (6, 48, 16, 64, 128, 72, 1e4, 64),
    "a window just past a page": (2, 32, 8, 128, 320, 40, 500.0, 33),
    "sixteen heads, a latent of 256": (16, 64, 32, 64, 256, 128, 1e4, 130),
    "a latent of 512": (8, 128, 64, 128, 512, 256, 1e4, 100),
    "one head": (1, 8, 16, 24, 16, 8, 100.0, 7),
    "two positions": (2, 8, 2, 8, 8, 8, 30.0, 2),
}


def spiked(x, W, m, rows, key, strength=8.0):
    """Rows `rows` ask loudly and row `key` answers loudly: input columns 0 and 1 (zero in every other row) feed one entry of the
    query's latent and one of the cached latent, which one entry of every head's unrotated query and key read and nothing else
    does, so that their score stands out by about 14 in front of the softmax."""
    W = {k: v.clone() for k, v in W.items()}
    p, H, D, R = "l0.mix.", m["heads"], m["dim"], m["rot_dim"]
    x = x.clone()
    x[:, :2] = 0
    x[list(rows), 0] = strength
    x[key, 1] = strength
    for name, col, up, step in (("dq", 0, "uq", D + R), ("dkv", 1, "uk", D)):
        W[p + name][0] = 0
        W[p + name][0, col] = 1.0
        W[p + name + ".norm"][0] = 1.0
        W[p + up][[h * step for h in range(H)]] = 0
        W[p + up][[h * step for h in range(H)], 0] = 1.0
    w = w64_of(W)
    n = x.double().numpy()
    qu, _ = P.latent_queries(n, m, w, p, 1e-5)
    c, _ = P.latent_keys(n, m, w, p, 1e-5)
    s = float(np.mean([qu[r, 0, 0] for r in rows]) * c[key, 0] * m["scale"])
    W[p + "uq"][[h * (D + R) for h in range(H)], 0] = torch.tensor(14.0 / s).to(torch.bfloat16).float()
    return x, W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(LATENT_CASES))
def test_latent_attention_sees_the_last_key_of_its_window_and_not_the_next(case, dtype):
    """One key that stands out, asked by the last row that sees it and by the next one, in prompts, in portions across pages' edges
    and decoded token by token."""
    H, D, R, VD, L, Q, base, window = LATENT_CASES[case]
    width, key = 56, 83
    T = key + window + 31
    layer = C.latent(H, D, R, VD, L, Q, 0.6 / (D + R) ** 0.5, base, window)
    m, pre = layer["mixer"], "l0.mix."
    spec, W = one_model([layer], width, seed=L + Q)
    inside, outside = key + window - 1, key + window
    x = torch.randn(T, width, generator=torch.Generator().manual_seed(6)).to(DT[dtype]).float()
    x, W = spiked(x, W, m, (inside, outside), key)
    w64, n64 = w64_of(W), x.double().numpy()
    want = P.mixer_latent_attention(n64, m, w64, pre, 1e-5)
    shorter = P.mixer_latent_attention(n64, dict(m, mask={"size": window - 1}), w64, pre, 1e-5)
    longer = P.mixer_latent_attention(n64, dict(m, mask={"size": window + 1}), w64, pre, 1e-5)
    assert rel(shorter[inside:inside + 1], want[inside:inside + 1]) > 0.2 and rel(longer[outside:outside + 1], want[outside:outside + 1]) > 0.2
    ungated = dict(w64)
    ungated[pre + "g"] = np.zeros((H, width))
    assert rel(P.mixer_latent_attention(n64, m, ungated, pre, 1e-5), want) > 0.05
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer, W, rt, width)
    assert part.halves and part.gate_heads
    tol = TOL[dtype] * (2 if dtype == "bfloat16" else 1)
    for sizes in ([T], [7, 2, 33, 3, 16, 5], [key + 2] + [1] * (T - key - 2)):
        cache, step = stepper([part.cache_need()], rt, requests=2)
        got = in_portions(part, x.to(DT[dtype]), cache, step, cuts(T, sizes))
        assert rel(got, want) < tol, sizes
        assert any(p < 0 for p in cache.table(0, "r"))              # pages behind the window went back


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rot,window", [(1000.0, None), (None, None), (None, 50)])
def test_latent_attention_over_all_keys_and_without_a_rotation(dtype, rot, window):
    layer = C.latent(4, 24, 8, 20, 40, 24, 0.5, rot, window)
    spec, W = one_model([layer], 56, seed=9)
    x = torch.randn(290, 56, generator=torch.Generator().manual_seed(6)).to(DT[dtype]).float()
    x, W = spiked(x, W, layer["mixer"], (288,), 3)
    want = P.mixer_latent_attention(x.double().numpy(), layer["mixer"], w64_of(W), "l0.mix.", 1e-5)
    rt = rt_of(dtype)
    part = bound(spec.layers[0].mixer, W, rt, 56)
    for sizes in ([290], [7, 2, 33, 3, 16, 5], [240] + [1] * 50):
        cache, step = stepper([part.cache_need()], rt, requests=2)
        assert rel(in_portions(part, x.to(DT[dtype]), cache, step, cuts(290, sizes)), want) < TOL[dtype] * (2 if dtype == "bfloat16" else 1), sizes


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,ff,rows", [(44, 52, 1), (44, 52, 37), (72, 40, 300), (128, 256, 1), (128, 256, 8), (128, 256, 40), (256, 192, 129),
                                           (1024, 512, 150), (1024, 2048, 600), (2048, 512, 20)])
def test_dense_feed_forward_with_biases_and_the_tanh_form_of_gelu(dtype, width, ff, rows):
    """Down products that stay in partial sums add the bias once; biases as large as the sums they are added to."""
    spec, W = one_model([C.retention(1, 8, 8, None, ff=ff)], width, seed=ff)
    for k in ("gate.b", "up.b", "down.b"):
        W["l0.mlp." + k] *= 3
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(8)).to(DT[dtype]).float()
    w64 = w64_of(W)
    want = P.dense_gated(x.double().numpy(), w64, "l0.mlp.")
    for k in ("gate.b", "up.b", "down.b"):
        assert rel(P.dense_gated(x.double().numpy(), dict(w64, **{"l0.mlp." + k: 0 * w64["l0.mlp." + k]}), "l0.mlp."), want) > 0.1
    part = bound(spec.layers[0].feed_forward, W, rt_of(dtype), width, family="feed_forward")
    assert rel(plain(part.forward(x.to(DT[dtype]).to(DEV), None)), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_tanh_form_of_gelu_as_a_plain_activation(dtype):
    from tandemllm_b200.kernels import ops
    z = torch.cat([torch.linspace(-12, 12, 4001), torch.tensor([-1e4, -300.0, 300.0, 1e4])]).to(DT[dtype])
    out = torch.empty_like(z, device=DEV)
    ops.activation(z.to(DEV), out, ops.ACTIVATIONS["gelu_tanh"])
    want = torch.from_numpy(P.gelu_tanh(z.double().numpy()))
    assert torch.allclose(out.double().cpu(), want, rtol=2e-6 if dtype == "float32" else 8e-3, atol=2e-7)


EXPERT_CASES = [(5, 2, 24, 37, 72, 20), (8, 3, 64, 300, 128, 128), (1, 1, 40, 5, 72, None), (4, 4, 16, 1, 72, 24), (24, 5, 48, 20, 72, 40),
                (16, 1, 64, 8, 256, 96), (16, 4, 64, 7, 256, 64), (16, 4, 64, 15, 256, 64), (16, 4, 128, 40, 256, 128), (64, 2, 64, 40, 128, 64),
                (16, 4, 128, 700, 256, None), (32, 2, 64, 3000, 64, 64), (8, 2, 256, 1500, 512, 256)]


def routed_and_shared(W, ffp, norm, x, rt):
    """The feed-forward of `ffp` behind the norm that runs its router, and the same from the plain functions with the rows that the
    experts read in the compute dtype. (The rows whose choice is no close call.)"""
    width, rows = x.shape[1], x.shape[0]
    route = ffp.router_args(rows, torch.device(DEV))
    fed_rows = norm.add_norm(x.to(DEV), None, route=route)
    out = plain(ffp.forward(fed_rows, None, routing=(route["ids"], route["wts"])))
    w = w64_of(W)
    n = P.plain_norm(x.double().numpy(), w["l0.norm1"], 1e-5)
    return out, n, P.sigmoid(n @ w["l0.mlp.router"].T), torch.from_numpy(n).to(rt.dtype).double().numpy(), w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,k,ff,rows,width,shared", EXPERT_CASES)
def test_experts_weighed_at_their_input_and_a_shared_one(dtype, E, k, ff, rows, width, shared):
    spec, W = one_model([C.retention(1, 8, 8, None, ff=(E, k, ff, shared))], width, seed=E + k)
    W["l0.mlp.router"] *= 0.5               # scores that are not close to one
    rt = rt_of(dtype)
    ffp = bound(spec.layers[0].feed_forward, W, rt, width, family="feed_forward")
    from tandemllm_b200.parts import make_part
    norm = make_part("norm", spec.layers[0].mixer_norm, prefix="l0.", size=width)
    norm.bind(reader(W), rt)
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(8))
    out, n, s, fed, w64 = routed_and_shared(W, ffp, norm, x, rt)
    mlp = C.mlp((E, k, ff, shared))
    want = P.routed_experts(fed, mlp, w64, "l0.mlp.", scores=s)
    outside = np.zeros_like(want)
    for t in range(min(rows, 4)):
        for e in np.argsort(-s[t], kind="stable")[:k]:
            outside[t] += s[t, e] * P.expert(fed[t:t + 1], w64, f"l0.mlp.e{e}.")[0]
    assert rel(outside[:4], want[:4]) > 0.05        # the weight behind the expert would be another answer
    if shared:
        want = want + P.expert(fed, w64, "l0.mlp.shared.")
    z = np.sort(np.log(s / (1 - s)), axis=-1)[:, ::-1]
    clear = (z[:, k - 1] - z[:, k] > 1e-4) if k < E else np.ones(rows, bool)
    assert clear.sum() >= max(1, int(0.9 * rows))
    assert rel(out[torch.from_numpy(clear)], want[clear]) < TOL[dtype]


@pytest.mark.parametrize("product", ["pair", "single"])
def test_experts_weighed_at_their_input_in_every_form_of_the_grouped_product(product):
    """bfloat16: 18 rows an expert up to 190, on the swapped tcgen05 kernel, on pairs of SMs two and one an SM, and on the persistent
    kernel that stands behind `PROMPT_PRODUCT` single."""
    from tandemllm_b200.kernels import tensorcore
    from tandemllm_b200.parts import make_part
    before = tensorcore.PROMPT_PRODUCT
    tensorcore.PROMPT_PRODUCT = product
    try:
        for rows in (36, 150, 380):
            spec, W = one_model([C.retention(1, 8, 8, None, ff=(4, 2, 136, 72))], 264, seed=rows)
            rt = rt_of("bfloat16")
            ffp = bound(spec.layers[0].feed_forward, W, rt, 264, family="feed_forward")
            norm = make_part("norm", spec.layers[0].mixer_norm, prefix="l0.", size=264)
            norm.bind(reader(W), rt)
            x = torch.randn(rows, 264, generator=torch.Generator().manual_seed(rows))
            out, n, s, fed, w64 = routed_and_shared(W, ffp, norm, x, rt)
            want = P.routed_experts(fed, C.mlp((4, 2, 136, 72)), w64, "l0.mlp.", scores=s) + P.expert(fed, w64, "l0.mlp.shared.")
            z = np.sort(np.log(s / (1 - s)), axis=-1)[:, ::-1]
            clear = z[:, 1] - z[:, 2] > 1e-4
            assert rel(out[torch.from_numpy(clear)], want[clear]) < TOL["bfloat16"], rows
    finally:
        tensorcore.PROMPT_PRODUCT = before


@pytest.mark.parametrize("rows", [20, 40, 60])
def test_a_mixer_a_shared_and_a_routed_part_keep_their_partial_sums_apart(rows):
    """bfloat16 at sizes where the routed down product, the shared expert's down product and the mixer's out projection are all left
    in partial sums that the next norm adds: a whole layer and the norm behind it against the plain functions."""
    from tandemllm_b200.parts.block import Layer
    width = 512
    layer = C.retention(4, 64, 64, None, ff=(64, 2, 512, 1024))
    spec, W = one_model([layer], width, seed=4)
    rt = rt_of("bfloat16")
    built = Layer(spec.layers[0], width)
    built.bind(reader(W), rt)
    cache, step = stepper([built.mixer.cache_need()], rt, requests=1)
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(8))
    w64 = w64_of(W)
    n = torch.from_numpy(P.plain_norm(x.double().numpy(), w64["l0.norm1"], 1e-5)).to(torch.bfloat16).double().numpy()
    want = x.double().numpy() + P.mixer_retention(n, layer["mixer"], w64, "l0.mix.", 1e-5) + P.feed_forward(n, layer["mlp"], w64, "l0.mlp.")
    residual = x.to(DEV)
    left = built.run(residual, None, step([("r", rows)]), cache.site_cache[0])
    rms = built.mixer_norm.add_norm(residual, left)
    z = np.sort(n @ w64["l0.mlp.router"].T, axis=-1)[:, ::-1]
    clear = torch.from_numpy(z[:, 1] - z[:, 2] > 0.03)
    assert int(clear.sum()) > rows // 2
    assert rel(residual[clear.to(DEV)], want[clear.numpy()]) < 1.5e-2
    assert rel(rms[clear.to(DEV)].float(), P.plain_norm(want, w64["l0.norm1"], 1e-5)[clear.numpy()]) < 2e-2


# ------------------------------------------------------------------------------------------ whole models
def engine_of(name, dtype, pages=64, parallel=4, cfg=None, W=None, graph=False, **kw):
    from tandemllm_b200.config import DipivikConfig
    from tandemllm_b200.engine import Engine, EngineArgs
    from tandemllm_b200.weights.loader import DictWeights
    cfg = cfg or C.CONFIGS[name]
    W = W or C.weights(name, bf16_exact=True)
    spec = DipivikConfig.from_dict(cfg).to_spec()
    args = EngineArgs(dtype=dtype, parallel=parallel, block_size=16, kv_blocks=pages, graph=graph, **dict({"max_len": 4096}, **kw))
    return Engine._build(None, spec, DictWeights({k: v.clone() for k, v in W.items()}), args), cfg, W


def held_to_the_plain_model(engine, cfg, W, requests, schedule, dtype, what="", slack=1.0, outliers=0.0):
    """32-bit: every row within the tolerance. bfloat16: nine rows in ten (of all requests together) within the tolerance and every
    row within four times that (where a normed head of a dozen numbers happens to be small, its norm multiplies the rounding of
    what went in), but for rows one of whose routed layers chooses between two scores that rounding can exchange, and but for
    the share `outliers` of the others. A fault moves a row by its own size."""
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
@pytest.mark.parametrize("name", ["d1", "d2", "d3", "d4"])
def test_whole_prompts_decoding_and_portions_agree_with_the_plain_model(name, dtype):
    engine, cfg, W = engine_of(name, dtype)
    toks = C.tokens(name, 150, seed=3)
    reqs = {"a": toks}
    whole = held_to_the_plain_model(engine, cfg, W, reqs, [[("a", len(toks))]], dtype, "whole")["a"]
    # the first tokens of a sequence alone
    held_to_the_plain_model(engine, cfg, W, {"a": toks[:3]}, [[("a", 1)], [("a", 1)], [("a", 1)]], dtype, "first tokens")
    # most of it at once, then token by token across pages' and windows' edges
    held_to_the_plain_model(engine, cfg, W, reqs, [[("a", 60)]] + [[("a", 1)]] * 90, dtype, "decode")
    # token by token from the very first
    held_to_the_plain_model(engine, cfg, W, {"a": toks[:70]}, [[("a", 1)]] * 70, dtype, "every token alone")
    # portions of changing size, down to two tokens
    for sizes in ([2], [7, 2, 33, 3, 16, 5], [64, 2, 31]):
        got = held_to_the_plain_model(engine, cfg, W, reqs, [[("a", c)] for c in cuts(len(toks), sizes)], dtype, f"portions {sizes}")["a"]
        if dtype == "float32":          # how the prompt was cut changes nothing beyond rounding
            assert rel(got, whole) < 4e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["d1", "d4"])
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
@pytest.mark.parametrize("name", ["d1", "d2", "d4"])
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
    engine, cfg, W = engine_of("d2", dtype, pages=28)
    toks = C.tokens("d2", 330, seed=8)
    held_to_the_plain_model(engine, cfg, W, {"a": toks}, [[("a", 9)]] + [[("a", 1)]] * 321, dtype, "long decoding")


def agrees_greedily(cfg, W, prompt, out, dtype):
    text = list(prompt)
    for t in out:
        row = P.forward(cfg, W, text)[-1]
        assert float(row.max() - row[t]) <= (2e-3 if dtype == "float32" else 0.12) * float(np.abs(row).max())
        text.append(t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype, tmp_path):
    """A folder on disk (config.json chooses the architecture), `Engine.generate`, several requests at once, decode steps
    from CUDA graphs where the engine takes them."""
    from tandemllm_b200.engine import Engine, EngineArgs
    from tandemllm_b200.sampling import SamplingParams
    name = "d2"
    folder = C.write_folder(str(tmp_path / "m"), name)
    engine = Engine.from_folder(folder, EngineArgs(dtype=dtype, max_len=256, parallel=3, chunk_size=32, max_batched_tokens=64))
    assert engine.model.spec.architecture == "Dipivik" and engine.model.graph_safe
    prompts = [C.tokens(name, n, seed=40 + n) for n in (70, 3, 21, 45)]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12))
    assert engine.step_function.graph_replays > 0
    for prompt, out in zip(prompts, outs):
        assert len(out) == 12
        agrees_greedily(C.CONFIGS[name], C.weights(name, bf16_exact=True), prompt, out, dtype)


def test_the_last_token_follows_graphs_steps_launched_ahead_and_preemption():
    """A model that is little more than its table of token pairs: what a step predicts hangs on the token before. Decode steps from
    graphs whose tokens are fed on the device, requests that lose their place and are recomputed, a stop id that ends a request
    after its next step was launched: always the text each request gives alone."""
    from tandemllm_b200.sampling import SamplingParams
    cfg = C.model(60, 64, 1e-5, [C.latent(2, 16, 8, 16, 16, 16, 0.2, 100.0, None), C.retention(2, 16, 16, (100.0, 16), ff=32)],
                  bigram=(401, 61, 7))
    W = C.random_weights(cfg, 5)
    W["bigram"] *= 3
    W["l0.mix.o"] *= 0.1
    g = torch.Generator().manual_seed(2)
    prompts = [torch.randint(0, 60, (n,), generator=g).tolist() for n in (40, 2, 33, 17, 1)]
    alone = []
    for p in prompts:
        engine, _, _ = engine_of(None, "float32", cfg=cfg, W=W, pages=16, parallel=1, overlap=False)
        alone.append(engine.generate([p], SamplingParams(temperature=0.0, max_tokens=30))[0])
        agrees_greedily(cfg, W, p, alone[-1], "float32")
    w = w64_of(W)
    other = P.embedding([prompts[0][0], prompts[0][-1]], cfg, w)[1] - P.embedding([(prompts[0][0] + 1) % 60, prompts[0][-1]], cfg, w)[1]
    assert np.abs(other).max() > 1.0                                    # the token before matters
    engine, _, _ = engine_of(None, "float32", cfg=cfg, W=W, pages=11, parallel=4, graph=True, max_len=128, chunk_size=16)
    assert engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=30)) == alone
    assert engine.stats()["scheduler"]["preemptions"] > 0 and engine.step_function.graph_replays > 0
    stop = alone[0][11]
    cut = [o[:o.index(stop) + 1] if stop in o else o for o in alone]
    outs = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=30, stop_token_ids=(stop,)))
    for o, c in zip(outs, cut):
        assert o == c or o == c[:-1]
    engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_on_a_folder(dtype, tmp_path):
    name = "d1"
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
    assert rel(a, wx[[0, 24]]) < TOL[dtype] * (2 if dtype == "bfloat16" else 1)
    assert rel(b, np.stack([wx[39], wy[18]])) < TOL[dtype] * (2 if dtype == "bfloat16" else 1)
    assert not (out / "2.f32").exists()


@pytest.mark.parametrize("seed", range(12))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_models_drawn_at_random(seed, dtype):
    cfg = C.random_config(seed)
    W = C.random_weights(cfg, 100 + seed)
    engine, cfg, W = engine_of(None, dtype, cfg=cfg, W=W, pages=32)
    g = torch.Generator().manual_seed(seed)
    toks = {r: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for r, n in (("a", 97), ("b", 30), ("c", 2))}
    schedule = [[("a", 40), ("b", 1)], [("a", 2), ("b", 17), ("c", 2)], [("a", 1), ("b", 1)], [("a", 31), ("b", 11)],
                [("a", 23)]]
    held_to_the_plain_model(engine, cfg, W, toks, schedule, dtype, f"random {seed}", slack=3.0 if dtype == "bfloat16" else 1.0,
                            outliers=0.015)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_command_line_writes_a_random_model_and_generates_from_it(dtype, tmp_path):
    """`random-weights` from a config.json of this design, then `generate` on the folder: greedy tokens that the plain model agrees
    with."""
    from tandemllm_b200.weights.safetensors_io import index_file, read_tensor
    cfg_path, folder, out = tmp_path / "config.json", tmp_path / "m", tmp_path / "out.json"
    cfg_path.write_text(json.dumps(C.D1))
    base = [sys.executable, "-m", "tandemllm_b200"]
    r = subprocess.run(base + ["random-weights", "--config", str(cfg_path), "--seed", "5", "--out", str(folder)], cwd=ROOT,
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    prompt = C.tokens("d1", 19, seed=6)
    r = subprocess.run(base + ["generate", "--model", str(folder), "--dtype", dtype, "--prompt-ids", ",".join(map(str, prompt)),
                               "--tokens", "8", "--json", str(out)], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = json.loads(out.read_text())["outputs"][0]
    assert len(got) == 8
    W = {k: read_tensor(v).double().numpy() for k, v in index_file(str(folder / "model.safetensors")).items()}
    assert set(W) == set(C.tensor_shapes(C.D1))
    agrees_greedily(C.D1, W, prompt, got, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_model_of_real_layer_widths(dtype):
    """Layer sizes of a model that would be served (width 1024, heads of 64 and 128, 16 experts), few layers and a small vocabulary:
    the products, attentions and scans run the forms they take at such sizes. A prompt in two portions, then decoding beside a
    second request."""
    cfg = C.model(1000, 1024, 1e-6, [C.latent(16, 64, 32, 64, 256, 384, 96 ** -0.5, 10000.0, 112, ff=(16, 4, 256, 512)),
                                     C.retention(8, 128, 128, (1e6, 128), ff=1024), C.latent(8, 128, 64, 128, 512, 256, 192 ** -0.5, 10000.0, 90, ff=512),
                                     C.retention(16, 64, 64, (1e6, 64), ff=(16, 4, 256, 512))], bigram=(2003, 31, 17), cap=25.0)
    W = C.random_weights(cfg, 77)
    engine, cfg, W = engine_of(None, dtype, cfg=cfg, W=W, pages=32)
    g = torch.Generator().manual_seed(9)
    toks = {r: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for r, n in (("a", 200), ("b", 70))}
    schedule = [[("a", 150)], [("a", 40), ("b", 64)]] + [[("a", 1), ("b", 1)]] * 6 + [[("a", 4)]]
    held_to_the_plain_model(engine, cfg, W, toks, schedule, dtype, "real widths")


@pytest.mark.parametrize("only", ["retention", "latent_attention"])
def test_a_model_of_one_kind_of_layer(only):
    """Nothing but retention: no page is ever held, only slots. Nothing but latent attention: no state but the last token."""
    layers = {"retention": [C.retention(2, 16, 8, (100.0, 16), ff=24), C.retention(1, 8, 16, None, ff=None)],
              "latent_attention": [C.latent(2, 16, 8, 8, 16, 16, 0.2, 100.0, 20, ff=24), C.latent(1, 8, 2, 16, 8, 8, 0.3, 100.0, 20, ff=None)]}
    from tandemllm_b200.sampling import SamplingParams
    cfg = C.model(40, 36, 1e-5, layers[only], bigram=(11, 5, 3), cap=8.0)
    W = C.random_weights(cfg, 3)
    engine, _, _ = engine_of(None, "float32", cfg=cfg, W=W, pages=12, parallel=2, graph=True, max_len=128, chunk_size=16)
    g = torch.Generator().manual_seed(1)
    texts = {r: torch.randint(0, 40, (n,), generator=g).tolist() for r, n in (("a", 60), ("b", 21))}
    held_to_the_plain_model(engine, cfg, W, texts, [[("a", 33), ("b", 1)], [("a", 2), ("b", 19)], [("b", 1)], [("a", 25)]], "float32", only)
    outs = engine.generate([texts["a"], texts["b"], texts["a"][:5]], SamplingParams(temperature=0.0, max_tokens=10))
    for p, o in zip((texts["a"], texts["b"], texts["a"][:5]), outs):
        assert len(o) == 10
        agrees_greedily(cfg, W, p, o, "float32")
