"""Dipivik without a GPU: the configuration reader, the caches it asks for, the tensors the parts ask for, and the plain
implementation's own consistency (a prefix does not change when the sequence goes on; retention equals its sum written out;
windows, gates, token pairs and experts do what they say)."""

import copy

import numpy as np
import pytest

from tests import dipivik_configs as C
from tests import plain_dipivik as P


def w64(name):
    return {k: v.double().numpy() for k, v in C.weights(name).items()}


def test_the_reader_names_every_tensor_of_the_design():
    from tandemllm_b200.config import DipivikConfig, architecture_of
    from tandemllm_b200.parts.model import DecoderModel
    for name, cfg in list(C.CONFIGS.items()) + [(s, C.random_config(s)) for s in range(40)]:
        assert architecture_of(cfg).name == "dipivik"
        spec = DipivikConfig.from_dict(cfg).to_spec()
        assert {s.name: tuple(s.shape) for s in DecoderModel(spec).weight_specs(None)} == C.tensor_shapes(cfg), name
        assert DipivikConfig.from_dict(DipivikConfig.from_dict(cfg).to_dict()).to_spec() == spec


def test_what_every_site_keeps_and_the_slot_behind_the_sites():
    import torch

    from tandemllm_b200.cache import CacheManager
    from tandemllm_b200.config import DipivikConfig
    from tandemllm_b200.parts.base import PagedNeed, SlotNeed
    from tandemllm_b200.parts.model import DecoderModel
    needs = DecoderModel(DipivikConfig.from_dict(C.D1).to_spec()).cache_needs()
    assert needs[0] == SlotNeed((3, 8, 6)) and needs[1] == PagedNeed(1, 26, 19, values=False)
    assert len(needs) == 6 and needs[5] == SlotNeed((1,), torch.int32) and needs[5].init == -1      # a request's last token
    assert len(DecoderModel(DipivikConfig.from_dict(C.D3).to_spec()).cache_needs()) == 3              # no table of pairs: no such slot
    cache = CacheManager(needs, num_pages=4, max_requests=2, device=torch.device("cpu"))
    last = cache.site_cache[5].state
    slot = cache.admit("a")
    assert last[slot].item() == -1
    last[slot] = 7
    cache.free("a")
    assert cache.admit("b") == slot and last[slot].item() == -1


def test_unknown_keys_and_bad_sizes_are_refused_by_name():
    from tandemllm_b200.config import DipivikConfig

    def refused(match, change, base=C.D2):
        bad = copy.deepcopy(base)
        change(bad)
        with pytest.raises(ValueError, match=match):
            DipivikConfig.from_dict(bad)

    refused("sink", lambda c: c["layers"][0]["mixer"].update(sink=1))
    refused("logit_scale", lambda c: c.update(logit_scale=2.0))
    refused("trigram", lambda c: c["embedding"].update(trigram={}))
    refused("mul_cur", lambda c: c["embedding"]["bigram"].pop("mul_cur"))
    refused("buckets", lambda c: c["embedding"]["bigram"].update(buckets=0))
    refused("q_rank", lambda c: c["layers"][0]["mixer"].pop("q_rank"))
    refused("kv_rank", lambda c: c["layers"][0]["mixer"].update(kv_rank=0))
    refused("rotated entries", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34))
    refused("rotated entries", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))
    refused("mask.size", lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    refused("3 decays for 4 heads", lambda c: c["layers"][1]["mixer"]["decay"].pop())
    refused("top 9 of 8", lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    refused("shared", lambda c: c["layers"][0]["mlp"].update(shared={"width": 4}))
    refused("mamba2", lambda c: c["layers"][0].update(type="mamba2"))
    refused("glu", lambda c: c["layers"][0]["mlp"].update(kind="glu"))


def test_a_prefix_does_not_change_when_the_sequence_goes_on():
    for name in C.CONFIGS:
        toks = C.tokens(name, 40, seed=2)
        whole = P.forward(C.CONFIGS[name], w64(name), toks)
        assert np.allclose(P.forward(C.CONFIGS[name], w64(name), toks[:17]), whole[:17], rtol=1e-9, atol=1e-9)


def test_token_pairs_read_the_token_before_and_the_first_one_the_last_row():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert P.bigram_rows([4, 1, 1, 9], b).tolist() == [10, 19 % 10, 10 % 10, 66 % 10]
    assert P.bigram_rows([4], b).tolist() == [10]
    cfg = {"embedding": {"bigram": b}}
    w = {"embed": np.eye(12), "bigram": np.arange(11.0)[:, None] * np.ones((11, 12))}
    x = P.embedding([4, 1], cfg, w)
    assert x[0, 4] == 11.0 and x[0, 0] == 10.0 and x[1, 1] == 10.0 and x[1, 0] == 9.0
    assert np.array_equal(P.embedding([4, 1], {}, w), np.eye(12)[[4, 1]])


def test_retention_is_the_decayed_sum_over_all_tokens():
    m = {"heads": 2, "dim": 6, "vdim": 5, "decay": [0.9, 0.995], "rot": {"base": 50.0, "dims": 4}}
    g = np.random.default_rng(3)
    width, T, eps = 9, 14, 1e-4
    w = {"q": g.normal(size=(12, width)), "k": g.normal(size=(12, width)), "v": g.normal(size=(10, width)), "g": g.normal(size=(10, width)),
         "o": np.eye(10)}
    n = g.normal(size=(T, width))
    got = (P.mixer_retention(n, m, w, "", eps) / P.silu(n @ w["g"].T)).reshape(T, 2, 5)
    q, k, v = P.retention_inputs(n, m, w, "")
    for h in range(2):
        for t in range(T):
            o = sum(m["decay"][h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(got[t, h], P.unit_rms(o, eps), rtol=1e-9)
    a, S = P.retention_scan(q[:5], k[:5], v[:5], m["decay"])
    b, S = P.retention_scan(q[5:], k[5:], v[5:], m["decay"], S)
    whole, end = P.retention_scan(q, k, v, m["decay"])
    assert np.allclose(np.concatenate([a, b]), whole) and np.allclose(S, end)


def test_halves_turn_the_rest_passes_and_only_differences_of_positions_count():
    x = np.random.default_rng(2).normal(size=(3, 1, 6))
    r = P.rotate_halves(x, np.array([0, 1, 5]), 100.0, 4)
    assert np.array_equal(r[0], x[0]) and np.array_equal(r[..., 4:], x[..., 4:])
    a = 5 * 100.0 ** (-2.0 / 4)
    assert np.allclose(r[2, 0, [1, 3]], [x[2, 0, 1] * np.cos(a) - x[2, 0, 3] * np.sin(a), x[2, 0, 3] * np.cos(a) + x[2, 0, 1] * np.sin(a)])
    far = P.rotate_halves(x, np.array([1000, 1001, 1005]), 100.0, 4)
    assert np.allclose(far[1, 0] @ far[2, 0], r[1, 0] @ r[2, 0])


def test_the_window_holds_its_size_and_the_gate_is_a_number_a_head():
    seen = P.window_mask(6, 3)
    assert seen[5, 3] and not seen[5, 2] and seen[2, 0] and not seen[0, 1] and P.window_mask(5, None).sum() == 15
    assert np.array_equal(P.window_mask(4, 1), np.eye(4, dtype=bool))
    m, W, pre = C.D1["layers"][1]["mixer"], w64("d1"), "l1.mix."
    n = np.random.default_rng(1).normal(size=(30, 44))
    base = P.mixer_latent_attention(n, m, W, pre, 1e-4)
    n2 = n.copy()
    n2[:11] = 0.5               # out of the window of every row from 29 on (29 - 18 = 11 is the first one inside)
    assert np.allclose(P.mixer_latent_attention(n2, m, W, pre, 1e-4)[29:], base[29:], rtol=1e-9, atol=1e-12)
    assert not np.allclose(P.mixer_latent_attention(n2, m, W, pre, 1e-4)[28], base[28], rtol=1e-3)
    closed = dict(W)
    closed[pre + "g"] = np.zeros((4, 44))
    open_ = dict(closed)
    open_[pre + "o"] = 2 * W[pre + "o"]
    assert np.allclose(P.mixer_latent_attention(n, m, open_, pre, 1e-4), 2 * P.mixer_latent_attention(n, m, closed, pre, 1e-4))
    # with a window of one a row only sees itself: its heads are its own values, gated
    own = P.mixer_latent_attention(n, dict(m, mask={"size": 1}), W, pre, 1e-4)
    c, _ = P.latent_keys(n, m, W, pre, 1e-4)
    v = (c @ W[pre + "uv"].T).reshape(30, 4, 10) * P.sigmoid(n @ W[pre + "g"].T)[:, :, None]
    assert np.allclose(own, v.reshape(30, 40) @ W[pre + "o"].T)


def test_an_experts_weight_multiplies_its_input():
    W, n = w64("d1"), np.random.default_rng(5).normal(size=(6, 44))
    ff = C.D1["layers"][0]["mlp"]
    s = P.sigmoid(n @ W["l0.mlp.router"].T)
    out, t = P.routed_experts(n, ff, W, "l0.mlp."), 3
    a, b = np.argsort(-s[t])[:2]
    want = P.expert(s[t, a] * n[t:t + 1], W, f"l0.mlp.e{a}.") + P.expert(s[t, b] * n[t:t + 1], W, f"l0.mlp.e{b}.")
    assert np.allclose(out[t], want[0], rtol=1e-10)
    outside = s[t, a] * P.expert(n[t:t + 1], W, f"l0.mlp.e{a}.") + s[t, b] * P.expert(n[t:t + 1], W, f"l0.mlp.e{b}.")
    assert not np.allclose(want, outside, rtol=0.05)
    both = P.feed_forward(n, ff, W, "l0.mlp.")
    assert np.allclose(both - out, P.expert(n, W, "l0.mlp.shared."))


def test_the_tanh_form_of_gelu_and_the_biases():
    assert np.allclose(P.gelu_tanh(np.array([-30.0, 0.0, 1.0, 30.0])), [0.0, 0.0, 0.841192, 30.0], atol=1e-6)
    W = w64("d1")
    zero = np.zeros((1, 44))
    want = (P.gelu_tanh(W["l1.mlp.gate.b"]) * W["l1.mlp.up.b"]) @ W["l1.mlp.down"].T + W["l1.mlp.down.b"]
    assert np.allclose(P.dense_gated(zero, W, "l1.mlp.")[0], want)


def test_mixer_and_feed_forward_read_one_norm_of_one_residual():
    cfg = C.model(9, 24, 1e-5, [C.retention(2, 6, 8, (40.0, 6), ff=20)], bigram=(4, 3, 2), cap=3.0)
    W = {k: v.double().numpy() for k, v in C.random_weights(cfg, 3).items()}
    toks = [1, 5, 7, 2]
    logits, layers = P.forward(cfg, W, toks, return_layers=True)
    x = P.embedding(toks, cfg, W)
    n = P.plain_norm(x, W["l0.norm1"], 1e-5)
    want = x + P.mixer_retention(n, cfg["layers"][0]["mixer"], W, "l0.mix.", 1e-5) + P.dense_gated(n, W, "l0.mlp.")
    assert np.allclose(layers[0], want, rtol=1e-12)
    raw = P.plain_norm(want, W["final.norm"], 1e-5) @ W["embed"].T
    assert np.allclose(logits, 3.0 * np.tanh(raw / 3.0)) and np.abs(logits).max() <= 3.0
