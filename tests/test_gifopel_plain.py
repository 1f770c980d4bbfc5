"""Gifopel without a GPU: the configuration reader, the caches it asks for, the tensors the parts ask for, chunked page groups in the
cache manager, and the plain implementation's own consistency (a prefix does not change when the sequence goes on; the
recurrences equal their definitions written out another way; chunks, sinks and experts do what they say)."""

import copy

import numpy as np
import pytest

from tests import gifopel_configs as C
from tests import plain_gifopel as P


def w64(name):
    return {k: v.double().numpy() for k, v in C.weights(name).items()}


def test_the_reader_names_every_tensor_of_the_design():
    from tandemllm_b200.config import GifopelConfig, architecture_of
    from tandemllm_b200.parts.model import DecoderModel
    for name, cfg in C.CONFIGS.items():
        assert architecture_of(cfg).name == "gifopel"
        spec = GifopelConfig.from_dict(cfg).to_spec()
        model = DecoderModel(spec)
        shapes = C.tensor_shapes(cfg, C.RANKS[name])
        for layer in model.layers:
            for part in layer.parts:
                if hasattr(part, "shapes_from"):
                    part.shapes_from(lambda n: shapes.get(n))
        assert {s.name: tuple(s.shape) for s in model.weight_specs(None)} == shapes, name
        assert GifopelConfig.from_dict(GifopelConfig.from_dict(cfg).to_dict()).to_spec() == spec
        assert len(spec.schedule) == len(cfg["layers"])
        assert all(s.cache_of is None for s in spec.schedule)           # a layer run again has a cache of its own


def test_layers_that_run_anothers_tensors_and_what_every_site_keeps():
    from tandemllm_b200.config import GifopelConfig
    from tandemllm_b200.parts.base import PagedNeed, SlotNeed
    from tandemllm_b200.parts.model import DecoderModel
    spec = GifopelConfig.from_dict(C.F1).to_spec()
    assert [s.layer for s in spec.schedule] == [0, 1, 2, 0] and [l.prefix for l in spec.layers] == ["l0.", "l1.", "l2."]
    needs = DecoderModel(spec).cache_needs()
    assert needs[0] == needs[3] and needs[0][0] == PagedNeed(2, 12, None, value_dim=10, chunk=24)
    # a slot: the convolution's last inputs (q, k, v each filled up to a multiple of 8 columns), then the state
    assert isinstance(needs[1], SlotNeed) and needs[1].shape == ((4 - 1) * (24 + 24 + 40) + 6 * 8 * 6,)
    assert needs[2].shape == (4 + 3 * 13 * 8,)                           # running maxima (filled up to 4), state and sum of keys
    chain = GifopelConfig.from_dict(C.F3).to_spec()
    assert [s.layer for s in chain.schedule] == [0, 1, 2, 1, 1]
    assert DecoderModel(chain).cache_needs()[0][0].reach is None         # no chunks: all earlier keys
    # the owner may come behind the layer that runs its tensors
    cfg = copy.deepcopy(C.F2)
    cfg["layers"] = [dict(cfg["layers"][1], weights_of=1), cfg["layers"][1]]
    spec = GifopelConfig.from_dict(cfg).to_spec()
    assert [s.layer for s in spec.schedule] == [0, 0] and spec.layers[0].prefix == "l1."


def test_unknown_keys_and_bad_sizes_are_refused_by_name():
    from tandemllm_b200.config import GifopelConfig

    def refused(match, change, base=C.F2):
        bad = copy.deepcopy(base)
        change(bad)
        with pytest.raises(ValueError, match=match):
            GifopelConfig.from_dict(bad)

    refused("window", lambda c: c["layers"][1]["mixer"]["left"].update(window=4))
    refused("logit_scale", lambda c: c.update(logit_scale=2.0))
    refused("gate_cap", lambda c: c["layers"][0]["mixer"].pop("gate_cap"))
    refused("kv_heads", lambda c: c["layers"][2]["mixer"].update(kv_heads=3))
    refused("conv", lambda c: c["layers"][2]["mixer"].update(conv=0))
    refused("rotated entries", lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=66))
    refused("mask.size", lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0))
    refused("top 9 of 8", lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    refused("attention", lambda c: c["layers"][0].update(type="attention"))
    refused("differs", lambda c: c["layers"][3]["mixer"].update(gate_cap=3.0))
    refused("weights_of 7", lambda c: c["layers"][3].update(weights_of=7))
    refused("weights_of 3", lambda c: c["layers"][3].update(weights_of=3))
    refused("glu", lambda c: c["layers"][0]["mlp"].update(kind="glu"))


def test_chunked_pages_go_back_when_the_chunk_is_over():
    from tandemllm_b200.cache import CacheManager
    from tandemllm_b200.parts.base import PagedNeed
    need = PagedNeed(1, 8, chunk=40)
    cache = CacheManager([need, PagedNeed(1, 8)], num_pages=8, max_requests=2, page_size=16)
    cache.admit("a")
    cache.reserve("a", 79)
    cache.advance("a", 39)
    assert all(p >= 0 for p in cache.table(0, "a"))
    cache.advance("a", 40)              # the next row begins a chunk: pages 0 and 1 are behind it, page 2 holds 40..47
    assert [p >= 0 for p in cache.table(0, "a")] == [False, False, True, True, True]
    assert all(p >= 0 for p in cache.table(1, "a"))
    cache.advance("a", 79)
    assert [p >= 0 for p in cache.table(0, "a")] == [False, False, True, True, True]
    cache.reserve("a", 81)
    cache.advance("a", 80)
    assert [p >= 0 for p in cache.table(0, "a")] == [False] * 5 + [True]
    cache.check()
    cache.free("a")
    assert all(g.pool.free == 8 for g in cache.groups)
    with pytest.raises(ValueError, match="chunk"):
        CacheManager([PagedNeed(1, 8, window=4, chunk=4)], num_pages=1, max_requests=1)


def test_a_prefix_does_not_change_when_the_sequence_goes_on():
    for name in ("f1", "f3", "f4"):
        toks = C.tokens(name, 40, seed=2)
        whole = P.forward(C.CONFIGS[name], w64(name), toks)
        assert np.allclose(P.forward(C.CONFIGS[name], w64(name), toks[:17]), whole[:17], rtol=1e-9, atol=1e-9)


def test_the_delta_rule_reads_what_it_wrote_and_carries_its_state():
    g = np.random.default_rng(0)
    T, H, D, V = 9, 2, 5, 3
    q, k = P.unit_vector(g.normal(size=(T, H, D))), P.unit_vector(g.normal(size=(T, H, D)))
    v, beta, dec = g.normal(size=(T, H, V)), P.sigmoid(g.normal(size=(T, H))), np.exp(-np.abs(g.normal(size=(T, H, D))))
    o, S = P.delta_scan(q, k, v, beta, dec)
    # one token: S = beta k v^T, so reading with the key itself gives beta |k|^2 v
    one, _ = P.delta_scan(k[:1], k[:1], v[:1], beta[:1], dec[:1])
    assert np.allclose(one[0], beta[0][:, None] * (k[0] ** 2).sum(-1)[:, None] * v[0], rtol=1e-10)
    # the same key written twice with full strength and no decay leaves the second value
    ones = np.ones((2, H))
    kk = np.stack([k[0] / np.sqrt((k[0] ** 2).sum(-1, keepdims=True))] * 2)
    again, _ = P.delta_scan(kk, kk, v[:2], ones, np.ones((2, H, D)))
    assert np.allclose(again[1], v[1], rtol=1e-10)
    # as a matrix recurrence: S <- (1 - beta k k^T) diag(g) S + beta k v^T
    for h in range(H):
        M = np.zeros((D, V))
        for t in range(T):
            M = (np.eye(D) - beta[t, h] * np.outer(k[t, h], k[t, h])) @ (dec[t, h][:, None] * M) + beta[t, h] * np.outer(k[t, h], v[t, h])
            assert np.allclose(o[t, h], M.T @ q[t, h], rtol=1e-9, atol=1e-12)
    a, Sa = P.delta_scan(q[:4], k[:4], v[:4], beta[:4], dec[:4])
    b, Sb = P.delta_scan(q[4:], k[4:], v[4:], beta[4:], dec[4:], Sa)
    assert np.allclose(np.concatenate([a, b]), o) and np.allclose(Sb, S)


def test_the_convolution_ends_at_the_current_token():
    u = np.arange(1.0, 6.0)[:, None]
    assert np.array_equal(P.causal_conv(u, np.array([[0.0, 0.0, 1.0]])), u)
    assert np.array_equal(P.causal_conv(u, np.array([[1.0, 0.0, 0.0]]))[:, 0], [0, 0, 1, 2, 3])
    assert np.array_equal(P.causal_conv(u, np.array([[2.0]])), 2 * u)


def test_the_matrix_memory_equals_its_sum_with_the_maximum_taken_out():
    """The running maximum only rescales: numerator and normaliser are sums over the tokens weighed by exp(i_s + f_(s+1) + .. + f_t),
    and the floor exp(-m) becomes 1 against them; m starts at 0, so a first token with a tiny input gate is not blown up to one."""
    m = {"heads": 2, "dim": 4, "vdim": 3, "gate_cap": 6.0}
    g = np.random.default_rng(3)
    width, T = 10, 12
    w = {"q": g.normal(size=(8, width)), "k": g.normal(size=(8, width)), "v": g.normal(size=(6, width)), "g": g.normal(size=(6, width)),
         "o": np.eye(6), "norm": np.ones(6), "i": g.normal(size=(2, width)), "i.b": g.normal(size=2) - 3.0,
         "f": g.normal(size=(2, width)), "f.b": g.normal(size=2) + 2.0}
    n = g.normal(size=(T, width))
    got = P.mixer_mlstm(n, m, w, "", 1e-5) / P.sigmoid(n @ w["g"].T)
    i, f = P.memory_gates(n, m, w, "")
    assert (np.abs(i) <= 6.0).all() and (f < 0).all()
    q, k, v = (n @ w["q"].T).reshape(T, 2, 4) * 0.5, (n @ w["k"].T).reshape(T, 2, 4), (n @ w["v"].T).reshape(T, 2, 3)
    for h in range(2):
        for t in range(T):
            e = np.array([i[s, h] + f[s + 1:t + 1, h].sum() for s in range(t + 1)])
            wt = np.exp(e)
            num, nq = (wt * (k[:t + 1, h] @ q[t, h])) @ v[:t + 1, h], (wt * (k[:t + 1, h] @ q[t, h])).sum()
            top = max(e.max(), f[:t + 1, h].sum())                     # m starts at 0 and decays with the forget gates
            o = num / (max(abs(nq), 1.0) + P.READ_FLOOR * np.exp(top))
            assert np.allclose(got.reshape(T, 2, 3)[t, h], P.unit_rms(o, 1e-5), rtol=1e-7, atol=1e-9)


def test_chunks_count_from_position_zero_and_a_sink_only_takes_weight_away():
    seen = P.chunk_mask(9, 4)
    assert seen[3, 0] and not seen[4, 3] and seen[4, 4] and seen[7, 4] and not seen[8, 7] and not seen[0, 1]
    assert P.chunk_mask(5, None).sum() == 15 and np.array_equal(P.chunk_mask(4, 1), np.eye(4, dtype=bool))
    m, W = C.F1["layers"][0]["mixer"]["left"], w64("f1")
    pre = "l0.mix.left."
    n = np.random.default_rng(1).normal(size=(30, 44))
    base = P.mixer_chunked_attention(n, m, W, pre, 1e-4)
    # the first row of a chunk sees itself only: its heads are v exp(s) / (exp(s) + exp(sink)), gated
    n2 = n.copy()
    n2[:24] = 0.5
    assert np.allclose(P.mixer_chunked_attention(n2, m, W, pre, 1e-4)[24:], base[24:], rtol=1e-9, atol=1e-12)
    high = dict(W)
    high[pre + "sink"] = np.full(4, 60.0)
    assert np.abs(P.mixer_chunked_attention(n, m, high, pre, 1e-4)).max() < 1e-12
    low = dict(W)
    low[pre + "sink"] = np.full(4, -60.0)
    assert not np.allclose(P.mixer_chunked_attention(n, m, low, pre, 1e-4), base, rtol=1e-2)


def test_neighbouring_entries_turn_and_the_rest_pass():
    x = np.random.default_rng(2).normal(size=(3, 1, 6))
    r = P.rotate_neighbours(x, np.array([0, 1, 5]), 100.0, 4)
    assert np.array_equal(r[0], x[0]) and np.array_equal(r[..., 4:], x[..., 4:])
    a = 5 * 100.0 ** (-2.0 / 4)
    assert np.allclose(r[2, 0, 2:4], [x[2, 0, 2] * np.cos(a) - x[2, 0, 3] * np.sin(a), x[2, 0, 3] * np.cos(a) + x[2, 0, 2] * np.sin(a)])


def test_the_routers_bias_is_part_of_the_logits_and_only_the_chosen_share_the_weight():
    W = w64("f1")
    n = np.random.default_rng(5).normal(size=(6, 44))
    ff = C.F1["layers"][0]["mlp"]
    z = P.router_logits(n, W, "l0.mlp.")
    out = P.routed_experts(n, ff, W, "l0.mlp.")
    t = 3
    a, b = np.argsort(-z[t])[:2]
    pa = 1 / (1 + np.exp(z[t, b] - z[t, a]))
    want = pa * P.squared_relu_expert(n[t:t + 1], W, f"l0.mlp.e{a}.") + (1 - pa) * P.squared_relu_expert(n[t:t + 1], W, f"l0.mlp.e{b}.")
    assert np.allclose(out[t], want[0], rtol=1e-10)
    pushed = dict(W)
    pushed["l0.mlp.router.b"] = np.array([0, 0, 0, 50.0, 0])
    assert np.allclose(P.routed_experts(n, ff, pushed, "l0.mlp."), P.squared_relu_expert(n, W, "l0.mlp.e3."), rtol=1e-9)


def test_mixer_and_feed_forward_read_the_same_residual():
    cfg = {"architecture": "Gifopel", "vocab": 9, "width": 24, "norm": {"eps": 1e-5}, "layers": [C.memory(2, 4, 6, 5.0, ff=20)]}
    W = {k: v.double().numpy() for k, v in C.random_weights(cfg, (2, 2), 3).items()}
    toks = [1, 5, 7, 2]
    _, layers = P.forward(cfg, W, toks, return_layers=True)
    x = W["embed"][toks]
    want = x + P.mixer_mlstm(P.plain_norm(x, W["l0.norm1"], 1e-5), cfg["layers"][0]["mixer"], W, "l0.mix.", 1e-5) + \
        P.dense_gated(P.plain_norm(x, W["l0.norm2"], 1e-5), W, "l0.mlp.")
    assert np.allclose(layers[0], want, rtol=1e-12)


def test_models_drawn_at_random_can_be_read():
    from tandemllm_b200.config import GifopelConfig
    from tandemllm_b200.parts.model import DecoderModel
    for seed in range(40):
        cfg, ranks = C.random_config(seed)
        model = DecoderModel(GifopelConfig.from_dict(cfg).to_spec())
        shapes = C.tensor_shapes(cfg, ranks)
        for layer in model.layers:
            for part in layer.parts:
                if hasattr(part, "shapes_from"):
                    part.shapes_from(lambda n: shapes.get(n))
        assert {s.name: tuple(s.shape) for s in model.weight_specs(None)} == shapes, seed
