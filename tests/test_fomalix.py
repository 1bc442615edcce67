"""CPU: the Fomalix oracle's mechanisms on cases with known answers, config.json reading, the model registry, and what the library
refuses before it touches a device."""
import json

import numpy as np
import pytest

import fomalix_models as M
from oracle import fomalix as F


def test_activations():
    np.testing.assert_allclose(F.softplus(np.array([0.0, 800.0, -800.0])), [np.log(2), 800.0, 0.0])
    np.testing.assert_allclose(F.gelu_tanh(np.array([0.0, 1.0, 9.0, -9.0])), [0.0, 0.841192, 9.0, 0.0], atol=1e-6)
    np.testing.assert_allclose(np.sum(F.unit(np.array([3.0, 4.0])) ** 2), 1.0, rtol=1e-6)


def test_position_vector_interleaves_sine_and_cosine():
    s = F.sinusoid([0, 2], 6)
    assert s[0].tolist() == [0, 1, 0, 1, 0, 1]
    np.testing.assert_allclose(s[1, 2:4], [np.sin(2 * 10000 ** (-2 / 6)), np.cos(2 * 10000 ** (-2 / 6))])
    np.testing.assert_allclose(F.embedding([1], np.array([[5.0, 5], [2.0, 3]]), 10.0), [[20.0, 31.0]])


def test_chunk_mask_edges():
    m = F.chunk_mask(7, 3)
    assert m[2].tolist() == [True] * 3 + [False] * 4 and m[3].tolist() == [False] * 3 + [True] + [False] * 3 and m[5].sum() == 3 and m[6].sum() == 1
    assert (F.chunk_mask(4, 1) == np.eye(4, dtype=bool)).all() and (F.chunk_mask(4, 9) == np.tril(np.ones((4, 4), bool))).all()


def test_the_sink_takes_weight_and_gives_no_value():
    score = np.array([[[1.0, 2.0, -np.inf]]])
    e = np.exp([1.0, 2.0])
    np.testing.assert_allclose(F.sink_softmax(score, np.array([3.0]))[0, 0, :2], e / (e.sum() + np.exp(3.0)))
    assert F.sink_softmax(score, np.array([700.0])).max() < 1e-250


def test_convolution_sees_the_past_and_zeros_before_the_start():
    x = np.arange(1.0, 5.0)[:, None]
    assert F.causal_conv(x, np.array([[100.0, 10.0, 1.0]]))[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0]
    assert F.causal_conv(x, np.array([[2.0]]), 1.0)[:, 0].tolist() == [3.0, 5.0, 7.0, 9.0]


def test_the_delta_rule_replaces_what_a_key_held():
    k = np.array([[[1.0, 0.0]], [[0.0, 1.0]], [[1.0, 0.0]]])
    v = np.array([[[3.0]], [[5.0]], [[7.0]]])
    one = np.ones((3, 1))
    o = F.delta_rule(k, k, v, one, one)
    assert o[:, 0, 0].tolist() == [3.0, 5.0, 7.0]                       # a token reads what it just wrote; 7 took the place of 3
    o = F.delta_rule(k, k, v, 0.5 * one, 0.5 * one)
    np.testing.assert_allclose(o[:, 0, 0], [1.5, 2.5, 0.375 + 0.5 * (7 - 0.375)])


def test_the_state_space_sums_decayed_writes_and_skips():
    x, B = np.array([[[1.0]], [[2.0]]]), np.ones((2, 1, 1))
    dt = np.array([[0.5], [0.25]])
    y = F.state_space(x, B, 3 * B, dt, np.array([np.log(2.0)]), np.array([10.0]))
    np.testing.assert_allclose(y[:, 0, 0], [1.5 + 10, 3 * (0.5 * np.exp(-0.5) + 0.5) + 20])


def test_order_of_looped_layers():
    cfg = M.config([(M.delta(), None)] * 5, loop=(1, 3, 3))
    assert F.layer_runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    cfg["loop"] = None
    assert [i for i, _ in F.layer_runs(cfg)] == [0, 1, 2, 3, 4]


def test_every_mechanism_shows_in_the_logits():
    cfg = M.config([(M.delta(), None), (M.mamba(), 30), (M.attn(), 40)], loop=(1, 3, 2))
    w, t = M.random_weights(cfg), M.tokens(cfg, 60)
    base, rng = F.forward(cfg, w, t), np.random.default_rng(1)
    for name in w:
        v = dict(w)
        v[name] = w[name] + 0.3 * np.abs(w[name]).max() * rng.standard_normal(w[name].shape)
        assert M.error(F.forward(cfg, v, t), base) > 1e-3, name
    far = list(t)
    far[2] = M.MARK
    assert M.error(F.forward(cfg, w, far)[-1:], base[-1:]) > 1e-3        # the slow heads carry a write to the end
    trace = []
    F.forward(cfg, w, t, trace)
    assert len(trace) == 5


def test_the_planted_key_shows_inside_its_chunk_only():
    cfg = M.config([(M.attn(chunk=10), 30)])
    w = M.plant_marker(cfg, M.random_weights(cfg))
    t = M.tokens(cfg, 40)
    plain = F.forward(cfg, w, t)
    t[13] = M.MARK
    marked = F.forward(cfg, w, t)
    assert np.array_equal(plain[:13], marked[:13]) and np.array_equal(plain[20:], marked[20:])
    assert min(M.error(marked[p:p + 1], plain[p:p + 1]) for p in range(13, 20)) > 0.1


def test_config_reading():
    from skainet_b200.fomalix import ATTENTION, DELTA, MAMBA2, FomalixConfig
    cfg = M.config([(M.delta(), None), (M.mamba(), 30), (M.attn(), 40)], loop=(1, 3, 2))
    c = FomalixConfig.from_json(cfg, max_seq=50, dtype="float32")
    assert (c.width, c.vocab, c.eps, c.max_seq, c.embed_scale, c.loop) == (72, 97, 1e-3, 50, 3.0, (1, 3, 2))
    d, m, a = c.layers
    assert (d.type, d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.ff) == (DELTA, 6, 3, 20, 12, 4, 0)
    assert (m.type, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, m.norm_groups, m.ff) == (MAMBA2, 6, 2, 24, 10, 3, 3, 30)
    assert (a.type, a.heads, a.kv_heads, a.dim, a.vdim, a.chunk, a.scale, a.ff) == (ATTENTION, 6, 2, 14, 18, 9, 0.35, 40)
    raw, layers = c.to_c()
    assert (raw.act_f32, raw.loop_start, raw.loop_stop, raw.loop_times) == (1, 1, 3, 2) and layers[2].chunk == 9 and abs(raw.embed_scale - 3.0) < 1e-6
    del cfg["loop"], cfg["layers"][0]["mlp"]
    raw, _ = FomalixConfig.from_json(cfg).to_c()
    assert (raw.loop_start, raw.loop_stop, raw.loop_times, raw.act_f32) == (0, 3, 1, 0)
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d.update(extra=1), lambda d: d["layers"][2]["mixer"].update(rot={}),
                   lambda d: d["layers"][1]["mlp"].update(kind="other"), lambda d: d["layers"][2]["mixer"]["mask"].update(kind="x"),
                   lambda d: d["layers"][2]["mixer"]["mask"].update(size=0), lambda d: d["layers"][1]["mixer"].update(clamp=1.0), lambda d: d.update(loop={"start": 0, "stop": 1, "times": 2, "x": 0})):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            FomalixConfig.from_json(bad)
    with pytest.raises(ValueError):
        FomalixConfig.from_json(cfg, dtype="float16").to_c()


def test_registry_name():
    from skainet_b200 import models
    assert models.FOLDERS["Fomalix"].__self__ is models.Fomalix


def test_create_refuses_bad_configurations_before_any_device_work(cuda_lib):
    from skainet_b200.fomalix import Fomalix, FomalixConfig
    for edit, text in ((lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads in 4 groups"),
                       (lambda c: c["layers"][0]["mixer"].update(conv=0), "0 taps"),
                       (lambda c: c["layers"][0]["mixer"].update(dim=513), "key size 513"),
                       (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "norm in 7 parts"),
                       (lambda c: c["layers"][2]["mixer"].update(dim=0), "bad sizes"),
                       (lambda c: c["loop"].update(stop=4), "layers 1 to 4 of 3"),
                       (lambda c: c["loop"].update(times=0), "0 times"),
                       (lambda c: c.update(width=0), "non-positive")):
        cfg = M.config([(M.delta(), None), (M.mamba(), 30), (M.attn(), 40)], loop=(1, 3, 2))
        edit(cfg)
        with pytest.raises(ValueError, match=text):
            Fomalix(FomalixConfig.from_json(cfg))
