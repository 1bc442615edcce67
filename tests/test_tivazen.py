"""CPU: the Tivazen oracle's mechanisms on cases with known answers, config.json and safetensors reading, the model registry,
sequence slots, and what the library refuses before it touches a device."""
import json
import struct

import numpy as np
import pytest

import tivazen_models as M
from oracle import tivazen as T


def test_norms_and_activations():
    x = np.array([[3.0, -4.0, 0.0, 0.0]])
    np.testing.assert_allclose(T.rms_norm(x, 2.0, 0.0), 2 * x / 2.5)
    np.testing.assert_allclose(T.rms_norm(x, np.array([1.0, 0.0, 1.0, 1.0]), 2.75), [[1.0, 0, 0, 0]])      # eps inside the root
    np.testing.assert_allclose(T.silu(np.array([0.0, 50.0])), [0.0, 50.0])


def test_rotation_pairs_the_halves_and_preserves_relative_positions():
    v = np.zeros((2, 4)); v[:, 1] = 1.0
    r = T.rotate_half(v, [0, 3], 10000.0)
    np.testing.assert_allclose(r[0], v[0])
    np.testing.assert_allclose(r[1], [0, np.cos(0.03), 0, np.sin(0.03)], atol=1e-12)      # second pair: 10000^(-1/2)
    rng = np.random.default_rng(0)
    a, b = rng.standard_normal(8), rng.standard_normal(8)
    dot = lambda i, j: T.rotate_half(a[None], [i], 77.0)[0] @ T.rotate_half(b[None], [j], 77.0)[0]
    assert abs(dot(5, 2) - dot(105, 102)) < 1e-9 and abs(dot(5, 2) - dot(5, 3)) > 1e-6


def test_window_mask_edges():
    m = T.window_mask(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5
    assert (T.window_mask(6, 1) == np.eye(6, dtype=bool)).all()


def test_routing_takes_the_largest_scores_unnormalised_and_scales_the_input():
    h = np.array([[1.0, 0.0]])
    pick, weight = T.route(h, np.array([[0.0, 0], [2.0, 0], [-1.0, 0]]), 2)
    assert pick.tolist() == [[1, 0]]
    np.testing.assert_allclose(weight, [[T.sigmoid(2.0), 0.5]])
    ex = [(np.eye(2), np.eye(2), np.eye(2))] * 3
    s = weight[0]
    np.testing.assert_allclose(T.expert_ff(h, np.array([[0.0, 0], [2.0, 0], [-1.0, 0]]), ex, 2)[0, 0], sum(T.silu(v) * v for v in s))


def test_attention_of_one_key_returns_its_gated_value():
    mix = M.attn(heads=2, dim=4, rot_dim=2, vdim=3, kv_rank=5, window=1)
    rng = np.random.default_rng(3)
    w = {"q": rng.standard_normal((12, 6)), "uk": rng.standard_normal((8, 5)), "uv": rng.standard_normal((6, 5)), "g": rng.standard_normal((2, 6)), "o": np.eye(6)}
    h, c = rng.standard_normal((4, 6)), rng.standard_normal((4, 5))
    out = T.latent_attention(h, w, mix, (c, rng.standard_normal((4, 2))))
    np.testing.assert_allclose(out, (c @ w["uv"].T) * np.repeat(T.sigmoid(h @ w["g"].T), 3, axis=1))


def test_depth_average_and_shared_latent_enter_the_model():
    cfg = M.config([(M.attn(), M.dense()), (M.attn(kv_from=0, window=4, heads=2), None), (M.attn(kv_rank=12), M.moe())])
    w, t = M.random_weights(cfg), M.tokens(M.config([]), 14)
    base = T.forward(cfg, w, t)
    for name, at in (("l1.dwa", 0), ("l2.dwa", 1), ("l0.mix.dkv.norm", 0)):
        v = {k: a.copy() for k, a in w.items()}
        v[name][at] += 0.5
        assert M.error(T.forward(cfg, v, t), base) > 1e-3, name
    trace = []
    T.forward(cfg, w, t, trace)
    assert len(trace) == 3 and trace[0].shape == (14, 72)


def test_the_planted_key_shows_inside_the_window_and_not_outside():
    cfg = M.config([(M.attn(window=9), M.dense())])
    w = M.plant_marker(cfg, M.random_weights(cfg))
    t = M.tokens(cfg, 40)
    plain = T.forward(cfg, w, t)
    t[20] = M.MARK
    marked = T.forward(cfg, w, t)
    assert np.array_equal(plain[:20], marked[:20]) and np.array_equal(plain[29:], marked[29:])
    assert min(M.error(marked[p:p + 1], plain[p:p + 1]) for p in range(20, 29)) > 0.1


def test_config_reading():
    from skainet_b200.tivazen import MLP_MOE, MLP_NONE, TivazenConfig
    cfg = M.config([(M.attn(), M.moe()), (M.attn(kv_from=0), None)])
    c = TivazenConfig.from_json(cfg, max_seq=50, dtype="float32")
    assert (c.width, c.vocab, c.eps, c.max_seq) == (72, 97, 1e-3, 50)
    a, b = c.layers
    assert (a.kv_from, a.mlp, a.experts, a.top, a.ff) == (None, MLP_MOE, 5, 3, 18) and (b.kv_from, b.mlp) == (0, MLP_NONE)
    del cfg["layers"][1]["mlp"]
    assert TivazenConfig.from_json(cfg).layers[1].mlp == MLP_NONE
    raw, layers = c.to_c()
    assert raw.act_f32 == 1 and layers[0].kv_from == -1 and layers[1].kv_from == 0 and layers[0].window == 9
    for change in (lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), lambda d: d.update(extra=1),
                   lambda d: d["layers"][0]["mixer"].update(sinks=2), lambda d: d["layers"][0]["mlp"].update(kind="other"), lambda d: d["layers"][0]["mixer"]["mask"].update(kind="x")):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            TivazenConfig.from_json(bad)
    with pytest.raises(ValueError):
        TivazenConfig.from_json(cfg, dtype="float16").to_c()


def test_safetensors_reader(tmp_path):
    from skainet_b200.safetensors import SafetensorsReader, write
    p = str(tmp_path / "a.safetensors")
    v = np.array([[1.5, -2.0, 3.25]])
    write(p, {"m": ("BF16", (1, 3), M.round_bf16(v)), "s": ("BF16", (), M.round_bf16(np.array(0.5))), "i": ("I32", (2,), np.array([4, -5], np.int32)),
              "f": ("F32", (2,), np.array([1e-3, 7.0], np.float32))})
    r = SafetensorsReader(p)
    assert r.floats("m").tolist() == v.tolist() and float(r.floats("s")) == 0.5 and r.floats("f")[1] == 7.0 and r.tensor("i").dtype == "I32"
    with pytest.raises(ValueError, match="not found"):
        r.raw("none")
    with pytest.raises(ValueError, match="expected BF16"):
        r.weight("m", 3, 1)
    with pytest.raises(ValueError, match="not a floating-point"):
        r.floats("i")
    r.close()
    raw = bytearray(open(p, "rb").read())
    for cut in (4, 40, len(raw) - 2):
        with pytest.raises(ValueError):
            open(p, "wb").write(raw[:cut])
            SafetensorsReader(p)
    h = json.dumps({"x": {"dtype": "BF16", "shape": [4], "data_offsets": [0, 6]}}).encode()
    open(p, "wb").write(struct.pack("<Q", len(h)) + h + bytes(8))
    with pytest.raises(ValueError):
        SafetensorsReader(p)


def test_bf16_rounding_helper_is_nearest_even():
    x = np.array([1.0, 1.0 + 2 ** -8, 1.0 + 3 * 2 ** -8, 1.0 + 2 ** -7, -3.14159, 1e-30], np.float32)
    assert M.widen(M.round_bf16(x)).tolist()[:4] == [1.0, 1.0, 1.0 + 2 ** -6, 1.0 + 2 ** -7]


def test_registry_names(tmp_path):
    from skainet_b200 import models
    assert "Tivazen" in models.FOLDERS and "llama" in models.GGUF
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unknown"}))
    with pytest.raises(ValueError, match="'Unknown' is not one of"):
        models.load_model(str(tmp_path))


def test_sequence_slots(monkeypatch):
    from skainet_b200 import decoder
    resets = []
    monkeypatch.setattr(decoder.Decoder, "reset", lambda self, seq=None: resets.append(seq))
    d = decoder.Decoder(0, 10, 10, 2)
    assert (d.acquire(), d.acquire()) == (0, 1)
    with pytest.raises(RuntimeError):
        d.acquire()
    d.release(0)
    with pytest.raises(ValueError):
        d.release(0)
    assert d.acquire() == 0 and resets == [0, 1, 0, 0]


def test_create_refuses_bad_configurations_before_any_device_work(cuda_lib):
    from skainet_b200.tivazen import Tivazen, TivazenConfig
    for edit, text in ((lambda c: c["layers"][0]["mixer"].update(rot_dim=5, rot={"base": 10.0, "dims": 5}), "must be even"),
                       (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "none of its own"),
                       (lambda c: c["layers"][1]["mixer"].update(kv_rank=8), "differ in kv_rank"),
                       (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window 0"),
                       (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "6 of 5 experts"),
                       (lambda c: c.update(width=0), "non-positive")):
        cfg = M.config([(M.attn(), M.moe()), (M.attn(kv_from=0), None)])
        edit(cfg)
        with pytest.raises(ValueError, match=text):
            Tivazen(TivazenConfig.from_json(cfg))
