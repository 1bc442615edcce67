"""GPU: the Fomalix design and the mechanisms it added, against the plain oracle, through the framework's own loader, caches,
steps and scheduler. fp32 models are held to fp32 rounding, bf16 models to bf16 rounding."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import fomalix_models as M
from oracle import fomalix as F

pytestmark = pytest.mark.gpu

TOL = {"float32": 3e-5, "bfloat16": 0.1}
DTYPES = ("float32", "bfloat16")
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))

A, D, S = M.attn, M.delta, M.mamba
CONFIGS = {
    # every branch at once: the three mixers inside and outside the loop, feed-forwards on some layers, odd sizes
    "mixed": M.config([(D(), None), (S(), 30), (A(), None), (D(heads=4, kv_heads=1, dim=33, vdim=24, conv=2), 50), (A(heads=4, kv_heads=4, chunk=21), 36)], loop=(1, 4, 3)),
    # nothing a multiple of anything: scalar paths of the row kernels, ragged tiles everywhere, a convolution of one tap
    "odd": M.config([(D(heads=3, kv_heads=3, dim=7, vdim=5, conv=1), 35), (S(heads=5, groups=1, state=11, vdim=7, conv=5, norm_groups=5), None),
                     (A(heads=3, kv_heads=1, dim=5, vdim=9, chunk=13), 17), (S(heads=3, groups=3, state=1, vdim=3, conv=2, norm_groups=1), None)], loop=(0, 1, 2), width=67, vocab=101),
    # heads of real models
    "heads": M.config([(D(heads=4, kv_heads=2, dim=128, vdim=128), None), (S(heads=4, groups=2, state=128, vdim=64, conv=4, norm_groups=1), 96),
                       (A(heads=16, kv_heads=2, dim=128, vdim=64, chunk=70, scale=0.09), 96), (A(heads=4, kv_heads=4, dim=64, vdim=128, chunk=300, scale=0.12), None)], width=128, vocab=300),
    # keys and states at and beyond what the tile kernels hold
    "wide": M.config([(D(heads=2, kv_heads=2, dim=192, vdim=80), None), (S(heads=2, groups=1, state=300, vdim=40, conv=4, norm_groups=2), 64),
                      (A(heads=3, kv_heads=1, dim=256, vdim=256, chunk=50, scale=0.06), None), (A(heads=20, kv_heads=1, dim=272, vdim=300, chunk=33, scale=0.06), 40)], width=96, vocab=130),
    "plain": M.config([(D(heads=4, kv_heads=4, dim=32, vdim=32), 64), (S(heads=4, groups=1, state=32, vdim=32, conv=4, norm_groups=1), 64), (A(heads=4, kv_heads=2, dim=32, vdim=32, chunk=40), 64)], width=64, vocab=150),
}


@pytest.fixture(scope="module")
def make(gpu, tmp_path_factory):
    from skainet_b200.fomalix import Fomalix
    made = []

    def build(cfg, w, dtype, **kw):
        path = M.save(tmp_path_factory.mktemp("model"), cfg, w)
        made.append(Fomalix.from_dir(path, dtype=dtype, **{"max_seq": 400, **kw}))
        return made[-1]
    yield build
    for m in made:
        m.free()
    from skainet_b200 import _lib
    assert _lib.lib().skainet_cuda_device_status() == 0


_models = {}


@pytest.fixture
def small(make):
    """(config, weights, model) by configuration name and dtype; passes of at most 48 rows, so caches wrap and prompts are cut."""
    def get(name, dtype, **kw):
        key = (name, dtype, tuple(kw.items()))
        if key not in _models:
            w = M.random_weights(CONFIGS[name], seed=len(name))
            _models[key] = (CONFIGS[name], w, make(CONFIGS[name], w, dtype, **{"prefill_rows": 48, **kw}))
        _models[key][2].reset()
        return _models[key]
    return get


_refs = {}


def reference(name, n, seed=7):
    """(tokens, logits, stream after every layer run) of a named configuration; computed once."""
    if (name, n, seed) not in _refs:
        cfg, trace = CONFIGS[name], []
        t = M.tokens(cfg, n, seed)
        _refs[name, n, seed] = (t, F.forward(cfg, M.random_weights(cfg, seed=len(name)), t, trace), trace)
    return _refs[name, n, seed]


def portions(m, t, cut, seq=0):
    """Logits of every token of t, run in portions of the given sizes."""
    rows, p = [], 0
    for k in cut:
        rows.append(m.forward(t[p:p + k], list(range(k)), seq))
        p += k
    return np.concatenate(rows)


# ---- mechanisms alone -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mixer", [
    D(), D(heads=4, kv_heads=4, dim=128, vdim=128), D(heads=2, kv_heads=1, dim=48, vdim=200, conv=3), D(heads=8, kv_heads=2, dim=16, vdim=16, conv=2), D(heads=1, kv_heads=1, dim=3, vdim=5, conv=1), D(heads=1, kv_heads=1, dim=16, vdim=520), D(heads=2, kv_heads=2, dim=256, vdim=96),
    S(), S(heads=4, groups=4, state=128, vdim=64, conv=4, norm_groups=1), S(heads=10, groups=2, state=16, vdim=64, conv=4, norm_groups=1), S(heads=3, groups=1, state=40, vdim=343, norm_groups=1), S(heads=4, groups=1, state=240, vdim=64, norm_groups=4), S(heads=2, groups=1, state=200, vdim=17, conv=2, norm_groups=2), S(heads=8, groups=2, state=16, vdim=64, conv=4, norm_groups=8), S(heads=1, groups=1, state=1, vdim=3, conv=1, norm_groups=1),
    A(), A(heads=8, kv_heads=1, dim=128, vdim=128, chunk=64, scale=0.1), A(heads=5, kv_heads=5, dim=40, vdim=24, chunk=100, scale=0.4), A(heads=12, kv_heads=4, dim=64, vdim=192, chunk=150, scale=0.2), A(heads=40, kv_heads=2, dim=24, vdim=40, chunk=1000, scale=0.4), A(heads=1, kv_heads=1, dim=1, vdim=1, chunk=1, scale=1.0),
], ids=lambda m: f"{m[0]}-{'-'.join(str(v) for v in m[1].values() if not isinstance(v, dict))}")
def test_one_mixer_in_prompts_and_decoding(make, dtype, mixer):
    """One layer without a feed-forward: whole prompts, then portions on both sides of every tile size, then single tokens."""
    cfg = M.config([(mixer, None)], width=64)
    w = M.random_weights(cfg, 11)
    m = make(cfg, w, dtype, prefill_rows=160)
    n = 330
    t = M.tokens(cfg, n, 5)
    ref = F.forward(cfg, w, t)
    for cut in ([n], [64, 65, 63, 128, 10], [16, 17, 15, 2, 3, 1, 31, 33, 32, 180], [200] + [1] * 40):
        m.reset()
        got = portions(m, t, cut)
        assert M.error(got, ref[:len(got)]) < TOL[dtype], cut[:4]


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer(make, dtype):
    cfg = CONFIGS["mixed"]
    w = M.random_weights(cfg, 5)
    t, W = M.tokens(cfg, 40), cfg["width"]
    for k in range(1, len(cfg["layers"]) + 1):
        c = dict(cfg, layers=cfg["layers"][:k], loop=dict(start=min(1, k - 1), stop=min(4, k), times=3))
        trace = []
        F.forward(c, w, t, trace)
        m = make(c, {n: v for n, v in w.items() if n[0] != "l" or int(n[1]) < k}, dtype)
        m.forward(t)
        assert M.error(m.peek(0, 40 * W).reshape(40, W), trace[-1]) < TOL[dtype], k


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_keep_their_vector(make, dtype):
    """A layer that adds nothing leaves embedding and position vector, which the final norm and the head turn into logits."""
    cfg = M.config([(A(chunk=4), None)], width=64, scale=1.0)
    w = M.random_weights(cfg, 3)
    w["l0.norm1b"] *= 0.0
    m = make(cfg, w, dtype, max_seq=70000, prefill_rows=4096)
    t = M.tokens(cfg, 69000)
    at = [0, 1, 4095, 4096, 33333, 68998, 68999]
    x = w["embed"][np.array(t)[at]] + F.sinusoid(at, 64)
    assert M.error(m.forward(t, at), F.rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T) < (1e-5 if dtype == "float32" else 0.02)


# ---- whole models ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_oracle(small, name, dtype):
    cfg, w, m = small(name, dtype)
    n = 200
    t, ref, _ = reference(name, n)
    for cut in ([n], [150] + [1] * 50, [2] * 100, [3, 1, 2, 5, 48, 49, 7, 20, 64, 1], [1] * 90 + [110]):
        m.reset()
        assert sum(cut) == n and M.error(portions(m, t, cut), ref) < TOL[dtype], cut[:4]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 2, 15, 64, 65, 100])
def test_chunk_edges_in_prompts_and_decoding(make, dtype, chunk):
    """A marked token is seen to the end of its chunk and by no later position, whichever step brings them."""
    cfg = M.config([(A(heads=4, kv_heads=2, dim=16, vdim=16, chunk=chunk, scale=0.4), 40)], width=64)
    w = M.plant_marker(cfg, M.random_weights(cfg, chunk))
    m = make(cfg, w, dtype, prefill_rows=40)
    n, at = 240, 67
    t = M.tokens(cfg, n)
    s = list(t)
    s[at] = M.MARK
    last = at // chunk * chunk + chunk - 1
    ref = F.forward(cfg, w, s)
    for cut in ([n], [at + 1] + [1] * (n - at - 1), [at, 2] + [3] * ((n - at - 2) // 3), [last + 1] + [2] * ((n - last - 1) // 2), [last] + [1] * 30):
        out = []
        for seq in (t, s):
            m.reset()
            out.append(portions(m, seq, cut))
        plain, marked = out
        assert M.error(marked, ref[:len(marked)]) < TOL[dtype], cut[:4]
        assert np.array_equal(plain[last + 1:], marked[last + 1:]) and np.array_equal(plain[:at], marked[:at]), cut[:4]
        seen = [M.error(marked[p:p + 1], plain[p:p + 1]) for p in range(at, min(last + 1, len(marked)))]
        assert not seen or min(seen) > 0.05, (cut[:4], seen)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", [-30.0, 0.0, 6.0, 60.0])
def test_sinks_of_every_strength(make, dtype, sink):
    """Scores reach dim * scale = 6.4: sinks far below, among and far above them, over one key and over many, split and whole."""
    cfg = M.config([(A(heads=4, kv_heads=2, dim=16, vdim=16, chunk=3000, scale=0.4), None)], width=64)
    w = M.random_weights(cfg, 2)
    w["l0.mix.sink"][:] = sink
    m = make(cfg, w, dtype, max_seq=1600, prefill_rows=1000)
    t = M.tokens(cfg, 1500, 4)
    ref = F.forward(cfg, w, t)
    at = [0, 1, 2, 63, 64, 500, 1200, 1499]
    assert M.error(m.forward(t, at), ref[at]) < TOL[dtype]
    m.reset()
    m.forward(t[:1480])
    assert M.error(np.concatenate([m.forward([k], [0]) for k in t[1480:]]), ref[1480:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mixer", [D(heads=4, kv_heads=2, dim=32, vdim=32), S(heads=4, groups=2, state=32, vdim=32, norm_groups=1)], ids=["delta", "mamba2"])
def test_a_far_write_survives_every_cut(make, dtype, mixer):
    """With almost no decay a write early in the sequence shows hundreds of tokens later, and whatever cut the prompt keeps it."""
    cfg = M.config([(mixer, None)], width=64)
    w = M.plant_write(cfg, M.random_weights(cfg, 8))
    m = make(cfg, w, dtype, max_seq=700, prefill_rows=256)
    t = M.tokens(cfg, 600, 6)
    s = list(t)
    s[3] = M.MARK
    ref = F.forward(cfg, w, s)
    assert M.error(F.forward(cfg, w, t)[-1:], ref[-1:]) > 0.15
    for cut in ([600], [4] + [149] * 4, [5, 95, 64, 36, 300, 100], [2] * 30 + [500] + [1] * 40):
        m.reset()
        assert M.error(portions(m, s, cut), ref) < 0.6 * TOL[dtype], cut[:3]


@pytest.mark.parametrize("dtype", DTYPES)
def test_strong_decay_and_wide_ranges_stay_finite(make, dtype):
    """Decays that underflow within a few tokens, step sizes far from one and large values."""
    cfg = M.config([(D(heads=4, kv_heads=2, dim=32, vdim=32), None), (S(heads=4, groups=2, state=32, vdim=32, norm_groups=1), None)], width=64)
    w = M.random_weights(cfg, 8)
    for l in range(2):
        w[f"l{l}.mix.A_log"][:] = [6.0, 3.0, -9.0, 0.0]
        w[f"l{l}.mix.dt_bias"][:] = [4.0, -6.0, 2.0, 30.0]
    w["l0.mix.v"] *= 64.0
    w["l1.mix.in"][:] *= 16.0
    m = make(cfg, w, dtype, prefill_rows=200)
    t = M.tokens(cfg, 200, 6)
    ref = F.forward(cfg, w, t)
    for cut in ([200], [100] + [1] * 20, [16] * 12):
        m.reset()
        got = portions(m, t, cut)
        assert M.error(got, ref[:len(got)]) < 2 * TOL[dtype], cut[:3]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_the_ring_many_times(small, dtype):
    cfg, w, m = small("plain", dtype, prefill_rows=8)
    t, ref, _ = reference("plain", 380, 3)
    got = [m.forward(t[:5], [4])] + [m.forward([k], [0]) for k in t[5:]]
    assert M.error(np.concatenate(got), ref[4:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [2, 4, 7, 20])
def test_batched_decoding_of_unequal_sequences(small, dtype, batch):
    """Each sequence of a batch gets the logits it gets alone, through the streaming and the tensor-core linears."""
    cfg, w, m = small("mixed", dtype, max_batch=20)
    seqs = [M.tokens(cfg, 3 + (17 * b) % 90, 50 + b) for b in range(batch)]
    for b, t in enumerate(seqs):
        m.prefill(t[:-1], b, want_next=False)
    tin, tout = np.array([t[-1] for t in seqs], np.int32), np.zeros(batch, np.int32)
    for step in range(4):
        m.decode(tin, tout)
        got = m.logits(batch)
        ref = np.stack([F.forward(cfg, w, t)[-1] for t in seqs])
        assert M.error(got, ref) < TOL[dtype], step
        assert tout.tolist() == got.argmax(-1).tolist()
        tin = np.array([(7 * step + 3 * b) % cfg["vocab"] for b in range(batch)], np.int32)      # not the greedy ones: unequal inputs
        for b in range(batch):
            seqs[b].append(int(tin[b]))


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_mates_and_slots_do_not_matter(small, dtype):
    """The same sequence in every slot of a batch, at every slot's own time, gives the same logits bit for bit."""
    cfg, w, m = small("mixed", dtype, max_batch=20)
    t = M.tokens(cfg, 60, 3)
    for b in (0, 3, 6):
        m.prefill(t[:50], b, want_next=False)
    for b in (1, 2, 4, 5):
        m.prefill(M.tokens(cfg, 20 + b, b), b, want_next=False)
    tout = np.zeros(7, np.int32)
    for k in t[50:]:
        m.decode(np.array([k, 5, 6, k, 7, 8, k], np.int32), tout)
        got = m.logits(7)
        assert np.array_equal(got[0], got[3]) and np.array_equal(got[0], got[6])
    assert M.error(got[:1], F.forward(cfg, w, t)[-1:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_freed_slots_are_used_again(small, dtype):
    cfg, w, m = small("mixed", dtype, max_batch=3)
    t, u = M.tokens(cfg, 120, 1), M.tokens(cfg, 33, 2)
    first = [m.forward(u, list(range(33)), s) for s in (m.acquire(), m.acquire())]
    assert np.array_equal(first[0], first[1])                      # the slot does not matter
    m.forward(t, (), m.acquire())
    for s in (1, 2, 0):
        m.release(s)
    ref = F.forward(cfg, w, u + [5])
    for _ in range(3):
        s = m.acquire()
        assert np.array_equal(m.forward(u, list(range(33)), s), first[0])      # nor what it held before
        assert M.error(m.forward([5], [0], s), ref[-1:]) < TOL[dtype]
    for s in range(3):
        m.release(s)
    s = m.acquire()                                                # a slot that is used again from its first token on, one by one
    got = np.concatenate([m.forward([k], [0], s) for k in u])
    assert M.error(got, ref[:33]) < TOL[dtype]
    m.release(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_in_any_order_and_number(small, dtype):
    cfg, w, m = small("plain", dtype)
    t = M.tokens(cfg, 130)
    every = m.forward(t, list(range(130)))
    want = [129, 0, 47, 48, 49, 0, 95, 96] + list(range(100, 10, -1))
    m.reset()
    assert np.abs(m.forward(t, want) - every[want]).max() < (1e-4 if dtype == "float32" else 0.05)
    m.reset()
    assert m.forward(t[:9]).shape == (0, cfg["vocab"])
    with pytest.raises(ValueError, match="outside"):
        m.forward([1], [1])
    with pytest.raises(ValueError, match="vocabulary"):
        m.forward([cfg["vocab"]], [0])
    with pytest.raises(ValueError, match="max_seq"):
        m.forward([1] * 392, [0])


def test_greedy_generation_through_the_registry_and_the_command_line(gpu, tmp_path):
    from skainet_b200 import models
    cfg = CONFIGS["mixed"]
    w = M.random_weights(cfg, 20)
    path = M.save(tmp_path, cfg, w)
    prompt, steps = M.tokens(cfg, 19), 14
    seq, margins = list(prompt), []
    for _ in range(steps):
        row = F.forward(cfg, w, seq)[-1]
        top = np.sort(row)[-2:]
        margins.append(top[1] - top[0])
        seq.append(int(row.argmax()))
    assert min(margins) > 1e-2                                     # no token hangs on rounding
    m = models.load_model(path, "float32", max_seq=64)
    for _ in range(2):
        assert models.generate(m, prompt, steps) == seq[19:]
    m.free()
    out = subprocess.run([sys.executable, "-m", "skainet_b200.models", "--model", path, "--tokens", ",".join(map(str, prompt)), "--steps", str(steps), "--dtype", "float32"],
                         cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0 and out.stdout.strip() == ",".join(map(str, seq[19:])), out.stderr[-2000:]


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_replays_steps(gpu, tmp_path, dtype):
    cfg = CONFIGS["plain"]
    w = M.random_weights(cfg, 5)
    path = M.save(tmp_path / "m", cfg, w)
    a, b = M.tokens(cfg, 70, 1), M.tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [3, 59]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[60:68], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[68:69], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [8, 0]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "70"],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {k}" for k in range(5)], r.stderr[-2000:]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    ra, rb = F.forward(cfg, w, a), F.forward(cfg, w, b)
    for k, ref in ((0, ra[[3, 59]]), (2, ra[[68]]), (3, ra[[69]]), (4, rb[[8, 0]])):
        got = np.fromfile(out / f"{k}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert M.error(got, ref) < TOL[dtype], k


def test_missing_and_misshaped_tensors_are_named(gpu, tmp_path):
    from skainet_b200.fomalix import Fomalix
    cfg = CONFIGS["plain"]
    w = M.random_weights(cfg)
    for name in ("l0.mix.v.conv", "l1.mix.conv.b", "l2.mix.sink", "l2.norm2b", "final.norm"):
        v = dict(w)
        del v[name]
        with pytest.raises(ValueError, match=name):
            Fomalix.from_dir(M.save(tmp_path, cfg, v))
    for name in ("l0.mix.a", "l2.mix.k.b", "l1.mix.norm"):
        v = dict(w)
        v[name] = v[name][:-1]
        with pytest.raises(ValueError, match=name):
            Fomalix.from_dir(M.save(tmp_path, cfg, v))
