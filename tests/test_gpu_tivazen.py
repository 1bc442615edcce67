"""GPU: the Tivazen design and the mechanisms it added, against the plain oracle, through the framework's own loader, cache,
steps and scheduler. fp32 models are held to fp32 rounding, bf16 models to bf16 rounding."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import tivazen_models as M
from oracle import tivazen as T

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 0.12}
DTYPES = ("float32", "bfloat16")

A, D, X = M.attn, M.dense, M.moe
CONFIGS = {
    # every branch at once: shared caches with other windows and head counts, routed, dense and absent feed-forward, odd sizes
    "mixed": M.config([(A(), D()), (A(kv_from=0, window=4, heads=5, dim=12, vdim=9, scale=0.2), X()), (A(kv_rank=33, rot_dim=2, window=30, base=100.0), None),
                       (A(kv_from=2, kv_rank=33, rot_dim=2, base=100.0, window=17), X(7, 1, 10)), (A(kv_from=0, window=21), D(50))]),
    # more heads than one MMA row group and more than one group of rows, a window across several key tiles
    "heads": M.config([(A(heads=20, dim=32, rot_dim=16, vdim=24, kv_rank=64, window=70), D(96)), (A(heads=70, dim=8, rot_dim=4, vdim=6, kv_rank=40, window=150), X(16, 1, 40))], width=128, vocab=300),
    # the widest latent the tile kernel holds, and one beyond it
    "wide": M.config([(A(heads=4, dim=64, rot_dim=64, vdim=40, kv_rank=512, window=33, scale=0.05), D(64)), (A(heads=3, dim=16, rot_dim=8, vdim=20, kv_rank=560, window=50, scale=0.05), None)], width=96, vocab=130),
    # nothing a multiple of anything: scalar paths of the row kernels, ragged tiles everywhere
    "odd": M.config([(A(heads=3, dim=7, rot_dim=2, vdim=5, kv_rank=17, window=11), D(35)), (A(heads=7, dim=5, rot_dim=2, vdim=3, kv_rank=17, window=29, kv_from=0), X(9, 4, 13)), (A(heads=2, dim=1, rot_dim=4, vdim=9, kv_rank=13, window=300), None)], width=67, vocab=101),
    "plain": M.config([(A(heads=8, dim=16, rot_dim=8, vdim=16, kv_rank=48, window=40), D(64)), (A(heads=8, dim=16, rot_dim=8, vdim=16, kv_rank=48, window=40), X(8, 2, 32))], width=64, vocab=150),
}


@pytest.fixture(scope="module")
def make(gpu, tmp_path_factory):
    from skainet_b200.tivazen import Tivazen
    made = []

    def build(cfg, w, dtype, **kw):
        path = M.save(tmp_path_factory.mktemp("model"), cfg, w)
        made.append(Tivazen.from_dir(path, dtype=dtype, **{"max_seq": 400, **kw}))
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


# ---- mechanisms alone -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,cols", [(1, 1), (17, 8), (100, 72), (130, 64), (300, 200), (512, 328)])
def test_bf16_linear_at_every_row_count(gpu, rows, cols):
    """The streaming, tensor-core and fp32 kernels over one weight; row counts on both sides of every switch and tile edge."""
    rng = np.random.default_rng(rows)
    h = M.round_bf16(rng.standard_normal((rows, cols)))
    w = gpu.Weight.upload(h.view(np.uint8), "BF16", rows, cols)
    assert np.array_equal(w.export().view(np.uint16), h.reshape(-1)) and np.array_equal(w.dequant(), M.widen(h).astype(np.float32))
    for m in (1, 2, 7, 8, 9, 16, 17, 31, 33, 64, 127, 129, 300):
        x = rng.standard_normal((m, cols)).astype(np.float32)
        xb = M.widen(M.round_bf16(x))
        scale = np.sqrt(cols)
        assert np.abs(gpu.matmul_host(w, x) - xb @ M.widen(h).T).max() < 2e-6 * scale * 10, m
        assert np.abs(gpu.matmul_host(w, x, 1) - x.astype(np.float64) @ M.widen(h).T).max() < 2e-6 * scale * 10, m
    w.free()


def test_bf16_linear_wide_tiles(gpu):
    """A product large enough for the tiles of 256 weight rows on every SM, several tiles per CTA, with a ragged last one."""
    rng = np.random.default_rng(5)
    rows, cols, m = 256 * 45 + 60, 192, 1000
    h = M.round_bf16(rng.standard_normal((rows, cols)))
    w = gpu.Weight.upload(h.view(np.uint8), "BF16", rows, cols)
    x = M.widen(M.round_bf16(rng.standard_normal((m, cols)))).astype(np.float32)
    ref = x @ M.widen(h).T.astype(np.float32)
    assert np.abs(gpu.matmul_host(w, x) - ref).max() < 2e-4
    w.free()


def test_bf16_embedding_rows_and_concat(gpu):
    h = M.round_bf16(np.random.default_rng(1).standard_normal((30, 20)))
    w = gpu.Weight.upload(h.view(np.uint8), "BF16", 30, 20)
    ids, out = gpu.DeviceBuffer.from_host(np.array([3, 29, 0], np.int32)), gpu.DeviceBuffer(3 * 20 * 4)
    gpu.embed(w, ids.ptr, 3, out.ptr)
    assert np.array_equal(out.download(np.float32, 60).reshape(3, 20), M.widen(h)[[3, 29, 0]])
    c = gpu.concat_rows(w, w)
    assert np.array_equal(c.export().view(np.uint16), np.concatenate([h, h]).reshape(-1))
    with pytest.raises(ValueError, match="row-major"):
        gpu.Weight.upload(h.view(np.uint8), "BF16", 30, 20, 1)


@pytest.mark.parametrize("dtype", DTYPES)
def test_depth_average_and_states(make, dtype):
    """Every state X_j of a prompt, and the stream after the last average."""
    cfg = CONFIGS["mixed"]
    w = M.random_weights(cfg, 9)
    m = make(cfg, w, dtype)
    t, trace = M.tokens(cfg, 40), []
    T.forward(cfg, w, t, trace)
    m.forward(t)
    W = cfg["width"]
    states = [m.peek(16 + j, 40 * W).reshape(40, W).astype(np.float64) for j in range(len(cfg["layers"]) + 1)]
    assert np.array_equal(states[0], w["embed"][t])
    for i, x in enumerate(trace):
        assert M.error(T.depth_average(w[f"l{i}.dwa"], states), x) < TOL[dtype], i
    assert M.error(m.peek(0, 40 * W).reshape(40, W), trace[-1]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top", [(1, 1), (4, 2), (40, 2), (40, 7), (6, 6)])
def test_routing_by_row_count(make, dtype, experts, top):
    """One routed layer: the one-CTA and the many-slot routing, runs of 8, 32 and 128 rows of an expert."""
    cfg = M.config([(A(window=5), X(experts, top, 24))], width=64)
    w = M.random_weights(cfg, 3)
    rng = np.random.default_rng(experts)
    m = make(cfg, w, dtype, max_seq=800, prefill_rows=700)
    for n in (1, 3, 30, 200, 700):
        t = rng.integers(0, cfg["vocab"], n).tolist()
        m.reset()
        want = list(range(max(0, n - 40), n))
        assert M.error(m.forward(t, want), T.forward(cfg, w, t)[want]) < TOL[dtype], n


@pytest.mark.parametrize("dtype", DTYPES)
def test_expert_weight_multiplies_the_input(make, dtype):
    """With a score well below one, scaling the input and scaling the output differ far beyond rounding."""
    cfg = M.config([(A(window=3), X(3, 1, 24))], width=64)
    w = M.random_weights(cfg, 4)
    w["l0.mlp.router"] *= 0.0
    w["l0.mlp.router"][1, 0] = 0.25
    w["embed"][:, 0] = 1.0
    w["l0.mix.o"][0] = 0.0
    m, t = make(cfg, w, dtype), M.tokens(cfg, 30)
    assert M.error(m.forward(t, list(range(30))), T.forward(cfg, w, t)) < TOL[dtype]


# ---- whole models ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_oracle(small, name, dtype):
    cfg, w, m = small(name, dtype)
    n = 200
    t = M.tokens(cfg, n, 7)
    ref = T.forward(cfg, w, t)
    for cut in ([n], [150] + [1] * 50, [2] * 100, [3, 1, 2, 5, 48, 49, 7, 20, 64, 1], [1] * 90 + [110]):
        m.reset()
        at, rows = 0, []
        for k in cut:
            rows.append(m.forward(t[at:at + k], list(range(k))))
            at += k
        got = np.concatenate(rows)
        assert at == n and M.error(np.concatenate(rows), ref) < TOL[dtype], cut[:4]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 15, 64, 65, 100])
def test_window_edges_in_prompts_and_decoding(make, dtype, window):
    """A marked token is seen by the window - 1 positions after it and by no later one, whichever step brings them."""
    cfg = M.config([(A(heads=4, dim=16, rot_dim=8, vdim=16, kv_rank=32, window=window), D(40))], width=64)
    w = M.plant_marker(cfg, M.random_weights(cfg, window))
    m = make(cfg, w, dtype, prefill_rows=40)
    n, at = 200, 60
    t = M.tokens(cfg, n)
    s = list(t)
    s[at] = M.MARK
    last = at + window - 1
    ref = T.forward(cfg, w, s)
    for cut in ([n], [at + 1] + [1] * (n - at - 1), [at, 2] + [3] * ((n - at - 2) // 3), [last + 1] + [2] * ((n - last - 1) // 2), [last] + [1] * 30):
        out = []
        for seq in (t, s):
            m.reset()
            rows, p = [], 0
            for k in cut:
                rows.append(m.forward(seq[p:p + k], list(range(k))))
                p += k
            out.append(np.concatenate(rows))
        plain, marked = out
        assert M.error(marked, ref[:len(marked)]) < TOL[dtype], cut[:4]
        assert np.array_equal(plain[last + 1:], marked[last + 1:]) and np.array_equal(plain[:at], marked[:at]), cut[:4]
        seen = [M.error(marked[p:p + 1], plain[p:p + 1]) for p in range(at, min(last + 1, len(marked)))]
        assert min(seen) > 0.05, (cut[:4], seen)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_borrowed_cache_keeps_its_own_window(make, dtype):
    """Layer 1 reads layer 0's latents through a wider window of its own: the ring holds what the widest reader sees."""
    cfg = M.config([(A(heads=4, dim=16, rot_dim=8, vdim=16, kv_rank=32, window=3), None), (A(heads=5, dim=12, rot_dim=8, vdim=10, kv_rank=32, window=77, kv_from=0), D(40))], width=64)
    w = M.plant_marker(cfg, M.random_weights(cfg, 2), layer=1)
    w["l1.dwa"][:] = [0.2, 0.3, 1.0]
    w = {k: M.widen(M.round_bf16(v)).reshape(v.shape) for k, v in w.items()}
    m = make(cfg, w, dtype, prefill_rows=20)
    t = M.tokens(cfg, 180)
    t[50] = M.MARK
    ref = T.forward(cfg, w, t)
    for cut in ([180], [55] + [1] * 125, [7] * 25):
        m.reset()
        rows, p = [], 0
        for k in cut:
            rows.append(m.forward(t[p:p + k], list(range(k))))
            p += k
        got = np.concatenate(rows)
        assert M.error(got, ref[:len(got)]) < TOL[dtype], cut[:3]
    other = list(t)
    other[50] = 2
    assert M.error(T.forward(cfg, w, other)[126:127], ref[126:127]) > 0.05      # the far edge of the wide window really shows


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_the_ring_many_times(small, dtype):
    cfg, w, m = small("plain", dtype, prefill_rows=8)
    t = M.tokens(cfg, 380, 3)
    ref = T.forward(cfg, w, t)
    got = [m.forward(t[:5], [4])] + [m.forward([k], [0]) for k in t[5:]]
    assert M.error(np.concatenate(got), ref[4:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [2, 4, 7, 20])
def test_batched_decoding_of_unequal_sequences(small, dtype, batch):
    """Each sequence of a batch gets the logits it gets alone, through the few-row, the streaming and the tensor-core kernels."""
    cfg, w, m = small("mixed", dtype, max_batch=20)
    seqs = [M.tokens(cfg, 3 + (17 * b) % 90, 50 + b) for b in range(batch)]
    for b, t in enumerate(seqs):
        m.prefill(t[:-1], b, want_next=False)
    tin, tout = np.array([t[-1] for t in seqs], np.int32), np.zeros(batch, np.int32)
    for step in range(6):
        m.decode(tin, tout)
        got = m.logits(batch)
        ref = np.stack([T.forward(cfg, w, t)[-1] for t in seqs])
        assert M.error(got, ref) < TOL[dtype], step
        assert tout.tolist() == got.argmax(-1).tolist()
        tin = np.array([(7 * step + 3 * b) % cfg["vocab"] for b in range(batch)], np.int32)      # not the greedy ones: unequal inputs
        for b in range(batch):
            seqs[b].append(int(tin[b]))


@pytest.mark.parametrize("dtype", DTYPES)
def test_freed_slots_are_used_again(small, dtype):
    cfg, w, m = small("mixed", dtype, max_batch=3)
    t, u = M.tokens(cfg, 120, 1), M.tokens(cfg, 33, 2)
    first = [m.forward(u, list(range(33)), s) for s in (m.acquire(), m.acquire())]
    assert np.array_equal(first[0], first[1])                      # the slot does not matter
    m.forward(t, (), m.acquire())
    for s in (1, 2, 0):
        m.release(s)
    for _ in range(3):
        s = m.acquire()
        assert np.array_equal(m.forward(u, list(range(33)), s), first[0])      # nor what it held before
        tail = m.forward([5], [0], s)
        assert M.error(tail, T.forward(cfg, w, u + [5])[-1:]) < TOL[dtype]
    for s in range(3):
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
    w = M.random_weights(cfg, 12)
    path = M.save(tmp_path, cfg, w)
    prompt, steps = M.tokens(cfg, 19), 14
    seq, margins = list(prompt), []
    for _ in range(steps):
        row = T.forward(cfg, w, seq)[-1]
        top = np.sort(row)[-2:]
        margins.append(top[1] - top[0])
        seq.append(int(row.argmax()))
    assert min(margins) > 1e-3                                     # no token hangs on rounding
    m = models.load_model(path, "float32", max_seq=64)
    for _ in range(2):
        assert models.generate(m, prompt, steps) == seq[19:]
    m.free()
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, "-m", "skainet_b200.models", "--model", path, "--tokens", ",".join(map(str, prompt)), "--steps", str(steps), "--dtype", "float32"],
                         cwd=root, capture_output=True, text=True, timeout=300)
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
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "70"],
                       input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {k}" for k in range(5)], r.stderr[-2000:]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    ra, rb = T.forward(cfg, w, a), T.forward(cfg, w, b)
    for k, ref in ((0, ra[[3, 59]]), (2, ra[[68]]), (3, ra[[69]]), (4, rb[[8, 0]])):
        got = np.fromfile(out / f"{k}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert M.error(got, ref) < TOL[dtype], k


def test_missing_and_misshaped_tensors_are_named(gpu, tmp_path):
    from skainet_b200.tivazen import Tivazen
    cfg = CONFIGS["plain"]
    w = M.random_weights(cfg)
    for name, text in (("l1.mlp.e3.up", "l1.mlp.e3.up"), ("l0.dwa", "l0.dwa"), ("final.norm", "final.norm")):
        v = dict(w)
        del v[name]
        with pytest.raises(ValueError, match=text):
            Tivazen.from_dir(M.save(tmp_path, cfg, v))
    v = dict(w)
    v["l0.mix.uk"] = v["l0.mix.uk"][:-1]
    with pytest.raises(ValueError, match="l0.mix.uk"):
        Tivazen.from_dir(M.save(tmp_path, cfg, v))


# ---- the runtime the designs share -------------------------------------------------------------------------------------------
def test_llama_forward_and_slots(gpu):
    """The shared entries on the other design: logits of chosen prompt places, a decoded token, a slot emptied and used again."""
    from skainet_b200.llama import Llama, LlamaConfig
    m = Llama(LlamaConfig(2, 512, 8, 4, 64, 1024, 1000, max_seq=64, max_batch=2))
    m.synth(seed=3, std=0.05)
    m.finalize()
    t = list(range(5, 25))
    nxt = m.prefill(t, 0)
    m.reset(0)
    lg = m.forward(t, [19, 4])
    assert lg.shape == (2, 1000) and int(lg[0].argmax()) == nxt
    one = m.forward([7], [0])
    assert np.array_equal(one, m.logits(1))
    s = m.acquire(), m.acquire()
    assert s == (0, 1) and np.array_equal(m.forward(t, [19, 4], 0), lg) and np.array_equal(m.forward(t, [19, 4], 1), lg)
    m.release(0)
    assert m.acquire() == 0 and np.array_equal(m.forward(t, [19, 4], 0), lg)
    m.free()


def test_llama_from_gguf_by_the_registry(gpu, oracle, tmp_path):
    from test_ops_gguf import write_gguf
    from skainet_b200 import models
    from skainet_b200.llama import Llama, LlamaConfig, W_EMBED, W_HEAD
    cfg = LlamaConfig(1, 256, 4, 2, 64, 512, 300, rope_theta=5000.0, max_seq=48)
    m = Llama(cfg)
    m.synth(seed=8, std=0.05)
    parts = {n: m.export_weight(0, k) for n, k in (("attn_q", 4), ("attn_k", 5), ("attn_v", 6), ("attn_output", 7), ("ffn_gate", 9), ("ffn_up", 10), ("ffn_down", 11))}
    shapes = {"attn_q": (256, 256), "attn_k": (128, 256), "attn_v": (128, 256), "attn_output": (256, 256), "ffn_gate": (512, 256), "ffn_up": (512, 256), "ffn_down": (256, 512)}
    ones = np.ones(256, np.float32).tobytes()
    tensors = [("token_embd.weight", (300, 256), 8, m.export_weight(0, W_EMBED)), ("output.weight", (300, 256), 8, m.export_weight(0, W_HEAD)), ("output_norm.weight", (256,), 0, ones)]
    tensors += [(f"blk.0.{n}.weight", shapes[n], 12, b) for n, b in parts.items()] + [(f"blk.0.{n}.weight", (256,), 0, ones) for n in ("attn_norm", "ffn_norm")]
    path = str(tmp_path / "m.gguf")
    u = lambda v: (4, v)
    write_gguf(path, tensors, {"general.architecture": (8, "llama"), "llama.block_count": u(1), "llama.embedding_length": u(256), "llama.attention.head_count": u(4),
                               "llama.attention.head_count_kv": u(2), "llama.feed_forward_length": u(512), "llama.rope.freq_base": (6, 5000.0),
                               "llama.attention.layer_norm_rms_epsilon": (6, 1e-5)})
    m.finalize()
    g = models.load_model(path, max_seq=48)
    assert models.generate(g, [3, 9, 250, 7], 10) == models.generate(m, [3, 9, 250, 7], 10)
    m.free(); g.free()
