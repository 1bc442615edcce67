"""Small Fomalix configurations and weights for the tests: random ones, and ones in which a single key stands out so that a
chunk edge that is one token off, a lost key or a sink that is left out changes the logits beyond any rounding."""
import json
import os

import numpy as np

from tivazen_models import MARK, error, round_bf16, tokens, widen  # noqa: F401


def attn(heads=6, kv_heads=2, dim=14, vdim=18, chunk=9, scale=0.35):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": scale}


def delta(heads=6, kv_heads=3, dim=20, vdim=12, conv=4):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def mamba(heads=6, groups=2, state=24, vdim=10, conv=3, norm_groups=3):
    return "mamba2", {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}


def config(layers, loop=None, width=72, vocab=97, eps=1e-3, scale=3.0):
    """layers: (mixer, feed-forward size or None); loop: (start, stop, times)."""
    return {"architecture": "Fomalix", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None,
            "layers": [{"type": t, "mixer": dict(m), "mlp": {"kind": "dense", "ff": ff} if ff else None} for (t, m), ff in layers]}


def random_weights(cfg, seed=0):
    """name -> float64 array of bfloat16 values. Decays run from almost none to strong, so far writes and near ones both show."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = gain * rng.standard_normal((rows, cols)) / np.sqrt(cols)

    def gains(name, n):
        w[name] = 1 + 0.3 * rng.standard_normal(n)

    def taps(name, channels, n):
        w[name] = rng.standard_normal((channels, n)) / np.sqrt(n)

    w["embed"] = rng.standard_normal((V, W))
    mat("head", V, W)
    gains("final.norm", W)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        x = p + "mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            gains(p + n, W)
        H, inner = m["heads"], m["heads"] * m["vdim"]
        mat(x + "o", W, inner)
        if l["type"] == "attention":
            for c, n in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                mat(x + c, n, W)
                w[f"{x}{c}.b"] = 0.5 * rng.standard_normal(n)
            w[x + "sink"] = rng.uniform(-1, 4, H)
        else:
            w[x + "A_log"], w[x + "dt_bias"] = np.resize([-6.0, 0.0, -3.0, 1.0], H) + 0.2 * rng.standard_normal(H), rng.uniform(-2, 0.5, H)
        if l["type"] == "delta":
            for c, n in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", inner)):
                mat(x + c, n, W, 2.0)
                taps(f"{x}{c}.conv", n, m["conv"])
            mat(x + "b", H, W)
            mat(x + "a", H, W)
            mat(x + "g", inner, W)
            gains(x + "norm", m["vdim"])
        elif l["type"] == "mamba2":
            ch = inner + 2 * m["groups"] * m["state"]
            mat(x + "in", inner + ch + H, W)
            taps(x + "conv", ch, m["conv"])
            w[x + "conv.b"] = 0.3 * rng.standard_normal(ch)
            w[x + "D"] = rng.standard_normal(H)
            gains(x + "norm", inner)
        if f:
            mat(p + "mlp.gate", f["ff"], W, 1.5)
            mat(p + "mlp.up", f["ff"], W)
            mat(p + "mlp.down", W, f["ff"])
    return {k: widen(round_bf16(v)).reshape(v.shape) for k, v in w.items()}


def plant_marker(cfg, w, lift=1.0):
    """Head 0 of layer 0 (attention) looks for the token MARK: its query is a constant direction, which only MARK's key has; the
    coordinate that tells MARK apart is one the position vector hardly moves. The score of a marked key is dim * scale * lift."""
    m, W = cfg["layers"][0]["mixer"], cfg["width"]
    c = W - 2 - W % 2
    w["embed"][:, c] = 0.0
    w["embed"][MARK, c] = 8.0
    D = m["dim"]
    w["l0.norm1"][c] = 1.0
    w["l0.mix.q"][:D], w["l0.mix.q.b"][:D] = 0.0, 0.0
    w["l0.mix.q.b"][0] = 1.0
    w["l0.mix.k"][:D], w["l0.mix.k.b"][:D] = 0.0, 0.0
    w["l0.mix.k"][0, c] = 4.0 * lift
    w["l0.mix.k.b"][1] = 1.0
    w["l0.mix.sink"][0] = 1.0
    return {k: widen(round_bf16(v)).reshape(v.shape) for k, v in w.items()}


def plant_write(cfg, w):
    """Layer 0 (a recurrence) writes the token MARK where no other token writes and every token reads, without decay: key
    coordinate 0 of group 0 is driven by MARK alone, query coordinate 0 by a constant, the values by MARK most of all."""
    l, W = cfg["layers"][0], cfg["width"]
    m, c = l["mixer"], W - 2 - W % 2
    w["embed"][:, c], w["embed"][:, c - 2] = 0.0, 2.0
    w["embed"][MARK, c] = 8.0
    w["l0.norm1"][c] = w["l0.norm1"][c - 2] = 1.0
    w["l0.mix.A_log"][:] = -9.0
    inner = m["heads"] * m["vdim"]
    if l["type"] == "delta":
        q, k, v = (w[f"l0.mix.{n}"] for n in "qkv")
        taps = [w[f"l0.mix.{n}.conv"][0] for n in "qk"]
        q, k = q[0], k[0]
    else:
        n = inner + m["groups"] * m["state"]
        q, k, v = w["l0.mix.in"][inner + n], w["l0.mix.in"][2 * inner], w["l0.mix.in"][inner:2 * inner]
        taps = [w["l0.mix.conv"][n], w["l0.mix.conv"][inner]]
        w["l0.mix.conv.b"][[n, inner]] = 0.0
        w["l0.mix.D"] *= 0.2
    q[:], k[:] = 0.0, 0.0
    q[c - 2], k[c] = 4.0, 4.0
    for t in taps:
        t[:] = 0.0
        t[-1] = 1.0
    v[:, c] *= 32.0
    (w["l0.mix.b"] if l["type"] == "delta" else w["l0.mix.in"][-m["heads"]:])[:, c] = 1.0
    return {k: widen(round_bf16(v)).reshape(v.shape) for k, v in w.items()}


def save(path, cfg, w):
    from skainet_b200.safetensors import write
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write(os.path.join(path, "model.safetensors"), {k: ("BF16", v.shape, round_bf16(v)) for k, v in w.items()})
    return str(path)
