"""Small Tivazen configurations and weights for the tests: random ones, and ones in which a single key stands out so that a
window that is one token off, a lost key or a key of another sequence changes the logits beyond any rounding."""
import json
import os

import numpy as np


def attn(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, window=9, base=5000.0, scale=0.31, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot_dim}, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff=36):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=3, ff=18):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=72, vocab=97, eps=1e-3):
    return {"architecture": "Tivazen", "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


def round_bf16(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) >> 16
    return u.astype(np.uint16)


def widen(h):
    return (h.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def random_weights(cfg, seed=0):
    """name -> float64 array of bfloat16 values."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = gain * rng.standard_normal((rows, cols)) / np.sqrt(cols)

    w["embed"] = rng.standard_normal((V, W))
    mat("head", V, W)
    w["final.norm"] = np.array(1.3)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        w[p + "norm1"], w[p + "dwa"] = np.array(0.7 + 0.1 * i), np.concatenate([rng.normal(0, 0.3, i + 1), [1.1]])
        mat(p + "mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), W, 1.5)
        if m.get("kv_from") is None:
            mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W, 1.5)
            w[p + "mix.dkv.norm"] = 1 + 0.3 * rng.standard_normal(m["kv_rank"])
        mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"])
        mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "mix.g", m["heads"], W)
        mat(p + "mix.o", W, m["heads"] * m["vdim"])
        if f is None:
            continue
        w[p + "norm2"] = np.array(1.2 - 0.1 * i)
        if f["kind"] == "moe":
            mat(p + "mlp.router", f["router"]["experts"], W, 2.0)
        for e in range(f["router"]["experts"] if f["kind"] == "moe" else 1):
            q = p + (f"mlp.e{e}." if f["kind"] == "moe" else "mlp.")
            ff = f["expert"]["ff"] if f["kind"] == "moe" else f["ff"]
            mat(q + "gate", ff, W); mat(q + "up", ff, W); mat(q + "down", W, ff)
    w = {k: widen(round_bf16(v)).reshape(v.shape) for k, v in w.items()}
    return separate_routes(cfg, w, rng)


ROUTE0 = 8    # first of the coordinates separate_routes takes


def separate_routes(cfg, w, rng):
    """Makes every expert choice clear, so that rounding cannot change it: one coordinate per expert that no sublayer writes,
    in which each token's embedding holds the experts' logits in an order of its own, evenly spaced. The depth averages scale
    those coordinates by a factor known per layer, which the router's rows undo."""
    experts = [l["mlp"]["router"]["experts"] if l["mlp"] and l["mlp"]["kind"] == "moe" else 0 for l in cfg["layers"]]
    E = max(experts, default=0)
    if E == 0:
        return w
    assert ROUTE0 + E <= cfg["width"]
    at = slice(ROUTE0, ROUTE0 + E)
    w["embed"][:, at] = (np.argsort(rng.standard_normal((cfg["vocab"], E)), axis=1) - (E - 1) / 2) * (6.0 / E)
    factor, states = 1.0, [1.0]
    for i in range(len(cfg["layers"])):
        p = f"l{i}."
        for name in w:
            if name == p + "mix.o" or (name.startswith(p + "mlp.") and name.endswith("down")):
                w[name][at] = 0.0
        if experts[i]:
            r = w[p + "mlp.router"]
            r[:] = 0.0
            r[np.arange(experts[i]), ROUTE0 + np.arange(experts[i])] = 1.0 / factor
        states.append(factor)
        factor = float(np.dot(w[p + "dwa"], states))
        if abs(factor) < 0.2:
            w[p + "dwa"][-1] += 0.5
            factor = float(np.dot(w[p + "dwa"], states))
    return {k: widen(round_bf16(v)).reshape(v.shape) for k, v in w.items()}


MARK = 1      # the token that plant_marker makes every query look for


def plant_marker(cfg, w, layer=0, strength=1.0):
    """Head 0 of `layer` attends almost only to the token MARK when it is visible: every embedding carries a constant in
    coordinate 0 that drives the query, only MARK carries coordinate 1, which drives the latent. The latent of a layer that
    borrows its cache is the owner's."""
    m = cfg["layers"][layer]["mixer"]
    owner = m.get("kv_from") if m.get("kv_from") is not None else layer
    w["embed"][:, 0], w["embed"][:, 1] = 1.0, 0.0
    w["embed"][MARK, 1] = 8.0
    q = w[f"l{layer}.mix.q"]
    q[0, :] = 0.0
    q[0, 0] = 16.0 * strength / m["scale"]
    d = w[f"l{owner}.mix.dkv"]
    d[0, :] = 0.0
    d[0, 1] = 4.0
    uk = w[f"l{layer}.mix.uk"]
    uk[0, :] = 0.0
    uk[0, 0] = 1.0
    w[f"l{owner}.mix.dkv.norm"][0] = 1.0
    for k in ("embed", f"l{layer}.mix.q"):
        w[k] = widen(round_bf16(w[k])).reshape(w[k].shape)
    return w


def tokens(cfg, n, seed=1):
    """n tokens without MARK."""
    return np.random.default_rng(seed).integers(2, cfg["vocab"], size=n).tolist()


def save(path, cfg, w):
    from skainet_b200.safetensors import write
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write(os.path.join(path, "model.safetensors"), {k: ("BF16", v.shape, round_bf16(v)) for k, v in w.items()})
    return str(path)


def error(got, ref):
    """Largest over the rows of rms(difference, mean removed) / rms(reference)."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    assert got.shape == ref.shape and np.isfinite(got).all()
    d = got - ref
    d -= d.mean(axis=-1, keepdims=True)
    return float((np.sqrt((d * d).mean(axis=-1)) / np.sqrt(np.mean(ref * ref))).max()) if got.size else 0.0
