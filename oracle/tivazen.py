"""Plain restatement of a Tivazen decoder in numpy double precision: one function per mechanism, whole sequences at once,
no cache and no batching. It is the oracle of the tests of that design and shares no code with the product path.

A model is `cfg` (the parsed config.json) and `w`, a dict of float arrays under the names of model.safetensors."""
from __future__ import annotations

import numpy as np


def rms_norm(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain over the last axis; the gain is one number or one per coordinate."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rotate_half(v, positions, base):
    """Rotates v[..., n] (n even) at positions (one per row of axis 0): dimension i pairs with i + n/2."""
    n = v.shape[-1]
    freq = float(base) ** (-2.0 * np.arange(n // 2) / n)
    ang = np.asarray(positions, np.float64)[:, None] * freq
    ang = ang.reshape((ang.shape[0],) + (1,) * (v.ndim - 2) + (n // 2,))
    c, s = np.cos(ang), np.sin(ang)
    u, t = v[..., : n // 2], v[..., n // 2:]
    return np.concatenate([u * c - t * s, t * c + u * s], axis=-1)


def window_mask(n, size):
    """[query, key]: a query sees itself and the size - 1 positions before it."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i - j < size)


def latent_kv(h, w_dkv, norm_gain, kv_rank, base, eps):
    """(latent [n, kv_rank], rotated shared key part [n, rot_dim]) of a sequence."""
    y = h @ w_dkv.T
    return rms_norm(y[:, :kv_rank], norm_gain, eps), rotate_half(y[:, kv_rank:], np.arange(h.shape[0]), base)


def latent_attention(h, w, mix, kv):
    """The mixer over a whole sequence h [n, width]; w holds q, uk, uv, g, o; kv = (latent, rotated key part)."""
    n, H, D, R, V = h.shape[0], mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"]
    c, kr = kv
    q = (h @ w["q"].T).reshape(n, H, D + R)
    qr = rotate_half(q[:, :, D:], np.arange(n), mix["rot"]["base"])
    k = (c @ w["uk"].T).reshape(n, H, D)
    v = (c @ w["uv"].T).reshape(n, H, V)
    score = (np.einsum("ihd,jhd->hij", q[:, :, :D], k) + np.einsum("ihd,jd->hij", qr, kr)) * mix["scale"]
    score = np.where(window_mask(n, mix["mask"]["size"])[None], score, -np.inf)
    p = np.exp(score - score.max(axis=-1, keepdims=True))
    p /= p.sum(axis=-1, keepdims=True)
    out = np.einsum("hij,jhd->ihd", p, v) * sigmoid(h @ w["g"].T)[:, :, None]
    return out.reshape(n, H * V) @ w["o"].T


def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, w_router, top):
    """(chosen experts [n, top], their weights [n, top]): the largest sigmoid scores, not renormalised."""
    s = sigmoid(h @ w_router.T)
    pick = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return pick, np.take_along_axis(s, pick, axis=-1)


def expert_ff(h, w_router, experts, top):
    """Each chosen expert is applied to its weight times the input; experts = list of (gate, up, down)."""
    pick, weight = route(h, w_router, top)
    out = np.zeros_like(h)
    for e, (gate, up, down) in enumerate(experts):
        t, k = np.nonzero(pick == e)
        if t.size:
            np.add.at(out, t, gated_ff(h[t] * weight[t, k][:, None], gate, up, down))
    return out


def depth_average(coef, states):
    """sum_j coef[j] * states[j]; states = the embedding output and the results of the layers so far."""
    return sum(float(a) * s for a, s in zip(coef, states))


def forward(cfg, w, tokens, trace=None):
    """Logits [n, vocab] of a whole sequence; `trace`, if a list, receives x after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    states, kvs = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        mw = {k: w[p + "mix." + k] for k in ("q", "uk", "uv", "g", "o")}
        if mix.get("kv_from") is None:
            kvs[i] = latent_kv(x, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], mix["kv_rank"], mix["rot"]["base"], eps)
            kv = kvs[i]
        else:
            kv = kvs[mix["kv_from"]]
        x = x + rms_norm(latent_attention(x, mw, mix, kv), w[p + "norm1"], eps)
        if mlp is not None:
            if mlp["kind"] == "dense":
                y = gated_ff(x, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
            else:
                ex = [tuple(w[f"{p}mlp.e{e}.{k}"] for k in ("gate", "up", "down")) for e in range(mlp["router"]["experts"])]
                y = expert_ff(x, w[p + "mlp.router"], ex, mlp["router"]["top"])
            x = x + rms_norm(y, w[p + "norm2"], eps)
        states.append(x)
        x = depth_average(w[p + "dwa"], states)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
