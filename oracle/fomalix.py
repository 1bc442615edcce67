"""Plain restatement of a Fomalix decoder in numpy double precision: one function per mechanism, whole sequences at once, the
recurrences token by token, no cache and no batching. It is the oracle of the tests of that design and shares no code with the
product path.

A model is `cfg` (the parsed config.json) and `w`, a dict of float arrays under the names of model.safetensors."""
from __future__ import annotations

import numpy as np

from .tivazen import rms_norm, sigmoid, silu


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sinusoid(positions, width):
    """[positions, width]: sine and cosine of position / 10000^(2i/width) in coordinates 2i and 2i + 1."""
    i = np.arange((width + 1) // 2)
    ang = np.asarray(positions, np.float64)[:, None] * 10000.0 ** (-2.0 * i / width)
    return np.stack([np.sin(ang), np.cos(ang)], axis=-1).reshape(len(ang), -1)[:, :width]


def embedding(tokens, table, scale):
    return table[np.asarray(tokens)] * scale + sinusoid(np.arange(len(tokens)), table.shape[1])


def chunk_mask(n, size):
    """[query, key]: a query sees the keys up to itself in its own chunk of `size` positions, chunks counted from position 0."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def sink_softmax(score, sink):
    """Weights over the last axis of score [heads, query, key]; the denominator also holds exp(sink[head])."""
    s = sink[:, None, None]
    top = np.maximum(score.max(axis=-1, keepdims=True), s)
    e = np.exp(score - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(s - top))


def chunk_attention(h, w, mix, eps):
    """The attention mixer over a whole sequence h [n, width]; w holds q, k, v, their biases (q.b, ..), sink, o."""
    n, H, G, D, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms_norm((h @ w["q"].T + w["q.b"]).reshape(n, H, D), 1.0, eps)
    k = rms_norm((h @ w["k"].T + w["k.b"]).reshape(n, G, D), 1.0, eps)
    v = (h @ w["v"].T + w["v.b"]).reshape(n, G, V)
    of = np.arange(H) // (H // G)
    score = np.einsum("ihd,jhd->hij", q, k[:, of]) * mix["scale"]
    p = sink_softmax(np.where(chunk_mask(n, mix["mask"]["size"])[None], score, -np.inf), w["sink"])
    return np.einsum("hij,jhd->ihd", p, v[:, of]).reshape(n, H * V) @ w["o"].T


def causal_conv(x, taps, bias=0.0):
    """y[t, c] = sum_j taps[c, j] * x[t - (T - 1) + j, c] + bias[c], zeros before the start."""
    T = taps.shape[1]
    xp = np.concatenate([np.zeros((T - 1, x.shape[1])), x])
    return sum(xp[j:j + x.shape[0]] * taps[:, j] for j in range(T)) + bias


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k [n, H, K]; v [n, H, V]; beta, g [n, H] -> o [n, H, V] from a zero state."""
    n, H, K = q.shape
    S = np.zeros((H, K, v.shape[2]))
    out = np.empty_like(v)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hkv,hk->hv", S, q[t])
    return out


def delta_mixer(h, w, mix, eps):
    n, H, G, K, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q, k, v = (silu(causal_conv(h @ w[c].T, w[c + ".conv"])) for c in ("q", "k", "v"))
    of = np.arange(H) // (H // G)
    q = unit(q.reshape(n, G, K))[:, of] * K ** -0.5
    k = unit(k.reshape(n, G, K))[:, of]
    g = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = delta_rule(q, k, v.reshape(n, H, V), sigmoid(h @ w["b"].T), g)
    o = rms_norm(o, w["norm"], eps) * silu(h @ w["g"].T).reshape(n, H, V)
    return o.reshape(n, H * V) @ w["o"].T


def state_space(x, B, C, dt, A_log, D):
    """x [n, H, P]; B, C [n, H, N]; dt [n, H] -> y [n, H, P] from a zero state."""
    n, H, P = x.shape
    S = np.zeros((H, B.shape[2], P))
    out = np.empty_like(x)
    for t in range(n):
        S = np.exp(-np.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out[t] = np.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t]
    return out


def mamba2_mixer(h, w, mix, eps):
    n, H, P, N, G = h.shape[0], mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    inner, gn = H * P, G * N
    z, xbc, dt = np.split(h @ w["in"].T, [inner, 2 * inner + 2 * gn], axis=1)
    x, B, C = np.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, inner + gn], axis=1)
    of = np.arange(H) // (H // G)
    y = state_space(x.reshape(n, H, P), B.reshape(n, G, N)[:, of], C.reshape(n, G, N)[:, of], softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    y = (y.reshape(n, inner) * silu(z)).reshape(n, mix["norm_groups"], -1)
    return (rms_norm(y, 1.0, eps).reshape(n, inner) * w["norm"]) @ w["o"].T


def gated_ff(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


MIXERS = {"attention": chunk_attention, "delta": delta_mixer, "mamba2": mamba2_mixer}


def layer_runs(cfg):
    """(layer, whether the embedding output is added before it) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, trace=None):
    """Logits [n, vocab] of a whole sequence; `trace`, if a list, receives x after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = x = embedding(tokens, w["embed"], cfg["embedding"]["scale"])
    for i, again in layer_runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        mw = {k[len(p) + 4:]: v for k, v in w.items() if k.startswith(p + "mix.")}
        if again:
            x = x + x0
        x = x + rms_norm(MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), mw, layer["mixer"], eps), w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = gated_ff(rms_norm(x, w[p + "norm2"], eps), w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"])
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
