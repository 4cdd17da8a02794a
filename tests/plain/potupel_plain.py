"""A plain, slow implementation of the Potupel design in float64 numpy: one function per mechanism, whole sequences at
once, nothing shared with the package.  The tests compare the engine with it.

``cfg`` is the model's description as the configuration file gives it (a dict), ``P`` maps tensor names to arrays.
"""
from __future__ import annotations

import math

import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def rms_norm(x, w, eps):
    """The weight is stored around zero: the row over its root mean square, times (1 + w)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (1.0 + w)


def joined(x, y, w, scale, eps):
    """A sublayer's result on the residual stream: normed, scaled element by element, added."""
    return x + rms_norm(y, w, eps) * scale


def causal_conv(u, taps):
    """u [T, C], taps [C, n]: the last tap on the token itself, zeros before the sequence's start."""
    T, n = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, u.shape[1])), u])
    out = np.zeros_like(u)
    for j in range(n):
        out += taps[:, j] * padded[j:j + T]
    return out


def frequencies(dims, base, scaling=None):
    """Turns per position of each rotated pair, stretched by wavelength: short waves as they are, long ones slowed by
    ``factor``, a blend between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif not wave < scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return np.array(out)


def rotate_half(x, positions, freq):
    """x [T, heads, d]: dimension i turns with dimension i + len(freq); what lies beyond passes."""
    n = len(freq)
    a = np.asarray(positions, dtype=np.float64)[:, None] * freq
    c, s = np.cos(a)[:, None], np.sin(a)[:, None]
    out = x.copy()
    out[..., :n] = x[..., :n] * c - x[..., n:2 * n] * s
    out[..., n:2 * n] = x[..., n:2 * n] * c + x[..., :n] * s
    return out


def softmax_beside_one(s):
    """Weights of scores s [T, T] over the keys up to the query's own position, with one more term, exp(0), below the line."""
    T = s.shape[0]
    s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-m))


def attention(h, P, pre, m):
    """Grouped queries; convolutions over time on q, k and v straight behind their projections; partly rotated heads."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ P[pre + r].T, P[pre + r + ".conv"]) for r in ("q", "k", "v"))
    freq = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rotate_half(q.reshape(T, H, d), np.arange(T), freq)
    k = rotate_half(k.reshape(T, G, d), np.arange(T), freq)
    v = v.reshape(T, G, dv)
    out = np.empty((T, H, dv))
    for i in range(H):
        g = i // (H // G)
        out[:, i] = softmax_beside_one(q[:, i] @ k[:, g].T * m["scale"]) @ v[:, g]
    return out.reshape(T, H * dv) @ P[pre + "o"].T


def dense(h, P, pre):
    z = np.maximum(h @ P[pre + "up"].T, 0.0)
    return (z * z) @ P[pre + "down"].T


def expert(h, P, pre):
    return (silu(h @ P[pre + "gate"].T) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


def route(z, top):
    """The ``top`` largest logits of each row and the softmax over them alone: (indices, weights) [T, top]."""
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    e = np.exp(np.take_along_axis(z, ids, 1) - z.max(axis=-1, keepdims=True))
    return ids, e / e.sum(axis=-1, keepdims=True)


def experts(h, P, pre, f):
    ids, w = route(h @ P[pre + "router"].T + P[pre + "router.b"], f["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t], w[t]):
            out[t] += p * expert(h[t:t + 1], P, f"{pre}e{e}.")[0]
    if f.get("shared") is not None:
        out += expert(h, P, pre + "shared.")
    return out


def enter_pass(x, x0, P, t):
    """What stands before the first layer of pass t: the stream beside the embedded rows, through one matrix, plus the pass's vector."""
    return np.concatenate([x, x0], axis=1) @ P["loop.in"].T + P["loop.step"][t]


def running_order(cfg):
    """(layer, pass that begins right before it or None) for every run of a layer."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, P, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence from its first token; ``after_layer(run, x)`` sees what every run of a layer makes."""
    eps = cfg["norm"]["eps"]
    x = x0 = P["embed"][np.asarray(tokens)]
    for run, (i, begins) in enumerate(running_order(cfg)):
        if begins is not None:
            x = enter_pass(x, x0, P, begins)
        n, layer = f"l{i}.", cfg["layers"][i]
        x = joined(x, attention(rms_norm(x, P[n + "norm1"], eps), P, n + "mix.", layer["mixer"]), P[n + "norm1b"], P[n + "ls1"], eps)
        f = layer.get("mlp")
        if f is not None:
            h = rms_norm(x, P[n + "norm2"], eps)
            y = dense(h, P, n + "mlp.") if f["kind"] == "dense" else experts(h, P, n + "mlp.", f)
            x = joined(x, y, P[n + "norm2b"], P[n + "ls2"], eps)
        if after_layer is not None:
            after_layer(run, x)
    return rms_norm(x, P["final.norm"], eps) @ P["embed"].T


def tensor_shapes(cfg):
    """name -> shape of every tensor of a model."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,)}
    if cfg.get("loop"):
        out.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    for i, layer in enumerate(cfg["layers"]):
        n, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        p, H, G, d, dv = n + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({n + "norm1": (W,), n + "norm1b": (W,), n + "ls1": (W,), p + "o": (W, H * dv)})
        for r, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
            out.update({p + r: (rows, W), p + r + ".conv": (rows, m["conv"])})
        if f is None:
            continue
        out.update({n + "norm2": (W,), n + "norm2b": (W,), n + "ls2": (W,)})
        p = n + "mlp."
        if f["kind"] == "dense":
            out.update({p + "up": (f["ff"], W), p + "down": (W, f["ff"])})
            continue
        E = f["router"]["experts"]
        out.update({p + "router": (E, W), p + "router.b": (E,)})
        for q, F in [(f"{p}e{e}.", f["expert"]["ff"]) for e in range(E)] + ([(p + "shared.", f["shared"]["ff"])] if f.get("shared") else []):
            out.update({q + "gate": (F, W), q + "up": (F, W), q + "down": (W, F)})
    return out
