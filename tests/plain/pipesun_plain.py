"""A plain, slow implementation of the Pipesun design in float64 numpy: one function per mechanism, whole sequences at
once, nothing shared with the package.  The tests compare the engine with it.

``cfg`` is the model's description as the configuration file gives it (a dict), ``P`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def unit_rms(x, eps):
    """x over the root of (mean square + eps), along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def token_shift(h, mu, before=None):
    """Row t becomes h_t + (h_{t-1} - h_t) * mu; ``before`` (None: zeros) is the row ahead of the first one."""
    prev = np.concatenate([np.zeros_like(h[:1]) if before is None else before[None], h[:-1]])
    return h + (prev - h) * mu


def depth_average(history, weights):
    """The sum of the rows kept so far (embedded rows, then every layer's result), each times its own weight."""
    assert len(history) == len(weights)
    return sum(w * X for w, X in zip(weights, history))


def rotate_adjacent(x, positions, dims, base):
    """x [T, ..., d]: dimensions (2i, 2i + 1) below ``dims`` turn by position * base^(-2i/dims); the rest pass."""
    i = np.arange(dims // 2)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * i / dims)
    c, s = np.cos(ang), np.sin(ang)
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def causal_softmax(s, sink=None):
    """Weights of scores s [H, T, T]: keys up to the query's own position; ``sink`` [H] adds exp(sink) to each denominator."""
    T = s.shape[1]
    s = np.where(np.tril(np.ones((T, T), dtype=bool))[None], s, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink[:, None, None])
    e = np.exp(s - m)
    d = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        d = d + np.exp(sink[:, None, None] - m)
    return e / d


def keys_and_values(h, P, pre, m, eps):
    """What a layer with projections of its own keeps: keys [T, G, 2, dim], each map's normed by itself, and values [T, G, vdim]."""
    T, G, d, dv = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = (h @ P[pre + "k"].T + P[pre + "k.b"]).reshape(T, G, 2, d)
    v = (h @ P[pre + "v"].T + P[pre + "v.b"]).reshape(T, G, dv)
    return rms_norm(k, P[pre + "k.norm"], eps), v


def map_difference(a1, a2, lam, diff, eps):
    """The second map's output, times lambda, off the first's; unit root mean square a head; times (1 - diff)."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def lambda_of(P, pre, diff):
    return np.exp(np.sum(P[pre + "lq1"] * P[pre + "lk1"])) - np.exp(np.sum(P[pre + "lq2"] * P[pre + "lk2"])) + diff


def differential_attention(h, P, pre, m, eps, kv=None):
    """Two softmax maps a head over the same values, the second taken off the first.  ``kv``: another layer's keys and values."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ P[pre + "q"].T + P[pre + "q.b"]).reshape(T, H, 2, d), P[pre + "q.norm"], eps)
    k, v = keys_and_values(h, P, pre, m, eps) if kv is None else kv
    lam = lambda_of(P, pre, m["diff"])
    out = np.empty((T, H, dv))
    for hd in range(H):
        g = hd // (H // G)
        s = np.stack([q[:, hd, i] @ k[:, g, i].T for i in range(2)]) * m["scale"]
        a = causal_softmax(s) @ v[:, g]
        out[:, hd] = map_difference(a[0], a[1], lam, m["diff"], eps)
    return out.reshape(T, H * dv) @ P[pre + "o"].T


def latent_attention(h, P, pre, m, eps):
    """Keys and values from one normed latent a token plus one rotated key part that the heads share; a sink a head in the
    softmax; the heads' outputs gated element by element."""
    T, H, d, dr, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    rot = lambda x: rotate_adjacent(x, pos, m["rot"]["dims"], m["rot"]["base"])
    q = (h @ P[pre + "q"].T).reshape(T, H, d + dr)
    q_rot = rot(q[..., d:])
    down = h @ P[pre + "dkv"].T
    c = rms_norm(down[:, :r], P[pre + "dkv.norm"], eps)
    k_rot = rot(down[:, r:])
    k = (c @ P[pre + "uk"].T).reshape(T, H, d)
    v = (c @ P[pre + "uv"].T).reshape(T, H, dv)
    s = (np.einsum("ihd,jhd->hij", q[..., :d], k) + np.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    out = np.einsum("hij,jhd->ihd", causal_softmax(s, P[pre + "sink"]), v).reshape(T, H * dv)
    return (out * sigmoid(h @ P[pre + "g"].T)) @ P[pre + "o"].T


def gated_feed_forward(h, P, pre):
    z = h @ P[pre + "gate"].T
    return (z * sigmoid(z) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


def forward(cfg, P, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence from its first token; ``after_layer(i, x)`` sees what layer i hands on."""
    eps = cfg["norm"]["eps"]
    x = P["embed"][np.asarray(tokens)]
    history, kept = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        n, m = f"l{i}.", layer["mixer"]
        h = token_shift(rms_norm(x, P[n + "norm1"], eps), P[n + "shift"])
        if layer["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = keys_and_values(h, P, n + "mix.", m, eps)
            y = differential_attention(h, P, n + "mix.", m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = latent_attention(h, P, n + "mix.", m, eps)
        x = x + rms_norm(y, P[n + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = gated_feed_forward(rms_norm(x, P[n + "norm2"], eps), P, n + "mlp.")
            x = x + rms_norm(y, P[n + "norm2b"], eps)
        history.append(x)
        x = depth_average(history, P[n + "dwa"])
        if after_layer is not None:
            after_layer(i, x)
    return rms_norm(x, P["final.norm"], eps) @ P["head"].T


def tensor_shapes(cfg):
    """name -> shape of every tensor of a model."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        n, m = f"l{i}.", layer["mixer"]
        p = n + "mix."
        out.update({n + "norm1": (W,), n + "norm1b": (W,), n + "shift": (W,), n + "dwa": (i + 2,)})
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            out.update({p + "q": (2 * H * d, W), p + "q.b": (2 * H * d,), p + "q.norm": (d,), p + "o": (W, H * dv)})
            out.update({p + n2: (d,) for n2 in ("lq1", "lk1", "lq2", "lk2")})
            if m.get("kv_from") is None:
                out.update({p + "k": (2 * G * d, W), p + "k.b": (2 * G * d,), p + "k.norm": (d,), p + "v": (G * dv, W), p + "v.b": (G * dv,)})
        else:
            r, dr = m["kv_rank"], m["rot_dim"]
            out.update({p + "q": (H * (d + dr), W), p + "dkv": (r + dr, W), p + "dkv.norm": (r,), p + "uk": (H * d, r), p + "uv": (H * dv, r),
                        p + "sink": (H,), p + "g": (H * dv, W), p + "o": (W, H * dv)})
        f = layer.get("mlp")
        if f is not None:
            F = f["ff"]
            out.update({n + "norm2": (W,), n + "norm2b": (W,), n + "mlp.gate": (F, W), n + "mlp.up": (F, W), n + "mlp.down": (W, F)})
    return out
