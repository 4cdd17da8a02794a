"""Typed configuration of the Pipesun design, from its config.json.

A Pipesun model is a list of layers with a norm before and a norm after each sublayer (the block arrangement ``sandwich``):

    h = N1(x);  h_t <- h_t + (h_{t-1} - h_t) * s;   x += N1b(mixer(h));   x += N2b(ff(N2(x)));   x <- sum_j w_j X_j

with s the layer's token shift and the last step an average over depth: X_0 are the embedded rows, X_{i+1} what layer i makes,
and what goes on from layer i is the sum of X_0 .. X_{i+1} with the layer's own i + 2 weights.  Mixers:

* ``attention``: differential attention.  Grouped queries; a head has two softmax maps over the same values, and the second,
  times one learned number of the layer, is taken off the first; unit norm a head, a constant factor.  Biases on q, k and v, an
  RMS norm a map on queries and keys, no rotation.  A layer may read another layer's keys and values (``kv_from``).
* ``latent_attention``: attention over one shared latent a token with a rotated (neighbours paired) key part, a sink a head in
  the softmax, an element-wise sigmoid gate on the concatenated heads.

Feed-forward: dense, gated by silu, or none.  The keys read here:

    architecture "Pipesun";  vocab, width;  norm.eps
    layers[i].type "attention":        mixer {heads, kv_heads, dim, vdim, scale, diff}  (+ kv_from: index of an earlier attention layer)
    layers[i].type "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}}
    layers[i].mlp  null | {kind "dense", ff}

Tensor names: embed, l<i>.norm1|norm1b|norm2|norm2b|shift|dwa, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict

from .spec import ConfigError, FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from .tefezen import _get

# No position limit is part of the design; positions are exact in float32 up to here.
MAX_POSITIONS = 1 << 24


@dataclass(frozen=True)
class PipesunConfig:
    raw: Any                       # the config.json dict, checked
    architecture: str = "Pipesun"

    def __hash__(self):
        return id(self)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PipesunConfig":
        d = copy.deepcopy(d)
        _get(d, "width", int), _get(d, "vocab", int)
        if not _get(d, "norm.eps", float) > 0:
            raise ConfigError("norm.eps must be positive")
        layers = _get(d, "layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json key 'layers' must be a list with at least one layer")
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind, m = _get(layer, "type"), _get(layer, "mixer")
            heads = _get(m, "heads", int)
            _get(m, "dim", int), _get(m, "vdim", int), _get(m, "scale", float)
            if kind == "attention":
                if m.get("kv_from") is not None:
                    src = m["kv_from"]
                    if not isinstance(src, int) or isinstance(src, bool) or not 0 <= src < i:
                        raise ConfigError(f"{where}: kv_from {src!r} must name an earlier layer")
                    owner = layers[src]
                    if owner.get("type") != "attention" or owner["mixer"].get("kv_from") is not None:
                        raise ConfigError(f"{where}: kv_from names layer {src}, which has no keys and values of its own")
                kv = _get(m, "kv_heads", int)
                if heads % kv:
                    raise ConfigError(f"{where}: {heads} query heads are not a multiple of {kv} key/value heads")
                _get(m, "diff", float)
            elif kind == "latent_attention":
                rd = _get(m, "rot_dim", int)
                _get(m, "kv_rank", int)
                dims, base = _get(m, "rot.dims", int), _get(m, "rot.base", float)
                if dims % 2 or dims > rd or not base > 0:
                    raise ConfigError(f"{where}: rot.dims {dims} must be even and at most {rd}, rot.base positive")
            else:
                raise ConfigError(f"{where}: mixer type '{kind}' is not known (attention, latent_attention)")
            f = layer.get("mlp")
            if f is not None:
                if f.get("kind") != "dense":
                    raise ConfigError(f"{where}: feed-forward kind {f.get('kind')!r} is not known (dense)")
                _get(f, "ff", int)
        return cls(raw=d, architecture=d.get("architecture") or (d.get("architectures") or ["Pipesun"])[0])

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(self.raw)

    # ------------------------------------------------------------------ #
    def to_model_spec(self) -> ModelSpec:
        d = self.raw
        W, V, eps = d["width"], d["vocab"], float(d["norm"]["eps"])
        norm = lambda name, size=W: NormSpec("rmsnorm", size, eps, name)
        layers = []
        for i, layer in enumerate(d["layers"]):
            m = layer["mixer"]
            if layer["type"] == "attention":
                mixer = MixerSpec(
                    kind="differential_attention", hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                    qk_norm=norm("{}.norm", m["dim"]), softmax_scale=float(m["scale"]), prefix="mix.", cache_from=m.get("kv_from"),
                    names=tuple((r, r) for r in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")),
                    extra=(("value_dim", m["vdim"]), ("diff", float(m["diff"])), ("out_eps", eps), ("bias", True)))
            else:
                mixer = MixerSpec(
                    kind="latent_attention", hidden_size=W, num_heads=m["heads"], num_kv_heads=1, head_dim=m["dim"],
                    softmax_scale=float(m["scale"]), prefix="mix.",
                    position=PositionSpec("rope", rotary_dim=m["rot"]["dims"], theta=float(m["rot"]["base"]), pairing="adjacent"),
                    extra=(("rot_dim", m["rot_dim"]), ("value_dim", m["vdim"]), ("kv_rank", m["kv_rank"]),
                           ("latent_norm", norm("dkv.norm", m["kv_rank"])), ("sink", "sink"), ("out_gate", "g"), ("exact_weights", True)))
            f = layer.get("mlp")
            ffn = None if f is None else FeedForwardSpec(kind="gated_mlp", hidden_size=W, intermediate_size=f["ff"], activation="silu", prefix="mlp.",
                                                         names=(("gate", "gate"), ("up", "up"), ("down", "down")))
            after = (norm("norm1b"),) if ffn is None else (norm("norm1b"), norm("norm2b"))
            layers.append(LayerSpec(index=i, arrangement="sandwich", mixer=mixer, feed_forward=ffn, mixer_norm=norm("norm1"),
                                    feed_forward_norm=None if ffn is None else norm("norm2"), prefix=f"l{i}.", norms=after,
                                    extra=(("token_shift", "shift"), ("depth_average", ("dwa", i)))))
        spec = ModelSpec(architecture=self.architecture, hidden_size=W, vocab_size=V, layers=tuple(layers), order=tuple(range(len(layers))),
                         final_norm=norm("final.norm"), embedding="embed", lm_head="head", max_positions=MAX_POSITIONS,
                         ignorable_tensors=tuple(f"l{i}.{n}" for i, layer in enumerate(d["layers"]) if layer.get("mlp") is None for n in ("norm2", "norm2b")))
        spec.validate()
        return spec
