"""Typed configuration of the Potupel design, from its config.json.

A Potupel model is a list of layers with a norm before and a norm after each sublayer, whose normed results are scaled element by
element before they join the residual stream (the block arrangement ``sandwich`` with ``scales``); every norm's weight is stored
around zero:

    x += s1 * N1b(mixer(N1(x)));   x += s2 * N2b(ff(N2(x)))

A stretch of the layers may run several times in a row (``LoopSpec``): before each pass the stream is mixed with the embedded
rows by one matrix and takes the pass's own vector.  The logits come from the embedding table.

* Mixer ``attention``: grouped queries; a short causal convolution over time on every channel of q, k and v behind their
  projections; the first dimensions of a head rotated in halves, with frequencies scaled by wavelength; softmax with one added to
  the denominator.
* Feed-forward: ``dense``, down(max(up, 0)^2); ``moe``, experts gated by silu, chosen by their largest router logits (with a bias)
  and weighted by the softmax over those, beside an expert that every token uses; or none.

The keys read here:

    architecture "Potupel";  vocab, width;  norm.eps;  loop null | {start, stop, times}
    layers[i].type "attention": mixer {heads, kv_heads, dim, vdim, scale, conv, rot {base, dims, scaling null | {factor, low, high, original}}}
    layers[i].mlp  null | {kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top}, shared null | {ff}}

Tensor names: embed, loop.in|step, l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2, l<i>.mix.q|k|v|o, l<i>.mix.q|k|v.conv,
l<i>.mlp.up|down, l<i>.mlp.router, l<i>.mlp.router.b, l<i>.mlp.e<j>|shared.gate|up|down, final.norm.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict

from .spec import ConfigError, FeedForwardSpec, LayerSpec, LoopSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from .tefezen import _get

# No position limit is part of the design; positions are exact in float32 up to here.
MAX_POSITIONS = 1 << 24


def _index(d, path):
    """A key that holds a layer's number (0 allowed)."""
    v = _get(d, path)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"{path} {v!r} must be a layer's number")
    return v


@dataclass(frozen=True)
class PotupelConfig:
    raw: Any                       # the config.json dict, checked
    architecture: str = "Potupel"

    def __hash__(self):
        return id(self)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PotupelConfig":
        d = copy.deepcopy(d)
        _get(d, "width", int), _get(d, "vocab", int)
        if not _get(d, "norm.eps", float) > 0:
            raise ConfigError("norm.eps must be positive")
        layers = _get(d, "layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json key 'layers' must be a list with at least one layer")
        if d.get("loop") is not None:
            start, stop = _index(d, "loop.start"), _index(d, "loop.stop")
            _get(d, "loop.times", int)
            if not start < stop <= len(layers):
                raise ConfigError(f"loop: layers {start} .. {stop - 1} of {len(layers)}")
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind, m = _get(layer, "type"), _get(layer, "mixer")
            if kind != "attention":
                raise ConfigError(f"{where}: mixer type '{kind}' is not known (attention)")
            heads, kv, dim = _get(m, "heads", int), _get(m, "kv_heads", int), _get(m, "dim", int)
            _get(m, "vdim", int), _get(m, "scale", float)
            if heads % kv:
                raise ConfigError(f"{where}: {heads} query heads are not a multiple of {kv} key/value heads")
            if _get(m, "conv", int) > 64:
                raise ConfigError(f"{where}: a convolution of {m['conv']} taps (at most 64)")
            dims, base = _get(m, "rot.dims", int), _get(m, "rot.base", float)
            if dims % 2 or dims > dim or not base > 0:
                raise ConfigError(f"{where}: rot.dims {dims} must be even and at most dim {dim}, rot.base positive")
            if m["rot"].get("scaling") is not None:
                for key in ("factor", "low", "high", "original"):
                    if not _get(m, "rot.scaling." + key, float) > 0:
                        raise ConfigError(f"{where}: rot.scaling.{key} must be positive")
            f = layer.get("mlp")
            if f is None:
                continue
            if f.get("kind") == "dense":
                _get(f, "ff", int)
            elif f.get("kind") == "moe":
                _get(f, "expert.ff", int)
                experts, top = _get(f, "router.experts", int), _get(f, "router.top", int)
                if top > experts:
                    raise ConfigError(f"{where}: {top} of {experts} experts")
                if f.get("shared") is not None:
                    _get(f, "shared.ff", int)
            else:
                raise ConfigError(f"{where}: feed-forward kind {f.get('kind')!r} is not known (dense, moe)")
        return cls(raw=d, architecture=d.get("architecture") or (d.get("architectures") or ["Potupel"])[0])

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(self.raw)

    # ------------------------------------------------------------------ #
    def to_model_spec(self) -> ModelSpec:
        d = self.raw
        W, V, eps = d["width"], d["vocab"], float(d["norm"]["eps"])
        norm = lambda name: NormSpec("rmsnorm", W, eps, name, weight_offset=1.0)
        layers = []
        for i, layer in enumerate(d["layers"]):
            m, rot = layer["mixer"], layer["mixer"]["rot"]
            scaling = rot.get("scaling")
            if scaling is not None:
                scaling = tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))
            mixer = MixerSpec(
                kind="attention", hidden_size=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], softmax_scale=float(m["scale"]),
                prefix="mix.", position=PositionSpec("rope", rotary_dim=rot["dims"], theta=float(rot["base"]), pairing="half", scaling=scaling),
                names=tuple((r, r) for r in ("q", "k", "v", "o")),
                extra=(("value_dim", m["vdim"]), ("conv", m["conv"]), ("sink_value", 0.0), ("exact_weights", True)))
            f, ffn = layer.get("mlp"), None
            if f is not None and f["kind"] == "dense":
                ffn = FeedForwardSpec(kind="mlp", hidden_size=W, intermediate_size=f["ff"], activation="relu2", prefix="mlp.")
            elif f is not None:
                shared = f.get("shared")
                ffn = FeedForwardSpec(kind="moe", hidden_size=W, intermediate_size=f["expert"]["ff"], activation="silu", prefix="mlp.",
                                      extra=(("experts", f["router"]["experts"]), ("top", f["router"]["top"]), ("router_bias", True),
                                             ("shared_size", 0 if shared is None else shared["ff"]), ("shared_gate", False)))
            n = 1 if ffn is None else 2
            layers.append(LayerSpec(index=i, arrangement="sandwich", mixer=mixer, feed_forward=ffn, mixer_norm=norm("norm1"),
                                    feed_forward_norm=None if ffn is None else norm("norm2"), prefix=f"l{i}.",
                                    norms=(norm("norm1b"), norm("norm2b"))[:n], extra=(("scales", ("ls1", "ls2")[:n]),)))
        loop = d.get("loop")
        if loop is not None:
            loop = LoopSpec(loop["start"], loop["stop"], int(loop["times"]), mix="loop.in", step="loop.step")
        spec = ModelSpec(architecture=self.architecture, hidden_size=W, vocab_size=V, layers=tuple(layers),
                         order=tuple(range(len(layers))) if loop is None else loop.order(len(layers)), final_norm=norm("final.norm"), embedding="embed",
                         lm_head=None, max_positions=MAX_POSITIONS, loop=loop,
                         # a file may carry the second sublayer's vectors of a layer that has none
                         ignorable_tensors=tuple(f"l{i}.{n}" for i, layer in enumerate(d["layers"]) if layer.get("mlp") is None for n in ("norm2", "norm2b", "ls2")))
        spec.validate()
        return spec
