"""Parts of a decoder and their registries; importing this package registers the built-in kinds."""
from __future__ import annotations

from typing import List

from ..weights.loader import WeightSpec
from .base import (BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS, FeedForward, Mixer, Norm, Part,
                   PositionEncoding, Registry)
from . import attention, block, diff_attention, gated_delta, latent_attention, lightning, loop, mlp, mlstm, moe, norm, parallel, retention, rotary, token_table, wkv  # noqa: F401  (registration)


def build_block(layer_spec):
    kind = layer_spec.arrangement
    if kind not in BLOCKS._classes:
        raise KeyError(f"no block arrangement '{kind}' is registered; known: {', '.join(BLOCKS.kinds())}")
    return BLOCKS._classes[kind](layer_spec)


def declare_weights(model_spec) -> List[WeightSpec]:
    """Every tensor the model owns, in file order, without touching a device."""
    specs = [WeightSpec(model_spec.embedding, (model_spec.vocab_size, model_spec.hidden_size))]
    specs += [WeightSpec(name, tuple(shape)) for name, shape in model_spec.shared_tensors]
    if model_spec.loop is not None:
        specs += loop.LoopEntry(model_spec.loop, model_spec.hidden_size).weight_specs()
    for layer in model_spec.layers:
        specs += build_block(layer).weight_specs()
    if model_spec.embedding_norm is not None:
        specs += NORMS.build(model_spec.embedding_norm).weight_specs("")
    specs += NORMS.build(model_spec.final_norm).weight_specs("")
    if model_spec.lm_head is not None:
        specs.append(WeightSpec(model_spec.lm_head, (model_spec.vocab_size, model_spec.hidden_size)))
    return specs


__all__ = ["BLOCKS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITIONS", "FeedForward", "Mixer", "Norm", "Part",
           "PositionEncoding", "Registry", "build_block", "declare_weights"]
