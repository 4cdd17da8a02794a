"""Arrangements of a block's parts around the residual stream.

``pre_norm``:  x += mixer(norm1(x));  x += feed_forward(norm2(x)); a norm whose consumer can fold it into
its first matrix product is handed over unevaluated (``norm.DeferredNorm``)
(berniehans/titan: engine/engine-core/src/forward_cpu.rs:281-386).  The
residual stream ``x`` is float32 and is updated in place: mixer and
feed-forward add into it in the epilogue of their last matrix product.  The other arrangements (``pre_norm_scaled``,
``output_norm``, ``hyper``, ``parallel``, ``sandwich``) are described at their classes.
"""
from __future__ import annotations

from typing import List

import torch

from ..cache.groups import CacheNeed
from ..weights.loader import WeightSpec
from .base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, Part


class PreNormBlock(Part):
    def __init__(self, spec):
        if spec.feed_forward is None or spec.mixer_norm is None or spec.feed_forward_norm is None or spec.norms:
            raise ValueError("the pre_norm arrangement takes a mixer, a feed-forward and exactly the two norms before them")
        self.spec = spec
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.feed_forward_norm = NORMS.build(spec.feed_forward_norm)
        self.feed_forward = FEED_FORWARDS.build(spec.feed_forward)

    def parts(self):
        return (self.mixer_norm, self.mixer, self.feed_forward_norm, self.feed_forward)

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        return out

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))

    @staticmethod
    def _normed(norm, consumer, x, ctx):
        """The norm's rows for the part that consumes them; not yet computed (a DeferredNorm) if the norm can be
        deferred and the part can fold it into its first product."""
        # up to 16 rows: measured after 2,048-token prompts, folding gains 3 % of the step at 12 and 16 sequences and
        # loses 1 to 3 % at 20 to 32 (the kernels take up to 32 rows: twice the float32 rows per weight tile through L2)
        if (getattr(consumer, "folds_norm", False) and hasattr(norm, "deferred") and getattr(norm, "groups", 1) == 1 and ctx.options.get("fold_norms", True)
                and x.shape[0] <= int(ctx.options.get("fold_norms_rows", 16))):
            return norm.deferred(x, ctx)
        return norm.forward(x, ctx)

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        self.mixer.forward(self._normed(self.mixer_norm, self.mixer, x, ctx), ctx, cache, x)
        self.feed_forward.forward(self._normed(self.feed_forward_norm, self.feed_forward, x, ctx), ctx, x)


BLOCKS.register("pre_norm", PreNormBlock)


class ScaledPreNormBlock(Part):
    """``pre_norm_scaled``: pre-norm with a learned scale on every sublayer's output ("layer scale"):

        x += s1 * mixer(norm1(x));   x += s2 * feed_forward(norm2(x))

    s1 and s2 are vectors as wide as the residual stream, named in ``LayerSpec.extra`` under "scales" (two tensor names
    relative to the layer's prefix).  The feed-forward, with its norm and scale, may be absent.  A sublayer adds into a
    zeroed float32 buffer of the step; one kernel then scales that buffer, adds it to the residual stream and leaves it
    zeroed.  Where the norm that follows is a ``dyt`` norm (its result depends on the element alone), the same kernel
    also writes the normed rows that the next sublayer reads: the feed-forward's input here, or the next block's
    mixer input, which the next block then finds in ``ctx.carried`` (the model names the block that runs next)."""

    def __init__(self, spec):
        if spec.mixer_norm is None or (spec.feed_forward is None) != (spec.feed_forward_norm is None) or spec.norms:
            raise ValueError("the pre_norm_scaled arrangement takes a mixer with its norm, and a feed-forward with its norm or neither")
        names = tuple(spec.option("scales", ()))
        if len(names) != (1 if spec.feed_forward is None else 2):
            raise ValueError("the pre_norm_scaled arrangement needs the name of one scale vector for each sublayer")
        self.spec, self.scale_names = spec, names
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.feed_forward_norm = None if spec.feed_forward_norm is None else NORMS.build(spec.feed_forward_norm)
        self.feed_forward = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward)
        self.scales: List[torch.Tensor] = []

    def parts(self):
        return (self.mixer_norm, self.mixer) + (() if self.feed_forward is None else (self.feed_forward_norm, self.feed_forward))

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        width = self.spec.mixer.hidden_size
        return out + [WeightSpec(self.spec.prefix + n, (width,), "vector", ("one_plus_normal", 0.1)) for n in self.scale_names]

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))
        self.scales = [get(self.spec.prefix + n) for n in self.scale_names]

    def _join(self, y, scale, x, ctx, next_norm):
        """x += scale * y, y zeroed; the rows of ``next_norm`` over the new x if that norm can ride along, else None."""
        from .. import kernels as K
        if next_norm is not None and hasattr(next_norm, "triple") and ctx.options.get("fuse_scaled_norm", True):
            h = ctx.empty(tuple(x.shape))
            K.scale_add(y, scale, x, ctx.stream, zero_y=True, norm=next_norm.triple(), h=h)
            return h
        K.scale_add(y, scale, x, ctx.stream, zero_y=True)
        return None

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        y = ctx.carried.get("sublayer_sum")
        if y is None or y.shape != x.shape:
            y = ctx.carried["sublayer_sum"] = torch.zeros_like(x)         # zeroed once a step; the joining kernel leaves it zeroed
        kept = ctx.carried.pop("normed_rows", None)
        h = kept[0] if kept is not None and kept[1] == ctx.run and kept[0].shape == x.shape else self.mixer_norm.forward(x, ctx)
        self.mixer.forward(h, ctx, cache, y)
        following = getattr(ctx.next_block, "mixer_norm", None) if isinstance(ctx.next_block, ScaledPreNormBlock) else None
        if self.feed_forward is None:
            h = self._join(y, self.scales[0], x, ctx, following)
        else:
            h = self._join(y, self.scales[0], x, ctx, self.feed_forward_norm)
            self.feed_forward.forward(h if h is not None else self.feed_forward_norm.forward(x, ctx), ctx, y)
            h = self._join(y, self.scales[1], x, ctx, following)
        if h is not None:
            ctx.carried["normed_rows"] = (h, ctx.run + 1)


BLOCKS.register("pre_norm_scaled", ScaledPreNormBlock)


class OutputNormBlock(Part):
    """``output_norm``: every sublayer reads the residual stream itself and its OUTPUT is normed before it is added:

        x += norm1(mixer(x));  x += norm2(feed_forward(x));  x += norm_k(extra_k(x)) for every further sublayer

    The feed-forward (with its norm) may be absent.  Further sublayers are feed-forward parts named in
    ``LayerSpec.extra`` under "sublayers" (a tuple of FeedForwardSpec), their norms are ``LayerSpec.norms`` in the same
    order.  A sublayer adds into a zeroed float32 buffer of the step; one kernel then norms that buffer's rows, adds them
    to the residual stream, leaves the buffer zeroed for the next sublayer and, in bfloat16, writes the new rows rounded
    for the next sublayer's first product (in float32 the sublayers read the residual stream in place)."""

    def __init__(self, spec):
        if spec.mixer_norm is None or (spec.feed_forward is None) != (spec.feed_forward_norm is None):
            raise ValueError("the output_norm arrangement takes a mixer with its norm, and a feed-forward with its norm or neither")
        self.spec = spec
        self.mixer = MIXERS.build(spec.mixer)
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.feed_forward = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward)
        self.feed_forward_norm = None if spec.feed_forward_norm is None else NORMS.build(spec.feed_forward_norm)
        for n in (spec.mixer_norm, spec.feed_forward_norm) + tuple(spec.norms):
            if n is not None and (n.kind != "rmsnorm" or getattr(n, "groups", 1) != 1):
                raise ValueError("the output_norm arrangement folds a plain RMS norm (one group) into the kernel that adds a sublayer's output")
        more = tuple(spec.option("sublayers", ()))
        if len(more) != len(spec.norms):
            raise ValueError(f"{len(more)} further sublayers with {len(spec.norms)} norms")
        self.more = [(FEED_FORWARDS.build(f), NORMS.build(n)) for f, n in zip(more, spec.norms)]

    def parts(self):
        first = (self.mixer, self.mixer_norm) + (() if self.feed_forward is None else (self.feed_forward, self.feed_forward_norm))
        return first + tuple(p for pair in self.more for p in pair)

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        return out

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))

    def bind_shared(self, shared) -> None:
        for part in self.parts():
            if hasattr(part, "bind_shared"):
                part.bind_shared(shared)

    def _input(self, x, ctx):
        """The residual rows as a sublayer's first product reads them: x itself in float32; in bfloat16 the rounded copy
        that the kernel before left (if it was made for exactly this state of x), else one made now."""
        if ctx.dtype == torch.float32:
            return x, None
        kept = ctx.carried.pop("rounded_rows", None)
        if kept is not None and kept[1] == ctx.run and kept[0].shape == x.shape:
            return kept[0], kept[0]
        from .. import kernels as K
        h = ctx.empty(tuple(x.shape))
        K.round_rows(x, h, ctx.stream)
        return h, h

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        from .. import kernels as K
        y = ctx.carried.get("sublayer_sum")
        if y is None or y.shape != x.shape:
            y = ctx.carried["sublayer_sum"] = torch.zeros_like(x)         # zeroed once a step; the norm kernel leaves it zeroed
        h, lowp = self._input(x, ctx)
        steps = [(lambda: self.mixer.forward(h, ctx, cache, y), self.mixer_norm)]
        if self.feed_forward is not None:
            steps.append((lambda: self.feed_forward.forward(h, ctx, y), self.feed_forward_norm))
        steps += [((lambda part=part: part.forward(h, ctx, y)), norm) for part, norm in self.more]
        for run_sublayer, norm in steps:
            run_sublayer()
            K.rmsnorm_add(y, norm.weight, x, norm.spec.eps, ctx.stream, lowp=lowp, zero_y=True)
        if lowp is not None:
            ctx.carried["rounded_rows"] = (lowp, ctx.run + 1)             # valid for the next run of the order, if nothing else touches x


BLOCKS.register("output_norm", OutputNormBlock)


class HyperConnectionBlock(Part):
    """``hyper``: a pre-norm block over several residual streams ("hyper-connections").  The model keeps S copies of the
    residual stream side by side, [T, S * H].  For each sublayer, with three small tensors ``in`` [S], ``out`` [S] and
    ``mix`` [S, S] (indexed [from, to]):

        u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_r <- sum_s mix[s, r] x_s + out[r] * y   (all r from the old streams)

    The tensors' names are ``<name>.in|out|mix`` with one name per sublayer in ``LayerSpec.extra["connections"]``; the number
    of streams is ``LayerSpec.extra["streams"]``.  The feed-forward, with its norm and connection, may be absent.  A sublayer
    adds into a zeroed float32 buffer of the step; ONE kernel then writes it into the streams, mixes them, leaves the buffer
    zeroed and reads the blend for the sublayer that follows, normed (the feed-forward's input here, or the next block's
    mixer input, which that block finds in ``ctx.carried``; after the last block the plain sum of the streams, which the
    model takes as the residual stream that goes to the final norm)."""

    def __init__(self, spec):
        if spec.mixer_norm is None or (spec.feed_forward is None) != (spec.feed_forward_norm is None) or spec.norms:
            raise ValueError("the hyper arrangement takes a mixer with its norm, and a feed-forward with its norm or neither")
        names = tuple(spec.option("connections", ()))
        if len(names) != (1 if spec.feed_forward is None else 2):
            raise ValueError("the hyper arrangement needs the name of one connection for each sublayer")
        self.streams = int(spec.option("streams", 0))
        if self.streams < 1:
            raise ValueError("the hyper arrangement needs the number of streams")
        for n in (spec.mixer_norm, spec.feed_forward_norm):
            if n is not None and (n.kind != "rmsnorm" or getattr(n, "groups", 1) != 1):
                raise ValueError("the hyper arrangement folds a plain RMS norm (one group) into the kernel that reads the streams")
        self.spec, self.names = spec, names
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.feed_forward_norm = None if spec.feed_forward_norm is None else NORMS.build(spec.feed_forward_norm)
        self.feed_forward = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward)
        self.connections: List[tuple] = []          # per sublayer: (in, out, mix)

    def parts(self):
        return (self.mixer_norm, self.mixer) + (() if self.feed_forward is None else (self.feed_forward_norm, self.feed_forward))

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        S = self.streams
        for n in self.names:
            p = self.spec.prefix + n
            out += [WeightSpec(p + ".in", (S,), "vector", ("normal_around", 0.2, 1.0 / S)),
                    WeightSpec(p + ".out", (S,), "vector", ("one_plus_normal", 0.2)),
                    WeightSpec(p + ".mix", (S, S), "vector", ("normal_around", 0.2, 1.0 / S))]
        return out

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))
        self.connections = [tuple(get(self.spec.prefix + n + s).contiguous() for s in (".in", ".out", ".mix")) for n in self.names]

    def _read(self, x, ctx, which: int, norm):
        from .. import kernels as K
        h = ctx.empty((x.shape[0], self.spec.mixer.hidden_size))
        K.hyper(x, self.streams, ctx.stream, in_w=self.connections[which][0], norm_w=norm.weight, eps=norm.spec.eps, h=h)
        return h

    def _join(self, y, which: int, x, ctx, following):
        """Sublayer ``which`` has left its result in y: write it into the streams, and read for what follows.  ``following``:
        (in, norm) of the next sublayer, or "sum" after the last block of the model, or None."""
        from .. import kernels as K
        _, out_w, mix = self.connections[which]
        W = self.spec.mixer.hidden_size
        if following == "sum":
            ones = ctx.scratch.get("stream_ones")
            if ones is None or ones.numel() != self.streams:
                ones = ctx.scratch["stream_ones"] = torch.ones(self.streams, dtype=torch.float32, device=ctx.device)
            total = ctx.empty((x.shape[0], W), torch.float32)
            K.hyper(x, self.streams, ctx.stream, y=y, mix=mix, out_w=out_w, in_w=ones, h=total)
            ctx.carried["stream_sum"] = (total, ctx.run + 1)
            return None
        if following is None:
            K.hyper(x, self.streams, ctx.stream, y=y, mix=mix, out_w=out_w)
            return None
        in_w, norm = following
        h = ctx.empty((x.shape[0], W))
        K.hyper(x, self.streams, ctx.stream, y=y, mix=mix, out_w=out_w, in_w=in_w, norm_w=norm.weight, eps=norm.spec.eps, h=h)
        return h

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        W = self.spec.mixer.hidden_size
        if x.shape[1] != self.streams * W:
            raise ValueError(f"the hyper arrangement of {self.streams} streams was given rows of {x.shape[1]} elements, not {self.streams * W}")
        y = ctx.carried.get("sublayer_sum")
        if y is None or y.shape != (x.shape[0], W):
            y = ctx.carried["sublayer_sum"] = torch.zeros((x.shape[0], W), dtype=torch.float32, device=ctx.device)   # zeroed once a step; the joining kernel leaves it zeroed
        kept = ctx.carried.pop("normed_rows", None)
        h = kept[0] if kept is not None and kept[1] == ctx.run and kept[0].shape == (x.shape[0], W) else self._read(x, ctx, 0, self.mixer_norm)
        self.mixer.forward(h, ctx, cache, y)
        nxt = ctx.next_block
        if nxt is None:
            following = "sum"
        elif isinstance(nxt, HyperConnectionBlock) and nxt.streams == self.streams and ctx.options.get("fuse_hyper", True):
            following = (nxt.connections[0][0], nxt.mixer_norm)
        else:
            following = None
        if self.feed_forward is None:
            h = self._join(y, 0, x, ctx, following)
        else:
            h = self._join(y, 0, x, ctx, (self.connections[1][0], self.feed_forward_norm))
            self.feed_forward.forward(h, ctx, y)
            h = self._join(y, 1, x, ctx, following)
        if h is not None:
            ctx.carried["normed_rows"] = (h, ctx.run + 1)


BLOCKS.register("hyper", HyperConnectionBlock)


class ParallelBlock(Part):
    """``parallel``: ONE norm, and both sublayers read its output:

        h = norm(x);   x += mult * (mixer(h) + feed_forward(h))

    ``mult`` is ``LayerSpec.extra["residual_mult"]`` (1 if absent); the feed-forward may be absent.  Mixer and feed-forward
    add into a zeroed float32 buffer of the step; one kernel then adds that buffer, times ``mult``, to the residual stream,
    leaves it zeroed and, where the block that runs next is of this arrangement with an RMS norm (in groups or not), writes
    that norm's rows, which the next block finds in ``ctx.carried``.  A layer runs one such kernel and, but for the first
    layer of a step, no norm kernel of its own."""

    def __init__(self, spec):
        if spec.mixer_norm is None or spec.feed_forward_norm is not None or spec.norms:
            raise ValueError("the parallel arrangement takes one norm (the mixer's), a mixer, and a feed-forward or none")
        self.spec = spec
        self.mult = float(spec.option("residual_mult", 1.0))
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.feed_forward = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward)

    def parts(self):
        return (self.mixer_norm, self.mixer) + (() if self.feed_forward is None else (self.feed_forward,))

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        return out

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        from .. import kernels as K
        y = ctx.carried.get("sublayer_sum")
        if y is None or y.shape != x.shape:
            y = ctx.carried["sublayer_sum"] = torch.zeros_like(x)         # zeroed once a step; the joining kernel leaves it zeroed
        kept = ctx.carried.pop("normed_rows", None)
        h = kept[0] if kept is not None and kept[1] == ctx.run and kept[0].shape == x.shape else self.mixer_norm.forward(x, ctx)
        self.mixer.forward(h, ctx, cache, y)
        if self.feed_forward is not None:
            self.feed_forward.forward(h, ctx, y)
        nxt = ctx.next_block
        following = nxt.mixer_norm if isinstance(nxt, ParallelBlock) and hasattr(nxt.mixer_norm, "groups") and ctx.options.get("fuse_parallel_norm", True) else None
        if following is None:
            K.residual_group_norm(y, self.mult, x, ctx.stream)
            return
        h = ctx.empty(tuple(x.shape))
        K.residual_group_norm(y, self.mult, x, ctx.stream, norm_w=following.weight, groups=following.groups, eps=following.spec.eps, h=h)
        ctx.carried["normed_rows"] = (h, ctx.run + 1)


BLOCKS.register("parallel", ParallelBlock)


class SandwichBlock(Part):
    """``sandwich``: a norm before AND after each sublayer, each if asked: a token shift in front of the mixer, and an average
    over depth behind the block:

        h = norm1(x);  h_t <- h_t + (h_{t-1} - h_t) * s;   x += norm1b(mixer(h));   x += norm2b(feed_forward(norm2(x)))
        x <- sum over j = 0 .. i + 1 of w_j X_j             X_0 the rows that entered the first block, X_{j+1} what block j made

    ``LayerSpec.norms`` are the norms after the sublayers (one a sublayer; the feed-forward, with both its norms, may be
    absent).  ``LayerSpec.extra``: "scales" = names of vectors [W], one a sublayer, that its normed result is multiplied by before it
    is added ("layer scale"; the vector and the norm's weight are one factor, formed once, in float32); "token_shift" = name of the factors s [W]; "depth_average" = (name of the weights w [i + 2], i)
    with i the block's place in the running order.

    A sublayer adds into a zeroed float32 buffer of the step; ONE kernel then norms that buffer, adds it to the residual stream,
    leaves it zeroed and goes on with what follows: the feed-forward's normed input, or the average over depth and, where
    the next block is of this arrangement, the rows its mixer reads.  With a token shift those need the previous token's row:
    in a step of single tokens that is the sequence's state, so the same kernel shifts too; in a step of longer runs the next
    block's own kernel norms and shifts (the row before is a neighbour's).  The previous token's normed row, before its own
    shift, is the block's state: float32, one row a sequence and run, in a ``state`` cache group (zero at a sequence's start).
    The rows X_j live in one scratch buffer ([runs, T, W] float32); none of them outlasts its step."""

    def __init__(self, spec):
        names = tuple(spec.option("scales", ()))
        if names and len(names) != len(spec.norms):
            raise ValueError(f"{len(names)} scale vectors with {len(spec.norms)} norms after sublayers")
        if spec.mixer_norm is None or (spec.feed_forward is None) != (spec.feed_forward_norm is None) or len(spec.norms) != (1 if spec.feed_forward is None else 2):
            raise ValueError("the sandwich arrangement takes a norm before and a norm after the mixer, and a feed-forward with two norms of its own or none")
        for n in (spec.mixer_norm, spec.feed_forward_norm) + tuple(spec.norms):
            if n is not None and (n.kind != "rmsnorm" or getattr(n, "groups", 1) != 1):
                raise ValueError("the sandwich arrangement folds plain RMS norms (one group) into the kernels around its sublayers")
        self.spec = spec
        self.W = spec.mixer.hidden_size
        self.mixer_norm = NORMS.build(spec.mixer_norm)
        self.mixer = MIXERS.build(spec.mixer)
        self.feed_forward_norm = None if spec.feed_forward_norm is None else NORMS.build(spec.feed_forward_norm)
        self.feed_forward = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward)
        self.after = [NORMS.build(n) for n in spec.norms]
        self.shift_name = spec.option("token_shift")
        self.depth_name, self.place = spec.option("depth_average", (None, 0))
        self.shift = self.depth_w = None
        self.scale_names, self.after_w = names, []

    def parts(self):
        ffn = () if self.feed_forward is None else (self.feed_forward_norm, self.feed_forward)
        return (self.mixer_norm, self.mixer) + ffn + tuple(self.after)

    def own_need(self):
        return None if self.shift_name is None else CacheNeed("state", state_shape=(self.W,), state_dtype=torch.float32)

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        out: List[WeightSpec] = []
        for part in self.parts():
            out += part.weight_specs(self.spec.prefix)
        out += [WeightSpec(self.spec.prefix + n, (self.W,), "vector", ("one_plus_normal", 0.1)) for n in self.scale_names]
        if self.shift_name is not None:
            out.append(WeightSpec(self.spec.prefix + self.shift_name, (self.W,), "vector", ("normal_around", 0.2, 0.3)))
        if self.depth_name is not None:
            n = self.place + 2
            out.append(WeightSpec(self.spec.prefix + self.depth_name, (n,), "vector", ("normal_around", 0.2, 1.0 / n)))
        return out

    def bind(self, get) -> None:
        for part in self.parts():
            part.bind(lambda name: get(self.spec.prefix + name))
        self.after_w = [n.weight for n in self.after]
        if self.scale_names:
            self.after_w = [(w.float() * get(self.spec.prefix + n).float()).contiguous() for w, n in zip(self.after_w, self.scale_names)]
        if self.shift_name is not None:
            self.shift = get(self.spec.prefix + self.shift_name).contiguous()
        if self.depth_name is not None:
            self.depth_w = get(self.spec.prefix + self.depth_name).contiguous()

    @staticmethod
    def _state(ctx, run):
        group, index = ctx.block_state(run)
        return group.layer_storage(index)

    def _read(self, x, ctx):
        """The mixer's input rows, by kernels of their own."""
        if self.shift is None:
            return self.mixer_norm.forward(x, ctx)
        from .. import kernels as K
        h = ctx.empty(tuple(x.shape))
        K.shift_norm(x, self.mixer_norm.weight, self.mixer_norm.spec.eps, self.shift, h, self._state(ctx, ctx.run), ctx.layout, ctx.stream)
        return h

    def _following(self, x, ctx):
        """What the kernel at this block's end may make for the next block: keyword arguments of the join, the next mixer's rows among them."""
        nxt = ctx.next_block
        if not isinstance(nxt, SandwichBlock) or nxt.W != self.W or not ctx.options.get("fuse_sandwich", True):
            return {}
        if nxt.shift is not None and not ctx.layout.all_single:
            return {}
        made = dict(pre_w=nxt.mixer_norm.weight, pre_eps=nxt.mixer_norm.spec.eps, h=ctx.empty(tuple(x.shape)))
        if nxt.shift is not None:
            made.update(mu=nxt.shift, state=self._state(ctx, ctx.run + 1), slot_of_row=ctx.layout.slot_of_seq)
        return made

    def forward(self, x: torch.Tensor, ctx, cache) -> None:
        from .. import kernels as K
        y = ctx.carried.get("sublayer_sum")
        if y is None or y.shape != x.shape:
            y = ctx.carried["sublayer_sum"] = torch.zeros_like(x)         # zeroed once a step; the joining kernel leaves it zeroed
        history = keep = None
        if self.depth_w is not None:
            if ctx.run != self.place:
                raise RuntimeError(f"a block with {self.place + 2} depth weights runs as number {ctx.run}")
            history = ctx.carried.get("depth_rows")
            if ctx.run == 0:                                              # the rows that enter the first block are depth 0: its first join keeps them
                held, n = ctx.scratch.get("depth_rows"), ctx.runs * x.numel()
                if held is None or held.numel() < n:                      # kept from step to step: as large as the longest one so far
                    held = ctx.scratch["depth_rows"] = ctx.empty((n,), torch.float32)
                history = ctx.carried["depth_rows"] = held[:n].view((ctx.runs,) + tuple(x.shape))
                keep = history[0]
            elif history is None:
                raise RuntimeError("an average over depth needs every block from the first on to keep its rows")
        kept = ctx.carried.pop("normed_rows", None)
        h = kept[0] if kept is not None and kept[1] == ctx.run and kept[0].shape == x.shape else self._read(x, ctx)
        self.mixer.forward(h, ctx, cache, y)
        if self.feed_forward is not None:
            n1, n2 = self.after[0], self.feed_forward_norm
            h = ctx.empty(tuple(x.shape))
            K.sandwich_join(y, self.after_w[0], n1.spec.eps, x, ctx.stream, keep=keep, pre_w=n2.weight, pre_eps=n2.spec.eps, h=h)
            keep = None
            self.feed_forward.forward(h, ctx, y)
        made, n = self._following(x, ctx), self.after[-1]
        K.sandwich_join(y, self.after_w[-1], n.spec.eps, x, ctx.stream, keep=keep, history=history, depth=self.place + 1 if history is not None else 0,
                        depth_w=self.depth_w, **made)
        if made:
            ctx.carried["normed_rows"] = (made["h"], ctx.run + 1)


BLOCKS.register("sandwich", SandwichBlock)
