"""Small Potupel configurations for the tests, each unlike the others in every size, option and layer order, and random
weights that a bfloat16 file holds exactly.  The list of a model's tensors is ``plain.potupel_plain.tensor_shapes``."""
import copy

import torch

from plain import potupel_plain as P


def attention(heads, kv_heads, dim, vdim, scale, conv, rot_dims, base=10000.0, scaling=None):
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv, "rot": rot}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return f if shared is None else dict(f, shared={"ff": shared})


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(layers, width, vocab, eps, loop=None):
    d = {"architecture": "Potupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    return d if loop is None else dict(d, loop=dict(zip(("start", "stop", "times"), loop)))


CASES = {
    # three passes over the middle of the model; convolutions of three, one, two and six taps; frequencies scaled in every way
    # (waves short, between and long) and left alone; every feed-forward, none at all
    "mix": lambda: model([layer(attention(4, 2, 12, 20, 0.3, 3, 8, 300.0, (8.0, 1.0, 4.0, 64)), dense(40)),
                          layer(attention(3, 1, 16, 8, 0.25, 1, 16, 77.0), moe(5, 2, 24, 32)),
                          layer(attention(4, 4, 8, 24, 0.4, 2, 4, 5000.0, (3.0, 0.5, 2.0, 200)), moe(3, 3, 17)),
                          layer(attention(6, 2, 10, 10, 0.35, 6, 10, 40.0))],
                         width=48, vocab=97, eps=1e-5, loop=(1, 3, 3)),
    # widths that are no multiples of 4 or 8, the residual's included; odd head sizes; one head; as many kv heads as heads; a
    # convolution longer than most portions; no loop; a mixture of one expert; no feed-forward first
    "odd": lambda: model([layer(attention(1, 1, 5, 9, 0.4, 9, 4, 77.0, (2.0, 1.0, 1.0, 30))),
                          layer(attention(3, 3, 7, 5, 0.5, 4, 6, 1e5), moe(1, 1, 11, 9)),
                          layer(attention(4, 1, 3, 29, 0.7, 5, 2, 900.0), dense(33)),
                          layer(attention(2, 2, 25, 40, 0.2, 2, 20, 60.0, (4.0, 2.0, 5.0, 50)), moe(9, 4, 7))],
                         width=51, vocab=131, eps=3e-6),
    # heads of 64 and 128, filled and padded: the sizes whose attention runs on tensor cores in bfloat16, with one, three and nine
    # query heads on a kv head; two passes from the first layer on; dense feed-forwards
    "wide": lambda: model([layer(attention(6, 2, 64, 64, 0.125, 4, 32, 10000.0, (8.0, 1.0, 4.0, 128)), dense(96)),
                           layer(attention(2, 2, 128, 100, 0.09, 3, 128, 500000.0), dense(160)),
                           layer(attention(9, 1, 60, 48, 0.13, 2, 48, 2000.0, (2.0, 1.0, 8.0, 100)), dense(64))],
                          width=136, vocab=211, eps=1e-6, loop=(0, 2, 2)),
    # the whole model runs twice; one expert a token, half of them, all but one
    "routed": lambda: model([layer(attention(3, 1, 64, 40, 0.13, 3, 24, 10000.0), moe(6, 1, 48, 40)),
                             layer(attention(4, 2, 32, 64, 0.18, 2, 32, 700.0, (16.0, 1.0, 3.0, 90)), moe(8, 4, 32)),
                             layer(attention(2, 1, 16, 16, 0.25, 3, 8, 100.0), moe(4, 3, 64, 72))],
                            width=64, vocab=150, eps=1e-5, loop=(0, 3, 2)),
}


def make_config(name):
    return copy.deepcopy(CASES[name]())


def random_weights(cfg, seed):
    """float32 torch tensors that bfloat16 holds exactly.  Matrices ~ N(0, 1/fan_in) (the embedding N(0, 1)); the small tensors are
    spread so that every mechanism matters: norm weights around zero, layer scales of both signs, taps of one size and any sign,
    router outputs of a few units with biases that change the choice, vectors of the passes of about the stream's size."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in P.tensor_shapes(cfg).items():
        n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = n()
        elif "norm" in last:
            t = n(0.3)
        elif last in ("ls1", "ls2"):
            t = n(0.5, 0.8)
        elif last == "conv":
            t = n(1.0 / shape[1] ** 0.5)
        elif last == "b":
            t = n(1.0)
        elif last == "router":
            t = n(3.0 / shape[-1] ** 0.5)
        elif last == "step":
            t = n(0.7)
        else:
            t = n(1.0 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16).float()
    return out


def as_numpy(weights):
    return {k: v.double().numpy() for k, v in weights.items()}
