"""Small Pipesun configurations for the tests, each unlike the others in every size, option and layer order, and random
weights that a bfloat16 file holds exactly.  The list of a model's tensors is ``plain.pipesun_plain.tensor_shapes``."""
import copy

import torch

from plain import pipesun_plain as P


def attention(heads, kv_heads, dim, vdim, scale, diff, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    return m if kv_from is None else dict(m, kv_from=kv_from)


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, rot_dims=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(layers, width, vocab, eps):
    return {"architecture": "Pipesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # an owner of keys and values first, read by the last layer with a factor and a scale of its own; a layer without feed-forward
    "mix": lambda: model([layer("attention", attention(4, 2, 12, 20, 0.3, 0.2), 40),
                          layer("latent_attention", latent(3, 16, 8, 12, 20, 0.2, base=300.0), 56),
                          layer("latent_attention", latent(2, 8, 4, 24, 28, 0.3, base=50.0)),
                          layer("attention", attention(4, 2, 12, 20, 0.45, 0.6, kv_from=0), 24)],
                         width=48, vocab=97, eps=1e-5),
    # widths that are no multiples of 4 or 8, the residual's included; odd sizes; one head; as many kv heads as heads; two owners
    # with a reader each, the readers in the other order; a rotation over part of the rotated dimensions; no feed-forward first
    "odd": lambda: model([layer("latent_attention", latent(1, 5, 6, 9, 11, 0.4, base=77.0, rot_dims=4)),
                          layer("attention", attention(3, 3, 7, 5, 0.5, 0.0), 33),
                          layer("attention", attention(2, 1, 3, 29, 0.7, 0.8), 21),
                          layer("attention", attention(2, 1, 3, 29, 0.3, 0.35, kv_from=2)),
                          layer("latent_attention", latent(5, 12, 2, 4, 6, 0.25, base=1e5), 16),
                          layer("attention", attention(3, 3, 7, 5, 0.2, 0.5, kv_from=1), 9)],
                         width=51, vocab=131, eps=3e-6),
    # rows of 128 and of 64 elements, filled and padded: the sizes whose attention runs on tensor cores in bfloat16, with six maps,
    # two and sixteen on a kv head; the latent sizes whose whole prompts run on tensor cores
    "wide": lambda: model([layer("attention", attention(6, 2, 64, 128, 0.125, 0.3), 96),
                           layer("latent_attention", latent(2, 128, 64, 128, 64, 0.07), 128),
                           layer("attention", attention(1, 1, 30, 56, 0.2, 0.1), 64),
                           layer("attention", attention(6, 2, 64, 128, 0.1, 0.45, kv_from=0)),
                           layer("attention", attention(8, 1, 60, 120, 0.15, 0.5), 64)],
                          width=128, vocab=211, eps=1e-6),
}


def make_config(name):
    return copy.deepcopy(CASES[name]())


def random_weights(cfg, seed):
    """float32 torch tensors that bfloat16 holds exactly.  Matrices ~ N(0, 1/fan_in) (the embedding N(0, 1)); the small tensors are
    spread so that every mechanism matters: shifts between minus a half and one and a half, depth weights of both signs, lambdas a
    few tenths from their constants, sinks of a few units, gates that open and close."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in P.tensor_shapes(cfg).items():
        n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = n()
        elif "norm" in last:
            t = n(0.2, 1.0)
        elif last == "shift":
            t = n(0.4, 0.4)
        elif last == "dwa":
            t = n(0.3)
            t[-1] += 1.0
        elif last == "b":
            t = n(0.3)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = n(0.6 / shape[0] ** 0.25)
        elif last == "sink":
            t = n(1.5)
        elif name.endswith("mix.g"):
            t = n(2.0 / shape[-1] ** 0.5)
        else:
            t = n(1.0 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16).float()
    return out


def as_numpy(weights):
    return {k: v.double().numpy() for k, v in weights.items()}
