"""The Pipesun design's configuration on the CPU: specs from the description, refusals, the declared tensors against the list
written out by hand, the block's own cache needs, and the plain implementation's mechanisms on hand-made numbers."""
import copy
import json
import math

import numpy as np
import pytest
import torch

from pipesun_cases import make_config, random_weights
from plain import pipesun_plain as P
from titan_b200.config import ConfigError, config_from_dict, load_config


def test_specs_follow_the_description():
    spec = config_from_dict(make_config("mix")).to_model_spec()
    assert spec.architecture == "Pipesun" and spec.hidden_size == 48 and spec.vocab_size == 97 and spec.lm_head == "head"
    assert [l.arrangement for l in spec.layers] == ["sandwich"] * 4
    assert [l.mixer.kind for l in spec.layers] == ["differential_attention", "latent_attention", "latent_attention", "differential_attention"]
    own, lat, bare, reader = spec.layers
    assert own.option("token_shift") == "shift" and [l.option("depth_average") for l in spec.layers] == [("dwa", i) for i in range(4)]
    assert [n.weight for n in own.norms] == ["norm1b", "norm2b"] and [n.weight for n in bare.norms] == ["norm1b"] and bare.feed_forward is None
    assert own.mixer.cache_from is None and reader.mixer.cache_from == 0
    assert (own.mixer.option("diff"), reader.mixer.option("diff"), own.mixer.softmax_scale, reader.mixer.softmax_scale) == (0.2, 0.6, 0.3, 0.45)
    assert own.mixer.option("value_dim") == 20 and own.mixer.qk_norm.size == 12 and own.mixer.position.kind == "none"
    assert lat.mixer.window is None and lat.mixer.option("sink") == "sink" and lat.mixer.option("out_gate") == "g"
    assert lat.mixer.position.pairing == "adjacent" and lat.mixer.position.theta == 300.0 and lat.mixer.position.rotary_dim == 8
    assert own.feed_forward.kind == "gated_mlp" and own.feed_forward.intermediate_size == 40 and own.feed_forward.activation == "silu"
    odd = config_from_dict(make_config("odd")).to_model_spec()
    assert odd.layers[0].mixer.position.rotary_dim == 4 and odd.layers[0].mixer.option("rot_dim") == 6
    assert [l.mixer.cache_from for l in odd.layers] == [None, None, None, 2, None, 1]
    assert set(odd.ignorable_tensors) == {"l0.norm2", "l0.norm2b", "l3.norm2", "l3.norm2b"}


@pytest.mark.parametrize("name", ["mix", "odd", "wide"])
def test_declared_tensors_are_the_list_written_by_hand(name):
    from titan_b200.parts import declare_weights
    cfg = make_config(name)
    declared = {w.name: tuple(w.shape) for w in declare_weights(config_from_dict(cfg).to_model_spec())}
    assert declared == {n: tuple(s) for n, s in P.tensor_shapes(cfg).items()}


def test_refusals():
    def broken(change, base="mix"):
        d = make_config(base)
        change(d)
        with pytest.raises(ConfigError):
            config_from_dict(d).to_model_spec()
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=1))                 # a layer without keys and values of this kind
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=3))                 # itself
    broken(lambda c: c["layers"][0]["mixer"].update(kv_from=3))                 # a later layer
    broken(lambda c: c["layers"][3]["mixer"].update(kv_heads=1))                # other head counts than the owner's
    broken(lambda c: c["layers"][3]["mixer"].update(heads=2))
    broken(lambda c: c["layers"][3]["mixer"].update(vdim=16))
    broken(lambda c: c["layers"][3]["mixer"].update(dim=8))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"].pop("diff"))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3))
    broken(lambda c: c["layers"][1]["mixer"].pop("kv_rank"))
    broken(lambda c: c["layers"][0].update(type="retention"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    broken(lambda c: c["norm"].update(eps=0))
    broken(lambda c: c.update(layers=[]))
    broken(lambda c: c["layers"][5]["mixer"].update(kv_from=3), base="odd")     # a reader is no owner


def test_every_block_keeps_a_state_of_its_own_beside_its_mixers_cache():
    """One float32 row a sequence and layer for the token shift, readers of another layer's keys included; keys and values only
    where a layer has projections of its own."""
    from titan_b200.cache import SequenceCache
    from titan_b200.engine.model import DecoderModel
    m = DecoderModel(config_from_dict(make_config("mix")).to_model_spec())
    needs = m.cache_needs()
    assert len(needs) == 8 and [n.kind if n else None for n in needs] == ["kv", "latent", "latent", None] + ["state"] * 4
    assert needs[0].head_dim == 32 and needs[0].num_kv_heads == 2           # two maps of 12, values of 20: rows of 32
    cache = SequenceCache(needs, 256, 3, 128, torch.float32, "cpu")
    places = [cache.view_for_layer(4 + i) for i in range(4)]
    assert len({id(g) for g, _ in places}) == 1 and [i for _, i in places] == [0, 1, 2, 3]
    s = cache.alloc_slot()
    group = places[0][0]
    group.layer_storage(2)[s] = 5.0
    cache.free_slot(s)
    assert cache.alloc_slot() == s and float(group.layer_storage(2)[s].abs().max()) == 0.0, "a slot used again starts from zero"


def test_weights_that_do_not_fit_are_named(tmp_path):
    from helpers import write_folder
    from titan_b200.parts import declare_weights
    from titan_b200.weights import FolderWeights, WeightError
    cfg = make_config("mix")
    w = {k: v.to(torch.bfloat16) for k, v in random_weights(cfg, 1).items()}
    w["l3.mix.k"] = w["l0.mix.k"].clone()                                   # a reader has no keys of its own
    del w["l2.dwa"]
    w["l2.norm2"] = w["l2.norm1"].clone()                                   # the norm of a feed-forward that is not there: ignored
    folder = write_folder(str(tmp_path / "m"), cfg, w)
    spec = load_config(folder).to_model_spec()
    with pytest.raises(WeightError) as e:
        FolderWeights(folder, declare_weights(spec), torch.float32, "cpu", spec.ignorable_tensors)
    assert e.value.missing == ["l2.dwa"] and e.value.unexpected == ["l3.mix.k"]


def test_plain_mechanisms_on_hand_made_numbers():
    h = np.array([[1.0, 2.0], [3.0, 4.0], [5.0, 8.0]])
    assert np.allclose(P.token_shift(h, np.array([0.5, 1.0])), [[0.5, 0.0], [2.0, 2.0], [4.0, 4.0]])
    assert np.allclose(P.token_shift(h[1:], np.array([0.5, 1.0]), before=h[0]), [[2.0, 2.0], [4.0, 4.0]])
    assert np.allclose(P.depth_average([h, 2 * h, 4 * h], [1.0, -1.0, 0.5]), h)
    s = np.zeros((1, 2, 2))
    w = P.causal_softmax(s, np.array([math.log(3.0)]))
    assert np.allclose(w[0], [[0.25, 0.0], [0.2, 0.2]])                     # a sink of three keys' weight
    assert np.allclose(P.map_difference(np.array([3.0, 4.0]), np.array([0.0, 0.0]), 0.7, 0.2, 0.0), np.array([3.0, 4.0]) / math.sqrt(12.5) * 0.8)
    q = P.rotate_adjacent(np.array([[1.0, 0.0, 5.0]] * 3), [0, 1, 2], 2, 10.0)
    assert np.allclose(q[2], [math.cos(2.0), math.sin(2.0), 5.0])


def test_a_random_weights_folder_is_written_and_read_back(tmp_path):
    from titan_b200.parts import declare_weights
    from titan_b200.weights import FolderWeights, write_model_folder
    cfg = make_config("odd")
    folder = str(tmp_path / "m")
    write_model_folder(folder, config_from_dict(cfg), seed=4)
    again = load_config(folder)
    back = again.to_dict()
    back.pop("torch_dtype", None)                       # what the writer adds
    assert json.loads(json.dumps(back)) == json.loads(json.dumps(cfg))
    declared = declare_weights(again.to_model_spec())
    source = FolderWeights(folder, declared, torch.float32, "cpu", [])
    by = {w.name: w for w in declared}
    assert tuple(source.get(by["l5.dwa"]).shape) == (7,) and tuple(source.get(by["l3.mix.q"]).shape) == (12, 51)
    assert "l3.mix.k" not in by and "l3.norm2" not in by
