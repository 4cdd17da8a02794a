"""The Potupel design's configuration on the CPU: specs from the description, refusals, the declared tensors against the list
written out by hand, the caches of the passes, the scaled frequencies, and the plain implementation's mechanisms on hand-made
numbers."""
import json
import math

import numpy as np
import pytest
import torch

from plain import potupel_plain as P
from potupel_cases import make_config, random_weights
from titan_b200.config import ConfigError, config_from_dict, load_config
from titan_b200.config.spec import LoopSpec, PositionSpec

NAMES = ["mix", "odd", "wide", "routed"]


def test_specs_follow_the_description():
    spec = config_from_dict(make_config("mix")).to_model_spec()
    assert spec.architecture == "Potupel" and spec.hidden_size == 48 and spec.vocab_size == 97 and spec.lm_head is None
    assert spec.order == (0, 1, 2, 1, 2, 1, 2, 3) and spec.loop == LoopSpec(1, 3, 3, "loop.in", "loop.step")
    assert [l.arrangement for l in spec.layers] == ["sandwich"] * 4 and spec.final_norm.weight_offset == 1.0
    a, b, c, bare = spec.layers
    assert a.option("scales") == ("ls1", "ls2") and bare.option("scales") == ("ls1",) and bare.feed_forward is None
    assert [n.weight for n in a.norms] == ["norm1b", "norm2b"] and all(n.weight_offset == 1.0 for n in a.norms + (a.mixer_norm, a.feed_forward_norm))
    assert (a.mixer.num_heads, a.mixer.num_kv_heads, a.mixer.head_dim, a.mixer.option("value_dim"), a.mixer.softmax_scale) == (4, 2, 12, 20, 0.3)
    assert [l.mixer.option("conv") for l in spec.layers] == [3, 1, 2, 6] and a.mixer.option("sink_value") == 0.0 and a.mixer.window is None
    assert a.mixer.position == PositionSpec("rope", 8, 300.0, "half", (8.0, 1.0, 4.0, 64.0)) and b.mixer.position.scaling is None
    assert (a.feed_forward.kind, a.feed_forward.activation, a.feed_forward.intermediate_size) == ("mlp", "relu2", 40)
    assert (b.feed_forward.kind, b.feed_forward.activation, b.feed_forward.intermediate_size) == ("moe", "silu", 24)
    assert [b.feed_forward.option(k) for k in ("experts", "top", "shared_size", "shared_gate", "router_bias")] == [5, 2, 32, False, True]
    assert c.feed_forward.option("shared_size") == 0
    assert set(spec.ignorable_tensors) == {"l3.norm2", "l3.norm2b", "l3.ls2"}
    odd = config_from_dict(make_config("odd")).to_model_spec()
    assert odd.loop is None and odd.order == (0, 1, 2, 3)
    d = make_config("odd")
    d["loop"], d["layers"][1]["mlp"]["shared"], d["layers"][1]["mixer"]["rot"]["scaling"] = None, None, None       # absent by name
    spec = config_from_dict(d).to_model_spec()
    assert spec.loop is None and spec.layers[1].feed_forward.option("shared_size") == 0


@pytest.mark.parametrize("name", NAMES)
def test_declared_tensors_are_the_list_written_by_hand(name):
    from titan_b200.parts import declare_weights
    cfg = make_config(name)
    declared = {w.name: tuple(w.shape) for w in declare_weights(config_from_dict(cfg).to_model_spec())}
    assert declared == {n: tuple(s) for n, s in P.tensor_shapes(cfg).items()}


@pytest.mark.parametrize("name", NAMES)
def test_the_running_order_is_the_one_written_by_hand(name):
    cfg = make_config(name)
    spec = config_from_dict(cfg).to_model_spec()
    runs = P.running_order(cfg)
    assert spec.order == tuple(i for i, _ in runs)
    if spec.loop is not None:
        assert [spec.loop.pass_at(r) for r in range(len(runs))] == [t for _, t in runs]


def test_loops_by_place():
    loop = LoopSpec(2, 3, 2)
    assert loop.order(4) == (0, 1, 2, 2, 3) and [loop.pass_at(r) for r in range(6)] == [None, None, 0, 1, None, None]
    loop = LoopSpec(0, 2, 1)
    assert loop.order(3) == (0, 1, 2) and [loop.pass_at(r) for r in range(4)] == [0, None, None, None]


def test_refusals():
    def broken(change, base="mix"):
        d = make_config(base)
        change(d)
        with pytest.raises(ConfigError):
            config_from_dict(d).to_model_spec()
    broken(lambda c: c["loop"].update(stop=5))                                  # beyond the last layer
    broken(lambda c: c["loop"].update(start=3))                                 # empty
    broken(lambda c: c["loop"].update(times=0))
    broken(lambda c: c["loop"].update(start=-1))
    broken(lambda c: c["loop"].pop("times"))
    broken(lambda c: c["layers"][0].update(type="retention"))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][0]["mixer"].pop("conv"))
    broken(lambda c: c["layers"][0]["mixer"].update(conv=65))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3))
    broken(lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("high"))
    broken(lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda c: c["layers"][1]["mlp"].pop("expert"))
    broken(lambda c: c["norm"].update(eps=0))
    broken(lambda c: c.update(layers=[]))


def test_every_pass_has_its_own_keys_and_windows():
    """One entry a run of a layer: keys and values, and, where the convolution reaches back, the window's rows beside them."""
    from titan_b200.cache import SequenceCache
    from titan_b200.engine.model import DecoderModel
    m = DecoderModel(config_from_dict(make_config("mix")).to_model_spec())
    needs = m.cache_needs()
    assert len(needs) == 8
    assert [tuple(n.kind for n in (need if isinstance(need, tuple) else (need,))) for need in needs] == \
        [("kv", "state"), ("kv",), ("kv", "state")] + [("kv",), ("kv", "state")] * 2 + [("kv", "state")]
    kv, state = needs[0]
    assert kv.head_dim == 32 and kv.num_kv_heads == 2                           # keys of 12, values of 20: heads of 32
    assert state.state_shape == (2 * (4 + 2 * 2) * 32,) and state.state_dtype == torch.float32
    cache = SequenceCache(needs, 256, 3, 128, torch.float32, "cpu")
    views = [cache.view_for_layer(r) for r in (2, 4, 6)]                        # one layer, three passes
    assert len({id(v[0][0]) for v in views}) == 1 and [v[0][1] for v in views] == [0, 1, 2] and [v[1][1] for v in views] == [0, 1, 2]
    s = cache.alloc_slot()
    group, index = views[1][1]
    group.layer_storage(index)[s] = 5.0
    cache.free_slot(s)
    assert cache.alloc_slot() == s and float(group.layer_storage(index)[s].abs().max()) == 0.0, "a slot used again starts from zero"


@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 8192.0), (4.0, 1.0, 4.0, 100.0), (2.5, 0.7, 9.0, 400.0), (3.0, 2.0, 2.0, 60.0), (1.0, 1.0, 4.0, 64.0)])
@pytest.mark.parametrize("dims,base", [(2, 10000.0), (10, 77.0), (64, 10000.0), (128, 500000.0)])
def test_scaled_frequencies(dims, base, scaling):
    from titan_b200.parts import POSITIONS
    part = POSITIONS.build(PositionSpec("rope", dims, base, "half", scaling))
    got = part.tables("cpu")["inv_freq"].double().numpy()
    want = P.frequencies(dims, base, None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling)))
    assert np.allclose(got, want, rtol=1e-7)
    if scaling == (2.5, 0.7, 9.0, 400.0) and dims == 64:                         # all three stretches are there, each with its own rule
        raw = P.frequencies(dims, base)
        ratio = want / raw
        assert (np.isclose(ratio, 1.0)).sum() > 2 and (np.isclose(ratio, 1 / 2.5)).sum() > 2 and ((ratio > 1 / 2.49) & (ratio < 0.999)).sum() > 2
        assert (np.diff(want) < 0).all()


def test_weights_that_do_not_fit_are_named(tmp_path):
    from helpers import write_folder
    from titan_b200.parts import declare_weights
    from titan_b200.weights import FolderWeights, WeightError
    cfg = make_config("mix")
    w = {k: v.to(torch.bfloat16) for k, v in random_weights(cfg, 1).items()}
    w["l0.mlp.gate"] = w["l0.mlp.up"].clone()                               # the dense feed-forward has no gate
    w["loop.step"] = w["loop.step"][:2].clone()
    del w["l1.mlp.router.b"]
    w["l3.ls2"] = w["l3.ls1"].clone()                                       # the scale of a feed-forward that is not there: ignored
    folder = write_folder(str(tmp_path / "m"), cfg, w)
    spec = load_config(folder).to_model_spec()
    with pytest.raises(WeightError) as e:
        FolderWeights(folder, declare_weights(spec), torch.float32, "cpu", spec.ignorable_tensors)
    assert e.value.missing == ["l1.mlp.router.b"] and e.value.unexpected == ["l0.mlp.gate"] and e.value.wrong_shape == [("loop.step", (2, 48), (3, 48))]


def test_plain_mechanisms_on_hand_made_numbers():
    u = np.array([[1.0, 1.0], [2.0, 0.0], [4.0, -1.0]])
    assert np.allclose(P.causal_conv(u, np.array([[0.5, 10.0], [1.0, 0.0]])), [[10.0, 0.0], [20.5, 1.0], [41.0, 0.0]])
    w = P.softmax_beside_one(np.log(np.array([[1.0, 1.0], [2.0, 3.0]])))
    assert np.allclose(w, [[0.5, 0.0], [2 / 6, 3 / 6]])
    assert np.allclose(P.softmax_beside_one(np.array([[800.0]])), [[1.0]]) and np.allclose(P.softmax_beside_one(np.array([[-800.0]])), [[0.0]])
    q = P.rotate_half(np.array([[[1.0, 7.0, 0.0, 8.0, 5.0]]] * 3), [0, 1, 2], np.array([1.0, 0.0]))
    assert np.allclose(q[2, 0], [math.cos(2.0), 7.0, math.sin(2.0), 8.0, 5.0])
    assert np.allclose(P.rms_norm(np.array([3.0, 4.0]), np.array([0.0, 1.0]), 0.0), np.array([3.0, 8.0]) / math.sqrt(12.5))
    ids, w = P.route(np.log(np.array([[1.0, 6.0, 2.0]])), 2)
    assert ids.tolist() == [[1, 2]] and np.allclose(w, [[0.75, 0.25]])
    assert np.allclose(P.dense(np.array([[3.0, -2.0]]), {"up": np.eye(2), "down": np.ones((1, 2))}, ""), [[9.0]])
    x = P.enter_pass(np.array([[1.0]]), np.array([[10.0]]), {"loop.in": np.array([[2.0, 3.0]]), "loop.step": np.array([[0.5], [0.25]])}, 1)
    assert np.allclose(x, [[32.25]])


def test_a_random_weights_folder_is_written_and_read_back(tmp_path):
    from titan_b200.parts import declare_weights
    from titan_b200.weights import FolderWeights, write_model_folder
    cfg = make_config("mix")
    folder = str(tmp_path / "m")
    write_model_folder(folder, config_from_dict(cfg), seed=4)
    again = load_config(folder)
    back = again.to_dict()
    back.pop("torch_dtype", None)                       # what the writer adds
    assert json.loads(json.dumps(back)) == json.loads(json.dumps(cfg))
    declared = declare_weights(again.to_model_spec())
    source = FolderWeights(folder, declared, torch.float32, "cpu", [])
    by = {w.name: w for w in declared}
    assert tuple(source.get(by["loop.in"]).shape) == (48, 96) and tuple(source.get(by["l3.mix.q.conv"]).shape) == (60, 6)
    assert abs(float(source.get(by["l0.norm1"]).mean())) < 0.2, "a norm weight that is stored around zero is drawn around zero"
