"""Sopalorn without a GPU: the configuration and its errors, the model as data (tensor names, whose keys a layer reads, the states
a layer's parts keep), and the plain rules on hand cases."""
import copy
import math

import numpy as np
import pytest

import plain_sopalorn as PS
from kapel_b200.config import ConfigError, RopeScaling, config_from_json

ROT = {"base": 50.0, "dims": 4, "scaling": {"factor": 4.0, "original": 90, "fast": 16.0, "slow": 2.0}}
RAW = {"architecture": "Sopalorn", "vocab": 50, "width": 24, "streams": 3, "norm": {"eps": 1e-4}, "embedding": {"scale": 3.0}, "logit_scale": 0.5,
       "layers": [
           {"type": "attention", "mlp": {"kind": "dense", "ff": 20, "limit": 0.7},
            "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3, "rot": ROT}},
           {"type": "lightning", "mlp": None, "mixer": {"heads": 3, "dim": 10, "vdim": 4, "decay": [0.5, 1.0, 0.875]}},
           {"type": "parallel", "mlp": {"kind": "moe", "router": {"experts": 5, "identity": 2, "top": 3, "scale": 1.5}, "expert": {"ff": 12}},
            "mixer": {"left": {"heads": 4, "kv_heads": 4, "dim": 6, "vdim": 10, "scale": 0.2, "mask": {"size": 9}},
                      "right": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "conv": 3}}},
           {"type": "attention", "mlp": None, "mixer": {"heads": 6, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.1, "rot": ROT, "kv_from": 0}},
       ]}


def test_round_trip_and_the_model_as_data():
    c = config_from_json(RAW)
    assert type(c).__name__ == "SopalornConfig" and config_from_json(c.to_json()) == c
    spec = c.to_spec()
    assert [(e.layer, e.cache_of) for e in spec.schedule] == [(0, 0), (1, 1), (2, 2), (3, 0)] and spec.streams == 3
    assert all(l.kind == "streams" and l.norms["pre_mixer"].kind == "layer" and l.norms["pre_mixer"].bias.endswith("norm1.b") for l in spec.layers)
    assert spec.embed.scale == 3.0 and not spec.embed.round_scale and spec.head.scale == 0.5 and spec.head.weight == "head"
    assert spec.final_norm.bias == "final.norm.b" and spec.final_norm.eps == 1e-4
    a, b = spec.layers[0].mixer, spec.layers[3].mixer
    assert a.unit_sink and a.q_norm.width == 32 and a.k_norm.width == 16 and not a.borrows_kv and a.v_head_dim == 6 and a.scale == 0.3
    assert a.position.pairing == "neighbours" and a.position.rotary_dim == 4 and a.position.scaling == RopeScaling(4.0, 90.0, 16.0, 2.0)
    assert b.borrows_kv and b.k_norm is None and b.q_norm.width == 48 and set(b.weights) == {"q", "o"}
    ret = spec.layers[1].mixer
    assert ret.decay == (0.5, 1.0, 0.875) and ret.activation == "silu" and ret.key_scale == 1.0 and ret.whole_norm and ret.gate == "sigmoid"
    assert spec.layers[1].ffn is None and spec.layers[1].streams[1] is None and set(spec.layers[1].norms) == {"pre_mixer"}
    both, moe = spec.layers[2].mixer, spec.layers[2].ffn
    assert both.left.sink and both.left.window == 9 and both.right.conv == 3 and (both.left_scale, both.right_scale) == (0.5, 0.5)
    assert both.left_norm.weight == "l2.mix.left.out" and both.right_norm.width == 24
    assert (moe.experts, moe.identity, moe.top, moe.route_scale, moe.scoring, moe.renormalize, moe.activation) == (5, 2, 3, 1.5, "softmax", True, "silu")
    assert (spec.layers[0].ffn.activation, spec.layers[0].ffn.limit) == ("clamped_swish", 0.7)
    plain = copy.deepcopy(RAW)
    del plain["layers"][0]["mixer"]["rot"]["scaling"], plain["layers"][2]["mlp"]["router"]["identity"]
    spec = config_from_json(plain).to_spec()
    assert spec.layers[0].mixer.position.scaling is None and spec.layers[2].ffn.identity == 0


def test_tensor_names_and_shapes():
    from kapel_b200.parts import expected_tensors

    t = expected_tensors(config_from_json(RAW).to_spec())
    assert t["embed"] == (50, 24) and t["head"] == (50, 24) and t["final.norm"] == t["final.norm.b"] == (24,)
    assert t["l0.mix.q"] == (32, 24) and t["l0.mix.k"] == (16, 24) and t["l0.mix.v"] == (12, 24) and t["l0.mix.o"] == (24, 24)
    assert t["l0.mix.q.norm"] == (32,) and t["l0.mix.k.norm"] == (16,) and t["l0.norm1.b"] == (24,) and t["l0.ls1"] == t["l0.ls2"] == (24,)
    assert t["l0.hc1.in"] == t["l0.hc2.out"] == (3,) and t["l0.hc1.mix"] == (3, 3) and t["l0.mlp.gate"] == (20, 24)
    assert t["l1.mix.norm"] == (12,) and t["l1.mix.g"] == (12, 24) and t["l1.mix.k"] == (30, 24)
    assert not any(n.startswith(("l1.mlp", "l1.hc2", "l1.norm2", "l1.ls2")) for n in t)
    assert t["l2.mix.left.sink"] == (4,) and t["l2.mix.left.out"] == t["l2.mix.right.out"] == (24,) and t["l2.mix.left.o"] == (24, 40)
    assert t["l2.mix.right.k.conv"] == (12, 3) and t["l2.mix.right.b"] == (4, 24) and t["l2.mix.right.norm"] == (10,)
    assert t["l2.mlp.router"] == (7, 24) and t["l2.mlp.correction"] == (7,) and t["l2.mlp.e4.down"] == (24, 12) and "l2.mlp.e5.gate" not in t
    assert {n for n in t if n.startswith("l3.mix")} == {"l3.mix.q", "l3.mix.o", "l3.mix.q.norm"}


@pytest.mark.parametrize("edit,words", [
    (lambda r: r["layers"][0].update(type="conv"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=10), "at most"),
    (lambda r: r["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(kind="mlp"), "kind"),
    (lambda r: r["layers"][1]["mixer"].update(decay=[0.5]), "3 numbers"),
    (lambda r: r["layers"][2]["mixer"]["left"].pop("mask"), "mask"),
    (lambda r: r["layers"][2]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda r: r["layers"][2]["mixer"]["right"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][2]["mixer"]["right"].update(conv=0), "conv"),
    (lambda r: r["layers"][2]["mlp"]["router"].update(top=8), "top"),
    (lambda r: r["layers"][2]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=1), "earlier"),
    (lambda r: r["layers"][3]["mixer"].update(kv_from=3), "earlier"),
    (lambda r: r["layers"][3]["mixer"].update(kv_heads=3), "kv heads"),
    (lambda r: r.update(streams=0), "streams"),
    (lambda r: r.pop("streams"), "streams"),
])
def test_what_the_file_cannot_say(edit, words):
    raw = copy.deepcopy(RAW)
    edit(raw)
    with pytest.raises(ConfigError, match=words):
        config_from_json(raw)


def test_the_states_a_layers_parts_keep():
    """A layer that reads another's keys keeps nothing; a parallel layer keeps its window's pages and, under its side's name, a memory."""
    import torch

    from kapel_b200.cache import StateSpec
    from kapel_b200.engine.model import ModelParts
    from kapel_b200.parts import BuildContext

    m = ModelParts(config_from_json(RAW).to_spec(), BuildContext(dtype=torch.float32, device=torch.device("cpu")))
    needs = m.cache_needs()
    assert sorted(needs) == [0, 1, 2] and m.graph_safe()
    assert needs[0].paged.window is None and needs[0].paged.v_head_dim == 6 and needs[0].state is None
    assert needs[1].paged is None and needs[1].state == StateSpec((3 * 10 * 4,))
    assert needs[2].paged.window == 9 and dict(needs[2].states) == {"right": StateSpec((2 * (2 * 12 + 40) + 4 * 6 * 10,))}


def test_blocks_of_several_streams_and_of_one_do_not_mix():
    import dataclasses

    import torch

    from kapel_b200.engine.model import ModelParts
    from kapel_b200.parts import BuildContext

    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"))
    spec = config_from_json(RAW).to_spec()
    with pytest.raises(ValueError, match="streams"):
        ModelParts(dataclasses.replace(spec, streams=0), ctx)
    first = dataclasses.replace(spec.layers[1], kind="prenorm", streams=None)
    with pytest.raises(ValueError, match="streams"):
        ModelParts(dataclasses.replace(spec, layers=(spec.layers[0], first, *spec.layers[2:])), ctx)


# -------------------------------------------------------------------------------------- the plain rules on hand cases
def test_streams_by_hand():
    x = np.array([[[1.0, 2.0]], [[10.0, 20.0]]])                       # two streams, one token
    assert np.allclose(PS.read_streams(x, np.array([2.0, -1.0])), [[-8.0, -16.0]])
    mix = np.array([[1.0, 5.0], [0.0, 3.0]])                           # stream 0 goes to both, stream 1 only to itself
    y = PS.write_streams(x, mix, np.array([7.0, 0.0]), np.array([[1.0, 1.0]]))
    assert np.allclose(y, [[[8.0, 9.0]], [[35.0, 70.0]]])


def test_layer_norm_and_window_by_hand():
    assert np.allclose(PS.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 2.0]), np.array([0.5, -0.5]), 0.0), [[-1.5, 1.5]])
    w = PS.masked_softmax(np.zeros((4, 4)), 2, 0.0)
    assert np.allclose(w, [[1 / 2, 0, 0, 0], [1 / 3, 1 / 3, 0, 0], [0, 1 / 3, 1 / 3, 0], [0, 0, 1 / 3, 1 / 3]])
    assert np.allclose(PS.masked_softmax(np.zeros((3, 3)), None, math.log(2.0))[2], [1 / 5] * 3)


def test_rotation_by_hand_and_against_the_parts_frequencies():
    from kapel_b200.parts.position import scaled_frequencies

    y = PS.rotate_neighbours(np.array([[[1.0, 0.0, 0.0, 1.0, 7.0]]]), [3], {"base": 100.0, "dims": 4})[0, 0]       # pairs (0, 1) and (2, 3)
    assert np.allclose(y, [math.cos(3), math.sin(3), -math.sin(0.3), math.cos(0.3), 7.0])
    rot = {"base": 20.0, "dims": 10, "scaling": {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 0.5}}
    f, magnitude = scaled_frequencies(10, 20.0, RopeScaling(3.0, 64.0, 4.0, 0.5))
    want, m = PS.frequencies(rot)
    assert np.allclose(f, want, rtol=1e-14) and magnitude == m and math.isclose(m, 0.1 * math.log(3.0) + 1.0)
    assert len(set(np.round(PS.frequencies({"base": 20.0, "dims": 10})[0] / want, 6))) > 2


def test_memories_by_hand():
    q = k = np.array([[1.0, 0.0]] * 3)
    v = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(PS.decay_recurrence(q, k, v, 0.5)[:, 0], [1.0, 10.5, 105.25])
    one = np.ones(3)
    assert np.allclose(PS.delta_recurrence(q, k, v, one, one)[:, 0], [1.0, 10.0, 100.0])                # a step of one replaces what lies there
    assert np.allclose(PS.delta_recurrence(q, k, v, 0.5 * one, 0.5 * one)[:, 0], [0.5, 5.125, 51.28125])


def test_router_by_hand():
    """The correction chooses and does not weigh; the weights are those of the softmax over all outputs, renormalised and scaled."""
    z = np.log(np.array([1.0, 2.0, 3.0, 4.0]))
    chosen, w = PS.route(z, np.zeros(4), 2, 1.0)
    assert list(chosen) == [3, 2] and np.allclose(w, [4 / 7, 3 / 7])
    chosen, w = PS.route(z, np.array([1.0, 0.0, 0.0, 0.0]), 2, 3.0)
    assert list(chosen) == [0, 3] and np.allclose(w, [3 / 5, 12 / 5])


def test_bounded_unit_by_hand():
    t = {"m.gate": np.array([[1.0]]), "m.up": np.array([[2.0]]), "m.down": np.array([[1.0]])}
    unit = lambda h: PS.dense(np.array([[h]]), t, "m", {"limit": 1.5})[0, 0]
    g = lambda x: x / (1.0 + math.exp(-1.702 * x))
    assert math.isclose(unit(0.5), g(0.5) * 2.0) and math.isclose(unit(4.0), g(1.5) * 2.5) and math.isclose(unit(-4.0), g(-4.0) * -0.5)
