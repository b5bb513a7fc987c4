"""Mukunex without a GPU: the configuration and its errors, the model as data (tensor names, the sizes only a tensor gives, the
states a layer's parts keep), and the plain rules on hand cases."""
import copy
import math

import numpy as np
import pytest

import plain_mukunex as PM
from kapel_b200.config import ConfigError, RopeBands, config_from_json

DENSE = {"kind": "dense", "ff": 20}
RAW = {"architecture": "Mukunex", "vocab": 50, "width": 24, "norm": {"eps": 1e-5}, "layers": [
    {"type": "channel_delta", "mlp": DENSE, "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 10, "conv": 3, "decay_rank": 5, "gate_rank": 7}},
    {"type": "parallel", "mlp": None, "mixer": {
        "left": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3,
                 "rot": {"base": 50.0, "dims": 4, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}}},
        "right": {"heads": 3, "dim": 10, "vdim": 4, "decay": [0.5, 1.0, 0.875], "rot": {"base": 90.0, "dims": 6}},
        "left_scale": 0.5, "right_scale": 2.0}},
    {"type": "rglru", "mlp": DENSE, "mixer": {"width": 30, "blocks": 5, "conv": 2}},
]}


def test_round_trip_and_the_model_as_data():
    c = config_from_json(RAW)
    assert type(c).__name__ == "MukunexConfig" and config_from_json(c.to_json()) == c
    spec = c.to_spec()
    assert [(e.layer, e.replica, e.before) for e in spec.schedule] == [(0, 0, None), (1, 0, None), (2, 0, None)]
    assert all(l.kind == "prenorm" and l.norms["pre_mixer"].offset == 0.0 for l in spec.layers)
    assert spec.layers[1].ffn is None and set(spec.layers[1].norms) == {"pre_mixer"} and spec.layers[0].ffn.activation == "gelu_tanh"
    assert spec.head.weight == "head" and spec.embed.weight == "embed" and spec.embed.scale == 1.0 and spec.final_norm.offset == 0.0
    both = spec.layers[1].mixer
    assert (both.left_scale, both.right_scale) == (0.5, 2.0)
    left, right = both.left, both.right
    assert left.sink and left.gated and left.gate_by_head and left.v_head_dim == 6 and left.scale == 0.3 and left.window is None
    assert left.position.rotary_dim == 4 and left.position.pairing == "half" and left.position.scaling == RopeBands(4.0, 1.0, 3.0, 40.0)
    assert right.decay == (0.5, 1.0, 0.875) and right.position.rotary_dim == 6 and right.position.scaling is None and right.position.theta == 90.0
    assert spec.layers[2].mixer.rate == 8.0 and spec.layers[0].mixer.unit_eps == 1e-6
    plain = copy.deepcopy(RAW)
    del plain["layers"][1]["mixer"]["left"]["rot"]["scaling"]
    assert config_from_json(plain).to_spec().layers[1].mixer.left.position.scaling is None


def test_tensor_names_shapes_and_the_sizes_only_tensors_give():
    from kapel_b200.parts import expected_tensors

    t = expected_tensors(config_from_json(RAW).to_spec())
    assert t["embed"] == (50, 24) and t["head"] == (50, 24) and t["final.norm"] == (24,)
    assert t["l0.mix.q"] == (12, 24) and t["l0.mix.v"] == (40, 24) and t["l0.mix.k.conv"] == (12, 3) and t["l0.mix.v.conv"] == (40, 3)
    assert t["l0.mix.b"] == (4, 24) and t["l0.mix.A_log"] == (4,) and t["l0.mix.a1"] == (5, 24) and t["l0.mix.a2"] == (24, 5)
    assert t["l0.mix.dt_bias"] == (24,) and t["l0.mix.g1"] == (7, 24) and t["l0.mix.g2"] == (40, 7) and t["l0.mix.norm"] == (10,)
    assert t["l0.mix.o"] == (24, 40) and t["l0.norm2"] == (24,) and t["l0.mlp.down"] == (24, 20)
    assert t["l1.mix.left.sink"] == (4,) and t["l1.mix.left.g"] == (4, 24) and t["l1.mix.left.v"] == (12, 24) and t["l1.mix.left.o"] == (24, 24)
    assert t["l1.mix.right.q"] == (30, 24) and t["l1.mix.right.g"] == (12, 24) and t["l1.mix.right.o"] == (24, 12)
    assert "l1.norm2" not in t and not any(n.startswith("l1.mlp") for n in t)
    assert t["l2.mix.ra"] == (5, 6, 6) and t["l2.mix.ra.b"] == (5, 6) and t["l2.mix.conv.b"] == (30,) and t["l2.mix.lam"] == (30,)
    assert t["l2.mix.y.b"] == (30,) and t["l2.mix.o"] == (24, 30)
    bare = copy.deepcopy(RAW)
    del bare["layers"][0]["mixer"]["decay_rank"], bare["layers"][0]["mixer"]["gate_rank"]
    c = config_from_json(bare)
    with pytest.raises(ConfigError, match="tensors"):
        c.to_spec()
    shapes = {"l0.mix.a1": (9, 24), "l0.mix.g1": (3, 24)}
    m = c.with_shapes(lambda n: shapes[n]).layers[0].mixer
    assert (m.decay_rank, m.gate_rank) == (9, 3)
    with pytest.raises(ConfigError, match="missing"):
        c.with_shapes(lambda n: {}[n])


@pytest.mark.parametrize("edit,words", [
    (lambda r: r["layers"][0].update(type="conv"), "type"),
    (lambda r: r["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(dims=3), "even"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"].update(dims=10), "at most"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(high=0.5), "below"),
    (lambda r: r["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5]), "3 numbers"),
    (lambda r: r["layers"][1]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]), "between"),
    (lambda r: r["layers"][1]["mixer"]["right"].pop("rot"), "rot"),
    (lambda r: r["layers"][1]["mixer"].pop("left"), "left"),
    (lambda r: r["layers"][2]["mixer"].update(blocks=4), "multiple"),
    (lambda r: r["layers"][2]["mixer"].pop("width"), "width"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda r: r["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda r: r.pop("width"), "width"),
])
def test_what_the_file_cannot_say(edit, words):
    raw = copy.deepcopy(RAW)
    edit(raw)
    with pytest.raises(ConfigError, match=words):
        config_from_json(raw)


def test_frequencies_in_three_bands():
    from kapel_b200.parts.position import scaled_frequencies

    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}}
    want = PM.frequencies(rot)
    got, magnitude = scaled_frequencies(32, 10000.0, RopeBands(8.0, 1.0, 4.0, 512.0))
    assert magnitude == 1.0 and np.allclose(got, want, rtol=1e-14)
    plain = PM.frequencies({"base": 10000.0, "dims": 32})
    ratio = plain / want
    assert ratio[0] == 1.0 and math.isclose(ratio[-1], 8.0) and np.any((ratio > 1.001) & (ratio < 7.999))
    same, _ = scaled_frequencies(32, 10000.0, RopeBands(8.0, 2.0, 2.0, 512.0))         # no band between: kept or divided, nothing else
    assert set(np.round(plain / np.array(same), 9)) == {1.0, 8.0}


def test_the_states_a_layers_parts_keep():
    """A parallel layer: pages for one side, the other side's memory under its name."""
    import torch

    from kapel_b200.cache import StateSpec
    from kapel_b200.parts import BuildContext, build_part

    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"))
    spec = config_from_json(RAW).to_spec()
    delta, par, lru = (build_part("mixer", l.mixer, ctx).cache_needs() for l in spec.layers)
    assert par.paged is not None and par.paged.kv_heads == 2 and par.paged.head_dim == 8 and dict(par.states) == {"right": StateSpec((3 * 10 * 4,))}
    assert delta.state == StateSpec((4 * 6 * 10,)) and dict(delta.states) == {"conv": StateSpec((2 * (2 * 12 + 40),))} and delta.paged is None
    assert lru.state == StateSpec((30,)) and dict(lru.states) == {"conv": StateSpec((30,))}


# -------------------------------------------------------------------------------------- the plain rules on hand cases
def test_softmax_with_a_sink_by_hand():
    w = PM.causal_softmax(np.zeros((3, 3)), math.log(2.0))
    assert np.allclose(w, [[1 / 3, 0, 0], [1 / 4, 1 / 4, 0], [1 / 5, 1 / 5, 1 / 5]])
    assert PM.causal_softmax(np.full((1, 1), -30.0), 0.0)[0, 0] < 1e-12
    assert np.isclose(PM.causal_softmax(np.full((1, 1), 5.0), -1e9)[0, 0], 1.0)


def test_rotation_and_convolution_by_hand():
    x = np.array([[[1.0, 0.0, 0.0, 1.0, 7.0]]])
    y = PM.rotate_halves(x, [3], {"base": 100.0, "dims": 4})[0, 0]                     # pairs (0, 2) and (1, 3), the fifth passes
    assert np.allclose(y, [math.cos(3), -math.sin(0.3), math.sin(3), math.cos(0.3), 7.0])
    assert np.allclose(PM.short_conv(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 1.0]])), [[1.0], [12.0], [24.0]])


def test_retention_by_hand():
    q = k = np.array([[1.0, 0.0]] * 3)
    v = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(PM.retention_recurrence(q, k, v, 0.5)[:, 0], [1.0, 10.5, 105.25])
    assert np.allclose(PM.retention_recurrence(q, k, v, 1.0)[:, 0], [1.0, 11.0, 111.0])


def test_recurrent_unit_by_hand():
    """With its recurrence gate shut (r = 0) the state stays and takes nothing; with a gate open and a large rate it is replaced
    by i u; the first row is like any other."""
    u = np.array([[2.0], [3.0], [5.0]])
    one, zero = np.ones((3, 1)), np.zeros((3, 1))
    assert np.allclose(PM.lru_recurrence(u, zero, one, np.array([1.0])), 0.0)
    assert np.allclose(PM.lru_recurrence(u, one, 0.5 * one, np.array([50.0])), 0.5 * u)
    lam = math.log(math.expm1(math.log(2.0) / 8.0))                                    # 8 softplus(lam) = log 2: a = 1/2
    b = math.sqrt(0.75)
    assert np.allclose(PM.lru_recurrence(u, one, one, np.array([lam]))[:, 0], [2 * b, 4 * b, 7 * b])
    r, i = PM.lru_gates(np.array([[1.0, 2.0, 3.0, 4.0]]), np.array([[[0.0, 1.0], [0.0, 0.0]], [[1.0, 0.0], [0.0, 0.0]]]), np.zeros((2, 2)),
                        np.zeros((2, 2, 2)), np.array([[0.0, 1.0], [2.0, 3.0]]))
    assert np.allclose(r[0], PM.sigmoid(np.array([2.0, 0.0, 3.0, 0.0]))) and np.allclose(i[0], PM.sigmoid(np.array([0.0, 1.0, 2.0, 3.0])))


def test_delta_rule_with_a_decay_a_channel_by_hand():
    """A step size of one puts the value under its key; another decay on another channel fades only that row."""
    d = 3
    k = np.eye(d)[[0, 1, 0]].astype(np.float64)
    v = np.array([[1.0, 2.0], [3.0, 4.0], [5.0, 6.0]])
    q = np.ones((3, d))
    g = np.tile(np.array([0.5, 1.0, 1.0]), (3, 1))
    out = PM.channel_delta_recurrence(q, k, v, g, np.ones(3))
    assert np.allclose(out[0], v[0]) and np.allclose(out[1], 0.5 * v[0] + v[1]) and np.allclose(out[2], v[1] + v[2])
    half = PM.channel_delta_recurrence(q, k, v, np.ones((3, d)), np.full(3, 0.5))
    assert np.allclose(half[2], 0.5 * v[1] + 0.5 * v[0] + 0.5 * (v[2] - 0.5 * v[0]))
