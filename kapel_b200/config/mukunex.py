"""Mukunex's configuration: a list of layers, each naming its mixer and its feed-forward.

config.json gives `architecture`, `vocab`, `width`, `norm.eps` and `layers`. A layer record is {type,
mixer, mlp}; its two RMS norms have plain weights (a layer without a feed-forward has one). `type`:

* "parallel": two mixers side by side, {left, right, left_scale, right_scale}. `left` is grouped-query
  attention with a sink a head in the softmax's denominator and one sigmoid gate a head on its output,
  {heads, kv_heads, dim, vdim, scale, rot{base, dims, scaling{factor, low, high, original}}}; `right` is
  retention, linear attention with a fixed decay a head, {heads, dim, vdim, decay[heads], rot}.
  Both turn the first `rot.dims` components of queries and keys, i with i + dims / 2.
* "rglru": a real-gated linear recurrent unit behind a short convolution, times a gelu branch
  {width, blocks, conv}; its two gates are `blocks` square matrices each.
* "channel_delta": the gated delta rule with a decay a head and key channel {heads, kv_heads, dim, vdim,
  conv}. The decay and the output gate come through low ranks, the number of rows of the tensors `a1`
  and `g1` (`decay_rank` and `gate_rank` may also be given here, as a model with random weights needs it).

`mlp` is {kind: "dense", ff} (gated, the tanh form of gelu) or null. The head is a table of its own.
Every size and constant is read from the file; the constants written here are those the design fixes
(the unit's rate of 8, the unit vectors' 1e-6).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional, Tuple

from .gemma2 import ConfigError, _MAX_HEAD_DIM, _MAX_HEADS, _MAX_HIDDEN, _MAX_INTERMEDIATE, _MAX_LAYERS, _MAX_VOCAB, _float, _int
from .lokedra import _flat, _record
from .spec import (
    AttentionSpec,
    BlockSpec,
    ChannelDeltaSpec,
    EmbedSpec,
    GatedMLPSpec,
    HeadSpec,
    LRUSpec,
    ModelSpec,
    NormSpec,
    ParallelMixerSpec,
    PositionSpec,
    RetentionSpec,
    RopeBands,
    default_schedule,
)

TYPES = ("parallel", "rglru", "channel_delta")
LRU_RATE = 8.0
UNIT_EPS = 1e-6


@dataclass(frozen=True)
class MukunexRotation:
    dims: int
    base: float
    scaling: Optional[RopeBands] = None


@dataclass(frozen=True)
class MukunexAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: MukunexRotation


@dataclass(frozen=True)
class MukunexRetention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: MukunexRotation


@dataclass(frozen=True)
class MukunexParallel:
    left: MukunexAttention
    right: MukunexRetention
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class MukunexLRU:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class MukunexDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None             # None until the tensors' shapes are known
    gate_rank: Optional[int] = None


@dataclass(frozen=True)
class MukunexLayer:
    type: str
    mixer: object
    ff: Optional[int]                            # the dense feed-forward's inner size; None: no feed-forward


def _heads_over(f: dict, where: str) -> Tuple[int, int]:
    heads = _int(f, [f"{where}heads"], hi=_MAX_HEADS)
    kv_heads = _int(f, [f"{where}kv_heads"], heads, hi=_MAX_HEADS)
    if heads % kv_heads:
        raise ConfigError(f"config.json: `{where}heads` = {heads} is not a multiple of `{where}kv_heads` = {kv_heads}")
    return heads, kv_heads


def _read_rot(m: dict, where: str, dim: int) -> MukunexRotation:
    rot = _record(m, "rot", where)
    f = _flat(rot, f"{where}rot.")
    dims = _int(f, [f"{where}rot.dims"], dim, lo=2, hi=_MAX_HEAD_DIM)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: `{where}rot.dims` = {dims} must be even and at most `{where}dim` = {dim}")
    base = _float(f, [f"{where}rot.base"], required=True)
    sc = _record(rot, "scaling", f"{where}rot.", required=False)
    bands = None
    if sc is not None:
        g = _flat(sc, f"{where}rot.scaling.")
        bands = RopeBands(*(_float(g, [f"{where}rot.scaling.{k}"], required=True) for k in ("factor", "low", "high", "original")))
        if bands.high < bands.low:
            raise ConfigError(f"config.json: `{where}rot.scaling.high` = {bands.high} must not be below `{where}rot.scaling.low` = {bands.low}")
    return MukunexRotation(dims, base, bands)


def _read_decay(m: dict, where: str, heads: int) -> Tuple[float, ...]:
    raw = m.get("decay")
    if not isinstance(raw, list) or len(raw) != heads or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in raw):
        raise ConfigError(f"config.json: `{where}decay` must be a list of {heads} numbers, one a head")
    if any(not 0.0 <= float(x) <= 1.0 for x in raw):
        raise ConfigError(f"config.json: `{where}decay` must lie between 0 and 1")
    return tuple(float(x) for x in raw)


def _read_mixer(kind: str, m: dict, where: str):
    w = f"{where}mixer."
    f = _flat(m, w)
    if kind == "parallel":
        left, right = _record(m, "left", w), _record(m, "right", w)
        fl, fr = _flat(left, f"{w}left."), _flat(right, f"{w}right.")
        heads, kv_heads = _heads_over(fl, f"{w}left.")
        dim = _int(fl, [f"{w}left.dim"], hi=_MAX_HEAD_DIM)
        attention = MukunexAttention(heads, kv_heads, dim, _int(fl, [f"{w}left.vdim"], dim, hi=_MAX_HEAD_DIM),
                                     _float(fl, [f"{w}left.scale"], required=True), _read_rot(left, f"{w}left.", dim))
        rheads = _int(fr, [f"{w}right.heads"], hi=_MAX_HEADS)
        rdim = _int(fr, [f"{w}right.dim"], hi=_MAX_HEAD_DIM)
        retention = MukunexRetention(rheads, rdim, _int(fr, [f"{w}right.vdim"], rdim, hi=_MAX_HEAD_DIM),
                                     _read_decay(right, f"{w}right.", rheads), _read_rot(right, f"{w}right.", rdim))
        return MukunexParallel(attention, retention, _float(f, [f"{w}left_scale"], 1.0, positive=False),
                               _float(f, [f"{w}right_scale"], 1.0, positive=False))
    if kind == "rglru":
        width = _int(f, [f"{w}width"], hi=_MAX_HIDDEN)
        blocks = _int(f, [f"{w}blocks"], hi=_MAX_HIDDEN)
        if width % blocks:
            raise ConfigError(f"config.json: `{w}width` = {width} is not a multiple of `{w}blocks` = {blocks}")
        return MukunexLRU(width, blocks, _int(f, [f"{w}conv"], hi=16))
    heads, kv_heads = _heads_over(f, w)
    dim = _int(f, [f"{w}dim"], hi=_MAX_HEAD_DIM)
    return MukunexDelta(heads, kv_heads, dim, _int(f, [f"{w}vdim"], dim, hi=_MAX_HEAD_DIM), _int(f, [f"{w}conv"], hi=16),
                        _int(f, [f"{w}decay_rank"], hi=_MAX_HIDDEN, required=False), _int(f, [f"{w}gate_rank"], hi=_MAX_HIDDEN, required=False))


def _read_mlp(m, where: str) -> Optional[int]:
    if m is None:
        return None
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: `{where}mlp` must be an object or null")
    if m.get("kind", "dense") != "dense":
        raise ConfigError(f"config.json: `{where}mlp.kind` = {m.get('kind')!r} is not known (\"dense\")")
    return _int(_flat(m, f"{where}mlp."), [f"{where}mlp.ff"], hi=_MAX_INTERMEDIATE)


@dataclass(frozen=True)
class MukunexConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[MukunexLayer, ...]

    architecture = "Mukunex"
    model_type = "mukunex"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_json(cls, raw: dict) -> "MukunexConfig":
        if not isinstance(raw, dict):
            raise ConfigError("config.json must hold a JSON object")
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw or len(layers_raw) > _MAX_LAYERS:
            raise ConfigError("config.json: `layers` must be a list of 1 to 4096 layer records")
        layers = []
        for i, rec in enumerate(layers_raw):
            where = f"layers[{i}]."
            if not isinstance(rec, dict):
                raise ConfigError(f"config.json: `layers[{i}]` must be an object")
            kind = rec.get("type")
            if kind not in TYPES:
                raise ConfigError(f"config.json: `{where}type` = {kind!r} is not known {TYPES}")
            layers.append(MukunexLayer(kind, _read_mixer(kind, _record(rec, "mixer", where), where), _read_mlp(rec.get("mlp"), where)))
        norm = _record(raw, "norm", "", required=False) or {}
        return cls(
            vocab=_int(raw, ["vocab"], hi=_MAX_VOCAB),
            width=_int(raw, ["width"], hi=_MAX_HIDDEN),
            eps=_float({"norm.eps": norm.get("eps")}, ["norm.eps"], 1e-6),
            layers=tuple(layers),
        )

    def with_shapes(self, shape_of) -> "MukunexConfig":
        """The configuration with the sizes that only the tensors give (`shape_of(name)` is a tensor's
        shape): the ranks behind a delta layer's decay and output gate are the rows of its `a1` and `g1`."""

        def rows(name: str, what: str) -> int:
            try:
                shape = tuple(shape_of(name))
            except KeyError:
                raise ConfigError(f"the tensor `{name}`, whose rows give {what}, is missing") from None
            if len(shape) != 2 or shape[0] < 1:
                raise ConfigError(f"the tensor `{name}` has shape {shape}, expected [rows, {self.width}]")
            return int(shape[0])

        layers = []
        for i, l in enumerate(self.layers):
            if l.type == "channel_delta":
                m = l.mixer
                if m.decay_rank is None:
                    m = replace(m, decay_rank=rows(f"l{i}.mix.a1", f"the rank of layer {i}'s decay"))
                if m.gate_rank is None:
                    m = replace(m, gate_rank=rows(f"l{i}.mix.g1", f"the rank of layer {i}'s output gate"))
                l = replace(l, mixer=m)
            layers.append(l)
        return replace(self, layers=tuple(layers))

    def to_json(self) -> dict:
        def rot_json(r: MukunexRotation) -> dict:
            out = {"base": r.base, "dims": r.dims}
            if r.scaling is not None:
                out["scaling"] = {"factor": r.scaling.factor, "low": r.scaling.low, "high": r.scaling.high, "original": r.scaling.original}
            return out

        layers = []
        for l in self.layers:
            m = l.mixer
            if l.type == "parallel":
                a, r = m.left, m.right
                mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "rot": rot_json(a.rot)},
                         "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay), "rot": rot_json(r.rot)},
                         "left_scale": m.left_scale, "right_scale": m.right_scale}
            elif l.type == "rglru":
                mixer = {"width": m.width, "blocks": m.blocks, "conv": m.conv}
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv}
                if m.decay_rank is not None:
                    mixer["decay_rank"] = m.decay_rank
                if m.gate_rank is not None:
                    mixer["gate_rank"] = m.gate_rank
            layers.append({"type": l.type, "mixer": mixer, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": layers}

    # ------------------------------------------------------------------ the model as data
    def _mixer_spec(self, i: int, l: MukunexLayer):
        w, p, m = self.width, f"l{i}.mix", l.mixer
        if l.type == "parallel":
            a, r = m.left, m.right
            names = {role: f"{p}.left.{role}" for role in ("q", "k", "v", "g", "o", "sink")}
            left = AttentionSpec(
                hidden=w, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, scale=a.scale, softcap=None,
                window=None, position=PositionSpec(theta=a.rot.base, rotary_dim=a.rot.dims, scaling=a.rot.scaling), weights=names,
                gated=True, gate_by_head=True, sink=True)
            right = RetentionSpec(
                hidden=w, num_heads=r.heads, head_dim=r.dim, v_head_dim=r.vdim, decay=r.decay, eps=self.eps,
                position=PositionSpec(theta=r.rot.base, rotary_dim=r.rot.dims, scaling=r.rot.scaling),
                weights={role: f"{p}.right.{role}" for role in ("q", "k", "v", "g", "o")})
            return ParallelMixerSpec(left=left, right=right, left_scale=m.left_scale, right_scale=m.right_scale)
        if l.type == "rglru":
            names = {role: f"{p}.{role}" for role in ("y", "x", "conv", "ra", "ri", "lam", "o")}
            names.update({f"{role}_bias": f"{p}.{role}.b" for role in ("y", "x", "conv", "ra", "ri")})
            return LRUSpec(hidden=w, width=m.width, blocks=m.blocks, conv=m.conv, weights=names, rate=LRU_RATE)
        if m.decay_rank is None or m.gate_rank is None:
            raise ConfigError(f"layer {i}: the ranks of the decay and the output gate are known from the tensors only (`with_shapes`), "
                              f"or from `layers[{i}].mixer.decay_rank` and `gate_rank`")
        names = {role: f"{p}.{role}" for role in ("q", "k", "v", "b", "A_log", "norm", "a1", "a2", "dt_bias", "g1", "g2", "o")}
        names.update({f"{role}_conv": f"{p}.{role}.conv" for role in ("q", "k", "v")})
        return ChannelDeltaSpec(
            hidden=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, conv=m.conv, decay_rank=m.decay_rank,
            gate_rank=m.gate_rank, eps=self.eps, weights=names, unit_eps=UNIT_EPS)

    def to_spec(self) -> ModelSpec:
        w = self.width
        blocks = []
        for i, l in enumerate(self.layers):
            norm = lambda name: NormSpec(width=w, eps=self.eps, offset=0.0, weight=f"l{i}.{name}")
            norms, ffn = {"pre_mixer": norm("norm1")}, None
            if l.ff is not None:
                norms["pre_ffn"] = norm("norm2")
                ffn = GatedMLPSpec(hidden=w, intermediate=l.ff, activation="gelu_tanh",
                                   weights={role: f"l{i}.mlp.{role}" for role in ("gate", "up", "down")})
            blocks.append(BlockSpec(kind="prenorm", mixer=self._mixer_spec(i, l), ffn=ffn, norms=norms))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=w,
            embed=EmbedSpec(weight="embed", scale=1.0, round_scale=False),
            layers=tuple(blocks), schedule=default_schedule(len(blocks)),
            final_norm=NormSpec(width=w, eps=self.eps, offset=0.0, weight="final.norm"),
            head=HeadSpec(weight="head", softcap=None), max_positions=None,
        )

    # ------------------------------------------------------------------ random weights
    def init_std(self, name: str, shape) -> float:
        """Tables N(0, inner width^-1/2) (the embedding N(0, 1)); vectors (norm weights, biases, sinks, rates)
        and convolution filters N(0, 0.5)."""
        if name == "embed":
            return 1.0
        if len(shape) <= 1 or name.endswith((".conv", ".b")):
            return 0.5
        return float(shape[-1]) ** -0.5
