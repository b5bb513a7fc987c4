"""Sopalorn's configuration: a list of layers over several residual streams, each naming its mixer and its feed-forward.

config.json gives `architecture`, `vocab`, `width`, `streams`, `embedding.scale`, `logit_scale`, `norm.eps` and `layers`. A
layer record is {type, mixer, mlp}. Every sublayer reads the streams through its own weights and a layer norm with a bias,
and writes its result, times a weight a channel, back into all of them. `type`:

* "attention": grouped queries, RMS norms over the whole query and key projections, the first `rot.dims` components turned
  (2i with 2i + 1), 1 in the softmax's denominator {heads, kv_heads, dim, vdim, scale, rot{base, dims, scaling{factor,
  original, fast, slow}}}. With `kv_from` the layer takes that layer's keys and values and has none of its own.
* "lightning": linear attention with a fixed decay a head behind silu, one RMS norm over all heads, a sigmoid gate
  {heads, dim, vdim, decay[heads]}.
* "parallel": half the sum of two mixers that read the same input, each RMS-normed over the width. `left`: attention over a
  sliding window with a learned sink a head and no positions {heads, kv_heads, dim, vdim, scale, mask{size}}; `right`: the
  gated delta rule {heads, kv_heads, dim, vdim, conv}.

`mlp` is {kind: "dense", ff, limit} (the gated unit with both halves bounded), {kind: "moe", router{experts, identity, top,
scale}, expert{ff}} (silu-gated experts; the last `identity` outputs of the router give the input back) or null. The head is
a table of its own. Every size and constant is read from the file; the constants written here are those the design fixes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .gemma2 import ConfigError, _MAX_HEAD_DIM, _MAX_HEADS, _MAX_HIDDEN, _MAX_INTERMEDIATE, _MAX_LAYERS, _MAX_VOCAB, _float, _int
from .lokedra import _flat, _record
from .mukunex import _heads_over, _read_decay
from .spec import (
    AttentionSpec,
    BlockSpec,
    DeltaSpec,
    EmbedSpec,
    GatedMLPSpec,
    HeadSpec,
    ModelSpec,
    MoESpec,
    NormSpec,
    ParallelMixerSpec,
    PositionSpec,
    RetentionSpec,
    RopeScaling,
    ScheduleEntry,
    StreamsSpec,
)

TYPES = ("attention", "lightning", "parallel")
SWISH_ALPHA = 1.702
UNIT_EPS = 1e-6
SIDE_SCALE = 0.5
_MAX_STREAMS = 16


@dataclass(frozen=True)
class SopalornRotation:
    dims: int
    base: float
    scaling: Optional[RopeScaling] = None


@dataclass(frozen=True)
class SopalornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: SopalornRotation
    kv_from: Optional[int] = None                # the layer whose keys and values this one takes; None: its own


@dataclass(frozen=True)
class SopalornLightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class SopalornWindow:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int


@dataclass(frozen=True)
class SopalornDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class SopalornParallel:
    left: SopalornWindow
    right: SopalornDelta


@dataclass(frozen=True)
class SopalornDense:
    ff: int
    limit: float


@dataclass(frozen=True)
class SopalornExperts:
    experts: int
    identity: int
    top: int
    scale: float
    ff: int


@dataclass(frozen=True)
class SopalornLayer:
    type: str
    mixer: object
    mlp: object                                  # SopalornDense, SopalornExperts or None


def _sizes(m: dict, where: str) -> Tuple[int, int, int, int]:
    """heads, kv_heads, dim and vdim of a record."""
    f = _flat(m, where)
    heads, kv_heads = _heads_over(f, where)
    dim = _int(f, [f"{where}dim"], hi=_MAX_HEAD_DIM)
    return heads, kv_heads, dim, _int(f, [f"{where}vdim"], dim, hi=_MAX_HEAD_DIM)


def _read_rot(m: dict, where: str, dim: int) -> SopalornRotation:
    rot = _record(m, "rot", where)
    f = _flat(rot, f"{where}rot.")
    dims = _int(f, [f"{where}rot.dims"], dim, lo=2, hi=_MAX_HEAD_DIM)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: `{where}rot.dims` = {dims} must be even and at most `{where}dim` = {dim}")
    base = _float(f, [f"{where}rot.base"], required=True)
    sc = _record(rot, "scaling", f"{where}rot.", required=False)
    scaling = None
    if sc is not None:
        g = _flat(sc, f"{where}rot.scaling.")
        scaling = RopeScaling(*(_float(g, [f"{where}rot.scaling.{k}"], required=True) for k in ("factor", "original", "fast", "slow")))
        if base <= 1.0:
            raise ConfigError(f"config.json: `{where}rot.base` = {base} must be above 1 where `scaling` is given")
    return SopalornRotation(dims, base, scaling)


def _read_mixer(kind: str, m: dict, where: str):
    w = f"{where}mixer."
    f = _flat(m, w)
    if kind == "attention":
        heads, kv_heads, dim, vdim = _sizes(m, w)
        kv_from = None if m.get("kv_from") is None else _int(f, [f"{w}kv_from"], lo=0, hi=_MAX_LAYERS)
        return SopalornAttention(heads, kv_heads, dim, vdim, _float(f, [f"{w}scale"], required=True, positive=False), _read_rot(m, w, dim), kv_from)
    if kind == "lightning":
        heads = _int(f, [f"{w}heads"], hi=_MAX_HEADS)
        dim = _int(f, [f"{w}dim"], hi=_MAX_HEAD_DIM)
        return SopalornLightning(heads, dim, _int(f, [f"{w}vdim"], dim, hi=_MAX_HEAD_DIM), _read_decay(m, w, heads))
    left, right = _record(m, "left", w), _record(m, "right", w)
    mask = _record(left, "mask", f"{w}left.")
    window = SopalornWindow(*_sizes(left, f"{w}left."), _float(_flat(left, f"{w}left."), [f"{w}left.scale"], required=True, positive=False),
                            _int(_flat(mask, f"{w}left.mask."), [f"{w}left.mask.size"], hi=1 << 30))
    delta = SopalornDelta(*_sizes(right, f"{w}right."), _int(_flat(right, f"{w}right."), [f"{w}right.conv"], hi=16))
    return SopalornParallel(window, delta)


def _read_mlp(m, where: str):
    if m is None:
        return None
    if not isinstance(m, dict):
        raise ConfigError(f"config.json: `{where}mlp` must be an object or null")
    w = f"{where}mlp."
    kind = m.get("kind", "dense")
    if kind == "dense":
        f = _flat(m, w)
        return SopalornDense(_int(f, [f"{w}ff"], hi=_MAX_INTERMEDIATE), _float(f, [f"{w}limit"], required=True))
    if kind != "moe":
        raise ConfigError(f"config.json: `{w}kind` = {kind!r} is not known (\"dense\", \"moe\")")
    router, expert = _record(m, "router", w), _record(m, "expert", w)
    f = _flat(router, f"{w}router.")
    experts = _int(f, [f"{w}router.experts"], hi=1 << 16)
    identity = _int(f, [f"{w}router.identity"], 0, lo=0, hi=1 << 16)
    return SopalornExperts(experts, identity, _int(f, [f"{w}router.top"], hi=experts + identity),
                           _float(f, [f"{w}router.scale"], 1.0, positive=False), _int(_flat(expert, f"{w}expert."), [f"{w}expert.ff"], hi=_MAX_INTERMEDIATE))


@dataclass(frozen=True)
class SopalornConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    embed_scale: float
    logit_scale: float
    layers: Tuple[SopalornLayer, ...]

    architecture = "Sopalorn"
    model_type = "sopalorn"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_json(cls, raw: dict) -> "SopalornConfig":
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
            layers.append(SopalornLayer(kind, _read_mixer(kind, _record(rec, "mixer", where), where), _read_mlp(rec.get("mlp"), where)))
        for i, l in enumerate(layers):
            if l.type != "attention" or l.mixer.kv_from is None:
                continue
            j, where = l.mixer.kv_from, f"layers[{i}].mixer.kv_from"
            if j >= i or layers[j].type != "attention" or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: `{where}` = {j} must name an earlier attention layer with keys and values of its own")
            a, b = l.mixer, layers[j].mixer
            if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                raise ConfigError(f"config.json: `{where}` = {j}: that layer has {b.kv_heads} kv heads of {b.dim} and {b.vdim}, this one reads "
                                  f"{a.kv_heads} of {a.dim} and {a.vdim}")
        norm = _record(raw, "norm", "", required=False) or {}
        embedding = _record(raw, "embedding", "", required=False) or {}
        return cls(
            vocab=_int(raw, ["vocab"], hi=_MAX_VOCAB),
            width=_int(raw, ["width"], hi=_MAX_HIDDEN),
            streams=_int(raw, ["streams"], hi=_MAX_STREAMS),
            eps=_float({"norm.eps": norm.get("eps")}, ["norm.eps"], 1e-5),
            embed_scale=_float({"embedding.scale": embedding.get("scale")}, ["embedding.scale"], 1.0, positive=False),
            logit_scale=_float(raw, ["logit_scale"], 1.0, positive=False),
            layers=tuple(layers),
        )

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.type == "attention":
                rot = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.scaling is not None:
                    s = m.rot.scaling
                    rot["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": rot}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            elif l.type == "lightning":
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
            else:
                a, r = m.left, m.right
                mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "mask": {"size": a.window}},
                         "right": {"heads": r.heads, "kv_heads": r.kv_heads, "dim": r.dim, "vdim": r.vdim, "conv": r.conv}}
            mlp = None
            if isinstance(l.mlp, SopalornDense):
                mlp = {"kind": "dense", "ff": l.mlp.ff, "limit": l.mlp.limit}
            elif l.mlp is not None:
                e = l.mlp
                mlp = {"kind": "moe", "router": {"experts": e.experts, "identity": e.identity, "top": e.top, "scale": e.scale}, "expert": {"ff": e.ff}}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale, "layers": layers}

    # ------------------------------------------------------------------ the model as data
    def _mixer_spec(self, i: int, l: SopalornLayer):
        w, eps, p, m = self.width, self.eps, f"l{i}.mix", l.mixer
        if l.type == "attention":
            borrows = m.kv_from is not None
            names = {role: f"{p}.{role}" for role in (("q", "o") if borrows else ("q", "k", "v", "o"))}
            return AttentionSpec(
                hidden=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, scale=m.scale, softcap=None, window=None,
                position=PositionSpec(theta=m.rot.base, rotary_dim=m.rot.dims, pairing="neighbours", scaling=m.rot.scaling), weights=names,
                q_norm=NormSpec(width=m.heads * m.dim, eps=eps, offset=0.0, weight=f"{p}.q.norm"),
                k_norm=None if borrows else NormSpec(width=m.kv_heads * m.dim, eps=eps, offset=0.0, weight=f"{p}.k.norm"),
                unit_sink=True, borrows_kv=borrows)
        if l.type == "lightning":
            return RetentionSpec(
                hidden=w, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim, decay=m.decay, eps=eps, position=PositionSpec(kind="none"),
                weights={role: f"{p}.{role}" for role in ("q", "k", "v", "g", "norm", "o")}, activation="silu", key_scale=1.0, whole_norm=True,
                gate="sigmoid")
        a, r = m.left, m.right
        left = AttentionSpec(
            hidden=w, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, scale=a.scale, softcap=None, window=a.window,
            position=PositionSpec(kind="none"), weights={role: f"{p}.left.{role}" for role in ("q", "k", "v", "sink", "o")}, sink=True)
        names = {role: f"{p}.right.{role}" for role in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")}
        names.update({f"{role}_conv": f"{p}.right.{role}.conv" for role in ("q", "k", "v")})
        right = DeltaSpec(hidden=w, num_heads=r.heads, num_kv_heads=r.kv_heads, head_dim=r.dim, v_head_dim=r.vdim, conv=r.conv, eps=eps,
                          weights=names, unit_eps=UNIT_EPS)
        over = lambda side: NormSpec(width=w, eps=eps, offset=0.0, weight=f"{p}.{side}.out")
        return ParallelMixerSpec(left=left, right=right, left_scale=SIDE_SCALE, right_scale=SIDE_SCALE, left_norm=over("left"), right_norm=over("right"))

    def _ffn_spec(self, i: int, m):
        if m is None:
            return None
        f = f"l{i}.mlp"
        if isinstance(m, SopalornDense):
            return GatedMLPSpec(hidden=self.width, intermediate=m.ff, activation="clamped_swish", limit=m.limit, swish_alpha=SWISH_ALPHA,
                                weights={role: f"{f}.{role}" for role in ("gate", "up", "down")})
        weights = {"router": f"{f}.router", "correction": f"{f}.correction"}
        weights.update({role: f"{f}.e{{e}}.{role}" for role in ("gate", "up", "down")})
        return MoESpec(hidden=self.width, experts=m.experts, identity=m.identity, top=m.top, intermediate=m.ff, activation="silu", weights=weights,
                       scoring="softmax", renormalize=True, route_scale=m.scale, gated=True)

    def to_spec(self) -> ModelSpec:
        w = self.width
        norm = lambda name: NormSpec(width=w, eps=self.eps, offset=0.0, weight=name, bias=f"{name}.b", kind="layer")
        blocks, schedule = [], []
        for i, l in enumerate(self.layers):
            ffn = self._ffn_spec(i, l.mlp)
            streams = lambda q: StreamsSpec(count=self.streams, read=f"l{i}.hc{q}.in", write=f"l{i}.hc{q}.out", mix=f"l{i}.hc{q}.mix")
            norms = {"pre_mixer": norm(f"l{i}.norm1")}
            if ffn is not None:
                norms["pre_ffn"] = norm(f"l{i}.norm2")
            blocks.append(BlockSpec(kind="streams", mixer=self._mixer_spec(i, l), ffn=ffn, norms=norms,
                                    scales=(f"l{i}.ls1", f"l{i}.ls2" if ffn is not None else None),
                                    streams=(streams(1), streams(2) if ffn is not None else None)))
            source = l.mixer.kv_from if l.type == "attention" else None
            schedule.append(ScheduleEntry(i, i if source is None else source))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=w,
            embed=EmbedSpec(weight="embed", scale=self.embed_scale, round_scale=False),
            layers=tuple(blocks), schedule=tuple(schedule), final_norm=norm("final.norm"),
            head=HeadSpec(weight="head", softcap=None, scale=self.logit_scale), max_positions=None, streams=self.streams,
        )

    # ------------------------------------------------------------------ random weights
    def init_std(self, name: str, shape) -> float:
        """Tables N(0, inner width^-1/2) (the embedding N(0, 1)); vectors (norm weights and biases, branch weights, sinks, rates, the
        streams' weights) and convolution filters N(0, 0.5); the experts' corrections N(0, 0.1), below the scores' own spread."""
        if name == "embed":
            return 1.0
        if name.endswith(".correction"):
            return 0.1
        if len(shape) <= 1 or name.endswith(".conv"):
            return 0.5
        return float(shape[-1]) ** -0.5
