"""Typed configuration of the Zazulix decoder, read from its config.json.

A Zazulix model is a token embedding, a list of pre-norm layers (``x += mixer(N1 x)``, ``x += ff(N2 x)``), a final norm and the
embedding table again as the head.  An RMS norm multiplies by one plus its tensor.  Three mixers:
``latent_attention``, a windowed softmax attention through a latent without positions, its merged heads times a sigmoid
gate per channel; ``attention``, a differential attention (a head subtracts a multiple of one softmax from another) behind
short filters, with a rotation and a gate per head; ``retention``, a linear recurrence whose heads fade at constant rates.
A layer's feed-forward is absent, dense (both branches clamped, an activation of its own) or a mixture of experts: sigmoid scores,
choice by corrected scores inside the best groups of neighbours (a group's score: its two largest), and a shared expert
times a gate per token.

config.json keys (every size and every constant that differs between models is read from here):

    architecture            "Zazulix"
    vocab, width
    norm.eps
    layers[i].type          "latent_attention" | "attention" | "retention"
    layers[i].mixer         latent_attention: heads, dim, vdim, kv_rank, scale, mask {size} (absent: every earlier key);
                            attention: heads, kv_heads, dim, vdim, scale, diff, conv (absent: no filter), rot {base, dims};
                            retention: heads, dim, vdim, decay [heads], rot {base, dims}
    layers[i].mlp           null, {kind: "dense", ff, limit}, or {kind: "moe", expert {ff}, router {experts, top, scale,
                            groups {count, keep}}, shared {ff}}

Tensor names: ``embed``, ``final.norm``; layer i's start with ``l<i>.``: ``norm1``, ``norm2``, ``mix.q`` / ``k`` / ``v`` (+
``.conv``), ``mix.lq1`` / ``lk1`` / ``lq2`` / ``lk2``, ``mix.g``, ``mix.o``, ``mix.dkv`` (+ ``.norm``), ``mix.uk``, ``mix.uv``, ``mlp.gate`` /
``up`` / ``down``, ``mlp.router``, ``mlp.correction``, ``mlp.e<k>.gate`` / ``up`` / ``down``, ``mlp.shared.gate`` / ``up`` / ``down`` /
``sg``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional, Tuple

from .specs import (ConfigError, DifferentialAttentionNames, DifferentialAttentionSpec, GatedMLPNames, GatedMLPSpec,
                    LatentAttentionNames, LatentAttentionSpec, LayerSpec, ModelSpec, NormSpec, RetentionNames, RetentionSpec,
                    RotarySpec, RoutedExpertsSpec, default_schedule)

ARCHITECTURE = "Zazulix"
MAX_POSITIONS = 1 << 24          # the design sets no limit of its own; positions are 32-bit integers
ACTIVATION_SLOPE = 1.702         # the dense feed-forward's g * sigmoid(1.702 g) * (u + 1)
GROUP_TOP = 2                    # a group of experts is scored by the sum of its two largest choice scores
LATENT_NAMES = LatentAttentionNames(q="mix.q", down="mix.dkv", down_norm="mix.dkv.norm", up_k="mix.uk", up_v="mix.uv",
                                    o="mix.o", gate="mix.g")
DIFFERENTIAL_NAMES = DifferentialAttentionNames(q="mix.q", k="mix.k", v="mix.v", o="mix.o", gate="mix.g", lambda_q1="mix.lq1",
                                                lambda_k1="mix.lk1", lambda_q2="mix.lq2", lambda_k2="mix.lk2")
RETENTION_NAMES = RetentionNames(q="mix.q", k="mix.k", v="mix.v", gate="mix.g", o="mix.o")


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where}: required key '{key}' is missing")
    return d[key]


def _int(d, key: str, where: str, least: int = 1) -> int:
    v = _need(d, key, where)
    if isinstance(v, bool) or int(v) != v or int(v) < least:
        raise ConfigError(f"config.json: {where}.{key} must be an integer of at least {least}, got {v!r}")
    return int(v)


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int

    @classmethod
    def from_dict(cls, d, where, most: int) -> Optional["RotationConfig"]:
        """None where nothing is turned (no ``rot``, or ``dims`` of 0)."""
        if not d or not d.get("dims"):
            return None
        c = cls(base=float(_need(d, "base", where)), dims=_int(d, "dims", where))
        if c.dims % 2 or c.dims > most:
            raise ConfigError(f"config.json: {where}.dims={c.dims} must be even and at most {most}")
        if not c.base > 0:
            raise ConfigError(f"config.json: {where}.base={c.base} must be positive")
        return c

    def spec(self) -> RotarySpec:
        return RotarySpec(theta=self.base, dim=self.dims, max_positions=MAX_POSITIONS, variant="half_partial")


@dataclass(frozen=True)
class WindowedLatentConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int]                       # None: every earlier key is seen

    @classmethod
    def from_dict(cls, d, where):
        mask = d.get("mask") or {}
        return cls(heads=_int(d, "heads", where), dim=_int(d, "dim", where), vdim=_int(d, "vdim", where),
                   kv_rank=_int(d, "kv_rank", where), scale=float(_need(d, "scale", where)),
                   window=None if not mask.get("size") else _int(mask, "size", where + ".mask"))


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    conv: Optional[int]                         # taps; None: no filter
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, d, where):
        h, g = _int(d, "heads", where), _int(d, "kv_heads", where)
        if h % g:
            raise ConfigError(f"config.json: {where}: heads={h} is no multiple of kv_heads={g}")
        dim = _int(d, "dim", where)
        return cls(heads=h, kv_heads=g, dim=dim, vdim=_int(d, "vdim", where), scale=float(_need(d, "scale", where)),
                   diff=float(_need(d, "diff", where)), conv=None if not d.get("conv") else _int(d, "conv", where),
                   rot=RotationConfig.from_dict(d.get("rot"), where + ".rot", dim))


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, d, where):
        heads, dim = _int(d, "heads", where), _int(d, "dim", where)
        decay = tuple(float(x) for x in _need(d, "decay", where))
        if len(decay) != heads:
            raise ConfigError(f"config.json: {where}.decay holds {len(decay)} numbers for {heads} heads")
        if not all(0.0 <= x <= 1.0 for x in decay):
            raise ConfigError(f"config.json: {where}.decay={list(decay)} must lie between 0 and 1")
        return cls(heads=heads, dim=dim, vdim=_int(d, "vdim", where), decay=decay,
                   rot=RotationConfig.from_dict(d.get("rot"), where + ".rot", dim))


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                                   # "dense" | "moe"
    ff: int                                     # dense: its inner size; moe: an expert's
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    groups: int = 1
    keep: int = 1
    shared_ff: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        kind = _need(d, "kind", where)
        if kind == "dense":
            c = cls(kind=kind, ff=_int(d, "ff", where), limit=float(_need(d, "limit", where)))
            if not c.limit >= 0:
                raise ConfigError(f"config.json: {where}.limit={c.limit} must not be negative")
            return c
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind={kind!r}; the design has 'dense' and 'moe'")
        r, shared = _need(d, "router", where), d.get("shared")
        rw = where + ".router"
        g = r.get("groups") or {}
        count = 1 if not g.get("count") else _int(g, "count", rw + ".groups")
        c = cls(kind=kind, ff=_int(_need(d, "expert", where), "ff", where + ".expert"), experts=_int(r, "experts", rw),
                top=_int(r, "top", rw), scale=1.0 if r.get("scale") is None else float(r["scale"]), groups=count,
                keep=count if not g.get("keep") else _int(g, "keep", rw + ".groups"),
                shared_ff=None if not shared else _int(shared, "ff", where + ".shared"))
        if c.experts % c.groups or c.keep > c.groups or c.top > c.keep * (c.experts // c.groups):
            raise ConfigError(f"config.json: {rw}: {c.experts} experts in {c.groups} groups of which {c.keep} are kept, "
                              f"{c.top} per token: that many cannot be chosen")
        return c


@dataclass(frozen=True)
class ZazulixLayer:
    type: str
    latent: Optional[WindowedLatentConfig] = None
    attention: Optional[DifferentialConfig] = None
    retention: Optional[RetentionConfig] = None
    mlp: Optional[FeedForwardConfig] = None


# a layer's type -> (the field of ZazulixLayer, its class)
MIXERS = {"latent_attention": ("latent", WindowedLatentConfig), "attention": ("attention", DifferentialConfig),
          "retention": ("retention", RetentionConfig)}


@dataclass(frozen=True)
class ZazulixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[ZazulixLayer, ...]
    raw: dict = None                            # config.json as read (written back unchanged)
    architecture: str = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # ------------------------------------------------------------------ read
    @classmethod
    def from_dict(cls, d: dict) -> "ZazulixConfig":
        name = d.get("architecture") or (d.get("architectures") or [None])[0]
        if name != ARCHITECTURE:
            raise ConfigError(f"config.json: architecture={name!r}, expected {ARCHITECTURE!r}")
        layers = []
        for i, L in enumerate(_need(d, "layers", "config")):
            where = f"layers[{i}]"
            kind = _need(L, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}.type={kind!r}; the design has {sorted(MIXERS)}")
            field, mixer = MIXERS[kind]
            mlp = None if L.get("mlp") is None else FeedForwardConfig.from_dict(L["mlp"], where + ".mlp")
            layers.append(ZazulixLayer(type=kind, mlp=mlp, **{field: mixer.from_dict(_need(L, "mixer", where), where + ".mixer")}))
        if not layers:
            raise ConfigError("config.json: 'layers' is empty")
        cfg = cls(vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"),
                  norm_eps=float(_need(_need(d, "norm", "config"), "eps", "norm")), layers=tuple(layers), raw=copy.deepcopy(d))
        if not cfg.norm_eps >= 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        return cfg

    # ----------------------------------------------------------------- write
    def to_dict(self) -> dict:
        d = copy.deepcopy(self.raw)
        d.setdefault("architecture", ARCHITECTURE)
        return d

    # ------------------------------------------------------------ translation
    def _norm_spec(self) -> NormSpec:
        return NormSpec(size=self.width, eps=self.norm_eps, weight="", weight_offset=1.0)

    def _mixer_spec(self, L: ZazulixLayer):
        W, eps = self.width, self.norm_eps
        if L.latent is not None:
            m = L.latent
            return LatentAttentionSpec(hidden=W, n_heads=m.heads, plain_dim=m.dim, rot_dim=0, value_dim=m.vdim, kv_rank=m.kv_rank,
                                       softmax_scale=m.scale, eps=eps, window=m.window, gate=True, names=LATENT_NAMES)
        if L.attention is not None:
            a = L.attention
            return DifferentialAttentionSpec(hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, key_dim=a.dim, value_dim=a.vdim,
                                             softmax_scale=a.scale, diff=a.diff, eps=eps, conv_taps=a.conv,
                                             position=None if a.rot is None else a.rot.spec(), names=DIFFERENTIAL_NAMES)
        r = L.retention
        return RetentionSpec(hidden=W, heads=r.heads, key_dim=r.dim, value_dim=r.vdim, decay=r.decay, eps=eps,
                             position=None if r.rot is None else r.rot.spec(), names=RETENTION_NAMES)

    def _ff_spec(self, c: Optional[FeedForwardConfig]):
        if c is None:
            return None
        W = self.width
        if c.kind == "dense":
            return GatedMLPSpec(hidden=W, intermediate=c.ff, activation="clamped", limit=c.limit, slope=ACTIVATION_SLOPE,
                                names=GatedMLPNames(gate="mlp.gate", up="mlp.up", down="mlp.down"))
        shared = None
        if c.shared_ff:
            shared = GatedMLPSpec(hidden=W, intermediate=c.shared_ff, activation="silu",
                                  names=GatedMLPNames(gate="mlp.shared.gate", up="mlp.shared.up", down="mlp.shared.down"))
        return RoutedExpertsSpec(hidden=W, intermediate=c.ff, n_experts=c.experts, top=c.top, groups=c.groups, groups_keep=c.keep,
                                 group_top=GROUP_TOP, scale=c.scale, scores="sigmoid", activation="silu", shared=shared,
                                 shared_gate=None if shared is None else "mlp.shared.sg", router="mlp.router",
                                 correction="mlp.correction", expert="mlp.e{}.")

    def to_model_spec(self) -> ModelSpec:
        specs = []
        for i, L in enumerate(self.layers):
            ff = self._ff_spec(L.mlp)
            specs.append(LayerSpec(prefix=f"l{i}.", mixer=self._mixer_spec(L), feed_forward=ff, mixer_norm=self._norm_spec(),
                                   feed_forward_norm=None if ff is None else self._norm_spec(), mixer_norm_prefix="norm1",
                                   feed_forward_norm_prefix="norm2"))
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden=self.width, layers=tuple(specs),
            schedule=default_schedule(len(specs)), final_norm=self._norm_spec(), tie_embeddings=True,
            max_positions=MAX_POSITIONS, embed_name="embed", final_norm_prefix="final.norm", head_name="head")
