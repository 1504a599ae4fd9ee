"""Typed configuration of the Tosodra decoder, read from its config.json.

A Tosodra model is a scaled token embedding, a list of layers, a final norm and the embedding table again as the head.
A layer's sublayers read the stream itself and a norm takes the stream and a sublayer's output together: ``x <-
N(alpha x + sublayer(x))``, with ``N`` an RMS norm in groups (the row in equal parts, each over its own root mean
square, times a weight).  Two mixers: ``attention``, a grouped-query attention inside chunks of the sequence, whose
weights are sigmoids of the scores plus a learned number per head (no softmax), whose q and k are normed over the whole
projection and turned by neighbours, whose values are normed per head, and whose merged heads are multiplied by a
sigmoid gate; ``latent_attention``, an ordinary softmax attention through a latent with a rotated key part shared by all
heads.  A layer's feed-forward is absent or a mixture of experts: sigmoid scores, the largest are chosen, a chosen
expert's score multiplies its INPUT, and a shared expert runs for every token.

config.json keys (every size and every constant that differs between models is read from here):

    architecture            "Tosodra"
    vocab, width
    embedding.scale         (absent: 1)
    norm.eps, norm.groups   (groups absent: 1)
    postln_alpha
    layers[i].type          "attention" | "latent_attention"
    layers[i].mixer         attention: heads, kv_heads, dim, vdim, scale, rot {base, dims}, mask {size} (absent: no chunks);
                            latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}
    layers[i].mlp           null, or {kind: "moe", expert {ff}, router {experts, top}, shared {ff}}

Tensor names: ``embed``, ``final.norm``; layer i's start with ``l<i>.``: ``norm1``, ``norm2``, ``mix.q`` / ``k`` / ``v`` (+
``.b``), ``mix.q.norm``, ``mix.k.norm``, ``mix.pb``, ``mix.g``, ``mix.o``, ``mix.dkv`` (+ ``.norm``), ``mix.uk``, ``mix.uv``,
``mlp.router``, ``mlp.e<k>.gate`` / ``up`` / ``down``, ``mlp.shared.gate`` / ``up`` / ``down``.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional, Tuple

from .specs import (ConfigError, GatedMLPNames, GatedMLPSpec, GroupedRMSNormSpec, HeadAttentionNames, HeadAttentionSpec,
                    LatentAttentionNames, LatentAttentionSpec, ModelSpec, RotarySpec, RoutedExpertsSpec, SumNormLayerSpec,
                    default_schedule)

ARCHITECTURE = "Tosodra"
MAX_POSITIONS = 1 << 24          # the design sets no limit of its own; positions are 32-bit integers
ATTENTION_NAMES = HeadAttentionNames(q="mix.q", k="mix.k", v="mix.v", o="mix.o", q_norm="mix.q.norm", k_norm="mix.k.norm",
                                     gate="mix.g", sink="mix.sink", score_bias="mix.pb")
LATENT_NAMES = LatentAttentionNames(q="mix.q", down="mix.dkv", down_norm="mix.dkv.norm", up_k="mix.uk", up_v="mix.uv",
                                    o="mix.o", sink="mix.sink")


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


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int]                        # None: every earlier key is seen
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, d, where):
        h, g = _int(d, "heads", where), _int(d, "kv_heads", where)
        if h % g:
            raise ConfigError(f"config.json: {where}: heads={h} is no multiple of kv_heads={g}")
        mask = d.get("mask") or {}
        dim = _int(d, "dim", where)
        return cls(heads=h, kv_heads=g, dim=dim, vdim=_int(d, "vdim", where), scale=float(_need(d, "scale", where)),
                   chunk=None if not mask.get("size") else _int(mask, "size", where + ".mask"),
                   rot=RotationConfig.from_dict(d.get("rot"), where + ".rot", dim))


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, d, where):
        rot_dim = _int(d, "rot_dim", where)
        return cls(heads=_int(d, "heads", where), dim=_int(d, "dim", where), rot_dim=rot_dim, vdim=_int(d, "vdim", where),
                   kv_rank=_int(d, "kv_rank", where), scale=float(_need(d, "scale", where)),
                   rot=RotationConfig.from_dict(d.get("rot"), where + ".rot", rot_dim))


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int                                     # an expert's inner size
    experts: int
    top: int
    shared_ff: Optional[int] = None

    @classmethod
    def from_dict(cls, d, where):
        kind = _need(d, "kind", where)
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind={kind!r}; the design has 'moe' (or no feed-forward)")
        r, shared = _need(d, "router", where), d.get("shared")
        c = cls(ff=_int(_need(d, "expert", where), "ff", where + ".expert"), experts=_int(r, "experts", where + ".router"),
                top=_int(r, "top", where + ".router"), shared_ff=None if not shared else _int(shared, "ff", where + ".shared"))
        if c.top > c.experts:
            raise ConfigError(f"config.json: {where}.router: {c.top} of {c.experts} experts cannot be chosen")
        return c


@dataclass(frozen=True)
class TosodraLayer:
    type: str
    attention: Optional[ChunkedAttentionConfig] = None
    latent: Optional[LatentConfig] = None
    mlp: Optional[ExpertsConfig] = None


@dataclass(frozen=True)
class TosodraConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    alpha: float
    layers: Tuple[TosodraLayer, ...]
    embed_scale: float = 1.0
    raw: dict = None                            # config.json as read (written back unchanged)
    architecture: str = ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # ------------------------------------------------------------------ read
    @classmethod
    def from_dict(cls, d: dict) -> "TosodraConfig":
        name = d.get("architecture") or (d.get("architectures") or [None])[0]
        if name != ARCHITECTURE:
            raise ConfigError(f"config.json: architecture={name!r}, expected {ARCHITECTURE!r}")
        layers = []
        for i, L in enumerate(_need(d, "layers", "config")):
            where = f"layers[{i}]"
            kind = _need(L, "type", where)
            m = _need(L, "mixer", where)
            mlp = None if L.get("mlp") is None else ExpertsConfig.from_dict(L["mlp"], where + ".mlp")
            if kind == "attention":
                layers.append(TosodraLayer(type=kind, mlp=mlp, attention=ChunkedAttentionConfig.from_dict(m, where + ".mixer")))
            elif kind == "latent_attention":
                layers.append(TosodraLayer(type=kind, mlp=mlp, latent=LatentConfig.from_dict(m, where + ".mixer")))
            else:
                raise ConfigError(f"config.json: {where}.type={kind!r}; the design has 'attention' and 'latent_attention'")
        if not layers:
            raise ConfigError("config.json: 'layers' is empty")
        norm = _need(d, "norm", "config")
        scale = (d.get("embedding") or {}).get("scale")
        cfg = cls(vocab=_int(d, "vocab", "config"), width=_int(d, "width", "config"), norm_eps=float(_need(norm, "eps", "norm")),
                  norm_groups=1 if norm.get("groups") is None else _int(norm, "groups", "norm"),
                  alpha=float(_need(d, "postln_alpha", "config")), layers=tuple(layers),
                  embed_scale=1.0 if scale is None else float(scale), raw=copy.deepcopy(d))
        if not cfg.norm_eps >= 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        if cfg.width % cfg.norm_groups:
            raise ConfigError(f"config.json: width={cfg.width} cannot be cut into norm.groups={cfg.norm_groups} equal parts")
        return cfg

    # ----------------------------------------------------------------- write
    def to_dict(self) -> dict:
        d = copy.deepcopy(self.raw)
        d.setdefault("architecture", ARCHITECTURE)
        return d

    # ------------------------------------------------------------ translation
    def _norm_spec(self, weight: str) -> GroupedRMSNormSpec:
        return GroupedRMSNormSpec(size=self.width, eps=self.norm_eps, groups=self.norm_groups, weight=weight)

    def _mixer_spec(self, L: TosodraLayer):
        W, eps = self.width, self.norm_eps

        def position(rot, variant):
            return None if rot is None else RotarySpec(theta=rot.base, dim=rot.dims, max_positions=MAX_POSITIONS, variant=variant)
        if L.type == "attention":
            a = L.attention
            return HeadAttentionSpec(hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, key_dim=a.dim, value_dim=a.vdim,
                                     softmax_scale=a.scale, eps=eps, position=position(a.rot, "interleaved"), bias_in=True,
                                     qk_norm_over="projection", value_norm=True, chunk=a.chunk, weights="sigmoid",
                                     channel_gate=True, names=ATTENTION_NAMES)
        m = L.latent
        return LatentAttentionSpec(hidden=W, n_heads=m.heads, plain_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim,
                                   kv_rank=m.kv_rank, softmax_scale=m.scale, eps=eps, position=position(m.rot, "half_partial"),
                                   names=LATENT_NAMES)

    def _ff_spec(self, c: Optional[ExpertsConfig]):
        if c is None:
            return None
        shared = None
        if c.shared_ff:
            shared = GatedMLPSpec(hidden=self.width, intermediate=c.shared_ff, activation="silu",
                                  names=GatedMLPNames(gate="mlp.shared.gate", up="mlp.shared.up", down="mlp.shared.down"))
        return RoutedExpertsSpec(hidden=self.width, intermediate=c.ff, n_experts=c.experts, top=c.top, scores="sigmoid",
                                 renormalize=False, weight_on="input", correction=None, activation="silu", shared=shared,
                                 router="mlp.router", expert="mlp.e{}.")

    def to_model_spec(self) -> ModelSpec:
        specs = []
        for i, L in enumerate(self.layers):
            ff = self._ff_spec(L.mlp)
            specs.append(SumNormLayerSpec(prefix=f"l{i}.", mixer=self._mixer_spec(L), mixer_norm=self._norm_spec("norm1"),
                                          feed_forward=ff, feed_forward_norm=None if ff is None else self._norm_spec("norm2"),
                                          alpha=self.alpha))
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden=self.width, layers=tuple(specs),
            schedule=default_schedule(len(specs)), final_norm=self._norm_spec("norm"), tie_embeddings=True,
            max_positions=MAX_POSITIONS, embed_name="embed", final_norm_prefix="final.", head_name="head",
            embed_scale=self.embed_scale)
