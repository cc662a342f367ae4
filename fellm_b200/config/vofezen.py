"""Typed configuration of the Vofezen design, read from its config.json.

The file is nested like Robazen's, Samusun's, Meresun's and Nalizen's: `layers` is a list of {type, mixer, mlp}, `norm` =
{eps}, beside `vocab` and `width`.  A layer's `type` is 'attention' or 'latent_attention'; its `mlp` is null or a dense
feed-forward {kind: dense, ff}.  Every size and every constant that can differ between two models of the design is read
here; a missing or ill-typed key raises ConfigError with the key's path.  What a file leaves out does not exist: no
rotation (`rot`), no scaling of its frequencies (`rot.scaling`), no value mixing (`v_mix`); `kv_heads` defaults to
`heads`, `vdim` to `dim`.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from .errors import ConfigError
from .meresun import FrequencyScaling
from .robazen import _get

NAME = "Vofezen"
LAYER_TYPES = ("attention", "latent_attention")


@dataclass(frozen=True)
class Rotation:
    """Rotary positions: `dims` elements in pairs (i, i + dims/2), frequencies base^(-2i/dims), scaled or not."""
    dims: int
    base: float
    scaling: Optional[FrequencyScaling]

    @staticmethod
    def read(d, where, most):
        """`d`: the mixer; most: how many elements can be rotated."""
        rot = _get(d, "rot", dict, where, required=False)
        if rot is None:
            return None
        where += ".rot"
        scaling = _get(rot, "scaling", dict, where, required=False)
        r = Rotation(dims=_get(rot, "dims", int, where), base=_get(rot, "base", float, where),
                     scaling=None if scaling is None else FrequencyScaling.read(scaling, where + ".scaling"))
        if r.dims % 2 or not 0 <= r.dims <= most:
            raise ConfigError(f"config.json: '{where}.dims' ({r.dims}) must be even and at most {most}")
        if r.base <= 0 or (r.scaling is not None and r.base <= 1):
            raise ConfigError(f"config.json: '{where}.base' must be positive (above 1 with scaling), got {r.base}")
        return r if r.dims else None

    def to_dict(self):
        d = dict(base=self.base, dims=self.dims)
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class AttentionConfig:
    """The 'attention' mixer: grouped queries, keys of `dim` and values of `vdim`, a rotation of a head's leading
    elements, a sink per head, values mixed with those of the first layer that mixes."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation]
    v_mix: bool

    @staticmethod
    def read(d, where):
        heads = _get(d, "heads", int, where, positive=True)
        dim = _get(d, "dim", int, where, positive=True)
        c = AttentionConfig(
            heads=heads, kv_heads=_get(d, "kv_heads", int, where, positive=True, required=False, default=heads),
            dim=dim, vdim=_get(d, "vdim", int, where, positive=True, required=False, default=dim),
            scale=_get(d, "scale", float, where), rot=Rotation.read(d, where, dim),
            v_mix=_get(d, "v_mix", bool, where, required=False, default=False))
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: '{where}.heads' ({c.heads}) is not a multiple of kv_heads ({c.kv_heads})")
        return c

    def to_dict(self):
        d = dict(dim=self.dim, heads=self.heads, kv_heads=self.kv_heads, scale=self.scale, v_mix=self.v_mix, vdim=self.vdim)
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class LatentAttentionConfig:
    """The 'latent_attention' mixer: queries through a latent of q_rank, keys and values through one latent of kv_rank and
    one rotated key part of rot_dim shared by the heads."""
    heads: int
    dim: int                  # unrotated query / key elements of a head
    rot_dim: int              # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[Rotation]

    @staticmethod
    def read(d, where):
        rot_dim = _get(d, "rot_dim", int, where, required=False, default=0)
        if rot_dim < 0:
            raise ConfigError(f"config.json: '{where}.rot_dim' must not be negative, got {rot_dim}")
        return LatentAttentionConfig(
            heads=_get(d, "heads", int, where, positive=True), dim=_get(d, "dim", int, where, positive=True),
            rot_dim=rot_dim, vdim=_get(d, "vdim", int, where, positive=True),
            q_rank=_get(d, "q_rank", int, where, positive=True), kv_rank=_get(d, "kv_rank", int, where, positive=True),
            scale=_get(d, "scale", float, where), rot=Rotation.read(d, where, rot_dim))

    def to_dict(self):
        d = dict(dim=self.dim, heads=self.heads, kv_rank=self.kv_rank, q_rank=self.q_rank, rot_dim=self.rot_dim,
                 scale=self.scale, vdim=self.vdim)
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class FeedForwardConfig:
    """kind 'dense': one feed-forward of `ff` with biases."""
    kind: str
    ff: int

    @staticmethod
    def read(d, where):
        kind = _get(d, "kind", str, where)
        if kind != "dense":
            raise ConfigError(f"config.json: '{where}.kind' is {kind!r}; known: dense")
        return FeedForwardConfig("dense", _get(d, "ff", int, where, positive=True))

    def to_dict(self):
        return dict(ff=self.ff, kind="dense")


@dataclass(frozen=True)
class VofezenLayer:
    type: str
    mixer: object
    mlp: Optional[FeedForwardConfig]          # None: the layer has no feed-forward

    def to_dict(self):
        return dict(mixer=self.mixer.to_dict(), mlp=None if self.mlp is None else self.mlp.to_dict(), type=self.type)


@dataclass
class VofezenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[VofezenLayer] = field(default_factory=list)

    @staticmethod
    def from_dict(d: dict) -> "VofezenConfig":
        vocab = _get(d, "vocab", int, "", positive=True)
        width = _get(d, "width", int, "", positive=True)
        eps = _get(_get(d, "norm", dict, ""), "eps", float, "norm")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]"
            kind = _get(L, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: '{where}.type' is {kind!r}; known: {', '.join(LAYER_TYPES)}")
            m = _get(L, "mixer", dict, where)
            mixer = (AttentionConfig if kind == "attention" else LatentAttentionConfig).read(m, where + ".mixer")
            mlp = None if L.get("mlp") is None else FeedForwardConfig.read(L["mlp"], where + ".mlp")
            layers.append(VofezenLayer(kind, mixer, mlp))
        mixing = [(i, L.mixer) for i, L in enumerate(layers) if getattr(L.mixer, "v_mix", False)]
        for i, m in mixing[1:]:
            j, first = mixing[0]
            if m.kv_heads * m.vdim != first.kv_heads * first.vdim:
                raise ConfigError(f"config.json: 'layers[{i}].mixer.v_mix': {m.kv_heads} x {m.vdim} values a token cannot be "
                                  f"mixed with layer {j}'s {first.kv_heads} x {first.vdim}")
        return VofezenConfig(vocab=vocab, width=width, norm_eps=eps, layers=layers)

    def to_dict(self) -> dict:
        return dict(architecture=NAME, layers=[L.to_dict() for L in self.layers], norm=dict(eps=self.norm_eps),
                    vocab=self.vocab, width=self.width)
