"""Typed configuration of the Petelix design, read from its config.json.

The file is nested like the designs' before it: `layers` is a list of {type, mixer, mlp}, `norm` = {eps}, beside
`embedding.scale`, `vocab` and `width`.  A layer's `type` is 'attention'; its `mlp` is null or routed experts {kind: moe,
expert: {ff}, router: {experts, identity, top, groups: {count, keep}}}.  A mixer may read the keys and values of an earlier
layer (`kv_from`).  Every size and every constant that can differ between two models of the design is read here; a missing
or ill-typed key raises ConfigError with the key's path.  What a file leaves out does not exist: no window (`mask`), no
rotation (`rot`), no soft cap, no groups of experts, no identity experts; `kv_heads` defaults to `heads`, `vdim` to `dim`,
`embedding.scale` to 1.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from .errors import ConfigError
from .robazen import _get

NAME = "Petelix"
LAYER_TYPES = ("attention",)


@dataclass(frozen=True)
class CappedAttentionConfig:
    """The 'attention' mixer: queries and keys normed over their whole projections, a rotation of a head's leading elements
    (neighbouring pairs), scores under a soft cap, a sliding window, a sink of score 0, a sigmoid gate on the heads' outputs;
    `kv_from`: the layer whose keys and values it reads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    window: Optional[int]
    rot_dims: int
    rot_base: float
    kv_from: Optional[int]

    @staticmethod
    def read(d, where):
        mask = _get(d, "mask", dict, where, required=False)
        rot = _get(d, "rot", dict, where, required=False)
        heads = _get(d, "heads", int, where, positive=True)
        dim = _get(d, "dim", int, where, positive=True)
        c = CappedAttentionConfig(
            heads=heads, kv_heads=_get(d, "kv_heads", int, where, positive=True, required=False, default=heads),
            dim=dim, vdim=_get(d, "vdim", int, where, positive=True, required=False, default=dim),
            scale=_get(d, "scale", float, where), softcap=_get(d, "softcap", float, where, required=False),
            window=None if mask is None else _get(mask, "size", int, where + ".mask", positive=True),
            rot_dims=0 if rot is None else _get(rot, "dims", int, where + ".rot"),
            rot_base=10000.0 if rot is None else _get(rot, "base", float, where + ".rot"),
            kv_from=_get(d, "kv_from", int, where, required=False))
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: '{where}.heads' ({c.heads}) is not a multiple of kv_heads ({c.kv_heads})")
        if c.softcap is not None and not c.softcap > 0:
            raise ConfigError(f"config.json: '{where}.softcap' must be positive, got {c.softcap}")
        if c.rot_dims % 2 or not 0 <= c.rot_dims <= c.dim:
            raise ConfigError(f"config.json: '{where}.rot.dims' ({c.rot_dims}) must be even and at most dim ({c.dim})")
        if c.rot_base <= 0:
            raise ConfigError(f"config.json: '{where}.rot.base' must be positive, got {c.rot_base}")
        return c

    def to_dict(self):
        d = dict(dim=self.dim, heads=self.heads, kv_heads=self.kv_heads, scale=self.scale, vdim=self.vdim)
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        if self.window is not None:
            d["mask"] = dict(size=self.window)
        if self.rot_dims:
            d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
        if self.softcap is not None:
            d["softcap"] = self.softcap
        return d


@dataclass(frozen=True)
class RoutedExpertsConfig:
    """`experts` gated feed-forwards of `ff` each and `identity` experts that hand their input on, `top` a token, chosen
    inside `keep` of `groups` groups of neighbours (groups 0: no groups)."""
    ff: int
    experts: int
    identity: int
    top: int
    groups: int = 0
    keep: int = 0

    @staticmethod
    def read(d, where):
        kind = _get(d, "kind", str, where)
        if kind != "moe":
            raise ConfigError(f"config.json: '{where}.kind' is {kind!r}; known: moe")
        router = _get(d, "router", dict, where)
        where_r = where + ".router"
        groups = _get(router, "groups", dict, where_r, required=False)
        c = RoutedExpertsConfig(
            ff=_get(_get(d, "expert", dict, where), "ff", int, where + ".expert", positive=True),
            experts=_get(router, "experts", int, where_r, positive=True),
            identity=_get(router, "identity", int, where_r, required=False, default=0),
            top=_get(router, "top", int, where_r, positive=True),
            groups=0 if groups is None else _get(groups, "count", int, where_r + ".groups", positive=True),
            keep=0 if groups is None else _get(groups, "keep", int, where_r + ".groups", positive=True))
        if c.identity < 0:
            raise ConfigError(f"config.json: '{where_r}.identity' must not be negative, got {c.identity}")
        n = c.experts + c.identity
        if c.top > n:
            raise ConfigError(f"config.json: '{where_r}.top' ({c.top}) is above experts and identity experts ({n})")
        if c.groups:
            if n % c.groups or c.keep > c.groups:
                raise ConfigError(f"config.json: '{where_r}.groups' ({c.groups}, keep {c.keep}) does not fit {n} experts")
            if c.top > (n // c.groups) * c.keep:
                raise ConfigError(f"config.json: '{where_r}.top' ({c.top}) is above the experts of {c.keep} groups")
        return c

    def to_dict(self):
        router = dict(experts=self.experts, top=self.top)
        if self.groups:
            router["groups"] = dict(count=self.groups, keep=self.keep)
        if self.identity:
            router["identity"] = self.identity
        return dict(expert=dict(ff=self.ff), kind="moe", router=router)


@dataclass(frozen=True)
class PetelixLayer:
    type: str
    mixer: CappedAttentionConfig
    mlp: Optional[RoutedExpertsConfig]          # None: the layer has no feed-forward

    def to_dict(self):
        return dict(mixer=self.mixer.to_dict(), mlp=None if self.mlp is None else self.mlp.to_dict(), type=self.type)


@dataclass
class PetelixConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    layers: List[PetelixLayer] = field(default_factory=list)

    @staticmethod
    def from_dict(d: dict) -> "PetelixConfig":
        vocab = _get(d, "vocab", int, "", positive=True)
        width = _get(d, "width", int, "", positive=True)
        eps = _get(_get(d, "norm", dict, ""), "eps", float, "norm")
        emb = _get(d, "embedding", dict, "", required=False, default={})
        emb_scale = _get(emb, "scale", float, "embedding", required=False, default=1.0)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]"
            kind = _get(L, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: '{where}.type' is {kind!r}; known: {', '.join(LAYER_TYPES)}")
            mixer = CappedAttentionConfig.read(_get(L, "mixer", dict, where), where + ".mixer")
            mlp = None if L.get("mlp") is None else RoutedExpertsConfig.read(L["mlp"], where + ".mlp")
            layers.append(PetelixLayer(kind, mixer, mlp))
        for i, L in enumerate(layers):
            j = L.mixer.kv_from
            if j is None:
                continue
            where = f"layers[{i}].mixer.kv_from"
            if not 0 <= j < i:
                raise ConfigError(f"config.json: '{where}' ({j}) must name an earlier layer")
            src = layers[j].mixer
            if src.kv_from is not None:
                raise ConfigError(f"config.json: '{where}' names layer {j}, which keeps no keys and values of its own")
            if (src.kv_heads, src.dim, src.vdim, src.rot_dims, src.rot_base) != \
                    (L.mixer.kv_heads, L.mixer.dim, L.mixer.vdim, L.mixer.rot_dims, L.mixer.rot_base):
                raise ConfigError(f"config.json: '{where}': layer {j}'s key/value heads, sizes and rotation differ from layer {i}'s")
        return PetelixConfig(vocab=vocab, width=width, norm_eps=eps, embedding_scale=emb_scale, layers=layers)

    def to_dict(self) -> dict:
        return dict(architecture=NAME, embedding=dict(scale=self.embedding_scale), layers=[L.to_dict() for L in self.layers],
                    norm=dict(eps=self.norm_eps), vocab=self.vocab, width=self.width)
