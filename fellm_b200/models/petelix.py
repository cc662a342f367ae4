"""Petelix: how the design is put together from parts.

A layer is `x += attention(norm1(x)); x += experts(norm2(x))`, both norms RMSNorms (the 'prenorm' arrangement).  A layer may
have no feed-forward.
  mixer 'attention'  grouped queries; q and k normed over their WHOLE projections (all heads' rows at once, weighted) before
                     they are split into heads and rotated on a head's leading elements, in neighbouring pairs (2i, 2i + 1);
                     scores under a soft cap; a sliding window; a sink of score 0 (one more in the softmax's denominator);
                     keys and values of different sizes; a sigmoid gate on the heads' outputs, from the mixer's own input; a
                     layer may read the keys and values of an earlier layer (`kv_from`: a schedule entry with cache_of)
                                                                                             (parts/attention.py)
  feed-forward       routed gated experts and identity experts behind one router: softmax scores over both, the choice by
                     score + correction inside the groups whose best choice score is largest, weights the plain scores
                                                                                             (parts/moe.py)
The embedding is scaled; the head is a matrix of its own.

Tensor names of the safetensors file: embed, head, final.norm, and per layer i: l<i>.norm1, l<i>.norm2,
l<i>.mix.{q,q.norm,k,k.norm,v,g,o} (no k, k.norm, v where the layer reads another's), l<i>.mlp.{router,correction} and
l<i>.mlp.e<j>.{gate,up,down}.
"""
from __future__ import annotations

from ..config.petelix import NAME, PetelixConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run
from .nalizen import kept_windows

MAX_POSITION = 1 << 20        # nothing ends a context but memory
SINK_SCORE = 0.0              # the score of every head's sink


def _norm(name: str, d: int, eps: float) -> PartSpec:
    return PartSpec.make("rmsnorm", names={"weight": name}, size=d, eps=eps)


def _attention(p: str, d: int, m, eps: float, cache_window) -> PartSpec:
    names = {"q_proj.weight": p + "q", "k_proj.weight": p + "k", "v_proj.weight": p + "v", "out_gate.weight": p + "g",
             "out_proj.weight": p + "o", "q_norm.weight": p + "q.norm", "k_norm.weight": p + "k.norm"}
    position = PartSpec.make("none")
    if m.rot_dims:
        position = PartSpec.make("rope", rot_dim=m.rot_dims, theta=m.rot_base, pairing="adjacent", table64=True)
    return PartSpec.make("attention", names=names, size=d, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim,
                         v_dim=m.vdim, qk_norm="whole", out_gate=True, norm_eps=eps, position=position, softcap=m.softcap,
                         window=m.window, cache_window=cache_window, scale=m.scale, sink=SINK_SCORE,
                         shares_cache=m.kv_from is not None)


def _feed_forward(p: str, d: int, f) -> PartSpec:
    names = {"router.weight": p + "router", "correction": p + "correction"}
    for e in range(f.experts):
        names.update({f"e{e}.{t}.weight": f"{p}e{e}.{t}" for t in ("gate", "up", "down")})
    return PartSpec.make("moe", names=names, size=d, ff=f.ff, experts=f.experts, identity=f.identity, top=f.top,
                         score="softmax", correction=True, groups=(f.groups, f.keep, 1) if f.groups else None)


def build_spec(cfg: PetelixConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    kept = kept_windows(cfg)
    layers, schedule, unused = [], [], []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        own = L.mixer.kv_from is None
        schedule.append(Run(i, cache_of=L.mixer.kv_from))              # (layers run once each: entry j is layer j)
        ffn = None if L.mlp is None else _feed_forward(p + "mlp.", d, L.mlp)
        if ffn is None:
            unused.append(p + "norm2")
        layers.append(LayerSpec(norm1=_norm(p + "norm1", d, eps),
                                mixer=_attention(p + "mix.", d, L.mixer, eps, kept[i] if own else "same"),
                                norm2=None if ffn is None else _norm(p + "norm2", d, eps), ffn=ffn))
    return ModelSpec(architecture=NAME, hidden_size=d, vocab_size=cfg.vocab, max_position=MAX_POSITION,
                     embedding=PartSpec.make("table", names={"weight": "embed"}, vocab=cfg.vocab, size=d,
                                             scale=cfg.embedding_scale),
                     layers=layers, final_norm=_norm("final.norm", d, eps),
                     head=PartSpec.make("linear", names={"weight": "head"}, vocab=cfg.vocab, size=d, tied=False),
                     schedule=schedule, unused=unused)


register_architecture(NAME, PetelixConfig.from_dict, build_spec)
