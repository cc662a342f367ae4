"""Vofezen: how the design is put together from parts.

A layer is `x += norm1b(mixer(norm1(x))); x += norm2b(ff(norm2(x)))`: an RMSNorm in front of every sublayer and another on
its output (the 'sandwich' arrangement), all with weights stored around zero (parts/rmsnorm.py, `offset`).  A layer may
have no feed-forward.
  mixer 'attention'         grouped queries, keys and values of different sizes, rotation of a head's leading elements
                            (pairs i, i + r/2) with frequencies scaled for long contexts, a sink per head in the softmax's
                            denominator; in every mixing layer but the first, values mixed with the first mixing layer's
                            of the same token, (1 - l) v + l v_first, l a number of the layer     (parts/attention.py)
  mixer 'latent_attention'  queries through a normed latent, one normed key-value latent and one rotated key part a token
                            shared by the heads                                               (parts/latent_attention.py)
  feed-forward              W_down max(W_up h + b, 0)^2 + b'                                         (parts/plain_ff.py)

Tensor names of the safetensors file: embed, head, final.norm, and per layer i: l<i>.norm1, l<i>.norm1b, l<i>.norm2,
l<i>.norm2b, l<i>.mix.{q,k,v,vmix,sink,o} (attention) or l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o} (latent), and
l<i>.mlp.{up,up.b,down,down.b}.  The first mixing layer's vmix has no use; a file may hold it.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.vofezen import NAME, VofezenConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec

MAX_POSITION = 1 << 20        # nothing ends a context but memory
NORM_OFFSET = 1.0             # a norm multiplies by 1 + w


def _norm(name: str, d: int, eps: float) -> PartSpec:
    return PartSpec.make("rmsnorm", names={"weight": name}, size=d, eps=eps, offset=NORM_OFFSET)


def _position(rot) -> PartSpec:
    if rot is None:
        return PartSpec.make("none")
    s = rot.scaling
    return PartSpec.make("rope", rot_dim=rot.dims, theta=rot.base, pairing="split_half", table64=True,
                         scaling=None if s is None else (s.factor, s.original, s.fast, s.slow))


def _attention(p: str, d: int, m, eps: float, v_mix) -> PartSpec:
    names = {"q_proj.weight": p + "q", "k_proj.weight": p + "k", "v_proj.weight": p + "v", "out_proj.weight": p + "o",
             "sink": p + "sink", "vmix": p + "vmix"}
    return PartSpec.make("attention", names=names, size=d, heads=m.heads, kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim,
                         qk_norm=False, norm_eps=eps, position=_position(m.rot), scale=m.scale, sink=True, v_mix=v_mix)


def _latent(p: str, d: int, m, eps: float) -> PartSpec:
    names = {f"{t}.weight": p + t for t in ("dq", "uq", "dkv", "uk", "uv", "o")}
    names.update({"dq.norm": p + "dq.norm", "dkv.norm": p + "dkv.norm"})
    return PartSpec.make("latent_attention", names=names, size=d, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim,
                         v_dim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale, norm_eps=eps,
                         position=_position(m.rot))


def _feed_forward(p: str, d: int, f) -> PartSpec:
    return PartSpec.make("plain", names={"up.weight": p + "up", "up.bias": p + "up.b", "down.weight": p + "down",
                                         "down.bias": p + "down.b"},
                         size=d, ff=f.ff, act="relu2", bias=True)


def build_spec(cfg: VofezenConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    layers, unused = [], []
    first = next((i for i, L in enumerate(cfg.layers) if getattr(L.mixer, "v_mix", False)), None)
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        if L.type == "attention":
            v_mix = None if not L.mixer.v_mix else ("first" if i == first else "mix")
            mixer = _attention(p + "mix.", d, L.mixer, eps, v_mix)
            if v_mix != "mix":
                unused.append(p + "mix.vmix")
        else:
            mixer = _latent(p + "mix.", d, L.mixer, eps)
        ffn = None if L.mlp is None else _feed_forward(p + "mlp.", d, L.mlp)
        if ffn is None:
            unused += [p + "norm2", p + "norm2b"]
        layers.append(LayerSpec(norm1=_norm(p + "norm1", d, eps), mixer=mixer, norm1b=_norm(p + "norm1b", d, eps),
                                norm2=None if ffn is None else _norm(p + "norm2", d, eps), ffn=ffn,
                                norm2b=None if ffn is None else _norm(p + "norm2b", d, eps), arrangement="sandwich"))
    return ModelSpec(architecture=NAME, hidden_size=d, vocab_size=cfg.vocab, max_position=MAX_POSITION,
                     embedding=PartSpec.make("table", names={"weight": "embed"}, vocab=cfg.vocab, size=d),
                     layers=layers, final_norm=_norm("final.norm", d, eps),
                     head=PartSpec.make("linear", names={"weight": "head"}, vocab=cfg.vocab, size=d, tied=False),
                     unused=unused)


register_architecture(NAME, VofezenConfig.from_dict, build_spec)
