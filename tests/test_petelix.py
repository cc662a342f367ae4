"""Petelix without a GPU: the configuration reader, the model description made from it, the tensors it asks for, what its layers
keep between steps, the planning of its attention, and the plain implementation's own mechanisms."""
from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import petelix_util as U
import plain_petelix as P
from fellm_b200 import ops
from fellm_b200.cache.manager import CacheManager
from fellm_b200.config.errors import ConfigError, WeightError
from fellm_b200.config.registry import config_from_dict
from fellm_b200.models.model import build_model
from fellm_b200.parts.base import PagedKV, build_part
from fellm_b200.parts.spec import PartSpec
from fellm_b200.weights.loader import bind_tensors
from fellm_b200.weights.random_init import random_tensors


def _spec(cfg):
    arch, c = config_from_dict(cfg)
    return arch, c, arch.build_spec(c)


def test_config_round_trip_and_registry():
    for name, (cfg, _) in U.CONFIGS.items():
        arch, c, spec = _spec(cfg)
        assert arch.name == "Petelix" and c.to_dict() == cfg, name
        assert spec.vocab_size == cfg["vocab"] and spec.hidden_size == cfg["width"]
        assert all(ls.arrangement == "prenorm" and (ls.ffn is None) == (ls.norm2 is None) for ls in spec.layers)
        assert [r.cache_of for r in spec.schedule] == [L["mixer"].get("kv_from") for L in cfg["layers"]]
    for seed in range(40):
        cfg = U.random_config(seed)
        assert _spec(cfg)[1].to_dict() == cfg, seed


def test_what_a_file_leaves_out_does_not_exist():
    cfg = copy.deepcopy(U.CFG_A)
    m = cfg["layers"][1]["mixer"]
    del m["kv_heads"], m["vdim"], m["rot"], m["mask"], m["softcap"], cfg["embedding"]
    r = cfg["layers"][1]["mlp"]["router"]
    del r["groups"], r["identity"]
    _, c, _ = _spec(cfg)
    m, f = c.layers[1].mixer, c.layers[1].mlp
    assert m.kv_heads == m.heads and m.vdim == m.dim and m.rot_dims == 0 and m.window is None and m.softcap is None
    assert f.groups == 0 and f.identity == 0 and c.embedding_scale == 1.0


@pytest.mark.parametrize("path,value,word", [
    (("width",), None, "width"), (("norm",), {}, "norm.eps"), (("vocab",), 0, "vocab"), (("layers",), [], "layers"),
    (("layers", 0, "type"), "conv", "layers[0].type"), (("layers", 0, "mixer", "heads"), 0, "heads"),
    (("layers", 0, "mixer", "heads"), 5, "kv_heads"), (("layers", 0, "mixer", "scale"), None, "scale"),
    (("layers", 0, "mixer", "softcap"), 0.0, "softcap"), (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 0, "mixer", "rot", "dims"), 26, "rot.dims"),
    (("layers", 0, "mixer", "rot", "base"), 0.0, "rot.base"), (("layers", 0, "mixer", "kv_from"), 0, "layers[0].mixer.kv_from"),
    (("layers", 3, "mixer", "kv_from"), 2, "keeps no keys"), (("layers", 3, "mixer", "vdim"), 24, "layers[3].mixer.kv_from"),
    (("layers", 2, "mixer", "rot", "base"), 10.0, "rotation"), (("layers", 0, "mlp", "kind"), "dense", "mlp.kind"),
    (("layers", 0, "mlp", "expert", "ff"), 0, "expert.ff"), (("layers", 0, "mlp", "router", "identity"), -1, "identity"),
    (("layers", 0, "mlp", "router", "identity"), 8, "router.groups"), (("layers", 0, "mlp", "router", "groups", "keep"), 6, "router.groups"),
    (("layers", 0, "mlp", "router", "top"), 7, "router.top"), (("layers", 4, "mlp", "router", "top"), 9, "router.top")])
def test_config_errors_name_the_key(path, value, word):
    cfg = copy.deepcopy(U.CFG_A)
    d = cfg
    for k in path[:-1]:
        d = d[k]
    if value is None:
        del d[path[-1]]
    else:
        d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        _spec(cfg)
    assert word in str(e.value)


def test_tensor_names_and_shapes():
    table = build_model(_spec(U.CFG_A)[2], "bfloat16").param_table()
    shape = {n: d.shape for n, (_, _, d) in table.items()}
    assert shape["embed"] == (211, 96) and shape["head"] == (211, 96) and shape["final.norm"] == (96,)
    assert shape["l0.mix.q"] == (144, 96) and shape["l0.mix.k"] == (48, 96) and shape["l0.mix.v"] == (80, 96)
    assert shape["l0.mix.q.norm"] == (144,) and shape["l0.mix.k.norm"] == (48,)               # over the whole projections
    assert shape["l0.mix.g"] == (240, 96) and shape["l0.mix.o"] == (96, 240) and "l0.mix.sink" not in shape
    assert shape["l3.mix.q.norm"] == (240,)
    assert not {n for n in shape if n.startswith(("l2.mix.k", "l2.mix.v", "l3.mix.k", "l3.mix.v"))}
    assert shape["l0.mlp.router"] == (15, 96) and shape["l0.mlp.correction"] == (15,)          # identity experts included
    assert shape["l0.mlp.e5.gate"] == (40, 96) and shape["l0.mlp.e5.down"] == (96, 40) and "l0.mlp.e6.gate" not in shape
    assert "l3.norm2" not in shape and "l3.mlp.router" not in shape


def test_unknown_and_missing_tensors_are_named():
    _, c, spec = _spec(U.CFG_A)
    tensors = random_tensors(build_model(spec, "float32"), 3)
    tensors["l3.norm2"] = torch.ones(96)                       # a norm of a layer without experts may lie unread
    bind_tensors(build_model(spec, "float32"), tensors, "cpu")
    tensors["l2.mix.k"] = torch.zeros(48, 96)
    del tensors["l0.mlp.correction"]
    with pytest.raises(WeightError) as e:
        bind_tensors(build_model(spec, "float32"), tensors, "cpu")
    assert "l2.mix.k" in str(e.value) and "l0.mlp.correction" in str(e.value) and "norm2" not in str(e.value)


def test_pages_are_kept_for_the_widest_window_of_their_readers():
    needs = build_model(_spec(U.CFG_A)[2], "float32").cache_needs()
    assert needs[0] == PagedKV(2, 24, 50, None, 40, False) and needs[2] is None and needs[3] is None
    assert needs[1] == PagedKV(4, 10, 33, None, 6, False) and needs[4] == PagedKV(1, 16, 64, None, 8, False)
    assert build_model(_spec(U.CFG_M)[2], "float32").cache_needs()[0].window is None            # one reader has no window
    cache = CacheManager(needs, page_tokens=16, max_tokens=256, max_requests=2, n_ctx=256, dtype=None, device="cpu")
    assert cache.views(None)[0].pool.shape[1:] == (1, 2 * 16 * (24 + 40))


def test_the_fixed_sink_and_the_input_products_columns():
    part = build_part("mixer", PartSpec.make("attention", size=16, heads=3, kv_heads=1, head_dim=5, v_dim=7, qk_norm="whole", out_gate=True,
                                             norm_eps=1e-6, position=PartSpec.make("none"), softcap=3.0, window=4, sink=0.5), "float32")
    g = torch.Generator().manual_seed(1)
    part.bind({k: torch.randn(d.shape, generator=g) for k, d in part.decls.items()})
    assert torch.equal(part.w["sink"], torch.full((3,), 0.5)) and "sink" not in part.decls
    assert part.gate_off % 8 == 0 and part.gate_off >= 15 + 5 + 7 and part.w["qkv.weight"].shape[0] >= part.gate_off + 21
    zero = build_part("mixer", PartSpec.make("attention", size=16, heads=2, kv_heads=1, head_dim=16, qk_norm="whole", norm_eps=1e-6,
                                             position=PartSpec.make("none"), sink=0.0), "float32")
    assert zero.sink and zero.sink_score == 0.0                  # a score of zero is a sink; False is none


@pytest.mark.parametrize("kw,word", [(dict(qk_norm="row"), "qk_norm"), (dict(qk_norm="whole", v_mix="mix"), "mixing"),
                                     (dict(qk_norm="whole", bias=True), "bias"), (dict(qk_norm="whole", chunk=4), "chunk"),
                                     (dict(qk_norm=False, sink=0.0, softcap=4.0), "soft cap")])
def test_attention_refuses_what_it_does_not_combine(kw, word):
    with pytest.raises(ConfigError) as e:
        build_part("mixer", PartSpec.make("attention", size=32, heads=2, kv_heads=1, head_dim=16, norm_eps=1e-6,
                                          position=PartSpec.make("none"), **kw), "float32")
    assert word in str(e.value)


def test_key_ranges_of_a_window_start_at_its_first_page():
    for window in (1, 64, 65, 100, 1000, 5000, None):
        for rows in (1, 8, 64):
            split, ranges, stages, cluster = ops.decode_wide_plan(3000, rows, 4, 128, 64, window)
            span = 3072 if window is None else min(3072, window + 63)       # the longest stretch from the first page's start
            assert split % 64 == 0 and split * ranges >= span and split * (ranges - 1) < -(-span // 64) * 64
    assert ops.umma_prefill_takes(16, 4, 128, 64, 64, 100, 0.1, True) and not ops.umma_prefill_takes(16, 4, 128, 64, 64, 100, 0.1)


# ----------------------------------------------------------------------------- the plain implementation's own mechanisms

def test_plain_softmax_with_one_more():
    s = np.array([[1.0, -2.0, -np.inf]])
    z = 1.0 + math.e + math.exp(-2.0)
    assert np.allclose(P.softmax_with_one_more(s), [[math.e / z, math.exp(-2.0) / z, 0.0]])
    assert np.allclose(P.softmax_with_one_more(s - 800.0), 0.0) and np.allclose(P.softmax_with_one_more(s + 800.0).sum(), 1.0)


def test_plain_window_and_cap():
    see = P.visible(5, 2)
    assert see.sum(1).tolist() == [1, 2, 2, 2, 2] and see[3].tolist() == [False, False, True, True, False]
    assert P.visible(4, 1).sum() == 4 and P.visible(4, None).sum() == 10
    assert np.allclose(P.soft_cap(np.array([0.01, 1e6, -1e6]), 5.0), [0.01, 5.0, -5.0], atol=1e-6)


def test_plain_rotation_turns_neighbours_and_depends_on_distance_alone():
    f = P.rotary_frequencies(6, 50.0)
    g = np.random.default_rng(0)
    a, b = g.standard_normal((1, 1, 8)), g.standard_normal((1, 1, 8))
    dot = lambda i, j: float((P.rotate(a, [i], f) * P.rotate(b, [j], f)).sum())
    assert abs(dot(17, 5) - dot(12, 0)) < 1e-5 and abs(dot(17, 5) - dot(17, 6)) > 1e-3
    r = P.rotate(a, [9], f)
    assert np.array_equal(r[..., 6:], a[..., 6:]) and np.allclose(r[..., 0] ** 2 + r[..., 1] ** 2, a[..., 0] ** 2 + a[..., 1] ** 2)


def test_plain_choice():
    s = np.array([0.4, 0.1, 0.05, 0.05, 0.3, 0.1])
    assert P.choose(s, 0 * s, 2, 1, 1) == [0, 4]
    assert P.choose(s, 0 * s, 3, 3, 2) == [0, 4, 1]                        # groups (0,1) (2,3) (4,5): the second is out
    assert P.choose(s, 0 * s, 2, 3, 1) == [0, 1]                           # group (0,1) alone: 0.1 beats the others' 0.3
    down = np.array([-1.0, -1.0, -0.1, -0.2, -1.0, -1.0])                  # negative choice scores: group (2,3), never a zero
    assert P.choose(s, down, 2, 3, 1) == [2, 3]
    assert P.choose(s, down - 5.0, 6, 3, 3)[:2] == [2, 3]


def test_plain_identity_experts_hand_on_their_input():
    g = np.random.default_rng(1)
    h = g.standard_normal((3, 6))
    w = {"router": g.standard_normal((4, 6)), "correction": np.array([-9.0, -9.0, 0.0, 0.0])}
    for e in range(2):
        w.update({f"e{e}.gate": g.standard_normal((5, 6)), f"e{e}.up": g.standard_normal((5, 6)), f"e{e}.down": g.standard_normal((6, 5))})
    out = P.experts(h, w, "", dict(router=dict(experts=2, identity=2, top=2, groups=dict(count=1, keep=1))))
    z = h @ w["router"].T
    s = np.exp(z) / np.exp(z).sum(-1, keepdims=True)
    assert np.allclose(out, s[:, 2:].sum(-1, keepdims=True) * h)


def test_plain_model_shows_every_mechanism():
    """A change to any mechanism of configuration A moves the logits of the plain model far beyond rounding."""
    cfg, w = U.plain_model("A")
    toks = U.tokens("A", 60, 0)
    want = U.plain_run(cfg, w, toks)
    for change in ("softcap", "scale", "rot", "window", "reader's window", "gate", "q norm", "k norm", "correction", "groups", "identity", "kv_from"):
        c2, w2 = copy.deepcopy(cfg), dict(w)
        L = c2["layers"]
        if change == "softcap":
            L[2]["mixer"]["softcap"] = 40.0
        elif change == "scale":
            L[1]["mixer"]["scale"] *= 1.5
        elif change == "rot":
            L[0]["mixer"]["rot"]["base"] = 30.0
        elif change == "window":
            L[4]["mixer"]["mask"]["size"] = 30
        elif change == "reader's window":
            L[3]["mixer"]["mask"]["size"] = 21
        elif change == "gate":
            w2["l1.mix.g"] = 0 * w["l1.mix.g"]
        elif change == "q norm":
            w2["l2.mix.q.norm"] = np.ones_like(w["l2.mix.q.norm"])
        elif change == "k norm":
            w2["l0.mix.k.norm"] = np.ones_like(w["l0.mix.k.norm"])
        elif change == "correction":
            w2["l0.mlp.correction"] = 0 * w["l0.mlp.correction"]
        elif change == "groups":
            L[0]["mlp"]["router"]["groups"]["keep"] = 5
        elif change == "identity":                   # an expert in the place of the first identity expert
            L[0]["mlp"]["router"].update(experts=7, identity=8)
            w2.update({f"l0.mlp.e6.{t}": w[f"l0.mlp.e5.{t}"] for t in ("gate", "up", "down")})
        else:
            w2.update({f"l3.mix.{t}": w[f"l0.mix.{t}"] for t in ("k", "v", "k.norm")})
            del L[3]["mixer"]["kv_from"]
        moved = U.row_distances(U.plain_run(c2, w2, toks), want)[40:]
        assert float(torch.quantile(moved, 0.8)) > 3e-3, (change, float(torch.quantile(moved, 0.8)))
