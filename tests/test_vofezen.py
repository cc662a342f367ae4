"""Vofezen without a GPU: the configuration reader, the model description made from it, the tensors it asks for (and those
it lets lie), what its layers keep between steps, which products the tensor-core attention takes, and the plain
implementation's own mechanisms."""
from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_vofezen as P
import vofezen_util as U
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
        assert arch.name == "Vofezen" and c.to_dict() == cfg, name
        assert spec.vocab_size == cfg["vocab"] and spec.hidden_size == cfg["width"]
        assert all(ls.arrangement == "sandwich" and ls.norm1b is not None for ls in spec.layers)
        assert all((ls.ffn is None) == (ls.norm2 is None) == (ls.norm2b is None) for ls in spec.layers)
    for seed in range(40):
        cfg = U.random_config(seed)
        _, c, _ = _spec(cfg)
        assert c.to_dict() == cfg, seed


def test_what_a_file_leaves_out_does_not_exist():
    cfg = copy.deepcopy(U.CFG_A)
    m = cfg["layers"][2]["mixer"]
    del m["kv_heads"], m["vdim"], m["rot"], m["v_mix"]
    del cfg["layers"][4]["mixer"]["rot_dim"]
    _, c, _ = _spec(cfg)
    m = c.layers[2].mixer
    assert m.kv_heads == m.heads and m.vdim == m.dim and m.rot is None and m.v_mix is False
    assert c.layers[4].mixer.rot_dim == 0 and c.layers[4].mixer.rot is None
    cfg["layers"][1]["mixer"]["rot"] = dict(base=10000.0, dims=0)           # a rotation of nothing is none
    assert _spec(cfg)[1].layers[1].mixer.rot is None


@pytest.mark.parametrize("path,value,word", [
    (("width",), None, "width"), (("norm",), {}, "norm.eps"), (("vocab",), 0, "vocab"), (("layers",), [], "layers"),
    (("layers", 0, "type"), "conv", "layers[0].type"), (("layers", 1, "mixer", "heads"), 0, "heads"),
    (("layers", 1, "mixer", "heads"), 5, "kv_heads"), (("layers", 1, "mixer", "scale"), None, "scale"),
    (("layers", 1, "mixer", "v_mix"), 1, "v_mix"), (("layers", 3, "mixer", "vdim"), 24, "layers[3].mixer.v_mix"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 1, "mixer", "rot", "dims"), 26, "rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), 1.0, "rot.base"), (("layers", 0, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0, "rot.scaling"),
    (("layers", 1, "mixer", "rot", "scaling", "fast"), None, "fast"),
    (("layers", 0, "mixer", "q_rank"), None, "q_rank"), (("layers", 0, "mixer", "kv_rank"), 0, "kv_rank"),
    (("layers", 0, "mixer", "rot", "dims"), 10, "rot.dims"), (("layers", 0, "mixer", "rot_dim"), -1, "rot_dim"),
    (("layers", 0, "mlp", "kind"), "moe", "mlp.kind"), (("layers", 1, "mlp", "ff"), 0, "mlp.ff")])
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
    _, c, spec = _spec(U.CFG_A)
    table = build_model(spec, "bfloat16").param_table()
    shape = {n: d.shape for n, (_, _, d) in table.items()}
    assert shape["embed"] == (211, 96) and shape["head"] == (211, 96) and shape["final.norm"] == (96,)
    assert shape["l0.mix.dq"] == (40, 96) and shape["l0.mix.dq.norm"] == (40,) and shape["l0.mix.uq"] == (84, 40)
    assert shape["l0.mix.dkv"] == (64, 96) and shape["l0.mix.dkv.norm"] == (56,) and shape["l0.mix.uk"] == (60, 56)
    assert shape["l0.mix.uv"] == (36, 56) and shape["l0.mix.o"] == (96, 36) and "l0.mix.sink" not in shape
    assert shape["l1.mix.q"] == (144, 96) and shape["l1.mix.k"] == (48, 96) and shape["l1.mix.v"] == (80, 96)
    assert shape["l1.mix.sink"] == (6,) and shape["l1.mix.o"] == (96, 240)
    assert "l1.mix.vmix" not in shape and "l2.mix.vmix" not in shape                # nothing to mix with; mixes nothing
    assert shape["l3.mix.vmix"] == () and shape["l5.mix.vmix"] == ()
    assert shape["l1.norm1"] == shape["l1.norm1b"] == shape["l1.norm2"] == shape["l1.norm2b"] == (96,)
    assert shape["l3.norm1b"] == (96,) and "l3.norm2" not in shape and "l3.norm2b" not in shape and "l3.mlp.up" not in shape
    assert shape["l1.mlp.up"] == (160, 96) and shape["l1.mlp.up.b"] == (160,)
    assert shape["l1.mlp.down"] == (96, 160) and shape["l1.mlp.down.b"] == (96,)


def test_a_file_may_hold_the_first_mixing_layers_number_but_nothing_unknown():
    _, c, spec = _spec(U.CFG_A)
    model = build_model(spec, "float32")
    tensors = random_tensors(model, 3)
    tensors["l1.mix.vmix"] = torch.tensor(0.5).bfloat16()
    bind_tensors(model, tensors, "cpu")
    # a norm around zero multiplies by 1 + w
    assert torch.equal(model.blocks[1].norm1b.w["weight"], tensors["l1.norm1b"].float() + 1.0)
    tensors["l1.mix.gate"] = torch.zeros(4)
    with pytest.raises(WeightError) as e:
        bind_tensors(build_model(spec, "float32"), tensors, "cpu")
    assert "l1.mix.gate" in str(e.value) and "vmix" not in str(e.value)


def test_what_the_layers_keep():
    _, c, spec = _spec(U.CFG_A)
    needs = build_model(spec, "float32").cache_needs()
    assert needs[0] == PagedKV(1, 64, None, None, None, True)                 # one latent and one rotated part a token
    assert needs[1] == PagedKV(2, 24, None, None, 40, False) and needs[3] == PagedKV(4, 8, None, None, 20, False)
    cache = CacheManager(needs, page_tokens=16, max_tokens=256, max_requests=3, n_ctx=256, dtype=None, device="cpu")
    views = cache.views(None)
    assert views[1].pool.shape[1:] == (1, 2 * 16 * 64) and views[0].pool.shape[1:] == (1, 16 * 64)


def test_split_half_rotation_of_a_latent_layer_is_the_neighbours_rotation_of_permuted_rows():
    """Pairs (i, i + n/2) of the queries' and the key's rotated parts are put side by side in the weights; the elements
    behind the rotated ones keep their places."""
    H, dn, dr, rk, rq, n = 2, 3, 7, 5, 4, 6
    part = build_part("mixer", PartSpec.make("latent_attention", size=8, heads=H, dim=dn, rot_dim=dr, v_dim=2, q_rank=rq, kv_rank=rk,
                                             scale=0.3, norm_eps=1e-6,
                                             position=PartSpec.make("rope", rot_dim=n, theta=50.0, pairing="split_half", table64=True)), "float32")
    g = torch.Generator().manual_seed(1)
    w = {k: torch.randn(d.shape, generator=g) for k, d in part.decls.items()}
    part.bind(dict(w))
    x = torch.randn(1, 8, generator=g).double()
    cq = torch.randn(1, rq, generator=g).double()
    q = (cq @ w["uq.weight"].double().T).view(H, dn + dr)
    q2 = (cq @ part.w["uq.weight"][:H * (dn + dr)].double().T).view(H, dn + dr)
    kr = (x @ w["dkv.weight"].double().T)[0, rk:]
    kr2 = (x @ part.w["down.weight"].double().T)[0, part.r_off:part.r_off + dr]
    f, _ = P.rotary_frequencies(n, 50.0)

    def neighbours(v, pos):
        out = v.clone()
        for i, fi in enumerate(f):
            c, s = math.cos(pos * fi), math.sin(pos * fi)
            out[..., 2 * i], out[..., 2 * i + 1] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s, v[..., 2 * i + 1] * c + v[..., 2 * i] * s
        return out
    want = [(P.rotate(q[None, :, dn:].numpy(), [9], f)[0] @ P.rotate(kr.numpy()[None, None], [4], f)[0, 0])]
    got = [(neighbours(q2[:, dn:], 9) @ neighbours(kr2, 4)).numpy()]
    assert np.allclose(got, want, atol=1e-5) and torch.equal(q[:, :dn], q2[:, :dn])


def test_sizes_the_tensor_core_attention_of_portions_takes():
    takes = lambda H, G, hd, vd, page=64, window=None, scale=0.1: ops.umma_prefill_takes(H, G, hd, vd, page, window, scale)
    assert takes(16, 4, 64, 64) and takes(8, 1, 128, 64) and takes(8, 8, 48, 80) and takes(32, 2, 128, 128) and takes(4, 4, 16, 16)
    assert not takes(6, 2, 64, 64)                 # three heads a kv head: 128 rows are no whole number of tokens
    assert not takes(8, 1, 128, 64, page=16) and not takes(8, 1, 128, 64, window=100) and not takes(8, 1, 128, 64, scale=-0.1)
    assert not takes(8, 1, 256, 64) and not takes(8, 1, 64, 144) and not takes(8, 1, 40, 64) and not takes(8, 1, 64, 24)


@pytest.mark.parametrize("kw,word", [(dict(v_mix="last"), "v_mix"), (dict(sink=True, softcap=5.0), "sink"), (dict(sink=True, bias=True), "sink"),
                                     (dict(v_mix="mix", shares_cache=True), "cache"), (dict(sink=True, v_dim=2048), "v_dim"),
                                     (dict(sink=True, out_gate=True), "gate")])
def test_attention_refuses_what_it_does_not_combine(kw, word):
    with pytest.raises(ConfigError) as e:
        build_part("mixer", PartSpec.make("attention", size=32, heads=2, kv_heads=1, head_dim=16, qk_norm=False, norm_eps=1e-6,
                                          position=PartSpec.make("none"), **kw), "float32")
    assert word in str(e.value)


# ----------------------------------------------------------------------------- the plain implementation's own mechanisms

def test_plain_softmax_with_a_sink():
    s = np.array([[1.0, 2.0, -np.inf]])
    p = P.softmax_with_sink(s, 0.5)
    z = math.e + math.e ** 2 + math.e ** 0.5
    assert np.allclose(p, [[math.e / z, math.e ** 2 / z, 0.0]]) and np.allclose(P.softmax_with_sink(s).sum(), 1.0)
    assert np.allclose(P.softmax_with_sink(s, 500.0), 0.0) and np.allclose(P.softmax_with_sink(s - 500.0, -800.0).sum(), 1.0)


def test_plain_frequencies_keep_the_fast_and_divide_the_slow():
    f, mag = P.rotary_frequencies(32, 10000.0, dict(factor=4.0, original=256, fast=16.0, slow=1.0))
    plain, one = P.rotary_frequencies(32, 10000.0)
    assert one == 1.0 and abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    assert np.allclose(f[:2], plain[:2]) and np.allclose(f[-3:], plain[-3:] / 4.0) and np.all(np.diff(f) < 0)


def test_plain_rotation_depends_on_distance_alone():
    f, _ = P.rotary_frequencies(6, 50.0)
    g = np.random.default_rng(0)
    a, b = g.standard_normal((1, 1, 8)), g.standard_normal((1, 1, 8))
    dot = lambda i, j: float((P.rotate(a, [i], f) * P.rotate(b, [j], f)).sum())
    assert abs(dot(17, 5) - dot(12, 0)) < 1e-5 and abs(dot(17, 5) - dot(17, 6)) > 1e-3
    assert np.array_equal(P.rotate(a, [9], f)[..., 6:], a[..., 6:])


def test_plain_value_mixing_and_norm_around_zero():
    assert np.allclose(P.mix_values(np.ones(3), np.full(3, 5.0), 0.25), 2.0)
    x = np.array([[3.0, -4.0]])
    assert np.allclose(P.norm(x, np.array([0.0, 1.0]), 0.0), [[3.0 / math.sqrt(12.5), -8.0 / math.sqrt(12.5)]])


def test_plain_model_shows_every_mechanism():
    """A change to any mechanism of configuration A moves the logits of the plain model far beyond rounding."""
    cfg, w = U.plain_model("A")
    toks = U.tokens("A", 60, 0)
    want = U.plain_run(cfg, w, toks)
    for change in ("sink", "vmix", "norm1b", "magnitude", "bias", "rot", "scale"):
        c2, w2 = copy.deepcopy(cfg), dict(w)
        if change == "sink":
            w2["l1.mix.sink"] = w["l1.mix.sink"] - 30.0
        elif change == "vmix":
            w2["l5.mix.vmix"] = np.zeros(())
        elif change == "norm1b":
            w2["l2.norm1b"] = w["l2.norm1b"] - 1.0
        elif change == "magnitude":
            del c2["layers"][1]["mixer"]["rot"]["scaling"]
        elif change == "bias":
            w2["l1.mlp.up.b"] = 0 * w["l1.mlp.up.b"]
        elif change == "rot":
            c2["layers"][0]["mixer"]["rot"]["base"] = 30.0
        else:
            c2["layers"][3]["mixer"]["scale"] *= 1.5
        moved = U.row_distances(U.plain_run(c2, w2, toks), want)[1:]
        assert float(moved.median()) > 5e-3, (change, float(moved.median()))
