"""Small Vofezen configurations for the tests, their model folders (random weights in a temporary folder), and helpers
that run the engine and the plain implementation (tests/plain_vofezen.py) side by side.

The configurations differ from one another in every size: keys larger and smaller than values and of one size, that are and
are not multiples of 8 or 16; one key/value head and as many as query heads; rotations of a whole head, of a part, of two
elements and none, scaled and not; value mixing in every attention layer, in some, in one (which then has nothing to mix
with) and in none, with a latent layer in front of, between and behind them; latents of many sizes with the rotated part
rotated whole, in part and not at all; layers without a feed-forward."""
from __future__ import annotations

import functools
import json
import tempfile
from pathlib import Path

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, rot=None, base=10000.0, scaling=None, v_mix=False):
    m = dict(dim=dim, heads=heads, kv_heads=kv_heads, scale=scale, v_mix=v_mix, vdim=vdim)
    if rot:
        m["rot"] = _rot(rot, base, scaling)
    return dict(type="attention", mixer=m)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot=None, base=10000.0, scaling=None):
    m = dict(dim=dim, heads=heads, kv_rank=kv_rank, q_rank=q_rank, rot_dim=rot_dim, scale=scale, vdim=vdim)
    if rot:
        m["rot"] = _rot(rot, base, scaling)
    return dict(type="latent_attention", mixer=m)


def _rot(dims, base, scaling):
    r = dict(base=base, dims=dims)
    if scaling is not None:
        factor, original, fast, slow = scaling
        r["scaling"] = dict(factor=factor, fast=fast, original=original, slow=slow)
    return r


def dense(ff):
    return dict(ff=ff, kind="dense")


def layer(mix, mlp=None):
    return dict(mix, mlp=mlp)


def config(vocab, width, layers, eps=1e-5):
    return dict(architecture="Vofezen", layers=layers, norm=dict(eps=eps), vocab=vocab, width=width)


# A: a latent layer first; keys of 24 with values of 40; three heads a key/value head; two layers that mix behind the first,
# one attention layer between them that does not; a layer without a feed-forward
CFG_A = config(211, 96, [
    layer(latent(3, 20, 8, 12, 40, 56, 0.2, rot=8, base=300.0), dense(80)),
    layer(attention(6, 2, 24, 40, 0.2, rot=8, scaling=(4.0, 64, 8.0, 1.0), v_mix=True), dense(160)),
    layer(attention(3, 3, 10, 6, 0.3, rot=10, base=77.0), dense(40)),
    layer(attention(4, 4, 8, 20, 0.35, rot=4, base=500.0, v_mix=True)),
    layer(latent(5, 8, 4, 16, 24, 32, 0.3), dense(64)),
    layer(attention(8, 1, 12, 80, 0.25, v_mix=True), dense(96)),
])

# B: attention first and last, ONE mixing layer only; a rotation of the whole head, of two elements, and none; one key/value
# head and as many as heads; a latent layer that rotates part of its rotated elements, scaled
CFG_B = config(300, 128, [
    layer(attention(4, 4, 16, 16, 0.3, rot=16, base=500.0), dense(192)),
    layer(attention(5, 1, 9, 40, 0.35, rot=2, base=1e6, v_mix=True)),
    layer(latent(2, 64, 16, 24, 8, 64, 0.12, rot=12, base=5e5, scaling=(8.0, 256, 16.0, 2.0)), dense(64)),
    layer(attention(2, 2, 33, 7, 0.2), dense(256)),
], eps=1e-6)

# C: sizes that are multiples of nothing: width and vocabulary odd, heads of 5, 7 and 9, ranks of 3 and 11
CFG_C = config(97, 37, [
    layer(attention(3, 1, 7, 5, 0.4, rot=6, base=50.0, scaling=(2.0, 16, 4.0, 1.0), v_mix=True), dense(21)),
    layer(latent(3, 5, 3, 9, 3, 11, 0.4, rot=2, base=20.0), dense(13)),
    layer(attention(5, 5, 9, 1, 0.4, rot=4, base=50.0, v_mix=True), dense(50)),
], eps=1e-3)

# M: small, and of the sizes the tensor-core kernels of the bfloat16 engine take (multiples of 16), with pages of 64: keys
# larger and smaller than values, two atoms of 64 elements and one, a whole one and a part of one
CFG_M = config(180, 128, [
    layer(attention(8, 2, 80, 48, 0.11, rot=32, scaling=(4.0, 64, 8.0, 1.0), v_mix=True), dense(96)),
    layer(latent(4, 32, 16, 32, 48, 64, 0.15, rot=16, base=2000.0), dense(256)),
    layer(attention(2, 1, 48, 96, 0.15, rot=48, base=500000.0, v_mix=True), dense(128)),
    layer(attention(16, 1, 128, 96, 0.09, rot=64, v_mix=True)),
    layer(attention(3, 1, 64, 32, 0.12, rot=16, base=100.0)),           # three heads a kv head: portions on mma.sync
])

# W: not tiny: the sizes at which the products run on their large tiles
CFG_W = config(256, 1024, [
    layer(attention(16, 4, 128, 64, 0.088, rot=32, scaling=(8.0, 128, 32.0, 1.0), v_mix=True), dense(2048)),
    layer(latent(8, 64, 32, 64, 384, 256, 0.1, rot=32), dense(1536)),
    layer(attention(16, 4, 64, 64, 0.125, rot=64, v_mix=True), dense(2048)),
])

CONFIGS = {"A": (CFG_A, 61), "B": (CFG_B, 62), "C": (CFG_C, 63), "M": (CFG_M, 64), "W": (CFG_W, 65)}
PAGE_TOKENS = {"M": 64, "W": 64}          # (the other small configurations run with pages of 16)
_tmp = tempfile.TemporaryDirectory(prefix="fellm_b200_vofezen_")

# random weights as the framework's random mode makes them, then some scaled so that no mechanism hides behind small numbers
SCALES = ((".mix.q", 3.0), (".mix.k", 3.0), (".mix.uq", 3.0), (".mix.uk", 3.0), (".mlp.up", 4.0), (".mix.dkv", 2.0))


def write_folder(folder, cfg, seed, scales=SCALES):
    from fellm_b200.config.registry import config_from_dict
    from fellm_b200.models.model import build_model
    from fellm_b200.weights.random_init import random_tensors
    from fellm_b200.weights.safetensors_io import write_safetensors
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    arch, typed = config_from_dict(cfg)
    tensors = random_tensors(build_model(arch.build_spec(typed), "float32"), seed)
    for name in tensors:
        for pat, s in scales:
            if pat in name and tensors[name].dim() == 2:
                tensors[name] = (tensors[name].float() * s).bfloat16()
    (folder / "config.json").write_text(json.dumps(typed.to_dict(), indent=1))
    write_safetensors(folder / "model.safetensors", tensors)
    return str(folder)


@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    cfg, seed = CONFIGS[name]
    # (the wide model's queries and keys are large already: scaled up, single scores would decide every softmax, and a close
    # call between two of them would be the rounding's)
    return write_folder(Path(_tmp.name) / f"vofezen_{name}", cfg, seed, SCALES if name != "W" else ((".mlp.up", 2.0),))


def load_folder(folder):
    """(config dict, {name: float64 array}) read with the safetensors reader."""
    from fellm_b200.weights.safetensors_io import SafetensorsFile
    cfg = json.loads((Path(folder) / "config.json").read_text())
    f = SafetensorsFile(Path(folder) / "model.safetensors")
    w = {n: f.tensor(n).clone().double().numpy() for n in f.names()}
    f.close()
    return cfg, w


@functools.lru_cache(maxsize=None)
def plain_model(name: str):
    return load_folder(model_folder(name))


def tokens(name: str, length: int, seed: int):
    cfg, _ = CONFIGS[name]
    rng = np.random.default_rng(9000 + seed)
    return [int(t) for t in rng.integers(0, cfg["vocab"], size=length)]


def plain_run(cfg, w, toks) -> torch.Tensor:
    import plain_vofezen
    return torch.from_numpy(plain_vofezen.run(cfg, w, toks))


@functools.lru_cache(maxsize=None)
def plain_logits(name: str, length: int, seed: int) -> torch.Tensor:
    cfg, w = plain_model(name)
    return plain_run(cfg, w, tokens(name, length, seed))


def make_engine(name_or_folder: str, dtype: str, **opts):
    from fellm_b200.config.options import EngineOptions
    from fellm_b200.engine import Engine
    folder = model_folder(name_or_folder) if name_or_folder in CONFIGS else name_or_folder
    o = dict(dtype=dtype, n_ctx=1024, ctx_past_model=True, max_requests=4, max_tokens=2048,
             page_tokens=PAGE_TOKENS.get(name_or_folder, 16), cuda_graphs=False, n_batch=2048)
    o.update(opts)
    return Engine.open(folder, EngineOptions(**o))


def row_distances(got, want) -> torch.Tensor:
    """Row by row: the root mean square difference of the logits with their means taken off, relative to the root mean
    square of all the wanted logits."""
    got, want = got.double().cpu(), want.double().cpu()
    got = got - got.mean(-1, keepdim=True)
    want = want - want.mean(-1, keepdim=True)
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


# (bfloat16: models 37 to 128 wide that norm every sublayer's OUTPUT to full size do not average a product's rounding out;
# the float32 engine is the sharp comparison)
LIMIT = {"float32": 1e-4, "bfloat16": 5e-2}


def assert_close(got, want, dtype: str, times: float = 1.0, note=None):
    assert got.shape == want.shape, (got.shape, want.shape)
    d = row_distances(got, want)
    assert float(d.max()) < LIMIT[dtype] * times, (note, float(d.max()), int(d.argmax()), float(d.median()))


def run_cuts(engine, req, toks, cuts):
    """Feeds toks in portions of the given sizes (the rest one by one) and returns the logits of every position."""
    from fellm_b200.engine import StepItem
    engine.add_request(req)
    out, at = [], 0
    sizes = list(cuts)
    while at < len(toks):
        n = sizes.pop(0) if sizes else 1
        n = min(n, len(toks) - at)
        out.append(engine.step([StepItem(req, toks[at:at + n], list(range(n)))]).clone())
        at += n
    engine.check_status()
    engine.release(req)
    return torch.cat(out)


def random_config(seed: int):
    """A configuration drawn at random: 1 to 6 layers of either kind in any order, heads and sizes that are and are not
    multiples of anything, any rotation or none, mixing or not, a feed-forward or none."""
    rng = np.random.default_rng(9700 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = int(pick([40, 72, 96, 120, 144]))
    mixed = int(pick([12, 48, 96]))                     # key/value heads x values of the layers that mix
    layers = []
    for i in range(int(rng.integers(1, 7))):
        scaling = None
        if rng.random() < 0.6:
            scaling = (float(pick([2.0, 4.0, 8.0])), int(pick([16, 64, 512])), float(pick([4.0, 16.0, 32.0])), float(pick([0.5, 1.0, 2.0])))
        base = float(pick([10.0, 10000.0, 5e5]))
        if rng.random() < 0.4:
            rot_dim = int(pick([0, 4, 7, 16]))
            rot = int(pick([0, 2, rot_dim // 2 * 2])) if rot_dim else 0
            mix = latent(int(pick([1, 2, 3, 8])), int(pick([4, 9, 16, 32])), rot_dim, int(pick([3, 8, 16, 33])), int(pick([1, 8, 20, 64])),
                         int(pick([5, 16, 32, 64])), float(rng.uniform(0.1, 0.5)), rot=rot, base=base, scaling=scaling)
        else:
            G = int(pick([1, 2, 3, 4]))
            v_mix = bool(rng.random() < 0.6)
            dim = int(pick([4, 7, 16, 24, 32, 48, 64]))
            vdim = mixed // G if v_mix else int(pick([3, 8, 16, 40, 64]))
            mix = attention(G * int(pick([1, 2, 4, 5])), G, dim, vdim, float(rng.uniform(0.05, 0.5)),
                            rot=int(pick([0, 2, 4, dim // 2 * 2])), base=base, scaling=scaling, v_mix=v_mix)
        layers.append(layer(mix, None if rng.random() < 0.2 else dense(int(pick([8, 24, 40, 64, 100])))))
    return config(int(pick([50, 101, 128, 200, 333])), width, layers, eps=float(pick([1e-5, 1e-6])))
