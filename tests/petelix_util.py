"""Small Petelix configurations for the tests, their model folders (random weights in a temporary folder), and helpers
that run the engine and the plain implementation (tests/plain_petelix.py) side by side.

The configurations differ from one another in every size: keys larger and smaller than values and of one size, that are and
are not multiples of 8 or 16; one key/value head and as many as query heads; rotations of a whole head, of a part, of two
elements and none; windows of one position, shorter and longer than a cache page, equal to one, and none; soft caps that bend
most scores, few and none; layers that read another layer's pages through a wider, a narrower and an equal window, two
readers of one layer; routers with many, one and no identity experts, with one group, all groups and none kept out, that
keep one expert, several and all; layers without experts."""
from __future__ import annotations

import functools
import json
import tempfile
from pathlib import Path

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, window, scale, cap=20.0, rot=None, base=10000.0, kv_from=None):
    m = dict(dim=dim, heads=heads, kv_heads=kv_heads, scale=scale, vdim=vdim)
    if window is not None:
        m["mask"] = dict(size=window)
    if rot:
        m["rot"] = dict(base=base, dims=rot)
    if cap is not None:
        m["softcap"] = cap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m)


def moe(ff, experts, top, identity=0, groups=None):
    router = dict(experts=experts, top=top)
    if groups:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    if identity:
        router["identity"] = identity
    return dict(expert=dict(ff=ff), kind="moe", router=router)


def layer(mix, mlp=None):
    return dict(mix, mlp=mlp)


def config(vocab, width, layers, eps=1e-5, emb=1.0):
    return dict(architecture="Petelix", embedding=dict(scale=emb), layers=layers, norm=dict(eps=eps), vocab=vocab, width=width)


# A: values larger than keys, three query heads a key/value head; a layer read twice, through a WIDER window and a narrower
# one (21, 50 and 7; pages of 16 divide none), with another cap and scale each; nine identity experts of fifteen, groups of
# three that mix both kinds; a layer without experts
CFG_A = config(211, 96, [
    layer(attention(6, 2, 24, 40, 21, 0.2, cap=3.0, rot=8, base=300.0), moe(40, 6, 4, 9, (5, 2))),
    layer(attention(4, 4, 10, 6, 33, 0.4, cap=8.0, rot=10, base=77.0), moe(24, 5, 3, 1, (3, 3))),
    layer(attention(2, 2, 24, 40, 50, 0.3, cap=1.5, rot=8, base=300.0, kv_from=0), moe(24, 4, 2, 2, (2, 1))),
    layer(attention(10, 2, 24, 40, 7, 0.15, cap=12.0, rot=8, base=300.0, kv_from=0)),
    layer(attention(3, 1, 16, 8, 64, 0.3, cap=5.0, rot=2), moe(16, 8, 8, 0, (4, 4))),
], emb=3.0)

# B: no window, a window of ONE position and one of a page; no cap; no rotation; no groups; one expert beside one identity
# expert; a router that keeps everything
CFG_B = config(300, 128, [
    layer(attention(4, 4, 16, 16, None, 0.3, cap=6.0, rot=16, base=500.0), moe(24, 4, 4, 3)),
    layer(attention(5, 1, 8, 32, 1, 0.35, cap=None), moe(56, 1, 1, 1)),
    layer(attention(4, 4, 16, 16, 16, 0.3, cap=50.0, rot=16, base=500.0, kv_from=0), moe(16, 3, 5, 2, (1, 1))),
    layer(attention(8, 2, 32, 16, 17, 0.15, cap=0.7, rot=12, base=1e6), moe(32, 2, 1, 14, (8, 3))),
], emb=0.6)

# C: sizes that are multiples of nothing: width 71, vocabulary 101, heads of 10, 7 and 9, seven experts of 9
CFG_C = config(101, 71, [
    layer(attention(3, 3, 10, 7, 16, 0.45, cap=4.0, rot=6, base=77.0), moe(9, 7, 3, 2, (3, 2))),
    layer(attention(3, 3, 10, 7, 15, 0.45, cap=2.0, rot=6, base=77.0, kv_from=0), moe(9, 5, 3, 2, (7, 4))),
    layer(attention(5, 1, 9, 5, 31, 0.4, cap=9.0, rot=4), moe(11, 3, 2, 3, (2, 2))),
], eps=1e-6, emb=1.7)

# M: small, and of the sizes the tensor-core kernels of the bfloat16 engine take, run with pages of 64: groups of heads that
# do and do not divide 128 rows, more than eight heads a key head, windows around a page, two readers
CFG_M = config(180, 128, [
    layer(attention(4, 2, 32, 48, 70, 0.2, cap=4.0, rot=16), moe(24, 6, 3, 2, (4, 2))),
    layer(attention(6, 2, 48, 16, 128, 0.2, cap=2.0, rot=48, base=500000.0), moe(32, 8, 3, 4, (2, 1))),
    layer(attention(8, 2, 32, 48, 33, 0.2, cap=15.0, rot=16, kv_from=0), moe(32, 8, 3)),
    layer(attention(12, 1, 64, 64, 64, 0.15, cap=6.0, rot=16), moe(40, 5, 2, 1)),
    layer(attention(2, 2, 32, 48, None, 0.2, cap=3.0, rot=16, kv_from=0)),
], emb=1.5)

# W: not tiny: the sizes at which the products and the experts' grouped products run on their tensor-core kernels
CFG_W = config(256, 1024, [
    layer(attention(16, 4, 128, 64, 100, 0.09, cap=30.0, rot=32), moe(512, 8, 3, 4, (4, 2))),
    layer(attention(16, 4, 128, 64, 1000, 0.09, cap=3.0, rot=32, kv_from=0), moe(256, 16, 4, 8, (6, 3))),
])

CONFIGS = {"A": (CFG_A, 51), "B": (CFG_B, 52), "C": (CFG_C, 53), "M": (CFG_M, 54), "W": (CFG_W, 55)}
PAGE_TOKENS = {"M": 64, "W": 64}          # (the other small configurations run with pages of 16)
_tmp = tempfile.TemporaryDirectory(prefix="fellm_b200_petelix_")

# random weights as the framework's random mode makes them, then some scaled so that no mechanism hides behind small
# numbers: experts whose outputs differ, gates away from one half (q and k are normed: their scale does not matter)
SCALES = ((".mlp.e", 5.0), (".mix.g", 8.0), (".mix.v", 4.0), (".mix.o", 4.0))


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
        if name.endswith(".correction"):
            # choice scores on both sides of zero, and far apart where the scores are small: fewer choices that rounding decides
            n = tensors[name].numel()
            order = np.random.default_rng(seed + n).permutation(n)
            tensors[name] = torch.from_numpy(0.2 - 0.9 * order / max(n, 10)).bfloat16()
    (folder / "config.json").write_text(json.dumps(typed.to_dict(), indent=1))
    write_safetensors(folder / "model.safetensors", tensors)
    return str(folder)


@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    cfg, seed = CONFIGS[name]
    return write_folder(Path(_tmp.name) / f"petelix_{name}", cfg, seed)


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
    rng = np.random.default_rng(8000 + seed)
    return [int(t) for t in rng.integers(0, cfg["vocab"], size=length)]


def plain_run(cfg, w, toks) -> torch.Tensor:
    import plain_petelix
    return torch.from_numpy(plain_petelix.run(cfg, w, toks))


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


LIMIT = {"float32": 2e-5, "bfloat16": 5e-2}
NOISE = {"M": 3.0, "W": 3.0}        # (sharp scores and experts on top of one another: rounding itself is that much larger)


def assert_close(got, want, dtype: str, times: float = 1.0, note=None):
    """In 32-bit every row is within the limit.  In bfloat16 a router's close call may go the other way for a token (its
    input is rounded), and experts that differ by design then move that row, and faintly the rows that read it, far beyond
    rounding: nine rows in ten are within the limit and the median row within a third of it, which no fault of a mechanism
    passes (a fault moves every row)."""
    assert got.shape == want.shape, (got.shape, want.shape)
    d = row_distances(got, want)
    limit = LIMIT[dtype] * times
    if dtype == "float32":
        assert float(d.max()) < limit, (note, float(d.max()), int(d.argmax()))
    else:
        assert float(torch.quantile(d, 0.9)) < limit and float(d.median()) < limit / 3, (note, float(torch.quantile(d, 0.9)), float(d.median()))


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
    """A configuration drawn at random: 1 to 6 layers, heads and sizes that are and are not multiples of anything, windows from
    1 to beyond the prompt or none, readers of earlier layers' pages, experts of any kind or none."""
    rng = np.random.default_rng(9300 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = int(pick([48, 72, 96, 120, 144]))
    layers, owners = [], []
    for i in range(int(rng.integers(1, 7))):
        cap = pick([None, 0.5, 2.0, 10.0, 50.0])
        if owners and rng.random() < 0.4:
            j = int(pick(owners))
            m = {k: v for k, v in layers[j]["mixer"].items() if k not in ("mask", "softcap")}
            m.update(kv_from=j, heads=m["kv_heads"] * int(pick([1, 2, 3])), scale=float(rng.uniform(0.05, 0.5)))
            window = pick([1, 5, 16, 17, 40, 100, None])
            if window is not None:
                m["mask"] = dict(size=window)
            if cap is not None:
                m["softcap"] = cap
            mix = dict(type="attention", mixer=m)
        else:
            G = int(pick([1, 2, 3]))
            dim = int(pick([4, 6, 8, 16, 24, 32, 48, 80]))
            vdim = int(pick([dim, 1, 3, 8, 16, 32, 48]))
            mix = attention(G * int(pick([1, 2, 4, 5])), G, dim, vdim, pick([1, 2, 15, 16, 17, 31, 64, 100, 1000, None]),
                            float(rng.uniform(0.05, 0.5)), cap=cap, rot=int(pick([0, 2, 4, dim, dim // 2 // 2 * 2])),
                            base=float(pick([10.0, 10000.0, 5e5])))
            owners.append(i)
        if rng.random() < 0.2:
            mlp = None
        else:
            per, count = int(pick([1, 2, 3, 4])), int(pick([1, 2, 3, 5]))
            n = per * count
            experts = int(rng.integers(1, n + 1))
            keep = int(rng.integers(1, count + 1))
            groups = (count, keep) if rng.random() < 0.8 else None
            mlp = moe(int(pick([8, 9, 16, 24, 40])), experts, int(rng.integers(1, (per * keep if groups else n) + 1)), n - experts, groups)
        layers.append(layer(mix, mlp))
    return config(int(pick([50, 101, 128, 200, 333])), width, layers, eps=float(pick([1e-5, 1e-6])), emb=float(rng.uniform(0.5, 8.0)))
