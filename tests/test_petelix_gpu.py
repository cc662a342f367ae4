"""Petelix on the GPU against the plain implementation (tests/plain_petelix.py).

First each mechanism alone, through its kernel's Python face with inputs made so that a fault shows (heads a thousand times
different in size under a norm over the whole row; a cache page that is not the next one; attention over pages that hold NaN
behind a request's end, with queries that point at the first and the last key of a window and at the key just outside it,
scores far beyond the soft cap, rows whose scores the sink outweighs; routers whose correction, whose groups and whose
negative choice scores decide); then whole models of four small configurations and a wide one: whole prompts, layer by
layer, prompts against token-by-token decoding, portions down to two tokens, unequal batches against each request alone,
pages and slots that are freed and come again, long decoding, a far key among hundreds at a window's edge, configurations
drawn at random, and greedy generation through the scheduler, the command line and the replay program."""
from __future__ import annotations

import copy
import json
import math
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import petelix_util as U
import plain_petelix as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


def _np(t):
    return t.detach().double().cpu().numpy()


@pytest.fixture(scope="module", autouse=True)
def kernels():
    """The attention libraries of every (key, value) size below, built side by side."""
    from fellm_b200 import ops
    from fellm_b200.csrc import jit
    sizes = [(128, 80), (128, 64), (48, 96), (80, 16), (64, 48), (64, 32), (256, 32), (32, 48), (48, 16), (64, 64), (32, 16)]
    mods = [("attention_mma", ops._mma_defines(hd, vd, True, True)) for hd, vd in sizes]
    mods += [("attention_umma", ops._umma_defines(hd, vd, True)) for hd, vd in sizes if ops.umma_prefill_takes(4, 2, hd, vd, 64, 9, 1.0, True)]
    jit.compile_many(mods + [(name, None) for name in ("attention_simt", "qk_rope_write", "moe", "sublayer")])


# ----------------------------------------------------------------------------- mechanisms alone

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,hd,vd,rot,pairing,page", [
    (6, 2, 24, 40, 8, "adjacent", 16), (8, 1, 128, 80, 128, "adjacent", 64), (4, 4, 48, 16, 16, "split_half", 64), (3, 3, 9, 5, 4, "adjacent", 16),
    (5, 1, 10, 7, 10, "split_half", 16), (16, 4, 128, 64, 32, "adjacent", 64), (2, 1, 16, 8, 0, "adjacent", 16), (6, 0, 24, 40, 12, "adjacent", 16),
    (7, 0, 64, 32, 16, "adjacent", 64), (64, 8, 128, 128, 64, "adjacent", 64), (1, 1, 2, 1, 2, "adjacent", 16)])
def test_norm_over_the_whole_projection_rotation_and_the_cache_write(dtype, H, G, hd, vd, rot, pairing, page):
    from fellm_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + hd)
    T, ld = 5, (H * hd + G * (hd + vd) + 7) // 8 * 8 + 16
    rows = torch.randn(T, ld, generator=g)
    sizes = 10.0 ** torch.linspace(-1.5, 1.5, H + G)                     # heads of very different size: the norm is not per head
    rows[:, :(H + G) * hd] *= sizes.repeat_interleave(hd)
    rows = rows.to(dtype)
    q_w, k_w = torch.rand(H * hd, generator=g) + 0.5, torch.rand(max(G, 1) * hd, generator=g) + 0.5
    eps = 0.25                                                          # inside the root, large enough to show
    positions, slots = [0, 5, page - 1, page, 2 * page + 3], [1, 0, 1, 0, 1]
    table = torch.tensor([[4, 2, 0], [5, 1, 3]], dtype=torch.int32)
    layer = 1
    pool = torch.full((6, 2, max(G, 1) * page * (hd + vd)), 7.0, dtype=dtype, device=DEV)
    freq = torch.from_numpy(P.rotary_frequencies(rot, 500.0)).float() if rot else None
    cache = SimpleNamespace(pool=pool, block_table=table.to(DEV), layer=layer, page_tokens=page)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = rows.to(DEV)
    args = (H, G, hd, vd, q_w.to(DEV), k_w.to(DEV) if G else None, eps, rot, freq.to(DEV) if rot else None, pairing)
    ops.qkv_norm_rotate_write(dev, *args, _i32(positions), _i32(slots), cache, status=status)
    assert int(status.item()) == 0
    r = _np(rows)

    def turned(x):
        if not rot:
            return x
        if pairing == "adjacent":
            return P.rotate(x, positions, freq.numpy())
        half = rot // 2
        order = [e for i in range(half) for e in (i, i + half)] + list(range(rot, hd))
        out = np.empty_like(x)
        out[..., order] = P.rotate(x[..., order], positions, freq.numpy())
        return out
    q = turned(P.norm(r[:, :H * hd], _np(q_w), eps).reshape(T, H, hd))
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    got = _np(dev)
    close = lambda a, b: np.all(np.abs(a - b) <= tol * (np.abs(b) + (1e-2 if dtype == torch.float32 else 2e-2)))
    assert close(got[:, :H * hd].reshape(T, H, hd), q)
    assert np.array_equal(got[:, H * hd:], r[:, H * hd:])
    want = np.full((6, 2, max(G, 1) * page * (hd + vd)), 7.0)
    if G:
        k = turned(P.norm(r[:, H * hd:(H + G) * hd], _np(k_w), eps).reshape(T, G, hd))
        v = r[:, (H + G) * hd:(H + G) * hd + G * vd].reshape(T, G, vd)
        for t in range(T):
            rec = want[table[slots[t], positions[t] // page], layer]
            at = positions[t] % page
            rec[:G * page * hd].reshape(G, page, hd)[:, at] = k[t]
            rec[G * page * hd:].reshape(G, page, vd)[:, at] = v[t]
    assert close(_np(pool), want) and np.array_equal(_np(pool)[want == 7.0], want[want == 7.0])
    if G:                                                               # a position without a page: recorded, nothing written
        before = pool.clone()
        bad = cache.block_table.clone()
        bad[:] = -1
        ops.qkv_norm_rotate_write(rows.to(DEV), *args, _i32(positions), _i32(slots),
                                  SimpleNamespace(pool=pool, block_table=bad, layer=layer, page_tokens=page), status=status)
        assert int(status.item()) == 2 and torch.equal(before, pool)


def _attention_case(H, G, hd, vd, page, T, window, seed):
    """Two requests of T tokens: bfloat16 keys, values and queries, pages in a random order and interleaved (NaN behind the
    requests' ends), query i pointing hard at ONE key: its own, the first of its window, the one just in front of that, a
    page's first or last, the first of all."""
    g = torch.Generator().manual_seed(seed)
    k, v = torch.randn(2, T, G, hd, generator=g).bfloat16(), torch.randn(2, T, G, vd, generator=g).bfloat16()
    q = torch.randn(2, T, H, hd, generator=g)
    R, w = H // G, window or T
    for r in range(2):
        for i in range(T):
            for h in range(i % 3, H, 3):
                j = [i, i - w + 1, i - w, i // page * page, i // page * page - 1, 0, i - w // 2][(i + h) % 7]
                q[r, i, h] = k[r, max(j, 0), h // R].float() * 1.3
    q = q.bfloat16()
    n_pages = -(-T // page)
    perm = torch.randperm(2 * n_pages + 2, generator=g)[:2 * n_pages].view(2, n_pages)
    pool = torch.full((2 * n_pages + 2, 1, G * page * (hd + vd)), float("nan"), dtype=torch.bfloat16)
    for r in range(2):
        for p in range(n_pages):
            n = min(page, T - p * page)
            rec = pool[perm[r, p], 0]
            rec[:G * page * hd].view(G, page, hd)[:, :n] = k[r, p * page:p * page + n].transpose(0, 1)
            rec[G * page * hd:].view(G, page, vd)[:, :n] = v[r, p * page:p * page + n].transpose(0, 1)
    return q, k, v, pool.to(DEV), perm.to(torch.int32).to(DEV), torch.randn(2, T, H * vd, generator=g).bfloat16() * 2.0


@pytest.mark.parametrize("cap", [2.0, 25.0, None])
@pytest.mark.parametrize("H,G,hd,vd,page,T,window", [
    (8, 1, 128, 80, 64, 300, 70), (16, 4, 128, 64, 64, 270, 128), (4, 4, 48, 96, 64, 150, 1), (8, 2, 80, 16, 64, 200, None),
    (2, 1, 128, 80, 64, 330, 65), (32, 1, 64, 48, 64, 100, 31), (6, 2, 64, 48, 64, 200, 64), (4, 2, 64, 32, 16, 130, 33),
    (3, 1, 256, 32, 64, 100, 50), (4, 1, 24, 40, 16, 90, 17), (2, 2, 7, 5, 16, 70, 16), (12, 3, 64, 32, 64, 400, 150)])
def test_attention_with_window_cap_sink_and_gate_over_written_pages(H, G, hd, vd, page, T, window, cap):
    """Portions that start and end in front of, on and behind the edges of pages, of windows and of the kernels' blocks,
    single tokens alone (the key walk split over CTAs) and beside portions, of two requests in one step: tcgen05 where the
    sizes allow, mma.sync, the split decode and the CUDA-core kernel, in bfloat16; and the CUDA-core kernel in float32,
    sharp.  The same float64 attention over the same bfloat16 numbers is the yardstick.  Pages that lie wholly in front of
    every window a step asks for hold NaN, as pages that were given away may."""
    from fellm_b200 import ops
    q, k, v, pool, table, gate = _attention_case(H, G, hd, vd, page, T, window, H * 1000 + hd)
    scale = 3.0 / math.sqrt(hd)
    want = [torch.from_numpy(P.attend(_np(q[r]), _np(k[r]), _np(v[r]), scale, cap, window).reshape(T, H * vd) * P.sigmoid(_np(gate[r])))
            for r in range(2)]
    g_off = (H * hd + 7) // 8 * 8
    flat = torch.zeros(2, T, g_off + (H * vd + 7) // 8 * 8, dtype=torch.bfloat16, device=DEV)
    flat[:, :, :H * hd] = q.view(2, T, H * hd).to(DEV)
    flat[:, :, g_off:g_off + H * vd] = gate.to(DEV)
    zero = torch.zeros(H, device=DEV)

    def run(items, x):
        n_rows = [n for _, _, n in items]
        ctx = SimpleNamespace(positions=_i32([i for r, a, n in items for i in range(a, a + n)]), row_slot=_i32([r for r, a, n in items for _ in range(n)]),
                              item_start=_i32([0] + list(np.cumsum(n_rows))), n_items=len(items), max_item_rows=max(n_rows),
                              max_len=max(a + n for _, a, n in items), all_single=max(n_rows) == 1)
        p = pool.clone()
        if window:
            for r in range(2):
                first = min([a for s, a, _ in items if s == r], default=0) - window + 1
                for i in range(max(first, 0) // page):
                    p[table[r, i].item()] = float("nan")
        if x.dtype == torch.float32:
            p = torch.nan_to_num(p.float(), nan=1e4)
        cache = SimpleNamespace(pool=p, block_table=table, layer=0, page_tokens=page)
        rows = torch.cat([x[r, a:a + n] for r, a, n in items])
        return ops.attention_written(rows, H, G, hd, vd, cache, ctx, scale, window=window, softcap=cap, sinks=zero,
                                     gate=rows[:, g_off:g_off + H * vd], ext=True)

    steps, at = [], 0
    for n in [1, 2, 29, 1, 31, 1, 64, 3, 66, 2, T]:
        n = min(n, T - at)
        if n <= 0:
            break
        steps.append([(0, at, n), (1, at, n)] if n > 2 else [(1, at, n), (0, at, n)])
        at += n
    steps += [[(0, T - 1, 1), (1, 5, 9)], [(0, T - 1, 1)], [(1, T // 2, 1), (0, T - 3, 1)], [(0, 0, T)], [(1, 3, T - 7), (0, 60, 2)]]
    for items in steps:
        ref = torch.cat([want[r][a:a + n] for r, a, n in items])
        top = max(1.0, float(ref.abs().max()))
        got = run(items, flat).double().cpu()
        assert torch.isfinite(got).all(), items
        assert float((got - ref).abs().max()) < 2e-2 * top, (items, float((got - ref).abs().max()))
        got = run(items, flat.float()).double().cpu()
        assert float((got - ref).abs().max()) < 2e-5 * top, (items, float((got - ref).abs().max()))
    ops.check_umma_status(DEV)


@pytest.mark.parametrize("H,G,hd,vd,rot,pairing,window,cap,own", [
    (8, 1, 128, 80, 64, "adjacent", 100, 5.0, True), (16, 4, 128, 64, 32, "adjacent", 1000, 30.0, True), (4, 4, 48, 96, 0, "adjacent", 64, 2.0, True),
    (16, 1, 80, 16, 2, "adjacent", None, 9.0, True), (12, 1, 128, 80, 128, "split_half", 1, 20.0, True), (4, 2, 80, 16, 48, "adjacent", 65, None, True),
    (6, 2, 48, 96, 16, "split_half", 600, 1.0, True), (12, 3, 64, 32, 24, "adjacent", 150, 40.0, False), (10, 1, 64, 48, 64, "adjacent", 31, 4.0, False),
    (8, 2, 128, 64, 32, "adjacent", None, 7.0, False)])
@pytest.mark.parametrize("ranges,stages,cluster", [(8, 0, True), (8, 2, False), (40, 4, False), (1, 0, True)])
def test_decode_from_the_input_products_rows(monkeypatch, H, G, hd, vd, rot, pairing, window, cap, own, ranges, stages, cluster):
    """The one-kernel decode step against the two-kernel one (norm, rotation and cache write, then attention): contexts of
    1 token, of a page less, exactly and one more, of windows and of many pages, in every way of splitting the key walk and
    merging the ranges; pages hold NaN behind the requests' ends and in front of their windows; what is written into the pages
    is the same up to the last bit of a bfloat16 (nothing, where the layer reads another's)."""
    from fellm_b200 import ops
    for name, val in (("WIDE_MAX_RANGES", ranges), ("WIDE_STAGES", stages), ("WIDE_CLUSTER", cluster)):
        monkeypatch.setattr(ops, name, val)
    page = 64
    g = torch.Generator().manual_seed(H * 7 + hd)
    lens = [1, 64, 65, 2, 700, 129, 1500, 128]
    T = len(lens)
    n_pages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(n_pages) + 1, generator=g)
    table = torch.full((T, max(n_pages)), -1, dtype=torch.int32)
    pool = torch.full((sum(n_pages) + 1, 2, G * page * (hd + vd)), float("nan"), dtype=torch.bfloat16)
    at = 0
    for r in range(T):
        table[r, :n_pages[r]] = perm[at:at + n_pages[r]].to(torch.int32)
        at += n_pages[r]
        for p in range(n_pages[r]):
            n = min(page, lens[r] - (0 if not own else 1) - p * page)
            if window and (p + 1) * page <= lens[r] - window:
                continue                                               # wholly in front of the window: given away
            rec = pool[table[r, p], 1]
            if n > 0:
                rec[:G * page * hd].view(G, page, hd)[:, :n] = torch.randn(G, n, hd, generator=g).bfloat16()
                rec[G * page * hd:].view(G, page, vd)[:, :n] = torch.randn(G, n, vd, generator=g).bfloat16()
    kv = G * (hd + vd) if own else 0
    g_off = (H * hd + kv + 7) // 8 * 8
    rows = (torch.randn(T, g_off + H * vd + 8 - (H * vd) % 8, generator=g) * 3.0).bfloat16().to(DEV)
    freq = torch.from_numpy(P.rotary_frequencies(rot, 500.0)).float().to(DEV) if rot else None
    q_w = ((torch.rand(H * hd, generator=g) + 0.5) * 2.0).to(DEV)
    k_w = (torch.rand(G * hd, generator=g) + 0.5).to(DEV) if own else None
    ctx = SimpleNamespace(positions=_i32([n - 1 for n in lens]), row_slot=_i32(list(range(T))), max_len=max(lens), all_single=True,
                          item_start=_i32(list(range(T + 1))), n_items=T, max_item_rows=1)
    scale, zero = 2.0 / math.sqrt(hd), torch.zeros(H, device=DEV)
    kw = dict(window=window, softcap=cap, sinks=zero, gate=rows[:, g_off:g_off + H * vd], ext=True)
    pool_a, pool_b = pool.to(DEV), pool.to(DEV)
    cache = lambda p: SimpleNamespace(pool=p, block_table=table.to(DEV), layer=1, page_tokens=page)
    assert ops.decode_wide_takes(rows, H, G, hd, vd, page, pool_a)
    before = rows.clone()
    got = ops.attention_decode_wide(rows, H, G, hd, vd, cache(pool_a), ctx, scale, rot_dim=rot, inv_freq=freq, pairing=pairing, q_w=q_w,
                                    k_w=k_w, eps=1e-2, reads_only=not own, **kw)
    ops.check_umma_status(DEV)
    assert torch.equal(rows, before)
    ops.qkv_norm_rotate_write(rows, H, G if own else 0, hd, vd, q_w, k_w, 1e-2, rot, freq, pairing, ctx.positions, ctx.row_slot, cache(pool_b))
    want = ops.attention_written(rows, H, G, hd, vd, cache(pool_b), ctx, scale, **kw)
    a, b = torch.nan_to_num(pool_a.float(), nan=9e9), torch.nan_to_num(pool_b.float(), nan=9e9)
    assert float(((a - b).abs() / (b.abs() + 1e-3)).max()) < 1e-2, "pages"
    assert own or torch.equal(a, torch.nan_to_num(pool.to(DEV).float(), nan=9e9))
    assert torch.isfinite(got).all()
    assert float((got.float() - want.float()).abs().max()) < 2e-2 * max(1.0, float(want.float().abs().max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [37, 301])                 # (a block a token, a warp a token)
@pytest.mark.parametrize("K,E,ident,top,count,keep", [(96, 6, 9, 4, 5, 2), (71, 7, 2, 3, 3, 2), (128, 1, 1, 1, 1, 1), (64, 2, 14, 1, 8, 3),
                                                      (256, 40, 24, 16, 16, 5), (40, 3, 0, 3, 3, 3), (1024, 96, 160, 8, 8, 4)])
def test_router_choice(dtype, T, K, E, ident, top, count, keep):
    """Softmax scores over experts and identity experts, the choice by score + correction (all choice scores negative; in every
    second case the correction outweighs the scores) inside the best groups, the weights the plain scores."""
    from fellm_b200 import ops
    g = torch.Generator().manual_seed(K + E)
    n = E + ident
    h = torch.randn(T, K, generator=g).to(dtype)
    wr = (torch.randn(n, K, generator=g) * (2.0 / math.sqrt(K))).to(dtype)
    corr = -1.0 - torch.rand(n, generator=g) * (0.7 if K % 3 else 0.02)
    idx, w = ops.moe_router(h.to(DEV), wr.to(DEV), top, correction=corr.to(DEV), groups=(count, keep, 1))
    z = _np(h) @ _np(wr).T
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    for t in range(T):
        chosen = P.choose(s[t], _np(corr), top, count, keep)
        c = np.sort(s[t] + _np(corr))
        if np.diff(c).min() > 1e-6:                       # no close call
            assert idx[t].tolist() == chosen, t
        assert np.allclose(_np(w[t]), s[t][idx[t].tolist()], rtol=2e-5, atol=1e-9)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,ff,E,ident,top,groups", [(96, 40, 6, 9, 4, (5, 2)), (72, 9, 7, 2, 3, (3, 2)), (128, 64, 1, 1, 1, None), (256, 128, 4, 4, 2, (4, 2)),
                                                     (64, 24, 2, 14, 5, (4, 3)), (37, 11, 3, 2, 2, None)])
@pytest.mark.parametrize("T", [1, 3, 40, 300, 700])
def test_experts_and_identity_experts(dtype, d, ff, E, ident, top, groups, T):
    """The part on every path of its products (a warp a column, mma.sync, tcgen05, CUDA cores), steps in which some tokens have
    identity experts alone and some none, added into a stream and stored; more than a thousand pairs."""
    from fellm_b200.parts.base import build_part
    from fellm_b200.parts.spec import PartSpec
    g = torch.Generator().manual_seed(d + T)
    part = build_part("feed_forward", PartSpec.make("moe", size=d, ff=ff, experts=E, identity=ident, top=top, score="softmax", correction=True,
                                                    groups=None if groups is None else (*groups, 1)), dtype)
    dt = getattr(torch, dtype)
    w = {}
    for name, decl in part.decls.items():
        t = torch.randn(decl.shape, generator=g) * (0.3 if name == "correction" else 1.5 / math.sqrt(decl.shape[-1]))
        w[name] = t.bfloat16()
    part.bind({n: t.to(DEV, torch.float32 if n == "correction" else dt) for n, t in w.items()})
    h = torch.randn(T, d, generator=g).bfloat16()
    x = torch.randn(T, d, generator=g)
    cfg = dict(router=dict(experts=E, identity=ident, top=top, groups=None if groups is None else dict(count=groups[0], keep=groups[1])))
    plain = {n.replace(".weight", ""): _np(t) for n, t in w.items()}
    want = P.experts(_np(h), plain, "", cfg)
    out = x.to(DEV).clone()
    part.forward(h.to(DEV, dt), None, out)
    err = np.abs(_np(out) - _np(x) - want).max(-1) / np.abs(want).max()
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert np.quantile(err, 0.99) < tol, (np.quantile(err, 0.99), err.max())           # (a close call of the choice may differ)
    stored = part.forward(h.to(DEV, dt), None, torch.full((T, d), float("nan"), device=DEV), store=True)
    assert float((stored - (out - x.to(DEV))).abs().max()) < 1e-4


def test_the_sink_counts_once_and_unscaled():
    """One key with score s: its weight is exp(s) / (1 + exp(s)), whatever the scale; a capped score enters as it is capped."""
    from fellm_b200 import ops
    H, hd, vd, page = 4, 32, 16, 64
    for dtype in (torch.float32, torch.bfloat16):
        pool = torch.zeros(1, 1, page * (hd + vd), dtype=dtype, device=DEV)
        pool[0, 0, 0] = 1.0                                        # key 0: the first unit vector
        pool[0, 0, page * hd:page * hd + vd] = 1.0                 # its value: ones
        q = torch.zeros(1, H * hd + 8, dtype=dtype, device=DEV)
        q[0, :H * hd:hd] = torch.tensor([0.0, 2.0, -3.0, 40.0], dtype=dtype)
        ctx = SimpleNamespace(positions=_i32([0]), row_slot=_i32([0]), item_start=_i32([0, 1]), n_items=1, max_item_rows=1, max_len=1, all_single=True)
        cache = SimpleNamespace(pool=pool, block_table=_i32([[0]]), layer=0, page_tokens=page)
        for single in (True, False):
            ctx.all_single = single
            got = ops.attention_written(q, H, 1, hd, vd, cache, ctx, 0.5, window=5, softcap=3.0, sinks=torch.zeros(H, device=DEV), ext=True)
            s = 3.0 * np.tanh(np.array([0.0, 1.0, -1.5, 20.0]) / 3.0)
            want = (1.0 / (1.0 + np.exp(-s)))[:, None].repeat(vd, 1)
            assert np.abs(_np(got).reshape(H, vd) - want).max() < (1e-5 if dtype == torch.float32 else 4e-3)


# ----------------------------------------------------------------------------- whole models

@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def engines(request):
    made = {}

    def get(name, **opts):
        key = (name, tuple(sorted(opts.items())))
        if key not in made:
            made[key] = U.make_engine(name, request.param, **opts)
        return made[key]
    get.dtype = request.param
    yield get
    made.clear()


@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_whole_prompt(engines, name):
    T = 150
    got = U.run_cuts(engines(name), "a", U.tokens(name, T, 0), [T])
    U.assert_close(got, U.plain_logits(name, T, 0), engines.dtype, U.NOISE.get(name, 1.0))


@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_layers_one_by_one(engines, name):
    cfg, w = U.plain_model(name)
    toks = U.tokens(name, 40, 1)
    want = torch.from_numpy(np.stack(P.streams(cfg, w, toks)))              # [layers, tokens, width]
    eng = engines(name)
    kept = []
    eng.model.after_run = lambda n, x: kept.append(x.clone())
    try:
        U.run_cuts(eng, "a", toks, [40])
    finally:
        eng.model.after_run = None
    got = torch.stack(kept).double().cpu()
    assert got.shape == want.shape
    for i in range(got.shape[0]):
        rows = (got[i] - want[i]).abs().amax(-1) / want[i].abs().max()
        err = float(rows.max() if engines.dtype == "float32" else torch.quantile(rows, 0.9))      # (a router's close call moves a row)
        assert err < U.LIMIT[engines.dtype] * U.NOISE.get(name, 1.0), (i, err)


@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_prompt_against_token_by_token(engines, name):
    T = 90
    eng = engines(name)
    toks = U.tokens(name, T, 2)
    whole = U.run_cuts(eng, "a", toks, [T])
    single = U.run_cuts(eng, "b", toks, [])
    U.assert_close(single, whole, engines.dtype, U.NOISE.get(name, 1.0))
    U.assert_close(single, U.plain_logits(name, T, 2), engines.dtype, U.NOISE.get(name, 1.0))


@pytest.mark.parametrize("name,cuts", [("A", [2, 2, 3, 17, 2, 21, 1, 1, 23, 2, 48]), ("B", [7, 2, 71, 2, 9, 64, 3]),
                                       ("C", [15, 2, 1, 16, 17, 2, 33]), ("M", [31, 2, 30, 1, 2, 63, 2, 7]), ("M", [64, 2, 69]),
                                       ("M", [2] * 40 + [3] * 20)])
def test_portions_of_many_sizes(engines, name, cuts):
    T = 170
    eng = engines(name)
    toks = U.tokens(name, T, 3)
    got = U.run_cuts(eng, "a", toks, cuts)
    U.assert_close(got, U.plain_logits(name, T, 3), engines.dtype, U.NOISE.get(name, 1.0))


@pytest.mark.parametrize("name", ["A", "C", "M"])
def test_unequal_batch_against_each_alone_with_slots_and_pages_that_come_again(engines, name):
    """Requests of different lengths share steps (portions beside single tokens), are left out of steps, end at different
    times and are followed by new ones in the slots and pages they gave back; the pool holds less than all of them."""
    from fellm_b200.engine import StepItem
    eng = engines(name, max_tokens=640 if name == "M" else 448)
    lengths = [97, 5, 140, 33, 61, 120, 2, 75]
    plans = {i: (U.tokens(name, n, 10 + i), [3, 1, 2, 40, 1, 1, 17, 2, 64][i % 3:]) for i, n in enumerate(lengths)}
    waiting, live, got = list(plans), {}, {i: [] for i in plans}
    step = 0
    while waiting or live:
        while waiting and len(live) < 4 and eng.cache.free_pages() * eng.cache.page_tokens >= lengths[waiting[0]] + 16 * len(live):
            i = waiting.pop(0)
            eng.add_request(i)
            live[i] = [0, list(plans[i][1])]
        items = []
        for i, st in live.items():
            if (step + i) % 5 == 4:
                continue                                    # left out of this step, goes on later
            n = min(st[1].pop(0) if st[1] else 1, len(plans[i][0]) - st[0])
            items.append((i, StepItem(i, plans[i][0][st[0]:st[0] + n], list(range(n)))))
            st[0] += n
        if items:
            lg = eng.step([it for _, it in items])
            at = 0
            for i, it in items:
                got[i].append(lg[at:at + len(it.tokens)].clone())
                at += len(it.tokens)
        for i in [i for i, st in live.items() if st[0] == len(plans[i][0])]:
            eng.release(i)
            del live[i]
        eng.cache.audit()
        step += 1
    eng.check_status()
    cfg, w = U.plain_model(name)
    alone = engines(name)
    for i in plans:
        U.assert_close(torch.cat(got[i]), U.plain_run(cfg, w, plans[i][0]), engines.dtype, U.NOISE.get(name, 1.0), note=i)
        if i in (1, 3):
            single = U.run_cuts(alone, f"alone{i}", plans[i][0], [len(plans[i][0])])
            U.assert_close(torch.cat(got[i]), single, engines.dtype, 0.2 if engines.dtype == "float32" else 1.0, note=i)


def test_logits_of_some_rows_only(engines):
    """A step whose wanted rows are not all rows takes the other way to the final norm; the logits are the same."""
    from fellm_b200.engine import StepItem
    eng = engines("M")
    toks = U.tokens("M", 100, 8)
    want = U.plain_logits("M", 100, 8)
    eng.add_request("a")
    eng.step([StepItem("a", toks[:70], [])])
    got = eng.step([StepItem("a", toks[70:], [0, 3, 29])])
    eng.release("a")
    U.assert_close(got, want[[70, 73, 99]], engines.dtype, U.NOISE["M"])


def test_wide_model(engines):
    """Width 1,024: the sizes at which the products and the experts run on their large tiles, attention of keys of 128 and values
    of 64 on tcgen05; portions, then token by token."""
    name, T = "W", 150
    got = U.run_cuts(engines(name), "a", U.tokens(name, T, 7), [140, 2, 5])
    U.assert_close(got, U.plain_logits(name, T, 7), engines.dtype, U.NOISE[name])


@pytest.mark.parametrize("cuts", [[170], [], [31, 2, 30, 1, 2, 63, 2, 7], [2] * 40 + [3] * 20])
def test_attention_alone_in_bfloat16(cuts):
    """The tensor-core configuration without experts: no router's close call hides a fault of the bfloat16 attention kernels (every
    row within rounding, under every cut, from graphs and without)."""
    cfg = copy.deepcopy(U.CFG_M)
    for L in cfg["layers"]:
        L["mlp"] = None
    folder = U.write_folder(Path(U._tmp.name) / "attention_alone", cfg, 56)
    _, w = U.load_folder(folder)
    toks = U.tokens("M", 170, 9)
    want = U.plain_run(cfg, w, toks)
    for graphs in (False, True):
        got = U.run_cuts(U.make_engine(folder, "bfloat16", page_tokens=64, cuda_graphs=graphs), "a", toks, cuts)
        assert float(U.row_distances(got, want).max()) < 2.5e-2


@pytest.mark.parametrize("name", ["A", "M"])
def test_long_decoding(engines, name):
    T = 420
    got = U.run_cuts(engines(name, max_tokens=512), "a", U.tokens(name, T, 5), [20])
    U.assert_close(got, U.plain_logits(name, T, 5), engines.dtype, U.NOISE.get(name, 1.0))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,page", [("wide", 64), ("wide", 16), ("narrow", 16), ("reader", 64), ("reader", 16)])
def test_a_far_key_at_the_windows_edge(dtype, kind, page):
    """Sharp scores.  A token's key is read from the first half of its embedding, its query from the second: the last tokens'
    query is made to find the token at position 3 among keys at random, with a window in which the last but one token still sees
    it and the last does not.  `reader`: the layer reads the pages of a layer whose own window is much narrower.  With
    another token in that place the last but one row is another one, and the last is not."""
    T, far = 604, 3
    window = T - 1 - far                      # the token at position T - 2 sees j >= far, the one at T - 1 does not
    hd, vd = (20, 12) if kind == "narrow" else (32, 16)
    layers = [U.layer(U.attention(2, 1, hd, vd, window, 2.0 / math.sqrt(hd), cap=30.0))]
    if kind == "reader":
        layers = [U.layer(U.attention(2, 1, hd, vd, 9, 0.2)), U.layer(U.attention(2, 1, hd, vd, window, 2.0 / math.sqrt(hd), cap=30.0, kv_from=0))]
    cfg = U.config(64, 64, layers)
    folder = U.write_folder(Path(U._tmp.name) / f"far_{kind}", cfg, 77, scales=())
    from fellm_b200.weights.safetensors_io import write_safetensors
    cfg, w = U.load_folder(folder)
    rng = np.random.default_rng(3)
    w["embed"] = rng.standard_normal(w["embed"].shape)
    w["embed"][63, 32:] = w["embed"][0, :32]
    read = rng.standard_normal((hd, 32))
    w["l0.mix.k"] = np.concatenate([read, 0 * read], 1)
    w["l0.mix.v"] = rng.standard_normal(w["l0.mix.v"].shape)
    for i in range(len(layers)):
        w[f"l{i}.mix.q"] = np.concatenate([np.concatenate([0 * read, read], 1)] * 2)
        w[f"l{i}.mix.q.norm"], w[f"l{i}.norm1"] = np.full(2 * hd, 1.5), np.ones(64)
        w[f"l{i}.mix.o"] = rng.standard_normal(w[f"l{i}.mix.o"].shape) * (0.02 if i + 1 < len(layers) else 1.0)
    w["l0.mix.k.norm"] = np.full(hd, 1.5)
    w = {n: torch.from_numpy(np.asarray(t)).bfloat16().double().numpy() for n, t in w.items()}
    write_safetensors(Path(folder) / "model.safetensors", {n: torch.from_numpy(np.asarray(t)).bfloat16() for n, t in w.items()})
    toks = [int(t) for t in rng.integers(1, 63, T - 2)] + [63, 63]
    toks[far] = 0
    want = U.plain_run(cfg, w, toks)
    eng = U.make_engine(folder, dtype, page_tokens=page, max_tokens=1024)
    for cuts in ([590, 9, 2], [T], [T - 1]):                            # the last tokens one by one, in a portion, one alone
        U.assert_close(U.run_cuts(eng, "a", toks, cuts)[-2:], want[-2:], dtype, 1.0 if dtype == "float32" else 0.5)
    other = list(toks)
    other[far] = 1
    moved = U.row_distances(U.plain_run(cfg, w, other)[-2:], want[-2:])
    assert float(moved[0]) > 0.1 and float(moved[1]) < 1e-3, moved


@pytest.mark.parametrize("seed", range(10))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_configurations_drawn_at_random(seed, dtype):
    """Ten models of random shape, each under three regimes: the whole prompt, portions down to two tokens followed by
    single tokens, and two unequal requests sharing every step."""
    from fellm_b200.engine import StepItem
    cfg = U.random_config(seed)
    folder = U.write_folder(Path(U._tmp.name) / f"random_{seed}", cfg, 500 + seed)
    _, w = U.load_folder(folder)
    eng = U.make_engine(folder, dtype, max_tokens=512, page_tokens=(16, 64)[seed % 2])
    rng = np.random.default_rng(seed)
    T = 75
    toks = [int(t) for t in rng.integers(0, cfg["vocab"], T)]
    other = [int(t) for t in rng.integers(0, cfg["vocab"], 41)]
    want, want_other = U.plain_run(cfg, w, toks), U.plain_run(cfg, w, other)
    U.assert_close(U.run_cuts(eng, "whole", toks, [T]), want, dtype, note=cfg)
    U.assert_close(U.run_cuts(eng, "cut", toks, [2, 17, 2, 3, 31]), want, dtype, note=cfg)
    eng.add_request("a")
    eng.add_request("b")
    got_a, got_b, at_a, at_b = [], [], 0, 0
    sizes_a, sizes_b = [5, 1, 30, 2], [1, 1, 16, 7, 2]
    while at_a < T or at_b < len(other):
        items = []
        na = min(sizes_a.pop(0) if sizes_a else 1, T - at_a)
        nb = min(sizes_b.pop(0) if sizes_b else 1, len(other) - at_b)
        if na > 0:
            items.append(StepItem("a", toks[at_a:at_a + na], list(range(na))))
        if nb > 0:
            items.append(StepItem("b", other[at_b:at_b + nb], list(range(nb))))
        lg = eng.step(items)
        if na > 0:
            got_a.append(lg[:na].clone())
        if nb > 0:
            got_b.append(lg[max(na, 0):max(na, 0) + nb].clone())
        at_a, at_b = at_a + max(na, 0), at_b + max(nb, 0)
    eng.check_status()
    U.assert_close(torch.cat(got_a), want, dtype, note=cfg)
    U.assert_close(torch.cat(got_b), want_other, dtype, note=cfg)


def _follows_greedily(cfg, w, prompt, got):
    seq = list(prompt)
    for k, t in enumerate(got):
        lg = U.plain_run(cfg, w, seq)[-1]
        top = torch.topk(lg, 2).values
        if int(lg.argmax()) != t:
            assert float(top[0] - top[1]) < 1e-4 * float(lg.abs().max()), (k, got, int(lg.argmax()))
            return
        seq.append(t)


@pytest.mark.parametrize("name", ["A", "B", "M"])
def test_greedy_generation_through_the_scheduler(name):
    """Engine.generate_batch (scheduler, sampler, CUDA graphs on) in float32 against the plain implementation's greedy
    continuation; prompts longer than a portion so that the scheduler cuts them."""
    from fellm_b200.engine import GenParams
    eng = U.make_engine(name, "float32", cuda_graphs=True, n_ubatch=32, n_batch=64, max_tokens=1024)
    cfg, w = U.plain_model(name)
    prompts = [U.tokens(name, n, 20 + i) for i, n in enumerate([70, 3, 41])]
    outs, stats = eng.generate_batch(prompts, GenParams.greedy(12))
    for p, got in zip(prompts, outs):
        assert len(got) == 12
        _follows_greedily(cfg, w, p, got)
    assert all(s is not None for s in stats)


def test_bfloat16_generation_with_graphs_is_the_direct_engines():
    """Decode steps replayed from CUDA graphs give the
    tokens of the engine that launches every step directly."""
    from fellm_b200.engine import GenParams
    outs = []
    for graphs in (True, False):
        eng = U.make_engine("M", "bfloat16", cuda_graphs=graphs, n_ubatch=16, n_batch=64)
        outs.append([list(o) for o in eng.generate_batch([U.tokens("M", 50, 30), U.tokens("M", 21, 31)], GenParams.greedy(24))[0]])
    assert outs[0] == outs[1] and all(len(o) == 24 for o in outs[0])


def test_command_line_runs_the_design(capsys):
    from fellm_b200 import cli
    folder = U.model_folder("A")
    assert cli.main(["inspect", "--model", folder]) == 0
    out = capsys.readouterr().out
    assert "architecture: Petelix" in out and "l0.mix.k.norm" in out and "l0.mlp.e5.down" in out and "l2.mix.k" not in out
    assert cli.main(["run", folder, "--prompt", "5 17 3 9 100", "--max-tokens", "6", "--temperature", "0", "--repetition-penalty", "1.0",
                     "--dtype", "float32", "--page-tokens", "16", "-c", "256", "--kv-device-budget", "4194304"]) == 0
    toks = [int(t) for t in capsys.readouterr().out.split()]
    cfg, w = U.plain_model("A")
    assert len(toks) == 6
    _follows_greedily(cfg, w, [5, 17, 3, 9, 100], toks)


def test_trace_replay_program(tmp_path):
    """bin/trace_run on a written folder: steps of portions beside single tokens, a request that ends and one that takes
    its slot; the logits it writes are the plain implementation's."""
    import subprocess
    import sys
    root = Path(__file__).resolve().parent.parent
    folder = U.model_folder("C")
    cfg, w = U.plain_model("C")
    a, b, c = U.tokens("C", 40, 40), U.tokens("C", 9, 41), U.tokens("C", 30, 42)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:33], want=[0, 32]), dict(id="b", tokens=b[:2], want=[])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[33:34], want=[0]), dict(id="b", tokens=b[2:], want=[6])], end=["b"]),
             dict(step=2, entries=[dict(id="c", tokens=c, want=[29])], end=[]),
             dict(step=3, entries=[dict(id="a", tokens=a[34:], want=[5])], end=["a", "c"])]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb, wc = U.plain_run(cfg, w, a), U.plain_run(cfg, w, b), U.plain_run(cfg, w, c)
    want = {0: torch.stack([wa[0], wa[32]]), 1: torch.stack([wa[33], wb[8]]), 2: wc[29:30], 3: wa[39:40]}
    for i, wt in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        assert float(U.row_distances(got, wt).max()) < U.LIMIT["float32"], i
