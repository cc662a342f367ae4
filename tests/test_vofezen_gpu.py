"""Vofezen on the GPU against the plain implementation (tests/plain_vofezen.py).

First each mechanism alone, through its kernel's Python face with inputs made so that a fault shows (norms of rows of very
different size; a cache page that is not the next one, values mixed with rows of another stride; attention over pages that
hold NaN behind a request's end, with queries that point at one far key, sinks that outweigh most keys and scores that are
sharp; the squared relu on every path of a product); then whole models of four small configurations and a wide one: whole
prompts, layer by layer, prompts against token-by-token decoding, portions down to two tokens, unequal batches against each
request alone, pages and slots that are freed and come again, long decoding, a far key among hundreds, ten configurations
drawn at random, and greedy generation through the scheduler, the command line and the replay program."""
from __future__ import annotations

import json
import math
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_vofezen as P
import vofezen_util as U

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _i32(xs):
    return torch.tensor(xs, dtype=torch.int32, device=DEV)


def _np(t):
    return t.detach().double().cpu().numpy()


# ----------------------------------------------------------------------------- mechanisms alone

@pytest.mark.parametrize("T,d", [(1, 96), (5, 72), (40, 128), (3, 250), (2, 2048), (7, 6), (300, 1024), (2, 8192), (2, 9000), (1, 16400), (3, 37)])
def test_norm_into_the_stream_and_the_norm_that_follows(T, d):
    from fellm_b200 import ops
    g = torch.Generator().manual_seed(d)
    size = 10.0 ** torch.randint(-3, 4, (T, 1), generator=g)
    y, x = torch.randn(T, d, generator=g) * size, torch.randn(T, d, generator=g) * 3.0
    w, wn = torch.randn(d, generator=g), torch.randn(d, generator=g)
    new = _np(x) + P.norm(_np(y), _np(w) - 1.0, 1e-5)
    after = P.norm(new, _np(wn) - 1.0, 1e-3)
    for out_dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        xs = x.to(DEV).clone()
        h = ops.add_rmsnorm(xs, y.to(DEV), w.to(DEV), 1e-5, wn.to(DEV), 1e-3, out_dtype=out_dtype)
        assert np.abs(_np(xs) - new).max() < 1e-5 * np.abs(new).max()
        assert h.dtype == out_dtype and np.abs(_np(h) - after).max() < tol * np.abs(after).max()
    xs = x.to(DEV).clone()
    assert ops.add_rmsnorm(xs, y.to(DEV), w.to(DEV), 1e-5) is None
    assert np.abs(_np(xs) - new).max() < 1e-5 * np.abs(new).max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,hd,vd,rot,pairing,mix,page", [(6, 2, 24, 40, 8, "split_half", True, 16), (8, 1, 128, 80, 64, "split_half", True, 64),
                                                            (3, 3, 10, 6, 10, "split_half", False, 16), (5, 1, 7, 5, 2, "adjacent", True, 16),
                                                            (4, 4, 64, 64, 0, "split_half", True, 64), (2, 1, 48, 16, 48, "split_half", False, 64),
                                                            (2, 2, 96, 32, 80, "split_half", True, 16)])
def test_rotation_value_mixing_and_the_cache_write(dtype, H, G, hd, vd, rot, pairing, mix, page):
    """Two requests whose pages interleave, at positions up to 100,000; values mixed with rows of another stride; what lies
    in the pages beside the written rows stays as it was, and a row whose page is not mapped writes nothing and is reported."""
    from fellm_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + hd)
    positions, slots = [5, 6, 99999, 0, page - 1, page], [0, 0, 1, 2, 2, 2]
    T, width = len(positions), H * hd + G * (hd + vd)
    ld = (width + 7) // 8 * 8 + 8
    rows = torch.randn(T, ld, generator=g).to(dtype)
    first = torch.randn(T, G * vd + 16, generator=g).to(dtype)[:, 8:8 + G * vd]
    n_pages = 100000 // page + 1
    table = np.full((3, n_pages), -1, dtype=np.int32)
    table[0, 0], table[1, 99999 // page], table[2, 0], table[2, 1] = 3, 1, 4, 0
    if page == 16:
        assert table[0, 6 // page] == 3
    pool = torch.full((6, 2, G * page * (hd + vd)), 7.0, dtype=dtype, device=DEV)
    freq = torch.tensor([40.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32)
    mag, lam, layer = 1.2, 0.3, 1
    cache = SimpleNamespace(pool=pool, block_table=torch.from_numpy(table).to(DEV), layer=layer, page_tokens=page)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    dev = rows.to(DEV).clone()
    kw = dict(v_first=first.to(DEV), lam=torch.tensor(lam, device=DEV)) if mix else {}
    ops.qkv_rotate_write(dev, H, G, hd, vd, rot, freq.to(DEV) if rot else None, pairing, mag, _i32(positions), _i32(slots), cache,
                         status=status, **kw)
    assert int(status.item()) == 0
    r = _np(rows)
    q, k = r[:, :H * hd].reshape(T, H, hd), r[:, H * hd:(H + G) * hd].reshape(T, G, hd)
    v = r[:, (H + G) * hd:width].reshape(T, G, vd)

    def turned(x):
        if not rot:
            return x
        if pairing == "adjacent":
            order = [i for i in range(0, rot, 2)] + [i for i in range(1, rot, 2)] + list(range(rot, hd))
            y = P.rotate(x[..., order], positions, freq.numpy(), mag)
            out = np.empty_like(y)
            out[..., order] = y
            return out
        return P.rotate(x, positions, freq.numpy(), mag)
    want_v = P.mix_values(v, _np(first).reshape(T, G, vd), float(np.float32(lam))) if mix else v
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    got = _np(dev)
    assert np.abs(got[:, :H * hd].reshape(T, H, hd) - turned(q)).max() < tol * 5
    assert np.array_equal(got[:, H * hd:], r[:, H * hd:])
    want = np.full((6, 2, G * page * (hd + vd)), 7.0)
    kt = turned(k)
    for t in range(T):
        rec = want[table[slots[t], positions[t] // page], layer]
        at = positions[t] % page
        rec[:G * page * hd].reshape(G, page, hd)[:, at] = kt[t]
        rec[G * page * hd:].reshape(G, page, vd)[:, at] = want_v[t]
    assert np.abs(_np(pool) - want).max() < tol * 5
    # (elements behind the rotated part, and values that mix with nothing, are copies)
    if rot < hd or not mix:
        assert np.array_equal(_np(pool)[want == 7.0], want[want == 7.0])
    before = pool.clone()
    ops.qkv_rotate_write(rows.to(DEV).clone(), H, G, hd, vd, rot, freq.to(DEV) if rot else None, pairing, mag, _i32([page * 3] * T),
                         _i32(slots), cache, status=status, **kw)
    assert int(status.item()) == 2 and torch.equal(before, pool)


def _attention_case(H, G, hd, vd, page, T, seed):
    """Two requests of T tokens: bfloat16 keys, values and queries, pages in a random order and interleaved (NaN behind the
    requests' ends), query i pointing hard at ONE key: the first, a page's first or last, its own, or one far back."""
    g = torch.Generator().manual_seed(seed)
    k, v = torch.randn(2, T, G, hd, generator=g).bfloat16(), torch.randn(2, T, G, vd, generator=g).bfloat16()
    q = torch.randn(2, T, H, hd, generator=g)
    R = H // G
    for r in range(2):
        for i in range(T):
            h = (i * 5 + r) % H
            j = [0, i, max(i - 1, 0), i // page * page, max(i // page * page - 1, 0), int(i * 0.37), i // 2][(i // 3) % 7]
            q[r, i, h] = k[r, j, h // R].float() * 1.3
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
    return q, k, v, pool.to(DEV), perm.to(torch.int32).to(DEV), (torch.randn(H, generator=g) + 2.5)


@pytest.mark.parametrize("H,G,hd,vd,page,T", [
    (8, 1, 128, 80, 64, 300), (16, 4, 64, 64, 64, 270), (4, 4, 48, 96, 64, 150), (8, 2, 80, 16, 64, 200), (16, 1, 16, 128, 64, 140),
    (2, 1, 128, 128, 64, 200), (32, 1, 96, 112, 64, 100), (6, 2, 64, 48, 64, 200), (4, 2, 32, 64, 16, 130), (3, 1, 256, 32, 64, 100),
    (4, 1, 24, 40, 16, 90), (2, 2, 7, 5, 16, 70)])
def test_attention_with_sinks_over_written_pages(H, G, hd, vd, page, T):
    """Portions that start and end in front of, on and behind the edges of pages and of the kernels' blocks, single tokens
    alone (the key walk split over CTAs) and beside portions, of two requests in one step: tcgen05 where the sizes allow,
    mma.sync, the split decode and the CUDA-core kernel, in bfloat16; and the CUDA-core kernel in float32, sharp.  The same
    float64 attention over the same bfloat16 numbers is the yardstick."""
    from fellm_b200 import ops
    q, k, v, pool, table, sinks = _attention_case(H, G, hd, vd, page, T, H * 1000 + hd)
    scale = 3.0 / math.sqrt(hd)
    want = [torch.from_numpy(P.attend(_np(q[r]), _np(k[r]), _np(v[r]), scale, _np(sinks))) for r in range(2)]
    ld = (H * hd + 7) // 8 * 8 + 16
    flat = torch.zeros(2, T, ld, dtype=torch.bfloat16, device=DEV)
    flat[:, :, :H * hd] = q.view(2, T, H * hd).to(DEV)
    pool32 = torch.nan_to_num(pool.float(), nan=0.0)

    def run(items, p, x):
        n_rows = [n for _, _, n in items]
        ctx = SimpleNamespace(positions=_i32([i for r, a, n in items for i in range(a, a + n)]), row_slot=_i32([r for r, a, n in items for _ in range(n)]),
                              item_start=_i32([0] + list(np.cumsum(n_rows))), n_items=len(items), max_item_rows=max(n_rows),
                              max_len=max(a + n for _, a, n in items), all_single=max(n_rows) == 1)
        cache = SimpleNamespace(pool=p, block_table=table, layer=0, page_tokens=page)
        rows = torch.cat([x[r, a:a + n] for r, a, n in items])
        return ops.attention_written(rows, H, G, hd, vd, cache, ctx, scale, sinks=sinks.to(DEV))

    steps, at = [], 0
    for n in [1, 2, 29, 1, 31, 1, 64, 3, 66, 2, T]:
        n = min(n, T - at)
        if n <= 0:
            break
        steps.append([(0, at, n), (1, at, n)] if n > 2 else [(1, at, n), (0, at, n)])
        at += n
    steps += [[(0, T - 1, 1), (1, 5, 9)], [(0, T - 1, 1)], [(1, T // 2, 1), (0, T - 3, 1)], [(0, 0, T)], [(1, 3, T - 7), (0, 60, 2)]]
    for items in steps:
        ref = torch.cat([want[r][a:a + n] for r, a, n in items]).reshape(-1, H * vd)
        top = max(1.0, float(ref.abs().max()))
        got = run(items, pool, flat).double().cpu()
        assert torch.isfinite(got).all(), items
        assert float((got - ref).abs().max()) < 2e-2 * top, (items, float((got - ref).abs().max()))
        got = run(items, pool32, flat.float()).double().cpu()
        assert float((got - ref).abs().max()) < 2e-5 * top, (items, float((got - ref).abs().max()))
    ops.check_umma_status(DEV)


@pytest.mark.parametrize("H,G,hd,vd,rot,pairing,mix,window", [
    (8, 1, 128, 80, 64, "split_half", True, None), (16, 4, 64, 64, 64, "adjacent", True, None), (4, 4, 48, 96, 0, "split_half", False, None),
    (16, 1, 80, 16, 2, "split_half", True, None), (12, 1, 128, 128, 128, "split_half", False, None), (4, 2, 192, 32, 96, "split_half", True, None),
    (6, 2, 32, 176, 16, "adjacent", True, None), (8, 2, 64, 48, 32, "split_half", True, 100)])
@pytest.mark.parametrize("ranges,stages,cluster", [(8, 0, True), (8, 2, False), (40, 4, False), (1, 0, True)])
def test_decode_from_the_input_products_rows(monkeypatch, H, G, hd, vd, rot, pairing, mix, window, ranges, stages, cluster):
    """The one-kernel decode step against the two-kernel one (rotation, mixing and cache write, then attention): contexts of
    1 token, of a page less, exactly and one more, and of many pages, in every way of splitting the key walk and merging the
    ranges; pages of one request hold NaN behind its end; what is written into the pages is the same bits."""
    from fellm_b200 import ops
    for name, v in (("WIDE_MAX_RANGES", ranges), ("WIDE_STAGES", stages), ("WIDE_CLUSTER", cluster)):
        monkeypatch.setattr(ops, name, v)
    page = 64
    g = torch.Generator().manual_seed(H * 7 + hd)
    lens = [1, 64, 65, 2, 700, 129, 1500]
    T = len(lens)
    n_pages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(n_pages) + 1, generator=g)
    table = torch.full((T, max(n_pages)), -1, dtype=torch.int32)
    pool = torch.full((sum(n_pages) + 1, 2, G * page * (hd + vd)), float("nan"), dtype=torch.bfloat16)
    at = 0
    for r in range(T):
        for p in range(n_pages[r]):
            table[r, p] = perm[at]
            n = min(page, lens[r] - 1 - p * page)                     # (the last position is the step's own)
            rec = pool[perm[at], 1]
            if n > 0:
                rec[:G * page * hd].view(G, page, hd)[:, :n] = torch.randn(G, n, hd, generator=g).bfloat16()
                rec[G * page * hd:].view(G, page, vd)[:, :n] = torch.randn(G, n, vd, generator=g).bfloat16()
            at += 1
    width = H * hd + G * (hd + vd)
    rows = torch.randn(T, (width + 15) // 8 * 8, generator=g).bfloat16().to(DEV)
    first = torch.randn(T, G * vd + 8, generator=g).bfloat16().to(DEV)[:, 8:]
    freq = torch.tensor([40.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32).to(DEV) if rot else None
    sinks, lam = (torch.randn(H, generator=g) + 2.0).to(DEV), torch.tensor(0.3, device=DEV)
    scale = 2.0 / math.sqrt(hd)
    kw = dict(v_first=first, lam=lam) if mix else {}
    ctx = SimpleNamespace(positions=_i32([n - 1 for n in lens]), row_slot=_i32(list(range(T))), item_start=_i32(list(range(T + 1))), n_items=T,
                          max_item_rows=1, max_len=max(lens), all_single=True)
    a, b = (SimpleNamespace(pool=pool.to(DEV).clone(), block_table=table.to(DEV), layer=1, page_tokens=page) for _ in range(2))
    before = rows.clone()
    got = ops.attention_decode_wide(rows, H, G, hd, vd, a, ctx, scale, rot_dim=rot, inv_freq=freq, pairing=pairing, mag=1.1, window=window,
                                    sinks=sinks, **kw)
    assert torch.equal(rows, before)
    ops.qkv_rotate_write(rows, H, G, hd, vd, rot, freq, pairing, 1.1, ctx.positions, ctx.row_slot, b, **kw)
    assert torch.equal(torch.nan_to_num(a.pool.float(), nan=99.0), torch.nan_to_num(b.pool.float(), nan=99.0))
    b.pool = torch.nan_to_num(b.pool, nan=0.0)
    want = ops.paged_attention_general(rows.float(), H, hd, vd, b.pool.float(), b.block_table, ctx.positions, ctx.row_slot, 1, page, G, scale,
                                       window=window, warps=4, sinks=sinks)
    assert torch.isfinite(got).all() and float((got.float() - want).abs().max()) < 2e-2 * max(1.0, float(want.abs().max()))
    # a row whose page is not mapped is reported and writes nothing
    table[0, 0] = -1
    a.block_table, kept = table.to(DEV), a.pool.clone()
    one = SimpleNamespace(positions=_i32([0]), row_slot=_i32([0]), max_len=1, all_single=True)
    ops.attention_decode_wide(rows[:1], H, G, hd, vd, a, one, scale, rot_dim=rot, inv_freq=freq, pairing=pairing, mag=1.1, sinks=sinks,
                              **(dict(v_first=first[:1], lam=lam) if mix else {}))
    from fellm_b200.config.errors import KernelError
    with pytest.raises(KernelError):
        ops.check_umma_status(DEV)
    assert torch.equal(torch.nan_to_num(kept.float(), nan=99.0), torch.nan_to_num(a.pool.float(), nan=99.0))


def test_a_sink_counts_once_and_unscaled():
    """Keys that score zero: a row at position i gives each of its i + 1 keys the weight 1 / (i + 1 + exp(sink)), whatever
    the scale, in portions and decoding, on every kernel."""
    from fellm_b200 import ops
    H, G, page, T = 8, 2, 64, 200
    for hd, vd in ((64, 48), (128, 64), (48, 80), (20, 12)):
        n_pages = -(-T // page)
        pool = torch.zeros(n_pages, 1, G * page * (hd + vd), dtype=torch.bfloat16, device=DEV)
        pool[:, :, G * page * hd:] = 1.0
        table = _i32([list(range(n_pages))])
        sinks = torch.linspace(-3.0, 6.0, H).to(DEV)
        q = torch.randn(T, H * hd).bfloat16().to(DEV)
        for dtype in (torch.bfloat16, torch.float32):
            cache = SimpleNamespace(pool=pool.to(dtype), block_table=table, layer=0, page_tokens=page)
            for rows in (range(T), [T - 1], [0]):
                n = len(rows)
                ctx = SimpleNamespace(positions=_i32(list(rows)), row_slot=_i32([0] * n), item_start=_i32([0, n]), n_items=1, max_item_rows=n,
                                      max_len=rows[-1] + 1, all_single=n == 1)
                got = ops.attention_written(q[list(rows)].to(dtype).contiguous(), H, G, hd, vd, cache, ctx, 5.0, sinks=sinks).double().cpu().view(n, H, vd)
                count = torch.tensor([i + 1.0 for i in rows]).double()[:, None]
                want = count / (count + sinks.double().cpu().exp()[None])
                assert float((got - want[:, :, None]).abs().max()) < (1e-2 if dtype == torch.bfloat16 else 1e-5), (hd, vd, n)


@pytest.mark.parametrize("M,N,K", [(1, 256, 128), (8, 4096, 1024), (16, 96, 1536), (3, 40, 80), (5, 64, 16384), (24, 512, 256), (50, 1024, 512), (64, 80, 64),
                                   (100, 2048, 512), (128, 120, 96), (130, 64, 64), (200, 384, 2048), (300, 256, 512), (2048, 2048, 256), (700, 3000, 128)])
@pytest.mark.parametrize("with_bias", [True, False])
def test_squared_relu_behind_a_product(M, N, K, with_bias):
    """The up product's epilogue on every kernel gemm_bf16 picks from (weight-streaming, few rows, persistent, CTA pairs, K
    over two CTAs), on mma.sync tiles and in float32."""
    from fellm_b200 import ops
    g = torch.Generator().manual_seed(M + N + K)
    x, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) / math.sqrt(K)).bfloat16()
    b = torch.randn(N, generator=g) if with_bias else None
    z = x.double() @ w.double().T + (b.double() if with_bias else 0.0)
    want = z.clamp(min=0) ** 2
    bd = b.to(DEV) if with_bias else None
    got = ops.gemm_bf16(x.to(DEV), w.to(DEV), bd, act="relu2")
    top = float(want.max())
    assert got.dtype == torch.bfloat16 and float((got.double().cpu() - want).abs().max()) < 1e-2 * top
    got = ops.gemm_tiled(x.to(DEV), w.to(DEV), bd, out=torch.empty(M, N, dtype=torch.bfloat16, device=DEV), epi=6)
    assert float((got.double().cpu() - want).abs().max()) < 1e-2 * top
    got = ops.gemm_simt(x.float().to(DEV), w.float().to(DEV), bd, act="relu2")
    assert got.dtype == torch.float32 and float((got.double().cpu() - want).abs().max()) < 1e-5 * top
    ops.check_umma_status(DEV)


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
    U.assert_close(got, U.plain_logits(name, T, 0), engines.dtype)


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
        err = float((got[i] - want[i]).abs().max() / want[i].abs().max())
        assert err < U.LIMIT[engines.dtype], (i, err)


@pytest.mark.parametrize("name", ["A", "B", "C", "M"])
def test_prompt_against_token_by_token(engines, name):
    T = 90
    eng = engines(name)
    toks = U.tokens(name, T, 2)
    whole = U.run_cuts(eng, "a", toks, [T])
    single = U.run_cuts(eng, "b", toks, [])
    U.assert_close(single, whole, engines.dtype)
    U.assert_close(single, U.plain_logits(name, T, 2), engines.dtype)


@pytest.mark.parametrize("name,cuts", [("A", [2, 2, 3, 17, 2, 21, 1, 1, 23, 2, 48]), ("B", [7, 2, 71, 2, 9, 64, 3]),
                                       ("C", [15, 2, 1, 16, 17, 2, 33]), ("M", [31, 2, 30, 1, 2, 63, 2, 7]), ("M", [64, 2, 69]),
                                       ("M", [2] * 40 + [3] * 20)])
def test_portions_of_many_sizes(engines, name, cuts):
    T = 170
    eng = engines(name)
    toks = U.tokens(name, T, 3)
    got = U.run_cuts(eng, "a", toks, cuts)
    U.assert_close(got, U.plain_logits(name, T, 3), engines.dtype)


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
        U.assert_close(torch.cat(got[i]), U.plain_run(cfg, w, plans[i][0]), engines.dtype, note=i)
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
    U.assert_close(got, want[[70, 73, 99]], engines.dtype)


def test_wide_model(engines):
    """Width 1,024: the sizes at which the products run on their large tiles, attention of keys of 128 and values of 64 on
    tcgen05; portions, then token by token."""
    name, T = "W", 150
    got = U.run_cuts(engines(name), "a", U.tokens(name, T, 7), [140, 2, 5])
    U.assert_close(got, U.plain_logits(name, T, 7), engines.dtype)


@pytest.mark.parametrize("name", ["A", "M"])
def test_long_decoding(engines, name):
    T = 420
    got = U.run_cuts(engines(name, max_tokens=512), "a", U.tokens(name, T, 5), [20])
    U.assert_close(got, U.plain_logits(name, T, 5), engines.dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,page", [("attention", 64), ("attention", 16), ("latent", 64), ("narrow", 16)])
def test_a_far_key_among_hundreds(dtype, kind, page):
    """One layer with a sharp score.  A token's key is read from the first half of its embedding, its query from the second:
    the last token's query is made to find the token at position 3, 600 positions back, among keys at random.  With another
    token in that place the last row is another one."""
    if kind == "latent":
        mix = U.latent(2, 32, 16, 24, 32, 64, 0.5)
    else:
        mix = U.attention(2, 1, 32, 16, 0.35) if kind == "attention" else U.attention(2, 1, 20, 12, 0.55)
    cfg = U.config(64, 64, [U.layer(mix)])
    folder = U.write_folder(Path(U._tmp.name) / f"far_{kind}", cfg, 77, scales=())
    from fellm_b200.weights.safetensors_io import write_safetensors
    cfg, w = U.load_folder(folder)
    rng = np.random.default_rng(3)
    w["embed"] = rng.standard_normal(w["embed"].shape)
    w["embed"][63, 32:] = w["embed"][0, :32]
    w["l0.norm1"][:32] = w["l0.norm1"][32:]
    n = 32 if kind == "latent" else cfg["layers"][0]["mixer"]["dim"]
    read = rng.standard_normal((n, 32)) * 0.3
    key, query = np.concatenate([read, 0 * read], 1), np.concatenate([0 * read, read], 1)
    if kind == "latent":
        w["l0.mix.dkv"] *= 0.0
        w["l0.mix.dkv"][:32], w["l0.mix.dq"] = key, query
        w["l0.mix.dq.norm"][:], w["l0.mix.dkv.norm"][:] = 1.0, 1.0
        w["l0.mix.uq"], w["l0.mix.uk"] = np.zeros_like(w["l0.mix.uq"]), np.zeros_like(w["l0.mix.uk"])
        for h in range(2):
            w["l0.mix.uq"][48 * h:48 * h + 32] = np.eye(32)
            w["l0.mix.uk"][32 * h:32 * h + 32, :32] = np.eye(32)
        w["l0.mix.uv"] = rng.standard_normal(w["l0.mix.uv"].shape)
    else:
        w["l0.mix.k"], w["l0.mix.q"] = key, np.concatenate([query, query])
        w["l0.mix.v"] = rng.standard_normal(w["l0.mix.v"].shape)
    w["l0.mix.o"] = rng.standard_normal(w["l0.mix.o"].shape)
    w = {n: torch.from_numpy(np.asarray(t)).bfloat16().double().numpy() for n, t in w.items()}
    write_safetensors(Path(folder) / "model.safetensors", {n: torch.from_numpy(np.asarray(t)).bfloat16() for n, t in w.items()})
    toks = [int(t) for t in rng.integers(1, 63, 604)] + [63]
    toks[3] = 0
    want = U.plain_run(cfg, w, toks)
    eng = U.make_engine(folder, dtype, page_tokens=page, max_tokens=1024)
    got = U.run_cuts(eng, "a", toks, [590, 9, 2])                   # the last tokens one by one
    U.assert_close(got, want, dtype)
    got = U.run_cuts(eng, "b", toks, [len(toks)])
    U.assert_close(got, want, dtype)
    # without the old position (another token in its place) the last row is another one
    other = list(toks)
    other[3] = 1
    moved = U.row_distances(U.plain_run(cfg, w, other)[-1:], want[-1:])
    assert float(moved) > 0.1, float(moved)


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
    """Decode steps replayed from CUDA graphs (the rows an earlier layer left live in the graph's own memory) give the
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
    assert "architecture: Vofezen" in out and "l3.mix.vmix" in out and "l0.mix.dkv.norm" in out
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
