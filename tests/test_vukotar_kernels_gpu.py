"""The kernels behind the Vukotar parts, each alone against the plain functions (tests/plain/vukotar_plain.py): positions
added to embedding rows, the sum of two branches under the next norm, capped logits, the selection with sigmoid scores
and groups worth their two best (each launch form), the experts' products with the square of relu, attention with one
more in the denominator (keys that stand out at the far end, at page borders and on the diagonal)."""
import math
import os

import numpy as np
import pytest
import torch

from plain import vukotar_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16


def dev(a, dtype=F32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV).contiguous()


def bf16(a):
    return torch.tensor(np.asarray(a), dtype=F32).to(BF16).float().numpy().astype(np.float64)


def rel(got, want):
    got = got.detach().float().cpu().numpy().astype(np.float64)
    return np.abs(got - want).max() / max(1e-30, np.abs(want).max())


@pytest.mark.parametrize("width", [1, 7, 64, 1030])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_rows_with_positions(width, dtype):
    from turboquant_cpp_b200.kernels import elementwise as KE
    from turboquant_cpp_b200.models.decoder import position_turns
    rng = np.random.default_rng(width)
    V, scale = 23, 3.5
    table = bf16(rng.standard_normal((V, width)))
    pos = np.array([0, 1, 2, 63, 64, 65, 1000, 8191, 131071, 7000000])
    toks = rng.integers(0, V, size=len(pos))
    out = torch.full((len(pos), width), float("nan"), dtype=F32, device=DEV)
    KE.embed_position_rows(dev(toks, torch.int32), dev(pos, torch.int32), dev(table, dtype),
                           position_turns(width, 10000.0).to(DEV), scale, out)
    want = np.stack([table[t] * scale + P.position_vector(int(p), width) for t, p in zip(toks, pos)])
    assert np.abs(out.cpu().numpy() - want).max() < 2e-6 * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("H", [5, 37, 64, 1028, 2048])
@pytest.mark.parametrize("wdtype,odtype", [(F32, F32), (BF16, BF16), (BF16, F32)])
def test_two_branches_summed_under_the_next_norm(H, wdtype, odtype):
    from turboquant_cpp_b200.kernels import elementwise as KE
    rng = np.random.default_rng(H)
    T, k = 9, 3
    x, a, b = rng.standard_normal((T, H)) * 2, rng.standard_normal((T, H)), rng.standard_normal((T, H))
    s1, s2 = rng.standard_normal(H), rng.standard_normal(H)
    w = {"n": bf16(rng.standard_normal(H)), "n.b": bf16(rng.standard_normal(H)), "n.alpha": np.float32(0.37)}
    places = rng.permutation(T * k)
    rows_b, wts = rng.standard_normal((T * k, H)), rng.random((T, k))
    routed = np.stack([sum(wts[t, j] * rows_b[places[t * k + j]] for j in range(k)) for t in range(T)])
    norm = dict(alpha=float(w["n.alpha"]), weight=dev(w["n"], wdtype), bias=dev(w["n.b"], wdtype))
    tol = 2e-6 if odtype == F32 else 5e-3
    expert = dict(b=dev(rows_b), row_of_pair=dev(places, torch.int32), pair_weights=dev(wts))
    for kw, f, f_scale in ((dict(b=dev(b)), b, s2), (expert, routed, s2), ({}, np.zeros((T, H)), None), (expert, routed, None)):
        first = s1 if f_scale is not None else None               # without factors: plain sums
        kw = dict(kw, b_scale=dev(f_scale) if f_scale is not None and "b" in kw else None)
        total = x + (a if first is None else a * first) + (f if f_scale is None else f * f_scale)
        dx = dev(x)
        out = torch.full((T, H), float("nan"), dtype=odtype, device=DEV)
        KE.branches_dyt(dx, dev(a), dev(first) if first is not None else None, out=out, **norm, **kw)
        assert rel(dx, total) < 1e-6 and rel(out, P.dyt(total, w, "n")) < tol
        dx = dev(x)                                               # the sum alone
        assert KE.branches_dyt(dx, dev(a), dev(first) if first is not None else None, **kw) is dx
        assert rel(dx, total) < 1e-6
        dx, pick = dev(x), np.array([7, 0, 7, 3])                 # chosen rows: the stream stays as it is
        out = torch.full((4, H), float("nan"), dtype=odtype, device=DEV)
        KE.branches_dyt(dx, dev(a), dev(first) if first is not None else None, rows=dev(pick, torch.int32), out=out, **norm, **kw)
        assert torch.equal(dx, dev(x)) and rel(out, P.dyt(total, w, "n")[pick]) < tol


@pytest.mark.parametrize("T,N", [(1, 33), (7, 97), (3, 5000)])
def test_capped_logits(T, N):
    from turboquant_cpp_b200.kernels import elementwise as KE
    x = 40.0 * np.random.default_rng(N).standard_normal((T, N))
    assert rel(KE.scale_bias_cols(dev(x), cap=12.0), P.softcap(x, 12.0)) < 1e-6
    assert rel(KE.scale_bias_cols(dev(x), 0.5, cap=12.0), P.softcap(0.5 * x, 12.0)) < 1e-6
    assert torch.equal(KE.scale_bias_cols(dev(x)), dev(x))


ROUTES = [(12, 3, 3, 2), (8, 2, 1, 1), (6, 4, 6, 5), (64, 8, 8, 3), (300, 5, 10, 4), (40, 1, 20, 1), (2600, 4, 26, 3), (7, 7, 1, 1)]


@pytest.mark.parametrize("E,k,groups,keep", ROUTES)
def test_selection_with_sigmoid_scores_and_groups_of_two_best(E, k, groups, keep):
    from turboquant_cpp_b200.kernels import moe as KM
    rng = np.random.default_rng(E * 31 + k)
    T = 61
    z = 1.5 * rng.standard_normal((T, E)).astype(np.float32).astype(np.float64)
    logits = np.concatenate([z, rng.standard_normal((T, 1))], axis=1)
    ids = torch.full((T, k), -1, dtype=torch.int32, device=DEV)
    wts = torch.full((T, k), float("nan"), dtype=F32, device=DEV)
    KM.router_select_corrected(dev(logits), None, k, True, P.WEIGHT_FLOOR, groups, keep, ids, wts, None, sigmoid=True, group_top=2)
    gi, gw = ids.cpu().numpy(), wts.cpu().numpy()
    r = {"experts": E, "top": k, "groups": {"count": groups, "keep": keep} if groups > 1 else None}
    clear = decided = 0
    for t in range(T):
        want, w, s, gap = P.route_row(z[t], r)
        if gap < 1e-6:
            continue
        clear += 1
        assert sorted(gi[t]) == sorted(want), (t, gap)
        assert np.abs(gw[t][np.argsort(gi[t])] - w[np.argsort(want)]).max() < 1e-6
        # would a group's single best have chosen differently?
        if groups > 1:
            best = s.reshape(groups, -1).max(axis=1)
            kept = np.argsort(-best, kind="stable")[:keep]
            decided += not set(want // (E // groups)) <= set(kept)
    assert clear > 0.8 * T
    if groups > 1 and E // groups > 1 and keep < groups:
        assert decided > 0, "no token in this test tells the two best from the single best"


@pytest.mark.parametrize("T,E,k,groups,keep,H", [(1, 12, 3, 3, 2, 64), (4, 60, 4, 4, 2, 128), (8, 60, 4, 12, 5, 256), (5, 8, 8, 1, 1, 40),
                                                 (24, 16, 2, 8, 3, 72), (1, 300, 3, 10, 2, 512)])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("sigmoid", [True, False])
@pytest.mark.parametrize("form", ["", "TQ_ROUTER_NO_TINY", "TQ_ROUTER_NO_CLUSTER"])
def test_every_one_launch_router_chooses_like_the_separate_kernels(T, E, k, groups, keep, H, dtype, sigmoid, form, monkeypatch):
    from turboquant_cpp_b200.kernels import elementwise as KE, moe as KM
    if form:
        monkeypatch.setenv("TQ_ROUTER_NO_TINY", "1")
        monkeypatch.setenv(form, "1")
    rng = np.random.default_rng(T * 100 + E)
    x = dev(rng.standard_normal((T, H)), dtype)
    wr = dev(rng.standard_normal((E, H)) / math.sqrt(H), dtype)
    i32, f32 = dict(dtype=torch.int32, device=DEV), dict(dtype=F32, device=DEV)
    ids_a, w_a, ids_b, w_b = torch.empty((T, k), **i32), torch.empty((T, k), **f32), torch.empty((T, k), **i32), torch.empty((T, k), **f32)
    how = dict(sigmoid=sigmoid, group_top=2)
    logits = KM.router_logits(x, wr, None, torch.empty((T, E + 1), **f32))
    KM.router_select_corrected(logits, None, k, True, P.WEIGHT_FLOOR, groups, keep, ids_a, w_a, None, **how)
    lay_a, lay_b = KM.ExpertLayout(T * k, E, 16, DEV), KM.ExpertLayout(T * k, E, 16, DEV)
    KM.moe_align(ids_a, lay_a)
    rows_a = KE.gather_rows(x, lay_a.sorted_pair, k, torch.empty((T * k, H), dtype=dtype, device=DEV))
    rows_b = torch.empty((T * k, H), dtype=dtype, device=DEV)
    KM.router_small(x, wr, None, k, True, ids_b, w_b, None, lay_b, rows_b, corrected=True, floor=P.WEIGHT_FLOOR,
                    n_groups=groups, keep_groups=keep, **how)
    # the forms add a row's products up in different orders: the choices agree where they are clear, the weights to rounding
    z = logits[:, :E].double().cpu().numpy()
    same = (ids_a == ids_b).all(dim=1).cpu().numpy()
    for t in range(T):
        if not same[t] and sigmoid:
            assert P.route_row(z[t], {"experts": E, "top": k, "groups": {"count": groups, "keep": keep}})[3] < 1e-5, t
    assert same.mean() > 0.9
    assert (w_a - w_b).abs().max().item() < 1e-5 or not same.all()
    if same.all():
        assert torch.equal(lay_a.sorted_pair[:T * k], lay_b.sorted_pair[:T * k])
        assert torch.equal(lay_a.row_of_pair[:T * k], lay_b.row_of_pair[:T * k])
        n = int(lay_a.n_tiles.item())
        assert n == int(lay_b.n_tiles.item()) and torch.equal(lay_a.tile_expert[:n], lay_b.tile_expert[:n])
        assert torch.equal(rows_a, rows_b)


@pytest.mark.parametrize("R,N,K,G", [(3, 24, 40, 4), (70, 64, 48, 5), (300, 136, 192, 8), (900, 260, 128, 2)])
@pytest.mark.parametrize("form", ["tensor cores", "exact"])
def test_experts_products_with_the_square_of_relu(R, N, K, G, form):
    from turboquant_cpp_b200.kernels import elementwise as KE, gemm_tc as KT, moe as KM
    rng = np.random.default_rng(R + N)
    a, w = bf16(rng.normal(size=(R, K))), bf16(1.5 * rng.normal(size=(G, N, K)) / math.sqrt(K))
    ids = rng.integers(0, G, size=(R, 1)).astype(np.int32)

    def layout(tile):
        lay = KM.ExpertLayout(R, G, tile, DEV)
        KM.moe_align(dev(ids, torch.int32), lay)
        order = lay.sorted_pair.cpu().numpy()[:R]
        want = np.stack([np.maximum(w[ids[o, 0]] @ a[o], 0.0) ** 2 for o in order])
        return lay, a[order], want

    if form == "tensor cores":
        packed = KT.pack_weights(dev(w, BF16), False)
        for tile in KT.TOKEN_TILES:
            lay, x, want = layout(tile)
            for pair in ((False, True) if tile >= 128 else (False,)):
                for dt, tol in ((BF16, 6e-3), (F32, 1e-5)):
                    out = torch.full((R, N), float("nan"), dtype=dt, device=DEV)
                    KT.gemm_tc(dev(x, BF16), packed, out, lay, tile, pair=pair, map=KE.MAP_RELU_SQUARED)
                    KT.check_status()
                    assert rel(out, want) < tol, (tile, pair, dt)
        return
    lay, x, want = layout(64)
    for few in (False, True):
        for dt, tol in ((F32, 2e-5), (BF16, 6e-3)):
            out = torch.full((R, N), float("nan"), dtype=dt, device=DEV)
            KM.grouped_gemm(dev(x, dt), dev(w, dt), out, lay, False, few_rows=few, map=KE.MAP_RELU_SQUARED)
            assert rel(out, want) < tol, (few, dt)


def test_an_element_function_is_refused_where_the_product_has_another_activation():
    from turboquant_cpp_b200.kernels import elementwise as KE, gemm_tc as KT, moe as KM
    from turboquant_cpp_b200.kernels._call import KernelError
    x, w = torch.zeros((4, 16), dtype=BF16, device=DEV), torch.zeros((1, 32, 16), dtype=BF16, device=DEV)
    out = torch.zeros((4, 16), dtype=BF16, device=DEV)
    for bad in (lambda: KT.gemm_tc(x, KT.pack_weights(w, True), out, None, 16, map=KE.MAP_RELU_SQUARED),
                lambda: KT.gemm_tc(x, KT.pack_weights(w[:, :16], False), out, None, 16, map=9),
                lambda: KM.grouped_gemm(x, w, out, None, True, map=KE.MAP_RELU_SQUARED),
                lambda: KM.router_select_corrected(torch.zeros((2, 5), device=DEV), None, 2, True, 0.0, 2, 1,
                                                   torch.zeros((2, 2), dtype=torch.int32, device=DEV), torch.zeros((2, 2), device=DEV),
                                                   None, group_top=3)):
        with pytest.raises(KernelError):
            bad()


def scattered_cache(T, G, dr, dtype, rng, extra_pages=3):
    n = -(-T // 64)
    cache = torch.full((n + extra_pages, 1, G, 64, dr), 1e30, dtype=dtype, device=DEV)
    table = torch.tensor(rng.permutation(n + extra_pages)[:n].reshape(1, n), dtype=torch.int32, device=DEV)
    return cache, table


@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 32, 64), (3, 3, 64, 128), (8, 1, 128, 32), (6, 2, 24, 40), (2, 1, 9, 7)])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("special", [None, 0, 63, 64, 127, 128, 250])
def test_attention_with_one_more_in_the_denominator(H, G, dk, dv, dtype, special):
    """special: the place of a key that every query likes far better than the others (its own value stands out too),
    at a sequence's start, at page borders, on the last query's diagonal; None: weak scores, so that the one in the
    denominator takes a visible share."""
    from turboquant_cpp_b200.kernels import bias_attention as KB
    T = 251
    rng = np.random.default_rng(H * 7 + (special or 0))
    scale = 0.8 / math.sqrt(dk)
    q, k, v = (0.3 * rng.standard_normal((T, n, d)) for n, d in ((H, dk), (G, dk), (G, dv)))
    if special is not None:
        u = rng.standard_normal(dk)
        u *= math.sqrt(12.0 / scale) / np.linalg.norm(u)
        q += u
        k[special] += u
        v[special] += 5.0
    qkv = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], axis=1)
    if dtype == BF16:
        q, k, v = bf16(q), bf16(k), bf16(v)
    want = P.attention_core(q, k, v, scale).reshape(T, H * dv)
    cache, table = scattered_cache(T, G, dk + dv, dtype, rng)
    positions, seq = torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
    qd = torch.empty((T, H, dk), dtype=dtype, device=DEV)
    KB.kv_write(dev(qkv), qd, cache, None, None, 0.0, positions, seq, table, 64, H, G, dk, dv)
    sink = torch.zeros(H, dtype=F32, device=DEV)
    tol = 2e-5 if dtype == F32 else 1.5e-2
    for n_splits in (1, 3, 16):
        out = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
        KB.attention(qd, cache, None, sink, positions, seq, table, 64, 0, 0, scale, out, H, G, dk, dv, n_splits=n_splits)
        assert rel(out, want) < tol, n_splits
    if KB.runs_usable(dtype, dk, dv, 64):
        for start in (0, 100):
            out = torch.full((T - start, H * dv), float("nan"), dtype=dtype, device=DEV)
            cu = torch.tensor([0, T - start], dtype=torch.int32, device=DEV)
            st = torch.tensor([start], dtype=torch.int32, device=DEV)
            KB.attention_runs(qd[start:].contiguous(), cache, None, sink, cu, st, table, 64, 0, 0, scale, out, 1, T - start, H, G, dk, dv)
            assert rel(out, want[start:]) < tol, start
    # the oracle tells a missing key, and a missing one in the denominator, from the right answer
    if special is not None:
        less = P.attention_core(q, np.where(np.arange(T)[:, None, None] == special, -k, k), v, scale).reshape(T, H * dv)
        assert np.abs(less - want)[special:].max() > 0.1 * np.abs(want).max()
    else:
        s = k[:2, 0] @ q[1, 0] * scale
        e = np.exp(s) / np.exp(s).sum()
        assert np.abs(e @ v[:2, 0] - want[1].reshape(H, dv)[0]).max() > 0.1 * np.abs(want[1]).max()
