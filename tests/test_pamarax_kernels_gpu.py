"""The kernels behind the Pamarax parts, each alone against the plain functions (tests/plain/pamarax_plain.py): the
matrix memory's gates, recurrence, chunks side by side and one-launch step, the delta rule with one decay per head in its
three forms, the convolution of single tokens, the cache write with norms over whole rows, values that are keys and the
query temperature, the element-wise gate, attention with one more in the denominator, gated activation and closing
projection with biases, and the weighted sum of two branches under a norm."""
import numpy as np
import pytest
import torch

from plain import pamarax_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV).contiguous()


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


def host(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def rel(got, want):
    return np.abs(host(got) - want).max() / max(1e-30, np.abs(want).max())


def area(slots, size, used, lead=0):
    """A state area of float32 rows in which every slot but the used ones holds other values; the first `lead` elements of
    a row belong to somebody else."""
    a = torch.full((slots, lead + size), 3.0, device=DEV)
    for sl in used:
        a[sl, lead:] = 0.0
    return a


# ---- the matrix memory --------------------------------------------------------------------------------------------
FLOOR = P.MEMORY_FLOOR
MEMORY_CASES = [
    # heads, key size, value size, cap
    (3, 8, 12, 9.0),
    (2, 64, 40, 15.0),
    (1, 100, 31, 4.0),
    (2, 200, 21, 15.0),
    (1, 1, 1, 2.0),
    (2, 128, 128, 20.0),
    (5, 33, 32, 6.0),
]


def memory_inputs(rng, n, case, i_off, f_off, width):
    H, dk, dv, cap = case
    proj = rng.standard_normal((n, width)) * 1.5
    return host(dev(proj))


def memory_reference(proj, case, offs, bi, bf, w, eps):
    """(outputs behind norm, weight and gate [n, H * dv], end states per head, raw outputs)."""
    H, dk, dv, cap = case
    q0, k0, v0, g0, i0, f0 = offs
    n = proj.shape[0]
    gi = cap * np.tanh((proj[:, i0:i0 + H] + bi) / cap)
    gf = P.log_sigmoid(cap * np.tanh((proj[:, f0:f0 + H] + bf) / cap))
    outs, ends = np.zeros((n, H, dv)), []
    for a in range(H):
        q = proj[:, q0 + a * dk:q0 + (a + 1) * dk] * dk ** -0.5
        o, st = P.memory_recurrence(q, proj[:, k0 + a * dk:k0 + (a + 1) * dk], proj[:, v0 + a * dv:v0 + (a + 1) * dv], gi[:, a], gf[:, a])
        outs[:, a] = o
        ends.append(st)
    full = P.unit_rms(outs, eps).reshape(n, H * dv) * w * P.sigmoid(proj[:, g0:g0 + H * dv])
    return full, ends, outs.reshape(n, H * dv)


def memory_layout(case, lead=5):
    """Columns of a projection's row: something else, then q, k, v, gate and the two gates' logits, then something else."""
    H, dk, dv, _ = case
    at, offs = lead, []
    for size in (H * dk, H * dk, H * dv, H * dv, H, H):
        offs.append(at)
        at += size
    return offs, at + 2


def run_memory(KS, proj, case, offs, bi, bf, w, eps, state, tops, cu, slots, odtype, form, chunk=0):
    """One step of the memory in the named form ('step': one token each; 'scan': the launches for runs)."""
    H, dk, dv, cap = case
    q, k, v, g, i, f = offs
    T = proj.shape[0]
    pd, out = dev(proj), torch.full((T, H * dv), float("nan"), dtype=odtype, device=DEV)
    if form == "step":
        return KS.memory_step(pd, q, k, v, g, i, f, dev(bi), dev(bf), cap, dk ** -0.5, state, tops, slots, w, out, H, dk, dv, FLOOR, eps)
    new = lambda *s: torch.full(s, float("nan"), device=DEV)
    gates, m, y, dots = new(T, H, 2), new(T, H), new(T, H * dv), new(T, H)
    KS.memory_gates(pd, i, f, dev(bi), dev(bf), cap, tops, gates, m, H, cu, slots)
    if not chunk:
        KS.memory_scan(pd, q, k, v, gates, state, y, dots, H, dk, dv, cu, slots)
    else:
        lens = np.diff(cu.cpu().numpy())
        cc, sc = [0], [0]
        for n in lens:
            base = cc[-1]
            cc += [base + min(int(n), c + chunk) for c in range(0, int(n), chunk)]
            sc.append(len(cc) - 1)
        N = len(cc) - 1
        ends, starts, decays = torch.zeros((N, H, dv + 1, dk), device=DEV), new(N, H, dv + 1, dk), new(N, H)
        KS.memory_scan(pd, q, k, v, gates, ends, None, decays, H, dk, dv, i32(cc), i32(list(range(N))))
        KS.memory_combine(state, slots, ends, starts, i32(sc), decays)
        KS.memory_scan(pd, q, k, v, gates, starts, y, dots, H, dk, dv, i32(cc), i32(list(range(N))))
    return KS.gated_group_norm(y, pd, g, w, H, eps, out, gate_after=True, sigmoid_gate=True, dots=dots, tops=m,
                               dot_scale=dk ** -0.5, floor=FLOOR)


@pytest.mark.parametrize("wdtype,odtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("case", MEMORY_CASES)
def test_memory_over_portions_in_used_slots(case, wdtype, odtype):
    """Three sequences in portions of unequal sizes, down to single tokens (the one-launch step), in slots in another
    order than the batch; the states and maxima pass from portion to portion and from form to form."""
    from turboquant_cpp_b200.kernels import ssm as KS
    H, dk, dv, cap = case
    rng = np.random.default_rng(dk * 10 + dv)
    offs, width = memory_layout(case)
    lens, eps = [61, 9, 330], 2e-5
    bi, bf = host(dev(rng.standard_normal(H))), host(dev(2.0 + rng.standard_normal(H)))
    w = host(dev(1 + 0.2 * rng.standard_normal(H * dv), wdtype))
    data = [memory_inputs(rng, n, case, 0, 0, width) for n in lens]
    want = [memory_reference(d, case, offs, bi, bf, w, eps) for d in data]
    size, slots = H * (dv + 1) * dk, [3, 0, 4]
    a = area(5, size + H + 3, slots)
    state, tops = a[:, :size].unflatten(1, (H, dv + 1, dk)), a[:, size:size + H]
    done = [0, 0, 0]
    tol = 1e-4 if odtype == torch.float32 else 1e-2
    for portion in ([1, 2, 17], [1, 1, 1], [40, 5, 300], [1, 1, 1], [18, 0, 11]):
        live = [i for i in range(3) if done[i] < lens[i]]
        take = [min(portion[i], lens[i] - done[i]) for i in live]
        rows = np.concatenate([data[i][done[i]:done[i] + n] for i, n in zip(live, take)])
        cu = i32(np.concatenate([[0], np.cumsum(take)]))
        out = run_memory(KS, rows, case, offs, bi, bf, dev(w, wdtype), eps, state, tops, cu, i32([slots[i] for i in live]), odtype,
                         "step" if max(take) == 1 else "scan")
        ref = np.concatenate([want[i][0][done[i]:done[i] + n] for i, n in zip(live, take)])
        assert rel(out, ref) < tol, portion
        for i, n in zip(live, take):
            done[i] += n
    assert done == lens
    for i, sl in enumerate(slots):
        for h, (S, n, m) in enumerate(want[i][1]):
            assert rel(state[sl, h, :dv].t(), S) < 1e-4 and rel(state[sl, h, dv], n) < 1e-4 and abs(float(tops[sl, h]) - m) < 1e-4
    assert float(a[1].min()) == 3.0 and float(a[2].max()) == 3.0 and float(a[:, size + H:][slots].abs().max()) == 0.0


@pytest.mark.parametrize("case", MEMORY_CASES)
@pytest.mark.parametrize("chunk", [16, 70])
def test_memory_in_chunks_side_by_side(case, chunk):
    """Runs cut into chunks give what the runs in one piece give, from kept states that are not zero."""
    from turboquant_cpp_b200.kernels import ssm as KS
    H, dk, dv, cap = case
    rng = np.random.default_rng(dk + dv)
    offs, width = memory_layout(case, lead=2)
    eps, lens, slots = 1e-5, [210, 3, 145], [2, 0, 3]
    bi, bf, w = host(dev(rng.standard_normal(H))), host(dev(3.0 + rng.standard_normal(H))), np.ones(H * dv)
    data = [memory_inputs(rng, n + 20, case, 0, 0, width) for n in lens]
    want = [memory_reference(d, case, offs, bi, bf, w, eps) for d in data]
    size = H * (dv + 1) * dk
    a = area(4, size + H, slots)
    state, tops = a[:, :size].unflatten(1, (H, dv + 1, dk)), a[:, size:]
    go = lambda rows, cu, chunk: run_memory(KS, rows, case, offs, bi, bf, dev(w), eps, state, tops, i32(cu), i32(slots), torch.float32,
                                            "scan", chunk)
    first = go(np.concatenate([d[:20] for d in data]), [0, 20, 40, 60], 0)
    assert rel(first, np.concatenate([x[0][:20] for x in want])) < 1e-4
    rest = go(np.concatenate([d[20:] for d in data]), [0, lens[0], lens[0] + lens[1], sum(lens)], chunk)
    assert rel(rest, np.concatenate([x[0][20:] for x in want])) < 1e-4
    for i, sl in enumerate(slots):
        for h, (S, n, m) in enumerate(want[i][1]):
            assert rel(state[sl, h, :dv].t(), S) < 1e-4 and rel(state[sl, h, dv], n) < 1e-4 and abs(float(tops[sl, h]) - m) < 1e-4


@pytest.mark.parametrize("form", ["scan", "step"])
def test_memory_where_each_side_of_the_denominator_decides(form):
    """Tokens whose |n . q| is far below e^-m and tokens where it is far above, input gates from closed to open, a first
    token whose gate lies below the starting maximum of zero, and a token that is written, kept over hundreds of others
    with open forget gates and found again by its key."""
    from turboquant_cpp_b200.kernels import ssm as KS
    case = (2, 16, 8, 15.0)
    H, dk, dv, cap = case
    rng = np.random.default_rng(4)
    offs, width = memory_layout(case)
    n, eps = 300, 1e-6
    proj = rng.standard_normal((n, width)) * 0.3
    q, k, v, g, i, f = offs
    proj[:, i:i + H] = rng.choice([-12.0, -6.0, 0.0, 2.0], size=(n, H))
    proj[:, f:f + H] = 9.0                                         # almost nothing is forgotten
    proj[0, i:i + H] = -14.0
    proj[::3, q:q + H * dk] *= 1e-3                                # queries that meet nothing: e^-m is the larger side
    for h in range(H):                                             # the far token: a key of its own, asked for at the end
        key = np.zeros(dk)
        key[3] = 6.0
        proj[5, k + h * dk:k + (h + 1) * dk] = key
        proj[5, i + h] = 6.0
        proj[n - 1, q + h * dk:q + (h + 1) * dk] = key * 3
    proj = host(dev(proj))
    zero = np.zeros(H)
    w = np.ones(H * dv)
    want, _, raw = memory_reference(proj, case, offs, zero, zero, w, eps)
    dots_decide = 0
    for h in range(H):
        gi = cap * np.tanh(proj[:, i + h] / cap)
        gf = P.log_sigmoid(cap * np.tanh(proj[:, f + h] / cap))
        nn, m = np.zeros(dk), 0.0
        for t in range(n):
            top = max(gf[t] + m, gi[t])
            nn = np.exp(gf[t] + m - top) * nn + np.exp(gi[t] - top) * proj[t, k + h * dk:k + (h + 1) * dk]
            m = top
            dots_decide += abs(nn @ proj[t, q + h * dk:q + (h + 1) * dk]) * dk ** -0.5 > np.exp(-m)
    assert 0.1 < dots_decide / (n * H) < 0.9                       # both sides occur
    forget = proj.copy()
    forget[5, i:i + H] = -14.0                                     # without the far token the last output is another one
    moved = memory_reference(forget, case, offs, zero, zero, w, eps)[0]
    assert np.abs(moved[-1] - want[-1]).max() > 0.05 * np.abs(want).max()
    size = H * (dv + 1) * dk
    a = area(2, size + H, [1])
    state, tops = a[:, :size].unflatten(1, (H, dv + 1, dk)), a[:, size:]
    if form == "scan":
        got = run_memory(KS, proj, case, offs, zero, zero, dev(w), eps, state, tops, i32([0, n]), i32([1]), torch.float32, "scan")
    else:
        got = torch.cat([run_memory(KS, proj[t:t + 1], case, offs, zero, zero, dev(w), eps, state, tops, None, i32([1]), torch.float32, "step")
                         for t in range(n)])
    assert rel(got, want) < 2e-4


# ---- the delta rule with one decay per head -----------------------------------------------------------------------
DELTA_CASES = [
    # H, G, dk, dv
    (4, 2, 8, 12),
    (2, 2, 64, 40),
    (3, 1, 100, 16),
    (1, 1, 200, 21),
    (2, 1, 1, 1),
    (2, 2, 128, 128),
    (6, 3, 31, 33),
]
UNIT_EPS = P.UNIT_EPS


def delta_data(rng, n, case, per_channel):
    """xqkv, projection and raw decays of n tokens, and what the plain rule makes of them: raw outputs, end states."""
    H, G, dk, dv = case
    C, b_off, a_off = 2 * G * dk + H * dv, 3, 2
    dper = dk if per_channel else 1
    xqkv = host(dev(rng.standard_normal((n, C))))
    proj = host(dev(rng.standard_normal((n, b_off + H + 4)) * 2))
    raw = host(dev(rng.standard_normal((n, a_off + H * dper + 1)) * 2 - 2))
    return xqkv, proj, raw


def delta_reference(d, case, a_log, dt_bias, per_channel):
    from plain import tasadra_plain
    H, G, dk, dv = case
    xqkv, proj, raw = d
    n = len(xqkv)
    q = P.unit_vector(xqkv[:, :G * dk].reshape(n, G, dk)) * dk ** -0.5
    k = P.unit_vector(xqkv[:, G * dk:2 * G * dk].reshape(n, G, dk))
    v = xqkv[:, 2 * G * dk:].reshape(n, H, dv)
    beta = P.sigmoid(proj[:, 3:3 + H])
    if per_channel:
        decay = np.exp(-np.exp(a_log)[None, :, None] * P.softplus(raw[:, 2:2 + H * dk] + dt_bias).reshape(n, H, dk))
        outs = [tasadra_plain.delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], decay[:, a]) for a in range(H)]
    else:
        decay = np.exp(-np.exp(a_log) * P.softplus(raw[:, 2:2 + H] + dt_bias))
        outs = [P.gated_delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], decay[:, a]) for a in range(H)]
    return np.stack([o for o, _ in outs], axis=1), np.stack([S for _, S in outs])


@pytest.mark.parametrize("form", ["delta_scan", "delta_scan_runs"])
@pytest.mark.parametrize("case", DELTA_CASES)
def test_delta_rule_with_a_decay_per_head_over_portions(case, form):
    from turboquant_cpp_b200.kernels import ssm as KS
    H, G, dk, dv = case
    rng = np.random.default_rng(dk * 10 + dv)
    lens = [61, 9, 143]
    a_log, dt_bias = host(dev(rng.standard_normal(H) * 0.7)), host(dev(rng.standard_normal(H)))
    data = [delta_data(rng, n, case, False) for n in lens]
    want = [delta_reference(d, case, a_log, dt_bias, False) for d in data]
    slots = [3, 0, 4]
    a = area(5, H * dv * dk, slots, lead=11)
    state = a[:, 11:].unflatten(1, (H, dv, dk))
    done = [0, 0, 0]
    for portion in ([1, 2, 17], [2, 1, 1], [40, 6, 113], [18, 0, 12]):
        live = [i for i in range(3) if done[i] < lens[i]]
        take = [min(portion[i], lens[i] - done[i]) for i in live]
        parts = [np.concatenate([data[i][j][done[i]:done[i] + n] for i, n in zip(live, take)]) for j in range(3)]
        cu = np.concatenate([[0], np.cumsum(take)])
        y = torch.full((int(cu[-1]), H * dv), float("nan"), device=DEV)
        getattr(KS, form)(dev(parts[0]), 0, G * dk, 2 * G * dk, dev(parts[1]), 3, dev(parts[2]), 2, dev(dt_bias), dev(a_log),
                          state, y, H, G, dk, dv, UNIT_EPS, dk ** -0.5, i32(cu), i32([slots[i] for i in live]))
        ref = np.concatenate([want[i][0][done[i]:done[i] + n] for i, n in zip(live, take)]).reshape(len(y), -1)
        assert rel(y, ref) < 3e-5, portion
        for i, n in zip(live, take):
            done[i] += n
    assert done == lens
    for i, sl in enumerate(slots):
        assert rel(state[sl].transpose(1, 2), want[i][1]) < 3e-5
    assert float(a[1].min()) == 3.0 and float(a[:, :11].min()) == 3.0


@pytest.mark.parametrize("sigmoid_gate,per_channel,wdtype,odtype", [
    (False, False, torch.float32, torch.float32), (True, True, torch.float32, torch.float32),
    (False, False, torch.bfloat16, torch.bfloat16), (True, False, torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("case", DELTA_CASES)
def test_delta_rule_token_by_token_in_one_launch(case, sigmoid_gate, per_channel, wdtype, odtype):
    from turboquant_cpp_b200.kernels import ssm as KS
    H, G, dk, dv = case
    rng = np.random.default_rng(dk + dv)
    n, eps = 23, 3e-5
    a_log, dt_bias = host(dev(rng.standard_normal(H) * 0.7)), host(dev(rng.standard_normal(H * (dk if per_channel else 1))))
    data = [delta_data(rng, n, case, per_channel) for _ in range(2)]
    gates = [host(dev(rng.standard_normal((n, 4 + H * dv)) * 2)) for _ in range(2)]
    w = host(dev(1 + 0.2 * rng.standard_normal(dv), wdtype))
    slots = [2, 0]
    a = area(3, H * dv * dk, slots, lead=6)
    state = a[:, 6:].unflatten(1, (H, dv, dk))
    want = []
    for d, z in zip(data, gates):
        o, S = delta_reference(d, case, a_log, dt_bias, per_channel)
        z = z[:, 4:].reshape(n, H, dv)
        want.append((P.unit_rms(o, eps) * w * (P.sigmoid(z) if sigmoid_gate else P.silu(z)), S))
    for t in range(n):
        rows = [np.stack([d[j][t] for d in data]) for j in range(3)]
        out = torch.full((2, H * dv), float("nan"), dtype=odtype, device=DEV)
        KS.delta_step(dev(rows[0]), 0, G * dk, 2 * G * dk, dev(rows[1]), 3, dev(rows[2]), 2, dev(dt_bias), dev(a_log),
                      dev(np.stack([z[t] for z in gates])), 4, sigmoid_gate, dev(np.tile(w, H), wdtype), state, i32(slots), out, H, G, dk, dv,
                      UNIT_EPS, dk ** -0.5, eps)
        assert rel(out, np.stack([x[0][t].reshape(-1) for x in want])) < (5e-5 if odtype == torch.float32 else 1e-2), t
    for i, sl in enumerate(slots):
        assert rel(state[sl].transpose(1, 2), want[i][1]) < 3e-5
    assert float(a[1].min()) == 3.0 and float(a[:, :6].min()) == 3.0


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8])
@pytest.mark.parametrize("wdtype", [torch.float32, torch.bfloat16])
def test_short_convolution_over_portions_and_token_by_token(taps, wdtype):
    """Runs (short steps and steps long enough for several tokens a thread), then single tokens in one launch, from the
    kept inputs the launches before left."""
    from turboquant_cpp_b200.kernels import ssm as KS
    rng = np.random.default_rng(taps)
    C, off, lens, slots = 150, 7, [290, 45, 4], [1, 3, 0]
    w = host(dev(rng.standard_normal((C, taps)), wdtype))
    u = [host(dev(rng.standard_normal((n, off + C + 2)))) for n in lens]
    want = [P.silu(P.short_convolution(x[:, off:off + C], w)) for x in u]
    a = area(4, (taps - 1) * C, slots, lead=3)
    kept = a[:, 3:].unflatten(1, (taps - 1, C)) if taps > 1 else torch.empty((4, 0, C), device=DEV)
    done = [0, 0, 0]
    for portion in ([2, 1, 1], [1, 1, 1], [280, 30, 1], [1, 1, 1], [1, 1, 0], [5, 11, 0]):
        live = [i for i in range(3) if done[i] < lens[i]]
        take = [min(portion[i], lens[i] - done[i]) for i in live]
        rows = np.concatenate([u[i][done[i]:done[i] + n] for i, n in zip(live, take)])
        out = torch.full((len(rows), C), float("nan"), device=DEV)
        sl = i32([slots[i] for i in live])
        if max(take) == 1:
            KS.conv_silu_step(dev(rows), off, dev(w, wdtype), None, kept, out, sl)
        else:
            KS.conv_silu(dev(rows), off, dev(w, wdtype), None, kept, out, i32(np.repeat(np.arange(len(live)), take)),
                         i32(np.concatenate([[0], np.cumsum(take)])), sl)
        assert rel(out, np.concatenate([want[i][done[i]:done[i] + n] for i, n in zip(live, take)])) < 1e-5, portion
        for i, n in zip(live, take):
            done[i] += n
    assert done == lens
    assert float(a[2].min()) == 3.0 and float(a[:, :3].min()) == 3.0


# ---- attention's pieces -----------------------------------------------------------------------------------------------
def scattered_cache(T, G, dr, dtype, rng, extra_pages=3):
    """More pages than the sequence needs, a large value where nothing is written, pages visited in a shuffled order."""
    n = -(-T // 64)
    cache = torch.full((n + extra_pages, 1, G, 64, dr), 1e30, dtype=dtype, device=DEV)
    table = torch.tensor(rng.permutation(n + extra_pages)[:n].reshape(1, n), dtype=torch.int32, device=DEV)
    return cache, table


def cached_rows(cache, table, T, G, dr):
    pos = np.arange(T)
    c = host(cache)[table.cpu().numpy()[0][pos // 64], 0, :, pos % 64]
    return c.reshape(T, G, dr)


WRITE_CASES = [
    # H, G, dk, dv, norm, rotated elements, base, values are keys, temperature
    (4, 2, 16, 16, "row", 8, 500.0, True, None),
    (3, 1, 40, 40, "row", 40, 10000.0, True, None),
    (16, 4, 20, 20, "row", 20, 77.0, True, None),
    (5, 5, 6, 9, "row", 0, 1.0, False, (0.3, 7)),
    (4, 2, 12, 20, "head", 0, 1.0, False, (0.7, 24)),
    (1, 1, 256, 5, "head", 0, 1.0, False, (2.0, 1)),
    (6, 3, 64, 32, "head", 16, 30.0, False, (-0.2, 200)),
    (2, 2, 1, 1, None, 0, 1.0, True, (1.0, 64)),
]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", WRITE_CASES)
def test_cache_write_with_row_norms_shared_values_and_temperature(case, dtype):
    from turboquant_cpp_b200.kernels import bias_attention as KB
    H, G, dk, dv, norm, dims, base, shared, temp = case
    rng = np.random.default_rng(H * dk + dv)
    T, eps = 210, 4e-5
    pos = np.arange(T)
    rows = host(dev(rng.standard_normal((T, H * dk + G * dk + (0 if shared else G * dv) + 3)) * 1.3))
    q, k = rows[:, :H * dk], rows[:, H * dk:(H + G) * dk]
    v = k.reshape(T, G, dk) if shared else rows[:, (H + G) * dk:(H + G) * dk + G * dv].reshape(T, G, dv)
    wq, wk = (host(dev(1 + 0.3 * rng.standard_normal(n * dk if norm == "row" else dk))) for n in (H, G))
    if norm == "row":
        q, k = P.unit_rms(q, eps) * wq, P.unit_rms(k, eps) * wk
    q, k = q.reshape(T, H, dk), k.reshape(T, G, dk)
    if norm == "head":
        q, k = P.unit_rms(q, eps) * wq, P.unit_rms(k, eps) * wk
    if dims:
        q, k = P.rotate_halves(q, pos, dims, base), P.rotate_halves(k, pos, dims, base)
    if temp:
        q = q * P.query_temperature(pos, *temp)[:, None, None]
    freq = dev([base ** (-2.0 * i / dims) for i in range(dims // 2)]) if dims else None
    cache, table = scattered_cache(T, G, dk + dv, dtype, rng)
    out = torch.full((T, H, dk), float("nan"), dtype=dtype, device=DEV)
    KB.kv_write_rot(dev(rows), out, cache, freq, dims, True, 0.0, i32(pos), torch.zeros(T, dtype=torch.int32, device=DEV), table, 64,
                    H, G, dk, dv, q_norm=dev(wq) if norm else None, k_norm=dev(wk) if norm else None, norm_eps=eps, norm_rows=norm == "row",
                    values_are_keys=shared, temperature=temp)
    tol = 5e-5 if dtype == torch.float32 else 8e-3
    assert rel(out, q) < tol
    got = cached_rows(cache, table, T, G, dk + dv)
    assert np.abs(got[..., :dk] - k).max() < tol * np.abs(k).max() and np.abs(got[..., dk:] - v).max() < tol * np.abs(v).max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,off,pad", [(64, 4, 0), (33, 5, 2), (1, 0, 0), (130, 8, 2)])
def test_elements_gated(N, off, pad, dtype):
    from turboquant_cpp_b200.kernels import bias_attention as KB
    rng = np.random.default_rng(N)
    T = 19
    o, gates = host(dev(rng.standard_normal((T, N)), dtype)), host(dev(rng.standard_normal((T, off + N + pad)) * 4))
    od = dev(o, dtype)
    KB.elements_gate(od, dev(gates), off, od)
    assert rel(od, o * P.sigmoid(gates[:, off:off + N])) < (1e-5 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 12, 20), (4, 1, 64, 32), (2, 2, 128, 128), (3, 1, 9, 9)])
@pytest.mark.parametrize("sink", [True, False])
def test_attention_over_scattered_pages_with_a_key_that_stands_out(H, G, dk, dv, sink, dtype):
    """Every query sees all earlier positions: a marked key at a sequence's start, at both sides of a page border and at the
    query's own position decides its output; weak scores show the one in the denominator."""
    from turboquant_cpp_b200.kernels import bias_attention as KB
    rng = np.random.default_rng(dk + H)
    T, scale = 200, 0.5
    q, k, v = (host(dev(rng.standard_normal(s), dtype)) for s in ((T, H, dk), (T, G, dk), (T, G, dv)))
    k[:64] *= 0.05
    q[:70] *= 0.1                                                 # early positions: weak scores, the added one weighs
    for mark, readers in ((0, (90, 199)), (63, (120,)), (64, (121, 150)), (180, (180,))):
        k[mark] = rng.choice([-1.0, 1.0], size=(G, dk)) * 2
        for t in readers:
            for a in range(H):
                q[t, a] = k[mark, a // (H // G)] * 3
    q, k = host(dev(q, dtype)), host(dev(k, dtype))
    want = P.attend(q, k, v, scale, extra=1.0 if sink else 0.0)
    for mark, t in ((0, 199), (63, 120), (64, 150), (180, 180)):      # the marked keys do decide
        assert np.abs(want[t, 0] - v[mark, 0]).max() < 0.05
    if sink:
        assert np.abs(want[:60] - P.attend(q[:60], k[:60], v[:60], scale)).max() > 0.02
    cache, table = scattered_cache(T, G, dk + dv, dtype, rng)
    pg, sl = table.cpu().numpy()[0][np.arange(T) // 64], np.arange(T) % 64
    cache[torch.tensor(pg, device=DEV).long(), 0, :, torch.tensor(sl, device=DEV)] = dev(np.concatenate([k, v], axis=2), dtype)
    zero = torch.zeros(H, device=DEV) if sink else None
    tol = 3e-5 if dtype == torch.float32 else 1.5e-2
    for n_splits in (1, 3):
        out = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
        KB.attention(dev(q, dtype), cache, None, zero, i32(np.arange(T)), torch.zeros(T, dtype=torch.int32, device=DEV), table, 64, 0, 0,
                     scale, out, H, G, dk, dv, n_splits=n_splits)
        assert rel(out, want.reshape(T, -1)) < tol, n_splits
    if KB.runs_usable(dtype, dk, dv, 64):
        for start in (0, 77, T - 3):
            out = torch.full((T - start, H * dv), float("nan"), dtype=dtype, device=DEV)
            KB.attention_runs(dev(q[start:], dtype), cache, None, zero, i32([0, T - start]), i32([start]), table, 64, 0, 0, scale, out, 1,
                              T - start, H, G, dk, dv)
            assert rel(out, want[start:].reshape(T - start, -1)) < tol, start


# ---- element-wise pieces ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("odtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("I", [5, 64, 1023, 1024, 2500])
def test_gated_activation_with_biases(I, odtype):
    from turboquant_cpp_b200.kernels import elementwise as K
    rng = np.random.default_rng(I)
    gu, b = host(dev(rng.standard_normal((7, 2 * I)) * 2)), host(dev(rng.standard_normal(2 * I)))
    for bias in (b, None):
        z = gu if bias is None else gu + bias
        out = K.glu_mul(dev(gu), torch.full((7, I), float("nan"), dtype=odtype, device=DEV), bias=None if bias is None else dev(bias))
        assert rel(out, P.silu(z[:, :I]) * z[:, I:]) < (1e-5 if odtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("H", [37, 48, 2048, 4100])
@pytest.mark.parametrize("wdtype,odtype", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)])
def test_norms_on_outputs_with_a_bias_and_of_weighted_branches(H, wdtype, odtype):
    from turboquant_cpp_b200.kernels import elementwise as K
    rng = np.random.default_rng(H)
    R, eps, neps = 5, 2e-4, 3e-5
    x, a, b, y = (host(dev(rng.standard_normal((R, H)))) for _ in range(4))
    bias = host(dev(rng.standard_normal(H)))
    w, wn, wa, wb = (host(dev(1 + 0.3 * rng.standard_normal(H), wdtype)) for _ in range(4))
    d = lambda t: dev(t, wdtype)
    tol = 1e-5 if odtype == torch.float32 else 8e-3
    # the closing projection's bias under the norm
    xd, nxt = dev(x), torch.empty((R, H), dtype=odtype, device=DEV)
    K.add_rmsnorm(xd, dev(y), d(w), eps, None, d(wn), nxt, neps, y_bias=dev(bias))
    new = x + P.unit_rms(y + bias, eps) * w
    assert rel(xd, new) < 1e-5 and rel(nxt, P.unit_rms(new, neps) * wn) < tol
    # two branches with factors, as they are and normed
    for norms in (False, True):
        fa, fb = 0.7, -1.4
        m = fa * (P.unit_rms(a, 1e-4) * wa if norms else a) + fb * (P.unit_rms(b, 1e-4) * wb if norms else b)
        new = x + P.unit_rms(m, eps) * w
        xd, nxt = dev(x), torch.empty((R, H), dtype=odtype, device=DEV)
        args = (d(wa), dev(b), d(wb)) if norms else (None, dev(b), None)
        K.add_rmsnorm_pair(xd, dev(a), *args, 1e-4, d(w), eps, None, d(wn), nxt, neps, factors=(fa, fb))
        assert rel(xd, new) < 1e-5 and rel(nxt, P.unit_rms(new, neps) * wn) < tol
        out = K.mean_of_norms(dev(a), *args, 1e-4, torch.empty((R, H), device=DEV), factors=(fa, fb))
        assert rel(out, m) < 1e-5
