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
