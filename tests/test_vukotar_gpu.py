"""The Vukotar decoder in the engine against the plain implementation (tests/plain/vukotar_plain.py): whole prompts,
decoding token by token, prompts in portions, batches of unequal requests, pages and slots used again, far tokens, layers
that share weights, other sizes, generation through the entry point, and trace replay as a user runs it."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from conftest import ROOT
from plain.vukotar_plain import PlainVukotar
from replay_util import batched, whole, with_tail
from vukotar_util import (CONFIGS, attention, check_against_plain, config, layer, make_weights, moe, run_steps_with_routing,
                          write_folder)

pytestmark = pytest.mark.gpu

_plain = {}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_folder(str(tmp_path_factory.mktemp(f"vukotar_{name}")), cfg, make_weights(cfg, 700 + i))
            for i, (name, cfg) in enumerate(CONFIGS.items())}


def plain_model(folder):
    if folder not in _plain:
        _plain[folder] = PlainVukotar(folder)
    return _plain[folder]


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def engine_for(folder, dtype, max_tokens=1024, **kw):
    import turboquant_cpp_b200 as tq
    return tq.Engine(tq.load_model(folder, dtype), max_tokens=max_tokens, record_routing=True, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_decoding_and_batches_agree_with_plain(folders, name, dtype):
    cfg, folder = CONFIGS[name], folders[name]
    reqs = {"r0": tokens_for(cfg, 100, 1), "r1": tokens_for(cfg, 1, 2), "r2": tokens_for(cfg, 57, 3), "r3": tokens_for(cfg, 140, 4)}
    eng = engine_for(folder, dtype, max_tokens=64 * 12)
    try:
        modes = {}
        steps, ends = [], {}
        for rid, toks in reqs.items():                        # each alone and whole, one after another
            s, e = whole(rid, toks)
            ends.update({k + len(steps): v for k, v in e.items()})
            steps += s
        modes["whole"] = run_steps_with_routing(eng, steps, ends)
        steps, ends = [], {}
        for rid, toks in reqs.items():                        # the last 50 tokens one by one
            s, e = with_tail(rid, toks, 50)
            ends.update({k + len(steps): v for k, v in e.items()})
            steps += s
        modes["tail"] = run_steps_with_routing(eng, steps, ends)
        s, e = batched(reqs, {"r0": 70, "r1": 1, "r2": 40, "r3": 129})      # unequal prompts, then decoded together
        modes["batched"] = run_steps_with_routing(eng, s, e)
        eng.cache.book.check_invariants()
        assert eng.cache.book.slots.n_held == 0 and all(p.n_held == 0 for p in eng.cache.book.pools)
        for rid, toks in reqs.items():
            for mode, (got, routing) in modes.items():
                assert sorted(got[rid]) == list(range(len(toks))), f"{mode} {rid}"
                check_against_plain(plain_model(folder), toks, got[rid], routing[rid], dtype, f"{name} {mode} {rid}")
    finally:
        eng.release()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,sizes", [("a", (2, 3, 50, 2, 64, 9)), ("b", (63, 2, 2, 65)), ("c", (17, 2, 2, 47, 30))])
def test_prompts_in_portions(folders, name, sizes, dtype):
    """A prompt cut into portions, down to two tokens, beside a request that goes on token by token: positions go on from
    portion to portion, and every layer finds its keys."""
    cfg, folder = CONFIGS[name], folders[name]
    toks, other = tokens_for(cfg, sum(sizes), 7), tokens_for(cfg, len(sizes) + 20, 8)
    eng = engine_for(folder, dtype)
    try:
        steps, at = [], 0
        for i, n in enumerate(sizes):
            step = [("p", toks[at:at + n], list(range(n)))]
            step.append(("o", other[:21], list(range(21))) if i == 0 else ("o", [other[20 + i]], [0]))
            steps.append(step)
            at += n
        got, routing = run_steps_with_routing(eng, steps, {len(steps) - 1: ["p", "o"]})
        check_against_plain(plain_model(folder), toks, got["p"], routing["p"], dtype, f"{name} portions")
        check_against_plain(plain_model(folder), other, got["o"], routing["o"], dtype, f"{name} beside portions")
    finally:
        eng.release()


def test_slots_and_pages_used_again_carry_nothing_over(folders):
    """A request run after others have ended gets their slot and pages; its logits are those of a fresh engine."""
    cfg, folder = CONFIGS["a"], folders["a"]
    eng = engine_for(folder, "float32", max_tokens=64 * 4, max_slots=2)
    try:
        a, b, c = tokens_for(cfg, 130, 11), tokens_for(cfg, 90, 12), tokens_for(cfg, 140, 13)
        run_steps_with_routing(eng, *batched({"a": a, "b": b}, {"a": 100, "b": 80}))
        got, routing = run_steps_with_routing(eng, *with_tail("c", c, 30))
        check_against_plain(plain_model(folder), c, got["c"], routing["c"], "float32", "after reuse")
        eng.cache.book.check_invariants()
    finally:
        eng.release()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    """250 tokens decoded one by one from a 3-token prompt through replayed graphs (both streams inside them)."""
    cfg, folder = CONFIGS["c"], folders["c"]
    toks = tokens_for(cfg, 253, 21)
    eng = engine_for(folder, dtype)
    try:
        got, routing = run_steps_with_routing(eng, *with_tail("x", toks, 250))
        assert eng.graphs is not None and eng.graphs.replays >= 240
        check_against_plain(plain_model(folder), toks, got["x"], routing["x"], dtype, "long decoding")
    finally:
        eng.release()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoding_in_growing_batches(folders, dtype):
    """One to twelve requests decoded together: every form of the decode router and of the token attention."""
    cfg, folder = CONFIGS["a"], folders["a"]
    for n in (1, 2, 5, 12):
        reqs = {f"r{i}": tokens_for(cfg, 12 + 3 * i, 60 + i) for i in range(n)}
        eng = engine_for(folder, dtype, max_tokens=64 * 16, max_slots=16)
        try:
            got, routing = run_steps_with_routing(eng, *batched(reqs, {r: 6 + 3 * i for i, r in enumerate(reqs)}))
            for rid, toks in reqs.items():
                check_against_plain(plain_model(folder), toks, got[rid], routing[rid], dtype, f"{n} together, {rid}")
        finally:
            eng.release()


VARIANTS = {
    # everything one
    "ones": ([layer(attention(heads=1, kv_heads=1, dim=1, vdim=1), moe(experts=1, top=1, groups=None, ff=1))], 4),
    # no feed-forward anywhere
    "attention_alone": ([layer(attention()), layer(attention(heads=1, kv_heads=1, dim=8, vdim=16)), layer(attention(), weights_of=0)], 36),
    # all experts of every token; as many kept groups as there are
    "all_chosen": ([layer(attention(), moe(experts=6, top=6, groups=(2, 2), ff=10))], 36),
    # more experts than the width (the separate router kernels), heads of 200
    "many_experts": ([layer(attention(heads=2, kv_heads=1, dim=200, vdim=180, scale=0.1), moe(experts=72, top=5, groups=(9, 3), ff=8))], 40),
    # sixteen heads on one, sizes of the tensor-core kernels
    "wide_group": ([layer(attention(heads=16, kv_heads=1, dim=64, vdim=64, scale=0.2), moe(experts=16, top=2, groups=(4, 1), ff=72))], 80),
    # one layer's weights six times over
    "looped": ([layer(attention(heads=4, kv_heads=2, dim=16, vdim=8), moe(experts=4, top=1, groups=(2, 1), ff=12))] +
               [layer(attention(heads=4, kv_heads=2, dim=16, vdim=8), moe(experts=4, top=1, groups=(2, 1), ff=12), weights_of=0)] * 5, 24),
}


@pytest.mark.parametrize("variant", sorted(VARIANTS))
def test_other_sizes_and_options(tmp_path, variant):
    layers, width = VARIANTS[variant]
    cfg = config(layers, vocab=50, width=width, scale=3.0, cap=20.0)
    folder = write_folder(str(tmp_path / variant), cfg, make_weights(cfg, 5))
    toks = tokens_for(cfg, 150, 31)
    for dtype in ("float32", "bfloat16"):
        eng = engine_for(folder, dtype)
        try:
            got, routing = run_steps_with_routing(eng, *with_tail("x", toks, 40))
            check_against_plain(plain_model(folder), toks, got["x"], routing.get("x", []), dtype, variant)
        finally:
            eng.release()


def test_a_wrong_constant_a_lost_key_or_a_shared_cache_would_show(folders, tmp_path):
    """The tests above mean something only if the plain model itself reacts to these faults by far more than the
    tolerance: positions off by one, another embedding factor, cap or score scale, no sink, factors per element left
    out, groups worth their single best, a layer's first key lost."""
    from plain import vukotar_plain as P
    cfg, folder = CONFIGS["a"], folders["a"]
    toks = tokens_for(cfg, 60, 1)
    w = P.load(folder)[1]
    ref = P.forward(cfg, w, toks)

    def moved(c, weights=w, at=slice(None)):
        return np.abs(P.forward(c, weights, toks) - ref)[at].max() / ref.std()

    for edit in (lambda c: c["embedding"].update(scale=5.2), lambda c: c.update(logit_softcap=11.5),
                 lambda c: c["layers"][0]["mixer"].update(scale=0.31)):
        c = copy.deepcopy(cfg)
        edit(c)
        assert moved(c) > 1e-2
    for leaf in ("l0.ls1", "l0.ls2", "l1.ls1", "l0.norm1.b"):
        assert moved(cfg, dict(w, **{leaf: np.ones_like(w[leaf])})) > 1e-2, leaf
    saved = P.position_vector, P.sink_softmax, P.attention_core, P.route_row
    try:
        P.position_vector = lambda p, width: saved[0](p + 1, width)
        assert moved(cfg) > 1e-2
        P.position_vector = saved[0]
        P.sink_softmax = lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum()
        assert moved(cfg) > 1e-2
        P.sink_softmax = saved[1]
        P.attention_core = lambda q, k, v, scale: saved[2](q, k, np.concatenate([0 * v[:1], v[1:]]), scale)
        assert moved(cfg, at=slice(1, None)) > 1e-2
        P.attention_core = saved[2]
        P.route_row = lambda z, r: saved[3](z, {k: v for k, v in r.items() if k != "groups"})
        assert moved(cfg) > 1e-2
    finally:
        P.position_vector, P.sink_softmax, P.attention_core, P.route_row = saved


def test_a_far_token_reaches_through_every_page(tmp_path):
    """400 tokens back, through a key that stands out: the plain logits at the end change with the first token, and the
    engine follows that change in a prompt, in decoding and across portions."""
    cfg = config([layer(attention(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.0), moe(experts=4, top=1, groups=(2, 1), ff=16)),
                  layer(attention(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.0), moe(experts=4, top=1, groups=(2, 1), ff=16), weights_of=0)],
                 vocab=40, width=32, scale=3.0, cap=25.0)
    w = make_weights(cfg, 9)
    w["l0.mix.q"] = w["l0.mix.q"] * 0.05                                  # flat weights: every far token counts a little
    folder = write_folder(str(tmp_path / "far"), cfg, w)
    a = tokens_for(cfg, 400, 3)
    b = [(a[0] + 7) % cfg["vocab"]] + a[1:]
    plain = plain_model(folder)
    ra, rb = plain.forward(a), plain.forward(b)
    moved = np.abs(ra[-1] - rb[-1]).max() / ra.std()
    assert moved > 2e-4, f"the first token does not reach the last position ({moved:.1e})"
    eng = engine_for(folder, "float32")
    try:
        for toks, ref in ((a, ra), (b, rb)):
            portions = ([[("x", toks[:65], [])], [("x", toks[65:330], [])], [("x", toks[330:], [69])]], {2: ["x"]})
            for sched in (whole("x", toks, keep={399}), with_tail("x", toks, 90, keep={0}), portions):
                got, _ = run_steps_with_routing(eng, *sched)
                e = np.abs(got["x"][399] - ref[399]).max() / ra.std()
                assert e < moved / 20, f"the last position is off by {e:.1e}, the far token moves it by {moved:.1e}"
    finally:
        eng.release()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(folders, dtype):
    import turboquant_cpp_b200 as tq
    cfg, folder = CONFIGS["a"], folders["a"]
    prompts = [tokens_for(cfg, n, 40 + n) for n in (1, 9, 40, 70)]
    n_new = 12
    with tq.Model(folder, temperature=0.0, max_tokens=n_new, dtype=dtype, max_batch=4, context_length=128) as m:
        outs = m.generate_batch(prompts)
        again = m.generate_batch(prompts[::-1])[::-1]                 # another order in the batch, slots used again
        alone = [m.ask(p) for p in prompts]
        if dtype == "float32":                                        # (bfloat16: a close call of the router may fall either way)
            assert again == outs and alone == outs
        m.engine.cache.book.check_invariants()
        assert m.engine.cache.book.slots.n_held == 0
    plain = plain_model(folder)
    floor = 1e-4 if dtype == "float32" else 0.15
    for p, o in zip(prompts, outs):
        rec = []
        l = plain.forward(list(p) + o, routing=rec)
        for i, t in enumerate(o):
            at = len(p) - 1 + i
            top = np.sort(l[at])[-2:]
            if int(np.argmax(l[at])) != t:
                close = top[1] - top[0] < floor * l.std() or (dtype == "bfloat16" and min(r[2][:at + 1].min() for r in rec) < 2e-2)
                assert close, f"token {i}: engine {t}, plain {int(np.argmax(l[at]))}"


def test_command_line_and_trace_replay(folders, tmp_path):
    """The generation program on a folder and on random weights, and the replay program as a user runs it: steps on
    standard input, logits in files, a line per step."""
    cfg, folder = CONFIGS["c"], folders["c"]
    toks = tokens_for(cfg, 40, 77)
    env = dict(os.environ, PYTHONPATH=ROOT)
    import turboquant_cpp_b200 as tq
    quant = [sys.executable, os.path.join(ROOT, "bin", "quant")]
    common = ["-p", " ".join(map(str, toks[:9])), "-n", "5", "-T", "0", "--dtype", "float32"]
    out = subprocess.run(quant + [folder] + common, capture_output=True, text=True, env=env, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    with tq.Model(folder, temperature=0.0, max_tokens=5, dtype="float32") as m:
        assert [int(t) for t in out.stdout.split()] == m.ask(toks[:9])
    info = subprocess.run(quant + [folder, "--info"], capture_output=True, text=True, env=env, timeout=600)
    assert info.returncode == 0 and "Vukotar" in info.stdout
    json.dump(cfg, open(tmp_path / "cfg.json", "w"))
    run = subprocess.run(quant + ["--random", str(tmp_path / "cfg.json"), "--seed-weights", "3"] + common + ["--profile"],
                         capture_output=True, text=True, env=env, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert any(l.startswith("[Profile ") and "moe=" in l for l in run.stderr.splitlines())
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[32:], "want": [7]}], "end": ["x"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path / "o"),
                          "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, env=env, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(tmp_path / "o" / "1.f32")
    ref = plain_model(folder).forward(toks)
    got = np.concatenate([np.fromfile(tmp_path / "o" / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for s in (0, 2)])
    assert np.abs(got - ref[[0, 29, 39]]).max() < 1e-4 * ref.std()


@pytest.mark.parametrize("T", [1, 6, 40, 700])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ungated_experts_beside_a_shared_one(T, dtype):
    """The routed part with an option this design leaves out: a shared expert without a gate inside it (beside the routed
    experts on a second stream, its output weighted by a gate of its own)."""
    import types
    import torch
    from plain import vukotar_plain as P
    from turboquant_cpp_b200.parts import ExpertRows, make_feed_forward
    from turboquant_cpp_b200.weights import RandomSource, WeightStore
    H, E, k, I, S = 64, 10, 3, 24, 72
    names = {"router": "router", "expert": "e{e}.", "up": "up", "down": "down", "shared": "sh.", "shared_gate": "sg"}
    run = torch.float32 if dtype == "float32" else torch.bfloat16
    for shared in (S, 0):
        ff = make_feed_forward("moe", prefix="f.", hidden=H, n_experts=E, top_k=k, intermediate=I, norm_topk=True,
                               shared_intermediate=shared, n_groups=5, keep_groups=3, group_top=2, scores="sigmoid",
                               renorm_floor=P.WEIGHT_FLOOR, gated=False, names=names)
        specs = ff.weight_specs()
        store = WeightStore(RandomSource(specs, 4, std=0.2), specs, "cuda:0", run)
        w = {s.name: store.get(s.name).double().cpu().numpy() for s in specs}
        assert not any("gate" in n for n in w)
        ff.bind(store)
        x = torch.randn(T, H, device="cuda:0").to(run)
        ctx = types.SimpleNamespace(act_dtype=run, debug={}, status=None)
        y = ff.forward(x, ctx)
        h, ids = x.double().cpu().numpy(), ctx.debug["router_ids"][0].cpu().numpy()
        ml = {"router": {"experts": E, "top": k, "groups": {"count": 5, "keep": 3}}}
        rec = []
        P.experts(h, w, "f.", ml, record=rec)
        differ = np.any(np.sort(ids, axis=1) != np.sort(rec[0][0], axis=1), axis=1)
        assert rec[0][2][differ].max(initial=0.0) < 1e-5
        want = P.experts(h, w, "f.", ml, ids=ids)
        if shared:
            want += P.expert(h, w, "f.sh.") / (1.0 + np.exp(-(h @ w["f.sg"].T)))
        got = y.double().cpu().numpy()
        assert np.abs(got - want).max() < (1e-5 if dtype == "float32" else 2e-2) * np.abs(want).max()
        left = ff.forward(x, ctx, leave_rows=True)
        assert isinstance(left, ExpertRows) == (shared == 0)


def test_a_blocks_sum_left_open_or_not_and_the_two_streams_give_the_same(folders):
    """The block with its sum taken by the next norm, with a sum of its own, with the feed-forward behind the mixer on one
    stream, and with a norm that takes no open sum."""
    import torch
    import turboquant_cpp_b200 as tq
    from turboquant_cpp_b200.parts import ParallelBlock
    cfg, folder = CONFIGS["a"], folders["a"]
    toks = tokens_for(cfg, 70, 5)

    def logits(change, dtype="float32"):
        model = tq.load_model(folder, dtype)
        change(model)
        eng = tq.Engine(model, max_tokens=128)
        s = eng.open()
        out = eng.step([tq.StepEntry(s, toks, list(range(70)))])
        eng.close(s)
        eng.release()
        return out

    ref = logits(lambda m: None)

    def closed(m):
        for b in m.blocks:
            b.leave_open = False
    assert (logits(closed) - ref).abs().max().item() < 1e-5 * ref.abs().max().item()

    def other_norm(m):                                   # as if the norms that follow took sums of one tensor only
        for b in m.blocks:
            b.norm.adds_open_sums = False
    assert (logits(other_norm) - ref).abs().max().item() < 1e-5 * ref.abs().max().item()
    saved = ParallelBlock.SIDE_BY_SIDE, ParallelBlock.SIDE_MIN_ELEMENTS
    try:
        ParallelBlock.SIDE_MIN_ELEMENTS = 0                # two streams, whatever the step's size
        for _ in range(3):
            assert torch.equal(logits(lambda m: None), ref)
        ParallelBlock.SIDE_BY_SIDE = False
        assert torch.equal(logits(lambda m: None), ref)
    finally:
        ParallelBlock.SIDE_BY_SIDE, ParallelBlock.SIDE_MIN_ELEMENTS = saved
