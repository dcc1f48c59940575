"""The Pamarax decoder in the engine against the plain implementation (tests/plain/pamarax_plain.py): whole prompts,
decoding token by token, prompts in portions, batches of unequal requests, pages and slots used again, far tokens, other
sizes, generation through the entry point, and trace replay as a user runs it."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from conftest import ROOT
from pamarax_util import (CONFIGS, assert_close, attention, config, layer, left, make_weights, memory, parallel, right, run_steps,
                          write_folder)
from plain.pamarax_plain import PlainPamarax, keep, to_bfloat16
from replay_util import batched, whole, with_tail

pytestmark = pytest.mark.gpu

_plain, _logits = {}, {}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        out[name] = write_folder(str(tmp_path_factory.mktemp(f"pamarax_{name}")), cfg, make_weights(cfg, 700 + i, sharp=2.0))
    return out


def plain_logits(folder, toks, dtype="float32"):
    """The plain model's logits; for bfloat16 with activations rounded where the engine keeps them in that dtype (without
    that a tenth of the positions of these models move by 5e-2 of the logits' spread and more: norms on the sub-layers'
    outputs enlarge roundings)."""
    key = (folder, tuple(toks), dtype)
    if key not in _logits:
        if folder not in _plain:
            _plain[folder] = PlainPamarax(folder)
        _logits[key] = _plain[folder].forward(toks, store=to_bfloat16 if dtype == "bfloat16" else keep)
    return _logits[key]


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def engine_for(folder, dtype, max_tokens=1024, **kw):
    import turboquant_cpp_b200 as tq
    return tq.Engine(tq.load_model(folder, dtype), max_tokens=max_tokens, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_whole_prompts_decoding_and_batches_agree_with_plain(folders, name, dtype):
    cfg, folder = CONFIGS[name], folders[name]
    reqs = {"r0": tokens_for(cfg, 150, 1), "r1": tokens_for(cfg, 1, 2), "r2": tokens_for(cfg, 77, 3), "r3": tokens_for(cfg, 200, 4)}
    eng = engine_for(folder, dtype, max_tokens=64 * 12)
    try:
        modes = {}
        steps, ends = [], {}
        for rid, toks in reqs.items():                        # each alone and whole, one after another
            s, e = whole(rid, toks)
            ends.update({k + len(steps): v for k, v in e.items()})
            steps += s
        modes["whole"] = run_steps(eng, steps, ends)
        steps, ends = [], {}
        for rid, toks in reqs.items():                        # the last 80 tokens one by one
            s, e = with_tail(rid, toks, 80)
            ends.update({k + len(steps): v for k, v in e.items()})
            steps += s
        modes["tail"] = run_steps(eng, steps, ends)
        s, e = batched(reqs, {"r0": 100, "r1": 1, "r2": 64, "r3": 129})     # unequal prompts, then decoded together
        modes["batched"] = run_steps(eng, s, e)
        eng.cache.book.check_invariants()
        assert eng.cache.book.slots.n_held == 0 and all(p.n_held == 0 for p in eng.cache.book.pools)
        for rid, toks in reqs.items():
            for mode, got in modes.items():
                assert sorted(got[rid]) == list(range(len(toks))), f"{mode} {rid}"
                assert_close(got[rid], plain_logits(folder, toks, dtype), dtype, f"{name} {mode} {rid}")
    finally:
        eng.release()


@pytest.mark.parametrize("name,sizes", [("a", (2, 3, 50, 2, 64, 9)), ("b", (70, 2, 58, 2, 65)), ("c", (17, 2, 2, 2, 40))])
def test_prompts_in_portions(folders, name, sizes):
    """A prompt cut into portions, down to two tokens, beside a request that goes on token by token: the states, the
    maxima and the convolution's kept inputs pass from portion to portion."""
    cfg, folder = CONFIGS[name], folders[name]
    toks, other = tokens_for(cfg, sum(sizes), 7), tokens_for(cfg, len(sizes) + 20, 8)
    for dtype in ("float32", "bfloat16"):
        eng = engine_for(folder, dtype)
        try:
            steps, at = [], 0
            for i, n in enumerate(sizes):
                step = [("p", toks[at:at + n], list(range(n)))]
                if i == 0:
                    step.append(("o", other[:21], list(range(21))))
                else:
                    step.append(("o", [other[20 + i]], [0]))
                steps.append(step)
                at += n
            got = run_steps(eng, steps, {len(steps) - 1: ["p", "o"]})
            assert_close(got["p"], plain_logits(folder, toks, dtype), dtype, f"{name} portions")
            assert_close(got["o"], plain_logits(folder, other, dtype), dtype, f"{name} beside portions")
        finally:
            eng.release()


@pytest.mark.parametrize("name,sizes", [("a", [500]), ("b", [140, 300]), ("c", [333])])
def test_long_prompts_whose_memory_runs_in_chunks(folders, name, sizes, monkeypatch):
    """Runs long enough to be cut into chunks side by side, whole and in portions that go on from a kept state, beside a
    short request."""
    from turboquant_cpp_b200.parts import memory as part
    cfg, folder = CONFIGS[name], folders[name]
    toks, other = tokens_for(cfg, sum(sizes), 21), tokens_for(cfg, len(sizes) + 40, 22)
    cut, plan = [], part.cut_runs
    monkeypatch.setattr(part, "cut_runs", lambda *a: cut.append(plan(*a)) or cut[-1])
    eng = engine_for(folder, "float32")
    try:
        steps, at = [], 0
        for i, n in enumerate(sizes):
            step = [("p", toks[at:at + n], list(range(n)))]
            step.append(("o", other[:41], list(range(41))) if i == 0 else ("o", [other[40 + i]], [0]))
            steps.append(step)
            at += n
        got = run_steps(eng, steps, {len(steps) - 1: ["p", "o"]})
        assert any(c is not None for c in cut)
        assert_close(got["p"], plain_logits(folder, toks), "float32", f"{name} long prompt")
        assert_close(got["o"], plain_logits(folder, other), "float32", f"{name} beside a long prompt")
    finally:
        eng.release()


def test_slots_and_pages_used_again_carry_nothing_over(folders):
    """A request run after others have ended gets their slot and pages; its logits are those of a fresh engine."""
    cfg, folder = CONFIGS["a"], folders["a"]
    eng = engine_for(folder, "float32", max_tokens=64 * 4, max_slots=2)
    try:
        a, b, c = tokens_for(cfg, 130, 11), tokens_for(cfg, 90, 12), tokens_for(cfg, 140, 13)
        s1, e1 = batched({"a": a, "b": b}, {"a": 100, "b": 80})
        run_steps(eng, s1, e1)
        s2, e2 = with_tail("c", c, 30)
        got = run_steps(eng, s2, e2)
        assert_close(got["c"], plain_logits(folder, c), "float32", "after reuse")
        eng.cache.book.check_invariants()
    finally:
        eng.release()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    """300 tokens decoded one by one from a 3-token prompt: states and pages over many steps, graphs replayed."""
    cfg, folder = CONFIGS["b"], folders["b"]
    toks = tokens_for(cfg, 303, 21)
    eng = engine_for(folder, dtype, max_slots=1)                 # one slot: the states' rows have no stride to speak of
    try:
        s, e = with_tail("x", toks, 300)
        got = run_steps(eng, s, e)
        assert eng.graphs is not None and eng.graphs.replays >= 290
        assert_close(got["x"], plain_logits(folder, toks, dtype), dtype, "long decoding")
    finally:
        eng.release()


VARIANTS = {
    # everything one: one head, keys and values of one element, one tap, a temperature that grows with every position
    "ones": [layer("attention", attention(heads=1, kv_heads=1, dim=1, rot=None)),
             layer("mlstm", memory(heads=1, dim=1, vdim=1, gate_cap=1.0)),
             layer("parallel", parallel(left(heads=1, kv_heads=1, dim=1, vdim=1, temp=(1.0, 1)), right(heads=1, kv_heads=1, dim=1, vdim=1, conv=1),
                                        (1.0, 1.0)), ff=1)],
    # one kind of layer alone each, no feed-forward anywhere
    "memory_alone": [layer("mlstm", memory()), layer("mlstm", memory(heads=7, dim=5, vdim=3))],
    "attention_alone": [layer("attention", attention()), layer("attention", attention(heads=9, kv_heads=3, dim=12, rot=(12, 50.0)))],
    "parallel_alone": [layer("parallel", parallel()), layer("parallel", parallel(scales=(0.0, 1.0))), layer("parallel", parallel(scales=(1.0, 0.0)))],
    # sizes of the tensor-core kernels with sixteen query rows a key head, and keys of 128 beside values of 64
    "wide_groups": [layer("attention", attention(heads=16, kv_heads=1, dim=32, scale=0.2, rot=(32, 1e4)), ff=16),
                    layer("parallel", parallel(left(heads=16, kv_heads=1, dim=128, vdim=64, scale=0.1, temp=(0.1, 64)), right(heads=4, kv_heads=1)))],
    # keys of 256 elements in both recurrences and in attention, values that no block of columns divides
    "wide_state": [layer("mlstm", memory(heads=2, dim=256, vdim=33), ff=16),
                   layer("parallel", parallel(left(heads=2, kv_heads=1, dim=256, vdim=3), right(heads=2, kv_heads=1, dim=256, vdim=21, conv=5)))],
    # values much longer than keys
    "long_values": [layer("mlstm", memory(heads=1, dim=4, vdim=300), ff=8), layer("parallel", parallel(r=right(heads=2, kv_heads=1, dim=3, vdim=280)))],
    # odd sizes everywhere: width, heads, keys, feed-forward
    "odd_width": [layer("attention", attention(heads=3, kv_heads=1, dim=10, rot=(6, 77.0)), ff=11),
                  layer("parallel", parallel(left(heads=5, kv_heads=5, dim=3, vdim=7), right(heads=3, kv_heads=1, dim=5, vdim=9, conv=6)), ff=13),
                  layer("mlstm", memory(heads=5, dim=3, vdim=7), ff=7)],
}
WIDTHS = {"odd_width": 37}       # a stream no 16-byte access divides


@pytest.mark.parametrize("variant", sorted(VARIANTS))
def test_other_sizes_and_options(tmp_path, variant):
    cfg = config(VARIANTS[variant], vocab=50, width=WIDTHS.get(variant, 36), scale=5.0)
    folder = write_folder(str(tmp_path / variant), cfg, make_weights(cfg, 5, sharp=2.0))
    toks = tokens_for(cfg, 200, 31)
    for dtype in ("float32", "bfloat16"):
        eng = engine_for(folder, dtype)
        try:
            s, e = with_tail("x", toks, 40)
            got = run_steps(eng, s, e)
            assert_close(got["x"], plain_logits(folder, toks, dtype), dtype, variant)
        finally:
            eng.release()


def test_one_stream_or_two_give_the_same(folders, monkeypatch):
    """The branches of a parallel layer on one stream and beside each other on two, in prompts and in decoding."""
    from turboquant_cpp_b200.parts import ParallelMixer
    cfg, folder = CONFIGS["a"], folders["a"]
    toks = tokens_for(cfg, 120, 3)
    for on in (True, False):
        monkeypatch.setattr(ParallelMixer, "SIDE_BY_SIDE", on)
        monkeypatch.setattr(ParallelMixer, "SIDE_MIN_ELEMENTS", 1)
        eng = engine_for(folder, "float32")
        for b in eng.model.blocks:
            if isinstance(b.mixer, ParallelMixer):
                b.mixer.right.runs_alone = False
        try:
            got = run_steps(eng, *with_tail("x", toks, 40))
            assert_close(got["x"], plain_logits(folder, toks), "float32", f"two streams: {on}")
        finally:
            eng.release()


def test_a_wrong_constant_or_a_lost_state_would_show(folders, tmp_path):
    """The tests above mean something only if the plain model itself reacts to these faults: with the weights used here each
    of them moves the logits by far more than the tolerance."""
    cfg, folder = CONFIGS["a"], folders["a"]
    toks = tokens_for(cfg, 60, 1)
    ref = plain_logits(folder, toks)
    weights = make_weights(cfg, 700, sharp=2.0)

    def moved(change=None, w=None):
        wrong = copy.deepcopy(cfg)
        if change:
            change(wrong)
        f = write_folder(str(tmp_path / f"m{np.random.default_rng().integers(1 << 40)}"), wrong, w or weights)
        return np.abs(PlainPamarax(f).forward(toks) - ref)[26:].max() / ref.std()

    mix = lambda c, i: c["layers"][i]["mixer"]
    assert moved() < 1e-6
    assert moved(lambda c: mix(c, 0)["rot"].__setitem__("base", 6000.0)) > 1e-2
    assert moved(lambda c: mix(c, 1).__setitem__("gate_cap", 8.0)) > 1e-2
    assert moved(lambda c: mix(c, 2)["left"]["q_temp"].__setitem__("every", 23)) > 1e-3
    assert moved(lambda c: mix(c, 2).__setitem__("left_scale", 0.9)) > 1e-2
    assert moved(lambda c: c["embedding"].__setitem__("scale", 1.8)) > 1e-2
    for name in ("l1.mix.f.b", "l1.mix.i.b", "l1.mix.norm", "l2.mix.right.dt_bias", "l0.mlp.gate.b", "l0.mlp.down.b", "l0.norm1b", "l0.mix.k.norm"):
        w = dict(weights)
        w[name] = np.zeros_like(w[name]) if not name.endswith(".norm") else np.ones_like(w[name])
        assert moved(w=w) > 1e-2, name
    # a lost state: a portion run alone differs from the portion in place
    assert np.abs(PlainPamarax(folder).forward(toks[30:])[0] - ref[30]).max() > 1e-2 * ref.std()


def test_a_far_token_reaches_through_attention_and_through_both_states(tmp_path):
    """Hundreds of tokens back: the plain logits at the end change when the first token changes, and the engine follows that
    change through pages (attention) and through the recurrences' states, in prompts and in decoding."""
    kinds = {"attention": attention(heads=2, kv_heads=1, dim=16, scale=0.05),
             "mlstm": memory(heads=2, dim=16, vdim=8),
             "parallel": parallel(left(heads=2, kv_heads=1, dim=16, vdim=16, scale=0.05), right(heads=2, kv_heads=2, dim=16, vdim=8, conv=2), (0.0, 1.0))}
    for kind, mixer in kinds.items():
        cfg = config([layer(kind, mixer, ff=16)], vocab=40, width=32)
        w = make_weights(cfg, 9)
        if kind == "mlstm":
            w["l0.mix.f.b"] = np.full_like(w["l0.mix.f.b"], 8.0)                 # forget gates open
            w["l0.mix.f"] = w["l0.mix.f"] * 0.05
        if kind == "parallel":
            w["l0.mix.right.dt_bias"] = np.full_like(w["l0.mix.right.dt_bias"], -9.0)      # decays near one
            w["l0.mix.right.a"] = w["l0.mix.right.a"] * 0.05
        folder = write_folder(str(tmp_path / kind), cfg, w)
        a = tokens_for(cfg, 400, 3)
        b = [(a[0] + 7) % cfg["vocab"]] + a[1:]
        ra, rb = plain_logits(folder, a), plain_logits(folder, b)
        move = np.abs(ra[-1] - rb[-1]).max() / ra.std()
        assert move > 2e-4, f"{kind}: the first token does not reach the last position ({move:.1e})"
        eng = engine_for(folder, "float32")
        try:
            for toks, ref in ((a, ra), (b, rb)):
                for sched in (whole("x", toks, keep={399}), with_tail("x", toks, 90, keep={0})):
                    got = run_steps(eng, *sched)
                    e = np.abs(got["x"][399] - ref[399]).max() / ra.std()
                    assert e < move / 10, f"{kind}: the last position is off by {e:.1e}, the far token moves it by {move:.1e}"
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
        assert m.generate_batch(prompts[::-1])[::-1] == outs          # another order in the batch, slots used again
        assert [m.ask(p) for p in prompts] == outs                    # each alone
        m.engine.cache.book.check_invariants()
        assert m.engine.cache.book.slots.n_held == 0
    plain = PlainPamarax(folder)
    floor = 1e-4 if dtype == "float32" else 0.15
    for p, o in zip(prompts, outs):
        toks = list(p)
        for i, t in enumerate(o):
            l = plain.forward(toks)[-1]
            top = np.sort(l)[-2:]
            if int(np.argmax(l)) != t:
                assert top[1] - top[0] < floor * l.std(), f"token {i}: engine {t}, plain {int(np.argmax(l))}"
            toks.append(t)


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
    assert info.returncode == 0 and "Pamarax" in info.stdout
    json.dump(cfg, open(tmp_path / "cfg.json", "w"))
    res = subprocess.run(quant + ["--random", str(tmp_path / "cfg.json"), "--seed-weights", "3"] + common + ["--profile"],
                         capture_output=True, text=True, env=env, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert any(l.startswith("[Profile ") and "matmul=" in l for l in res.stderr.splitlines())
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[30:32], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[32:], "want": [7]}], "end": ["x"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path / "o"),
                          "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, env=env, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(tmp_path / "o" / "1.f32")
    ref = plain_logits(folder, toks)
    got0 = np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4").reshape(2, cfg["vocab"])
    got2 = np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4").reshape(1, cfg["vocab"])
    assert_close({0: got0[0], 29: got0[1], 39: got2[0]}, ref, "float32", "trace replay")
