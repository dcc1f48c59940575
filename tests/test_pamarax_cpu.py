"""Parts of the Pamarax decoder that need no GPU: the configuration reader, the model's plan of tensors, cache and state
needs, frequencies, and the plain implementation's own consistency."""
import copy

import numpy as np
import pytest

from pamarax_util import CONFIGS, make_weights, tensor_shapes, write_folder
from plain import pamarax_plain as P


def test_the_models_plan_names_every_tensor_with_its_shape():
    import turboquant_cpp_b200 as tq
    for name, cfg in CONFIGS.items():
        plan = {s.name: tuple(s.shape) for s in tq.build_model(cfg, "bfloat16").weight_specs()}
        assert plan == tensor_shapes(cfg), name


def test_cache_and_state_needs_follow_the_layers():
    import turboquant_cpp_b200 as tq
    model = tq.build_model(CONFIGS["a"], "float32")
    # attention: a row of key and value per key/value head, nothing given back; the memory: S and n of every head and m;
    # side by side: rows and, behind the convolution's kept inputs, the delta rule's state
    assert [(n.window, n.planes, n.n_kv_heads, n.head_dim) if n else None for n in model.cache_needs()] == \
        [(0, 1, 2, 32), None, (0, 1, 2, 32), None, (0, 1, 1, 16)]
    assert [s.shape if s else None for s in model.state_needs()] == \
        [None, (3 * 13 * 8 + 3,), (2 * (2 * 2 * 8 + 4 * 12) + 4 * 12 * 8,), (2 * 7 * 20 + 2,), (1 * (2 * 2 * 16 + 2 * 8) + 2 * 8 * 16,)]
    assert model.capturable() and all(e.cache_of is None for e in model.schedule)
    assert set(model.kernels()) == {"elementwise", "bias_attention", "ssm"}


def test_optional_keys_may_be_missing():
    import turboquant_cpp_b200 as tq
    cfg = copy.deepcopy(CONFIGS["a"])
    cfg.pop("embedding")
    cfg["layers"][0]["mixer"].pop("rot")
    cfg["layers"][0]["mixer"].pop("vdim")
    cfg["layers"][2]["mixer"]["left"].pop("q_temp")
    model = tq.build_model(cfg, "float32")
    assert model.embedding.scale == 1.0 and model.blocks[0].mixer.position is None and model.blocks[2].mixer.left.temperature is None


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].__setitem__("type", "mamba2"), "type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 18), "dims"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("vdim", 8), "vdim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("gate_cap", 0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("dim", 300), "dim"),
    (lambda c: c["layers"][2]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][2]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][2]["mixer"]["left"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda c: c["layers"][2]["mixer"]["left"].__setitem__("vdim", 257), "vdim"),
    (lambda c: c["layers"][2]["mixer"]["right"].__setitem__("conv", 9), "conv"),
    (lambda c: c["layers"][2]["mixer"]["right"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "kind"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_a_configuration_that_cannot_run_is_refused_with_the_key(change, word):
    import turboquant_cpp_b200 as tq
    cfg = copy.deepcopy(CONFIGS["a"])
    change(cfg)
    with pytest.raises(tq.ConfigError) as e:
        tq.build_model(cfg, "float32")
    assert word in str(e.value)


def test_plain_decoding_by_recomputation_is_causal(tmp_path):
    """The plain model has no cache: the logits of a prefix are the first rows of the logits of the whole."""
    cfg = CONFIGS["a"]
    m = P.PlainPamarax(write_folder(str(tmp_path / "m"), cfg, make_weights(cfg, 1)))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 40).tolist()
    assert np.abs(m.forward(toks)[:25] - m.forward(toks[:25])).max() < 1e-9


def test_the_plain_recurrences_continue_from_a_state():
    rng = np.random.default_rng(2)
    T, dk, dv = 30, 6, 5
    q, k, v = rng.standard_normal((T, dk)), rng.standard_normal((T, dk)), rng.standard_normal((T, dv))
    beta, decay, i, f = rng.random(T), rng.random(T), 3 * rng.standard_normal(T), P.log_sigmoid(3 * rng.standard_normal(T))
    whole, S = P.gated_delta_rule(q, k, v, beta, decay)
    first, S1 = P.gated_delta_rule(q[:11], k[:11], v[:11], beta[:11], decay[:11])
    rest, S2 = P.gated_delta_rule(q[11:], k[11:], v[11:], beta[11:], decay[11:], S=S1)
    assert np.abs(np.concatenate([first, rest]) - whole).max() < 1e-12 and np.abs(S2 - S).max() < 1e-12
    whole, end = P.memory_recurrence(q, k, v, i, f)
    first, st = P.memory_recurrence(q[:11], k[:11], v[:11], i[:11], f[:11])
    rest, end2 = P.memory_recurrence(q[11:], k[11:], v[11:], i[11:], f[11:], start=st)
    assert np.abs(np.concatenate([first, rest]) - whole).max() < 1e-12 and np.abs(end[0] - end2[0]).max() < 1e-12 and end[2] == end2[2]


def test_the_running_maximum_of_the_plain_memory_only_scales():
    """Without the floor of 1e-6 the outputs are those of the recurrence without a maximum, S <- e^f S + e^i k v^T with
    |n . q| or one below."""
    rng = np.random.default_rng(3)
    T, dk, dv = 25, 4, 3
    q, k, v = rng.standard_normal((T, dk)), rng.standard_normal((T, dk)), rng.standard_normal((T, dv))
    i, f = 2 * rng.standard_normal(T), P.log_sigmoid(2 * rng.standard_normal(T))
    got, _ = P.memory_recurrence(q, k, v, i, f)
    S, n = np.zeros((dk, dv)), np.zeros(dk)
    for t in range(T):
        S = np.exp(f[t]) * S + np.exp(i[t]) * np.outer(k[t], v[t])
        n = np.exp(f[t]) * n + np.exp(i[t]) * k[t]
        want = (S.T @ q[t]) / max(abs(n @ q[t]), 1.0)
        assert np.abs(got[t] - want).max() < 1e-3 * max(1.0, np.abs(want).max())
