"""Parts of the Vukotar decoder that need no GPU: the configuration reader, the model's plan of tensors, the schedule of
layers that share weights, cache needs, position frequencies, and the plain implementation's own consistency."""
import copy
import math

import numpy as np
import pytest

from plain import vukotar_plain as P
from vukotar_util import CONFIGS, attention, config, layer, make_weights, moe, tensor_shapes, write_folder


def test_the_models_plan_names_every_tensor_with_its_shape():
    import turboquant_cpp_b200 as tq
    for name, cfg in CONFIGS.items():
        specs = tq.build_model(cfg, "bfloat16").weight_specs()
        assert {s.name: tuple(s.shape) for s in specs if not s.optional} == tensor_shapes(cfg), name
        # the factor of a feed-forward that a layer does not have may be stored or not
        assert [s.name for s in specs if s.optional] == (["l1.ls2"] if name == "a" else [])


def test_a_tensor_nothing_reads_may_be_left_out_and_any_other_may_not():
    import torch
    import turboquant_cpp_b200 as tq
    from turboquant_cpp_b200.weights import WeightError, check_plan
    specs = tq.build_model(CONFIGS["a"], "bfloat16").weight_specs()
    index = {n: (torch.bfloat16, s) for n, s in tensor_shapes(CONFIGS["a"]).items()}
    check_plan(index, specs)
    check_plan(dict(index, **{"l1.ls2": (torch.bfloat16, (CONFIGS["a"]["width"],))}), specs)
    with pytest.raises(WeightError, match="l1.ls2"):
        check_plan(dict(index, **{"l1.ls2": (torch.bfloat16, (3,))}), specs)
    with pytest.raises(WeightError, match="l0.ls2"):
        check_plan({n: v for n, v in index.items() if n != "l0.ls2"}, specs)


def test_layers_that_share_weights_run_one_block_with_caches_of_their_own():
    import turboquant_cpp_b200 as tq
    m = tq.build_model(CONFIGS["a"], "float32")
    assert len(m.blocks) == 3 and [e.block for e in m.schedule] == [0, 1, 0, 2, 1]
    assert all(e.cache_of is None for e in m.schedule)
    assert [(n.n_kv_heads, n.head_dim, n.window, n.planes) for n in m.cache_needs()] == \
        [(2, 96, 0, 1), (2, 96, 0, 1), (2, 96, 0, 1), (4, 32, 0, 1), (2, 96, 0, 1)]
    assert all(s is None for s in m.state_needs()) and m.capturable()
    m = tq.build_model(CONFIGS["c"], "float32")                  # ahead of the layer named, and through another one
    assert len(m.blocks) == 2 and [e.block for e in m.schedule] == [0, 0, 0, 1]
    assert m.blocks[0].norm.name == "l1.norm1" and m.blocks[1].norm.name == "l3.norm1"


def test_constants_come_from_the_configuration():
    import turboquant_cpp_b200 as tq
    cfg = config([layer(attention(scale=0.77), moe(groups=(4, 3), experts=8, top=2))], scale=0.125, cap=3.5)
    m = tq.build_model(cfg, "float32")
    assert m.embedding.scale == 0.125 and m.head.softcap == 3.5 and m.head.name == "embed"
    b = m.blocks[0]
    assert b.mixer.scale == 0.77 and b.mixer.window == 0 and b.mixer.has_sink and b.mixer.bias_rows == 0
    assert (b.ffn.n_groups, b.ffn.keep_groups, b.ffn.group_top, b.ffn.sigmoid, b.ffn.gated) == (4, 3, 2, True, False)
    m = tq.build_model(CONFIGS["b"], "float32")
    assert m.embedding.scale == 1.0 and m.head.softcap == 0.0 and m.blocks[0].ffn.n_groups == 1


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].__setitem__("type", "window"), "type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("dim", 257), "dim"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 13), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("keep", 4), "kept"),
    (lambda c: c["layers"][3]["mlp"]["router"].update(top=5), "choices"),
    (lambda c: c["layers"][2].__setitem__("weights_of", 3), "weights_of"),
    (lambda c: c["layers"][2].__setitem__("weights_of", 9), "weights_of"),
    (lambda c: c["layers"][2].__setitem__("weights_of", 2), "weights_of"),
    (lambda c: c.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_a_configuration_that_cannot_run_is_refused_with_the_key(change, word):
    import turboquant_cpp_b200 as tq
    cfg = copy.deepcopy(CONFIGS["a"])
    change(cfg)
    with pytest.raises(tq.ConfigError) as e:
        tq.build_model(cfg, "float32")
    assert word in str(e.value)


def test_two_layers_that_name_each_other_are_refused():
    import turboquant_cpp_b200 as tq
    cfg = config([layer(attention(), weights_of=1), layer(attention(), weights_of=0), layer(attention())])
    with pytest.raises(tq.ConfigError, match="weights_of"):
        tq.build_model(cfg, "float32")


@pytest.mark.parametrize("width", [1, 2, 37, 64])
def test_position_steps_are_the_plain_frequencies(width):
    from turboquant_cpp_b200.models.decoder import position_turns
    turns = position_turns(width, 10000.0).numpy()
    assert turns.shape == ((width + 1) // 2,)
    for p in (0, 1, 5, 4097):
        want = P.position_vector(p, width)
        ang = 2.0 * math.pi * p * turns
        got = np.stack([np.sin(ang), np.cos(ang)], axis=1).reshape(-1)[:width]
        assert np.abs(got - want).max() < 1e-11


def test_plain_logits_of_a_prefix_are_the_first_rows_of_the_whole(tmp_path):
    cfg = CONFIGS["a"]
    m = P.PlainVukotar(write_folder(str(tmp_path / "m"), cfg, make_weights(cfg, 1)))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 30).tolist()
    assert np.abs(m.forward(toks)[:19] - m.forward(toks[:19])).max() < 1e-9


def test_the_plain_sink_takes_its_share_and_the_plain_router_ranks_groups_by_their_two_best():
    p = P.sink_softmax(np.array([0.0, 0.0, 0.0]))
    assert np.allclose(p, 0.25)                                               # three keys and the one
    assert P.sink_softmax(np.array([-800.0]))[0] == 0.0 and abs(P.sink_softmax(np.array([800.0]))[0] - 1.0) < 1e-12
    # the best single expert sits in group 0, the best pair in group 1
    z = np.array([3.0, -9.0, -9.0, 1.0, 1.2, -9.0])
    ids, w, s, _ = P.route_row(z, {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert sorted(ids) == [3, 4] and abs(w.sum() - 1.0) < 1e-12 and np.allclose(w, s[ids] / s[ids].sum())
    ids, _, _, _ = P.route_row(z, {"experts": 6, "top": 2})
    assert sorted(ids) == [0, 4]
