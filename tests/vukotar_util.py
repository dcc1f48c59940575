"""Helpers of the Vukotar tests: small configurations and model folders with weights made for the test."""
import numpy as np

from lumevik_util import check_against_plain, run_steps_with_routing      # noqa: F401  (schedules, the engine's expert choices)
from nuforax_util import write_folder                                     # noqa: F401


def attention(heads=6, kv_heads=2, dim=32, vdim=64, scale=0.3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}


def moe(experts=12, top=3, groups=(3, 2), ff=24):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(mixer, mlp=None, weights_of=None):
    out = {"type": "attention", "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def config(layers, vocab=97, width=48, eps=3e-5, scale=5.0, cap=11.0):
    out = {"architecture": "Vukotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        out["embedding"] = {"scale": scale}
    if cap is not None:
        out["logit_softcap"] = cap
    return out


# Configurations that differ in every size, in the order and sharing of layers, and in the options.
CONFIGS = {
    # grouped heads, values wider than keys, a layer without feed-forward, both kinds used a second time, layers of
    # several sizes in one model
    "a": config([layer(attention(), moe()), layer(attention()), layer(attention(), moe(), weights_of=0),
                 layer(attention(heads=4, kv_heads=4, dim=16, vdim=16, scale=0.5), moe(experts=8, top=2, groups=(4, 2), ff=40)),
                 layer(attention(), weights_of=1)]),
    # odd sizes (no 16-byte rows, no tensor-core shapes), a key/value head per head, no groups, one expert a token,
    # neither cap nor embedding factor
    "b": config([layer(attention(heads=3, kv_heads=3, dim=10, vdim=7, scale=1.0), moe(experts=5, top=1, groups=None, ff=21)),
                 layer(attention(heads=2, kv_heads=1, dim=9, vdim=20, scale=-0.7), moe(experts=7, top=4, groups=None, ff=13)),
                 layer(attention(heads=3, kv_heads=3, dim=10, vdim=7, scale=1.0), moe(experts=5, top=1, groups=None, ff=21), weights_of=0)],
                vocab=61, width=37, scale=None, cap=None),
    # one key/value head for eight, the sharing layer ahead of the one it names, a layer named through another one,
    # groups of one expert, wide key rows
    "c": config([layer(attention(heads=8, kv_heads=1, dim=64, vdim=32, scale=0.2), moe(experts=6, top=3, groups=(6, 4), ff=32), weights_of=1),
                 layer(attention(heads=8, kv_heads=1, dim=64, vdim=32, scale=0.2), moe(experts=6, top=3, groups=(6, 4), ff=32)),
                 layer(attention(heads=8, kv_heads=1, dim=64, vdim=32, scale=0.2), moe(experts=6, top=3, groups=(6, 4), ff=32), weights_of=0),
                 layer(attention(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.1), moe(experts=20, top=4, groups=(2, 1), ff=16))],
                vocab=128, width=64, scale=2.5, cap=6.0),
}


def tensor_shapes(cfg):
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "final.norm.b": (W,), "final.norm.alpha": ()}
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"], out[p + "norm1.b"], out[p + "norm1.alpha"], out[p + "ls1"] = (W,), (W,), (), (W,)
        q = p + "mix."
        out[q + "q"], out[q + "k"] = (m["heads"] * m["dim"], W), (m["kv_heads"] * m["dim"], W)
        out[q + "v"], out[q + "o"] = (m["kv_heads"] * m["vdim"], W), (W, m["heads"] * m["vdim"])
        if l["mlp"] is not None:
            out[p + "ls2"] = (W,)
            out[p + "mlp.router"] = (l["mlp"]["router"]["experts"], W)
            for e in range(l["mlp"]["router"]["experts"]):
                out[f"{p}mlp.e{e}.up"] = (l["mlp"]["expert"]["ff"], W)
                out[f"{p}mlp.e{e}.down"] = (W, l["mlp"]["expert"]["ff"])
    return out


def make_weights(cfg, seed, sharp=1.5):
    """Random weights with magnitudes that keep every mechanism visible: norm weights around 1 with biases, layer factors
    of both signs around 1, router rows that spread the scores.  `sharp` scales the query projections."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf == "alpha":
            w = np.asarray(0.3 + 0.5 * rng.random())
        elif leaf == "b":
            w = 0.3 * rng.standard_normal(shape)
        elif leaf in ("norm1", "norm"):
            w = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf in ("ls1", "ls2"):
            w = 0.8 + 0.5 * rng.standard_normal(shape)
        elif name == "embed":
            w = rng.standard_normal(shape) * 0.6
        elif leaf == "router":
            w = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])
        else:
            w = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if leaf == "q":
                w = w * sharp
        out[name] = np.asarray(w, dtype=np.float32)
    return out
