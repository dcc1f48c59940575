"""Helpers of the Pamarax tests: small configurations and model folders with weights made for the test."""
import numpy as np

from nuforax_util import run_steps, spread_error, write_folder      # noqa: F401  (file writing, schedules)

# float32: sums of a few thousand terms in another order than float64.  bfloat16, against the plain model rounded where the
# engine rounds: single activations fall on the other side of a rounding, the tensor-core attention kernels also round the
# softmax's weights, and norms on the sub-layers' outputs enlarge both at single positions.
TOL = {"float32": (1e-5, 1e-4), "bfloat16": (2e-2, 0.3)}      # (nine positions in ten, every position)


def assert_close(got_rows, ref, dtype, what):
    """got_rows {position: row} against the plain logits ref [T, vocab] at those positions."""
    ps = sorted(got_rows)
    e = spread_error(np.stack([got_rows[p] for p in ps]), ref[ps])
    most, every = TOL[dtype]
    assert np.all(np.isfinite(e)), f"{what}: not finite"
    assert e.max() < every, f"{what}: position {ps[int(e.argmax())]} differs by {e.max():.3e} (tolerance {every:.0e})"
    assert np.quantile(e, 0.9) < most, f"{what}: a tenth of the positions differ by more than {np.quantile(e, 0.9):.3e}"


def memory(heads=3, dim=8, vdim=12, gate_cap=9.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def attention(heads=4, kv_heads=2, dim=16, scale=0.4, rot=(8, 5000.0)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def left(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.5, temp=(0.7, 24)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def right(heads=4, kv_heads=2, dim=8, vdim=12, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(l=None, r=None, scales=(0.8, 1.3)):
    return {"left": l or left(), "right": r or right(), "left_scale": scales[0], "right_scale": scales[1]}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=97, width=48, eps=3e-5, scale=1.7):
    return {"architecture": "Pamarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# Configurations that differ in every size, in the order and kinds of layers, and in the options.
CONFIGS = {
    # grouped heads, a partial rotation, keys and values of different sizes, a layer without feed-forward
    "a": config([layer("attention", attention(), ff=40),
                 layer("mlstm", memory()),
                 layer("parallel", parallel(), ff=56),
                 layer("mlstm", memory(heads=2, dim=20, vdim=6, gate_cap=4.0), ff=24),
                 layer("parallel", parallel(left(heads=3, kv_heads=1, dim=10, vdim=6, temp=None), right(heads=2, kv_heads=2, dim=16, vdim=8, conv=2),
                                            (-0.7, 1.1)), ff=32)]),
    # sizes the tensor-core attention kernels take (32 / 64 / 128), side by side first, one and several query heads a
    # key/value head, whole heads rotated, factors that the design could make equal or one
    "b": config([layer("parallel", parallel(left(heads=4, kv_heads=1, dim=64, vdim=32, scale=0.2, temp=(0.3, 64)),
                                            right(heads=2, kv_heads=1, dim=64, vdim=40, conv=4), (1.0, 1.0)), ff=72),
                 layer("attention", attention(heads=2, kv_heads=2, dim=64, scale=0.15, rot=(64, 20000.0)), ff=48),
                 layer("mlstm", memory(heads=2, dim=64, vdim=40, gate_cap=20.0), ff=40),
                 layer("attention", attention(heads=4, kv_heads=1, dim=128, scale=0.12, rot=(32, 300.0)))],
                vocab=61, width=64, eps=1e-6, scale=1.0),
    # the memory first, odd sizes, one head, one tap and eight, keys of more than 128 elements, no rotation
    "c": config([layer("mlstm", memory(heads=1, dim=130, vdim=21), ff=24),
                 layer("parallel", parallel(left(heads=1, kv_heads=1, dim=7, vdim=40, temp=(1.5, 1)),
                                            right(heads=3, kv_heads=3, dim=20, vdim=7, conv=1)), ff=16),
                 layer("attention", attention(heads=3, kv_heads=1, dim=9, rot=None)),
                 layer("parallel", parallel(left(heads=6, kv_heads=3, dim=33, vdim=5, temp=(0.4, 100)),
                                            right(heads=1, kv_heads=1, dim=140, vdim=20, conv=8), (0.3, 2.0)), ff=28)],
                vocab=128, width=40, scale=0.6),
}


def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q = p + "mix."
        out[p + "norm1"] = out[p + "norm1b"] = (W,)
        if l["type"] == "mlstm":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            out.update({q + "q": (H * dk, W), q + "k": (H * dk, W), q + "v": (H * dv, W), q + "g": (H * dv, W), q + "o": (W, H * dv),
                        q + "norm": (H * dv,), q + "i": (H, W), q + "i.b": (H,), q + "f": (H, W), q + "f.b": (H,)})
        elif l["type"] == "attention":
            H, G, dk = m["heads"], m["kv_heads"], m["dim"]
            out.update({q + "q": (H * dk, W), q + "k": (G * dk, W), q + "q.norm": (H * dk,), q + "k.norm": (G * dk,),
                        q + "g": (H * dk, W), q + "o": (W, H * dk)})
        else:
            a, d, r = m["left"], m["right"], q + "right."
            H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q += "left."
            out.update({q + "q": (H * dk, W), q + "k": (G * dk, W), q + "v": (G * dv, W), q + "q.norm": (dk,), q + "k.norm": (dk,),
                        q + "o": (W, H * dv)})
            H, G, dk, dv, taps = d["heads"], d["kv_heads"], d["dim"], d["vdim"], d["conv"]
            out.update({r + "q": (G * dk, W), r + "k": (G * dk, W), r + "v": (H * dv, W), r + "q.conv": (G * dk, taps),
                        r + "k.conv": (G * dk, taps), r + "v.conv": (H * dv, taps), r + "b": (H, W), r + "a": (H, W), r + "A_log": (H,),
                        r + "dt_bias": (H,), r + "norm": (dv,), r + "g": (H * dv, W), r + "o": (W, H * dv)})
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (W,)
            for n, shape in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
                out[p + "mlp." + n], out[p + f"mlp.{n}.b"] = shape, (shape[0],)
    return out


def make_weights(cfg, seed, sharp=1.0):
    """Random weights with magnitudes that keep every mechanism visible: projections of unit gain, norm weights of both
    kinds away from their neutral value, gates from closed to open, decays from fast to slow, biases of order one.
    `sharp` scales the head norms' weights and the query projections (peaked attention)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            w = rng.standard_normal(shape)
        elif name == "final.norm" or leaf in ("norm1", "norm1b", "norm2", "norm2b"):
            w = 0.3 * rng.standard_normal(shape)                          # the distance from one
        elif leaf == "norm":
            w = 1.0 + 0.2 * rng.standard_normal(shape)
            if name.endswith("q.norm"):
                w = w * sharp
        elif name.endswith(".f.b"):
            w = 1.5 + 1.5 * rng.standard_normal(shape)                    # heads that forget and heads that keep
        elif leaf == "b" and len(shape) == 1:
            w = 0.5 * rng.standard_normal(shape)
        elif leaf in ("A_log", "dt_bias"):
            w = rng.standard_normal(shape) - 1.0
        elif leaf == "conv":
            w = rng.standard_normal(shape) * 0.6
        else:
            w = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if leaf in ("a", "b", "g", "i", "f"):
                w = w * 2.0
        out[name] = np.asarray(w, dtype=np.float32)
    return out
