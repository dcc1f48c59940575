"""A plain, slow implementation of the Pamarax decoder, one function per mechanism, in float64 on the CPU.

It reads a model folder (config.json, model.safetensors) with its own few lines of file parsing and shares no code
with the library.  Every function takes a whole sequence and loops over positions where the definition does; nothing
is cached, so the logits of a position are those of the definition itself.

With x the stream (the embedding's row times a factor at the start), every layer is

    x <- x + post1(mixer(pre1(x)));   x <- x + post2(ff(pre2(x)))       the second line only with a feed-forward

where pre and post are RMS norms whose stored weight is the distance from one.  Three mixers: a matrix memory with
exponential gates; softmax attention whose values are its unnormed, unrotated keys, with a norm over the whole query and
key rows, and a gate per element; and two branches side by side, softmax attention with one more in the softmax's
denominator and a temperature on the queries, and a delta rule with one decay per head.

`store` (identity by default) is applied wherever an implementation with 16-bit activations keeps one: what the norms hand
to the products, attention's queries, keys, values and sums, what enters a mixer's last product, and the feed-forward's
inner activations.  With `to_bfloat16` the model is what such an implementation computes, up to its float32 sums.
"""
import json
import math
import os
import struct

import numpy as np

F = np.float64
UNIT_EPS = 1e-6              # inside the root of the delta rule's unit vectors
MEMORY_FLOOR = 1e-6          # added to the matrix memory's denominator


# ---- file reading ---------------------------------------------------------------------------------------------
def read_safetensors(path):
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = data[lo:hi]
        if meta["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(F)
        elif meta["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(F)
        else:
            raise ValueError(f"dtype {meta['dtype']} of '{name}'")
        out[name] = arr.reshape(meta["shape"])
    return out


def load(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ---- small functions --------------------------------------------------------------------------------------------
def sigmoid(v):
    return 1.0 / (1.0 + np.exp(-v))


def silu(v):
    return v * sigmoid(v)


def softplus(v):
    return np.logaddexp(0.0, v)


def log_sigmoid(v):
    return -np.logaddexp(0.0, -v)


def unit_rms(v, eps):
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def keep(v):
    return v


def to_bfloat16(v):
    """To the nearest bfloat16, ties to even."""
    u = np.ascontiguousarray(v, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16).astype(np.uint32).view(np.float32).astype(F)


def around_one(v, w, eps):
    """An RMS norm whose stored weight is the distance from one."""
    return unit_rms(v, eps) * (1.0 + w)


# ---- mixer: matrix memory with exponential gates ------------------------------------------------------------------
def memory_recurrence(q, k, v, i, f, start=None):
    """One head: q, k [T, dim], v [T, vdim], log gates i, f [T]; start: (S [dim, vdim], n [dim], m) before the first
    token (zeros if None).  Returns (outputs [T, vdim], the state after the last token)."""
    T, dim = k.shape
    if start is None:
        S, n, m = np.zeros((dim, v.shape[1]), dtype=F), np.zeros(dim, dtype=F), 0.0
    else:
        S, n, m = start[0].astype(F).copy(), start[1].astype(F).copy(), float(start[2])
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        top = max(f[t] + m, i[t])                      # the running maximum that keeps the exponentials in range
        keep, take = math.exp(f[t] + m - top), math.exp(i[t] - top)
        S = keep * S + take * np.outer(k[t], v[t])
        n = keep * n + take * k[t]
        m = top
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + MEMORY_FLOOR)
    return out, (S, n, m)


def memory_gates(h, w, p, cap):
    """The log gates of every head, [T, heads] each: the input's, and the logarithm of a sigmoid for forgetting."""
    capped = lambda name: cap * np.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    return capped("i"), log_sigmoid(capped("f"))


def memory_mixer(h, w, p, m, eps, store=keep):
    T = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, dim)
    v = (h @ w[p + "v"].T).reshape(T, H, vdim)
    gi, gf = memory_gates(h, w, p, float(m["gate_cap"]))
    o = np.zeros((T, H, vdim), dtype=F)
    for a in range(H):
        o[:, a], _ = memory_recurrence(q[:, a], k[:, a], v[:, a], gi[:, a], gf[:, a])
    o = unit_rms(o, eps).reshape(T, H * vdim) * w[p + "norm"]
    return store(o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- softmax attention --------------------------------------------------------------------------------------------
def rotate_halves(v, positions, dims, base):
    """v [T, heads, n]: element i < dims/2 is paired with i + dims/2; position p turns the pair by p * base^(-2i/dims).
    Elements from `dims` on pass."""
    half = dims // 2
    out = v.copy()
    freq = np.array([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    ang = positions[:, None, None].astype(F) * freq[None, None, :]
    c, s = np.cos(ang), np.sin(ang)
    a, b = v[..., :half], v[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


def attend(q, k, v, scale, extra=0.0):
    """q [T, H, dim] over k [T, G, dim], v [T, G, vdim], causal; `extra` is added to the softmax's denominator (in
    units of exp(0))."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=F)
    for a in range(H):
        g = a // (H // G)
        for t in range(T):
            s = (k[:t + 1, g] @ q[t, a]) * scale
            top = max(float(s.max()), 0.0)
            e = np.exp(s - top)
            out[t, a] = (e / (e.sum() + extra * math.exp(-top))) @ v[:t + 1, g]
    return out


def shared_value_attention(h, w, p, m, eps, store=keep):
    T = h.shape[0]
    H, G, dim = m["heads"], m["kv_heads"], m["dim"]
    pos = np.arange(T)
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    v = k.reshape(T, G, dim)                                  # the keys as they leave the projection
    q = (unit_rms(q, eps) * w[p + "q.norm"]).reshape(T, H, dim)      # one root mean square for all heads
    k = (unit_rms(k, eps) * w[p + "k.norm"]).reshape(T, G, dim)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = (rotate_halves(u, pos, rot["dims"], rot["base"]) for u in (q, k))
    o = store(attend(store(q), store(k), store(v), m["scale"])).reshape(T, H * dim)
    return store(o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((positions + 1) / every) + 1.0)


def sink_attention(h, w, p, m, eps, store=keep):
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w[p + "q"].T).reshape(T, H, dim), eps) * w[p + "q.norm"]
    k = unit_rms((h @ w[p + "k"].T).reshape(T, G, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(T, G, vdim)
    temp = m.get("q_temp")
    if temp:
        q = q * query_temperature(np.arange(T), temp["coef"], temp["every"])[:, None, None]
    o = attend(store(q), store(k), store(v), m["scale"], extra=1.0)
    return store(o.reshape(T, H * vdim)) @ w[p + "o"].T


# ---- delta rule with one decay per head -----------------------------------------------------------------------------
def short_convolution(u, taps_w):
    """u [T, C], taps_w [C, taps]: the last column meets the current token, zeros before the start."""
    T, taps = u.shape[0], taps_w.shape[1]
    out = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1 - j)
            if src >= 0:
                out[t] += u[src] * taps_w[:, j]
    return out


def unit_vector(v):
    return v / np.sqrt(np.sum(v * v, axis=-1, keepdims=True) + UNIT_EPS)


def gated_delta_rule(q, k, v, beta, decay, S=None):
    """One head: q, k [T, dim], v [T, vdim], beta, decay [T]; S [dim, vdim] before the first token (zeros if None).
    Returns (outputs [T, vdim], the state after the last token)."""
    T, dim = k.shape
    S = np.zeros((dim, v.shape[1]), dtype=F) if S is None else S.astype(F).copy()
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        S = decay[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out, S


def delta_mixer(h, w, p, m, eps, store=keep):
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, dim)) * dim ** -0.5
    k = unit_vector(k.reshape(T, G, dim))
    v = v.reshape(T, H, vdim)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = np.zeros((T, H, vdim), dtype=F)
    for a in range(H):
        g = a // (H // G)
        o[:, a], _ = gated_delta_rule(q[:, g], k[:, g], v[:, a], beta[:, a], decay[:, a])
    o = unit_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, vdim)
    return store(o.reshape(T, H * vdim)) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps, store=keep):
    return (m["left_scale"] * sink_attention(h, w, p + "left.", m["left"], eps, store) +
            m["right_scale"] * delta_mixer(h, w, p + "right.", m["right"], eps, store))


MIXERS = {"mlstm": memory_mixer, "attention": shared_value_attention, "parallel": parallel_mixer}


# ---- feed-forward and model -----------------------------------------------------------------------------------------
def feed_forward(h, w, p, store=keep):
    lin = lambda u, n: u @ w[p + n].T + w[p + n + ".b"]
    return lin(store(silu(lin(h, "gate")) * lin(h, "up")), "down")


def forward(cfg, w, tokens, streams=None, store=keep):
    """Logits [T, vocab] of a whole sequence; `streams` (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](store(around_one(x, w[p + "norm1"], eps)), w, p + "mix.", layer["mixer"], eps, store)
        x = x + around_one(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(store(around_one(x, w[p + "norm2"], eps)), w, p + "mlp.", store)
            x = x + around_one(y, w[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.copy())
    return store(around_one(x, w["final.norm"], eps)) @ w["head"].T


class PlainPamarax:
    def __init__(self, folder):
        self.cfg, self.weights = load(folder)

    def forward(self, tokens, streams=None, store=keep):
        return forward(self.cfg, self.weights, tokens, streams, store)
