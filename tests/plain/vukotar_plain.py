"""A plain, slow implementation of the Vukotar decoder, one function per mechanism, in float64 on the CPU.

It reads a model folder (config.json, model.safetensors) with its own few lines of file parsing and shares no code
with the library.  Every function takes a whole sequence; nothing is cached, so the logits of a position are those of
the definition itself.

Notation: x_p is the stream at position p, d the model width, dyt(v) = tanh(alpha v) * w + b.

    x_p = a * E[token_p] + s(p),   s(p)_(2m) = sin(p w_m), s(p)_(2m+1) = cos(p w_m), w_m = 10000^(-2m/d)
    per layer:  h = dyt(x);  x <- x + ls1 * attention(h) + ls2 * experts(h)         (the last term only with experts)
    logits = c * tanh(E dyt(x) / c)

A layer may use the weights of another one; it still attends over keys and values of its own.
"""
import json
import math
import os
import struct

import numpy as np

F = np.float64
POSITION_BASE = 10000.0
WEIGHT_FLOOR = 1e-20


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
        a, b = meta["data_offsets"]
        raw = data[a:b]
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


# ---- the mechanisms -------------------------------------------------------------------------------------------
def position_vector(p, width):
    out = np.zeros(width, dtype=F)
    for c in range(width):
        angle = p * POSITION_BASE ** (-(c - c % 2) / width)
        out[c] = math.sin(angle) if c % 2 == 0 else math.cos(angle)
    return out


def embed(tokens, table, scale):
    return np.stack([table[t] * scale + position_vector(p, table.shape[1]) for p, t in enumerate(tokens)])


def dyt(v, w, name):
    return np.tanh(float(w[name + ".alpha"]) * v) * w[name] + w[name + ".b"]


def sink_softmax(s):
    """exp(s_j) / (1 + sum exp(s_j)), without overflow."""
    top = max(0.0, float(s.max()))
    e = np.exp(s - top)
    return e / (math.exp(-top) + e.sum())


def attention_core(q, k, v, scale):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] of one sequence from its start; [T, H, dv]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=F)
    for i in range(T):
        for a in range(H):
            g = a // per
            out[i, a] = sink_softmax(k[:i + 1, g] @ q[i, a] * scale) @ v[:i + 1, g]
    return out


def attention(h, w, p, m):
    T = h.shape[0]
    H, G = m["heads"], m.get("kv_heads", m["heads"])
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[p + "k"].T).reshape(T, G, m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
    return attention_core(q, k, v, m["scale"]).reshape(T, H * m["vdim"]) @ w[p + "o"].T


def route_row(z, r):
    """One token's logits z [E]: (the chosen experts, their weights, the scores, the smallest gap that decided)."""
    E, top = r["experts"], r["top"]
    s = 1.0 / (1.0 + np.exp(-z))
    allowed, gap = list(range(E)), math.inf
    if r.get("groups"):
        n, keep = r["groups"]["count"], r["groups"]["keep"]
        per = E // n
        value = [sum(sorted(s[g * per:(g + 1) * per])[-2:]) for g in range(n)]
        order = sorted(range(n), key=lambda g: (-value[g], g))
        if keep < n:
            gap = value[order[keep - 1]] - value[order[keep]]
        allowed = [e for e in range(E) if e // per in order[:keep]]
    order = sorted(allowed, key=lambda e: (-s[e], e))
    if top < len(order):
        gap = min(gap, s[order[top - 1]] - s[order[top]])
    ids = np.array(order[:top])
    return ids, s[ids] / (s[ids].sum() + WEIGHT_FLOOR), s, gap


def expert(h, w, p):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def experts(h, w, p, ml, ids=None, record=None):
    """The routed feed-forward of rows h [T, d].  ids [T, top]: these experts in place of the choice (their weights are
    still this model's); record: receives (ids, weights, gaps)."""
    y, seen = np.zeros_like(h), []
    for t in range(h.shape[0]):
        own, wts, s, gap = route_row(w[p + "router"] @ h[t], ml["router"])
        if ids is not None:
            own = np.asarray(ids[t])
            wts = s[own] / (s[own].sum() + WEIGHT_FLOOR)
        for e, a in zip(own, wts):
            y[t] += a * expert(h[t], w, f"{p}e{e}.")
        seen.append((own, wts, gap))
    if record is not None:
        record.append(tuple(np.array(c) for c in zip(*seen)))
    return y


def softcap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ---- the model ------------------------------------------------------------------------------------------------
def source_layer(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, w, tokens, streams=None, routing=None, forced=None):
    """Logits [T, vocab] of one sequence.  streams: receives the stream after every layer; routing: (experts, weights,
    gaps) of every layer with experts, in the order they run; forced: per such layer the experts [T, top] to take
    (a shorter list: the layers without an entry choose for themselves)."""
    x = embed(tokens, w["embed"], cfg.get("embedding", {}).get("scale", 1.0))
    routed = 0
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{source_layer(cfg['layers'], i)}."
        h = dyt(x, w, p + "norm1")
        y = attention(h, w, p + "mix.", layer["mixer"]) * w[p + "ls1"]
        if layer.get("mlp"):
            ids = forced[routed] if forced is not None and routed < len(forced) else None
            y = y + experts(h, w, p + "mlp.", layer["mlp"], ids, routing) * w[p + "ls2"]
            routed += 1
        x = x + y
        if streams is not None:
            streams.append(x.copy())
    return softcap(dyt(x, w, "final.norm") @ w["embed"].T, cfg.get("logit_softcap"))


class PlainVukotar:
    def __init__(self, folder):
        self.cfg, self.w = load(folder)

    def forward(self, tokens, streams=None, routing=None, forced=None):
        return forward(self.cfg, self.w, tokens, streams, routing, forced)
