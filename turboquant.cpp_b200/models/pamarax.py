"""The Pamarax decoder as a list of parts.

Scaled embedding; layers in the order config.json lists them, each a `SandwichBlock` of RMS norms whose stored weight is
the distance from one, before and after each sub-layer.  Three mixers: a matrix memory with exponential gates; attention
whose values are its unnormed, unrotated keys, with a norm over the whole query and key rows, rotation and a gate per
element; and two branches side by side with a factor each, attention with normed heads, a temperature on the queries
and one more in the softmax's denominator, and a delta rule with one decay per head.  Dense feed-forward (silu, biases),
final norm, a head of its own.
Tensors: embed, l<i>.norm1|norm1b|norm2|norm2b, l<i>.mix.<name> (a parallel mixer's under mix.left and mix.right),
l<i>.mlp.gate|up|down (+ .b), final.norm, head.
"""
from __future__ import annotations

import torch

from ..config.pamarax import ARCHITECTURE, PamaraxConfig
from ..config.registry import register_architecture
from ..parts import SandwichBlock, make_feed_forward, make_mixer, make_norm, make_position_encoding
from .decoder import DecoderModel, LMHead, PairEmbedding, ScheduleEntry


class PamaraxModel(DecoderModel):
    def __init__(self, cfg: PamaraxConfig, dtype: torch.dtype):
        W, eps = cfg.width, cfg.eps
        norm = lambda name: make_norm("rmsnorm", name=name, size=W, eps=eps, around_zero=True)
        blocks = []
        for i, layer in enumerate(cfg.layers):
            p, m = f"l{i}.", layer.mixer
            if layer.type == "mlstm":
                mixer = make_mixer("matrix_memory", prefix=p + "mix.", hidden=W, heads=m.heads, dim=m.dim, vdim=m.vdim,
                                   gate_cap=m.gate_cap, eps=eps)
            elif layer.type == "attention":
                position = make_position_encoding("rotary_scaled", dims=m.rot_dims, base=m.rot_base, pairing="halves") if m.rot_dims else None
                mixer = make_mixer("normed_attention", prefix=p + "mix.", hidden=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim,
                                   vdim=m.dim, scale=m.scale, eps=eps, norm="row", position=position, values_are_keys=True, gate=True)
            else:
                a, d = m.left, m.right
                left = make_mixer("normed_attention", prefix=p + "mix.left.", hidden=W, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim,
                                  vdim=a.vdim, scale=a.scale, eps=eps, norm="head", temperature=a.temperature, sink=True)
                right = make_mixer("head_delta", prefix=p + "mix.right.", hidden=W, heads=d.heads, kv_heads=d.kv_heads, dim=d.dim,
                                   vdim=d.vdim, taps=d.taps, eps=eps)
                mixer = make_mixer("parallel", left=left, right=right, hidden=W, eps=eps, factors=(m.left_scale, m.right_scale))
            ffn = ffn_norm = ffn_post = None
            if layer.mlp is not None:
                ffn_norm, ffn_post = norm(p + "norm2"), norm(p + "norm2b")
                ffn = make_feed_forward("glu", prefix=p + "mlp.", hidden=W, intermediate=layer.mlp.ff, bias=True)
            blocks.append(SandwichBlock(norm(p + "norm1"), mixer, norm(p + "norm1b"), ffn_norm, ffn, ffn_post))
        for b, nxt in zip(blocks, blocks[1:]):               # the layers run in the listed order, each once
            b.next_norm = nxt.mixer_norm
        super().__init__(cfg, dtype, embedding=PairEmbedding("embed", cfg.vocab, W, cfg.embedding_scale), blocks=blocks,
                         schedule=[ScheduleEntry(i) for i in range(len(blocks))], final_norm=norm("final.norm"),
                         head=LMHead("head", cfg.vocab, W))


register_architecture(ARCHITECTURE, PamaraxConfig, PamaraxModel)
