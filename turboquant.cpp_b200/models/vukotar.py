"""The Vukotar decoder as a list of parts.

Scaled embedding with sinusoidal positions added; layers in the order config.json lists them, each a `ParallelBlock`: one
dynamic-tanh norm, on its output attention (no rotation, a softmax with one more in its denominator) beside routed
experts (square of relu, sigmoid scores, groups of experts), each with a factor per element on the way into the
stream.  A layer may use another one's tensors: its schedule entry then names that layer's block and keeps a cache of its
own.  Final norm of the same kind; the head is the embedding's table, its logits capped.
Tensors: embed, l<i>.norm1 (+ .b, .alpha), l<i>.mix.q|k|v|o, l<i>.mlp.router, l<i>.mlp.e<n>.up|down, l<i>.ls1|ls2,
final.norm (+ .b, .alpha).
"""
from __future__ import annotations

import torch

from ..config.registry import register_architecture
from ..config.vukotar import ARCHITECTURE, GROUP_TOP, POSITION_BASE, ROUTER_WEIGHT_FLOOR, VukotarConfig
from ..kernels.elementwise import MAP_RELU_SQUARED
from ..parts import ParallelBlock, make_feed_forward, make_mixer, make_norm
from .decoder import DecoderModel, LMHead, PositionedEmbedding, ScheduleEntry

MOE_NAMES = {"router": "router", "expert": "e{e}.", "up": "up", "down": "down"}


class VukotarModel(DecoderModel):
    def __init__(self, cfg: VukotarConfig, dtype: torch.dtype):
        W = cfg.width
        norm = lambda name: make_norm("dyt", name=name, size=W)
        blocks, block_of = [], {}
        for i, layer in enumerate(cfg.layers):
            if layer.weights_of is not None:
                continue
            p, m, e = f"l{i}.", layer.mixer, layer.mlp
            mixer = make_mixer("window_bias_attention", prefix=p + "mix.", hidden=W, heads=m.heads, kv_heads=m.kv_heads,
                               dim=m.dim, vdim=m.vdim, scale=m.scale, sink=True)
            ffn = None
            if e is not None:
                ffn = make_feed_forward("moe", prefix=p + "mlp.", hidden=W, n_experts=e.experts, top_k=e.top,
                                        intermediate=e.ff, norm_topk=True, n_groups=e.groups, keep_groups=e.keep_groups,
                                        group_top=GROUP_TOP, scores="sigmoid", renorm_floor=ROUTER_WEIGHT_FLOOR,
                                        gated=False, map=MAP_RELU_SQUARED, names=MOE_NAMES)
            block_of[i] = len(blocks)
            blocks.append(ParallelBlock(norm(p + "norm1"), mixer, ffn, hidden=W, mixer_scale=p + "ls1",
                                        ffn_scale=p + "ls2", leave_open=True))
        schedule = [ScheduleEntry(block_of[i if layer.weights_of is None else layer.weights_of])
                    for i, layer in enumerate(cfg.layers)]
        super().__init__(cfg, dtype, embedding=PositionedEmbedding("embed", cfg.vocab, W, cfg.embedding_scale, POSITION_BASE),
                         blocks=blocks, schedule=schedule, final_norm=norm("final.norm"),
                         head=LMHead("embed", cfg.vocab, W, softcap=cfg.logit_softcap))


register_architecture(ARCHITECTURE, VukotarConfig, VukotarModel)
