"""Two mixers side by side: both read the same input, each output passes an RMS norm of its own (a plain weight over
the model width) or goes on as it is, and the result is a weighted sum.

    y = f_l * norm_left(left(h)) + f_r * norm_right(right(h))           (factors of 1/2: the mean)
    y = f_l * left(h) + f_r * right(h)                                   (without norms)

The branches are mixers of any kind; one may keep keys and values, one a per-sequence state (the block hands the
pair's needs on: the cache of whichever branch asks for one, the state likewise).  When both branches offer their
fused input projection (`input_weight()`, `take_input_weight()` and `forward(..., projected=...)`), the two projections
run as one product.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from ..kernels.linear import linear
from ..weights.loader import WeightSpec, WeightStore
from . import side
from .base import BranchPair, KVNeed, LayerCache, Mixer, StateNeed, StepContext, register_mixer


class ParallelMixer(Mixer):
    # The branches run on two streams: neither waits for the other.  Prompts stay on one where launches, not the GPU, bound
    # the step (a smaller stream), and where a branch wants the GPU to itself.  Measured on B200, one stream / two: decoding
    # with a delta rule beside attention 0.588 / 0.566 ms (batch 8, width 2,048), with retention 0.692 / 0.674 ms; a prompt
    # with retention 5.79 / 5.26 ms, with a delta rule 4.33 / 4.49 ms.
    SIDE_BY_SIDE = side.ENABLED
    SIDE_MIN_ELEMENTS = 3 << 20

    def __init__(self, left: Mixer, right: Mixer, hidden: int, eps: float, left_norm: Optional[str] = None,
                 right_norm: Optional[str] = None, factors: Tuple[float, float] = (0.5, 0.5)):
        """left_norm, right_norm: the names of the two norms' weights (both None: no norms)."""
        if (left_norm is None) != (right_norm is None):
            raise ValueError("mixers side by side: both branches have a norm or neither")
        needs = [m.cache_need() for m in (left, right)]
        states = [m.state_need() for m in (left, right)]
        if all(n is not None for n in needs) or all(s is not None for s in states):
            raise ValueError("mixers side by side: at most one branch may keep keys and values, and one a state")
        self.left, self.right, self.hidden, self.eps = left, right, int(hidden), float(eps)
        self.left_norm, self.right_norm, self.factors = left_norm, right_norm, (float(factors[0]), float(factors[1]))
        self.w_left = self.w_right = self.w_in = None

    def parts(self):
        return [self.left, self.right]

    def weight_specs(self) -> List[WeightSpec]:
        return self.left.weight_specs() + self.right.weight_specs() + \
            [WeightSpec(n, (self.hidden,), init="one_plus_normal") for n in (self.left_norm, self.right_norm) if n is not None]

    def bind(self, store: WeightStore) -> None:
        self.left.bind(store)
        self.right.bind(store)
        if self.left_norm is not None:
            self.w_left, self.w_right = store.get(self.left_norm), store.get(self.right_norm)
            if self.w_left.dtype != self.w_right.dtype:
                self.w_left, self.w_right = self.w_left.float(), self.w_right.float()
        if all(hasattr(m, "input_weight") for m in (self.left, self.right)):
            a, b = self.left.input_weight(), self.right.input_weight()
            if a.dtype == b.dtype:
                self.w_in = torch.cat([a, b], dim=0).contiguous()       # one product for both branches
                self.left.take_input_weight(self.w_in[:a.shape[0]])     # the branches keep views of it
                self.right.take_input_weight(self.w_in[a.shape[0]:])

    def kernels(self) -> List[str]:
        return ["elementwise"] + self.left.kernels() + self.right.kernels()

    def cache_need(self) -> Optional[KVNeed]:
        return self.left.cache_need() or self.right.cache_need()

    def state_need(self) -> Optional[StateNeed]:
        return self.left.state_need() or self.right.state_need()

    def capturable(self) -> bool:
        return self.left.capturable() and self.right.capturable()

    def step_work(self, n_tokens, kv_tokens):
        return {}                # the branches are listed among the block's parts and say what they do themselves

    def forward_branches(self, xn: torch.Tensor, ctx: StepContext, cache: LayerCache) -> BranchPair:
        """The two branches' outputs before their norms, for a block whose norm on the mixer's output takes the
        branches' norms and their weighted sum in its own pass."""
        left_in, right_in = {}, {}
        if self.w_in is not None:
            proj = linear(xn, self.w_in, out_dtype=torch.float32)
            left_in, right_in = {"projected": proj}, {"projected": proj, "offset": self.left.input_weight().shape[0]}
        runs_apart = xn.numel() >= self.SIDE_MIN_ELEMENTS and not (self.left.runs_alone or self.right.runs_alone)
        if self.SIDE_BY_SIDE and (ctx.max_q_len == 1 or runs_apart):
            other = side.fork(xn.device)
            with torch.cuda.stream(other):
                b = self.right.forward(xn, ctx, cache, **right_in)
            a = self.left.forward(xn, ctx, cache, **left_in)
            side.join(other)
        else:
            a = self.left.forward(xn, ctx, cache, **left_in)
            b = self.right.forward(xn, ctx, cache, **right_in)
        return BranchPair(a, self.w_left, b, self.w_right, self.eps, self.factors)

    def forward(self, xn: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        return self.forward_branches(xn, ctx, cache).sum()


register_mixer("parallel", ParallelMixer)
