"""A matrix memory with exponential gates (the mLSTM of xLSTM).

With h the mixer's input, H heads, key size dk, value size dv:

    q = W_q h * dk^-1/2, k = W_k h [H, dk],  v = W_v h [H, dv],  z = W_g h [H * dv]
    i = cap tanh((W_i h + b_i) / cap),  f = logsigmoid(cap tanh((W_f h + b_f) / cap))     log gates, one a head
    per head, from S = 0 [dk, dv], n = 0 [dk], m = 0:
        m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n <- e^(f + m - m') n + e^(i - m') k
        o  = S^T q / (max(|n . q|, e^(-m')) + 1e-6)
    out = W_o (concat_a o_a / sqrt(mean(o_a^2) + eps) * w * sigmoid(z))                   w [H * dv]

m only keeps the exponentials in range: with S e^m and n e^m the recurrence is linear with decay e^f.  A sequence's state
is one float32 row: S column by column with n as one more column (the value of which is one), [H, dv + 1, dk], and m [H].
The fused input projection [q | k | v | z | i | f] leaves the library's product as float32; everything behind it is
float32 up to the gated norm's output.  Long runs are cut into chunks where that fills the GPU (`chunks.cut_runs`).
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import gemv as KG
from ..kernels import ssm as KS
from ..kernels.linear import linear
from ..weights.loader import WeightSpec, WeightStore
from .base import LayerCache, Mixer, StateNeed, StepContext, register_mixer
from .chunks import cut_runs

DENOMINATOR_FLOOR = 1e-6


class MatrixMemoryMixer(Mixer):
    def __init__(self, prefix: str, hidden: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float):
        if heads < 1 or vdim < 1 or not 1 <= dim <= KS.MAX_STATE:
            raise ValueError(f"matrix memory '{prefix}': {heads} heads, keys of {dim} (1..{KS.MAX_STATE}), values of {vdim}")
        if not (gate_cap > 0.0 and eps > 0.0):
            raise ValueError(f"matrix memory '{prefix}': the gates' cap {gate_cap} and eps {eps} must be positive")
        self.prefix, self.hidden, self.heads, self.dim, self.vdim = prefix, int(hidden), int(heads), int(dim), int(vdim)
        self.cap, self.eps = float(gate_cap), float(eps)
        self.qk, self.inner = self.heads * self.dim, self.heads * self.vdim
        self.state_size = self.heads * (self.vdim + 1) * self.dim
        self.w_in = self.w_o = self.w_norm = self.i_bias = self.f_bias = None

    def weight_specs(self) -> List[WeightSpec]:
        p, W, H = self.prefix, self.hidden, self.heads
        return [WeightSpec(p + "q", (self.qk, W)), WeightSpec(p + "k", (self.qk, W)), WeightSpec(p + "v", (self.inner, W)),
                WeightSpec(p + "g", (self.inner, W)), WeightSpec(p + "i", (H, W)), WeightSpec(p + "i.b", (H,)),
                WeightSpec(p + "f", (H, W)), WeightSpec(p + "f.b", (H,)),
                WeightSpec(p + "norm", (self.inner,), init="one_plus_normal"), WeightSpec(p + "o", (W, self.inner))]

    def bind(self, store: WeightStore) -> None:
        p = self.prefix
        ws = [store.take(p + n) for n in ("q", "k", "v", "g", "i", "f")]
        dt = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        self.w_in = torch.cat([w.to(dt) for w in ws], dim=0).contiguous()
        self.i_bias, self.f_bias = (store.get(p + n).float().contiguous() for n in ("i.b", "f.b"))
        self.w_norm, self.w_o = store.get(p + "norm"), store.get(p + "o")

    def kernels(self) -> List[str]:
        return ["ssm"] + (["gemv"] if getattr(self, "run_dtype", None) == torch.bfloat16 else [])

    def state_need(self) -> StateNeed:
        return StateNeed((self.state_size + self.heads,), torch.float32)

    def step_work(self, n_tokens, kv_tokens):
        wb = lambda w: 0 if w is None else w.numel() * w.element_size()
        rows = 2 * self.qk + 2 * self.inner + 2 * self.heads
        return {"matmul": (wb(self.w_in) + wb(self.w_o), 2.0 * n_tokens * self.hidden * (rows + self.inner)),
                "other": (8.0 * self.state_size, 5.0 * n_tokens * self.state_size)}

    def input_weight(self) -> torch.Tensor:
        """The fused input projection's weight ([q | k | v | z | i | f] rows): see `forward(projected=...)`."""
        return self.w_in

    def take_input_weight(self, w: torch.Tensor) -> None:
        """The fused input projection as part of a wider one."""
        self.w_in = w

    def forward(self, xn: torch.Tensor, ctx: StepContext, cache: LayerCache, projected: Optional[torch.Tensor] = None,
                offset: int = 0) -> torch.Tensor:
        """projected: float32 rows of a wider product that hold this mixer's projection from column `offset`."""
        T, dev, H, dk, dv = xn.shape[0], xn.device, self.heads, self.dim, self.vdim
        proj = projected if projected is not None else linear(xn, self.w_in, out_dtype=torch.float32)
        q, k = offset, offset + self.qk
        v, z = k + self.qk, k + self.qk + self.inner
        i, f = z + self.inner, z + self.inner + H
        S = cache.state[:, :self.state_size].unflatten(1, (H, dv + 1, dk))
        tops = cache.state[:, self.state_size:self.state_size + H]
        o = torch.empty((T, self.inner), dtype=ctx.act_dtype, device=dev)
        if ctx.max_q_len == 1 and ctx.n_seqs == T:               # every sequence brings one token: one launch
            KS.memory_step(proj, q, k, v, z, i, f, self.i_bias, self.f_bias, self.cap, dk ** -0.5, S, tops, ctx.slots, self.w_norm, o,
                           H, dk, dv, DENOMINATOR_FLOOR, self.eps)
        else:
            f32 = lambda *shape: torch.empty(shape, dtype=torch.float32, device=dev)
            gates, m, y, dots = f32(T, H, 2), f32(T, H), f32(T, self.inner), f32(T, H)
            KS.memory_gates(proj, i, f, self.i_bias, self.f_bias, self.cap, tops, gates, m, H, ctx.cu_seqlens, ctx.slots)
            scan = lambda st, out, nq, cu, slots: KS.memory_scan(proj, q, k, v, gates, st, out, nq, H, dk, dv, cu, slots)
            plan = cut_runs(ctx, H, dv + 1)
            if plan is None:
                scan(S, y, dots, ctx.cu_seqlens, ctx.slots)
            else:
                # the chunks side by side from zero states without outputs, the states they should have started from, and
                # the chunks once more from those
                cu_chunks, chunk_ids, seq_chunks = plan
                ends = torch.zeros((chunk_ids.shape[0], H, dv + 1, dk), dtype=torch.float32, device=dev)
                starts = torch.empty_like(ends)
                decays = f32(chunk_ids.shape[0], H)
                scan(ends, None, decays, cu_chunks, chunk_ids)
                KS.memory_combine(S, ctx.slots, ends, starts, seq_chunks, decays)
                scan(starts, y, dots, cu_chunks, chunk_ids)
            KS.gated_group_norm(y, proj, z, self.w_norm, H, self.eps, o, gate_after=True, sigmoid_gate=True, dots=dots, tops=m,
                                dot_scale=dk ** -0.5, floor=DENOMINATOR_FLOOR)
        if KG.pays(o, self.w_o):
            return KG.gemv(o, self.w_o, torch.empty((T, self.hidden), dtype=torch.float32, device=dev))
        return linear(o, self.w_o, out_dtype=torch.float32)


register_mixer("matrix_memory", MatrixMemoryMixer)
