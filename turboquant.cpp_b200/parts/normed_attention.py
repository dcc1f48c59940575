"""Causal grouped-query attention with normed queries and keys, over the paged cache of rows [k | v].

With h the mixer's input, H query heads on G key/value heads (head a reads a // (H / G)), key size dk, value size dv:

    q = W_q h, k = W_k h, v = W_v h, z = W_g h             (one fused product, float32 result; v and z optional)
    q, k <- rms(q) * w_q, rms(k) * w_k                      `norm` 'head': each head by itself, weights [dk] the heads share;
                                                            'row': all query heads as one row, all key heads as another,
                                                            weights [H * dk] and [G * dk]; None: no norm
    q, k <- rotated by the position                         (`position`: frequencies, pairing; None: no rotation)
    q    <- q * (1 + coef * ln(floor((p + 1) / every) + 1)) (`temperature` (coef, every); None: as it is)
    p_ij  = exp(s_ij) / (c + sum_j exp(s_ij)),  s_ij = q_i . k_j * scale,  j <= i        c: 1 with `sink`, else 0
    out   = W_o (concat_a sum_j p_ij v_j * sigmoid(z))      (`gate`: a logit per element; without: the sums as they are)

`values_are_keys`: there is no W_v; the values are the keys as they leave the projection, before norm and rotation.  Norms,
rotation, temperature, scores and softmax are float32; queries, cached rows and the sums are kept in the activation dtype.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

import torch

from ..kernels import bias_attention as KB
from ..kernels.linear import linear
from ..weights.loader import WeightSpec, WeightStore
from .base import KVNeed, LayerCache, Mixer, StepContext, register_mixer
from .bias_attention import paged_attention
from .gated_attention import _fuse, _output


class NormedAttentionMixer(Mixer):
    RUNS_MIN = 16             # steps whose longest run of new tokens is at least this take the kernel for runs

    def __init__(self, prefix: str, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float,
                 norm: Optional[str] = "head", position=None, temperature: Optional[Tuple[float, int]] = None,
                 sink: bool = False, values_are_keys: bool = False, gate: bool = False, window: int = 0):
        if heads < 1 or kv_heads < 1 or heads % kv_heads:
            raise ValueError(f"attention '{prefix}': {heads} heads are not a multiple of {kv_heads} key/value heads")
        if not (1 <= dim <= KB.MAX_DIM and 1 <= vdim <= KB.MAX_DIM):
            raise ValueError(f"attention '{prefix}': key size {dim} and value size {vdim} must be in 1..{KB.MAX_DIM}")
        if norm not in (None, "head", "row"):
            raise ValueError(f"attention '{prefix}': norm must be 'head', 'row' or None, got {norm!r}")
        if position is not None and (not hasattr(position, "freq") or position.dims > dim):
            raise ValueError(f"attention '{prefix}': the position encoding must give frequencies for at most {dim} elements")
        if values_are_keys and dim != vdim:
            raise ValueError(f"attention '{prefix}': keys of {dim} elements cannot be values of {vdim}")
        if window < 0 or not eps > 0.0 or (temperature is not None and temperature[1] < 1):
            raise ValueError(f"attention '{prefix}': window {window}, eps {eps} and temperature {temperature}")
        self.prefix, self.hidden = prefix, int(hidden)
        self.heads, self.kv_heads, self.dim, self.vdim = int(heads), int(kv_heads), int(dim), int(vdim)
        self.scale, self.eps, self.norm, self.window = float(scale), float(eps), norm, int(window)
        self.position, self.has_sink, self.values_are_keys, self.has_gate = position, bool(sink), bool(values_are_keys), bool(gate)
        self.temperature = None if temperature is None else (float(temperature[0]), int(temperature[1]))
        self.q_size, self.k_size, self.v_size = self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim
        self.out_size = self.heads * self.vdim
        self.gate_off = self.q_size + self.k_size + (0 if self.values_are_keys else self.v_size)
        self.w_in = self.w_o = self.q_norm = self.k_norm = self.sink = None

    def weight_specs(self) -> List[WeightSpec]:
        p, W = self.prefix, self.hidden
        specs = [WeightSpec(p + "q", (self.q_size, W)), WeightSpec(p + "k", (self.k_size, W)), WeightSpec(p + "o", (W, self.out_size))]
        if not self.values_are_keys:
            specs.append(WeightSpec(p + "v", (self.v_size, W)))
        if self.has_gate:
            specs.append(WeightSpec(p + "g", (self.out_size, W)))
        if self.norm is not None:
            for n, rows in (("q.norm", self.q_size), ("k.norm", self.k_size)):
                specs.append(WeightSpec(p + n, (rows if self.norm == "row" else self.dim,), init="one_plus_normal"))
        return specs

    def bind(self, store: WeightStore) -> None:
        p = self.prefix
        names = ["q", "k"] + ([] if self.values_are_keys else ["v"]) + (["g"] if self.has_gate else [])
        self.w_in = _fuse([store.take(p + n) for n in names])
        self.w_o = store.get(p + "o")
        if self.norm is not None:
            self.q_norm, self.k_norm = (store.get(p + n).float().contiguous() for n in ("q.norm", "k.norm"))
        if self.has_sink:                                         # a sink of score zero per head
            self.sink = torch.zeros(self.heads, dtype=torch.float32, device=store.device)
        if self.position is not None:
            self.position.prepare(store.device)

    def kernels(self) -> List[str]:
        return ["bias_attention"] + (["gemv"] if getattr(self, "run_dtype", None) == torch.bfloat16 else [])

    def cache_need(self) -> KVNeed:
        return KVNeed(self.kv_heads, self.dim + self.vdim, self.window, planes=1)

    def step_work(self, n_tokens, kv_tokens):
        wb = lambda w: 0 if w is None else w.numel() * w.element_size()
        proj = self.hidden * (self.gate_off + (self.out_size if self.has_gate else 0) + self.out_size)
        el = 2 if getattr(self, "run_dtype", None) == torch.bfloat16 else 4
        seen = min(kv_tokens, n_tokens * self.window) if self.window else kv_tokens
        return {"matmul": (wb(self.w_in) + wb(self.w_o), 2.0 * n_tokens * proj),
                "attn": (float(self.kv_heads * (self.dim + self.vdim) * el * seen), 2.0 * self.heads * (self.dim + self.vdim) * seen)}

    def input_weight(self) -> torch.Tensor:
        """The fused input projection's weight [q | k | v | z rows, hidden]: see `forward(projected=...)`."""
        return self.w_in

    def take_input_weight(self, w: torch.Tensor) -> None:
        """The fused input projection as part of a wider one."""
        self.w_in = w

    def forward(self, xn: torch.Tensor, ctx: StepContext, cache: LayerCache, projected: Optional[torch.Tensor] = None) -> torch.Tensor:
        """projected: float32 rows of a wider product that begin with this mixer's projection."""
        T, act, dev = xn.shape[0], ctx.act_dtype, xn.device
        rows = projected if projected is not None else linear(xn, self.w_in, out_dtype=torch.float32)
        q = torch.empty((T, self.heads, self.dim), dtype=act, device=dev)
        pe = self.position if self.position is not None and self.position.dims else None
        KB.kv_write_rot(rows, q, cache.kv if cache.writes else None, pe.freq if pe is not None else None,
                        pe.dims if pe is not None else 0, pe is None or pe.halves, 0.0, ctx.positions, ctx.seq_of_token,
                        cache.page_table, cache.page_size, self.heads, self.kv_heads, self.dim, self.vdim,
                        mag=getattr(pe, "mag", 1.0), q_norm=self.q_norm, k_norm=self.k_norm, norm_eps=self.eps,
                        norm_rows=self.norm == "row", values_are_keys=self.values_are_keys, temperature=self.temperature)
        o = paged_attention(q, cache, ctx, self.heads, self.kv_heads, self.dim, self.vdim, self.scale, window=self.window,
                            sink=self.sink, runs_min=self.RUNS_MIN)
        if self.has_gate:
            KB.elements_gate(o, rows, self.gate_off, o)
        return _output(o, self.w_o, self.hidden)


register_mixer("normed_attention", NormedAttentionMixer)
