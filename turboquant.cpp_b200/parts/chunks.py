"""How a step's long runs of new tokens are cut into chunks for a recurrence that allows it (linear in its state)."""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ..kernels import ssm as KS
from .base import StepContext

MIN_CHUNK = 64           # the shortest chunk worth cutting a run into
# measured on B200, 2,048 tokens, 16 heads of 128 x 129, microseconds of both walks: one run 313, 4 chunks 251, 8 chunks 225,
# 16 chunks 212, 32 chunks 220
ROUNDS = 4
_sm_counts = {}


def cut_runs(ctx: StepContext, heads: int, columns: int) -> Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]]:
    """None, or how this step's runs are cut: (token offsets of the chunks [chunks + 1], chunk numbers [chunks], each
    sequence's chunks [sequences + 1]) on the device.  The recurrence kernel walks a run token by token with a warp per
    four of a head's `columns` columns of state; where those warps fill at most half of the GPU and a run is long,
    cutting the runs fills it (ROUNDS times over, so that the last round of blocks costs little), at the price of walking
    them once more for the states alone (half the work of a walk with outputs).  The plan depends on the step's runs and on heads and columns only, and is kept for the step's other layers."""
    lens = list(ctx.host_q_lens)
    if not lens or len(lens) != ctx.n_seqs or max(lens) < 2 * MIN_CHUNK:
        return None
    key = str(ctx.device)
    if key not in _sm_counts:
        _sm_counts[key] = torch.cuda.get_device_properties(ctx.device).multi_processor_count
    room, warps = _sm_counts[key] * KS.SCAN_WARPS_PER_SM, KS.scan_warps(len(lens), heads, columns)
    if room // warps < 2:
        return None
    cuts = ROUNDS * room // warps
    size = max(MIN_CHUNK, -(-max(lens) // cuts))
    size = -(-size // 16) * 16
    if max(lens) < 2 * size:
        return None
    name = f"run_chunks_{size}"
    plan = ctx.carry.get(name) if ctx.carry is not None else None
    if plan is None:
        cu, seq_chunks, at = [0], [0], 0
        for n in lens:
            for c0 in range(0, n, size):
                cu.append(at + min(n, c0 + size))
            at += n
            seq_chunks.append(len(cu) - 1)
        i32 = lambda v: torch.tensor(v, dtype=torch.int32).to(ctx.device, non_blocking=True)
        plan = (i32(cu), torch.arange(len(cu) - 1, dtype=torch.int32, device=ctx.device), i32(seq_chunks))
        if ctx.carry is not None:
            ctx.carry[name] = plan
    return plan
