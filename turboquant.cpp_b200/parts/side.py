"""A second stream for work that does not wait for what the main stream does meanwhile.

    side = fork(device);  with torch.cuda.stream(side): ...;  main-stream work;  join(side)

What is allocated on the second stream may be read on the main one after the join, and is not handed out again before the
second stream has waited for the main one at the next fork; what the main stream allocated and the second reads stays
referenced until the join.  Decode graphs record the fork and the join."""
from __future__ import annotations

import os

import torch

ENABLED = os.environ.get("TQ_NO_SIDE_BY_SIDE", "") in ("", "0")
_streams = {}


def fork(device) -> torch.cuda.Stream:
    """The device's second stream, waiting for what the current one has been given so far."""
    key = torch.device(device).index
    if key not in _streams:
        _streams[key] = torch.cuda.Stream(device=device)
    _streams[key].wait_stream(torch.cuda.current_stream())
    return _streams[key]


def join(side: torch.cuda.Stream) -> None:
    torch.cuda.current_stream().wait_stream(side)
