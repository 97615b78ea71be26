"""Independent parts of a step on streams of their own.

Two parts that read the same rows and write different buffers (the sub-layers of a parallel block, two mixers side by
side) have no order between them.  A decode step is a chain of short kernels, each waiting for the one before, so running
such parts next to each other shortens the chain; captured in a CUDA graph the forks and joins are edges between its
nodes and cost nothing at replay.  Prompt steps fill the device with every kernel and stay on one stream.
"""
from __future__ import annotations

from typing import Callable

import torch

USE_SIDE_STREAMS = True  # off: everything on the caller's stream, in order


def run_both(step, ctx, name: str, first: Callable, second: Callable, apart: bool = True):
    """(first(), second()); with `apart` the second on the stream `name` of the model's device during steps of single tokens.  The two
    must not touch a buffer that the other writes; what either allocates is used by the other stream only behind the
    join at the end (or, in a later step, behind that step's fork)."""
    if not (apart and USE_SIDE_STREAMS and step.all_decode and ctx.device.type == "cuda"):
        return first(), second()
    key = ("side stream", name)
    if key not in ctx.shared:
        ctx.shared[key] = torch.cuda.Stream(ctx.device)
    side = ctx.shared[key]
    here = torch.cuda.current_stream(ctx.device)
    side.wait_stream(here)
    with torch.cuda.stream(side):
        there = second()
    mine = first()
    here.wait_stream(side)
    return mine, there
