"""
Work beside the current stream, for parts whose members do not depend on one another.

A step replayed from a CUDA graph is mostly small kernels in a row, each shorter than the machine is wide; where two chains
of them read the same input, the second goes to a stream of its own and the graph runs both at once.  Steps that are launched
kernel by kernel keep one stream: the host is what they wait for, or their kernels fill the device.

    side = fork(rt, ctx, "name")          # None: not overlapped, stay on the current stream
    with on(side): a = ...
    b = ...
    join(side)                            # from here on the current stream may read a

Between fork and join neither chain may write what the other reads.  Tensors made inside are freed to the side stream's
share of the allocator and handed out again there only after the next fork, which waits for everything the current stream
was given before it: a consumer enqueued before the next fork of the same name is safe.
"""

from __future__ import annotations

from contextlib import nullcontext

import torch


def fork(rt, ctx, name: str) -> torch.cuda.Stream | None:
    if not (getattr(ctx, "replayed", False) and rt.ops.overlap):
        return None
    key = ("side stream", name)
    if key not in rt.shared:
        rt.shared[key] = torch.cuda.Stream(device=rt.device)
    side = rt.shared[key]
    side.wait_stream(torch.cuda.current_stream(rt.device))
    return side


def on(side: torch.cuda.Stream | None):
    return torch.cuda.stream(side) if side is not None else nullcontext()


def join(side: torch.cuda.Stream | None) -> None:
    if side is not None:
        torch.cuda.current_stream(side.device).wait_stream(side)
