"""Streams beside the main one, for work that meets the rest of a layer only later.

``fork(device, name, apart)`` gives the named stream of a device, made to wait for everything enqueued so far on the current
one (inside a graph capture: a fork), or, when not ``apart``, the current stream itself; ``join(stream)`` makes the current
stream wait for it.  Parts that may run at the same time use different names.  A tensor made on such a stream may be read
on the stream that joined it; its memory goes back to the named stream, whose next use of it comes after the next fork and
so after that reader.

Decode steps are replayed as graphs of short kernels that leave most of the GPU idle: there a fork costs the host nothing
and halves of a layer run side by side (1.17 -> 0.83 ms a step at width 2048 and batch 8).  A prompt's kernels fill the GPU
one after the other and every stream switch is host time (width 1024: 4.8 against 5.4 ms; 4096: no difference), so parts
fork in decode-only steps alone.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

_streams: Dict[Tuple[int, str], "torch.cuda.Stream"] = {}


def fork(device: torch.device, name: str, apart: bool = True) -> "torch.cuda.Stream":
    current = torch.cuda.current_stream(device)
    if not apart:
        return current
    key = (torch.device(device).index or 0, name)
    s = _streams.get(key)
    if s is None:
        s = _streams[key] = torch.cuda.Stream(device=device)
    s.wait_stream(current)
    return s


def join(stream: "torch.cuda.Stream") -> None:
    current = torch.cuda.current_stream(stream.device)
    if stream != current:
        current.wait_stream(stream)
