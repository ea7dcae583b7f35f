"""Streams beside the main one, for work that meets the rest of a layer only later.

``fork(device, name)`` gives the named stream of a device, made to wait for everything enqueued so far on the current one
(inside a graph capture: a fork; the caller joins with ``current.wait_stream(stream)``).  Parts that may run at the same
time use different names.  A tensor made on such a stream may be read on the stream that joined it; its memory goes back
to the named stream, whose next use of it comes after the next fork and so after that reader."""
from __future__ import annotations

from typing import Dict, Tuple

import torch

_streams: Dict[Tuple[int, str], "torch.cuda.Stream"] = {}


def fork(device: torch.device, name: str) -> "torch.cuda.Stream":
    key = (torch.device(device).index or 0, name)
    s = _streams.get(key)
    if s is None:
        s = _streams[key] = torch.cuda.Stream(device=device)
    s.wait_stream(torch.cuda.current_stream(device))
    return s
