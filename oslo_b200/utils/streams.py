"""Two independent pieces of a step at the same time: a fork and a join inside a captured CUDA graph."""
from __future__ import annotations

from typing import Any, Callable, Dict, Tuple

import torch
from torch import Tensor

_SIDE: Dict[int, "torch.cuda.Stream"] = {}


def beside(main: Callable[[], Any], side: Callable[[], Any], like: Tensor) -> Tuple[Any, Any]:
    """``(main(), side())``. While ``like``'s device captures a graph ``side`` is captured on a stream of its own, so that a replay runs the two
    next to each other; what either returns may be used once both have been. Memory: the side stream starts from where the
    capturing one is and is joined before this returns, so a block that one of them gives back is never reused under the other."""
    if not (like.is_cuda and torch.cuda.is_initialized() and torch.cuda.is_current_stream_capturing()):
        return main(), side()
    current = torch.cuda.current_stream(like.device)
    stream = _SIDE.setdefault(current.device_index, torch.cuda.Stream(like.device))
    stream.wait_stream(current)
    with torch.cuda.stream(stream):
        second = side()
    first = main()
    current.wait_stream(stream)
    return first, second
