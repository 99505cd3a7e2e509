"""Two independent branches of a step on two CUDA streams (also while a graph is captured: the branch becomes a parallel path)."""
from __future__ import annotations

from typing import Callable, Dict

import torch

_side: Dict[torch.device, "torch.cuda.Stream"] = {}


def beside(device: torch.device, branch: Callable[[], None]) -> Callable[[], None]:
    """Starts ``branch`` on the device's side stream after everything issued so far; call the result to wait for it on the current
    stream. Tensors that the branch uses must live until then. On CPU the branch simply runs."""
    if device.type != "cuda":
        branch()
        return lambda: None
    if device not in _side:
        _side[device] = torch.cuda.Stream(device)
    side, cur = _side[device], torch.cuda.current_stream(device)
    side.wait_stream(cur)
    with torch.cuda.stream(side):
        branch()
    return lambda: cur.wait_stream(side)
