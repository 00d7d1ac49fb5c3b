"""Independent pieces of a few-token step beside one another.

A decode step's kernels are too small to fill the chip, so two chains that do not depend on each other
(the sides of a parallel mixer, a shared expert beside the routed ones) take less time next to each
other than one after the other::

    fork = Fork(device)          # the side stream waits for what has been launched so far
    with fork:
        ...                      # launches (and allocations) on the side stream
    ...                          # launches on the step's own stream
    fork.join()                  # what comes next waits for the side stream

Everything is stream order, so the same code is captured in a CUDA graph as a fork and a join.
Tensors made inside the ``with`` belong to the side stream; what they are read by outside it has to be
launched after ``join``, and they have to stay alive until then.
"""
from __future__ import annotations

import torch

# Steps of at most this many tokens fork; longer ones fill the chip with one chain.
FORK_MAX_TOKENS = 64
_STREAMS = {}
_off = False


def side_streams_off(on: bool) -> None:
    """Launch everything on the step's own stream (tests compare both ways)."""
    global _off
    _off = bool(on)


def forks(tokens: int) -> bool:
    return not _off and tokens <= FORK_MAX_TOKENS


class Fork:
    def __init__(self, device):
        key = torch.device(device).index or 0
        if key not in _STREAMS:
            _STREAMS[key] = torch.cuda.Stream(device=device)
        self.side = _STREAMS[key]
        self.main = torch.cuda.current_stream(device)
        self.side.wait_stream(self.main)
        self._within = torch.cuda.stream(self.side)

    def __enter__(self):
        self._within.__enter__()
        return self

    def __exit__(self, *exc):
        return self._within.__exit__(*exc)

    def join(self) -> None:
        self.main.wait_stream(self.side)
