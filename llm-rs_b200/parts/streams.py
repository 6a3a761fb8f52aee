"""Independent branches of a captured step on streams of their own.

A decode step is a chain of small kernels that leave most of the device idle. Where a part knows two chains that do not read
each other's results, it runs one of them ``beside`` the other while the step is captured in a CUDA graph: they become parallel
branches of the graph. Steps that are not captured stay on one stream (prompt portions fill the device by themselves).

Memory: what is allocated inside ``beside`` belongs to the side stream and is used again by it only; what the side stream reads
must be kept alive by the caller until ``join``."""
from __future__ import annotations

import os

import torch

# LLMRS_FORK_BRANCHES=0 keeps the branches of a captured step one after the other.
FORK_BRANCHES = os.environ.get("LLMRS_FORK_BRANCHES", "1") != "0"
FORK_MAX_TOKENS = 64
_STREAMS = {}


def forks(n_tokens: int) -> bool:
    """Whether a step of so many tokens runs independent branches side by side."""
    return FORK_BRANCHES and n_tokens <= FORK_MAX_TOKENS and torch.cuda.is_current_stream_capturing()


class beside:
    """``with beside(k, device) as branch: ...`` runs the body on side stream ``k`` after what the current stream has been given so
    far; ``branch.join()`` makes the current stream wait for it. Nested uses take different numbers."""

    def __init__(self, number: int, device):
        # Ahead of the main stream where both have work: the side branch is the longer one.
        if (number, device) not in _STREAMS:
            _STREAMS[number, device] = torch.cuda.Stream(device, priority=-1)
        self.stream = _STREAMS[number, device]

    def __enter__(self):
        self.stream.wait_stream(torch.cuda.current_stream())
        self._guard = torch.cuda.stream(self.stream)
        self._guard.__enter__()
        return self

    def __exit__(self, *exc):
        return self._guard.__exit__(*exc)

    def join(self) -> None:
        torch.cuda.current_stream().wait_stream(self.stream)
