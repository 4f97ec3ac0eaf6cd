"""CUDA graph capture."""
from __future__ import annotations

import contextlib
import gc

import torch


@contextlib.contextmanager
def capture(graph: "torch.cuda.CUDAGraph"):
    """``torch.cuda.graph(graph)`` with the garbage collector held off: engines sit in reference cycles, and collecting
    one in the middle of a capture destroys its graphs, which CUDA forbids while a stream is capturing."""
    was_on = gc.isenabled()
    gc.disable()
    try:
        with torch.cuda.graph(graph):
            yield
    finally:
        if was_on:
            gc.enable()
