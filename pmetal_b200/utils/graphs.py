"""CUDA-graph capture."""
from __future__ import annotations

import contextlib
import gc

import torch


@contextlib.contextmanager
def capture(graph: "torch.cuda.CUDAGraph"):
    """``torch.cuda.graph(graph)`` during which the garbage collector rests: a graph that it frees meanwhile (models in reference
    cycles hold their graphs until a collection) resets on the capturing thread, which invalidates the capture."""
    gc.collect()
    was = gc.isenabled()
    gc.disable()
    try:
        with torch.cuda.graph(graph):
            yield
    finally:
        if was:
            gc.enable()
