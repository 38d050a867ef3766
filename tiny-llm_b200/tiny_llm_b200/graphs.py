"""CUDA graph capture with Python's cyclic garbage collector held back.

A model that was dropped may sit in a reference cycle with graphs of its own.  Collected in the middle of another capture, it
destroys those graphs, an operation that invalidates the capture under way; inside ``capture`` the collector waits."""

from __future__ import annotations

import contextlib
import gc

import torch


@contextlib.contextmanager
def capture(graph: "torch.cuda.CUDAGraph", **kwargs):
    """``torch.cuda.graph(graph, **kwargs)``, during which nothing is collected."""
    collecting = gc.isenabled()
    gc.disable()
    try:
        with torch.cuda.graph(graph, **kwargs):
            yield
    finally:
        if collecting:
            gc.enable()
