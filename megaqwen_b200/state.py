"""What a sequence leaves behind for its next tokens, layer run by layer run.

A run is one pass of one layer: a layer that the model loops over has as many
runs as passes, and each keeps its own.  Two kinds exist: a *cache* with a row
per position (latents of latent attention, keys and values), whose rows beyond
the position are never read and need no clearing, and a *recurrent state* of fixed
size (lightning attention, gated linear attention, Mamba-2 with the last inputs of
its convolution), which must be zero where a sequence begins.
"""
from __future__ import annotations

import ctypes as C

import torch


class SequenceState:
    """Device memory of all runs.  ``sizes``: (bytes, recurrent) per run."""

    def __init__(self, sizes, device):
        self.recurrent = [bool(r) for _, r in sizes]
        self.buffers = [torch.zeros(int(n), dtype=torch.uint8, device=device) for n, _ in sizes]
        self.pointers = (C.c_void_p * len(self.buffers))(*[b.data_ptr() for b in self.buffers])

    def reset(self) -> None:
        for b, recurrent in zip(self.buffers, self.recurrent):
            if recurrent:
                b.zero_()

    def nbytes(self) -> int:
        return sum(b.numel() for b in self.buffers)

    def snapshot(self) -> list:
        """Copies of the recurrent states (a cache needs none: its rows stay valid)."""
        return [b.clone() if r else None for b, r in zip(self.buffers, self.recurrent)]

    def restore(self, saved) -> None:
        for b, s in zip(self.buffers, saved):
            if s is not None:
                b.copy_(s)
