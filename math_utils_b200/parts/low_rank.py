"""A projection through two matrices of a small inner size, as the recurrent mixers use it for decays and gates.

The first matrix [rank, hidden] rides in the mixer's stacked input product; the second [n, rank] is applied by
``ops.low_rank`` together with what follows it (a bias, a decay's nonlinearity), in float32.  No key of a
configuration gives the rank: it is a ``FreeSize`` that the weight file fixes.
"""
from __future__ import annotations

import torch

from .base import FreeSize, TensorSpec


class LowRank:
    def __init__(self, part, down: str, up: str, n: int, hidden_size: int, default_rank: int):
        """``down`` and ``up``: the part's tensor roles of the two matrices; ``n``: outputs."""
        self.down_name, self.up_name = part.tensor_name(down), part.tensor_name(up)
        self.n, self.hidden_size = n, hidden_size
        self.free = FreeSize(self.down_name, max(1, default_rank))
        self.rank = 0                       # known once the weights are
        self._made = {}

    def tensor_specs(self):
        return (TensorSpec(self.down_name, (self.free, self.hidden_size)), TensorSpec(self.up_name, (self.n, self.free)))

    def bind(self, tensors) -> None:
        """The inner size is padded with zeros to a multiple of 16: whole pieces for the tensor cores."""
        self.down, self.up = tensors[self.down_name], tensors[self.up_name]
        pad = -self.down.shape[0] % 16
        if pad:
            self.down = torch.nn.functional.pad(self.down, (0, 0, 0, pad))
            self.up = torch.nn.functional.pad(self.up, (0, pad)).contiguous()
        self.rank = self.down.shape[0]

    def part(self, ops, col: int, out, **what):
        """What ``ops.low_rank`` takes for this projection: its first product's columns start at ``col``.  Made once
        per output buffer."""
        key = (out.data_ptr(), out.shape[0], col)
        made = self._made.get(key)
        if made is None:
            if len(self._made) > 64:
                self._made.clear()
            made = self._made[key] = ops.low_rank_part(self.up, col, out, **what)
        return made
