"""A mixer that can run beside others on one input.

A branch offers, beyond what every mixer does: ``in_names`` (its input matrices' tensor names, in the order of its columns), ``in_width`` and
``core_width`` (columns it takes of a combination's input product and gives to an output product), ``out_name``, and ``core(proj, col0, step,
cache, out, scale)``, which works from the branch's columns of the input product (kept in float) to what its output projection reads.
Used alone, a branch is an ordinary mixer.
"""
from __future__ import annotations

from typing import Mapping

import torch

from .. import ops
from .base import Mixer


def common_dtype(tensors) -> torch.dtype:
    return torch.float32 if any(t.dtype == torch.float32 for t in tensors) else tensors[0].dtype


class Branch(Mixer):
    in_names: tuple[str, ...]
    out_name: str
    in_width: int
    core_width: int
    hidden: int

    def core(self, proj: torch.Tensor, col0: int, step, cache, out: torch.Tensor, scale: float) -> None:
        """``proj`` [tokens, *] float: this branch's input projections start at column ``col0``.  Write what the output
        projection reads, times ``scale``, to ``out`` [tokens, core_width] (a view, activation type)."""
        raise NotImplementedError

    def load_core(self, tensors: Mapping[str, torch.Tensor]) -> None:
        """Everything but the input and output matrices."""

    def load(self, tensors: Mapping[str, torch.Tensor]) -> None:
        mats = [tensors[name] for name in self.in_names]
        dtype = common_dtype(mats)
        self.w_in = torch.cat([m.to(dtype) for m in mats], dim=0).contiguous()
        self.w_o = tensors[self.out_name].contiguous()
        self.load_core(tensors)

    def forward(self, x, step, cache, own_cache):
        if cache is None or not own_cache:
            raise ValueError(f"{type(self).__name__} keeps something per request; the schedule gave it none")
        proj = ops.linear(x, self.w_in, None, torch.float32)
        out = torch.empty((x.shape[0], self.core_width), dtype=self.dtype, device=x.device)
        self.core(proj, 0, step, cache, out, 1.0)
        return ops.linear(out, self.w_o, None, self.dtype, may_leave_partials=True)  # the result is a residual delta
