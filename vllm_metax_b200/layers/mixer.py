"""Sequence mixers between one merged input product and one output product.

A branch reads its parts of the input product's rows and writes its columns of the output product's operand:

    in_parts() -> {name: rows}      attach(proj, prefix)      in_slots(proj), out_slot(weight): where checkpoint tensors go
    out_width, runs                 mix(positions, h, p, out, run)

Several branches side by side share both products: the sum of their outputs is formed in the output product's accumulators,
with a branch's factor applied to its operand columns in fp32 (``out_scale`` of the branches).
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from .recurrent import StackedLinear, _param


class ProjectedMixer(nn.Module):
    def __init__(self, width: int, branches: dict[str, nn.Module], dtype=torch.bfloat16):
        """``branches``: name ("" for a single one) -> branch."""
        super().__init__()
        self.names = list(branches)
        self.branches = nn.ModuleList(branches.values())
        parts, biased = {}, []
        self.spans, at = [], 0
        for n, b in self.items():
            for name, rows in b.in_parts().items():
                parts[self.prefix(n) + name] = rows
            if getattr(b, "proj_bias", False):
                biased.append(n)
            self.spans.append((at, at + b.out_width))
            at += b.out_width
        self.in_proj = StackedLinear(width, parts, tuple(biased), dtype=dtype)
        self.out_proj = _param(width, at, dtype=dtype)
        for n, b in self.items():
            b.attach(self.in_proj, self.prefix(n))

    @staticmethod
    def prefix(name: str) -> str:
        return name + "." if name else ""

    def items(self):
        return zip(self.names, self.branches)

    def slots(self) -> dict:
        out = {}
        for (n, b), (lo, hi) in zip(self.items(), self.spans):
            named = {**b.in_slots(self.in_proj), "o": b.out_slot(self.out_proj.data[:, lo:hi])}
            out.update({self.prefix(n) + k: v for k, v in named.items()})
        return out

    def forward(self, positions: torch.Tensor, h: torch.Tensor, run: int = 0) -> torch.Tensor:
        p = self.in_proj(h)
        o = torch.empty(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)
        for b, (lo, hi) in zip(self.branches, self.spans):
            b.mix(positions, h, p, o[:, lo:hi], run)
        return ops.gemm(o, self.out_proj)
