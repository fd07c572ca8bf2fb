"""Rotation angles of a step, computed once per rotation and shared by all layers that have it."""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from ..attention.metadata import get_forward_context


class Rotation(nn.Module):
    """``inv_freq``: fp64 frequencies of the rotated pairs."""

    def __init__(self, inv_freq: torch.Tensor):
        super().__init__()
        self.key = ("rope_angles", tuple(inv_freq.tolist()))
        self.register_buffer("inv_freq", inv_freq.double().to(torch.get_default_device()), persistent=False)

    def angles(self, positions: torch.Tensor, tokens: int) -> torch.Tensor:
        """Cosines and sines ``[tokens, 2, pairs]`` of the step's tokens."""
        extra = get_forward_context().extra
        hit = extra.get(self.key)
        if hit is None:
            hit = extra[self.key] = ops.rope_angles(positions, self.inv_freq, tokens)
        return hit
