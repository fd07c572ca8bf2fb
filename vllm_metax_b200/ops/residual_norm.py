"""Sublayer boundary of decoders that norm both sides of a sublayer and keep an fp32 residual stream
(``csrc/residual_norm.cu``); with no stream to write, the last boundary in front of the LM head.

    x' = x + gain * y / sqrt(mean(y^2) + eps)                    fp32
    h  = gain_out * x' / sqrt(mean(x'^2) + eps)                  the next sublayer's input, in y's dtype

Gains have one entry or one per channel.  ``y`` may still be the expert-sorted rows of a mixture-of-experts layer
(:class:`ExpertRows`): the kernel forms the weighted sums itself.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Union

import torch


@dataclass
class ExpertRows:
    """What the grouped expert products left: the rows of pair (t, k) is ``rows[inv_pos[t * topk + k]]``; pairs whose id is at
    least ``identity_from`` are identity experts and stand for the token's own row of ``through``."""
    rows: torch.Tensor                       # [R, width], expert-sorted
    weights: Optional[torch.Tensor]          # fp32 [T, topk]; None: the rows are added as they are (weighted inputs)
    inv_pos: torch.Tensor                    # int32 [T * topk], -1: computed elsewhere
    ids: Optional[torch.Tensor] = None       # int32 [T, topk]
    through: Optional[torch.Tensor] = None   # [T, width]
    identity_from: int = 0
    shared: Optional[torch.Tensor] = None    # [T, width]
    top: int = 0                             # pairs per token (where there are no weights to tell)

    @property
    def topk(self) -> int:
        return self.top if self.weights is None else self.weights.shape[1]

    @property
    def tokens(self) -> int:
        return self.inv_pos.numel() // self.topk

    def combined(self) -> torch.Tensor:
        from .. import _custom_ops as ops

        identity = None if self.through is None else (self.ids, self.through, self.identity_from)
        w = self.weights
        if w is None:
            w = torch.ones(self.tokens, self.topk, dtype=torch.float32, device=self.rows.device)
        return ops.moe_combine(self.rows, w, self.inv_pos, self.tokens, self.shared, identity)


def normed(y: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    yf = y.float()
    return yf * torch.rsqrt(yf.pow(2).mean(-1, keepdim=True) + eps) * gain.float()


def boundary_norm(y: Union[torch.Tensor, ExpertRows], x: Optional[torch.Tensor], gain: Optional[torch.Tensor],
                  gain_out: torch.Tensor, eps: float, want_x: bool = True):
    """Returns ``(x', h)`` (``x' = None`` unless ``want_x``).  ``x=None``: ``x' = y``."""
    from .. import _custom_ops as ops

    late = isinstance(y, ExpertRows)
    rows = y.rows if late else y
    T = y.tokens if late else y.shape[0]
    if not ops._use_cuda(rows):
        yt = y.combined() if late else y
        xn = yt.float() if x is None else x + normed(yt, gain, eps)
        return (xn if want_x else None), normed(xn, gain_out, eps).to(rows.dtype)
    x_out = torch.empty(T, rows.shape[1], dtype=torch.float32, device=rows.device) if want_x else None
    h = torch.empty(T, rows.shape[1], dtype=rows.dtype, device=rows.device)
    extra = (y.weights, y.inv_pos, y.ids, y.through, y.identity_from, y.shared) if late else (None, None, None, None, 0, None)
    torch.ops.b200.residual_norm(h, x_out, rows, x, None if x is None else gain, gain_out, eps, 1.0, None, 0, *extra)
    return x_out, h


def embed_norm(table: torch.Tensor, ids: torch.Tensor, vocab: int, scale: float, gain_out: torch.Tensor, eps: float):
    """``x' = scale * table[ids]`` in fp32 and its norm: the embedding and the boundary in front of the first layer."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(table):
        xn = table[ids].float() * scale
        return xn, normed(xn, gain_out, eps).to(table.dtype)
    x_out = torch.empty(ids.numel(), table.shape[1], dtype=torch.float32, device=table.device)
    h = torch.empty(ids.numel(), table.shape[1], dtype=table.dtype, device=table.device)
    torch.ops.b200.residual_norm(h, x_out, table, None, None, gain_out, eps, scale, ids, vocab, None, None, None, None, 0, None)
    return x_out, h


def residual_norm(y: torch.Tensor, x: Optional[torch.Tensor], gain: Optional[torch.Tensor], gain_out: torch.Tensor,
                  eps: float) -> torch.Tensor:
    """``norm(x + norm(y))`` with gains ``gain_out`` and ``gain`` - the hidden states the LM head reads."""
    return boundary_norm(y, x, gain, gain_out, eps, want_x=False)[1]
