"""Sublayer boundary of pre-norm decoders with layer norms and an fp32 residual stream (``csrc/prenorm.cu``).

    x' = x + y (+ add)                                                   fp32
    h  = gain * (x' - mean(x')) / sqrt(mean((x' - mean)^2) + eps)        the next sublayer's input

``y`` is a sublayer's output, rows of an embedding table (``ids``), an fp32 product, or the expert-sorted rows of a
mixture-of-experts layer (:class:`ops.residual_norm.ExpertRows`): the kernel forms the sums itself.

Where the stream re-enters a loop through a product W [x'; x0], ``loop_operand`` writes that product's operand instead of h.
In 16-bit models it holds x' as the sum of two 16-bit numbers, so that the stream keeps its precision.
"""
from __future__ import annotations

from typing import Optional, Union

import torch

from .residual_norm import ExpertRows


def _sum(y, x, add, ids):
    if isinstance(y, ExpertRows):
        y = y.combined()
    xn = (y if ids is None else y[ids]).float()
    if x is not None:
        xn = x + xn
    return xn if add is None else xn + add.float()


def layer_normed(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps) * gain.float()


def _launch(y, x, add, ids, vocab, gain, eps, h, x_out, table=None, table_ids=None):
    late = isinstance(y, ExpertRows)
    extra = (y.weights, y.inv_pos, y.topk, y.shared) if late else (None, None, 0, None)
    torch.ops.b200.prenorm(h, x_out, y.rows if late else y, x, add, gain, eps, ids, vocab, *extra, table, table_ids)


def _tokens(y, ids):
    return ids.numel() if ids is not None else y.tokens if isinstance(y, ExpertRows) else y.shape[0]


def prenorm(y: Union[torch.Tensor, ExpertRows], x: Optional[torch.Tensor], gain: torch.Tensor, eps: float,
            add: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None, vocab: int = 0, want_x: bool = True):
    """Returns ``(x', h)``, ``h`` in ``gain``'s dtype (``x' = None`` unless ``want_x``).  ``x=None``: ``x' = y (+ add)``."""
    from .. import _custom_ops as ops

    rows = y.rows if isinstance(y, ExpertRows) else y
    if not ops._use_cuda(rows):
        xn = _sum(y, x, add, ids)
        return (xn if want_x else None), layer_normed(xn, gain, eps).to(gain.dtype)
    T, W = _tokens(y, ids), rows.shape[1]
    x_out = torch.empty(T, W, dtype=torch.float32, device=rows.device) if want_x else None
    h = torch.empty(T, W, dtype=gain.dtype, device=rows.device)
    _launch(y, x, add, ids, vocab, gain, eps, h, x_out)
    return x_out, h


def loop_operand(y: Union[torch.Tensor, ExpertRows], x: Optional[torch.Tensor], table: torch.Tensor, ids: torch.Tensor,
                 vocab: int, gather: bool = False) -> torch.Tensor:
    """``[x'; table[ids]]`` of ``x' = x + y``: fp32 ``[T, 2 W]``, or 16-bit ``[T, 3 W]`` with x' split into ``hi + lo``.
    ``gather``: y is the table too (a loop in front of the first layer)."""
    from .. import _custom_ops as ops

    y_ids = ids if gather else None
    if not ops._use_cuda(table):
        xn, x0 = _sum(y, x, None, y_ids), table[ids]
        hi = xn.to(table.dtype)
        return torch.cat([hi, x0] if table.dtype == torch.float32 else [hi, (xn - hi.float()).to(table.dtype), x0], -1)
    T, W = ids.numel(), table.shape[1]
    out = torch.empty(T, (2 if table.dtype == torch.float32 else 3) * W, dtype=table.dtype, device=table.device)
    _launch(y, x, None, y_ids, vocab, None, 0.0, out, None, table, ids)
    return out
