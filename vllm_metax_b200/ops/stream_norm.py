"""Sublayer boundary of decoders whose residual is several fp32 streams (``csrc/stream_norm.cu``).

    x'_t = sum_s mix[s, t] x_s + write[t] y          (x: the streams before)
    u    = sum_t read[t] x'_t
    h    = gain * u / sqrt(mean(u^2) + eps)          the next sublayer's input

``coef`` holds ``read | write | mix`` (fp32, ``S (S + 2)`` numbers).  In front of the first sublayer there is no y and x' = x.
``Embedded`` stands for streams that nothing has been written to: all of them are the scaled embedding row.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Union

import torch

MAX_STREAMS = 8


@dataclass
class Embedded:
    table: torch.Tensor                      # [rows, width]
    ids: torch.Tensor                        # int64 [T]
    vocab: int
    scale: float
    streams: int

    def rows(self) -> torch.Tensor:
        e = self.table[self.ids].float() * self.scale
        return e[:, None].expand(-1, self.streams, -1)


def stream_norm(y: Optional[torch.Tensor], x: Union[torch.Tensor, Embedded], coef: torch.Tensor, gain: torch.Tensor, eps: float,
                want_x: bool = True):
    """Returns ``(x', h)``, ``h`` in the model's dtype.  Without ``y`` the streams pass as they are; a tensor ``x [T, S, width]`` is
    overwritten; ``x' = None`` unless ``want_x``."""
    from .. import _custom_ops as ops

    first = isinstance(x, Embedded)
    like = x.table if first else y
    S = x.streams if first else x.shape[1]
    if not ops._use_cuda(like):
        old = xn = x.rows() if first else x
        read, write, mix = coef[:S], coef[S: 2 * S], coef[2 * S:].view(S, S)
        if y is not None:
            xn = torch.einsum("st,nsw->ntw", mix, old) + write[:, None] * y.float()[:, None]
        u = torch.einsum("s,nsw->nw", read, xn)
        h = (u * torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps) * gain).to(like.dtype)
        return (x if y is None else xn) if want_x else None, h
    T, W = x.ids.numel() if first else x.shape[0], like.shape[1]
    h = torch.empty(T, W, dtype=like.dtype, device=like.device)
    x_out = None
    if want_x and y is not None:
        x_out = torch.empty(T, S, W, dtype=torch.float32, device=like.device) if first else x
    source = (x.table, x.ids, x.vocab, x.scale) if first else (None, None, 0, 1.0)
    torch.ops.b200.stream_norm(h, x_out, y, None if first else x, coef, gain, eps, *source, S)
    return (x if y is None else x_out) if want_x else None, h
