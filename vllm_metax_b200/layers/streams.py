"""Hyper-connections with fixed weights: the residual is several streams, a sublayer reads one combination of them, and its output
goes back to every stream while the streams mix.  What stands between two sublayers - the write of the one, the read and the norm
of the other - is one launch (``ops/stream_norm.py``)."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from ..ops.stream_norm import MAX_STREAMS, stream_norm
from .basic import NormAroundOne
from .recurrent import _param


class HyperConnection(nn.Module):
    """The weights of one sublayer: what it reads of each stream, what each stream takes of its output, and the mix [from, to]."""

    def __init__(self, streams: int, dtype):
        super().__init__()
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"{streams} residual streams; 1 to {MAX_STREAMS} are supported")
        self.read, self.write = _param(streams, dtype=dtype), _param(streams, dtype=dtype)
        self.mix = _param(streams, streams, dtype=dtype)

    def slots(self) -> dict:
        return {"in": self.read.data, "out": self.write.data, "mix": self.mix.data}


class StreamBoundary(nn.Module):
    """Between the sublayers of ``before`` and ``after`` (None at the ends: nothing to write; the sum of the streams is read)."""

    def __init__(self, streams: int, before: Optional[HyperConnection], after: Optional[HyperConnection], norm: NormAroundOne,
                 eps: float):
        super().__init__()
        self.streams, self.before, self.after, self.norm, self.eps = streams, before, after, norm, eps
        self.register_buffer("coef", torch.ones(streams * (streams + 2), dtype=torch.float32), persistent=False)

    def finalize_weights(self) -> None:
        S = self.streams
        if self.after is not None:
            self.coef[:S] = self.after.read.data.float()
        if self.before is not None:
            self.coef[S: 2 * S] = self.before.write.data.float()
            self.coef[2 * S:] = self.before.mix.data.float().flatten()
        self.norm.finalize_weights()

    def forward(self, y, x):
        return stream_norm(y, x, self.coef, self.norm.gain, self.eps, want_x=self.after is not None)
