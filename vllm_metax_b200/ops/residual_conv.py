"""Sublayer boundary of post-norm decoders with an fp32 residual stream and a short input convolution
(``csrc/residual_conv.cu``).

    x' = x + gain * y / sqrt(mean(y^2) + eps)                    fp32
    h  = x' + sum_j w[:, j] * x'[t - (K-1) + j]                  the next sublayer's input, in y's dtype

``gain`` has one entry or one per channel.  ``carry [slots, K-1, D]`` (fp32, oldest first) holds the last inputs of every
request between steps; sequences of a step are given by ``query_start_loc``, their slots by ``state_indices`` and whether
the slot holds history by ``has_initial_state``.
"""
from __future__ import annotations

from typing import Optional

import torch

from .residual_norm import normed


def residual_conv_ref(y, x, gain, w, eps, carry, query_start_loc, state_indices, has_initial_state):
    xn = y.float() if x is None else x + normed(y, gain, eps)
    T, D = xn.shape
    K = w.shape[1]
    h = torch.empty_like(xn)
    qsl = query_start_loc.tolist()
    wf = w.float()
    for b in range(len(qsl) - 1):
        s, e = qsl[b], qsl[b + 1]
        if e <= s:
            continue
        slot = int(state_indices[b]) if state_indices is not None else -1
        use = slot >= 0 and carry is not None and (has_initial_state is None or bool(has_initial_state[b]))
        prev = carry[slot] if use else torch.zeros(K - 1, D, dtype=xn.dtype, device=xn.device)
        ext = torch.cat([prev, xn[s:e]], 0)
        h[s:e] = xn[s:e] + (ext.unfold(0, K, 1) * wf[None]).sum(-1)
        if slot >= 0 and carry is not None and K > 1:
            carry[slot] = ext[-(K - 1):]
    return xn, h.to(y.dtype)


def residual_conv(y: torch.Tensor, x: Optional[torch.Tensor], gain: Optional[torch.Tensor], w: torch.Tensor, eps: float,
                  carry: Optional[torch.Tensor], query_start_loc: torch.Tensor,
                  state_indices: Optional[torch.Tensor] = None, has_initial_state: Optional[torch.Tensor] = None):
    """Returns ``(x', h)``; with ``x=None`` (in front of the first layer) ``x' = y``."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(y):
        return residual_conv_ref(y, x, gain, w, eps, carry, query_start_loc, state_indices, has_initial_state)
    x_out = torch.empty(y.shape, dtype=torch.float32, device=y.device)
    h = torch.empty_like(y)
    torch.ops.b200.residual_conv(x_out, h, y, x, None if x is None else gain, w, carry if w.shape[1] > 1 else None,
                                 query_start_loc, state_indices, has_initial_state, eps)
    return x_out, h
