"""Real-gated linear recurrent unit (``csrc/rglru.cu``), with its fp32 PyTorch statement.

    r = sigmoid(zr + br);  i = sigmoid(zi + bi);  log a = decay * r
    S <- a S + sqrt(1 - a^2) i u;   out = S * gelu_tanh(y)

``gates [T, blocks, 2, width / blocks]`` (fp32) holds the logits zr, zi and is overwritten; ``decay [width]`` is
``-8 softplus(lambda)``; ``state [slots, width]`` (fp32) is carried like every recurrent state.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F


def rglru_ref(u, y, gates, r_bias, i_bias, decay, state, query_start_loc, state_indices, has_initial_state):
    T, W = u.shape
    z = gates.float().reshape(T, gates.shape[1], 2, -1)
    r = torch.sigmoid(z[:, :, 0].reshape(T, W) + r_bias)
    i = torch.sigmoid(z[:, :, 1].reshape(T, W) + i_bias)
    log_a = decay * r
    a = torch.exp(log_a)
    v = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u.float()
    out = torch.zeros(T, W, dtype=torch.float32, device=u.device)
    qsl = query_start_loc.tolist()
    for b in range(len(qsl) - 1):
        slot = int(state_indices[b]) if state_indices is not None else -1
        use = slot >= 0 and (has_initial_state is None or bool(has_initial_state[b]))
        S = state[slot].clone() if use else torch.zeros(W, dtype=torch.float32, device=u.device)
        for t in range(qsl[b], qsl[b + 1]):
            S = a[t] * S + v[t]
            out[t] = S
        if slot >= 0 and qsl[b + 1] > qsl[b]:
            state[slot] = S
    return (out * F.gelu(y.float(), approximate="tanh")).to(u.dtype)


def rglru(u: torch.Tensor, y: torch.Tensor, gates: torch.Tensor, r_bias: torch.Tensor, i_bias: torch.Tensor,
          decay: torch.Tensor, state: torch.Tensor, query_start_loc: torch.Tensor, state_indices: Optional[torch.Tensor],
          has_initial_state: Optional[torch.Tensor], max_query_len: int) -> torch.Tensor:
    """``u, y [T, width]`` (row pitch free) -> ``[T, width]``; ``state`` is updated in place."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(u):
        return rglru_ref(u, y, gates, r_bias, i_bias, decay, state, query_start_loc, state_indices, has_initial_state)
    T, W = u.shape
    out = torch.empty(T, W, dtype=u.dtype, device=u.device)
    summary = None
    chunk = torch.ops.b200.rglru_chunk()
    if max_query_len > chunk:
        summary = torch.empty((T // chunk + query_start_loc.numel() - 1) * 2 * W, dtype=torch.float32, device=u.device)
        ops._launches += 2
    torch.ops.b200.rglru_scan(out, state, gates, u, y, r_bias, i_bias, decay, gates.shape[-1], summary, query_start_loc,
                              state_indices, has_initial_state, max_query_len)
    return out
