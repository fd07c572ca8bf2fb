"""Gated linear attention with a decay per key channel (``csrc/gla.cu``), with its fp32 PyTorch statement.

    S <- diag(alpha) S + k v^T;  o = S^T (scale q)
    out = o / sqrt(mean(o^2) + eps) * norm_w * silu(g)              per head over its value columns

``qkvg [T, *]`` is the merged projection's output with q, k, v and g (heads side by side) at column offsets; ``alpha`` is
fp32 ``[T, H * dim]``; ``state [slots, H, dim, vdim]`` (fp32) is read where ``has_initial_state`` says so and always written
back at ``state_indices``.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn.functional as F


def gated_linear_attention_ref(qkvg, offsets, alpha, norm_w, state, query_start_loc, state_indices, has_initial_state,
                               scale, eps):
    H, D, V = state.shape[1:]
    T = qkvg.shape[0]
    qo, ko, vo, go = offsets
    q = qkvg[:, qo: qo + H * D].float().reshape(T, H, D) * scale
    k = qkvg[:, ko: ko + H * D].float().reshape(T, H, D)
    v = qkvg[:, vo: vo + H * V].float().reshape(T, H, V)
    g = qkvg[:, go: go + H * V].float()
    alpha = alpha.float().reshape(T, H, D)
    o = torch.zeros(T, H, V, dtype=torch.float32, device=qkvg.device)
    qsl = query_start_loc.tolist()
    for b in range(len(qsl) - 1):
        slot = int(state_indices[b]) if state_indices is not None else -1
        use = slot >= 0 and (has_initial_state is None or bool(has_initial_state[b]))
        S = state[slot].clone() if use else torch.zeros(H, D, V, dtype=torch.float32, device=qkvg.device)
        for t in range(qsl[b], qsl[b + 1]):
            S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        if slot >= 0 and qsl[b + 1] > qsl[b]:
            state[slot] = S
    o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
    return (o.reshape(T, H * V) * F.silu(g)).to(qkvg.dtype)


def gated_linear_attention(qkvg: torch.Tensor, offsets: Sequence[int], alpha: torch.Tensor, norm_w: torch.Tensor,
                           state: torch.Tensor, query_start_loc: torch.Tensor, state_indices: Optional[torch.Tensor],
                           has_initial_state: Optional[torch.Tensor], scale: float, eps: float,
                           max_query_len: int) -> torch.Tensor:
    """``offsets`` = columns of (q, k, v, g) in ``qkvg``.  Returns ``[T, H * vdim]``; ``state`` is updated in place."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(qkvg):
        return gated_linear_attention_ref(qkvg, offsets, alpha, norm_w, state, query_start_loc, state_indices,
                                          has_initial_state, scale, eps)
    H, D, V = state.shape[1:]
    T = qkvg.shape[0]
    out = torch.empty(T, H * V, dtype=qkvg.dtype, device=qkvg.device)
    B = query_start_loc.numel() - 1
    scratch = None
    need = torch.ops.b200.gla_scratch_floats(qkvg, B, H, D, V, max_query_len)
    if need:                               # split heads or segments: further launches
        scratch = torch.empty(need, dtype=torch.float32, device=qkvg.device)
        ops._launches += 1
    torch.ops.b200.gla_recurrent(out, state, qkvg, *offsets, alpha, norm_w, scratch, query_start_loc, state_indices,
                                 has_initial_state, scale, eps, max_query_len)
    return out
