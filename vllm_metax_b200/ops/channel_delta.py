"""Gated delta rule with a decay per key channel (``csrc/channel_delta.cu``), with its fp32 PyTorch statement.

    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q         q, k unit vectors, q times dim^(-1/2)
    out = out_scale * unit_rms(o) * norm_w * sigmoid(gate)                      per head over its value columns

``qkv [T, *]`` holds q and k (``kv_heads`` x dim) and v (H x vdim) at column offsets, value head h using key head
h // (H / kv_heads); ``g`` (fp32 ``[T, H * dim]``) holds the decays, ``beta`` (fp32 ``[T, H]``) the logits of the step sizes;
``state [slots, H, dim, vdim]`` (fp32) is carried like every recurrent state.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from .gla import Steps, _carried


def channel_delta_rule_ref(qkv, offsets, kv_heads, g, beta, gate, norm_w, state, steps: Steps, eps, out_scale=1.0):
    H, D, V = state.shape[1:]
    T, G = qkv.shape[0], kv_heads
    qo, ko, vo = offsets
    q, k = (qkv[:, a: a + G * D].float().reshape(T, G, D) for a in (qo, ko))
    q, k = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6) for x in (q, k))
    q, k = (q * D ** -0.5).repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    v = qkv[:, vo: vo + H * V].float().reshape(T, H, V)
    g, b_ = g[:, : H * D].float().reshape(T, H, D), torch.sigmoid(beta[:, :H].float())
    o = torch.zeros(T, H, V, dtype=torch.float32, device=qkv.device)
    qsl = steps.query_start_loc.tolist()
    for b in range(len(qsl) - 1):
        slot, use = _carried(steps, b)
        S = state[slot].clone() if use else torch.zeros(H, D, V, dtype=torch.float32, device=qkv.device)
        for t in range(qsl[b], qsl[b + 1]):
            S = g[t][:, :, None] * S
            u = b_[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        if slot >= 0 and qsl[b + 1] > qsl[b]:
            state[slot] = S
    o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
    return (o.reshape(T, H * V) * torch.sigmoid(gate[:, : H * V].float()) * out_scale).to(qkv.dtype)


def channel_delta_rule(qkv: torch.Tensor, offsets: Sequence[int], kv_heads: int, g: torch.Tensor, beta: torch.Tensor,
                       gate: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor, steps: Steps, eps: float,
                       out_scale: float = 1.0, out: Optional[torch.Tensor] = None, shape: int = 0) -> torch.Tensor:
    """``offsets`` = columns of (q, k, v).  Returns ``[T, H * vdim]`` (``out``: rows may be part of wider ones); ``state`` is
    updated in place.  ``shape``: pins the kernel's lanes per column * 1000 + columns per CTA (0: chosen from the sizes)."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(qkv):
        y = channel_delta_rule_ref(qkv, offsets, kv_heads, g, beta, gate, norm_w, state, steps, eps, out_scale)
        return y if out is None else out.copy_(y)
    H, D, V = state.shape[1:]
    T, B = qkv.shape[0], steps.query_start_loc.numel() - 1
    if out is None:
        out = torch.empty(T, H * V, dtype=qkv.dtype, device=qkv.device)
    need = torch.ops.b200.channel_delta_scratch_floats(qkv, B, H, kv_heads, D, V, steps.max_query_len, shape)
    scratch = torch.empty(need, dtype=torch.float32, device=qkv.device) if need else None
    ops._launches += need > 0
    torch.ops.b200.channel_delta(out, state, qkv, *offsets, kv_heads, g, beta, gate, norm_w, scratch, *steps[:3], eps, out_scale,
                                 steps.max_query_len, shape)
    return out
