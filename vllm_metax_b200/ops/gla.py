"""Linear attention with a decay (``csrc/gla.cu``), with its fp32 PyTorch statement.

    S <- decay S + k v^T;  o = S^T (scale q)
    out = out_scale * unit_rms(o) * norm_w * act(g)              per head over its value columns, or over all heads together

The decay is one number per key channel and token (gated linear attention), per head (lightning attention) or per head and
token (matrix memory).  ``qkvg [T, *]`` is the merged projection's output with q, k, v and g (heads side by side) at column
offsets; ``state [slots, H, dim, vdim]`` (fp32) is read where ``has_initial_state`` says so and always written back at
``state_indices``.

The matrix memory of xLSTM stabilises its exponential gates with a running maximum (``memory_gates``) and divides the read-out
by a normaliser state that is carried like S with ones for v:

    top' = max(f + top, i);  decay = exp(f + top - top');  k <- exp(i - top') k;  floor = exp(-top')
    o = S^T q / (max(|n . q|, floor) + 1e-6)
"""
from __future__ import annotations

from typing import NamedTuple, Optional, Sequence

import torch
import torch.nn.functional as F


class Steps(NamedTuple):
    """The sequences of a step and where their carried state lives."""
    query_start_loc: torch.Tensor                   # int32 [B + 1]
    state_indices: Optional[torch.Tensor]           # int32 [B], negative: nothing is carried
    has_initial_state: Optional[torch.Tensor]       # int32 [B]
    max_query_len: int


class Normalizer(NamedTuple):
    """What turns linear attention into a matrix memory."""
    state: torch.Tensor                             # fp32 [slots, H, ceil(vdim / 16), dim], equal copies along the third
    k_mul: torch.Tensor                             # fp32 [T, H]
    floor: torch.Tensor                             # fp32 [T, H]


GATES = {"silu": F.silu, "sigmoid": torch.sigmoid}


def _carried(steps: Steps, b: int) -> tuple[int, bool]:
    slot = int(steps.state_indices[b]) if steps.state_indices is not None else -1
    return slot, slot >= 0 and (steps.has_initial_state is None or bool(steps.has_initial_state[b]))


def linear_attention_ref(qkvg, offsets, decay, norm_w, state, steps: Steps, scale, eps, gate="silu", silu_qkv=False,
                         whole_row=False, memory: Optional[Normalizer] = None, out_scale=1.0):
    H, D, V = state.shape[1:]
    T = qkvg.shape[0]
    qo, ko, vo, go = offsets
    q, k = (qkvg[:, a: a + H * D].float().reshape(T, H, D) for a in (qo, ko))
    v = qkvg[:, vo: vo + H * V].float().reshape(T, H, V)
    g = qkvg[:, go: go + H * V].float()
    if silu_qkv:
        q, k, v = F.silu(q), F.silu(k), F.silu(v)
    q = q * scale
    if memory is not None:
        k = k * memory.k_mul[:T].float()[..., None]
    if decay.dim() == 1:
        decay = decay.expand(T, H)
    alpha = decay.float()[..., None].expand(T, H, D) if decay.shape[1] == H and D > 1 else decay.float().reshape(T, H, D)
    o = torch.zeros(T, H, V, dtype=torch.float32, device=qkvg.device)
    qsl = steps.query_start_loc.tolist()
    for b in range(len(qsl) - 1):
        slot, use = _carried(steps, b)
        S = state[slot].clone() if use else torch.zeros(H, D, V, dtype=torch.float32, device=qkvg.device)
        n = memory.state[slot][:, 0].clone() if use and memory is not None else torch.zeros(H, D, device=qkvg.device)
        for t in range(qsl[b], qsl[b + 1]):
            S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
            if memory is not None:
                n = alpha[t] * n + k[t]
                o[t] /= (torch.maximum((n * q[t]).sum(-1).abs(), memory.floor[t].float()) + 1e-6)[:, None]
        if slot >= 0 and qsl[b + 1] > qsl[b]:
            state[slot] = S
            if memory is not None:
                memory.state[slot] = n[:, None]
    if whole_row:
        o = o.reshape(T, 1, H * V)
    o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
    o = o.reshape(T, H, V) * norm_w.float().reshape(-1, V)
    return (o.reshape(T, H * V) * GATES[gate](g) * out_scale).to(qkvg.dtype)


def linear_attention(qkvg: torch.Tensor, offsets: Sequence[int], decay: torch.Tensor, norm_w: torch.Tensor,
                     state: torch.Tensor, steps: Steps, scale: float, eps: float, gate: str = "silu", silu_qkv: bool = False,
                     whole_row: bool = False, memory: Optional[Normalizer] = None, out_scale: float = 1.0,
                     out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``offsets`` = columns of (q, k, v, g) in ``qkvg``; ``decay`` fp32 ``[T, H * dim]`` (per key channel), ``[T, H]`` or
    ``[H]``; ``norm_w`` has one entry per value column of a head or of all heads; ``silu_qkv``: q, k and v pass silu first;
    ``whole_row``: the norm runs over all heads.  Returns ``[T, H * vdim]`` (``out``: rows may be part of wider ones);
    states are updated in place."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(qkvg):
        y = linear_attention_ref(qkvg, offsets, decay, norm_w, state, steps, scale, eps, gate, silu_qkv, whole_row, memory,
                                 out_scale)
        return y if out is None else out.copy_(y)
    H, D, V = state.shape[1:]
    T = qkvg.shape[0]
    if out is None:
        out = torch.empty(T, H * V, dtype=qkvg.dtype, device=qkvg.device)
    B = steps.query_start_loc.numel() - 1
    scratch = None
    need = torch.ops.b200.gla_scratch_floats(qkvg, B, H, D, V, steps.max_query_len, whole_row)
    if need:                               # split heads or segments: further launches
        scratch = torch.empty(need, dtype=torch.float32, device=qkvg.device)
        ops._launches += 1
    torch.ops.b200.gla_recurrent(out, state, qkvg, *offsets, decay, norm_w, scratch, *steps[:3], scale, eps,
                                 steps.max_query_len, gate == "sigmoid", silu_qkv, whole_row,
                                 *(memory if memory is not None else (None, None, None)), out_scale)
    return out


def gated_linear_attention(qkvg, offsets, alpha, norm_w, state, query_start_loc, state_indices, has_initial_state, scale, eps,
                           max_query_len):
    """Decays per key channel, head norms, a silu gate."""
    return linear_attention(qkvg, offsets, alpha, norm_w, state,
                            Steps(query_start_loc, state_indices, has_initial_state, max_query_len), scale, eps)


def memory_gates_ref(logits, bias, cap, top, steps: Steps):
    H = top.shape[1]
    z = cap * torch.tanh((logits[:, : 2 * H].float() + bias) / cap)
    i, f = z[:, :H], F.logsigmoid(z[:, H:])
    decay, k_mul, floor = (torch.zeros(logits.shape[0], H, dtype=torch.float32, device=logits.device) for _ in range(3))
    qsl = steps.query_start_loc.tolist()
    for b in range(len(qsl) - 1):
        slot, use = _carried(steps, b)
        m = top[slot].clone() if use else torch.zeros(H, dtype=torch.float32, device=logits.device)
        for t in range(qsl[b], qsl[b + 1]):
            new = torch.maximum(f[t] + m, i[t])
            decay[t], k_mul[t], floor[t] = torch.exp(f[t] + m - new), torch.exp(i[t] - new), torch.exp(-new)
            m = new
        if slot >= 0 and qsl[b + 1] > qsl[b]:
            top[slot] = m
    return decay, k_mul, floor


def memory_gates(logits: torch.Tensor, bias: torch.Tensor, cap: float, top: torch.Tensor, steps: Steps):
    """``logits [T, >= 2H]`` (fp32): input gates, then forget gates, before ``bias [2H]`` and the cap ``cap tanh(z / cap)``;
    ``top [slots, H]`` (fp32): the running maximum, updated in place.  Returns ``(decay, k_mul, floor)``, fp32 ``[T, H]``."""
    from .. import _custom_ops as ops

    if not ops._use_cuda(logits):
        return memory_gates_ref(logits, bias, cap, top, steps)
    out = torch.empty(3, logits.shape[0], top.shape[1], dtype=torch.float32, device=logits.device)
    torch.ops.b200.memory_gates(out, top, logits, bias, cap, *steps)
    return tuple(out)
