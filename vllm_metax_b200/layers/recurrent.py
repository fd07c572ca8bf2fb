"""Recurrent sequence mixers whose per-request state lives in the runner's state slots, and the post-norm boundary with a
short input convolution.  Sizes and constants are constructor arguments, so that a model class picks them from its config.

Every module with state implements ``allocate_state(slots, device)`` (returns the bytes taken); the step's slots come with
the forward context (``state_indices``, ``state_has_init``).
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _custom_ops as ops
from ..attention.metadata import get_forward_context
from ..ops.gdn import causal_conv1d
from ..ops.gla import gated_linear_attention
from ..ops.residual_conv import residual_conv
from ..ops.rglru import rglru


def _param(*shape, dtype) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=dtype), requires_grad=False)


class StackedLinear(nn.Module):
    """Several bias-free (or biased) projections of one input as a single product.  Every part starts at a multiple of 8
    rows (zero rows in between), so each part of the output is a 16-byte aligned operand for the next kernel."""

    def __init__(self, in_features: int, parts: dict[str, int], bias_parts: tuple = (), dtype=torch.bfloat16):
        super().__init__()
        self.offsets, self.sizes = {}, dict(parts)
        n = 0
        for name, rows in parts.items():
            self.offsets[name] = n
            n += -(-rows // 8) * 8
        self.weight = _param(n, in_features, dtype=dtype)
        self.bias = _param(n, dtype=dtype) if bias_parts else None

    def rows(self, name: str) -> torch.Tensor:
        """The weight rows of one part (a view, for loading)."""
        return self.weight.data[self.offsets[name]: self.offsets[name] + self.sizes[name]]

    def bias_rows(self, name: str) -> torch.Tensor:
        return self.bias.data[self.offsets[name]: self.offsets[name] + self.sizes[name]]

    def part(self, out: torch.Tensor, name: str) -> torch.Tensor:
        return out[:, self.offsets[name]: self.offsets[name] + self.sizes[name]]

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return ops.gemm(x, self.weight, self.bias)


class InputConv(nn.Module):
    """Residual add of the previous sublayer's (normed) output, then ``h + conv(h)`` as the next sublayer's input."""

    def __init__(self, width: int, taps: int, dtype=torch.bfloat16):
        super().__init__()
        self.width, self.taps = width, taps
        self.weight = _param(width, taps, dtype=dtype)
        self.carry: Optional[torch.Tensor] = None

    def allocate_state(self, slots: int, device) -> int:
        self.carry = torch.zeros(slots, self.taps - 1, self.width, dtype=torch.float32, device=device)
        return self.carry.numel() * 4

    def forward(self, y, x, gain, eps):
        md = get_forward_context().attn_metadata
        return residual_conv(y, x, gain, self.weight, eps, self.carry, md.query_start_loc, md.extra["state_indices"],
                             md.extra["state_has_init"])


class GatedLinearAttention(nn.Module):
    """Linear attention with a decay per key channel, alpha = sigmoid(W2 W1 h + b)^(1/tau), and a gated head norm."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay_rank: int, tau: float, eps: float,
                 dtype=torch.bfloat16):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps, self.dtype = heads, dim, vdim, eps, dtype
        self.register_buffer("inv_tau", torch.full((1,), 1.0 / tau, dtype=torch.float32), persistent=False)
        self.in_proj = StackedLinear(width, {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim,
                                             "a1": decay_rank}, dtype=dtype)
        self.decay_proj = _param(heads * dim, decay_rank, dtype=dtype)
        self.decay_bias = _param(heads * dim, dtype=dtype)
        self.head_norm = _param(vdim, dtype=dtype)
        self.out_proj = _param(width, heads * vdim, dtype=dtype)
        self.state: Optional[torch.Tensor] = None

    def allocate_state(self, slots: int, device) -> int:
        self.state = torch.zeros(slots, self.heads, self.dim, self.vdim, dtype=torch.float32, device=device)
        return self.state.numel() * 4

    def forward(self, positions, h):
        md = get_forward_context().attn_metadata
        p = self.in_proj(h)
        alpha = ops.gemm(self.in_proj.part(p, "a1"), self.decay_proj, self.decay_bias, act="decay", act_params=self.inv_tau,
                         out_dtype=torch.float32)
        off = [self.in_proj.offsets[n] for n in ("q", "k", "v", "g")]
        o = gated_linear_attention(p, off, alpha, self.head_norm, self.state, md.query_start_loc, md.extra["state_indices"],
                                   md.extra["state_has_init"], self.dim ** -0.5, self.eps, md.max_query_len)
        return ops.gemm(o, self.out_proj)


class RGLRUMixer(nn.Module):
    """Griffin's recurrent block: a gelu branch times a real-gated linear recurrence over a short convolution."""

    def __init__(self, in_width: int, width: int, blocks: int, taps: int, dtype=torch.bfloat16):
        super().__init__()
        assert width % blocks == 0, "the recurrence width splits into equal blocks"
        self.width, self.blocks, self.taps, self.dtype = width, blocks, taps, dtype
        bw = self.block_width = width // blocks
        self.in_proj = StackedLinear(in_width, {"y": width, "x": width}, ("y", "x"), dtype=dtype)
        self.conv_weight = _param(width, taps, dtype=dtype)
        self.conv_bias = _param(width, dtype=dtype)
        self.gate_weight = _param(blocks, 2 * bw, bw, dtype=dtype)     # per block: rows of the r gate, then of the i gate
        self.r_bias = _param(width, dtype=torch.float32)
        self.i_bias = _param(width, dtype=torch.float32)
        self.lam = _param(width, dtype=torch.float32)
        self.register_buffer("decay", torch.zeros(width, dtype=torch.float32), persistent=False)
        self.out_proj = _param(in_width, width, dtype=dtype)
        self.conv_state: Optional[torch.Tensor] = None
        self.state: Optional[torch.Tensor] = None

    def finalize_weights(self) -> None:
        self.decay.copy_(-8.0 * F.softplus(self.lam.data))

    def allocate_state(self, slots: int, device) -> int:
        self.conv_state = torch.zeros(slots, self.taps - 1, self.width, dtype=self.dtype, device=device)
        self.state = torch.zeros(slots, self.width, dtype=torch.float32, device=device)
        return self.conv_state.numel() * self.conv_state.element_size() + self.state.numel() * 4

    def forward(self, positions, h):
        md = get_forward_context().attn_metadata
        idx, init, qsl = md.extra["state_indices"], md.extra["state_has_init"], md.query_start_loc
        T = h.shape[0]
        p = self.in_proj(h)
        u = causal_conv1d(self.in_proj.part(p, "x"), self.conv_weight, self.conv_bias, self.conv_state, qsl, idx, init,
                          silu=False)
        gates = torch.empty(T, self.blocks, 2, self.block_width, dtype=torch.float32, device=h.device)
        ops.gemm_batched(u.view(T, self.blocks, self.block_width).transpose(0, 1), self.gate_weight,
                         out=gates.view(T, self.blocks, 2 * self.block_width).transpose(0, 1))
        o = rglru(u, self.in_proj.part(p, "y"), gates, self.r_bias, self.i_bias, self.decay, self.state, qsl, idx, init,
                  md.max_query_len)
        return ops.gemm(o, self.out_proj)
