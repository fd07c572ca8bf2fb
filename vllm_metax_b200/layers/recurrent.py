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
from ..ops.channel_delta import channel_delta_rule
from ..ops.gla import Normalizer, Steps, gated_linear_attention, linear_attention, memory_gates
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


def current_steps() -> Steps:
    md = get_forward_context().attn_metadata
    return Steps(md.query_start_loc, md.extra["state_indices"], md.extra["state_has_init"], md.max_query_len)


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


class _HeadsBranch(nn.Module):
    """What the linear-attention branches of a :class:`layers.mixer.ProjectedMixer` share: heads of ``dim`` (padded to a
    multiple of 8 where rows of ``vdim`` leave the branch), states per pass (``runs``) and slot."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, eps: float, runs: int, out_scale: float, dtype):
        super().__init__()
        self.width, self.heads, self.dim, self.vdim, self.eps = width, heads, dim, vdim, eps
        self.runs, self.out_scale, self.dtype = runs, out_scale, dtype
        self.out_width = -(-heads * vdim // 8) * 8
        self.state: Optional[torch.Tensor] = None

    def attach(self, proj: StackedLinear, prefix: str = "") -> None:
        self.prefix = prefix
        self.at = {n: proj.offsets[prefix + n] for n in self.in_parts()}

    def out_slot(self, weight: torch.Tensor):
        return weight[:, : self.heads * self.vdim]

    def allocate_state(self, slots: int, device) -> int:
        self.state = torch.zeros(self.runs, slots, self.heads, self.dim, self.vdim, dtype=torch.float32, device=device)
        return self.state.numel() * 4

    def _rows(self, proj: StackedLinear, *names) -> dict:
        return {n: proj.rows(self.prefix + n) for n in names}

    def _out(self, out: torch.Tensor) -> torch.Tensor:
        n = self.heads * self.vdim
        if n < self.out_width:
            out[:, n:].zero_()
        return out[:, :n]


class LightningAttention(_HeadsBranch):
    """Linear attention with a fixed decay per head, silu on q, k and v, one norm over all heads and a sigmoid gate."""

    def __init__(self, width, heads, dim, vdim, decay, eps, runs: int = 1, out_scale: float = 1.0, dtype=torch.bfloat16):
        super().__init__(width, heads, dim, vdim, eps, runs, out_scale, dtype)
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        self.register_buffer("decay", torch.tensor(decay, dtype=torch.float32), persistent=False)
        self.norm = _param(heads * vdim, dtype=dtype)

    def in_parts(self) -> dict:
        k, v = self.heads * self.dim, self.heads * self.vdim
        return {"q": k, "k": k, "v": v, "g": v}

    def in_slots(self, proj) -> dict:
        return {**self._rows(proj, "q", "k", "v", "g"), "norm": self.norm.data}

    def mix(self, positions, h, p, out, run: int = 0) -> None:
        linear_attention(p, [self.at[n] for n in ("q", "k", "v", "g")], self.decay, self.norm, self.state[run], current_steps(),
                         1.0, self.eps, gate="sigmoid", silu_qkv=True, whole_row=True, out_scale=self.out_scale,
                         out=self._out(out))


class MatrixMemory(_HeadsBranch):
    """The matrix memory of xLSTM (mLSTM): exponential gates under a running maximum, a normaliser, head norms, a sigmoid gate."""

    def __init__(self, width, heads, dim, vdim, gate_cap, eps, runs: int = 1, out_scale: float = 1.0, dtype=torch.bfloat16):
        super().__init__(width, heads, dim, vdim, eps, runs, out_scale, dtype)
        self.gate_cap = float(gate_cap)
        self.gates = _param(2 * heads, width, dtype=dtype)                  # rows of the input gates, then of the forget gates
        self.gate_bias = _param(2 * heads, dtype=torch.float32)
        self.norm = _param(heads * vdim, dtype=dtype)
        self.normalizer = self.top = None

    def in_parts(self) -> dict:
        k, v = self.heads * self.dim, self.heads * self.vdim
        return {"q": k, "k": k, "v": v, "g": v}

    def in_slots(self, proj) -> dict:
        H = self.heads
        return {**self._rows(proj, "q", "k", "v", "g"), "norm": self.norm.data, "i": self.gates.data[:H], "f": self.gates.data[H:],
                "i.b": self.gate_bias.data[:H], "f.b": self.gate_bias.data[H:]}

    def allocate_state(self, slots: int, device) -> int:
        n = super().allocate_state(slots, device)
        self.normalizer = torch.zeros(self.runs, slots, self.heads, -(-self.vdim // 16), self.dim, dtype=torch.float32,
                                      device=device)
        self.top = torch.zeros(self.runs, slots, self.heads, dtype=torch.float32, device=device)
        return n + 4 * (self.normalizer.numel() + self.top.numel())

    def mix(self, positions, h, p, out, run: int = 0) -> None:
        steps = current_steps()
        decay, k_mul, floor = memory_gates(ops.router_logits(h, self.gates), self.gate_bias, self.gate_cap, self.top[run], steps)
        linear_attention(p, [self.at[n] for n in ("q", "k", "v", "g")], decay, self.norm, self.state[run], steps,
                         self.dim ** -0.5, self.eps, gate="sigmoid", memory=Normalizer(self.normalizer[run], k_mul, floor),
                         out_scale=self.out_scale, out=self._out(out))


class ChannelDeltaRule(_HeadsBranch):
    """Gated delta rule with a decay per key channel from a low-rank projection, short convolutions in front of q, k and v,
    head norms and a low-rank sigmoid gate."""

    def __init__(self, width, heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank, eps, runs: int = 1,
                 out_scale: float = 1.0, dtype=torch.bfloat16):
        super().__init__(width, heads, dim, vdim, eps, runs, out_scale, dtype)
        if heads % kv_heads:
            raise ValueError(f"{heads} value heads over {kv_heads} key heads")
        self.kv_heads, self.taps, self.decay_rank, self.gate_rank = kv_heads, taps, decay_rank, gate_rank
        pad = lambda n: -(-n // 8) * 8
        self.channels = 2 * pad(kv_heads * dim) + pad(heads * vdim)         # q | k | v as they lie in the input product
        self.conv_weight = _param(self.channels, taps, dtype=dtype)
        self.beta = _param(heads, width, dtype=dtype)
        self.decay_proj = _param(heads * dim, pad(decay_rank), dtype=dtype)
        self.dt_bias = _param(heads * dim, dtype=dtype)
        self.A_log = _param(heads, dtype=torch.float32)
        self.register_buffer("rate", torch.zeros(heads * dim, dtype=torch.float32), persistent=False)
        self.gate_proj = _param(heads * vdim, pad(gate_rank), dtype=dtype)
        self.norm = _param(vdim, dtype=dtype)
        self.conv_state: Optional[torch.Tensor] = None

    def finalize_weights(self) -> None:
        self.rate.copy_(torch.exp(self.A_log.data).repeat_interleave(self.dim))

    def in_parts(self) -> dict:
        k = self.kv_heads * self.dim
        return {"q": k, "k": k, "v": self.heads * self.vdim, "a1": self.decay_rank, "g1": self.gate_rank}

    def in_slots(self, proj) -> dict:
        out = {**self._rows(proj, "q", "k", "v", "a1", "g1"), "b": self.beta.data, "A_log": self.A_log.data,
               "a2": self.decay_proj.data[:, : self.decay_rank], "dt_bias": self.dt_bias.data,
               "g2": self.gate_proj.data[:, : self.gate_rank], "norm": self.norm.data}
        for n in ("q", "k", "v"):
            lo = self.at[n] - self.at["q"]
            out[n + ".conv"] = self.conv_weight.data[lo: lo + self.in_parts()[n]]
        return out

    def allocate_state(self, slots: int, device) -> int:
        n = super().allocate_state(slots, device)
        self.conv_state = torch.zeros(self.runs, slots, self.taps - 1, self.channels, dtype=self.dtype, device=device)
        return n + self.conv_state.numel() * self.conv_state.element_size()

    def mix(self, positions, h, p, out, run: int = 0) -> None:
        steps, at = current_steps(), self.at
        u = causal_conv1d(p[:, at["q"]: at["q"] + self.channels], self.conv_weight, None, self.conv_state[run], *steps[:3])
        g = ops.gemm(p[:, at["a1"]: at["a1"] + self.decay_proj.shape[1]], self.decay_proj, self.dt_bias, act="softplus_decay",
                     act_params=self.rate, out_dtype=torch.float32)
        gate = ops.gemm(p[:, at["g1"]: at["g1"] + self.gate_proj.shape[1]], self.gate_proj)
        channel_delta_rule(u, [at[n] - at["q"] for n in ("q", "k", "v")], self.kv_heads, g, ops.router_logits(h, self.beta), gate,
                           self.norm, self.state[run], steps, self.eps, self.out_scale, self._out(out))
