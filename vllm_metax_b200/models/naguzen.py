"""Naguzen: a small hybrid decoder whose ``config.json`` lists the layers one by one.

    x = embed[token]                                              fp32 residual stream
    per layer   x += norm1(mixer(h)),  x += norm2(ff(h)),         h = x + conv(x), a short causal convolution per sublayer
    logits = head . norm(x)

Norms divide by the root mean square and multiply by ONE number; they sit on the sublayers' outputs.  Mixers:
``latent_attention`` (windowed, layers/latent_attention.py), ``gla`` and ``rglru`` (layers/recurrent.py).  Feed-forward:
dense with the xIELU activation, or routed gelu experts (sigmoid scores, top-k, not renormalised, times a constant) plus a
shared expert, or none.

Between two products everything runs in one launch per boundary (csrc/residual_conv.cu: norm of the finished sublayer's
output, residual add, convolution with its carry); activations run in the GEMM epilogues.  Only latent-attention layers own
paged cache; everything else is in the runner's state slots.  Single rank.
"""
from __future__ import annotations

from typing import Iterable

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import _custom_ops as ops
from ..config import ModelConfig
from ..engine.loader import copy_to_slots, safetensors_shapes
from ..layers.basic import ParallelLMHead, VocabParallelEmbedding
from ..layers.fused_moe import FusedMoE
from ..layers.latent_attention import LatentAttention
from ..layers.recurrent import GatedLinearAttention, InputConv, RGLRUMixer, _param
from ..ops.residual_norm import residual_norm
from ..parallel import state as ps


class ScalarRMSNorm(nn.Module):
    """The gain of ``x / sqrt(mean(x^2) + eps) * g`` with one number for all coordinates; the arithmetic is fused into the
    boundary kernels."""

    def __init__(self, dtype):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(1, dtype=dtype), requires_grad=False)


class XieluMLP(nn.Module):
    def __init__(self, width: int, ff: int, dtype):
        super().__init__()
        self.up, self.down = _param(ff, width, dtype=dtype), _param(width, ff, dtype=dtype)
        self.act = _param(2, dtype=torch.float32)                      # p, q of the checkpoint
        self.register_buffer("coef", torch.zeros(2, dtype=torch.float32), persistent=False)

    def finalize_weights(self) -> None:
        self.coef.copy_(F.softplus(self.act.data) + torch.tensor([0.0, 0.5], device=self.act.device))

    def slots(self) -> dict:
        return {"up": self.up.data, "down": self.down.data, "act": self.act.data}

    def forward(self, h):
        return ops.gemm(ops.gemm(h, self.up, act="xielu", act_params=self.coef), self.down)


class GeluMLP(nn.Module):
    def __init__(self, width: int, ff: int, dtype):
        super().__init__()
        self.up, self.down = _param(ff, width, dtype=dtype), _param(width, ff, dtype=dtype)

    def forward(self, h):
        return ops.gemm(ops.gemm(h, self.up, act="gelu"), self.down)


class RoutedExperts(nn.Module):
    def __init__(self, width: int, spec: dict, dtype, prefix: str):
        super().__init__()
        r = spec["router"]
        self.gate = _param(r["experts"], width, dtype=dtype)
        self.experts = FusedMoE(r["experts"], r["top"], width, spec["expert"]["ff"], dtype, renormalize=False,
                                scoring_func="sigmoid", routed_scaling_factor=float(r["scale"]), gated=False,
                                activation="gelu", prefix=f"{prefix}.experts")
        self.shared = GeluMLP(width, spec["shared"]["ff"], dtype) if spec.get("shared") else None

    def slots(self) -> dict:
        e = self.experts
        out = {"router": self.gate.data}
        for i in range(e.num_experts):
            out[f"e{i}.up"], out[f"e{i}.down"] = e.w13_weight.data[i], e.w2_weight.data[i]
        if self.shared is not None:
            out["shared.up"], out["shared.down"] = self.shared.up.data, self.shared.down.data
        return out

    def forward(self, h):
        shared = self.shared(h) if self.shared is not None else None
        return self.experts(h, ops.router_logits(h, self.gate), shared)


class NaguzenLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, cache_idx: int, decay_rank: int):
        super().__init__()
        hf, dt = cfg.hf_config, cfg.dtype
        spec, W, eps = hf["layers"][i], hf["width"], float(hf["norm"]["eps"])
        self.kind, m, f = spec["type"], spec["mixer"], spec["mlp"]
        taps = int(hf["canon"]["taps"])
        self.conv1, self.out1_norm = InputConv(W, taps, dt), ScalarRMSNorm(dt)
        if self.kind == "latent_attention":
            window = int((m.get("mask") or {}).get("size") or 0)
            self.mixer = LatentAttention(W, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"],
                                         float(m["scale"]), window, float(m["rot"]["base"]), m["rot"]["dims"], eps,
                                         cache_idx, dt)
        elif self.kind == "gla":
            self.mixer = GatedLinearAttention(W, m["heads"], m["dim"], m["vdim"], decay_rank, float(m["tau"]), eps, dt)
        elif self.kind == "rglru":
            self.mixer = RGLRUMixer(W, m["width"], m["blocks"], m["conv"], dt)
        else:
            raise ValueError(f"layer {i}: unknown mixer type {self.kind!r}")
        self.mlp = None
        if f is not None:
            self.conv2, self.out2_norm = InputConv(W, taps, dt), ScalarRMSNorm(dt)
            if f["kind"] == "dense":
                self.mlp = XieluMLP(W, f["ff"], dt)
            elif f["kind"] == "moe":
                self.mlp = RoutedExperts(W, f, dt, f"l{i}.mlp")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")

    def slots(self) -> dict:
        """Checkpoint name within the layer -> the memory it is copied to."""
        out = {"norm1": self.out1_norm.weight.data, "canon1": self.conv1.weight.data}
        m = self.mixer
        if self.kind == "latent_attention":
            out.update({f"mix.{k}": v for k, v in m.slots().items()})
        elif self.kind == "gla":
            out.update({f"mix.{n}": m.in_proj.rows(n) for n in ("q", "k", "v", "g", "a1")})
            out.update({"mix.a2": m.decay_proj.data, "mix.a2.b": m.decay_bias.data, "mix.norm": m.head_norm.data,
                        "mix.o": m.out_proj.data})
        else:
            bw = m.block_width
            out.update({"mix.y": m.in_proj.rows("y"), "mix.y.b": m.in_proj.bias_rows("y"), "mix.x": m.in_proj.rows("x"),
                        "mix.x.b": m.in_proj.bias_rows("x"), "mix.conv": m.conv_weight.data,
                        "mix.conv.b": m.conv_bias.data, "mix.ra": m.gate_weight.data[:, :bw],
                        "mix.ri": m.gate_weight.data[:, bw:], "mix.ra.b": m.r_bias.data, "mix.ri.b": m.i_bias.data,
                        "mix.lam": m.lam.data, "mix.o": m.out_proj.data})
        if self.mlp is not None:
            out.update({"norm2": self.out2_norm.weight.data, "canon2": self.conv2.weight.data})
            out.update({f"mlp.{k}": v for k, v in self.mlp.slots().items()})
        return out


class NaguzenForCausalLM(nn.Module):
    supports_prefix_caching = False        # a cached prefix has latent rows but no recurrent state to resume from
    native_units = "hybrid"

    def __init__(self, cfg: ModelConfig):
        super().__init__()
        if ps.tp_size() > 1 or ps.get_pp_group().world_size > 1 or ps.get_dcp_group().world_size > 1 \
                or ps.get_pcp_group().world_size > 1:
            raise ValueError("Naguzen runs on one rank")
        if cfg.quantization:
            raise ValueError("Naguzen checkpoints are served unquantised")
        self.cfg = cfg
        hf = cfg.hf_config
        self.eps = float(hf["norm"]["eps"])
        ranks = decay_ranks(cfg)
        self.embed = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, cfg.dtype)
        self.layers = nn.ModuleList()
        n_cache = 0
        for i, spec in enumerate(hf["layers"]):
            self.layers.append(NaguzenLayer(cfg, i, n_cache, ranks.get(i, 16)))
            n_cache += spec["type"] == "latent_attention"
        self.final_norm = ScalarRMSNorm(cfg.dtype)
        self.lm_head = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, cfg.dtype)
        self._complete = False

    # ---- engine interface --------------------------------------------------------------------------------------
    def _latent(self) -> list:
        return [l.mixer for l in self.layers if l.kind == "latent_attention"]

    def num_kv_layers(self) -> int:
        return len(self._latent())

    def kv_cache_spec(self) -> dict:
        return {"kind": "latent"}

    def kv_bytes_per_block(self, block_size: int, kv_cache_dtype: str) -> int:
        return sum(m.cache_elems_per_token() for m in self._latent()) * block_size * torch.empty((), dtype=self.cfg.dtype).element_size()

    def allocate_kv_cache(self, num_blocks: int, block_size: int, kv_cache_dtype: str, device) -> list:
        if kv_cache_dtype not in ("auto", "bfloat16", "float16"):
            raise ValueError(f"the latent cache is kept in the model's dtype, not {kv_cache_dtype}")
        return [m.allocate_kv_cache(num_blocks, block_size, device) for m in self._latent()]

    def allocate_state(self, slots: int, device) -> int:
        return sum(m.allocate_state(slots, device) for m in self.modules() if m is not self and hasattr(m, "allocate_state"))

    def forward(self, input_ids, positions, intermediate=None):
        y, x, gain = self.embed(input_ids), None, None
        for l in self.layers:
            x, h = l.conv1(y, x, gain, self.eps)
            y, gain = l.mixer(positions, h), l.out1_norm.weight
            if l.mlp is not None:
                x, h = l.conv2(y, x, gain, self.eps)
                y, gain = l.mlp(h), l.out2_norm.weight
        return residual_norm(y, x, gain, self.final_norm.weight, self.eps)

    def compute_logits(self, hidden):
        return self.lm_head.logits(hidden)

    # ---- weights -----------------------------------------------------------------------------------------------
    def finalize_weights(self) -> None:
        for m in self.modules():
            if m is not self and hasattr(m, "finalize_weights"):
                m.finalize_weights()

    def slots(self) -> dict:
        V = self.cfg.vocab_size
        out = {"embed": self.embed.weight.data[:V], "head": self.lm_head.weight.data[:V],
               "final.norm": self.final_norm.weight.data}
        for i, l in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in l.slots().items()})
        return out

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        loaded = copy_to_slots(self.slots(), weights, complete=not self._complete)
        self._complete = True                  # later calls may bring a subset (weight updates)
        self.finalize_weights()
        return loaded


def decay_ranks(cfg: ModelConfig) -> dict[int, int]:
    """Low rank of every gla layer's decay projection.  The config does not carry it: it is the first dimension of the
    layer's ``mix.a1``, read from the checkpoint's headers (16 without a checkpoint)."""
    gla = [i for i, l in enumerate(cfg.hf_config["layers"]) if l["type"] == "gla"]
    if not gla or not cfg.model_path:
        return {}
    shapes = safetensors_shapes(cfg.model_path)
    return {i: shapes[f"l{i}.mix.a1"][0] for i in gla}
