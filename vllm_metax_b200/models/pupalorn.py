"""Pupalorn: a decoder whose ``config.json`` lists the layers one by one.

    x = scale * embed[token]                                     fp32 residual stream
    per layer   x += m * ls1 * norm1b(attention(norm1(x))),  x += m * ls2 * norm2b(experts(norm2(x)))
    logits = head . norm(x)

Norms divide by the root mean square; their weights are stored around zero.  Attention (layers/attention.py:QKNormAttention)
norms and partially rotates queries and keys and looks back over a sliding window; a layer with ``kv_from`` reads the keys and
values that layer cached and has no cache of its own.  Feed-forward: routed experts with a squared-relu (softmax scores, a
correction that moves the choice only, weights not renormalised), the last router outputs being identity experts.

Between two products everything runs in one launch per boundary (csrc/residual_norm.cu), which also forms the experts' weighted
sums: a layer's output norm, its layer scale and the residual multiplier are one fp32 gain.  Single rank.
"""
from __future__ import annotations

from typing import Iterable

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from ..config import ModelConfig
from ..engine.loader import copy_to_slots
from ..layers.attention import QKNormAttention
from ..layers.basic import NormAroundOne, ParallelLMHead, VocabParallelEmbedding
from ..layers.fused_moe import FusedMoE
from ..layers.recurrent import _param
from ..ops.reference import rope_frequencies
from ..ops.residual_norm import boundary_norm, embed_norm
from ..parallel import state as ps


class IdentityRoutedExperts(nn.Module):
    def __init__(self, width: int, spec: dict, dtype, prefix: str):
        super().__init__()
        r = spec["router"]
        identity = int(r.get("identity") or 0)
        self.gate = _param(r["experts"] + identity, width, dtype=dtype)
        self.experts = FusedMoE(r["experts"], r["top"], width, spec["expert"]["ff"], dtype, renormalize=False,
                                scoring_func="softmax", e_score_correction_bias=True, gated=False, activation="relu2",
                                num_identity=identity, prefix=f"{prefix}.experts")

    def slots(self) -> dict:
        e = self.experts
        out = {"router": self.gate.data, "correction": e.e_score_correction_bias.data}
        for i in range(e.num_experts):
            out[f"e{i}.up"], out[f"e{i}.down"] = e.w13_weight.data[i], e.w2_weight.data[i]
        return out

    def forward(self, h):
        return self.experts.forward_rows(h, ops.router_logits(h, self.gate))


def _rotation(rot: dict) -> torch.Tensor:
    s = rot.get("scaling")
    scaling = None if s is None else {
        "type": "llama3", "factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
        "original_max_position_embeddings": s["original"]}
    return rope_frequencies(int(rot["dims"]), float(rot["base"]), scaling)[0]


class PupalornLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, cache_idx: int, kv_from):
        super().__init__()
        hf, dt = cfg.hf_config, cfg.dtype
        spec, W, factor = hf["layers"][i], hf["width"], float(hf["residual_mult"])
        m, f = spec["mixer"], spec.get("mlp")
        if spec["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {spec['type']!r}")
        self.in1, self.out1 = NormAroundOne(W, dt), NormAroundOne(W, dt, factor, scaled=True)
        self.mixer = QKNormAttention(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                                     float(hf["norm"]["eps"]), _rotation(m["rot"]), cache_idx,
                                     window=int((m.get("mask") or {}).get("size") or 0) or None, kv_from=kv_from, dtype=dt)
        self.mlp = None
        if f is not None:
            if f["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            self.in2, self.out2 = NormAroundOne(W, dt), NormAroundOne(W, dt, factor, scaled=True)
            self.mlp = IdentityRoutedExperts(W, f, dt, f"l{i}.mlp")

    def slots(self) -> dict:
        """Checkpoint name within the layer -> where it is copied."""
        out = {"norm1": self.in1.weight.data, "norm1b": self.out1.weight.data, "ls1": self.out1.scale.data}
        out.update({f"mix.{k}": v for k, v in self.mixer.slots().items()})
        if self.mlp is not None:
            out.update({"norm2": self.in2.weight.data, "norm2b": self.out2.weight.data, "ls2": self.out2.scale.data})
            out.update({f"mlp.{k}": v for k, v in self.mlp.slots().items()})
        return out


class PupalornForCausalLM(nn.Module):
    native_units = "gqa"

    def __init__(self, cfg: ModelConfig):
        super().__init__()
        if ps.tp_size() > 1 or ps.get_pp_group().world_size > 1 or ps.get_dcp_group().world_size > 1 \
                or ps.get_pcp_group().world_size > 1:
            raise ValueError("Pupalorn runs on one rank")
        if cfg.quantization:
            raise ValueError("Pupalorn checkpoints are served unquantised")
        self.cfg = cfg
        hf = cfg.hf_config
        self.eps, self.embed_scale = float(hf["norm"]["eps"]), float(hf["embedding"]["scale"])
        self.embed = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, cfg.dtype)
        self.layers = nn.ModuleList()
        n_cache = 0
        for i, spec in enumerate(hf["layers"]):
            src = spec["mixer"].get("kv_from")
            if src is not None and not (0 <= src < i and self.layers[src].mixer.own_kv):
                raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with keys and values of its own")
            kv_from = None if src is None else self.layers[src].mixer
            self.layers.append(PupalornLayer(cfg, i, n_cache if src is None else kv_from.attn.layer_idx, kv_from))
            n_cache += src is None
        self.final_norm = NormAroundOne(cfg.hidden_size, cfg.dtype)
        self.lm_head = ParallelLMHead(cfg.vocab_size, cfg.hidden_size, cfg.dtype)
        self._complete = False

    # ---- engine interface --------------------------------------------------------------------------------------
    def _own(self) -> list:
        return [l.mixer for l in self.layers if l.mixer.own_kv]

    def num_kv_layers(self) -> int:
        return len(self._own())

    def kv_cache_spec(self) -> dict:
        return {"kind": "layers"}

    def kv_bytes_per_block(self, block_size: int, kv_cache_dtype: str) -> int:
        return (sum(m.cache_elems_per_token() for m in self._own()) * block_size
                * torch.empty((), dtype=self.cfg.dtype).element_size())

    def allocate_kv_cache(self, num_blocks: int, block_size: int, kv_cache_dtype: str, device) -> list:
        if kv_cache_dtype not in ("auto", "bfloat16", "float16"):
            raise ValueError(f"the cache is kept in the model's dtype, not {kv_cache_dtype}")
        return [m.allocate_kv_cache(num_blocks, block_size, device) for m in self._own()]

    def decode_workspace_floats(self, batch: int, max_seq_len: int) -> int:
        return max((l.mixer.decode_workspace_floats(batch, max_seq_len) for l in self.layers), default=0)

    def forward(self, input_ids, positions, intermediate=None):
        first = self.layers[0].in1 if len(self.layers) else self.final_norm
        x, h = embed_norm(self.embed.weight, input_ids, self.cfg.vocab_size, self.embed_scale, first.gain, self.eps)
        for i, l in enumerate(self.layers):
            after = self.layers[i + 1].in1 if i + 1 < len(self.layers) else self.final_norm
            y, out = l.mixer(positions, h), l.out1
            if l.mlp is not None:
                x, h = boundary_norm(y, x, out.gain, l.in2.gain, self.eps)
                y, out = l.mlp(h), l.out2
            x, h = boundary_norm(y, x, out.gain, after.gain, self.eps, want_x=i + 1 < len(self.layers))
        return h

    def compute_logits(self, hidden):
        return self.lm_head.logits(hidden)

    # ---- weights -----------------------------------------------------------------------------------------------
    def finalize_weights(self) -> None:
        for m in self.modules():
            if isinstance(m, NormAroundOne):
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
