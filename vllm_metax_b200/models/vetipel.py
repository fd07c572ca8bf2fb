"""Vetipel: an attention-only decoder whose ``config.json`` lists the layers one by one and whose residual is several streams.

    x_s = scale * embed[token]                                   fp32 streams
    per sublayer   y = f(norm(sum_s in[s] x_s)),  x_t = sum_s mix[s, t] x_s + out[t] y
    logits = head . norm(sum_s x_s)

Norms divide by the root mean square; their weights are stored around zero.  Mixers: ``attention`` (sigmoid weights instead of a
softmax, a slope per head, a sliding window), ``attention_2`` (biased projections, unit head norms, a learned temperature and
logarithmic distance bias per head, chunks, sinks) - both layers/attention.py:QKNormAttention with one output gate per head - and
``latent_attention`` (layers/latent_attention.py, queries straight from the input, rotation in adjacent pairs).  Feed-forward:
dense with a squared relu, or none.

Between two products everything runs in one launch per boundary (layers/streams.py).  Single rank.
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
from ..layers.latent_attention import LatentAttention
from ..layers.recurrent import _param
from ..layers.streams import HyperConnection, StreamBoundary
from ..ops.stream_norm import Embedded
from ..parallel import state as ps


class SquaredReluMLP(nn.Module):
    """down(relu(up h)^2); the number of hidden rows padded to a multiple of 8."""

    def __init__(self, width: int, ff: int, dtype):
        super().__init__()
        self.ff, pad = ff, -(-ff // 8) * 8
        self.up, self.down = _param(pad, width, dtype=dtype), _param(width, pad, dtype=dtype)

    def slots(self) -> dict:
        return {"up": self.up.data[: self.ff], "down": self.down.data[:, : self.ff]}

    def forward(self, h):
        return ops.gemm(ops.gemm(h, self.up, act="relu2"), self.down)


def _sigmoid_attention(W, m, eps, cache_idx, dtype) -> QKNormAttention:
    H = int(m["heads"])
    return QKNormAttention(W, H, m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), eps, None, cache_idx, dtype=dtype,
                           window=int(m["mask"]["size"]), norm="none", sigmoid=True, gated="head",
                           alibi_slopes=[2.0 ** (-8.0 * (h + 1) / H) for h in range(H)])


def _chunked_attention(W, m, eps, cache_idx, dtype) -> QKNormAttention:
    return QKNormAttention(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), eps, None, cache_idx, dtype=dtype,
                           chunk=int(m["mask"]["size"]), norm="unit", proj_bias=True, head_temp=True, log_bias=True, sinks=True,
                           gated="head")


def _latent_attention(W, m, eps, cache_idx, dtype) -> LatentAttention:
    return LatentAttention(W, m["heads"], m["dim"], m["rot_dim"], m["vdim"], None, m["kv_rank"], float(m["scale"]), 0,
                           float(m["rot"]["base"]), m["rot"]["dims"], eps, cache_idx, dtype, interleaved=True)


MIXERS = {"attention": _sigmoid_attention, "attention_2": _chunked_attention, "latent_attention": _latent_attention}


class VetipelLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int):
        super().__init__()
        hf, dt = cfg.hf_config, cfg.dtype
        spec, W, S = hf["layers"][i], hf["width"], int(hf["streams"])
        f = spec.get("mlp")
        if spec["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer type {spec['type']!r}")
        self.norm1, self.hc1 = NormAroundOne(W, dt), HyperConnection(S, dt)
        self.mixer = MIXERS[spec["type"]](W, spec["mixer"], float(hf["norm"]["eps"]), i, dt)
        self.mlp = None
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            self.norm2, self.hc2 = NormAroundOne(W, dt), HyperConnection(S, dt)
            self.mlp = SquaredReluMLP(W, f["ff"], dt)

    def slots(self) -> dict:
        """Checkpoint name within the layer -> where it is copied."""
        parts = [("norm1", {"": self.norm1.weight.data}), ("hc1.", self.hc1.slots()), ("mix.", self.mixer.slots())]
        if self.mlp is not None:
            parts += [("norm2", {"": self.norm2.weight.data}), ("hc2.", self.hc2.slots()), ("mlp.", self.mlp.slots())]
        return {pre + k: v for pre, d in parts for k, v in d.items()}


class VetipelForCausalLM(nn.Module):
    native_units = "streams"

    def __init__(self, cfg: ModelConfig):
        super().__init__()
        if ps.tp_size() > 1 or ps.get_pp_group().world_size > 1 or ps.get_dcp_group().world_size > 1 \
                or ps.get_pcp_group().world_size > 1:
            raise ValueError("Vetipel runs on one rank")
        if cfg.quantization:
            raise ValueError("Vetipel checkpoints are served unquantised")
        self.cfg = cfg
        hf, W, dt = cfg.hf_config, cfg.hidden_size, cfg.dtype
        self.streams, self.embed_scale = int(hf["streams"]), float(hf["embedding"]["scale"])
        self.embed = VocabParallelEmbedding(cfg.vocab_size, W, dt)
        self.layers = nn.ModuleList(VetipelLayer(cfg, i) for i in range(len(hf["layers"])))
        self.final_norm = NormAroundOne(W, dt)
        self.lm_head = ParallelLMHead(cfg.vocab_size, W, dt)
        # the sublayers in the order they run, and what stands in front of each and behind the last
        self.sublayers, before, bounds = [], None, []
        for l in self.layers:
            for f, norm, hc in ((l.mixer, l.norm1, l.hc1), *(((l.mlp, l.norm2, l.hc2),) if l.mlp is not None else ())):
                bounds.append(StreamBoundary(self.streams, before, hc, norm, float(hf["norm"]["eps"])))
                self.sublayers.append((f, f is l.mixer))
                before = hc
        bounds.append(StreamBoundary(self.streams, before, None, self.final_norm, float(hf["norm"]["eps"])))
        self.bounds = nn.ModuleList(bounds)
        self._complete = False

    # ---- engine interface --------------------------------------------------------------------------------------
    def num_kv_layers(self) -> int:
        return len(self.layers)

    def kv_cache_spec(self) -> dict:
        return {"kind": "layers"}

    def kv_bytes_per_block(self, block_size: int, kv_cache_dtype: str) -> int:
        return (sum(l.mixer.cache_elems_per_token() for l in self.layers) * block_size
                * torch.empty((), dtype=self.cfg.dtype).element_size())

    def allocate_kv_cache(self, num_blocks: int, block_size: int, kv_cache_dtype: str, device) -> list:
        if kv_cache_dtype not in ("auto", "bfloat16", "float16"):
            raise ValueError(f"the cache is kept in the model's dtype, not {kv_cache_dtype}")
        return [l.mixer.allocate_kv_cache(num_blocks, block_size, device) for l in self.layers]

    def decode_workspace_floats(self, batch: int, max_seq_len: int) -> int:
        return max((l.mixer.decode_workspace_floats(batch, max_seq_len) for l in self.layers), default=0)

    def forward(self, input_ids, positions, intermediate=None):
        x, h = self.bounds[0](None, Embedded(self.embed.weight, input_ids, self.cfg.vocab_size, self.embed_scale, self.streams))
        for (f, mixes), bound in zip(self.sublayers, self.bounds[1:]):
            x, h = bound(f(positions, h) if mixes else f(h), x)
        return h

    def compute_logits(self, hidden):
        return ops.gemm(hidden, self.lm_head.weight, out_dtype=torch.float32)[:, : self.cfg.vocab_size]

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
