"""Luluzen: a decoder whose ``config.json`` lists the layers one by one, with two mixers side by side in a layer and a run of
layers that is passed through several times.

    x = embed[token]                                              fp32 residual stream
    per layer   x += mixer(norm1(x)),  x += ff(norm2(x))          layer norms without a bias
    per pass    x = W_in [x; embedding] + step[pass]              in front of the loop's first layer
    logits = cap tanh(embed . norm(x) / cap)

Mixers: ``lightning`` (layers/recurrent.py:LightningAttention); ``parallel`` (attention with head norms, a query temperature and
a learned distance bias, beside a gated delta rule with a decay per key channel); ``parallel_2`` (windowed, capped attention with
whole-row norms, interleaved rotation, sinks and an output gate, beside the matrix memory of xLSTM).  Both sides of a layer share
one input and one output product (layers/mixer.py).  Feed-forward: dense with a tanh-gelu gate, or routed experts with a clamped
SwiGLU whose routing weights (sigmoid scores, as they are) multiply the expert's input.

Every pass through the loop has caches and states of its own.  Between two products everything runs in one launch per boundary
(csrc/prenorm.cu), which also forms the experts' sums and the loop's operand.  Single rank.
"""
from __future__ import annotations

from typing import Iterable

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from ..config import ModelConfig
from ..engine.loader import copy_to_slots, safetensors_shapes
from ..layers.attention import QKNormAttention
from ..layers.basic import VocabParallelEmbedding
from ..layers.fused_moe import FusedMoE
from ..layers.mixer import ProjectedMixer
from ..layers.recurrent import ChannelDeltaRule, LightningAttention, MatrixMemory, _param
from ..ops.prenorm import loop_operand, prenorm
from ..ops.reference import rope_frequencies
from ..parallel import state as ps

SWIGLU_SLOPE = 1.702


class GatedMLP(nn.Module):
    """down(gelu_tanh(gate h) * (up h)); gate and up rows interleaved, their number padded to a multiple of 8."""

    def __init__(self, width: int, ff: int, dtype):
        super().__init__()
        self.ff, pad = ff, -(-ff // 8) * 8
        self.gate_up, self.down = _param(2 * pad, width, dtype=dtype), _param(width, pad, dtype=dtype)

    def slots(self) -> dict:
        return {"gate": self.gate_up.data[0: 2 * self.ff: 2], "up": self.gate_up.data[1: 2 * self.ff: 2],
                "down": self.down.data[:, : self.ff]}

    def forward(self, h):
        return ops.gemm(ops.gemm(h, self.gate_up, act="gelu_tanh_gate"), self.down)


class ClampedExperts(nn.Module):
    def __init__(self, width: int, spec: dict, dtype, prefix: str):
        super().__init__()
        r, self.ff = spec["router"], spec["expert"]["ff"]
        self.gate = _param(r["experts"], width, dtype=dtype)
        self.experts = FusedMoE(r["experts"], r["top"], width, -(-self.ff // 8) * 8, dtype, renormalize=False,
                                scoring_func="sigmoid", activation="clamped_swiglu",
                                activation_params=(float(spec["expert"]["limit"]), SWIGLU_SLOPE), weight_input=True,
                                prefix=f"{prefix}.experts")
        self.experts.w13_weight.data.zero_()               # the padding of odd sizes
        self.experts.w2_weight.data.zero_()

    def slots(self) -> dict:
        e, n = self.experts, self.ff
        out = {"router": self.gate.data}
        for i in range(e.num_experts):
            w13 = e.w13_weight.data[i]
            out.update({f"e{i}.gate": w13[0: 2 * n: 2], f"e{i}.up": w13[1: 2 * n: 2], f"e{i}.down": e.w2_weight.data[i, :, :n]})
        return out

    def forward(self, h):
        return self.experts.forward_rows(h, ops.router_logits(h, self.gate))


def _biased_attention(W, m, eps, cache_idx, dtype, **kw) -> QKNormAttention:
    return QKNormAttention(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), eps, None, cache_idx, dtype=dtype,
                           standalone=False, q_temp=(float(m["q_temp"]["coef"]), int(m["q_temp"]["every"])),
                           bias_far=int(m["bias_max"]), proj_bias=True, **kw)


def _window_attention(W, m, eps, cache_idx, dtype, **kw) -> QKNormAttention:
    return QKNormAttention(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), eps,
                           rope_frequencies(int(m["rot"]["dims"]), float(m["rot"]["base"]))[0], cache_idx,
                           window=int(m["mask"]["size"]), dtype=dtype, standalone=False, whole_row_norm=True, interleaved=True,
                           softcap=float(m["softcap"]), sinks=True, gated=True, **kw)


class LuluzenLayer(nn.Module):
    def __init__(self, cfg: ModelConfig, i: int, cache_idx: int, runs: int, shapes: dict):
        super().__init__()
        hf, dt = cfg.hf_config, cfg.dtype
        spec, W, eps = hf["layers"][i], hf["width"], float(hf["norm"]["eps"])
        kind, m, f = spec["type"], spec["mixer"], spec.get("mlp")
        self.runs, self.cache_idx = runs, cache_idx
        self.norm1 = _param(W, dtype=dt)
        if kind == "lightning":
            branches = {"": LightningAttention(W, m["heads"], m["dim"], m["vdim"], m["decay"], eps, runs, dtype=dt)}
        elif kind == "parallel":
            rows = lambda name, default: shapes.get(f"l{i}.mix.{name}", (default,))[0]
            a, r = m["left"], m["right"]
            rank = max(16, r["dim"])                       # of the low-rank projections, where no checkpoint tells
            branches = {
                "left": _biased_attention(W, a, eps, cache_idx, dt, runs=runs, out_scale=float(m["left_scale"]),
                                          bias_rows=rows("left.rel", 32)),
                "right": ChannelDeltaRule(W, r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"], rows("right.a1", rank),
                                          rows("right.g1", rank), eps, runs, float(m["right_scale"]), dt)}
        elif kind == "parallel_2":
            r = m["right"]
            branches = {
                "left": _window_attention(W, m["left"], eps, cache_idx, dt, runs=runs, out_scale=float(m["left_scale"])),
                "right": MatrixMemory(W, r["heads"], r["dim"], r["vdim"], r["gate_cap"], eps, runs, float(m["right_scale"]), dt)}
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        self.mixer = ProjectedMixer(W, branches, dt)
        self.norm2 = self.mlp = None
        if f is not None:
            self.norm2 = _param(W, dtype=dt)
            if f["kind"] == "dense":
                self.mlp = GatedMLP(W, f["ff"], dt)
            elif f["kind"] == "moe":
                self.mlp = ClampedExperts(W, f, dt, f"l{i}.mlp")
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")

    def attention(self) -> list:
        return [b for b in self.mixer.branches if isinstance(b, QKNormAttention)]

    def slots(self) -> dict:
        """Checkpoint name within the layer -> where it is copied."""
        out = {"norm1": self.norm1.data, **{f"mix.{k}": v for k, v in self.mixer.slots().items()}}
        if self.mlp is not None:
            out.update({"norm2": self.norm2.data, **{f"mlp.{k}": v for k, v in self.mlp.slots().items()}})
        return out


class LoopEntry(nn.Module):
    """What stands in front of every pass: the product W_in [x; embedding] and the pass's own vector.  16-bit operands hold x
    in two parts (``ops/prenorm.py:loop_operand``), so the columns for x are there twice."""

    def __init__(self, width: int, times: int, dtype):
        super().__init__()
        self.width, self.parts = width, 2 if dtype == torch.float32 else 3
        self.weight = _param(width, self.parts * width, dtype=dtype)
        self.step = _param(times, width, dtype=dtype)

    def finalize_weights(self) -> None:
        if self.parts == 3:
            w = self.weight.data.view(self.width, 3, self.width)
            w[:, 1] = w[:, 0]

    def slots(self) -> dict:
        w = self.weight.data.view(self.width, self.parts, self.width)
        return {"in": (w[:, :: self.parts - 1], (self.width, 2 * self.width)), "step": self.step.data}

    def forward(self, operand):
        return ops.gemm(operand, self.weight, out_dtype=torch.float32)


class LuluzenForCausalLM(nn.Module):
    supports_prefix_caching = False        # a cached prefix has keys and values but no recurrent state to resume from
    native_units = "parallel"

    def __init__(self, cfg: ModelConfig):
        super().__init__()
        if ps.tp_size() > 1 or ps.get_pp_group().world_size > 1 or ps.get_dcp_group().world_size > 1 \
                or ps.get_pcp_group().world_size > 1:
            raise ValueError("Luluzen runs on one rank")
        if cfg.quantization:
            raise ValueError("Luluzen checkpoints are served unquantised")
        self.cfg = cfg
        hf, n = cfg.hf_config, len(cfg.hf_config["layers"])
        self.eps = float(hf["norm"]["eps"])
        loop = hf.get("loop") or {"start": n, "stop": n, "times": 0}
        lo, hi, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
        if not (0 <= lo <= hi <= n) or times < 0 or (lo < hi and times < 1):
            raise ValueError(f"loop {loop} over {n} layers")
        if lo == hi:
            times = 0
        shapes = safetensors_shapes(cfg.model_path) if cfg.model_path else {}
        self.embed = VocabParallelEmbedding(cfg.vocab_size, cfg.hidden_size, cfg.dtype)
        self.layers = nn.ModuleList()
        n_cache = 0
        for i in range(n):
            layer = LuluzenLayer(cfg, i, n_cache, times if lo <= i < hi else 1, shapes)
            self.layers.append(layer)
            n_cache += layer.runs * len(layer.attention())
        self.entry = LoopEntry(cfg.hidden_size, times, cfg.dtype) if times else None
        # the layers in the order they run: (layer, pass, whether it opens a pass)
        self.order = ([(i, 0, False) for i in range(lo)] + [(i, t, i == lo) for t in range(times) for i in range(lo, hi)]
                      + [(i, 0, False) for i in range(hi, n)])
        self.final_norm = _param(cfg.hidden_size, dtype=cfg.dtype)
        self.register_buffer("logit_cap", torch.tensor([float(hf["logit_softcap"])], dtype=torch.float32), persistent=False)
        self._complete = False

    # ---- engine interface --------------------------------------------------------------------------------------
    def _attention(self) -> list:
        return [a for l in self.layers for a in l.attention()]

    def num_kv_layers(self) -> int:
        return sum(a.runs for a in self._attention())

    def kv_cache_spec(self) -> dict:
        return {"kind": "layers"}

    def kv_bytes_per_block(self, block_size: int, kv_cache_dtype: str) -> int:
        return (sum(a.cache_elems_per_token() for a in self._attention()) * block_size
                * torch.empty((), dtype=self.cfg.dtype).element_size())

    def allocate_kv_cache(self, num_blocks: int, block_size: int, kv_cache_dtype: str, device) -> list:
        if kv_cache_dtype not in ("auto", "bfloat16", "float16"):
            raise ValueError(f"the cache is kept in the model's dtype, not {kv_cache_dtype}")
        return [a.allocate_kv_cache(num_blocks, block_size, device) for a in self._attention() for _ in range(a.runs)]

    def decode_workspace_floats(self, batch: int, max_seq_len: int) -> int:
        return max((a.decode_workspace_floats(batch, max_seq_len) for a in self._attention()), default=0)

    def allocate_state(self, slots: int, device) -> int:
        return sum(m.allocate_state(slots, device) for m in self.modules() if m is not self and hasattr(m, "allocate_state"))

    def forward(self, input_ids, positions, intermediate=None):
        table, vocab, eps = self.embed.weight, self.cfg.vocab_size, self.eps
        y, x, ids = table, None, input_ids                       # the stream is x + y (y: rows of the table at first)
        for i, run, opens in self.order:
            l, add = self.layers[i], None
            if opens:
                y = self.entry(loop_operand(y, x, table, input_ids, vocab, gather=ids is not None))
                x, ids, add = None, None, self.entry.step[run]
            x, h = prenorm(y, x, l.norm1, eps, add, ids, vocab)
            y, ids = l.mixer(positions, h, run), None
            if l.mlp is not None:
                x, h = prenorm(y, x, l.norm2, eps)
                y = l.mlp(h)
        return prenorm(y, x, self.final_norm, eps, None, ids, vocab, want_x=False)[1]

    def compute_logits(self, hidden):
        return ops.gemm(hidden, self.embed.weight, act="softcap", act_params=self.logit_cap,
                        out_dtype=torch.float32)[:, : self.cfg.vocab_size]

    # ---- weights -----------------------------------------------------------------------------------------------
    def finalize_weights(self) -> None:
        for m in self.modules():
            if m is not self and hasattr(m, "finalize_weights"):
                m.finalize_weights()

    def slots(self) -> dict:
        out = {"embed": self.embed.weight.data[: self.cfg.vocab_size], "final.norm": self.final_norm.data}
        if self.entry is not None:
            out.update({f"loop.{k}": v for k, v in self.entry.slots().items()})
        for i, l in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in l.slots().items()})
        return out

    def load_weights(self, weights: Iterable[tuple[str, torch.Tensor]]) -> set[str]:
        loaded = copy_to_slots(self.slots(), weights, complete=not self._complete)
        self._complete = True                  # later calls may bring a subset (weight updates)
        self.finalize_weights()
        return loaded
