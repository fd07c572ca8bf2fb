"""Prefill and decode throughput of the layer-list hybrid (Naguzen) beside the existing model closest to it, at sizes that
resemble a real model's layers (random weights), and the time of each of its kernels against its roofline
(``bench.py --hybrid``).

Model rows: device-resident workload (``engine/static_workload.py``), CUDA events, decode as graph replays; weights and
caches are larger than L2.  Kernel rows: CUDA events around single launches with L2 overwritten in between; the like kernel
of the closest model is timed the same way at the same sizes.
"""
from __future__ import annotations

import json
import statistics
from typing import Callable

import torch

from .. import _custom_ops as ops
from ..config import ModelConfig

TITLE = "hybrid decoder beside its closest models"
SIZES = {
    # width, heads, experts, top, expert ff (not gated), shared ff, dense ff
    "w2048": dict(width=2048, heads=16, experts=64, top=8, ff=768, shared=768, dense=8192),
    "w4096": dict(width=4096, heads=32, experts=32, top=4, ff=1536, shared=1536, dense=16384),
}


def _gated(ff: int) -> int:
    """Width of a gated feed-forward with the parameters of a plain one."""
    return ff * 2 // 3 // 64 * 64


def naguzen_config(s: dict, repeats: int = 2) -> ModelConfig:
    """``repeats`` x (gla, rglru, windowed latent attention, latent attention with experts)."""
    W, H = s["width"], s["heads"]
    moe = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"], "scale": 1.5}, "expert": {"ff": s["ff"]},
           "shared": {"ff": s["shared"]}}
    dense = {"kind": "dense", "ff": s["dense"]}
    lat = {"heads": H, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 1536, "kv_rank": 512, "mask": {"size": 2048},
           "rot": {"base": 500000.0, "dims": 64}, "scale": 192 ** -0.5}
    layers = [{"type": "gla", "mixer": {"heads": H, "dim": 128, "vdim": 128, "tau": 16.0}, "mlp": moe},
              {"type": "rglru", "mixer": {"width": W, "blocks": 16, "conv": 4}, "mlp": moe},
              {"type": "latent_attention", "mixer": lat, "mlp": dense},
              {"type": "latent_attention", "mixer": lat, "mlp": moe}] * repeats
    return ModelConfig.from_layer_list({"architecture": "Naguzen", "vocab": 32768, "width": W, "canon": {"taps": 4},
                                        "norm": {"eps": 1e-6}, "layers": layers})


def qwen3_next_config(s: dict, layers: int = 8) -> ModelConfig:
    """Gated-delta-rule hybrid of the same width, depth, state size and expert parameters (gated experts of 2/3 the width)."""
    W, H = s["width"], s["heads"]
    return ModelConfig.from_hf_dict(dict(
        architectures=["Qwen3NextForCausalLM"], vocab_size=32768, hidden_size=W, intermediate_size=_gated(s["dense"]),
        num_hidden_layers=layers, num_attention_heads=H, num_key_value_heads=max(2, H // 8), head_dim=128, rms_norm_eps=1e-6,
        rope_theta=500000.0, max_position_embeddings=16384, linear_num_value_heads=H, linear_num_key_heads=H,
        linear_key_head_dim=128, linear_value_head_dim=128, linear_conv_kernel_dim=4, full_attention_interval=4,
        num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=_gated(s["ff"]),
        shared_expert_intermediate_size=_gated(s["shared"]), norm_topk_prob=True))


def deepseek_config(s: dict, layers: int = 8) -> ModelConfig:
    """Latent attention in every layer, same sizes, without the window."""
    W, H = s["width"], s["heads"]
    return ModelConfig(
        architecture="DeepseekV3ForCausalLM", vocab_size=32768, hidden_size=W, intermediate_size=_gated(s["dense"]),
        num_hidden_layers=layers, num_attention_heads=H, num_key_value_heads=H, rms_norm_eps=1e-6, rope_theta=500000.0,
        max_position_embeddings=16384, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64,
        v_head_dim=128, first_k_dense_replace=2, num_experts=s["experts"], num_experts_per_tok=s["top"],
        moe_intermediate_size=_gated(s["ff"]), n_shared_experts=1, scoring_func="sigmoid", topk_method="greedy",
        norm_topk_prob=False, routed_scaling_factor=1.5)


MODELS = {"naguzen": naguzen_config, "qwen3_next": qwen3_next_config, "deepseek_v3": deepseek_config}


def model_rows(steps: int = 3, warmup: int = 2, sizes=("w2048", "w4096"), batches=((8, 1024), (64, 1024), (1, 8192)),
               models=None, table=None) -> list:
    """``models``: label -> config of one entry of ``table`` (sizes by name)."""
    from ..engine.llm import LLM
    from ..engine.static_workload import StaticWorkload

    rows = []
    for name in sizes:
        s = (table or SIZES)[name]
        for label, make in (models or MODELS).items():
            cfg = make(s)
            top_n = max(n for n, _ in batches)
            blocks = sum(-(-(p + 48) // 64) * n for n, p in batches) + 8
            llm = LLM(cfg, device="cuda", block_size=64, max_model_len=max(p for _, p in batches) + 128, max_num_seqs=top_n,
                      max_num_batched_tokens=8192, num_gpu_blocks=blocks, load_format="dummy", enforce_eager=True)
            params = sum(p.numel() for p in llm.engine.runner.model.parameters())
            for n, prompt in batches:
                out = 33
                wl = StaticWorkload(llm.engine.runner, n, prompt, out, 8192)
                wl.capture()
                pre, dec = [], []
                for i in range(warmup + steps):
                    wl.run()
                    torch.cuda.synchronize()
                    ph = wl.phase_ms()
                    if i >= warmup:
                        pre.append(ph["prefill_ms"])
                        dec.append(ph["decode_ms"] / (out - 1))
                ops.check_kernel_status(0)
                p, d = statistics.median(pre), statistics.median(dec)
                rows.append({"size": name, "model": label, "params_m": round(params / 1e6), "requests": n, "prompt": prompt,
                             "prefill_tok_s": round(n * prompt / p * 1e3), "decode_ms_per_step": round(d, 3),
                             "decode_tok_s": round(n / d * 1e3)})
                wl.graph = None
                del wl
            del llm
            torch.cuda.empty_cache()
    return rows


# ------------------------------------------------------------------------------------------------ single kernels
def _time_us(fn: Callable[[], object], flush: torch.Tensor, iters: int = 15, warmup: int = 3) -> float:
    """Median of ``iters`` launches, L2 overwritten before each; ``fn`` may launch several kernels."""
    ts = []
    for i in range(iters + warmup):
        flush.fill_(float(i))
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        if i >= warmup:
            ts.append(a.elapsed_time(b) * 1e3)
    return statistics.median(ts)


def _peaks() -> tuple[float, float]:
    """(bytes per us, flops per us): the driver's measured copy bandwidth and bf16 GEMM rate, or an earlier measurement."""
    import os

    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            m = json.load(f)
        return m["hbm_gbs"] * 1e3, m["bf16_tflops"] * 1e6
    except (OSError, KeyError, ValueError):
        return 6.65e6, 1.59e9


def kernel_rows(size: str = "w2048", only: str = "") -> list:
    """One row per new kernel and phase: time, roofline fraction, and the same for the like kernel of the closest model."""
    from ..ops.gdn import causal_conv1d, gated_delta_rule
    from ..ops.gla import gated_linear_attention
    from ..ops.residual_conv import residual_conv
    from ..ops.residual_norm import residual_norm
    from ..ops.rglru import rglru

    s = SIZES[size]
    W, H, D, K, R, V = s["width"], s["heads"], 128, 512, 64, 128
    dev, bf = torch.device("cuda"), torch.bfloat16
    ops.load_native()
    flush = torch.empty(64 << 20, dtype=torch.float32, device=dev)
    bw, fl = _peaks()
    rn = lambda *sh, dt=bf: torch.randn(*sh, device=dev, dtype=torch.float32).mul_(0.5).to(dt)
    rows: list = []

    def row(name, fn, nbytes, flops=0.0, like=None):
        if only and only not in name:
            return
        t = _time_us(fn, flush)
        ideal = max(nbytes / bw, flops / fl)
        r = {"size": size, "kernel": name, "us": round(t, 1), "roofline": round(ideal / t, 3)}
        if like is not None:
            ln, lf, lb, lfl = like
            lt = _time_us(lf, flush)
            r.update({"like": ln, "like_us": round(lt, 1), "like_roofline": round(max(lb / bw, lfl / fl) / lt, 3)})
        rows.append(r)

    for T, B in ((8192, 8), (64, 64)):
        phase = "prompt 8x1024" if T > B else "decode 64"
        per = T // B
        qsl = torch.arange(B + 1, dtype=torch.int32, device=dev) * per
        idx, init = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), int(T == B), dtype=torch.int32, device=dev)
        # -- boundaries
        y, x, g1, cw = rn(T, W), rn(T, W, dt=torch.float32), rn(1), rn(W, 4)
        carry, nw, res = torch.zeros(B, 3, W, device=dev), rn(W), rn(T, W)
        norm_like = ("fused_add_rms_norm", lambda: ops.fused_add_rms_norm(y, res, nw, 1e-6), 8.0 * T * W, 0)
        row(f"residual_conv, {phase}", lambda: residual_conv(y, x, g1, cw, 1e-6, carry, qsl, idx, init),
            12.0 * T * W + 4.0 * B * W * 3 * (1 + (T == B)), 0, norm_like)
        row(f"residual_norm, {phase}", lambda: residual_norm(y, x, g1, g1, 1e-6), 8.0 * T * W, 0, norm_like)
        # -- gated linear attention
        n = H * D
        p, al, hn = rn(T, 4 * n + 16), torch.rand(T, n, device=dev), rn(V)
        st = torch.zeros(B, H, D, V, device=dev)
        state_bytes = 4.0 * B * H * D * V * (1 + (T == B))
        q, k, v = rn(T, H, D), rn(T, H, D), rn(T, H, V)
        gg, bb = -torch.rand(T, H, device=dev), torch.rand(T, H, device=dev)
        gdn_bytes = T * H * (2.0 * (2 * D + 2 * V) + 8) + state_bytes
        gdn_like = ("gdn_recurrent", lambda: gated_delta_rule(q, k, v, gg, bb, qsl, st, idx, init), gdn_bytes, 0)
        row(f"gla_recurrent, {phase}",
            lambda: gated_linear_attention(p, (0, n, 2 * n, 3 * n), al, hn, st, qsl, idx, init, D ** -0.5, 1e-6, per),
            T * n * (2.0 * 5 + 4) + state_bytes, 0, gdn_like)
        # -- RG-LRU
        gates, u, yy = rn(T, 16, 2, W // 16, dt=torch.float32), rn(T, W), rn(T, 2 * W)[:, :W]
        f32 = [rn(W, dt=torch.float32) for _ in range(2)] + [-torch.rand(W, device=dev)]
        s1 = torch.zeros(B, W, device=dev)
        row(f"rglru_scan, {phase}", lambda: rglru(u, yy, gates, *f32, s1, qsl, idx, init, per),
            T * W * 14.0 + 4.0 * B * W * (1 + (T == B)), 0, gdn_like)
        gw = rn(16, W // 8, W // 16)
        pw = rn(W // 8, W // 16)
        row(f"block-diagonal gates, {phase}",
            lambda: ops.gemm_batched(u.view(T, 16, W // 16).transpose(0, 1), gw, out=gates.view(T, 16, W // 8).transpose(0, 1)),
            T * W * 10.0 + 2.0 * gw.numel(), 2.0 * T * W * W / 8, ("torch.bmm (bf16 out)", lambda: torch.bmm(
                u.view(T, 16, W // 16).transpose(0, 1), gw.transpose(1, 2)), T * W * 6.0 + 2.0 * gw.numel(), 2.0 * T * W * W / 8))
        cs, kw, kb = torch.zeros(B, 3, W, device=dev, dtype=bf), rn(W, 4), rn(W)
        row(f"causal_conv1d (shared), {phase}", lambda: causal_conv1d(yy, kw, kb, cs, qsl, idx, init, silu=False), 4.0 * T * W)
        # -- latent attention
        ctx, win, bs = 1024, 2048, 64
        nb = ctx // bs + 1
        cache = rn(B * nb, bs, K + R)
        table = torch.arange(B * nb, dtype=torch.int32, device=dev).view(B, nb)
        a, qw, kvw = rn(T, 1536 + K + R), rn(1536), rn(K)
        pos = (torch.arange(T, device=dev) % per) + (ctx - 1 if T == B else 0)
        blk = torch.arange(T, device=dev) // per
        slots = (table.long()[blk, pos // bs] * bs + pos % bs)
        angles = ops.rope_angles(pos, torch.rand(R // 2, device=dev, dtype=torch.float64), T)
        row(f"latent_insert, {phase}",
            lambda: ops.latent_insert(a, 0, 1536, qw, kvw, R, angles, cache, slots, 1e-6),
            2.0 * T * (1536 + K + R) * 2, 0, ("rms_norm (query latent only)", lambda: ops.rms_norm(y, nw, 1e-6), 4.0 * T * W, 0))
        qn, absorb, lat_q = rn(T, H, D + R), rn(H, K, D), rn(T, H, K + R)
        if T == B:
            row(f"absorb q, {phase}", lambda: ops.gemm_batched(qn[..., :D].transpose(0, 1), absorb, out=lat_q[..., :K].transpose(0, 1)),
                2.0 * (T * H * (D + K) + H * K * D), 2.0 * T * H * K * D,
                ("torch.bmm", lambda: torch.bmm(qn[..., :D].transpose(0, 1), absorb.transpose(1, 2)),
                 2.0 * (T * H * (D + K) + H * K * D), 2.0 * T * H * K * D))
            lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
            att = lambda w: (lambda: ops.mla_decode(lat_q, cache, table, lens, 0.07, max_seq_len=ctx, window=w))
            row(f"latent decode, window 2048, context {ctx}", att(win), 2.0 * B * ctx * (K + R), 2.0 * B * H * ctx * (2 * K + R),
                ("mla_decode", att(0), 2.0 * B * ctx * (K + R), 2.0 * B * H * ctx * (2 * K + R)))
            row(f"latent decode, window 512, context {ctx}", att(512), 2.0 * B * 512 * (K + R), 2.0 * B * H * 512 * (2 * K + R),
                ("mla_decode", att(0), 2.0 * B * ctx * (K + R), 2.0 * B * H * ctx * (2 * K + R)))
        else:
            kv = rn(T, H, D + R + V)
            pairs = lambda w: B * sum(min(i + 1, w) for i in range(per))
            kc, vc = kv[..., : D + R].contiguous(), kv[..., D + R:].contiguous()
            for w in (2048, 256):
                fw = 2.0 * H * pairs(w) * (D + R + V)
                row(f"prompt attention 192/128, window {w}", lambda: ops.varlen_attention(
                    qn, kv[..., : D + R], kv[..., D + R:], qsl, qsl, 0.07, max_q_len=per, window=w), 2.0 * T * H * (2 * (D + R) + 2 * V),
                    fw, ("without window, packed K / V", lambda: ops.varlen_attention(qn, kc, vc, qsl, qsl, 0.07, max_q_len=per),
                         2.0 * T * H * (2 * (D + R) + 2 * V), 2.0 * H * pairs(per) * (D + R + V)))
        # -- feed-forward products with their epilogues
        ff = s["dense"]
        wu, coef, gu = rn(ff, W), torch.tensor([0.7, 1.1], device=dev), rn(ff, W)
        by = 2.0 * (T * W + ff * W + T * ff)
        row(f"up product + xIELU, {phase}", lambda: ops.gemm(y, wu, act="xielu", act_params=coef), by, 2.0 * T * W * ff,
            ("gemm_silu_mul, same weight", lambda: ops.gemm_silu_mul(y, gu), by - T * ff, 2.0 * T * W * ff))
        E, top, I = s["experts"], s["top"], s["ff"]
        ids = torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(T)]).to(torch.int32)
        sid, be, total, inv = ops.moe_align_block_size(ids, 128, E, None, want_inverse=True)
        ar = ops.moe_gather(y, sid, total, top)
        w1, w13 = rn(E, I, W), rn(E, _gated(I) * 2, W)
        hit = float(len(torch.unique(ids)))
        eb = lambda n_out, n_rows: 2.0 * (T * top * (W + n_out) + hit * n_rows * W)
        row(f"expert up + gelu, {phase}", lambda: ops.gemm_grouped(ar, w1, be, total, epi=ops.EPI_CODES["gelu"]), eb(I, I),
            2.0 * T * top * I * W, ("expert gate/up + SiLU gate", lambda: ops.gemm_grouped(ar, w13, be, total, epi=1),
                                    eb(_gated(I), 2 * _gated(I)), 2.0 * T * top * 2 * _gated(I) * W))
        rw = rn(E, W)
        row(f"router product (fp32 out), {phase}", lambda: ops.gemm(y, rw, out_dtype=torch.float32), 2.0 * (T * W + E * W + 2 * T * E),
            2.0 * T * W * E, ("router product (bf16 out)", lambda: ops.gemm(y, rw), 2.0 * (T * W + E * W + T * E), 2.0 * T * W * E))
        a1, a2, ab, it = rn(T, 16), rn(n, 16), rn(n), torch.full((1,), 1 / 16, device=dev)
        row(f"decay product, {phase}", lambda: ops.gemm(a1, a2, ab, act="decay", act_params=it, out_dtype=torch.float32), 4.0 * T * n,
            2.0 * T * n * 16, ("bf16 out", lambda: ops.gemm(a1, a2), 2.0 * T * n, 2.0 * T * n * 16))
    ops.check_kernel_status(0)
    return rows
