"""Prefill and decode throughput of the looped layer-list decoder with two mixers side by side (Luluzen) beside the existing
models closest to it (Qwen3-Next: delta rule and attention in turn, routed experts; Naguzen: gated linear attention, latent
attention, routed experts), at sizes that resemble a real model's layers (random weights), and the time of each of its kernels
against its roofline (``bench.py --parallel``).

Same methods as ``bench_hybrid``.  Equal width, depth (layer runs), heads, state sizes and experts; all three models' experts have
the same number of parameters.
"""
from __future__ import annotations

import torch

from .. import _custom_ops as ops
from ..config import ModelConfig
from . import bench_hybrid
from .bench_hybrid import _peaks, _time_us, naguzen_config, qwen3_next_config

TITLE = "looped decoder with mixers side by side beside its closest models"
SIZES = {
    # width, query (and recurrent) heads, key / value heads, experts, top, expert ff (gated), dense ff, sliding window; moe_ff and
    # shared: what the closest models' tables call them (a plain feed-forward of the same parameters)
    "w2048": dict(width=2048, heads=16, kv=4, experts=64, top=8, gated_ff=512, ff=768, shared=768, dense=8192, window=1024),
    "w4096": dict(width=4096, heads=32, kv=8, experts=32, top=4, gated_ff=1024, ff=1536, shared=1536, dense=16384, window=1024),
}


def luluzen_config(s: dict) -> ModelConfig:
    """Eight layer runs: six layers, of which two are passed through twice."""
    H, G = s["heads"], s["kv"]
    moe = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"]}, "expert": {"ff": s["gated_ff"], "limit": 7.0}}
    dense = {"kind": "dense", "ff": s["dense"] * 2 // 3 // 64 * 64}
    att = {"heads": H, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    lightning = {"type": "lightning", "mlp": moe,
                 "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-2 - 6 * i / H) for i in range(H)]}}
    memory = {"type": "parallel_2", "mlp": dense, "mixer": {
        "left": {**att, "softcap": 50.0, "mask": {"size": s["window"]}, "rot": {"base": 500000.0, "dims": 64}},
        "right": {"heads": H, "dim": 128, "vdim": 128, "gate_cap": 15.0}, "left_scale": 0.8, "right_scale": 0.7}}
    delta = {"type": "parallel", "mlp": moe, "mixer": {
        "left": {**att, "bias_max": 512, "q_temp": {"coef": 0.1, "every": 4096}},
        "right": {"heads": H, "kv_heads": H, "dim": 128, "vdim": 128, "conv": 4}, "left_scale": 0.8, "right_scale": 0.7}}
    return ModelConfig.from_layer_list({
        "architecture": "Luluzen", "vocab": 32768, "width": s["width"], "norm": {"eps": 1e-6}, "logit_softcap": 30.0,
        "loop": {"start": 1, "stop": 3, "times": 2}, "layers": [memory, lightning, delta, lightning, {**memory, "mlp": moe}, delta]})


MODELS = {"luluzen": luluzen_config, "qwen3_next": qwen3_next_config, "naguzen": naguzen_config}


def model_rows(steps: int = 3, warmup: int = 2, sizes=("w2048", "w4096"), **kw) -> list:
    return bench_hybrid.model_rows(steps, warmup, sizes, models=kw.pop("models", MODELS), table=SIZES, **kw)


def kernel_rows(size: str = "w2048", only: str = "") -> list:
    """One row per kernel that is new or changed for this design, prompt and decode: time, roofline fraction, and the same for
    the like kernel of the closest model."""
    from ..layers.attention import distance_buckets
    from ..ops.channel_delta import channel_delta_rule
    from ..ops.gdn import causal_conv1d, gated_delta_rule
    from ..ops.gla import Normalizer, Steps, gated_linear_attention, linear_attention, memory_gates
    from ..ops.prenorm import loop_operand, prenorm
    from ..ops.residual_norm import ExpertRows

    s = SIZES[size]
    W, H, G, D, win = s["width"], s["heads"], s["kv"], 128, s["window"]
    dev, bf, f32 = torch.device("cuda"), torch.bfloat16, torch.float32
    ops.load_native()
    flush = torch.empty(64 << 20, dtype=f32, device=dev)
    bw, fl = _peaks()
    rn = lambda *sh, dt=bf: torch.randn(*sh, device=dev, dtype=f32).mul_(0.5).to(dt)
    rows: list = []

    def row(name, fn, nbytes, flops=0.0, like=None):
        if only and only not in name:
            return
        t = _time_us(fn, flush)
        r = {"size": size, "kernel": name, "us": round(t, 1), "roofline": round(max(nbytes / bw, flops / fl) / t, 3)}
        if like is not None:
            ln, lf, lb, lfl = like
            lt = _time_us(lf, flush)
            r.update({"like": ln, "like_us": round(lt, 1), "like_roofline": round(max(lb / bw, lfl / fl) / lt, 3)})
        rows.append(r)

    for T, B, ctx in ((8192, 8, 1024), (8192, 1, 8192), (64, 64, 2048)):
        decode = T == B
        per = T // B
        phase = f"decode {B}, context {ctx}" if decode else f"prompt {B}x{per}"
        qsl = torch.arange(B + 1, dtype=torch.int32, device=dev) * per
        idx, init = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), int(decode), dtype=torch.int32, device=dev)
        steps = Steps(qsl, idx, init, per)
        # -- recurrences
        n = H * D
        st = torch.zeros(B, H, D, D, device=dev)
        state_bytes = 4.0 * B * H * D * D * (1 + decode)
        p = rn(T, 4 * n + 16)
        off = (0, n, 2 * n, 3 * n)
        q, k, v = rn(T, H, D), rn(T, H, D), rn(T, H, D)
        gg, bb = -torch.rand(T, H, device=dev), torch.rand(T, H, device=dev)
        like = ("gated_delta_rule", lambda: gated_delta_rule(q, k, v, gg, bb, qsl, st, idx, init),
                T * H * (8.0 * D + 8) + state_bytes, 0)
        hn, rw = rn(D), rn(n)
        alpha = torch.rand(T, n, device=dev)
        gla_like = ("gated_linear_attention", lambda: gated_linear_attention(p, off, alpha, hn, st, qsl, idx, init, D ** -0.5, 1e-6, per),
                    T * n * 14.0 + state_bytes, 0)
        dec = torch.rand(H, device=dev)
        lin = lambda: linear_attention(p, off, dec, rw, st, steps, 1.0, 1e-6, "sigmoid", True, True)
        row(f"lightning attention, {phase}", lin, T * n * 10.0 + state_bytes, 0, like)
        row(f"lightning attention against gla, {phase}", lin, T * n * 10.0 + state_bytes, 0, gla_like)
        z, zb, top, nst = rn(T, 2 * H, dt=f32), rn(2 * H, dt=f32), torch.zeros(B, H, device=dev), torch.zeros(B, H, D // 16, D, device=dev)
        g3 = memory_gates(z, zb, 15.0, top, steps)
        row(f"memory gates, {phase}", lambda: memory_gates(z, zb, 15.0, top, steps), T * H * 20.0)

        def memory():
            g = memory_gates(z, zb, 15.0, top, steps)
            linear_attention(p, off, g[0], rw, st, steps, D ** -0.5, 1e-6, "sigmoid", memory=Normalizer(nst, g[1], g[2]))

        row(f"matrix memory with its gates, {phase}", memory, T * n * 10.0 + T * H * 32.0 + state_bytes * 1.0625, 0, like)
        row(f"matrix memory, {phase}", lambda: linear_attention(p, off, g3[0], rw, st, steps, D ** -0.5, 1e-6, "sigmoid",
                                                                  memory=Normalizer(nst, g3[1], g3[2])),
            T * n * 10.0 + T * H * 12.0 + state_bytes * 1.0625, 0, gla_like)
        gate = rn(T, n)
        row(f"channel delta rule, {phase}", lambda: channel_delta_rule(p, off[:3], H, alpha, bb, gate, hn, st, steps, 1e-6),
            T * n * 14.0 + T * H * 4.0 + state_bytes, 0, like)
        cs, kw_ = torch.zeros(B, 3, 3 * n, device=dev, dtype=bf), rn(3 * n, 4)
        row(f"causal_conv1d (shared), {phase}", lambda: causal_conv1d(p[:, : 3 * n], kw_, None, cs, qsl, idx, init), 12.0 * T * n)
        # -- attention
        bs, nb = 64, ctx // 64 + 1
        cache = rn(B * nb, 2, bs, G, D)
        bt = torch.arange(B * nb, dtype=torch.int32, device=dev).view(B, nb)
        pos = (torch.arange(T, device=dev) % per) + (ctx - 1 if decode else 0)
        kv = ops.kv_views(cache)
        q3 = rn(T, H, D)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        bias = rn(32, H, dt=f32)[distance_buckets(32, 512)].t().contiguous()
        tiles = {} if decode else {"bias_tiles": ops.distance_bias_tiles(bias, H // G)}
        sink = rn(H, dt=f32)
        wide = rn(T, 2 * n)
        ot = wide[:, :n].unflatten(1, (H, D))
        if decode:
            att = lambda **kw: (lambda: ops.paged_attention_decode(q3, cache, bt, lens, 0.09, max_seq_len=ctx, **kw))
            cost, flp = (lambda w: 4.0 * B * w * G * D + 4.0 * T * n), (lambda w: 4.0 * B * H * w * D)
        else:
            att = lambda **kw: (lambda: ops.paged_attention_prefill(q3, cache, bt, lens, qsl, 0.09, max_q_len=per, max_seq_len=ctx, **kw))
            cost = lambda w: 4.0 * T * n + 4.0 * T * G * D
            flp = lambda w: 4.0 * H * B * sum(min(i + 1, w) for i in range(per)) * D
        plain = lambda w: (f"plain, window {w}" if w < ctx else "plain", att(window=w if w < ctx else -1), cost(min(w, ctx)), flp(w))
        row(f"attention with a distance bias, {phase}", att(distance_bias=bias, out=ot, out_scale=0.8, **tiles), cost(ctx), flp(ctx), plain(ctx))
        row(f"capped window attention, sink and gate, {phase}",
            att(window=win, softcap=50.0, sinks=sink, gate=gate, out=ot, out_scale=0.8), cost(min(win, ctx)) + 2.0 * T * n, flp(win), plain(win))
        # -- the rest does not care how the tokens are cut
        if B == 1:
            continue
        slots = bt.long()[torch.arange(T, device=dev) // per, pos // bs] * bs + pos % bs
        qkv, qw, kw, qr, kr = rn(T, (H + 2 * G) * D), rn(D), rn(D), rn(H * D), rn(G * D)
        ang = ops.rope_angles(pos, torch.rand(32, device=dev, dtype=torch.float64), T)
        csn = torch.rand(16384, D, device=dev)
        qa, ka, va = qkv[:, : H * D], qkv[:, H * D: (H + G) * D], qkv[:, (H + G) * D:]
        at = (0, H * D, (H + G) * D)

        def separate():                    # what the closest model runs: head norms, then rotation and cache write
            ops.head_rms_norm(qa, qw, 1e-6, H, D)
            ops.head_rms_norm(ka, kw, 1e-6, G, D)
            ops.rope_and_cache(pos, qa, ka, va, D, csn, True, cache, slots)

        byts = 4.0 * T * (H + 2 * G) * D
        sep = ("head_rms_norm x 2 + rope_and_cache", separate, byts, 0)
        row(f"row norm + pair rotation + cache, {phase}", lambda: ops.head_norm_rope(
            qkv, at, qr, kr, H, D, ang, kv, slots, 1e-6, whole_row=True, interleaved=True), byts, 0, sep)
        row(f"head norm + temperature + cache, {phase}", lambda: ops.head_norm_rope(
            qkv, at, qw, kw, H, D, None, kv, slots, 1e-6, q_temp=(pos, 0.1, 4096)), byts, 0, sep)
        y, x, nw, res, g1 = rn(T, W), rn(T, W, dt=f32), rn(W), rn(T, W), rn(W)
        norm_like = ("fused_add_rms_norm", lambda: ops.fused_add_rms_norm(y, res, nw, 1e-6), 8.0 * T * W, 0)
        row(f"prenorm, {phase}", lambda: prenorm(y, x, g1, 1e-6), 12.0 * T * W, 0, norm_like)
        row(f"prenorm in front of the head, {phase}", lambda: prenorm(y, x, g1, 1e-6, want_x=False), 8.0 * T * W, 0, norm_like)
        row(f"prenorm behind the loop's product, {phase}", lambda: prenorm(x, None, g1, 1e-6, nw), 10.0 * T * W, 0, norm_like)
        table, ids = rn(32768, W), torch.randint(0, 32768, (T,), device=dev)
        row(f"prenorm of embeddings, {phase}", lambda: prenorm(table, None, g1, 1e-6, None, ids, 32768), 8.0 * T * W, 0,
            ("embedding", lambda: ops.embedding(table, ids), 4.0 * T * W, 0))
        row(f"loop operand, {phase}", lambda: loop_operand(y, x, table, ids, 32768), 14.0 * T * W, 0, norm_like)
        # -- products
        op, wi = rn(T, 3 * W), rn(W, 3 * W)
        row(f"loop product (fp32 out), {phase}", lambda: ops.gemm(op, wi, out_dtype=f32), 2.0 * (3 * T * W + 3 * W * W) + 4.0 * T * W,
            6.0 * T * W * W, ("bf16 out", lambda: ops.gemm(op, wi), 2.0 * (4 * T * W + 3 * W * W), 6.0 * T * W * W))
        ff = s["dense"] * 2 // 3 // 64 * 64
        gu = rn(2 * ff, W)
        by = 2.0 * (T * W + 2 * ff * W + T * ff)
        row(f"gate/up product + gelu gate, {phase}", lambda: ops.gemm(y, gu, act="gelu_tanh_gate"), by, 4.0 * T * W * ff,
            ("gemm_silu_mul", lambda: ops.gemm_silu_mul(y, gu), by, 4.0 * T * W * ff))
        a1, a2, ab, rate = rn(T, D), rn(n, D), rn(n), torch.rand(n, device=dev)
        row(f"decay product (softplus, fp32 out), {phase}", lambda: ops.gemm(a1, a2, ab, act="softplus_decay", act_params=rate, out_dtype=f32),
            2.0 * (T * D + n * D) + 4.0 * T * n, 2.0 * T * n * D,
            ("bf16 out", lambda: ops.gemm(a1, a2, ab), 2.0 * (T * D + n * D + T * n), 2.0 * T * n * D))
        if decode:
            cap = torch.full((1,), 30.0, device=dev)
            row(f"capped logits (fp32 out), {phase}", lambda: ops.gemm(y, table, act="softcap", act_params=cap, out_dtype=f32),
                2.0 * (T * W + table.numel()) + 4.0 * T * 32768, 2.0 * T * table.numel(),
                ("logits (bf16 out)", lambda: ops.gemm(y, table), 2.0 * (T * W + table.numel() + T * 32768), 2.0 * T * table.numel()))
        gw = rn(2 * H, W)
        row(f"recurrence gates product (fp32 out), {phase}", lambda: ops.router_logits(y, gw), 2.0 * (T * W + 2 * H * W) + 8.0 * T * H,
            4.0 * T * W * H, ("bf16 out", lambda: ops.gemm(y, gw), 2.0 * (T * W + 2 * H * W + 2 * T * H), 4.0 * T * W * H))
        # -- experts
        E, tp, gf = s["experts"], s["top"], s["gated_ff"]
        eids = torch.stack([torch.randperm(E, device=dev)[:tp] for _ in range(T)]).to(torch.int32)
        wt, limit = torch.rand(T, tp, device=dev), torch.tensor([7.0, 1.702], device=dev)
        sid, be, total, inv = ops.moe_align_block_size(eids, 128, E, None, want_inverse=True)
        hit = float(len(torch.unique(eids)))
        row(f"weighted gather, {phase}", lambda: ops.moe_gather(y, sid, total, tp, wt), 2.0 * T * W + 2.0 * T * tp * W, 0,
            ("moe_gather", lambda: ops.moe_gather(y, sid, total, tp), 2.0 * T * W + 2.0 * T * tp * W, 0))
        ar, w13, w2 = ops.moe_gather(y, sid, total, tp, wt), rn(E, 2 * gf, W), rn(E, W, gf)
        eb = 2.0 * (T * tp * (W + gf) + hit * 2 * gf * W)
        row(f"expert gate/up + clamped gate, {phase}",
            lambda: ops.gemm_grouped(ar, w13, be, total, ops.EPI_CODES["clamped_swiglu_gate"], limit), eb, 4.0 * T * tp * gf * W,
            ("expert gate/up + SiLU gate", lambda: ops.gemm_grouped(ar, w13, be, total, 1), eb, 4.0 * T * tp * gf * W))
        er = ops.gemm_grouped(ops.gemm_grouped(ar, w13, be, total, 1), w2, be, total)
        late = ExpertRows(er, None, inv, top=tp)

        def combine_then_norm():
            ops.fused_add_rms_norm(ops.moe_combine(er, wt, inv, T), res, nw, 1e-6)

        row(f"expert sums + prenorm, {phase}", lambda: prenorm(late, x, g1, 1e-6), 2.0 * T * tp * W + 10.0 * T * W, 0,
            ("moe_combine + fused_add_rms_norm", combine_then_norm, 2.0 * T * tp * W + 10.0 * T * W, 0))
    ops.check_kernel_status(0)
    return rows
