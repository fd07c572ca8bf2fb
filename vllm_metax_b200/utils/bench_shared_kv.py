"""Prefill and decode throughput of the layer-list decoder with windowed, cross-layer-shared attention and identity experts
(Pupalorn) beside the existing model closest to it (Qwen3-MoE: head norms, rotation, grouped-query attention, routed experts),
at sizes that resemble a real model's layers (random weights), and the time of each of its kernels against its roofline
(``bench.py --shared-kv``).

Same methods as ``bench_hybrid``.  Equal width, depth, heads, head size and experts; the gated experts of Qwen3-MoE are two thirds
as wide, so that an expert has the same number of parameters.
"""
from __future__ import annotations

import torch

from .. import _custom_ops as ops
from ..config import ModelConfig
from . import bench_hybrid
from .bench_hybrid import _gated, _peaks, _time_us

TITLE = "shared-KV decoder beside its closest model"
SIZES = {
    # width, query heads, key / value heads, experts, identity experts, top, expert ff, sliding window
    "w2048": dict(width=2048, heads=16, kv=4, experts=64, identity=8, top=8, ff=1152, window=1024),
    "w4096": dict(width=4096, heads=32, kv=8, experts=32, identity=4, top=4, ff=2304, window=1024),
}
ROT = {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}


def pupalorn_config(s: dict, layers: int = 8, share: bool = True, window: bool = True) -> ModelConfig:
    """The upper half of the layers reads the keys and values of the layer below it (``share``)."""
    mlp = {"kind": "moe", "router": {"experts": s["experts"], "identity": s["identity"], "top": s["top"]}, "expert": {"ff": s["ff"]}}
    out = []
    for i in range(layers):
        m = {"heads": s["heads"], "kv_heads": s["kv"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": ROT}
        if window:
            m["mask"] = {"size": s["window"]}
        if share and i >= layers // 2:
            m["kv_from"] = layers // 2 - 1
        out.append({"type": "attention", "mixer": m, "mlp": mlp})
    return ModelConfig.from_layer_list({"architecture": "Pupalorn", "vocab": 32768, "width": s["width"], "norm": {"eps": 1e-6},
                                        "embedding": {"scale": 8.0}, "residual_mult": 0.4, "layers": out})


def qwen3_moe_config(s: dict, layers: int = 8) -> ModelConfig:
    return ModelConfig.from_hf_dict(dict(
        architectures=["Qwen3MoeForCausalLM"], vocab_size=32768, hidden_size=s["width"], intermediate_size=4 * s["width"],
        num_hidden_layers=layers, num_attention_heads=s["heads"], num_key_value_heads=s["kv"], head_dim=128, rms_norm_eps=1e-6,
        rope_theta=500000.0, max_position_embeddings=16384, num_experts=s["experts"], num_experts_per_tok=s["top"],
        moe_intermediate_size=_gated(s["ff"]), norm_topk_prob=False, decoder_sparse_step=1, mlp_only_layers=[]))


MODELS = {"pupalorn": pupalorn_config,
          "pupalorn, own K / V everywhere, no window": lambda s: pupalorn_config(s, share=False, window=False),
          "qwen3_moe": qwen3_moe_config}


def model_rows(steps: int = 3, warmup: int = 2, sizes=("w2048", "w4096"), **kw) -> list:
    return bench_hybrid.model_rows(steps, warmup, sizes, models=MODELS, table=SIZES, **kw)


def kernel_rows(size: str = "w2048", only: str = "") -> list:
    """One row per kernel that is new or changed for this design, prompt and decode: time, roofline fraction, and the same for
    the like kernel of the closest model."""
    from ..layers.fused_moe import expert_rows
    from ..ops.residual_norm import ExpertRows, boundary_norm, embed_norm

    s = SIZES[size]
    W, H, G, D, win = s["width"], s["heads"], s["kv"], 128, s["window"]
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
        # -- boundaries
        y, x, nw, res = rn(T, W), rn(T, W, dt=torch.float32), rn(W), rn(T, W)
        g1, g2 = rn(W, dt=torch.float32), rn(W, dt=torch.float32)
        norm_like = ("fused_add_rms_norm", lambda: ops.fused_add_rms_norm(y, res, nw, 1e-6), 8.0 * T * W, 0)
        if B != 1:
            row(f"boundary_norm, {phase}", lambda: boundary_norm(y, x, g1, g2, 1e-6), 12.0 * T * W, 0, norm_like)
            row(f"boundary_norm in front of the head, {phase}", lambda: boundary_norm(y, x, g1, g2, 1e-6, want_x=False),
                8.0 * T * W, 0, norm_like)
            table, ids = rn(32768, W), torch.randint(0, 32768, (T,), device=dev)
            row(f"embed_norm, {phase}", lambda: embed_norm(table, ids, 32768, 8.0, g2, 1e-6), 8.0 * T * W, 0,
                ("embedding", lambda: ops.embedding(table, ids), 4.0 * T * W, 0))
        # -- projection epilogue
        bs, nb = 64, ctx // 64 + 1
        cache = rn(B * nb, 2, bs, G, D)
        bt = torch.arange(B * nb, dtype=torch.int32, device=dev).view(B, nb)
        pos = (torch.arange(T, device=dev) % per) + (ctx - 1 if decode else 0)
        slots = bt.long()[torch.arange(T, device=dev) // per, pos // bs] * bs + pos % bs
        qkv, qw, kw = rn(T, (H + 2 * G) * D), rn(D), rn(D)
        freq = torch.rand(32, device=dev, dtype=torch.float64)
        ang = ops.rope_angles(pos, freq, T)
        cs = torch.rand(16384, D, device=dev)
        q, k, v = qkv[:, : H * D], qkv[:, H * D: (H + G) * D], qkv[:, (H + G) * D:]
        kv = ops.kv_views(cache)
        off = (0, H * D, (H + G) * D)

        def separate():                    # what the closest model runs: head norms, then rotation and cache write
            ops.head_rms_norm(q, qw, 1e-6, H, D)
            ops.head_rms_norm(k, kw, 1e-6, G, D)
            ops.rope_and_cache(pos, q, k, v, D, cs, True, cache, slots)

        if B != 1:
            row(f"rope_angles (once a step), {phase}", lambda: ops.rope_angles(pos, freq, T), 4.0 * T * 64)
            byts = 4.0 * T * (H + 2 * G) * D
            row(f"head_norm_rope, {phase}", lambda: ops.head_norm_rope(qkv, off, qw, kw, H, D, ang, kv, slots, 1e-6), byts, 0,
                ("head_rms_norm x 2 + rope_and_cache", separate, byts, 0))
            qo = rn(T, H * D)
            row(f"head_norm_rope, queries only, {phase}",
                lambda: ops.head_norm_rope(qo, (0, 0, 0), qw, None, H, D, ang, None, slots, 1e-6), 4.0 * T * H * D, 0,
                ("head_rms_norm", lambda: ops.head_rms_norm(qo, qw, 1e-6, H, D), 4.0 * T * H * D, 0))
        # -- attention
        q3 = rn(T, H, D)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        if decode:
            att = lambda w: (lambda: ops.paged_attention_decode(q3, cache, bt, lens, 0.09, window=w, max_seq_len=ctx))
            cost = lambda n: 4.0 * B * n * G * D + 4.0 * T * H * D
            for w in (win, 128):
                short = torch.full((B,), w, dtype=torch.int32, device=dev)      # as many keys without a window
                row(f"paged decode, window {w}, {phase}", att(w), cost(w), 4.0 * B * H * w * D,
                    (f"paged decode, context {w}", lambda: ops.paged_attention_decode(q3, cache, bt, short, 0.09, max_seq_len=w),
                     cost(w), 4.0 * B * H * w * D))
        else:
            qsl = torch.arange(B + 1, dtype=torch.int32, device=dev) * per
            att = lambda w: (lambda: ops.paged_attention_prefill(q3, cache, bt, lens, qsl, 0.09, max_q_len=per, window=w, max_seq_len=ctx))
            pairs = lambda w: B * sum(min(i + 1, w) for i in range(per))
            byts = 4.0 * T * H * D + 4.0 * T * G * D
            row(f"paged prompt attention, window {win}, {phase}", att(win), byts, 4.0 * H * pairs(win) * D,
                ("without a window", att(-1), byts, 4.0 * H * pairs(per) * D))
            # a short window against prompts as short as it: as many key tiles per query tile
            n = T // 128
            bt2 = torch.arange(2 * n, dtype=torch.int32, device=dev).view(n, 2)
            len2, qsl2 = torch.full((n,), 128, dtype=torch.int32, device=dev), torch.arange(n + 1, dtype=torch.int32, device=dev) * 128
            row(f"paged prompt attention, window 128, {phase}", att(128), byts, 4.0 * H * pairs(128) * D,
                (f"prompts {n}x128 without a window", lambda: ops.paged_attention_prefill(
                    q3, cache, bt2, len2, qsl2, 0.09, max_q_len=128, max_seq_len=128), byts, 4.0 * H * n * 128 * 129 / 2 * D))
        if B == 1:
            continue
        # -- experts
        E, I, top, ff, gf = s["experts"], s["identity"], s["top"], s["ff"], _gated(s["ff"])
        gate, bias = rn(E + I, W), rn(E + I, dt=torch.float32)
        row(f"router product (fp32 out), {phase}", lambda: ops.router_logits(y, gate),
            2.0 * (T * W + (E + I) * W) + 4.0 * T * (E + I), 2.0 * T * W * (E + I),
            ("router product (bf16 out)", lambda: ops.gemm(y, gate[:E]), 2.0 * (T * W + E * W + T * E), 2.0 * T * W * E))
        z, zb = rn(T, E + I, dt=torch.float32), rn(T, E)
        row(f"topk_gating with correction, {phase}", lambda: ops.topk_gating(z, top, False, "softmax", bias), 4.0 * T * (E + I), 0,
            ("topk_gating", lambda: ops.topk_gating(zb, top, False), 2.0 * T * E, 0))
        ids = torch.stack([torch.randperm(E + I, device=dev)[:top] for _ in range(T)]).to(torch.int32)
        idr = torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(T)]).to(torch.int32)
        wt = torch.rand(T, top, device=dev)
        real = float((ids < E).sum())
        sid, be, total, inv = ops.moe_align_block_size(ids, 128, E, None, want_inverse=True)
        ar = ops.moe_gather(y, sid, total, top)
        w1, w13, w2, w2g = rn(E, ff, W), rn(E, 2 * gf, W), rn(E, W, ff), rn(E, W, gf)
        hit = float(len(torch.unique(ids[ids < E])))
        row(f"expert up + squared relu, {phase}", lambda: ops.gemm_grouped(ar, w1, be, total, epi=ops.EPI_CODES["relu2"]),
            2.0 * (real * (W + ff) + hit * ff * W), 2.0 * real * ff * W,
            ("expert gate/up + SiLU gate", lambda: ops.gemm_grouped(ar, w13, be, total, epi=1),
             2.0 * (real * (W + gf) + hit * 2 * gf * W), 4.0 * real * gf * W))
        er = ops.gemm_grouped(ops.gemm_grouped(ar, w1, be, total, epi=ops.EPI_CODES["relu2"]), w2, be, total)
        late = ExpertRows(er, wt, inv, ids, y, E)

        def combine_then_norm():
            ops.fused_add_rms_norm(ops.moe_combine(er, wt, inv, T), res, nw, 1e-6)

        row(f"expert combine + boundary_norm, {phase}", lambda: boundary_norm(late, x, g1, g2, 1e-6),
            2.0 * T * top * W + 10.0 * T * W, 0,
            ("moe_combine + fused_add_rms_norm", combine_then_norm, 2.0 * real * W + 2.0 * T * W + 8.0 * T * W, 0))
        row(f"experts, align to combine, {phase}",
            lambda: expert_rows(y, w1, w2, wt, ids, E, None, None, ops.EPI_CODES["relu2"], E).combined(),
            4.0 * hit * ff * W + 4.0 * T * W, 4.0 * real * ff * W,
            ("experts of the closest model", lambda: expert_rows(y, w13, w2g, wt, idr, E).combined(),
             2.0 * hit * 3 * gf * W + 4.0 * T * W, 6.0 * T * top * gf * W))
    ops.check_kernel_status(0)
    return rows
