"""Prefill and decode throughput of the attention-only decoder over several residual streams (Vetipel) beside the existing models
closest to it (Llama: grouped-query attention in every layer; DeepSeek-V3 with dense feed-forwards: latent attention in every
layer), at sizes that resemble a real model's layers (random weights), and the time of each of its kernels against its roofline
(``bench.py --streams``).

Same methods as ``bench_hybrid``.  Equal width, depth, heads and feed-forward parameters.
"""
from __future__ import annotations

import torch

from .. import _custom_ops as ops
from ..config import ModelConfig
from . import bench_hybrid
from .bench_hybrid import _gated, _peaks, _time_us

TITLE = "decoder over several residual streams beside its closest models"
SIZES = {
    # width, query heads, key / value heads, dense ff (not gated), residual streams, sliding window and chunk
    "w2048": dict(width=2048, heads=16, kv=4, dense=8192, streams=4, reach=1024),
    "w4096": dict(width=4096, heads=32, kv=8, dense=16384, streams=4, reach=1024),
}
LAYERS = 8


def vetipel_config(s: dict) -> ModelConfig:
    """Twice (windowed sigmoid attention, chunked attention, latent attention, chunked attention)."""
    dense = {"kind": "dense", "ff": s["dense"]}
    att = {"heads": s["heads"], "kv_heads": s["kv"], "dim": 128, "vdim": 128, "mask": {"size": s["reach"]}, "scale": 128 ** -0.5}
    lat = {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "rot": {"base": 500000.0, "dims": 64},
           "scale": 192 ** -0.5}
    kinds = [("attention", att), ("attention_2", att), ("latent_attention", lat), ("attention_2", att)] * (LAYERS // 4)
    return ModelConfig.from_layer_list({
        "architecture": "Vetipel", "vocab": 32768, "width": s["width"], "streams": s["streams"], "embedding": {"scale": 8.0},
        "norm": {"eps": 1e-6}, "layers": [{"type": t, "mixer": m, "mlp": dense} for t, m in kinds]})


def llama_config(s: dict) -> ModelConfig:
    return ModelConfig(architecture="LlamaForCausalLM", vocab_size=32768, hidden_size=s["width"],
                       intermediate_size=_gated(s["dense"]), num_hidden_layers=LAYERS, num_attention_heads=s["heads"],
                       num_key_value_heads=s["kv"], head_dim=128, rms_norm_eps=1e-6, rope_theta=500000.0,
                       max_position_embeddings=16384)


def deepseek_config(s: dict) -> ModelConfig:
    return ModelConfig(
        architecture="DeepseekV3ForCausalLM", vocab_size=32768, hidden_size=s["width"], intermediate_size=_gated(s["dense"]),
        num_hidden_layers=LAYERS, num_attention_heads=s["heads"], num_key_value_heads=s["heads"], rms_norm_eps=1e-6,
        rope_theta=500000.0, max_position_embeddings=16384, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
        qk_rope_head_dim=64, v_head_dim=128, first_k_dense_replace=LAYERS)


MODELS = {"vetipel": vetipel_config, "llama": llama_config, "deepseek_v3_dense": deepseek_config}


def model_rows(steps: int = 3, warmup: int = 2, sizes=("w2048", "w4096"), **kw) -> list:
    return bench_hybrid.model_rows(steps, warmup, sizes, models=kw.pop("models", MODELS), table=SIZES, **kw)


def kernel_rows(size: str = "w2048", only: str = "") -> list:
    """One row per kernel that is new or changed for this design, prompt and decode: time, roofline fraction, and the same for
    the like kernel of the closest model."""
    from ..ops.mhc import mhc_fused_post_pre
    from ..ops.stream_norm import Embedded, stream_norm

    s = SIZES[size]
    W, H, G, S, D, reach = s["width"], s["heads"], s["kv"], s["streams"], 128, s["reach"]
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

    for T, B, ctx in ((8192, 8, 1024), (8192, 1, 8192), (64, 64, 2048), (8, 8, 2048)):
        decode = T == B
        per = T // B
        phase = f"decode {B}, context {ctx}" if decode else f"prompt {B}x{per}"
        # -- attention
        bs, nb, n = 64, ctx // 64 + 1, H * D
        cache = rn(B * nb, 2, bs, G, D)
        bt = torch.arange(B * nb, dtype=torch.int32, device=dev).view(B, nb)
        pos = (torch.arange(T, device=dev) % per) + (ctx - 1 if decode else 0)
        kv, q3, gate = ops.kv_views(cache), rn(T, H, D), rn(T, H)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], device=dev)
        shift, sink = rn(H, dt=f32) - 4.0, rn(H, dt=f32)
        bias = -torch.rand(H, 1, device=dev) * torch.log1p(torch.arange(reach, device=dev, dtype=f32))[None]
        tiles = {} if decode else {"bias_tiles": ops.distance_bias_tiles(bias, H // G)}
        if decode:
            att = lambda **kw: (lambda: ops.paged_attention_decode(q3, cache, bt, lens, 0.09, max_seq_len=ctx, **kw))
            seen = lambda w: B * min(w, ctx)
            cost = lambda w: 4.0 * B * min(w, ctx) * G * D + 4.0 * T * n
        else:
            qsl = torch.arange(B + 1, dtype=torch.int32, device=dev) * per
            att = lambda **kw: (lambda: ops.paged_attention_prefill(q3, cache, bt, lens, qsl, 0.09, max_q_len=per, max_seq_len=ctx, **kw))
            seen = lambda w: B * sum(min(i + 1, w) for i in range(per))
            cost = lambda w: 4.0 * T * n + 4.0 * T * G * D
        flops = lambda pairs: 4.0 * H * pairs * D
        w = reach if reach < ctx else -1
        plain = (f"plain, window {w}" if w > 0 else "plain", att(window=w), cost(reach), flops(seen(reach)))
        row(f"sigmoid attention, slopes, window, head gate, {phase}", att(window=reach, sigmoid_shift=shift, alibi_slopes=slopes, gate=gate),
            cost(reach), flops(seen(reach)), plain)
        row(f"the same with a softmax, {phase}", att(window=reach, alibi_slopes=slopes, gate=gate), cost(reach), flops(seen(reach)), plain)
        in_chunk = B * ((ctx - 1) % reach + 1) if decode else B * sum(i % reach + 1 for i in range(per))
        chunk_cost = 4.0 * in_chunk * G * D + 4.0 * T * n if decode else cost(reach)
        row(f"chunked attention, log bias, sink, head gate, {phase}", att(chunk=reach, distance_bias=bias, sinks=sink, gate=gate, **tiles),
            chunk_cost, flops(in_chunk), plain)
        row(f"chunked attention, {phase}", att(chunk=reach), chunk_cost, flops(in_chunk), plain)
        # -- the rest does not care how the tokens are cut
        if B == 1 or T == 8:
            continue
        slots = bt.long()[torch.arange(T, device=dev) // per, pos // bs] * bs + pos % bs
        qkv, qw, kw = rn(T, (H + 2 * G) * D + 16), rn(D), rn(D)
        csn, temp = torch.rand(16384, D, device=dev), torch.rand(H, device=dev)
        qa, ka, va = (qkv[:, a: b] for a, b in ((0, n), (n, n + G * D), (n + G * D, n + 2 * G * D)))
        at = (0, n, n + G * D)

        def separate():                    # what a model with head norms runs: head norms, then rotation and cache write
            ops.head_rms_norm(qa, qw, 1e-6, H, D)
            ops.head_rms_norm(ka, kw, 1e-6, G, D)
            ops.rope_and_cache(pos, qa, ka, va, D, csn, True, cache, slots)

        byts = 4.0 * T * (H + 2 * G) * D
        row(f"unit head norm + temperature + cache, {phase}", lambda: ops.head_norm_rope(
            qkv, at, None, None, H, D, None, kv, slots, 1e-6, q_scale=temp, width=D), byts, 0,
            ("head_rms_norm x 2 + rope_and_cache", separate, byts, 0))
        row(f"cache write, {phase}", lambda: ops.head_norm_rope(qkv, at, None, None, H, D, None, kv, slots, 1e-6, normed=False, width=D),
            8.0 * T * G * D, 0, ("reshape_and_cache", lambda: ops.reshape_and_cache(ka, va, cache, slots), 8.0 * T * G * D, 0))
        K, R, QR = 512, 64, H * 192
        lat, a, kn = rn(B * nb, bs, K + R), rn(T, QR + K + R), rn(K)
        c512, krot = rn(T, K), rn(T, 1, R)
        ang = ops.rope_angles(pos, torch.rand(R // 2, device=dev, dtype=torch.float64), T)
        y, nw, res = rn(T, W), rn(W), rn(T, W)
        row(f"latent_insert without queries, {phase}", lambda: ops.latent_insert(a, 0, QR, None, kn, R, ang, lat, slots, 1e-6, interleaved=True),
            4.0 * T * (K + R), 0, ("rms_norm + concat_and_cache_mla", lambda: ops.concat_and_cache_mla(
                ops.rms_norm(c512, kn, 1e-6), krot[:, 0], lat, slots), 4.0 * T * (K + R), 0))
        ql = a[:, :QR].unflatten(1, (H, 192))
        row(f"latent_rope in place, {phase}", lambda: ops.latent_rope(ql[..., D:], ql[..., D:], ang, R, 0, interleaved=True), 4.0 * T * H * R, 0,
            ("rotary_embedding", lambda: ops.rotary_embedding(pos, qa, ka, D, csn, True), 4.0 * T * (H + G) * D, 0))
        # -- boundary
        x, gain, coef = rn(T, S, W, dt=f32), rn(W, dt=f32), torch.rand(S * (S + 2), device=dev) / S
        table, ids = rn(32768, W), torch.randint(0, 32768, (T,), device=dev)
        e = Embedded(table, ids, 32768, 8.0, S)
        norm_like = ("fused_add_rms_norm", lambda: ops.fused_add_rms_norm(y, res, nw, 1e-6), 8.0 * T * W, 0)
        row(f"stream_norm, {S} streams, {phase}", lambda: stream_norm(y, x, coef, gain, 1e-6), T * W * (8.0 * S + 4), 0, norm_like)
        row(f"stream_norm behind the last sublayer, {phase}", lambda: stream_norm(y, x, coef, gain, 1e-6, want_x=False),
            T * W * (4.0 * S + 4), 0, norm_like)
        row(f"stream_norm behind the first sublayer, {phase}", lambda: stream_norm(y, e, coef, gain, 1e-6), T * W * (4.0 * S + 6), 0, norm_like)
        row(f"stream_norm of embeddings, {phase}", lambda: stream_norm(None, e, coef, gain, 1e-6), 4.0 * T * W, 0,
            ("embedding", lambda: ops.embedding(table, ids), 4.0 * T * W, 0))
        x3, c3 = rn(T, 3, W, dt=f32), torch.rand(15, device=dev)
        row(f"stream_norm, 3 streams, {phase}", lambda: stream_norm(y, x3, c3, gain, 1e-6), T * W * 28.0, 0, norm_like)
        if S <= 4:                         # DeepSeek-V4's boundary, whose weights are computed per token
            xb, fn = rn(T, S, W), rn(2 * S + S * S, S * W, dt=f32)
            post, comb, sc, ba = torch.rand(T, S, device=dev), torch.rand(T, S, S, device=dev), torch.ones(3, device=dev), rn(2 * S + S * S, dt=f32)
            row(f"stream_norm, {S} streams, against mhc, {phase}", lambda: stream_norm(y, x, coef, gain, 1e-6), T * W * (8.0 * S + 4), 0,
                ("mhc_fused_post_pre (bf16 streams)",
                 lambda: mhc_fused_post_pre(y, xb, post, comb, fn, sc, ba, 1e-6, 1e-6, 1e-6, 2.0, 20), T * W * (4.0 * S + 4), 0))
        # -- products
        up, proj, pb = rn(s["dense"], W), rn((H + 2 * G) * D + H, W), rn((H + 2 * G) * D + H)
        by = 2.0 * (T * W + up.numel() + T * s["dense"])
        row(f"up product + squared relu, {phase}", lambda: ops.gemm(y, up, act="relu2"), by, 2.0 * T * up.numel(),
            ("gemm_silu_mul", lambda: ops.gemm_silu_mul(y, up), by - T * s["dense"], 2.0 * T * up.numel()))
        row(f"up product, squared relu or not, {phase}", lambda: ops.gemm(y, up, act="relu2"), by, 2.0 * T * up.numel(),
            ("without an activation", lambda: ops.gemm(y, up), by, 2.0 * T * up.numel()))
        by = 2.0 * (T * W + proj.numel() + T * proj.shape[0])
        row(f"q, k, v, gate product with biases, {phase}", lambda: ops.gemm(y, proj, pb), by, 2.0 * T * proj.numel(),
            ("without", lambda: ops.gemm(y, proj), by, 2.0 * T * proj.numel()))
        if decode:
            row(f"logits (fp32 out), {phase}", lambda: ops.gemm(y, table, out_dtype=f32),
                2.0 * (T * W + table.numel()) + 4.0 * T * 32768, 2.0 * T * table.numel(),
                ("bf16 out", lambda: ops.gemm(y, table), 2.0 * (T * W + table.numel() + T * 32768), 2.0 * T * table.numel()))
    ops.check_kernel_status(0)
    return rows
