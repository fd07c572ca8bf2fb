"""The GQA attention layer: fused RoPE + KV-cache write, then the split forward
(decode slice -> split-KV decode kernel, prefill slice -> tcgen05 varlen kernel).

One backend (``PAGED_GQA``) replaces the reference's FLASH_ATTN / TRITON_ATTN /
FLASHINFER family for decoder self-attention: bf16/fp16 caches, fp8 caches with a
static scale, and int8 / fp8 caches with per-(token, head) scales
(``int8_per_token_head``) all run through the same two kernels.  The split of a
mixed batch into a decode slice and a prefill slice follows
vllm_metax/v1/attention/backends/flash_attn.py:1302-1355 (VLLM_METAX_ENABLE_FA_SPLIT_FORWARD).
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from ..attention.metadata import get_forward_context
from ..ops import turboquant as tq
from .recurrent import StackedLinear, _param
from .rotation import Rotation

KV_DTYPES = {
    "auto": None, "bfloat16": torch.bfloat16, "float16": torch.float16, "fp8": torch.float8_e4m3fn,
    "fp8_e4m3": torch.float8_e4m3fn, "int8_per_token_head": torch.int8, "fp8_per_token_head": torch.float8_e4m3fn,
}


class PagedGQABackend:
    name = "PAGED_GQA"
    supported_head_sizes = (64, 128, 256)      # 8-bit caches; 16-bit ones take every multiple of 8 up to 256
    supported_kv_cache_dtypes = tuple(KV_DTYPES)

    @staticmethod
    def get_kv_cache_shape(num_blocks: int, block_size: int, num_kv_heads: int, head_size: int):
        return (num_blocks, 2, block_size, num_kv_heads, head_size)

    @staticmethod
    def get_scale_shape(num_blocks: int, block_size: int, num_kv_heads: int):
        return (num_blocks, 2, block_size, num_kv_heads)

    @staticmethod
    def supported_block_sizes():
        return (16, 32, 64, 128, 256)

    @staticmethod
    def allocate_pages(num_blocks, block_size, num_kv_heads, head_size, v_head_size, dtype, device):
        """Cache of a layer whose keys and values may differ in size: the usual 5-D tensor where they do not, otherwise one
        row per page, ``[K of the page's tokens | V of them]``."""
        if head_size == v_head_size:
            shape = PagedGQABackend.get_kv_cache_shape(num_blocks, block_size, num_kv_heads, head_size)
        else:
            shape = (num_blocks, block_size * num_kv_heads * (head_size + v_head_size))
        return torch.zeros(shape, dtype=dtype, device=device)

    @staticmethod
    def views(cache: torch.Tensor, block_size: int, num_kv_heads: int, head_size: int, v_head_size: int):
        """``(K, V)`` views ``[num_blocks, block_size, num_kv_heads, size]`` of what ``allocate_pages`` returned."""
        if cache.dim() == 5:
            return cache[:, 0], cache[:, 1]
        n = block_size * num_kv_heads
        shape = (cache.shape[0], block_size, num_kv_heads)
        return (cache[:, : n * head_size].view(*shape, head_size), cache[:, n * head_size:].view(*shape, v_head_size))

    @staticmethod
    def allocate(num_blocks, block_size, num_kv_heads, head_size, model_dtype, kv_cache_dtype: str, device):
        if tq.is_turboquant(kv_cache_dtype):
            # combined K+V slots; the second element carries the format instead of a scale tensor
            assert head_size == tq.D, "TurboQuant caches are built for head_dim 128"
            fmt = tq.TqFormat.from_name(kv_cache_dtype)
            return (tq.alloc_cache(num_blocks, block_size, num_kv_heads, fmt, device), fmt)
        dt = KV_DTYPES[kv_cache_dtype] or model_dtype
        cache = torch.zeros(PagedGQABackend.get_kv_cache_shape(num_blocks, block_size, num_kv_heads, head_size),
                            dtype=dt, device=device)
        scales = None
        if kv_cache_dtype.endswith("per_token_head"):
            scales = torch.ones(PagedGQABackend.get_scale_shape(num_blocks, block_size, num_kv_heads),
                                dtype=torch.float32, device=device)
        return (cache, scales)


class Attention(nn.Module):
    def __init__(self, num_heads: int, head_size: int, scale: float, num_kv_heads: int, layer_idx: int,
                 sliding_window: Optional[int] = None, softcap: float = 0.0, sinks: Optional[torch.Tensor] = None,
                 k_scale: float = 1.0, v_scale: float = 1.0, alibi_slopes: Optional[torch.Tensor] = None):
        super().__init__()
        self.alibi_slopes = alibi_slopes           # f32 [num_heads] (Bloom / MPT / Baichuan-13B style position bias)
        self.num_heads, self.head_size, self.scale, self.num_kv_heads = num_heads, head_size, scale, num_kv_heads
        self.layer_idx = layer_idx
        self.window = sliding_window or -1
        self.softcap = softcap
        self.sinks = sinks
        self.k_scale, self.v_scale = k_scale, v_scale
        self.distance_bias: Optional[torch.Tensor] = None      # f32 [num_heads, L]: bias by distance, the last entry from L - 1 on
        self.bias_tiles: Optional[torch.Tensor] = None         # the same for the prompt kernel (ops.distance_bias_tiles)
        self.out_scale = 1.0
        self.chunk = 0                                         # a position sees its own chunk of this many (0: no chunks)
        self.sigmoid_shift: Optional[torch.Tensor] = None      # f32 [num_heads]: weights are sigmoid(score + shift), no softmax

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, positions: Optional[torch.Tensor] = None,
                rope=None) -> torch.Tensor:
        """``q [T, Hq*D]``, ``k, v [T, Hkv*D]`` (views into the qkv GEMM output are fine).
        With ``rope`` given, RoPE is applied inside the cache-write kernel."""
        ctx = get_forward_context()
        md = ctx.attn_metadata
        kv_cache, kv_scales = ctx.kv_caches[self.layer_idx]
        T = q.shape[0]
        if isinstance(kv_scales, tq.TqFormat):
            return self._forward_turboquant(q, k, v, positions, rope, md, kv_cache, kv_scales)
        if "dcp_ctx_lens" in md.extra:
            return self._forward_dcp(q, k, v, positions, rope, md, kv_cache, kv_scales)
        pcp_slots = md.extra.get("pcp_slots_all")
        if pcp_slots is not None:
            # prefill context parallel: this copy computed a slice of every chunk; the copies exchange their K / V
            # rows and each writes all of them into its own (replicated) cache - parallel/pcp.py
            from ..parallel import state as ps

            if rope is not None:
                ops.rotary_embedding(positions, q, k, self.head_size, rope.cos_sin_cache, rope.is_neox)
            g, sizes = ps.get_pcp_group(), md.extra["pcp_sizes"]
            k_all, v_all = g.all_gatherv(k.contiguous(), sizes), g.all_gatherv(v.contiguous(), sizes)
            ops.reshape_and_cache(k_all, v_all, kv_cache, pcp_slots, kv_scales, self.k_scale, self.v_scale)
        elif rope is not None:
            ops.rope_and_cache(positions, q, k, v, self.head_size, rope.cos_sin_cache, rope.is_neox, kv_cache,
                               md.slot_mapping, kv_scales, self.k_scale, self.v_scale)
        else:
            ops.reshape_and_cache(k, v, kv_cache, md.slot_mapping, kv_scales, self.k_scale, self.v_scale)
        q3 = q.reshape(T, self.num_heads, self.head_size)
        if not q3.is_contiguous() and q3.stride(1) != self.head_size:
            q3 = q3.contiguous()
        if "cascade_blocks" in md.extra and self.window == -1 and self.alibi_slopes is None and self.sinks is None:
            return self._forward_cascade(q3, md, kv_cache, kv_scales)
        return self.attend(q3, md, kv_cache, kv_scales).reshape(T, self.num_heads * self.head_size)

    def attend(self, q3: torch.Tensor, md, kv_cache, kv_scales=None, out=None, gate=None) -> torch.Tensor:
        """``q3 [T, heads, D]`` over the cache, which already holds this step's keys and values (written by this layer or by the
        one whose cache it reads): decode rows, then prompt portions.  ``kv_cache``: 5-D or a pair of views.  ``out`` and
        ``gate``: as in ``ops.paged_attention_decode``."""
        if out is None:
            v_size = kv_cache[1].shape[-1] if isinstance(kv_cache, tuple) else self.head_size
            out = torch.empty(q3.shape[0], self.num_heads, v_size, dtype=q3.dtype, device=q3.device)
        nd, ndt = md.num_decodes, md.num_decode_tokens
        gates = (None, None) if gate is None else (gate[:ndt], gate[ndt:])
        if nd > 0:
            ops.paged_attention_decode(q3[:ndt], kv_cache, md.block_table[:nd], md.seq_lens[:nd], self.scale,
                                       out=out[:ndt], kv_scales=kv_scales, window=self.window, softcap=self.softcap,
                                       sinks=self.sinks, num_splits=md.decode_num_splits, max_seq_len=md.max_seq_len,
                                       k_scale=self.k_scale, v_scale=self.v_scale, workspace=md.decode_workspace,
                                       alibi_slopes=self.alibi_slopes, distance_bias=self.distance_bias, gate=gates[0],
                                       out_scale=self.out_scale, chunk=self.chunk, sigmoid_shift=self.sigmoid_shift)
        if md.num_prefills > 0:
            ops.paged_attention_prefill(q3[ndt:], kv_cache, md.block_table[nd:], md.seq_lens[nd:],
                                        md.prefill_query_start_loc, self.scale, out=out[ndt:], kv_scales=kv_scales,
                                        max_q_len=md.max_prefill_query_len, window=self.window, softcap=self.softcap,
                                        sinks=self.sinks, k_scale=self.k_scale, v_scale=self.v_scale,
                                        max_seq_len=md.max_seq_len, alibi_slopes=self.alibi_slopes,
                                        distance_bias=self.distance_bias, bias_tiles=self.bias_tiles, gate=gates[1],
                                        out_scale=self.out_scale, chunk=self.chunk, sigmoid_shift=self.sigmoid_shift)
        return out

    def _forward_cascade(self, q3, md, kv_cache, kv_scales) -> torch.Tensor:
        """Shared-prefix (cascade) attention: the leading ``cascade_blocks`` cache blocks are the same physical blocks
        for every request of the step, so all of the step's query tokens attend them in ONE pass (one pseudo request,
        no causal mask: the prefix precedes every query), every request attends the rest of its own context, and the
        two partial results are merged by their log-sum-exps.  The prefix is read once per step instead of once per
        request.  Mirrors the cascade path of vllm_metax/v1/attention/backends/flash_attn.py (``use_cascade_attention``
        / ``cascade_attention``: prefix pass + suffix pass + ``merge_attn_states``)."""
        T, H, D = q3.shape
        dev = q3.device
        n = md.extra["cascade_blocks"]
        nd, ndt = md.num_decodes, md.num_decode_tokens
        common = dict(kv_scales=kv_scales, softcap=self.softcap, k_scale=self.k_scale, v_scale=self.v_scale)
        o_p = torch.empty(T, H, D, dtype=q3.dtype, device=dev)
        lse_p = torch.empty(H, T, dtype=torch.float32, device=dev)
        ops.paged_attention_prefill(q3, kv_cache, md.block_table[:1, :n].contiguous(), md.extra["cascade_seq_len"],
                                    md.extra["cascade_qsl"], self.scale, out=o_p, lse_out=lse_p, max_q_len=T,
                                    causal=False, max_seq_len=n * md.block_size, **common)
        table, lens = md.extra["cascade_suffix_table"], md.extra["cascade_suffix_lens"]
        o_s = torch.empty(T, H, D, dtype=q3.dtype, device=dev)
        parts = []
        if nd > 0:
            lse_d = torch.empty(H, ndt, dtype=torch.float32, device=dev)
            ops.paged_attention_decode(q3[:ndt], kv_cache, table[:nd], lens[:nd], self.scale, out=o_s[:ndt],
                                       lse_out=lse_d, max_seq_len=md.max_seq_len, **common)
            parts.append(lse_d)
        if md.num_prefills > 0:
            lse_f = torch.empty(H, T - ndt, dtype=torch.float32, device=dev)
            ops.paged_attention_prefill(q3[ndt:], kv_cache, table[nd:], lens[nd:], md.prefill_query_start_loc, self.scale,
                                        out=o_s[ndt:], lse_out=lse_f, max_q_len=md.max_prefill_query_len,
                                        max_seq_len=md.max_seq_len, **common)
            parts.append(lse_f)
        lse_s = parts[0] if len(parts) == 1 else torch.cat(parts, dim=1)
        out = ops.merge_attn_states(o_p, lse_p, o_s, lse_s.contiguous())
        return out.reshape(T, H * D)

    def _forward_dcp(self, q, k, v, positions, rope, md, kv_cache, kv_scales) -> torch.Tensor:
        """Decode context parallel: this rank's cache holds every dcp-th token of each sequence (the slot mapping is
        -1 for the others).  Decode rows: all-gather q over the group's heads, attend the local shard, combine the
        partial outputs by their log-sum-exp and keep this rank's heads.  Prefill rows: causal attention over the
        chunk's own fresh K / V (every rank has them - its KV heads are replicated over the group) merged with the
        same gather / local / combine pass over the cached context, which needs no mask because all of it precedes
        the chunk.  Mirrors vllm_metax/v1/attention/backends/flash_attn.py:1450-1610."""
        from ..parallel import dcp
        from ..parallel import state as ps

        g = ps.get_dcp_group()
        d = g.world_size
        T, H, D = q.shape[0], self.num_heads, self.head_size
        if rope is not None:
            ops.rope_and_cache(positions, q, k, v, D, rope.cos_sin_cache, rope.is_neox, kv_cache, md.slot_mapping,
                               kv_scales, self.k_scale, self.v_scale)
        else:
            ops.reshape_and_cache(k, v, kv_cache, md.slot_mapping, kv_scales, self.k_scale, self.v_scale)
        q3 = q.reshape(T, H, D)
        out = torch.empty(T, H, D, dtype=q.dtype, device=q.device)
        nd, ndt = md.num_decodes, md.num_decode_tokens
        common = dict(kv_scales=kv_scales, window=self.window, softcap=self.softcap, k_scale=self.k_scale,
                      v_scale=self.v_scale, alibi_slopes=None)
        assert self.alibi_slopes is None and self.sinks is None, "ALiBi / sinks are not combined with DCP"

        def masked(o, lse, empty_rows):           # rows whose local shard is empty contribute nothing
            lse = torch.where(empty_rows[None, :], torch.full_like(lse, float("-inf")), lse)
            return torch.where(empty_rows[:, None, None], torch.zeros_like(o), o), lse.t().contiguous()

        if nd > 0:
            lens = md.seq_lens[:nd]

            def attend_decode(q_all):
                o = torch.empty(ndt, H * d, D, dtype=q.dtype, device=q.device)
                lse = torch.empty(H * d, ndt, dtype=torch.float32, device=q.device)
                ops.paged_attention_decode(q_all, kv_cache, md.block_table[:nd], lens.clamp_min(1), self.scale, out=o,
                                           lse_out=lse, num_splits=md.decode_num_splits, max_seq_len=md.max_seq_len,
                                           workspace=md.decode_workspace, **common)
                return masked(o, lse, lens == 0)

            out[:ndt] = dcp.decode_attention(q3[:ndt].contiguous(), attend_decode, g)
        if md.num_prefills > 0:
            Tp = T - ndt
            cu = md.prefill_query_start_loc
            Hkv = self.num_kv_heads
            qp = q3[ndt:].contiguous()
            kp = k[ndt:].reshape(Tp, Hkv, D).contiguous()
            vp = v[ndt:].reshape(Tp, Hkv, D).contiguous()
            o_self = torch.empty(Tp, H, D, dtype=q.dtype, device=q.device)
            lse_self = torch.empty(H, Tp, dtype=torch.float32, device=q.device)
            ops.varlen_attention(qp, kp, vp, cu, cu, self.scale, out=o_self, max_q_len=md.max_prefill_query_len,
                                 causal=True, window=self.window, softcap=self.softcap, lse_out=lse_self)
            if md.extra["dcp_any_context"]:
                ctx = md.extra["dcp_ctx_lens"][nd:]
                qlens = (cu[1:] - cu[:-1]).long()
                empty_tok = torch.repeat_interleave(ctx == 0, qlens, output_size=Tp)

                def attend_context(q_all):
                    o = torch.empty(Tp, H * d, D, dtype=q.dtype, device=q.device)
                    lse = torch.empty(H * d, Tp, dtype=torch.float32, device=q.device)
                    ops.paged_attention_prefill(q_all, kv_cache, md.block_table[nd:], ctx.clamp_min(1), cu, self.scale,
                                                out=o, lse_out=lse, max_q_len=md.max_prefill_query_len, causal=False,
                                                max_seq_len=md.max_seq_len, **{k_: v_ for k_, v_ in common.items()
                                                                               if k_ != "window"})
                    return masked(o, lse, empty_tok)

                o_ctx, lse_ctx = dcp.decode_attention(qp, attend_context, g, return_lse=True)
                out[ndt:] = ops.merge_attn_states(o_ctx, lse_ctx.t().contiguous(), o_self, lse_self)
            else:
                out[ndt:] = o_self
        return out.reshape(T, H * D)

    def _forward_turboquant(self, q, k, v, positions, rope, md, cache, fmt) -> torch.Tensor:
        """TurboQuant cache: RoPE, quantising store, then decode rows straight from the compressed slots and prefill
        rows against the de-quantised context (the cache is the only source of K / V, so a chunk sees its own keys
        through the same quantiser as every later step will).  Mirrors the split of
        vllm_metax/v1/attention/backends/turboquant_attn.py:286-942."""
        T = q.shape[0]
        if rope is not None:
            ops.rotary_embedding(positions, q, k, self.head_size, rope.cos_sin_cache, rope.is_neox)
        tq.store(k, v, cache, md.slot_mapping[:T], fmt)
        q3 = q.reshape(T, self.num_heads, self.head_size)
        if not q3.is_contiguous():
            q3 = q3.contiguous()
        out = torch.empty(T, self.num_heads, self.head_size, dtype=q.dtype, device=q.device)
        nd, ndt = md.num_decodes, md.num_decode_tokens
        if nd > 0 and ndt == nd:
            tq.decode_attention(q3[:nd], cache, md.block_table[:nd], md.seq_lens[:nd], self.scale, fmt, out=out[:nd])
            first = nd
        else:
            first = 0                   # multi-token decode rows (speculative drafts) take the prefill route
        if first < md.num_reqs:
            bs = cache.shape[1]
            lens = md.seq_lens[first: md.num_reqs].cpu()
            qsl = md.query_start_loc[first: md.num_reqs + 1]
            t0 = 0 if first == 0 else ndt
            slots = torch.cat([tq._slots_of(md.block_table[first + i], int(L), bs) for i, L in enumerate(lens.tolist())])
            kd, vd = tq.dequant(cache, slots, fmt, q.dtype)
            cu_k = torch.zeros(lens.numel() + 1, dtype=torch.int32)
            cu_k[1:] = lens.cumsum(0)
            cu_q = (qsl - qsl[0]).int()
            ops.varlen_attention(q3[t0:], kd, vd, cu_q, cu_k.to(q.device), self.scale, out=out[t0:],
                                 max_q_len=md.max_query_len, causal=True, window=self.window, softcap=self.softcap,
                                 sinks=self.sinks)
        return out.reshape(T, self.num_heads * self.head_size)


class QKNormAttention(nn.Module):
    """Grouped-query attention, by default with RMS-normed queries and keys, with key and value sizes of its own, an optional
    sliding window or chunks, and optionally the keys and values of another layer (``kv_from``: that layer's module, which must come earlier in the step)
    instead of projections and a cache of its own.

        merged q | k | v product -> ``head_norm_rope`` (norms, rotation, cache write) -> paged attention -> output product

    ``norm``: "weighted", "unit" (without weights) or "none"; ``whole_row_norm``: one norm over all heads.  ``inv_freq=None``: no
    rotation; ``interleaved``: pairs (2i, 2i + 1).  ``q_temp = (coef, every)``: queries grow with the position; ``head_temp``:
    scores are multiplied by a learned number per head.  ``bias_far`` and ``bias_rows``: a learned bias by distance, one row per
    bucket (``distance_buckets``).  ``alibi_slopes``: a fixed slope per head.  ``log_bias``: ``r1 ln(1 + r2 distance)`` with
    two learned numbers per head is taken off (the keys must be near: a window or chunks).  ``sigmoid``: weights are the sigmoid
    of the score plus a learned number per head, without a softmax.  ``gated``: the heads' outputs times the sigmoid of another
    projection, an entry each, or ("head") one number per head.

    Head sizes are padded to multiples of 8 with zero rows of the projections (and zero columns of the output product).
    ``standalone=False``: a branch of a :class:`layers.mixer.ProjectedMixer`, which owns the products.  ``runs``: how often a
    step passes through the layer; every pass has a cache of its own, from ``cache_idx`` on."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float,
                 inv_freq: Optional[torch.Tensor], cache_idx: int, window: Optional[int] = None,
                 kv_from: Optional["QKNormAttention"] = None, dtype=torch.bfloat16, *, standalone: bool = True, runs: int = 1,
                 whole_row_norm: bool = False, interleaved: bool = False, q_temp: Optional[tuple] = None, softcap: float = 0.0,
                 sinks: bool = False, bias_rows: int = 0, bias_far: int = 0, gated=False, proj_bias: bool = False,
                 out_scale: float = 1.0, norm: str = "weighted", chunk: int = 0, head_temp: bool = False,
                 alibi_slopes: Optional[list] = None, log_bias: bool = False, sigmoid: bool = False):
        super().__init__()
        if norm not in ("weighted", "unit", "none") or (whole_row_norm and norm != "weighted"):
            raise ValueError(f"norm {norm!r}" + (" over whole rows" if whole_row_norm else ""))
        if sigmoid and sinks:
            raise ValueError("a sink belongs to a softmax")
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads over {kv_heads} key / value heads")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim, self.eps = width, heads, kv_heads, dim, vdim, eps
        self.dim_pad, self.vdim_pad = -(-dim // 8) * 8, -(-vdim // 8) * 8
        self.own_kv = kv_from is None
        if kv_from is not None and (kv_from.kv_heads, kv_from.dim, kv_from.vdim) != (kv_heads, dim, vdim):
            raise ValueError("a layer that reads another layer's keys and values has its key / value heads and sizes")
        self.runs, self.whole_row_norm, self.interleaved, self.q_temp = runs, whole_row_norm, interleaved, q_temp
        self.proj_bias, self.gated = proj_bias, gated
        self.out_width = heads * self.vdim_pad
        rows = (heads, kv_heads) if whole_row_norm else (1, 1)
        self.norm, self.dtype = norm, dtype
        self.q_norm = _param(rows[0] * self.dim_pad, dtype=dtype) if norm == "weighted" else None
        self.k_norm = _param(rows[1] * self.dim_pad, dtype=dtype) if norm == "weighted" and self.own_kv else None
        self.rotation = Rotation(inv_freq) if inv_freq is not None else None
        self.head_temp = _param(heads, dtype=torch.float32) if head_temp else None
        self.attn = Attention(heads, self.dim_pad, scale, kv_heads, cache_idx, sliding_window=window, softcap=softcap)
        self.attn.out_scale, self.attn.chunk = out_scale, chunk
        if alibi_slopes is not None:
            self.register_buffer("slopes", torch.tensor(alibi_slopes, dtype=torch.float32), persistent=False)
            self.attn.alibi_slopes = self.slopes
        self.shift = _param(heads, dtype=torch.float32) if sigmoid else None
        self.attn.sigmoid_shift = self.shift
        self.sinks = _param(heads, dtype=torch.float32) if sinks else None
        self.attn.sinks = self.sinks
        self.rel = self.log_bias = None
        reach = 0                                  # distances of the bias table
        if bias_rows:
            self.buckets = distance_buckets(bias_rows, bias_far)
            self.rel, reach = _param(bias_rows, heads, dtype=dtype), len(self.buckets)
        elif log_bias:
            reach = min((n for n in (window, chunk) if n), default=0)
            if not reach:
                raise ValueError("a logarithmic distance bias needs a window or chunks")
            self.log_bias = _param(2, heads, dtype=torch.float32)
        if reach:
            self.register_buffer("distance_bias", torch.zeros(heads, reach, dtype=torch.float32), persistent=False)
            self.attn.distance_bias = self.distance_bias
            self.register_buffer("bias_tiles", ops.distance_bias_tiles(self.distance_bias, heads // kv_heads), persistent=False)
            self.attn.bias_tiles = self.bias_tiles
        if standalone:
            self.proj = StackedLinear(width, self.in_parts(), ("q", "k", "v") if proj_bias else (), dtype=dtype)
            self.attach(self.proj)
            self.out_proj = _param(width, self.out_width, dtype=dtype)

    # ---- the products around it -----------------------------------------------------------------------------------
    def in_parts(self) -> dict:
        parts = {"q": self.heads * self.dim_pad}
        if self.own_kv:
            parts.update(k=self.kv_heads * self.dim_pad, v=self.kv_heads * self.vdim_pad)
        if self.gated:
            parts["g"] = self.gate_width
        return parts

    @property
    def gate_width(self) -> int:
        return self.heads if self.gated == "head" else self.out_width

    def attach(self, proj: StackedLinear, prefix: str = "") -> None:
        """The product that yields q, k, v (and g) as its parts ``prefix + name``."""
        self.prefix = prefix
        self.offsets = tuple(proj.offsets.get(prefix + n, 0) for n in ("q", "k", "v"))
        self.gate_offset = proj.offsets.get(prefix + "g", 0)

    def finalize_weights(self) -> None:
        if self.rel is not None:
            self.distance_bias.copy_(self.rel.data.float()[self.buckets].t())
        if self.log_bias is not None:
            r1, r2 = self.log_bias.data.double()[..., None]
            far = torch.arange(self.distance_bias.shape[1], dtype=torch.float64, device=r1.device)
            self.distance_bias.copy_(-r1 * torch.log1p(r2 * far))
        if self.attn.distance_bias is not None:
            self.bias_tiles.copy_(ops.distance_bias_tiles(self.distance_bias, self.heads // self.kv_heads))

    def in_slots(self, proj: StackedLinear) -> dict:
        """Tensor name -> (memory it is copied to, its shape in a checkpoint), without the output product."""
        def heads(name, n, size, pad):
            return proj.rows(self.prefix + name).view(n, pad, self.width)[:, :size], (n * size, self.width)

        def bias(name, n, size, pad):
            return proj.bias_rows(self.prefix + name).view(n, pad)[:, :size], (n * size,)

        def norm(w, n):
            return (w.data.view(n, self.dim_pad)[:, : self.dim], (n * self.dim,)) if self.whole_row_norm else w.data[: self.dim]

        sizes = {"q": (self.heads, self.dim, self.dim_pad)}
        out = {"q.norm": norm(self.q_norm, self.heads)} if self.q_norm is not None else {}
        if self.own_kv:
            sizes.update(k=(self.kv_heads, self.dim, self.dim_pad), v=(self.kv_heads, self.vdim, self.vdim_pad))
        if self.k_norm is not None:
            out["k.norm"] = norm(self.k_norm, self.kv_heads)
        for name, s in sizes.items():
            out[name] = heads(name, *s)
            if self.proj_bias:
                out[name + ".b"] = bias(name, *s)
        if self.gated:
            out["g"] = proj.rows(self.prefix + "g") if self.gated == "head" else heads("g", self.heads, self.vdim, self.vdim_pad)
        if self.sinks is not None:
            out["sink"] = self.sinks.data
        if self.rel is not None:
            out["rel"] = self.rel.data
        if self.log_bias is not None:
            out["r1"], out["r2"] = self.log_bias.data
        if self.head_temp is not None:
            out["temp"] = self.head_temp.data
        if self.shift is not None:
            out["pb"] = self.shift.data
        return out

    def out_slot(self, weight: torch.Tensor) -> tuple:
        """The same for the output product, whose columns for this layer are ``weight [width, out_width]``."""
        return (weight.unflatten(1, (self.heads, self.vdim_pad))[..., : self.vdim], (self.width, self.heads * self.vdim))

    def slots(self) -> dict:
        return {**self.in_slots(self.proj), "o": self.out_slot(self.out_proj.data)}

    # ---- cache ------------------------------------------------------------------------------------------------------
    def decode_workspace_floats(self, batch: int, max_seq_len: int) -> int:
        """What the split decode of ``batch`` rows needs for its partial results (0: it does not split)."""
        tiles = -(-(self.heads // self.kv_heads) // 16)
        n = ops.decode_num_splits(batch, self.kv_heads, max_seq_len, tiles, window=self.attn.window, chunk=self.attn.chunk)
        return n * batch * self.heads * (self.vdim_pad + 1) if n > 1 else 0

    def cache_elems_per_token(self) -> int:
        return self.runs * self.kv_heads * (self.dim_pad + self.vdim_pad) if self.own_kv else 0

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device):
        return (PagedGQABackend.allocate_pages(num_blocks, block_size, self.kv_heads, self.dim_pad, self.vdim_pad,
                                               self.dtype, device), None)

    # ---- forward ----------------------------------------------------------------------------------------------------
    def mix(self, positions: torch.Tensor, h: torch.Tensor, p: torch.Tensor, out: torch.Tensor, run: int = 0) -> None:
        """From the input product's rows ``p`` to the output product's operand ``out [T, out_width]``."""
        ctx = get_forward_context()
        md = ctx.attn_metadata
        T = p.shape[0]
        cache = ctx.kv_caches[self.attn.layer_idx + run][0]
        kv = PagedGQABackend.views(cache, md.block_size, self.kv_heads, self.dim_pad, self.vdim_pad)
        angles = self.rotation.angles(positions, T) if self.rotation is not None else None
        q = ops.head_norm_rope(p, self.offsets, self.q_norm, self.k_norm, self.heads, self.dim, angles,
                               kv if self.own_kv else None, md.slot_mapping, self.eps, whole_row=self.whole_row_norm,
                               interleaved=self.interleaved, q_temp=(positions, *self.q_temp) if self.q_temp else None,
                               q_scale=self.head_temp, normed=self.norm != "none", width=self.dim_pad)
        gate = None
        if self.gated:
            gate = p[:, self.gate_offset: self.gate_offset + self.gate_width]
        self.attn.attend(q, md, kv, out=out.unflatten(1, (self.heads, self.vdim_pad)), gate=gate)

    def forward(self, positions: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        o = torch.empty(h.shape[0], self.out_width, dtype=h.dtype, device=h.device)
        self.mix(positions, h, self.proj(h), o)
        return ops.gemm(o, self.out_proj)


def distance_buckets(rows: int, far: int) -> list:
    """Row of a learned distance bias for every distance 0, 1, ... up to the first that has the last row, which all larger ones
    share: ``rows / 2`` rows for single distances, the others on a logarithmic scale that ends at ``far``."""
    half = rows // 2
    if half < 1 or far <= half:
        raise ValueError(f"a distance bias of {rows} rows up to distance {far}")
    out = list(range(half))
    while out[-1] != rows - 1:
        n = len(out)
        x = math.log(n / half) / math.log(far / half) * (rows - half)
        whole = round(x)                               # a quotient of logarithms that is a whole number, up to rounding
        out.append(min(rows - 1, half + (whole if abs(x - whole) < 1e-9 else math.floor(x))))
    return out
