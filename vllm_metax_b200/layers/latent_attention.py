"""Multi-head latent attention of any sizes with a sliding window (``layers/mla.py`` is the 512 + 64 DeepSeek form with its
sparse and distributed variants; both run the same attention kernels).

Cache: one row per token and layer, ``[latent kv_rank | rotated key part rot_dim | zeros to a multiple of 8]``, paged like
every KV cache; the rotated part is shared by the heads.

    down      one product for both latents (or the queries themselves and the key latent) -> ``latent_insert``: norms, rotation of
              the key part, cache write
    decode    absorbed form: q . W_UK per head (batched product), attention over the cached rows (``mla_decode``), . W_UV
    prompts   the cached rows a portion can see (its own tokens and up to window - 1 before it) are gathered and multiplied
              with ONE matrix that yields, head by head, [unrotated key | rotated key | value] - the rotated columns are an
              identity block over the gathered rotated part - and the tcgen05 varlen kernel runs on that.  Portions that
              are short next to the context they see, fp32, and sizes the varlen kernel does not take use the decode path.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import _custom_ops as ops
from ..attention.metadata import get_forward_context
from ..ops.reference import rope_frequencies
from .recurrent import StackedLinear, _param
from .rotation import Rotation

# A portion takes the up-projected path unless the context rows to up-project outnumber its tokens by more than this.
CONTEXT_PER_TOKEN = 4


class LatentCache:
    name = "LATENT"

    @staticmethod
    def row_elems(kv_rank: int, rot_dim: int) -> int:
        return -(-(kv_rank + rot_dim) // 8) * 8

    @staticmethod
    def allocate(num_blocks: int, block_size: int, kv_rank: int, rot_dim: int, dtype, device) -> torch.Tensor:
        return torch.zeros(num_blocks, block_size, LatentCache.row_elems(kv_rank, rot_dim), dtype=dtype, device=device)


def prompt_spans(md, window: int):
    """``(cu_rows [n + 1], first position [n], total rows)`` of the cache rows this step's prompt portions can see; computed
    once per step and window (models may mix windows)."""
    key = ("prompt_spans", window)
    hit = md.extra.get(key)
    if hit is None:
        nd = md.num_decodes
        lens = md.seq_lens_cpu if md.seq_lens_cpu is not None else md.seq_lens.cpu()
        qsl = md.query_start_loc_cpu if md.query_start_loc_cpu is not None else md.query_start_loc.cpu()
        lens, q = lens[nd: md.num_reqs].long(), (qsl[nd + 1: md.num_reqs + 1] - qsl[nd: md.num_reqs]).long()
        first = (lens - q - (window - 1)).clamp_min(0) if window > 0 else torch.zeros_like(lens)
        cu = torch.zeros(lens.numel() + 1, dtype=torch.int32)
        cu[1:] = (lens - first).cumsum(0)
        dev = md.seq_lens.device
        hit = md.extra[key] = (cu.to(dev, non_blocking=True), first.to(torch.int32).to(dev, non_blocking=True), int(cu[-1]))
    return hit


class LatentAttention(nn.Module):
    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: Optional[int], kv_rank: int,
                 scale: float, window: int, rot_base: float, rot_dims: int, eps: float, cache_idx: int, dtype=torch.bfloat16,
                 interleaved: bool = False):
        """``q_rank=None``: queries straight from the input.  ``window`` 0: none.  ``interleaved``: rotation in pairs (2i, 2i + 1)
        instead of (i, i + half)."""
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim = heads, dim, rot_dim, vdim
        self.q_rank, self.kv_rank, self.scale, self.window, self.eps = q_rank, kv_rank, scale, window, eps
        self.cache_idx, self.dtype = cache_idx, dtype
        self.row = LatentCache.row_elems(kv_rank, rot_dim)
        self.interleaved, q_rows = interleaved, heads * (dim + rot_dim)
        self.down = StackedLinear(width, {"dq" if q_rank else "q": q_rank or q_rows, "dkv": kv_rank + rot_dim}, dtype=dtype)
        self.q_norm = _param(q_rank, dtype=dtype) if q_rank else None
        self.kv_norm = _param(kv_rank, dtype=dtype)
        self.up_q = _param(q_rows, q_rank, dtype=dtype) if q_rank else None
        self.up_k = _param(heads * dim, kv_rank, dtype=dtype)
        self.up_v = _param(heads * vdim, kv_rank, dtype=dtype)
        self.out_proj = _param(width, heads * vdim, dtype=dtype)
        self.rotation = Rotation(rope_frequencies(int(rot_dims), float(rot_base))[0])
        # filled by finalize_weights: W_UK transposed per head, and the prompt path's [k | rotated k | v] matrix
        self.register_buffer("absorb_k", torch.zeros(heads, kv_rank, dim, dtype=dtype), persistent=False)
        qk = dim + rot_dim
        self.prompt_kernel = (dtype != torch.float32 and qk % 8 == 0 and vdim % 8 == 0 and qk <= 192 and vdim <= 128)
        if self.prompt_kernel:
            self.register_buffer("up_kv", torch.zeros(heads, qk + vdim, self.row, dtype=dtype), persistent=False)

    def finalize_weights(self) -> None:
        H, D, R, K = self.heads, self.dim, self.rot_dim, self.kv_rank
        uk = self.up_k.data.view(H, D, K)
        self.absorb_k.copy_(uk.transpose(1, 2))
        if self.prompt_kernel:
            self.up_kv.zero_()
            self.up_kv[:, :D, :K] = uk
            self.up_kv[:, D: D + R, K: K + R] = torch.eye(R, dtype=self.dtype, device=uk.device)
            self.up_kv[:, D + R:, :K] = self.up_v.data.view(H, self.vdim, K)

    def slots(self) -> dict:
        """Tensor name -> the memory it is copied to."""
        out = {"dkv": self.down.rows("dkv"), "dkv.norm": self.kv_norm.data, "uk": self.up_k.data, "uv": self.up_v.data,
               "o": self.out_proj.data}
        if self.q_rank:
            return {"dq": self.down.rows("dq"), "dq.norm": self.q_norm.data, "uq": self.up_q.data, **out}
        return {"q": self.down.rows("q"), **out}

    # ---- cache ------------------------------------------------------------------------------------------------------
    def cache_elems_per_token(self) -> int:
        return self.row

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device) -> torch.Tensor:
        return LatentCache.allocate(num_blocks, block_size, self.kv_rank, self.rot_dim, self.dtype, device)

    def decode_workspace_floats(self, batch: int, max_seq_len: int) -> int:
        """What the split decode of ``batch`` rows needs for its partial results (0: it does not split)."""
        n = ops.mla_decode_num_splits(batch, self.heads, max_seq_len, self.window)
        return n * batch * self.heads * (self.kv_rank + 1) if n > 1 else 0

    # ---- forward ----------------------------------------------------------------------------------------------------
    def _absorbed(self, q, angles, cache, md, n_req: int, out) -> None:
        """Rows [0, len(q)) of the step, which belong to its first ``n_req`` requests."""
        m, H, D, K = q.shape[0], self.heads, self.dim, self.kv_rank
        qa = torch.empty(m, H, self.row, dtype=q.dtype, device=q.device)
        ops.gemm_batched(q[..., :D].transpose(0, 1), self.absorb_k, out=qa[..., :K].transpose(0, 1))
        ops.latent_rope(qa[..., K:], q[..., D:], angles, self.rot_dim, self.row - K - self.rot_dim, self.interleaved)
        lat = ops.mla_decode(qa, cache, md.block_table[:n_req], md.seq_lens[:n_req], self.scale,
                             query_start_loc=md.query_start_loc[:n_req + 1], max_seq_len=md.max_seq_len,
                             window=self.window, kv_rank=K, workspace=md.decode_workspace)
        ops.gemm_batched(lat.transpose(0, 1), self.up_v.view(H, self.vdim, K), out=out.transpose(0, 1))

    def forward(self, positions, h):
        ctx = get_forward_context()
        md = ctx.attn_metadata
        cache = ctx.kv_caches[self.cache_idx]
        T, H, D, R, V = h.shape[0], self.heads, self.dim, self.rot_dim, self.vdim
        a, angles = self.down(h), self.rotation.angles(positions, T)
        cq = ops.latent_insert(a, self.down.offsets.get("dq", 0), self.down.offsets["dkv"], self.q_norm, self.kv_norm, R,
                               angles, cache, md.slot_mapping, self.eps, self.interleaved)
        q = (ops.gemm(cq, self.up_q) if self.q_rank else self.down.part(a, "q")).unflatten(1, (H, D + R))
        out = torch.empty(T, H, V, dtype=h.dtype, device=h.device)
        nd, ndt = md.num_decodes, md.num_decode_tokens
        mha = self.prompt_kernel and h.is_cuda and md.num_prefills > 0
        if mha:
            cu_rows, first, total = prompt_spans(md, self.window)
            mha = total <= CONTEXT_PER_TOKEN * (T - ndt)
        if not mha:
            self._absorbed(q, angles, cache, md, md.num_reqs, out)
        else:
            if ndt > 0:
                self._absorbed(q[:ndt], angles[:ndt], cache, md, nd, out[:ndt])
            qp = q[ndt:]
            ops.latent_rope(qp[..., D:], qp[..., D:], angles[ndt:], R, 0, self.interleaved)
            rows = ops.gather_mla_cache(cache, md.block_table[nd:], cu_rows, first, total)
            kv = ops.gemm(rows, self.up_kv.view(H * (D + R + V), self.row)).view(total, H, D + R + V)
            ops.varlen_attention(qp, kv[..., : D + R], kv[..., D + R:], md.prefill_query_start_loc, cu_rows, self.scale,
                                 out=out[ndt:], max_q_len=md.max_prefill_query_len, causal=True,
                                 window=self.window if self.window > 0 else -1)
        return ops.gemm(out.view(T, H * V), self.out_proj)
