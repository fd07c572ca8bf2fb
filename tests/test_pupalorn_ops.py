"""Every mechanism of the Pupalorn decoder alone, against the plain float64 statement in ``pupalorn_oracle.py``: on the CPU
(the PyTorch statements of the ops) and on the GPU (the kernels), in fp32 and bf16."""
import random

import pytest
import torch

from tests import pupalorn_oracle as O
from vllm_metax_b200 import _custom_ops as ops
from vllm_metax_b200.layers.attention import PagedGQABackend
from vllm_metax_b200.layers.fused_moe import FusedMoE, expert_rows
from vllm_metax_b200.ops.reference import rope_frequencies
from vllm_metax_b200.ops.residual_norm import ExpertRows, boundary_norm, embed_norm

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = [torch.float32, torch.bfloat16]
pytestmark = pytest.mark.usefixtures("kernel_status_ok")


def tol(dt):
    return 2e-5 if dt == torch.float32 else 1.5e-2


def close(got, want, dt, factor=1.0):
    got, want = got.detach().cpu().to(torch.float64), want.to(torch.float64)
    rms = want.pow(2).mean().sqrt().clamp_min(1e-6)
    err = float((got - want).abs().max() / rms)
    assert err < 6 * tol(dt) * factor, f"max error {err:.3g} of the rms"


def rnd(*shape, dt=torch.float32, scale=1.0, seed=None):
    g = torch.Generator().manual_seed(seed if seed is not None else sum(shape) * 7 + len(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dt)


def i32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


# ------------------------------------------------------------------ boundary: norm, residual, norm
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width", [37, 96, 264, 2048, 2056, 4096])
def test_boundary(device, dt, width):
    eps, T = 3e-3, 11
    y, x = rnd(T, width, dt=dt), rnd(T, width, seed=5, scale=3.0)
    g1, g2 = 0.4 * rnd(width, seed=6), 1 + rnd(width, seed=7)
    want_x = x.double() + O.unit_rms(y.double(), eps) * g1.double()
    want_h = O.unit_rms(want_x, eps) * g2.double()
    a = [t.to(device) for t in (y, x, g1, g2)]
    xo, h = boundary_norm(*a, eps)
    close(xo, want_x, torch.float32)
    close(h, want_h, dt)
    assert h.dtype == dt and xo.dtype == torch.float32
    none, h2 = boundary_norm(*a, eps, want_x=False)
    assert none is None and torch.equal(h2, h)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width", [30, 96, 1024])
def test_embedding_boundary(device, dt, width):
    table, g = rnd(64, width, dt=dt), 1 + 0.3 * rnd(width, seed=2)
    ids = torch.tensor([3, 0, 40, 3, 17])
    x, h = embed_norm(table.to(device), ids.to(device), 41, 7.25, g.to(device), 1e-4)
    want = table.double()[ids] * 7.25
    close(x, want, torch.float32)
    close(h, O.unit_rms(want, 1e-4) * g.double(), dt)


# ------------------------------------------------------------------ rotation frequencies
@pytest.mark.parametrize("scaling", [None, dict(factor=5.0, low=1.0, high=3.0, original=300),
                                     dict(factor=3.0, low=2.0, high=2.5, original=100), dict(factor=1.0, low=1.0, high=4.0, original=64)])
@pytest.mark.parametrize("dims,base", [(2, 500.0), (40, 8000.0), (96, 5e5)])
def test_frequencies(dims, base, scaling):
    hf = scaling and {"type": "llama3", "factor": scaling["factor"], "low_freq_factor": scaling["low"],
                      "high_freq_factor": scaling["high"], "original_max_position_embeddings": scaling["original"]}
    got = rope_frequencies(dims, base, hf)[0]
    want = torch.tensor(O.frequencies(dims, base, scaling), dtype=torch.float64)
    assert torch.allclose(got, want, rtol=1e-12, atol=0)


# ------------------------------------------------------------------ head norms, rotation, cache write
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,rot", [(4, 2, 64, 64, 32), (3, 1, 128, 64, 128), (2, 2, 10, 3, 6), (5, 5, 48, 40, 16),
                                              (16, 4, 256, 128, 64), (2, 1, 264, 8, 96), (8, 1, 72, 136, 24), (1, 1, 2, 1, 2)])
def test_head_norm_rope(device, dt, H, G, dim, vdim, rot):
    """Queries out, keys and values into pages in any order; rows without a slot leave the cache alone; far positions."""
    T, bs, blocks, eps = 9, 16, 5, 2e-3
    dp, vp = -(-dim // 8) * 8, -(-vdim // 8) * 8
    q, k, v = rnd(T, H, dim, dt=dt), rnd(T, G, dim, dt=dt, seed=3), rnd(T, G, vdim, dt=dt, seed=4)
    wq, wk = ((1 + 0.3 * rnd(dim, seed=s)).to(dt) for s in (8, 9))
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    qkv = torch.cat([pad(q, dp).flatten(1), pad(k, dp).flatten(1), pad(v, vp).flatten(1)], 1).to(device)
    off = (0, H * dp, (H + G) * dp)
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4097, 100000, 5])
    slots = torch.tensor([16, 17, 3, 79, 0, -1, 40, 41, 33])
    freqs = O.frequencies(rot, 9000.0)
    angles = ops.rope_angles(pos.to(device), torch.tensor(freqs, dtype=torch.float64, device=device), T)
    cache = torch.full_like(PagedGQABackend.allocate_pages(blocks, bs, G, dp, vp, dt, device), 7.0)
    kc, vc = PagedGQABackend.views(cache, bs, G, dp, vp)
    got = ops.head_norm_rope(qkv, off, pad(wq, dp).to(device), pad(wk, dp).to(device), H, dim, angles, (kc, vc),
                             slots.to(device), eps)
    norm = lambda x, w: O.rotate(O.unit_rms(x.double(), eps) * w.double(), pos, rot, freqs)
    close(got[..., :dim], norm(q, wq), dt)
    assert float(got[..., dim:].abs().sum()) == 0
    kw = norm(k, wk)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kc[s // bs, s % bs, :, :dim], kw[t], dt, 2.0)
            assert torch.equal(vc[s // bs, s % bs, :, :vdim].cpu(), v[t])
    written = {s for s in slots.tolist() if s >= 0}
    for s in range(blocks * bs):
        if s not in written:
            assert bool((kc[s // bs, s % bs] == 7).all()) and bool((vc[s // bs, s % bs] == 7).all())
    only = ops.head_norm_rope(qkv[:, : H * dp].contiguous(), (0, 0, 0), pad(wq, dp).to(device), None, H, dim, angles,
                              None, slots.to(device), eps)
    assert torch.equal(only, got)


# ------------------------------------------------------------------ paged attention
def paged_case(device, dt, lens, new, H, G, dim, vdim, bs, seed=0, spike=()):
    """Ragged batch over shuffled pages.  ``spike``: (sequence, query position, key position) whose score stands out."""
    rng = random.Random(seed)
    qs, ks, vs = [], [], []
    for b, n in enumerate(lens):
        qs.append(rnd(n, H, dim, seed=seed + 10 * b))
        ks.append(rnd(n, G, dim, seed=seed + 10 * b + 1))
        vs.append(rnd(n, G, vdim, seed=seed + 10 * b + 2))
    for b, i, j in spike:
        ks[b][j] *= 4.0
        for h in range(H):
            qs[b][i, h] = ks[b][j, h // (H // G)] * 2.0
    qs, ks, vs = ([t.to(dt) for t in l] for l in (qs, ks, vs))
    pages = [-(-n // bs) for n in lens]
    order = list(range(sum(pages) + 2))
    rng.shuffle(order)
    cache = PagedGQABackend.allocate_pages(len(order), bs, G, dim, vdim, dt, "cpu")
    cache.copy_(rnd(*cache.shape, seed=99).to(dt))                 # what is outside a sequence must not matter
    kc, vc = PagedGQABackend.views(cache, bs, G, dim, vdim)
    table = torch.zeros(len(lens), max(pages), dtype=torch.int32)
    for b, n in enumerate(lens):
        for p in range(pages[b]):
            table[b, p] = order.pop()
            m = min(bs, n - p * bs)
            kc[table[b, p], :m] = ks[b][p * bs: p * bs + m]
            vc[table[b, p], :m] = vs[b][p * bs: p * bs + m]
    q = torch.cat([qs[b][n - c:] for b, (n, c) in enumerate(zip(lens, new))])
    qsl = [0]
    for c in new:
        qsl.append(qsl[-1] + c)
    cache = cache.to(device)
    return (q.to(device), PagedGQABackend.views(cache, bs, G, dim, vdim) if cache.dim() == 2 else cache, table.to(device),
            i32(lens, device), i32(qsl, device), [t.double() for t in qs], [t.double() for t in ks], [t.double() for t in vs])


ATTN = [(4, 2, 64, 64, 64), (6, 2, 48, 40, 16), (3, 1, 128, 24, 32), (5, 5, 8, 16, 16), (4, 1, 136, 128, 64), (2, 2, 192, 104, 32),
        (2, 1, 200, 256, 64), (2, 2, 264, 16, 16), (1, 1, 16, 296, 32)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("window", [-1, 1, 5, 64, 130])
@pytest.mark.parametrize("H,G,dim,vdim,bs", ATTN)
def test_paged_attention(device, dt, window, H, G, dim, vdim, bs):
    """Decode rows and prompt portions of ragged batches, key and value sizes of any tile, windows over page borders; one key
    just inside and one just outside the window stand out."""
    lens, new = [1, 70, 129, 200, 16], [1, 3, 129, 40, 16]
    w = window if window > 0 else 0
    far = min(150, w or 150)
    spike = [(3, 180, 180 - far), (3, 195, 195 - far + 1), (2, 128, max(0, 128 - far)), (1, 69, max(0, 69 - far + 1))]
    q, cache, table, sl, qsl, qs, ks, vs = paged_case(device, dt, lens, new, H, G, dim, vdim, bs, spike=spike)
    want = [O.attend(a, b, c, dim ** -0.5, w) for a, b, c in zip(qs, ks, vs)]
    out = ops.paged_attention_prefill(q, cache, table, sl, qsl, dim ** -0.5, max_q_len=max(new), window=window, max_seq_len=200)
    close(out, torch.cat([x[n - c:] for x, n, c in zip(want, lens, new)]), dt, 2.0)
    last = (qsl[1:] - 1).long()
    for splits in (0, 1, 3):
        dec = ops.paged_attention_decode(q[last].contiguous(), cache, table, sl, dim ** -0.5, window=window, num_splits=splits,
                                         max_seq_len=200)
        close(dec, torch.stack([x[-1] for x in want]), dt, 2.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("window,far", [(-1, 1499), (-1, 700), (1000, 999), (1000, 1000), (600, 599)])
def test_far_keys(device, dt, window, far):
    lens = [1500, 3]
    q, cache, table, sl, qsl, qs, ks, vs = paged_case(device, dt, lens, [20, 3], 4, 2, 64, 32, 64, spike=[(0, 1499, 1499 - far)])
    want = [O.attend(a, b, c, 0.125, max(0, window)) for a, b, c in zip(qs, ks, vs)]
    out = ops.paged_attention_prefill(q, cache, table, sl, qsl, 0.125, max_q_len=20, window=window, max_seq_len=1500)
    close(out, torch.cat([want[0][-20:], want[1]]), dt, 2.0)
    dec = ops.paged_attention_decode(q[[19, 22]].contiguous(), cache, table, sl, 0.125, window=window, max_seq_len=1500)
    close(dec, torch.stack([want[0][-1], want[1][-1]]), dt, 2.0)


# ------------------------------------------------------------------ experts
def moe_weights(E, I, W, ff, dt, seed=0):
    w = {"x.router": rnd(E + I, W, dt=dt, seed=seed, scale=2.0 * W ** -0.5), "x.correction": rnd(E + I, dt=dt, seed=seed + 1, scale=0.05)}
    for e in range(E):
        w[f"x.e{e}.up"] = rnd(ff, W, dt=dt, seed=seed + 2 + 2 * e, scale=W ** -0.5)
        w[f"x.e{e}.down"] = rnd(W, ff, dt=dt, seed=seed + 3 + 2 * e, scale=ff ** -0.5)
    return w


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,I,top", [(12, 3, 2), (3, 5, 4), (8, 0, 1), (1, 1, 2), (40, 30, 6)])
def test_routing(device, E, I, top):
    """Softmax over all outputs, the correction in the choice and not in the weights, no renormalisation."""
    T = 33
    z, c = rnd(T, E + I, scale=1.5), rnd(E + I, scale=0.3, seed=4)
    w, ids = ops.topk_gating(z.to(device), top, False, "softmax", c.to(device))
    moved = 0
    for t in range(T):
        want = O.choose(z[t].double(), c.double(), top)
        assert ids[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].cpu().double(), torch.tensor([x for _, x in want], dtype=torch.float64), rtol=1e-5, atol=1e-7)
        moved += [e for e, _ in want] != [e for e, _ in O.choose(z[t].double(), 0 * c.double(), top)]
    assert moved > 0 or top >= E + I


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("E,I,top,W,ff,T", [(6, 2, 2, 96, 40, 17), (3, 5, 4, 64, 24, 40), (4, 0, 1, 48, 16, 5), (1, 1, 2, 30, 7, 3),
                                            (16, 4, 3, 128, 64, 300)])
def test_identity_experts(device, dt, E, I, top, W, ff, T):
    """The layer, combined by itself and inside the boundary."""
    w = moe_weights(E, I, W, ff, dt)
    f = {"router": {"experts": E, "identity": I, "top": top}, "expert": {"ff": ff}}
    h = rnd(T, W, dt=dt, seed=50)
    want = O.experts(h.double(), w, "x.", f)
    with torch.device(device):
        layer = FusedMoE(E, top, W, ff, dt, renormalize=False, scoring_func="softmax", e_score_correction_bias=True, gated=False,
                         activation="relu2", num_identity=I)
    for e in range(E):
        layer.weight_loader(layer.w13_weight, w[f"x.e{e}.up"], e, "w1")
        layer.weight_loader(layer.w2_weight, w[f"x.e{e}.down"], e, "w2")
    layer.weight_loader(layer.e_score_correction_bias, w["x.correction"].float())
    hd = h.to(device)
    logits = ops.router_logits(hd, w["x.router"].to(device))
    close(layer(hd, logits), want, dt, 2.0)
    rows = layer.forward_rows(hd, logits)
    assert isinstance(rows, ExpertRows)
    close(rows.combined(), want, dt, 2.0)
    x, g = rnd(T, W, seed=51), 1 + 0.2 * rnd(W, seed=52)
    xo, hn = boundary_norm(rows, x.to(device), g.to(device), g.to(device), 1e-3)
    want_x = x.double() + O.unit_rms(want, 1e-3) * g.double()
    close(xo, want_x, dt, 2.0)
    close(hn, O.unit_rms(want_x, 1e-3) * g.double(), dt, 2.0)


@pytest.mark.parametrize("device", DEVICES)
def test_only_identity_experts_are_chosen(device):
    """No pair has a row of its own: the output is the input times the weights' sum."""
    E, I, W, T = 2, 3, 64, 9
    x = rnd(T, W, dt=torch.bfloat16).to(device)
    w13, w2 = rnd(E, 16, W, dt=torch.bfloat16).to(device), rnd(E, W, 16, dt=torch.bfloat16).to(device)
    ids = torch.stack([torch.randperm(I)[:2] + E for _ in range(T)]).to(torch.int32).to(device)
    wt = torch.rand(T, 2).to(device)
    got = expert_rows(x, w13, w2, wt, ids, E, epi=ops.EPI_CODES["relu2"], identity_from=E).combined()
    close(got, wt.cpu().double().sum(1, keepdim=True) * x.cpu().double(), torch.bfloat16)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (70, 40, 24), (300, 256, 1024), (33, 7, 15), (1024, 4096, 256)])
def test_squared_relu_epilogue(device, dt, M, N, K):
    a, w = rnd(M, K, dt=dt), rnd(N, K, dt=dt, scale=K ** -0.5)
    close(ops.gemm(a.to(device), w.to(device), act="relu2"), O.relu_squared(a.double() @ w.double().t()), dt, 3.0)
