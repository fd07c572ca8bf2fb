"""Every mechanism of the Luluzen decoder alone, against the plain float64 statement in ``luluzen_oracle.py``: on the CPU (the
PyTorch statements of the ops) and on the GPU (the kernels), in fp32 and bf16."""
import math
import random

import pytest
import torch

from tests import luluzen_oracle as O
from vllm_metax_b200 import _custom_ops as ops
from vllm_metax_b200.layers.attention import PagedGQABackend, distance_buckets
from vllm_metax_b200.layers.fused_moe import FusedMoE
from vllm_metax_b200.ops.channel_delta import channel_delta_rule
from vllm_metax_b200.ops.gla import Normalizer, Steps, linear_attention, memory_gates
from vllm_metax_b200.ops.prenorm import loop_operand, prenorm
from vllm_metax_b200.ops.residual_norm import ExpertRows

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


# ------------------------------------------------------------------ boundary: add, layer norm
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width", [37, 96, 264, 2048, 2056, 4096])
def test_boundary(device, dt, width):
    """Rows far from zero: the mean is taken off before the squares are summed."""
    eps, T = 3e-3, 11
    y, x = rnd(T, width, dt=dt), rnd(T, width, seed=5, scale=3.0) + 40.0
    g, add = (1 + rnd(width, seed=7)).to(dt), rnd(width, seed=8, dt=dt)
    yd, xd, gd, ad = (t.to(device) for t in (y, x, g, add))
    want = x.double() + y.double()
    xo, h = prenorm(yd, xd, gd, eps)
    close(xo, want, torch.float32)
    close(h, O.layer_norm(want, g, eps), dt, 4.0)
    assert h.dtype == dt and xo.dtype == torch.float32
    none, h2 = prenorm(yd, xd, gd, eps, want_x=False)
    assert none is None and torch.equal(h2, h)
    z = rnd(T, width, seed=9)                                    # an fp32 product and a vector, as behind the loop's product
    xo, h = prenorm(z.to(device), None, gd, eps, ad)
    close(xo, z.double() + add.double(), torch.float32)
    close(h, O.layer_norm(z.double() + add.double(), g, eps), dt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width", [30, 96, 1024])
def test_embedding_and_loop_operand(device, dt, width):
    table, g = rnd(64, width, dt=dt), (1 + 0.3 * rnd(width, seed=2)).to(dt)
    ids = torch.tensor([3, 0, 40, 3, 17])
    t, i, gd = table.to(device), ids.to(device), g.to(device)
    x, h = prenorm(t, None, gd, 1e-4, None, i, 41)
    close(x, table.double()[ids], torch.float32)
    close(h, O.layer_norm(table.double()[ids], g, 1e-4), dt)
    y, x = rnd(5, width, dt=dt, seed=3), 9.0 * rnd(5, width, seed=4)
    parts = 2 if dt == torch.float32 else 3
    op = loop_operand(y.to(device), x.to(device), t, i, 41).view(5, parts, width).cpu().double()
    want = x.double() + y.double()
    close(op[:, :-1].sum(1), want, torch.float32)               # 16-bit parts add up to far more than 16 bits
    assert torch.equal(op[:, -1], table.double()[ids])
    first = loop_operand(t, None, t, i, 41, gather=True).view(5, parts, width).cpu().double()
    assert torch.equal(first[:, :-1].sum(1), table.double()[ids]) and torch.equal(first[:, -1], table.double()[ids])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,topk,width,weighted", [(7, 1, 96, False), (19, 3, 264, False), (5, 6, 50, True)])
def test_boundary_sums_expert_rows(device, dt, T, topk, width, weighted):
    rows, x = rnd(T * topk + 9, width, dt=dt), rnd(T, width, seed=5)
    inv = torch.randperm(T * topk + 9, generator=torch.Generator().manual_seed(1))[: T * topk].to(torch.int32)
    w = torch.rand(T, topk, generator=torch.Generator().manual_seed(2)) if weighted else None
    g = (1 + 0.3 * rnd(width, seed=2)).to(dt)
    late = ExpertRows(rows.to(device), None if w is None else w.to(device), inv.to(device), top=topk)
    xo, h = prenorm(late, x.to(device), g.to(device), 1e-5)
    picked = rows.double()[inv.long()].view(T, topk, width)
    want = x.double() + (picked if w is None else picked * w.double()[..., None]).sum(1)
    close(xo, want, torch.float32 if device == "cuda" else dt)
    close(h, O.layer_norm(want, g, 1e-5), dt, 2.0)


# ------------------------------------------------------------------ norms, rotation, query temperature, cache write
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("whole_row", [False, True])
@pytest.mark.parametrize("H,G,dim,vdim,rot", [(4, 2, 64, 64, 32), (3, 1, 128, 64, 128), (2, 2, 10, 3, 6), (5, 5, 48, 40, 0),
                                              (16, 4, 256, 128, 64), (2, 1, 264, 8, 98), (8, 1, 72, 136, 20), (1, 1, 2, 1, 2)])
def test_norm_rotation_temperature(device, dt, whole_row, H, G, dim, vdim, rot):
    """Adjacent pairs, one norm per head or over the row, a temperature or none; far positions; rows without a slot."""
    T, bs, blocks, eps = 9, 16, 5, 2e-3
    dp, vp = -(-dim // 8) * 8, -(-vdim // 8) * 8
    q, k, v = rnd(T, H, dim, dt=dt), rnd(T, G, dim, dt=dt, seed=3), rnd(T, G, vdim, dt=dt, seed=4)
    wq, wk = ((1 + 0.3 * rnd(n if whole_row else 1, dim, seed=s)).to(dt) for s, n in ((8, H), (9, G)))
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    qkv = torch.cat([pad(q, dp).flatten(1), pad(k, dp).flatten(1), pad(v, vp).flatten(1)], 1).to(device)
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4097, 100000, 5])
    slots = torch.tensor([16, 17, 3, 79, 0, -1, 40, 41, 33])
    base = 700.0
    angles = None
    if rot:
        freqs = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device=device)
        angles = ops.rope_angles(pos.to(device), freqs, T)
    temp = None if whole_row and rot else (pos.to(device), 0.4, 7)
    kc, vc = PagedGQABackend.views(torch.zeros_like(PagedGQABackend.allocate_pages(blocks, bs, G, dp, vp, dt, device)), bs, G, dp, vp)
    got = ops.head_norm_rope(qkv, (0, H * dp, (H + G) * dp), pad(wq, dp).flatten().to(device), pad(wk, dp).flatten().to(device), H,
                             dim, angles, (kc, vc), slots.to(device), eps, whole_row=whole_row, interleaved=True, q_temp=temp)

    def normed(x, w):
        x = x.double()
        y = O.unit_rms(x.flatten(1), eps).view_as(x) if whole_row else O.unit_rms(x, eps)
        return O.rotate_pairs(y * w.double(), pos, rot, base)

    want = normed(q, wq)
    if temp is not None:
        want = want * O.query_temperature(pos, 0.4, 7)[:, None, None]
    close(got[..., :dim], want, dt)
    assert float(got[..., dim:].abs().sum()) == 0
    kw = normed(k, wk)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kc[s // bs, s % bs, :, :dim], kw[t], dt, 2.0)
            assert torch.equal(vc[s // bs, s % bs, :, :vdim].cpu(), v[t])


# ------------------------------------------------------------------ paged attention
def test_distance_buckets():
    for rows, far in ((16, 110), (2, 2), (3, 9), (32, 128), (32, 1000), (6, 4), (10, 6), (16, 128), (7, 300)):
        index = distance_buckets(rows, far)
        assert len(index) <= far + 1
        for n in range(far + 40):
            assert index[min(n, len(index) - 1)] == O.distance_bucket(n, rows, far), (rows, far, n)
    for rows, far in ((1, 5), (16, 8), (16, 3)):
        with pytest.raises(ValueError):
            distance_buckets(rows, far)


def paged_case(device, dt, lens, new, H, G, dim, vdim, bs, spike=(), scale=1.0):
    """Ragged batch over shuffled pages.  ``spike``: (sequence, query position, key position) whose score stands out."""
    rng = random.Random(3)
    qs, ks, vs = ([rnd(n, h, d, seed=10 * b + s, dt=dt) for b, n in enumerate(lens)] for s, h, d in ((0, H, dim), (1, G, dim), (2, G, vdim)))
    for b, i, j in spike:
        u = rnd(dim, seed=77)
        u = (u / u.norm() * math.sqrt(6.0 / scale)).to(dt)
        qs[b][i], ks[b][j] = u, u
    nb = [-(-n // bs) for n in lens]
    pages = list(range(sum(nb) + 3))
    rng.shuffle(pages)
    kc, vc = PagedGQABackend.views(PagedGQABackend.allocate_pages(len(pages), bs, G, dim, vdim, dt, device), bs, G, dim, vdim)
    table = torch.zeros(len(lens), max(nb), dtype=torch.int32)
    at = 0
    for b, n in enumerate(lens):
        table[b, : nb[b]] = torch.tensor(pages[at: at + nb[b]])
        at += nb[b]
        for j in range(n):
            kc[table[b, j // bs], j % bs], vc[table[b, j // bs], j % bs] = ks[b][j].to(device), vs[b][j].to(device)
    q = torch.cat([qs[b][lens[b] - new[b]:] for b in range(len(lens))]).to(device)
    qsl = [0]
    for n in new:
        qsl.append(qsl[-1] + n)
    return qs, ks, vs, q, (kc, vc), table.to(device), i32(lens, device), i32(qsl, device)


ATTN = [  # H, G, dim, vdim, bs, options
    (4, 2, 64, 48, 64, dict(softcap=9.0, sink=True, gate=True, window=37)),
    (6, 2, 40, 64, 16, dict(bias=(16, 50))),
    (3, 3, 128, 128, 64, dict(bias=(6, 90), gate=True, sink=True)),
    (8, 1, 96, 104, 64, dict(bias=(32, 400), softcap=5.0)),
    (2, 1, 192, 128, 64, dict(sink=True, softcap=3.0)),
    (2, 2, 200, 160, 32, dict(bias=(8, 20), gate=True, window=64, sink=True)),
    (2, 1, 264, 16, 16, dict(bias=(4, 10), gate=True, softcap=4.0, sink=True)),
    (1, 1, 8, 8, 16, dict(bias=(2, 2), sink=True, window=1)),
]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,bs,opt", ATTN)
@pytest.mark.parametrize("decode", [False, True])
def test_paged_attention(device, dt, H, G, dim, vdim, bs, opt, decode):
    """Prompts, portions with context and single tokens; a key that alone matters sits at bucket and page borders and just
    inside and outside the window.  The output's rows are part of wider ones."""
    lens = [1, 63, 64, 65, 130, 259, 300, 17]
    new = [1] * 8 if decode else [1, 63, 1, 2, 70, 259, 130, 17]
    scale = dim ** -0.5
    win = opt.get("window", 0)
    spikes = [(1, 62, 10), (3, 64, 63), (4, 129, 129 - min(win or 64, 129) + 1), (5, 258, 258 - min(win or 128, 258)),
              (6, 299, 0), (7, 16, 0)]
    qs, ks, vs, q, kv, table, sl, qsl = paged_case(device, dt, lens, new, H, G, dim, vdim, bs, spikes, scale)
    rel = 2.0 * rnd(*((opt["bias"][0], H) if "bias" in opt else (2, H)), seed=5)
    bias = rel[distance_buckets(*opt["bias"])].t().contiguous().to(device) if "bias" in opt else None
    sink = rnd(H, seed=6) if opt.get("sink") else None
    T = q.shape[0]
    wide = torch.zeros(T, 8 + H * vdim + 16, dtype=dt, device=device)
    out = wide[:, 8: 8 + H * vdim].unflatten(1, (H, vdim))
    gates = rnd(T, 8 + H * vdim, seed=9, dt=dt).to(device)[:, 8:] if opt.get("gate") else None
    kw = dict(out=out, window=win or -1, softcap=opt.get("softcap", 0.0), sinks=None if sink is None else sink.to(device),
              max_seq_len=max(lens), distance_bias=bias, gate=gates, out_scale=0.7)
    if decode:
        ops.paged_attention_decode(q, kv, table, sl, scale, **kw)
    else:
        ops.paged_attention_prefill(q, kv, table, sl, qsl, scale, max_q_len=max(new), **kw)
    want = []
    for b, n in enumerate(lens):
        db = O.distance_bias(rel, opt["bias"][1], n) if "bias" in opt else None
        o = O.attend(qs[b].double(), ks[b].double(), vs[b].double(), scale, win, opt.get("softcap", 0.0), db, sink)
        want.append(o[n - new[b]:])
    want = 0.7 * torch.cat(want)
    if gates is not None:
        want = want * O.sigmoid(gates.cpu().double()).view_as(want)
    close(out, want, dt, 2.0)
    assert float(wide[:, :8].abs().sum()) == 0 and float(wide[:, 8 + H * vdim:].abs().sum()) == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("opt", [dict(bias=(32, 900), gate=True), dict(softcap=20.0, sink=True, gate=True, window=1500)])
def test_split_decoding_far_back(dt, opt):
    """Few requests with long contexts: the keys are split over CTAs, whose parts meet the sink, gate and factor once."""
    test_case = [2000, 1537, 31]
    H, G, dim, vdim = 4, 2, 64, 56
    win = opt.get("window", 0)
    qs, ks, vs, q, kv, table, sl, _ = paged_case("cuda", dt, test_case, [1, 1, 1], H, G, dim, vdim, 64,
                                                 [(0, 1999, 1999 - (win or 2000) + 1), (1, 1536, 1536 - 900)], dim ** -0.5)
    rel, sink = 2.0 * rnd(32, H, seed=5), rnd(H, seed=6)
    bias = rel[distance_buckets(32, 900)].t().contiguous().cuda() if "bias" in opt else None
    gates = rnd(3, H * vdim, seed=9, dt=dt).cuda()
    got = ops.paged_attention_decode(q, kv, table, sl, dim ** -0.5, window=win or -1, softcap=opt.get("softcap", 0.0),
                                     sinks=sink.cuda() if opt.get("sink") else None, max_seq_len=2000, distance_bias=bias,
                                     gate=gates, out_scale=1.3)
    want = torch.cat([O.attend(qs[b].double(), ks[b].double(), vs[b].double(), dim ** -0.5, win, opt.get("softcap", 0.0),
                               O.distance_bias(rel, 900, n) if "bias" in opt else None, sink if opt.get("sink") else None)[-1:]
                      for b, n in enumerate(test_case)])
    close(got, 1.3 * want * O.sigmoid(gates.cpu().double()).view_as(want), dt, 2.0)


# ------------------------------------------------------------------ recurrences over portions, slots used again
LENS = [5, 40, 1, 17, 70, 33]
CUTS = [[{0: 5, 1: 40, 2: 1, 3: 17, 4: 70, 5: 33}],                                       # whole
        [{0: 2, 1: 17}, {1: 1, 2: 1, 3: 16}, {0: 3, 3: 1, 4: 31, 1: 2}, {4: 2, 1: 20, 5: 1}, {4: 37, 5: 32}],
        [{i: 1 for i in range(6) if t < LENS[i]} for t in range(70)]]                    # token by token


def run_portions(cuts, lens, device, fn):
    """``fn(rows, steps)`` on the tokens of each step (``rows``: (sequence, position) pairs); sequences share a pool of slots in
    which they come and go, and whose contents are never cleared.  Returns the outputs per sequence."""
    at, slots, free = [0] * len(lens), {}, list(range(len(lens) + 1))
    outs = [[] for _ in lens]
    rng = random.Random(1)
    for step in cuts:
        order = list(step)
        rng.shuffle(order)
        rows, qsl, idx, init = [], [0], [], []
        for b in order:
            if b not in slots:
                slots[b] = free.pop(rng.randrange(len(free)))
            idx.append(slots[b])
            init.append(int(at[b] > 0))
            rows += [(b, at[b] + j) for j in range(step[b])]
            qsl.append(len(rows))
        o = fn(rows, Steps(i32(qsl, device), i32(idx, device), i32(init, device), max(step.values()))).cpu()
        for n, b in enumerate(order):
            outs[b].append(o[qsl[n]: qsl[n + 1]])
            at[b] += step[b]
            if at[b] == lens[b]:
                free.append(slots.pop(b))
    return [torch.cat(o) for o in outs]


def gather(seqs, rows, device):
    return torch.stack([seqs[b][t] for b, t in rows]).to(device)


def dirty(*shape, device):
    return torch.full(shape, 3.0, dtype=torch.float32, device=device)


RECURRENT = [(2, 64, 32), (3, 20, 12), (1, 33, 7), (4, 96, 136), (2, 136, 48), (2, 128, 128), (1, 256, 24)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,V", RECURRENT)
@pytest.mark.parametrize("cuts", range(len(CUTS)))
def test_lightning_over_portions(device, dt, H, D, V, cuts):
    W = 2 * H * D + 2 * H * V
    p = [rnd(n, W, seed=b, dt=dt) for b, n in enumerate(LENS)]
    decay, nw = torch.linspace(0.6, 0.999, H), (1 + 0.3 * rnd(H * V, seed=8)).to(dt)
    off = (0, H * D, 2 * H * D, 2 * H * D + H * V)
    state = dirty(7, H, D, V, device=device)
    got = run_portions(CUTS[cuts], LENS, device, lambda rows, s: linear_attention(
        gather(p, rows, device), off, decay.to(device), nw.to(device), state, s, 1.0, 1e-4, "sigmoid", True, True, out_scale=0.6))
    for b, n in enumerate(LENS):
        x = p[b].double()
        q, k, v = (O.silu(x[:, a: a + H * d]).view(n, H, d) for a, d in zip(off, (D, D, V)))
        o = O.unit_rms(O.decayed_states(q, k, v, decay.double()).reshape(n, -1), 1e-4) * nw.double()
        close(got[b], 0.6 * o * O.sigmoid(x[:, off[3]:]), dt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,V", RECURRENT)
@pytest.mark.parametrize("cuts", range(len(CUTS)))
def test_matrix_memory_over_portions(device, dt, H, D, V, cuts):
    """Gates with large swings: the running maximum, the normaliser's floor and the cap all take part."""
    W, cap = 2 * H * D + 2 * H * V, 7.0
    p, z = [rnd(n, W, seed=b, dt=dt) for b, n in enumerate(LENS)], [4.0 * rnd(n, 2 * H, seed=50 + b) for b, n in enumerate(LENS)]
    bias = torch.cat([rnd(H, seed=3), 2.0 + rnd(H, seed=4)])
    nw = (1 + 0.3 * rnd(H * V, seed=8)).to(dt)
    off = (0, H * D, 2 * H * D, 2 * H * D + H * V)
    state, norm, top = dirty(7, H, D, V, device=device), dirty(7, H, -(-V // 16), D, device=device), dirty(7, H, device=device)

    def run(rows, s):
        g = memory_gates(gather(z, rows, device), bias.to(device), cap, top, s)
        return linear_attention(gather(p, rows, device), off, g[0], nw.to(device), state, s, D ** -0.5, 1e-4, "sigmoid",
                                memory=Normalizer(norm, g[1], g[2]), out_scale=1.4)

    got = run_portions(CUTS[cuts], LENS, device, run)
    for b, n in enumerate(LENS):
        x = p[b].double()
        q, k, v = (x[:, a: a + H * d].view(n, H, d) for a, d in zip(off, (D, D, V)))
        g = O.cap(z[b].double() + bias.double(), cap)
        o = O.memory_states(q * D ** -0.5, k, v, g[:, :H], -O.softplus(-g[:, H:]))
        o = O.unit_rms(o, 1e-4).reshape(n, -1) * nw.double()
        close(got[b], 1.4 * o * O.sigmoid(x[:, off[3]:]), dt, 3.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,V", [(2, 2, 64, 32), (3, 1, 20, 12), (1, 1, 33, 7), (4, 2, 96, 136), (4, 4, 136, 48), (2, 1, 128, 128),
                                     (1, 1, 256, 24)])
@pytest.mark.parametrize("cuts", range(len(CUTS)))
def test_channel_delta_over_portions(device, dt, H, G, D, V, cuts):
    W = 2 * G * D + H * V
    p = [rnd(n, W, seed=b, dt=dt) for b, n in enumerate(LENS)]
    dec = [torch.sigmoid(4.0 + 2.0 * rnd(n, H * D, seed=20 + b)) for b, n in enumerate(LENS)]
    beta, gate = [rnd(n, H, seed=30 + b) for b, n in enumerate(LENS)], [rnd(n, H * V, seed=40 + b, dt=dt) for b, n in enumerate(LENS)]
    nw, off = (1 + 0.3 * rnd(V, seed=8)).to(dt), (0, G * D, 2 * G * D)
    state = dirty(7, H, D, V, device=device)
    wide = {}

    def run(rows, s):
        wide["o"] = torch.zeros(len(rows), H * V + 8, dtype=dt, device=device)
        return channel_delta_rule(*(gather(p, rows, device), off, G, gather(dec, rows, device), gather(beta, rows, device),
                                    gather(gate, rows, device), nw.to(device), state, s, 1e-4), 0.8, wide["o"][:, : H * V])

    got = run_portions(CUTS[cuts], LENS, device, run)
    for b, n in enumerate(LENS):
        x = p[b].double()
        q, k = (x[:, a: a + G * D].view(n, G, D) for a in off[:2])
        q, k = (y / torch.sqrt((y * y).sum(-1, keepdim=True) + 1e-6) for y in (q, k))
        q, k = (y.repeat_interleave(H // G, 1) for y in (q * D ** -0.5, k))
        o = O.delta_states(q, k, x[:, off[2]:].view(n, H, V), dec[b].double().view(n, H, D), O.sigmoid(beta[b].double()))
        o = (O.unit_rms(o, 1e-4) * nw.double()).reshape(n, -1)
        close(got[b], 0.8 * o * O.sigmoid(gate[b].double()), dt, 3.0)


@pytest.mark.gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("kind", ["lightning", "memory", "delta"])
@pytest.mark.parametrize("H,D,V", [(2, 64, 48), (1, 128, 160)])
def test_long_prompts_in_segments_and_columns(dt, kind, H, D, V):
    """Prompts long enough to be cut into segments and column blocks, with history, beside short ones: against the same op token
    by token on the CPU."""
    lens, first = [700, 20, 1030], [260, 20, 1]
    cuts = [{b: n for b, n in enumerate(first)}, {0: 439, 2: 1028}, {0: 1, 2: 1}]
    W = 2 * H * D + 2 * H * V
    p = [rnd(n, W, seed=b, dt=dt) for b, n in enumerate(lens)]
    f = [rnd(n, H * max(D, 2), seed=9 + b) for b, n in enumerate(lens)]
    off = (0, H * D, 2 * H * D, 2 * H * D + H * V)
    nw = (1 + 0.3 * rnd(H * V if kind != "delta" else V, seed=8)).to(dt)
    got = {}
    for device in ("cpu", "cuda"):
        st, norm, top = dirty(4, H, D, V, device=device), dirty(4, H, -(-V // 16), D, device=device), dirty(4, H, device=device)
        nwd = nw.to(device)

        def run(rows, s):
            x, y = gather(p, rows, device), gather(f, rows, device)
            if kind == "lightning":
                return linear_attention(x, off, torch.linspace(0.9, 0.998, H, device=device), nwd, st, s, 1.0, 1e-4, "sigmoid", True, True)
            if kind == "memory":
                g = memory_gates(3.0 * y, torch.full((2 * H,), 2.0, device=device), 9.0, top, s)
                return linear_attention(x, off, g[0], nwd, st, s, D ** -0.5, 1e-4, "sigmoid", memory=Normalizer(norm, g[1], g[2]))
            return channel_delta_rule(x, off[:3], H, torch.sigmoid(4.0 + y), y[:, :H].contiguous(), x[:, off[3]:], nwd, st, s, 1e-4)

        got[device] = run_portions(cuts, lens, device, run)
    for a, b in zip(got["cuda"], got["cpu"]):
        close(a, b, dt, 4.0)


# ------------------------------------------------------------------ product epilogues, experts
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 48, 24), (7, 208, 96), (33, 1280, 1040), (64, 512, 2048), (200, 272, 72), (300, 1024, 512),
                                   (3, 22, 13), (2100, 2048, 64)])
def test_product_epilogues(device, dt, M, N, K):
    a, w, b = rnd(M, K, dt=dt), rnd(N, K, dt=dt, seed=2, scale=K ** -0.5), rnd(N, dt=dt, seed=3)
    y = a.double() @ w.double().t() + b.double()
    ad, wd, bd = a.to(device), w.to(device), b.to(device)
    g, u = y[:, 0::2], y[:, 1::2]
    close(ops.gemm(ad, wd, bd, act="gelu_tanh_gate"), O.gelu_tanh(g) * u, dt, 2.0)
    lim = torch.tensor([0.8, 1.702], device=device)
    gc, uc = g.clamp(max=0.8), u.clamp(-0.8, 0.8)
    close(ops.gemm(ad, wd, bd, act="clamped_swiglu_gate", act_params=lim), gc * O.sigmoid(1.702 * gc) * (uc + 1), dt, 2.0)
    rate = torch.rand(N, generator=torch.Generator().manual_seed(4)) * 2
    close(ops.gemm(ad, wd, bd, act="softplus_decay", act_params=rate.to(device), out_dtype=torch.float32),
          torch.exp(-rate.double() * O.softplus(y)), torch.float32, 4.0)
    cap = torch.tensor([1.3], device=device)
    close(ops.gemm(ad, wd, act="softcap", act_params=cap, out_dtype=torch.float32), O.cap(y - b.double(), 1.3), torch.float32, 4.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W,E,ff,top", [(1, 96, 6, 40, 2), (37, 72, 5, 24, 1), (300, 136, 8, 64, 3), (9, 30, 3, 16, 3)])
def test_experts_with_weighted_inputs(device, dt, T, W, E, ff, top):
    m = FusedMoE(E, top, W, ff, dt, renormalize=False, scoring_func="sigmoid", activation="clamped_swiglu",
                 activation_params=(0.9, 1.702), weight_input=True)
    w = {}
    for e in range(E):
        for i, (n, shape) in enumerate((("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff)))):
            t = w[f"e{e}.{n}"] = rnd(*shape, dt=dt, seed=10 * e + i, scale=1.5 * shape[1] ** -0.5)
            (m.w13_weight.data[e, i::2] if i < 2 else m.w2_weight.data[e]).copy_(t)
    m = m.to(device)
    h, z = rnd(T, W, dt=dt), rnd(T, E, seed=4)
    want = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for e, s in O.choose(z[t].double(), top):
            want[t] += O.expert(s * h[t].double(), w, f"e{e}.", 0.9)
    got = m.forward_rows(h.to(device), z.to(device)).combined()
    close(got, want, dt, 3.0)
    close(m(h.to(device), z.to(device)), want, dt, 3.0)
