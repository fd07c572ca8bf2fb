"""Every mechanism of the Vetipel decoder alone, against the plain float64 statement in ``vetipel_oracle.py``: on the CPU (the
PyTorch statements of the ops) and on the GPU (the kernels), in fp32 and bf16."""
import pytest
import torch

from tests import vetipel_oracle as O
from tests.test_luluzen_ops import DEVICES, DTYPES, close, i32, paged_case, rnd
from vllm_metax_b200 import _custom_ops as ops
from vllm_metax_b200.layers.attention import PagedGQABackend, QKNormAttention
from vllm_metax_b200.ops.stream_norm import Embedded, stream_norm

pytestmark = pytest.mark.usefixtures("kernel_status_ok")


# ------------------------------------------------------------------ boundary over several streams
def boundary_weights(S, seed=0):
    read, write, mix = rnd(S, seed=seed + 1), rnd(S, seed=seed + 2), rnd(S, S, seed=seed + 3)      # (mix is not symmetric)
    return read, write, mix, torch.cat([read, write, mix.flatten()])


def boundary(y, streams, read, write, mix, gain, eps):
    """What the oracle makes of ``y [T, W]`` (or None) and ``streams [T, S, W]``."""
    xs = list(streams.double().unbind(1))
    if y is not None:
        xs = O.write_streams(xs, mix, write, y.double())
    return torch.stack(xs, 1), O.unit_rms(O.read_streams(xs, read), eps) * gain.double()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width,S", [(37, 1), (96, 2), (264, 3), (2048, 3), (2056, 4), (4096, 2), (4104, 3), (8192, 4), (96, 5),
                                     (2048, 8), (4096, 6), (50, 7)])
def test_stream_boundary(device, dt, width, S):
    T, eps = 13, 2e-3
    read, write, mix, coef = boundary_weights(S)
    y, x, gain = rnd(T, width, dt=dt), 3.0 * rnd(T, S, width, seed=5), 1 + 0.3 * rnd(width, seed=6)
    want_x, want_h = boundary(y, x, read, write, mix, gain, eps)
    xd = x.to(device)
    xo, h = stream_norm(y.to(device), xd, coef.to(device), gain.to(device), eps)
    close(xo, want_x, torch.float32)
    close(h, want_h, dt)
    assert h.dtype == dt and xo.dtype == torch.float32 and (device == "cpu" or xo.data_ptr() == xd.data_ptr())
    none, h2 = stream_norm(y.to(device), x.to(device), coef.to(device), gain.to(device), eps, want_x=False)
    assert none is None and torch.equal(h2, h)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width,S", [(30, 1), (96, 3), (1024, 2), (4096, 4), (72, 8)])
def test_stream_boundaries_of_the_embedding(device, dt, width, S):
    """In front of the first sublayer nothing is written; its output is the first to make the streams differ."""
    T, eps, scale, vocab = 700, 1e-5, 12.0, 41
    read, write, mix, coef = boundary_weights(S, 9)
    table, gain = rnd(64, width, dt=dt), 1 + 0.3 * rnd(width, seed=6)
    ids = torch.randint(0, vocab, (T,), generator=torch.Generator().manual_seed(2))
    e = Embedded(table.to(device), ids.to(device), vocab, scale, S)
    streams = (table.double()[ids] * scale)[:, None].expand(T, S, width)
    x, h = stream_norm(None, e, coef.to(device), gain.to(device), eps)
    assert x is e
    close(h, boundary(None, streams, read, write, mix, gain, eps)[1], dt)
    y = rnd(T, width, dt=dt, seed=3)
    want_x, want_h = boundary(y, streams, read, write, mix, gain, eps)
    x, h = stream_norm(y.to(device), e, coef.to(device), gain.to(device), eps)
    close(x, want_x, torch.float32)
    close(h, want_h, dt)


# ------------------------------------------------------------------ norms without weights, factors per head, cache write
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 64, 64), (3, 1, 128, 40), (2, 2, 10, 3), (16, 4, 256, 128), (2, 1, 264, 8), (1, 1, 2, 1),
                                          (8, 1, 72, 136)])
@pytest.mark.parametrize("normed", [True, False])
def test_unit_norm_and_head_factors(device, dt, H, G, dim, vdim, normed):
    """Unit norms with a factor per query head, or nothing but the cache write; rows without a slot."""
    T, bs, blocks, eps = 9, 16, 5, 2e-3
    dp, vp = -(-dim // 8) * 8, -(-vdim // 8) * 8
    q, k, v = rnd(T, H, dim, dt=dt), 3.0 * rnd(T, G, dim, dt=dt, seed=3), rnd(T, G, vdim, dt=dt, seed=4)
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    qkv = torch.cat([pad(q, dp).flatten(1), pad(k, dp).flatten(1), pad(v, vp).flatten(1)], 1).to(device)
    slots = torch.tensor([16, 17, 3, 79, 0, -1, 40, 41, 33])
    temp = rnd(H, seed=8) if normed else None
    kc, vc = PagedGQABackend.views(torch.zeros_like(PagedGQABackend.allocate_pages(blocks, bs, G, dp, vp, dt, device)), bs, G, dp, vp)
    got = ops.head_norm_rope(qkv, (0, H * dp, (H + G) * dp), None, None, H, dim, None, (kc, vc), slots.to(device), eps,
                             q_scale=None if temp is None else temp.to(device), normed=normed, width=dp)
    unit = (lambda x: O.unit_rms(x.double(), eps)) if normed else (lambda x: x.double())
    close(got[..., :dim], unit(q) * (temp.double()[:, None] if normed else 1.0), dt)
    assert float(got[..., dim:].abs().sum()) == 0 and got.shape == (T, H, dp)
    assert normed or got.data_ptr() == qkv.data_ptr()
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            close(kc[s // bs, s % bs, :, :dim], unit(k)[t], dt, 2.0)
            assert torch.equal(vc[s // bs, s % bs, :, :vdim].cpu(), v[t])
    assert float(kc[2, 10:].abs().sum()) == 0


# ------------------------------------------------------------------ paged attention
ATTN = [  # H, G, dim, vdim, bs, window, chunk, options
    (4, 2, 64, 48, 64, 37, 0, dict(sigmoid=True, gate="head", slopes=True)),
    (6, 2, 40, 64, 16, 0, 50, dict(log=True, sink=True, gate="head")),
    (3, 3, 128, 128, 64, 0, 64, dict(log=True, sink=True)),
    (8, 1, 96, 104, 64, 100, 0, dict(sigmoid=True, slopes=True, gate="all")),
    (2, 1, 192, 128, 64, 64, 0, dict(sigmoid=True, slopes=True)),
    (5, 1, 184, 120, 32, 0, 96, dict(log=True, sink=True, gate="head")),
    (2, 2, 200, 160, 32, 64, 0, dict(sigmoid=True, slopes=True, gate="head")),
    (2, 2, 208, 24, 32, 0, 130, dict(log=True, sink=True, gate="head")),
    (2, 1, 264, 16, 16, 20, 0, dict(sigmoid=True, slopes=True, gate="head")),
    (2, 1, 16, 264, 16, 0, 7, dict(log=True, sink=True)),
    (1, 1, 8, 8, 16, 1, 0, dict(sigmoid=True, gate="head")),
    (1, 1, 8, 8, 16, 0, 1, dict(sink=True, gate="head")),
    (4, 4, 64, 64, 64, 40, 64, dict(sink=True)),                          # a window inside chunks
    (4, 2, 64, 64, 64, 0, 0, dict(sigmoid=True, log=300)),               # sigmoid weights of every key
    (4, 1, 48, 64, 64, 0, 100, dict(slopes=True, gate="head")),
]


def attention_case(opt, H, window, chunk):
    """Options -> (keyword arguments of the ops on the CPU, score and weigh functions of the oracle for a sequence)."""
    kw = dict(window=window or -1, chunk=chunk)
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)])
    r1, r2, shift, sink = rnd(H, seed=5).abs(), rnd(H, seed=6).abs() + 0.1, rnd(H, seed=7) - 1.0, rnd(H, seed=8)
    if opt.get("slopes"):
        kw["alibi_slopes"] = slopes
    if opt.get("log"):
        far = torch.arange(opt["log"] if opt["log"] is not True else window or chunk, dtype=torch.float64)
        kw["distance_bias"] = -(r1.double()[:, None] * torch.log1p(r2.double()[:, None] * far)).float()
    if opt.get("sigmoid"):
        kw["sigmoid_shift"] = shift
    if opt.get("sink"):
        kw["sinks"] = sink

    def oracle(n, scale):
        seen = O.causal_mask(n)
        if window:
            seen = seen & O.window_mask(n, window)
        if chunk:
            seen = seen & O.chunk_mask(n, chunk)
        bias = torch.zeros(H, n, n, dtype=torch.float64)
        if opt.get("slopes"):
            bias = bias + O.linear_bias(n, H)
        if opt.get("log"):
            bias = bias + O.log_bias(n, r1, r2)
        score = lambda h, s: s * scale - bias[h]
        if opt.get("sigmoid"):
            return score, lambda h, s: O.sigmoid_weights(s, seen, shift[h])
        return score, lambda h, s: O.softmax_weights(s, seen, sink[h] if opt.get("sink") else None)

    return kw, oracle


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,dim,vdim,bs,window,chunk,opt", ATTN)
@pytest.mark.parametrize("decode", [False, True])
def test_paged_attention(device, dt, H, G, dim, vdim, bs, window, chunk, opt, decode):
    """Prompts, portions with context and single tokens.  A key whose score stands out sits just inside and just outside the
    window or chunk, at page borders and at the first token.  The output's rows are part of wider ones."""
    lens = [1, 63, 64, 65, 130, 259, 300, 17, 101]
    new = [1] * 9 if decode else [1, 63, 1, 2, 70, 259, 130, 17, 37]
    scale = dim ** -0.5
    start = lambda i: max(0, i - window + 1) if window else i // chunk * chunk if chunk else 0
    spikes = [(1, 62, start(62)), (2, 63, max(0, start(63) - 1)), (3, 64, 63), (4, 129, start(129)), (5, 258, max(0, start(258) - 1)),
              (6, 299, 0), (7, 16, 0), (8, 100, start(100))]
    qs, ks, vs, q, kv, table, sl, qsl = paged_case(device, dt, lens, new, H, G, dim, vdim, bs, spikes, scale)
    kw, oracle = attention_case(opt, H, window, chunk)
    T = q.shape[0]
    wide = torch.zeros(T, 8 + H * vdim + 16, dtype=dt, device=device)
    out = wide[:, 8: 8 + H * vdim].unflatten(1, (H, vdim))
    gates = None
    if opt.get("gate"):
        gates = rnd(T, 8 + (H if opt["gate"] == "head" else H * vdim), seed=9, dt=dt).to(device)[:, 8:]
    kw = {k: v.to(device) if torch.is_tensor(v) else v for k, v in kw.items()}
    kw.update(out=out, max_seq_len=max(lens), gate=gates, out_scale=0.7)
    if decode:
        ops.paged_attention_decode(q, kv, table, sl, scale, **kw)
    else:
        ops.paged_attention_prefill(q, kv, table, sl, qsl, scale, max_q_len=max(new), **kw)
    want = torch.cat([O.attend(qs[b].double(), ks[b].double(), vs[b].double(), *oracle(n, scale))[n - new[b]:]
                      for b, n in enumerate(lens)])
    if gates is not None:
        want = want * O.sigmoid(gates.cpu().double()).view(T, H, -1)
    close(out, 0.7 * want, dt, 2.0)
    assert float(wide[:, :8].abs().sum()) == 0 and float(wide[:, 8 + H * vdim:].abs().sum()) == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("window,chunk,opt", [(1500, 0, dict(sigmoid=True, slopes=True, gate=True)), (0, 1200, dict(log=True, sink=True, gate=True)),
                                              (0, 0, dict(sigmoid=True))])
def test_split_decoding_far_back(dt, window, chunk, opt):
    """Few requests with long contexts: the keys are split over CTAs, whose parts meet the sink, gate and factor once."""
    lens = [2000, 1537, 31]
    H, G, dim, vdim = 4, 2, 64, 56
    first = max(0, 2000 - window) if window else 1999 // chunk * chunk if chunk else 0
    qs, ks, vs, q, kv, table, sl, _ = paged_case("cuda", dt, lens, [1, 1, 1], H, G, dim, vdim, 64,
                                                 [(0, 1999, first), (1, 1536, 1536 - 300)], dim ** -0.5)
    kw, oracle = attention_case(opt, H, window, chunk)
    gates = rnd(3, H, seed=9, dt=dt).cuda() if opt.get("gate") else None
    got = [ops.paged_attention_decode(q, kv, table, sl, dim ** -0.5, max_seq_len=2000, gate=gates, out_scale=1.3, num_splits=n,
                                      **{k: v.cuda() if torch.is_tensor(v) else v for k, v in kw.items()}) for n in (0, 1, 3)]
    want = 1.3 * torch.cat([O.attend(qs[b].double(), ks[b].double(), vs[b].double(), *oracle(n, dim ** -0.5))[-1:]
                            for b, n in enumerate(lens)])
    if gates is not None:
        want = want * O.sigmoid(gates.cpu().double())[:, :, None]
    for g in got:
        close(g, want, dt, 2.0)


@pytest.mark.parametrize("device", DEVICES)
def test_large_sigmoid_scores(device):
    """Scores far beyond the exponent range: weights of exactly nothing and of one."""
    H, D, bs, n = 2, 64, 64, 130
    dt = torch.bfloat16
    qs, ks, vs, q, kv, table, sl, qsl = paged_case(device, dt, [n], [n], H, 1, D, D, bs)
    shift = torch.tensor([400.0, -900.0])
    out = ops.paged_attention_prefill(q, kv, table, sl, qsl, 1.0, max_q_len=n, max_seq_len=n, sigmoid_shift=shift.to(device))
    one = ops.paged_attention_decode(q[-1:], kv, table, sl, 1.0, max_seq_len=n, sigmoid_shift=shift.to(device))
    sums = vs[0].double().cumsum(0)[:, 0]
    close(out[:, 0], sums, dt)
    close(one[:, 0], sums[-1:], dt)
    assert float(out[:, 1].abs().max()) < 1e-12 and float(one[:, 1].abs().max()) < 1e-12


def test_split_counts_follow_what_is_seen():
    n = lambda **kw: ops.decode_num_splits(1, 2, 8192, **kw)
    assert n() > n(window=1024) == n(chunk=1024) > n(window=1024, chunk=512) == n(window=512) >= n(chunk=100) == 1


@pytest.mark.parametrize("kw,message", [
    (dict(norm="none", whole_row_norm=True), "whole rows"), (dict(norm="other"), "norm"), (dict(sigmoid=True, sinks=True), "softmax"),
    (dict(log_bias=True), "window or chunks")])
def test_attention_options_that_do_not_go_together(kw, message):
    with pytest.raises(ValueError, match=message):
        QKNormAttention(32, 2, 1, 16, 16, 1.0, 1e-6, None, 0, **kw)


# ------------------------------------------------------------------ latent pieces
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("K,R,dims", [(24, 12, 12), (30, 6, 4), (256, 64, 64), (512, 64, 64), (7, 2, 2)])
def test_latent_insert_without_a_query_latent(device, dt, K, R, dims):
    """Rotation in adjacent pairs, whole turns far from the start, rows without a slot."""
    T, base, eps, row, H = 11, 700.0, 1e-4, -(-(K + R) // 8) * 8, 3
    a, kw = rnd(T, 8 + K + R + 2, dt=dt), rnd(K, dt=dt) + 1
    pos = torch.tensor([0, 1, 2, 5, 63, 64, 65, 4095, 7, 70000, 3])
    slots = torch.tensor([5, 4, -1, 63, 64, 0, 30, 31, 32, 33, -1])
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    angles = ops.rope_angles(pos.to(device), freq.to(device), T)
    cache = torch.full((5, 16, row), 9.0, dtype=dt, device=device)
    assert ops.latent_insert(a.to(device), 0, 8, None, kw.to(device), R, angles, cache, slots.to(device), eps, interleaved=True) is None
    x, rows = a.double(), torch.zeros(T, row, dtype=torch.float64)
    rows[:, :K] = O.unit_rms(x[:, 8: 8 + K], eps) * kw.double()
    rows[:, K: K + R] = O.rotate_pairs(x[:, None, 8 + K: 8 + K + R], pos, dims, base)[:, 0]
    ok, flat = slots >= 0, cache.view(80, row).cpu()
    close(flat[slots[ok]], rows[ok], dt)
    rest = torch.ones(80, dtype=torch.bool)
    rest[slots[ok]] = False
    assert bool((flat[rest] == 9.0).all())
    q = rnd(T, H, R + 5, dt=dt).to(device)
    dst = torch.full((T, H, R + 4), 9.0, dtype=dt, device=device)
    ops.latent_rope(dst, q[..., 5:], angles, R, 3, interleaved=True)
    close(dst[..., :R], O.rotate_pairs(q[..., 5:].cpu().double(), pos, dims, base), dt)
    assert bool((dst[..., R: R + 3] == 0).all()) and bool((dst[..., R + 3:] == 9.0).all())


# ------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W,ff", [(1, 48, 40), (9, 50, 13), (300, 264, 520)])
def test_squared_relu_mlp(device, dt, T, W, ff):
    from vllm_metax_b200.models.vetipel import SquaredReluMLP

    w = {"up": rnd(ff, W, dt=dt, scale=W ** -0.5), "down": rnd(W, ff, dt=dt, scale=ff ** -0.5)}
    mlp = SquaredReluMLP(W, ff, dt).to(device)
    for k, dst in mlp.slots().items():
        dst.copy_(w[k])
    h = rnd(T, W, dt=dt, seed=4)
    close(mlp(h.to(device)), O.dense(h.double(), w, ""), dt, 2.0)
