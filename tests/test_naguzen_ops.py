"""Every mechanism of the Naguzen decoder alone, against the plain float64 statement in ``naguzen_oracle.py``: on the CPU
(the PyTorch statements of the ops) and on the GPU (the kernels), in fp32 and bf16."""
import pytest
import torch

from tests import naguzen_oracle as O
from vllm_metax_b200 import _custom_ops as ops
from vllm_metax_b200.ops.gdn import causal_conv1d
from vllm_metax_b200.ops.gla import gated_linear_attention
from vllm_metax_b200.ops.residual_conv import residual_conv
from vllm_metax_b200.ops.residual_norm import residual_norm
from vllm_metax_b200.ops.rglru import rglru

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


def split_steps(lens, cuts):
    """Sequences of ``lens`` tokens cut at ``cuts`` -> per step the (sequence, lo, hi) it brings."""
    edges = [0] + sorted(cuts) + [max(lens)]
    for lo, hi in zip(edges[:-1], edges[1:]):
        yield [(s, lo, min(hi, n)) for s, n in enumerate(lens) if lo < n]


def step_args(step, slots, dev):
    qsl = [0]
    for _, lo, hi in step:
        qsl.append(qsl[-1] + hi - lo)
    return i32(qsl, dev), i32([slots[s] for s, _, _ in step], dev), i32([int(lo > 0) for _, lo, _ in step], dev)


LENS, CUTS = [1, 5, 40, 91], [1, 2, 4, 7, 23, 24, 40, 63]
SLOTS = [3, 0, 4, 1]


# ------------------------------------------------------------------ boundary: residual + norm + convolution
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width,taps,per_channel", [(48, 4, False), (37, 3, False), (264, 1, True), (2056, 2, False),
                                                    (4608, 5, False), (72, 8, True)])
def test_residual_conv_over_portions(device, dt, width, taps, per_channel):
    eps = 3e-3
    w, gain = rnd(width, taps, dt=dt, scale=0.5), rnd(width if per_channel else 1, dt=dt) + 1
    ys = [rnd(n, width, dt=dt, seed=n) for n in LENS]
    xs = [rnd(n, width, seed=100 + n) for n in LENS]
    want_x = [x.double() + O.unit_rms(y.double(), eps) * gain.double() for x, y in zip(xs, ys)]
    want_h = [x + O.causal_conv(x, w.double()) for x in want_x]
    carry = rnd(6, taps - 1, width).to(device)            # old contents of freed slots must not leak in
    wd, gd = w.to(device), gain.to(device)
    for step in split_steps(LENS, CUTS):
        qsl, idx, init = step_args(step, SLOTS, device)
        y = torch.cat([ys[s][lo:hi] for s, lo, hi in step]).to(device)
        x = torch.cat([xs[s][lo:hi] for s, lo, hi in step]).to(device)
        xo, h = residual_conv(y, x, gd, wd, eps, carry, qsl, idx, init)
        close(xo, torch.cat([want_x[s][lo:hi] for s, lo, hi in step]), torch.float32)
        close(h, torch.cat([want_h[s][lo:hi] for s, lo, hi in step]), dt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width", [40, 51, 3000, 6000])
def test_first_and_last_boundary(device, dt, width):
    eps = 1e-4
    y, x = rnd(9, width, dt=dt), rnd(9, width, seed=5)
    g1, g2 = rnd(1, dt=dt) + 1, rnd(1, dt=dt, seed=9) + 2
    w = rnd(width, 3, dt=dt)
    xo, h = residual_conv(y.to(device), None, None, w.to(device), eps, None, i32([0, 9], device))
    close(xo, y.double(), torch.float32)
    close(h, y.double() + O.causal_conv(y.double(), w.double()), dt)
    want = O.scalar_norm(x.double() + O.scalar_norm(y.double(), g1.double(), eps), g2.double(), eps)
    close(residual_norm(y.to(device), x.to(device), g1.to(device), g2.to(device), eps), want, dt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 5])
def test_short_convolution_over_portions(device, dt, taps):
    C = 72
    w, b = rnd(C, taps, dt=dt), rnd(C, dt=dt)
    xs = [rnd(n, C, dt=dt, seed=n) for n in LENS]
    state = rnd(6, taps - 1, C, dt=dt).to(device)
    for step in split_steps(LENS, CUTS):
        qsl, idx, init = step_args(step, SLOTS, device)
        x = torch.cat([xs[s][lo:hi] for s, lo, hi in step]).to(device)
        got = causal_conv1d(x, w.to(device), b.to(device), state, qsl, idx, init, silu=False)
        want = torch.cat([(O.causal_conv(xs[s].double(), w.double()) + b.double())[lo:hi] for s, lo, hi in step])
        close(got, want, dt)


# ------------------------------------------------------------------ recurrences
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,V,tau,long", [(3, 20, 12, 9.0, 0), (2, 64, 48, 16.0, 0), (1, 33, 7, 1.0, 0), (2, 96, 136, 4.0, 0),
                                            (1, 130, 40, 16.0, 0), (1, 250, 260, 2.0, 0), (2, 40, 24, 16.0, 1),
                                            (1, 33, 150, 200.0, 1), (1, 170, 30, 50.0, 1)])
def test_gated_linear_attention_over_portions(device, dt, H, D, V, tau, long):
    """``long``: portions of several segments beside short ones (edges at 256 tokens), slow decays."""
    eps = 1e-5
    lens, cuts = ([300, 1, 800, 257], [1, 2, 258, 262, 775]) if long else (LENS, CUTS)
    widths = [H * D, H * D, H * V, H * V]
    off = [8, 8 + widths[0], 8 + 2 * widths[0], 8 + 2 * widths[0] + widths[2]]
    rows = [rnd(n, off[3] + widths[3] + 5, dt=dt, seed=n) for n in lens]
    zs = [O.sigmoid(rnd(n, H * D, seed=50 + n).double() * 2 + 3) ** (1 / tau) for n in lens]
    nw = rnd(V, dt=dt) + 1
    want = []
    for r, z in zip(rows, zs):
        n, p = r.shape[0], r.double()
        part = lambda i, w: p[:, off[i]: off[i] + widths[i]].reshape(n, H, w)
        alpha = z.float().double().view(n, H, D)
        o = O.gated_linear_recurrence(part(0, D) * D ** -0.5, part(1, D), part(2, V), alpha)
        g = p[:, off[3]: off[3] + widths[3]]
        want.append((O.unit_rms(o, eps) * nw.double()).reshape(n, H * V) * g * O.sigmoid(g))
    state = rnd(6, H, D, V).to(device)
    for step in split_steps(lens, cuts):
        qsl, idx, init = step_args(step, SLOTS, device)
        x = torch.cat([rows[s][lo:hi] for s, lo, hi in step]).to(device)
        z = torch.cat([zs[s][lo:hi] for s, lo, hi in step]).float().to(device)
        got = gated_linear_attention(x, off, z, nw.to(device), state, qsl, idx, init, D ** -0.5, eps,
                                     max(hi - lo for _, lo, hi in step))
        close(got, torch.cat([want[s][lo:hi] for s, lo, hi in step]), dt, 2.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("width,blocks", [(120, 3), (35, 1), (72, 9)])
def test_rglru_over_portions(device, dt, width, blocks):
    lens = [1, 70, 200, 333]
    us, ys = [rnd(n, width, dt=dt, seed=n) for n in lens], [rnd(n, width, dt=dt, seed=9 + n) for n in lens]
    zs = [rnd(n, blocks, 2, width // blocks, seed=70 + n) for n in lens]
    rb, ib, lam = rnd(width), rnd(width, seed=3), rnd(width, seed=4) * 2 - 3
    decay = -8.0 * torch.nn.functional.softplus(lam)
    want = []
    for u, y, z in zip(us, ys, zs):
        n = u.shape[0]
        r = O.sigmoid(z[:, :, 0].reshape(n, width).double() + rb.double())
        i = O.sigmoid(z[:, :, 1].reshape(n, width).double() + ib.double())
        la = -8.0 * r * O.softplus(lam.double())
        S, out = torch.zeros(width, dtype=torch.float64), []
        for t in range(n):
            S = torch.exp(la[t]) * S + torch.sqrt(1 - torch.exp(2 * la[t])) * i[t] * u[t].double()
            out.append(S * O.gelu_tanh(y[t].double()))
        want.append(torch.stack(out))
    state = rnd(6, width).to(device)
    for step in split_steps(lens, [1, 2, 66, 67, 131, 300, 301]):
        qsl, idx, init = step_args(step, SLOTS, device)
        cat = lambda a: torch.cat([a[s][lo:hi] for s, lo, hi in step]).to(device)
        got = rglru(cat(us), cat(ys), cat(zs).contiguous(), rb.to(device), ib.to(device), decay.to(device), state, qsl, idx,
                    init, max(hi - lo for _, lo, hi in step))
        close(got, torch.cat([want[s][lo:hi] for s, lo, hi in step]), dt)


# ------------------------------------------------------------------ products and their epilogues
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 40, 24), (7, 203, 96), (33, 1288, 1040), (64, 520, 2048), (200, 264, 72),
                                   (300, 1032, 1024), (1100, 2056, 136), (50, 33, 30), (5, 64, 16)])
def test_product_epilogues(device, dt, M, N, K):
    a, w = rnd(M, K, dt=dt), rnd(N, K, dt=dt, scale=K ** -0.5)
    p, q = 0.3, -0.8
    coef = torch.tensor([float(O.softplus(torch.tensor(p))), 0.5 + float(O.softplus(torch.tensor(q)))], device=device)
    z = a.double() @ w.double().t()
    ad, wd = a.to(device), w.to(device)
    close(ops.gemm(ad, wd), z, dt)
    close(ops.gemm(ad, wd, act="gelu"), O.gelu_erf(z), dt)
    close(ops.gemm(ad, wd, act="gelu_tanh"), O.gelu_tanh(z), dt)
    close(ops.gemm(ad, wd, act="xielu", act_params=coef), O.xielu(z, p, q), dt)
    b = rnd(N, dt=dt) + 2
    y = ops.gemm(ad, wd, b.to(device), act="decay", act_params=torch.full((1,), 1 / 16, device=device), out_dtype=torch.float32)
    close(y, O.sigmoid(z + b.double()) ** (1 / 16), torch.float32)
    y = ops.gemm(ad, wd, out_dtype=torch.float32)
    assert y.dtype == torch.float32
    close(y, z, torch.float32)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("Z,M,N,K", [(3, 1, 80, 40), (5, 9, 136, 24), (2, 60, 64, 128), (4, 150, 200, 72), (3, 77, 10, 9),
                                     (1, 260, 48, 16)])
def test_batched_product_on_strided_views(device, dt, Z, M, N, K):
    a = rnd(M, Z, K + 8, dt=dt).to(device)[..., :K].transpose(0, 1)          # [Z, M, K], rows of another pitch
    w = rnd(Z, N, K, dt=dt).to(device)
    want = torch.einsum("zmk,znk->zmn", a.double().cpu(), w.double().cpu())
    for out_dt in {dt, torch.float32}:
        buf = torch.full((M, Z, N + 8), 7.0, dtype=out_dt, device=device)
        ops.gemm_batched(a, w, out=buf[..., :N].transpose(0, 1))
        close(buf[..., :N].transpose(0, 1), want, out_dt)
        assert bool((buf[..., N:] == 7.0).all()), "columns behind the result were written"


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W,E,I,top,scale,shared", [(1, 96, 6, 40, 2, 0.7, 0), (37, 72, 5, 24, 1, 2.5, 48),
                                                      (300, 136, 33, 16, 7, 1.0, 8), (9, 50, 4, 18, 4, 1.3, 20)])
def test_routed_experts(device, dt, T, W, E, I, top, scale, shared):
    from vllm_metax_b200.models.naguzen import RoutedExperts

    spec = {"kind": "moe", "router": {"experts": E, "top": top, "scale": scale}, "expert": {"ff": I},
            "shared": {"ff": shared} if shared else None}
    cfg = {"vocab": 8, "width": W, "canon": {"taps": 1}, "norm": {"eps": 1e-6},
           "layers": [{"type": "rglru", "mixer": {"width": 8, "blocks": 1, "conv": 1}, "mlp": spec}]}
    w = O.random_weights(cfg, seed=T)
    with torch.device(device):
        m = RoutedExperts(W, spec, dt, "x")
    for k, dst in m.slots().items():
        dst.copy_(w["l0.mlp." + k])
    h = rnd(T, W, dt=dt)
    s = O.sigmoid(O.linear(w, "l0.mlp.router", h.double())).sort(-1, descending=True).values
    gap = s[:, top - 1] - s[:, top] if top < E else torch.ones(T)
    sure = gap > 1e-3                                        # rounding may decide between two equal experts
    got = m(h.to(device)).cpu()
    close(got[sure], O.moe_ff(h.double(), w, "l0.mlp.", spec)[sure], dt)


# ------------------------------------------------------------------ latent attention
def needle(T, H, D, pairs, seed=0, dt=torch.float32):
    """Queries and keys of small scores, except that query i meets key j with a score far above the rest."""
    q, k = rnd(T, H, D, seed=seed) * 0.3, rnd(T, H, D, seed=seed + 1) * 0.3
    for n, (i, j) in enumerate(pairs):
        d = torch.nn.functional.normalize(rnd(H, D, seed=100 + n), dim=-1) * 6
        q[i], k[j] = d, d
    return q.to(dt), k.to(dt)


@pytest.mark.gpu
@pytest.mark.parametrize("dqk,dv,H", [(32, 24, 3), (72, 64, 2), (96, 128, 5), (136, 40, 1), (192, 128, 2), (64, 64, 4)])
@pytest.mark.parametrize("window", [1, 17, 128, 1000])
def test_prompt_attention_sizes_and_windows(dqk, dv, H, window):
    T = 300
    inside = [(i, i - window + 1) for i in (window - 1, 130, 257, 299) if i < T and i >= window - 1]
    outside = [(i, i - window) for i in (window + 1, 200, 290) if i < T and i >= window]
    for pairs in (inside, outside):
        q, k = needle(T, H, dqk, pairs, dt=torch.bfloat16)
        v = rnd(T, H, dv, dt=torch.bfloat16)
        kv = torch.zeros(T, H, dqk + dv + 8, dtype=torch.bfloat16)
        kv[..., :dqk], kv[..., dqk: dqk + dv] = k, v
        kv = kv.cuda()
        want = O.window_attention(q.double(), k.double(), v.double(), 0.5, window)
        for lo in (0, 1, 128, 298):                          # the last T - lo tokens as queries over all keys
            cq, ck = i32([0, T - lo], "cuda"), i32([0, T], "cuda")
            got = ops.varlen_attention(q[lo:].cuda(), kv[..., :dqk], kv[..., dqk: dqk + dv], cq, ck, 0.5, window=window)
            close(got, want[lo:], torch.bfloat16, 2.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,K,R", [(3, 24, 12), (20, 64, 32), (40, 136, 16), (2, 30, 6), (5, 256, 64), (1, 512, 64),
                                   (33, 512, 8)])
@pytest.mark.parametrize("window", [1, 33, 600])
def test_absorbed_attention_over_pages(device, dt, H, K, R, window):
    """Decode rows and short portions over a paged latent cache whose pages are scattered; a key stands out just inside
    and just outside the window, and on both sides of a page border."""
    bs, row = 16, -(-(K + R) // 8) * 8
    lens, new = [1, 17, 70, 333], [1, 2, 1, 5]
    pages = torch.randperm(64, generator=torch.Generator().manual_seed(1))
    cache = torch.full((64, bs, row), float("nan"), dtype=dt)
    table = torch.zeros(4, 24, dtype=torch.int32)
    qs, want, n = [], [], 0
    for b, (L, m) in enumerate(zip(lens, new)):
        last = L - 1
        pairs = [(last, max(0, last - window + 1))] if b % 2 else [(last, max(0, last - window))]
        q, k = needle(L, H, K + R, pairs, seed=b, dt=dt)
        k = k[:, :1]                                         # one key per token, shared by the heads
        if pairs:
            q[last] = k[pairs[0][1]]
        nb = -(-L // bs)
        table[b, :nb] = pages[n: n + nb].int()
        n += nb
        flat = torch.zeros(nb * bs, row, dtype=dt)
        flat[:L, : K + R] = k[:, 0]
        flat[L:] = float("nan") if device == "cpu" else 0.0
        cache[table[b, :nb].long()] = flat.view(nb, bs, row)
        o = O.window_attention(q.double(), k.double().expand(L, H, K + R), k[..., :K].double().expand(L, H, K), 0.4, window)
        qa = torch.zeros(m, H, row, dtype=dt)
        qa[..., : K + R] = q[L - m:]
        qs.append(qa)
        want.append(o[L - m:])
    qsl = [0]
    for m in new:
        qsl.append(qsl[-1] + m)
    args = (torch.cat(qs).to(device), cache.to(device), table.to(device), i32(lens, device), 0.4)
    for splits in (1, 3) if device == "cuda" and dt != torch.float32 else (1,):
        got = ops.mla_decode(*args, query_start_loc=i32(qsl, device), max_seq_len=max(lens), window=window, kv_rank=K,
                             num_splits=splits)
        close(got, torch.cat(want), dt, 2.0)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("QR,K,R,dims", [(40, 24, 12, 12), (129, 30, 6, 4), (512, 256, 64, 64)])
def test_latent_insert_and_rotation(device, dt, QR, K, R, dims):
    T, base, eps, row = 11, 700.0, 1e-4, -(-(K + R) // 8) * 8
    kv_off = QR + 3
    a, qw, kw = rnd(T, kv_off + K + R + 2, dt=dt), rnd(QR, dt=dt) + 1, rnd(K, dt=dt) + 1
    pos = torch.tensor([0, 1, 2, 5, 63, 64, 65, 4095, 7, 70000, 3])
    slots = torch.tensor([5, 4, -1, 63, 64, 0, 30, 31, 32, 33, -1])
    freq = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    angles = ops.rope_angles(pos.to(device), freq.to(device), T)
    cache = torch.full((5, 16, row), 9.0, dtype=dt, device=device)
    cq = ops.latent_insert(a.to(device), 0, kv_off, qw.to(device), kw.to(device), R, angles, cache, slots.to(device), eps)
    x = a.double()
    close(cq, O.unit_rms(x[:, :QR], eps) * qw.double(), dt)
    want = torch.full((80, row), 9.0, dtype=torch.float64)
    rows = torch.zeros(T, row, dtype=torch.float64)
    rows[:, :K] = O.unit_rms(x[:, kv_off: kv_off + K], eps) * kw.double()
    rows[:, K: K + R] = O.rotate(x[:, kv_off + K: kv_off + K + R], pos, dims, base)
    want[slots[slots >= 0]] = rows[slots >= 0]
    flat = cache.view(80, row).cpu()
    close(flat[slots[slots >= 0]], want[slots[slots >= 0]], dt)
    rest = torch.ones(80, dtype=torch.bool)
    rest[slots[slots >= 0]] = False
    assert bool((flat[rest] == 9.0).all())
    q = rnd(T, 3, R + 5, dt=dt).to(device)
    dst = torch.full((T, 3, R + 4), 9.0, dtype=dt, device=device)
    ops.latent_rope(dst, q[..., 5:], angles, R, 3)
    close(dst[..., :R].cpu(), O.rotate(q[..., 5:].cpu().double(), pos, dims, base), dt)
    assert bool((dst[..., R: R + 3] == 0).all()) and bool((dst[..., R + 3:] == 9.0).all())
