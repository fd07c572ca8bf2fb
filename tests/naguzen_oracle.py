"""Plain statement of the Naguzen decoder, one function per mechanism, whole sequences at a time, in float64 on the CPU.

Nothing here uses the package: the tests compare the package with these functions.  ``w`` maps checkpoint tensor names
to tensors and ``cfg`` is the checkpoint's ``config.json`` as a dict.  Recurrences walk the tokens one by one,
attention builds the full score matrix of a head, convolutions sum their taps.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def get(w, name):
    return w[name].to(F64)


def linear(w, name, x):
    return x @ get(w, name).t()


# ------------------------------------------------------------------ elementwise pieces
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def xielu(z, p, q):
    p, q = torch.as_tensor(p, dtype=F64), torch.as_tensor(q, dtype=F64)
    pos = softplus(p) * z * z + 0.5 * z
    neg = (0.5 + softplus(q)) * (torch.exp(torch.clamp(z, max=0)) - 1.0 - z) + 0.5 * z
    return torch.where(z > 0, pos, neg)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(x, taps):
    """``x [T, C]``, ``taps [C, K]`` (last column = the current token), zeros before the start."""
    T, C = x.shape
    K = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return out


def rotate(x, positions, dims, base):
    """Rotate-half rotation of the first ``dims`` entries of the last axis; ``x [T, ..., D]``."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        a = positions.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a), torch.sin(a)
        shape = [x.shape[0]] + [1] * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ------------------------------------------------------------------ mixers
def window_attention(q, k, v, scale, window):
    """``q, k [T, H, D]``, ``v [T, H, Dv]``; token i sees j with 0 <= i - j < window."""
    T, H, _ = q.shape
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    seen = (dist >= 0) & (dist < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h].t()) * scale
        s = s.masked_fill(~seen, float("-inf"))
        s = s - s.max(-1, keepdim=True).values
        e = torch.exp(s)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, h]
    return out


def latent_attention(h, w, pre, m, eps):
    T, H = h.shape[0], m["heads"]
    dim, rd, vd, r = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = unit_rms(linear(w, pre + "dq", h), eps) * get(w, pre + "dq.norm")
    q = linear(w, pre + "uq", cq).view(T, H, dim + rd)
    kv = linear(w, pre + "dkv", h)
    c = unit_rms(kv[:, :r], eps) * get(w, pre + "dkv.norm")
    pos = torch.arange(T)
    kr = rotate(kv[:, r:], pos, m["rot"]["dims"], m["rot"]["base"])
    qr = rotate(q[..., dim:], pos, m["rot"]["dims"], m["rot"]["base"])
    q = torch.cat([q[..., :dim], qr], -1)
    k = torch.cat([linear(w, pre + "uk", c).view(T, H, dim), kr[:, None].expand(T, H, rd)], -1)
    v = linear(w, pre + "uv", c).view(T, H, vd)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"])
    return linear(w, pre + "o", o.reshape(T, H * vd))


def gated_linear_recurrence(q, k, v, alpha):
    """``q, k, alpha [T, H, dim]``, ``v [T, H, vdim]``: per head S = diag(alpha) S + k v^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def gla(h, w, pre, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(w, pre + "q", h).view(T, H, D) * D ** -0.5
    k = linear(w, pre + "k", h).view(T, H, D)
    v = linear(w, pre + "v", h).view(T, H, V)
    z = linear(w, pre + "a2", linear(w, pre + "a1", h)) + get(w, pre + "a2.b")
    alpha = sigmoid(z).view(T, H, D) ** (1.0 / m["tau"])
    o = gated_linear_recurrence(q, k, v, alpha)
    o = unit_rms(o, eps) * get(w, pre + "norm")
    g = linear(w, pre + "g", h)
    return linear(w, pre + "o", o.reshape(T, H * V) * g * sigmoid(g))


def rglru(h, w, pre, m, eps):
    T, B = h.shape[0], m["blocks"]
    y = gelu_tanh(linear(w, pre + "y", h) + get(w, pre + "y.b"))
    u = causal_conv(linear(w, pre + "x", h) + get(w, pre + "x.b"), get(w, pre + "conv")) + get(w, pre + "conv.b")
    ub = u.view(T, B, -1)
    gate = {}
    for n in ("ra", "ri"):
        gate[n] = torch.stack([sigmoid(ub[:, b] @ get(w, pre + n)[b].t() + get(w, pre + n + ".b")[b])
                               for b in range(B)], 1).reshape(T, -1)
    log_a = -8.0 * gate["ra"] * softplus(get(w, pre + "lam"))
    a = torch.exp(log_a)
    inp = torch.sqrt(-torch.expm1(2.0 * log_a)) * gate["ri"] * u
    S = torch.zeros(u.shape[1], dtype=F64)
    out = torch.zeros_like(u)
    for t in range(T):
        S = a[t] * S + inp[t]
        out[t] = S
    return linear(w, pre + "o", out * y)


MIXERS = {"latent_attention": latent_attention, "gla": gla, "rglru": rglru}


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, w, pre):
    p, q = get(w, pre + "act")
    return linear(w, pre + "down", xielu(linear(w, pre + "up", h), p, q))


def route(h, w, pre, r):
    s = sigmoid(linear(w, pre + "router", h))
    val, idx = s.topk(r["top"], -1)
    return val * r["scale"], idx


def moe_ff(h, w, pre, m):
    val, idx = route(h, w, pre, m["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for weight, e in zip(val[t], idx[t].tolist()):
            out[t] += weight * linear(w, f"{pre}e{e}.down", gelu_erf(linear(w, f"{pre}e{e}.up", h[t])))
    if m.get("shared"):
        out = out + linear(w, pre + "shared.down", gelu_erf(linear(w, pre + "shared.up", h)))
    return out


# ------------------------------------------------------------------ the model
def scalar_norm(x, g, eps):
    return unit_rms(x, eps) * g


def layer(x, w, i, spec, eps):
    pre = f"l{i}."
    h = x + causal_conv(x, get(w, pre + "canon1"))
    x = x + scalar_norm(MIXERS[spec["type"]](h, w, pre + "mix.", spec["mixer"], eps), get(w, pre + "norm1"), eps)
    if spec["mlp"] is None:
        return x
    h = x + causal_conv(x, get(w, pre + "canon2"))
    y = dense_ff(h, w, pre + "mlp.") if spec["mlp"]["kind"] == "dense" else moe_ff(h, w, pre + "mlp.", spec["mlp"])
    return x + scalar_norm(y, get(w, pre + "norm2"), eps)


def forward(tokens, w, cfg, want_layers=False):
    """Logits ``[T, vocab]`` of one sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = get(w, "embed")[torch.as_tensor(tokens, dtype=torch.long)]
    layers = []
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, eps)
        layers.append(x)
    logits = linear(w, "head", scalar_norm(x, get(w, "final.norm"), eps))
    return (logits, layers) if want_layers else logits


# ------------------------------------------------------------------ random checkpoints
def tensor_shapes(cfg):
    """Name -> shape of every tensor a checkpoint of ``cfg`` holds (the decay's low rank from ``cfg["decay_rank"]``,
    a key only the tests use)."""
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": ()}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        s[p + "norm1"], s[p + "canon1"] = (), (W, taps)
        if l["type"] == "latent_attention":
            H = m["heads"]
            s.update({p + "mix.dq": (m["q_rank"], W), p + "mix.dq.norm": (m["q_rank"],),
                      p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                      p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], W), p + "mix.dkv.norm": (m["kv_rank"],),
                      p + "mix.uk": (H * m["dim"], m["kv_rank"]), p + "mix.uv": (H * m["vdim"], m["kv_rank"]),
                      p + "mix.o": (W, H * m["vdim"])})
        elif l["type"] == "gla":
            H, D, VD, R = m["heads"], m["dim"], m["vdim"], cfg.get("decay_rank", 8)
            s.update({p + "mix.q": (H * D, W), p + "mix.k": (H * D, W), p + "mix.v": (H * VD, W),
                      p + "mix.g": (H * VD, W), p + "mix.o": (W, H * VD), p + "mix.norm": (VD,),
                      p + "mix.a1": (R, W), p + "mix.a2": (H * D, R), p + "mix.a2.b": (H * D,)})
        else:
            U, B = m["width"], m["blocks"]
            b = U // B
            s.update({p + "mix.y": (U, W), p + "mix.y.b": (U,), p + "mix.x": (U, W), p + "mix.x.b": (U,),
                      p + "mix.conv": (U, m["conv"]), p + "mix.conv.b": (U,), p + "mix.ra": (B, b, b),
                      p + "mix.ra.b": (B, b), p + "mix.ri": (B, b, b), p + "mix.ri.b": (B, b), p + "mix.lam": (U,),
                      p + "mix.o": (W, U)})
        f = l["mlp"]
        if f is None:
            continue
        s[p + "norm2"], s[p + "canon2"] = (), (W, taps)
        if f["kind"] == "dense":
            s.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"]), p + "mlp.act": (2,)})
        else:
            E, I = f["router"]["experts"], f["expert"]["ff"]
            s[p + "mlp.router"] = (E, W)
            for e in range(E):
                s[f"{p}mlp.e{e}.up"], s[f"{p}mlp.e{e}.down"] = (I, W), (W, I)
            if f.get("shared"):
                s[p + "mlp.shared.up"], s[p + "mlp.shared.down"] = (f["shared"]["ff"], W), (W, f["shared"]["ff"])
    return s


def random_weights(cfg, seed=0):
    """Weights at which every path carries signal: unit-gain projections, decays from fast to slow, gains about 1."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        n = torch.randn(shape, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.25 * n
        elif leaf == "act":
            t = 0.5 * n
        elif leaf in ("canon1", "canon2", "conv"):
            t = 0.35 * n
        elif leaf == "lam":
            t = -2.0 + 1.5 * n
        elif name.endswith("a2.b"):
            t = 2.0 + 2.0 * n
        elif leaf == "b":
            t = 0.3 * n
        elif leaf == "embed":
            t = n
        else:
            t = n * shape[-1] ** -0.5
            if leaf == "router":
                t = 2.0 * t
        w[name] = t.to(torch.bfloat16)
    # the experts of a layer are variations of one: where rounding decides between two of equal score, the output moves
    # little (a wrong expert still stands far above the fp32 limits)
    for name in w:
        head, _, leaf = name.rpartition(".")
        if ".mlp.e" in name and not head.endswith(".e0"):
            first = head[: head.rindex(".e")] + ".e0." + leaf
            w[name] = (w[first].float() + 0.25 * w[name].float()).to(torch.bfloat16)
    return w
