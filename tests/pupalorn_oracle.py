"""Plain statement of the Pupalorn decoder, one function per mechanism, whole sequences at a time, in float64 on the CPU.

Nothing here uses the package: the tests compare the package with these functions.  ``w`` maps checkpoint tensor names to
tensors and ``cfg`` is the checkpoint's ``config.json`` as a dict.  Attention builds the full score matrix of a head, experts
run token by token, rotations pair by pair.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def get(w, name):
    return w[name].to(F64)


def linear(w, name, x):
    return x @ get(w, name).t()


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, g, eps):
    """RMS norm whose stored weight is the gain's distance from one."""
    return unit_rms(x, eps) * (1.0 + g.to(F64))


# ------------------------------------------------------------------ rotation
def frequencies(dims, base, scaling=None):
    """base^(-2i/dims); with ``scaling`` long wavelengths are slowed down by ``factor``, short ones kept, blended between."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            wave, n = 2.0 * math.pi / f, float(scaling["original"])
            lo, hi, k = float(scaling["low"]), float(scaling["high"]), float(scaling["factor"])
            if wave > n / lo:
                f = f / k
            elif wave >= n / hi:
                s = (n / wave - lo) / (hi - lo)
                f = (1.0 - s) * f / k + s * f
        out.append(f)
    return out


def rotate(x, positions, dims, freqs):
    """Rotate-half rotation of the first ``dims`` entries of the last axis; ``x [T, heads, D]``."""
    half = dims // 2
    out = x.clone()
    for i, f in enumerate(freqs):
        a = (positions.to(F64) * f)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ------------------------------------------------------------------ attention
def attend(q, k, v, scale, window=0):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``: query head h reads key head h // (H / G); token i sees j with
    0 <= i - j < window (no lower bound without a window)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    seen = (dist >= 0) if not window else (dist >= 0) & (dist < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].t()) * scale).masked_fill(~seen, float("-inf"))
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, g]
    return out


def project_kv(h, w, pre, m, eps):
    """Keys (normed and rotated) and values of a layer that has its own."""
    T, G, r = h.shape[0], m["kv_heads"], m["rot"]
    k = linear(w, pre + "k", h).view(T, G, m["dim"])
    k = unit_rms(k, eps) * get(w, pre + "k.norm")
    k = rotate(k, torch.arange(T), r["dims"], frequencies(r["dims"], r["base"], r.get("scaling")))
    return k, linear(w, pre + "v", h).view(T, G, m["vdim"])


def attention(h, w, pre, m, eps, shared=None):
    """Returns the mixer's output and the keys and values it read (``shared`` = another layer's)."""
    T, r = h.shape[0], m["rot"]
    q = linear(w, pre + "q", h).view(T, m["heads"], m["dim"])
    q = unit_rms(q, eps) * get(w, pre + "q.norm")
    q = rotate(q, torch.arange(T), r["dims"], frequencies(r["dims"], r["base"], r.get("scaling")))
    k, v = shared if shared is not None else project_kv(h, w, pre, m, eps)
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size") or 0)
    return linear(w, pre + "o", o.reshape(T, -1)), (k, v)


# ------------------------------------------------------------------ experts
def choose(z, correction, top):
    """Router logits ``[n]`` -> [(expert, weight)]: softmax scores over all outputs, the correction moves the choice only,
    weights as they are."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    order = sorted(range(z.numel()), key=lambda e: (-float(s[e] + correction[e]), e))
    return [(e, float(s[e])) for e in order[:top]]


def relu_squared(z):
    return torch.clamp(z, min=0) ** 2


def expert(h, w, pre):
    return linear(w, pre + ".down", relu_squared(linear(w, pre + ".up", h)))


def experts(h, w, pre, f):
    """The outputs past the real experts hand the input through, times their weight."""
    r = f["router"]
    z = linear(w, pre + "router", h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in choose(z[t], get(w, pre + "correction"), r["top"]):
            out[t] += wt * (expert(h[t], w, f"{pre}e{e}") if e < r["experts"] else h[t])
    return out


# ------------------------------------------------------------------ model
def forward(tokens, w, cfg, residuals=None):
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the stream after every layer."""
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = get(w, "embed")[torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    kv = {}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = l["mixer"]
        shared = kv[mix["kv_from"]] if mix.get("kv_from") is not None else None
        y, kv[i] = attention(norm_around_one(x, w[p + "norm1"], eps), w, p + "mix.", mix, eps, shared)
        x = x + m * norm_around_one(y, w[p + "norm1b"], eps) * get(w, p + "ls1")
        if l.get("mlp") is not None:
            y = experts(norm_around_one(x, w[p + "norm2"], eps), w, p + "mlp.", l["mlp"])
            x = x + m * norm_around_one(y, w[p + "norm2b"], eps) * get(w, p + "ls2")
        if residuals is not None:
            residuals.append(x)
    return linear(w, "head", norm_around_one(x, w["final.norm"], eps))


# ------------------------------------------------------------------ checkpoints for tests
def tensor_shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l.get("mlp")
        out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "ls1": (W,), p + "mix.q": (m["heads"] * m["dim"], W),
                    p + "mix.q.norm": (m["dim"],), p + "mix.o": (W, m["heads"] * m["vdim"])})
        if m.get("kv_from") is None:
            out.update({p + "mix.k": (m["kv_heads"] * m["dim"], W), p + "mix.v": (m["kv_heads"] * m["vdim"], W),
                        p + "mix.k.norm": (m["dim"],)})
        if f is not None:
            r, ff = f["router"], f["expert"]["ff"]
            n = r["experts"] + r.get("identity", 0)
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "ls2": (W,), p + "mlp.router": (n, W),
                        p + "mlp.correction": (n,)})
            for e in range(r["experts"]):
                out.update({f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return out


def random_weights(cfg, seed=0, decisive=False):
    """bf16 tensors under the checkpoint's names; gains that are stored around zero stay there, others around one.
    ``decisive``: corrections so far apart that they alone choose the experts."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        leaf = name.split(".", 1)[-1]
        if leaf.endswith((".q.norm", ".k.norm")) or leaf in ("ls1", "ls2"):
            t = 1.0 + 0.3 * t
        elif decisive and leaf.endswith("correction"):
            t = 2.0 * torch.randperm(shape[0], generator=g)
        elif len(shape) == 1:
            t = (0.05 if leaf.endswith("correction") else 0.3) * t
        elif name != "embed":
            t = t * shape[1] ** -0.5 * (2.0 if leaf.endswith("router") else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out
