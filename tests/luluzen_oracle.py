"""Plain statement of the Luluzen decoder, one function per mechanism, whole sequences at a time, in float64 on the CPU.

Nothing here uses the package: the tests compare the package with these functions.  ``w`` maps checkpoint tensor names to
tensors and ``cfg`` is the checkpoint's ``config.json`` as a dict.  Attention builds the full score matrix of a head,
recurrences and experts run token by token, rotations pair by pair.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def get(w, name):
    return w[name].to(F64)


def linear(w, name, x):
    y = x @ get(w, name).t()
    return y + get(w, name + ".b") if name + ".b" in w else y


def silu(x):
    return x / (1.0 + torch.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def cap(x, c):
    return c * torch.tanh(x / c)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, g, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * g.to(F64)


# ------------------------------------------------------------------ attention
def distance_bucket(n, rows, far):
    """Distances below ``rows / 2`` have a bucket each, larger ones share the rest on a logarithmic scale that ends at ``far``."""
    half = rows // 2
    if n < half:
        return n
    steps = math.log(n / half) / math.log(far / half) * (rows - half)
    near = round(steps)                                       # (a step that is a whole number, up to float rounding)
    return min(rows - 1, half + (near if abs(steps - near) < 1e-9 else math.floor(steps)))


def distance_bias(table, far, T):
    """``table [rows, heads]`` -> ``[heads, T, T]``, entry (h, i, j) for i >= j."""
    rows = table.shape[0]
    by_distance = torch.stack([table[distance_bucket(n, rows, far)] for n in range(T)]).to(F64)        # [T, heads]
    i = torch.arange(T)
    return by_distance[(i[:, None] - i[None, :]).clamp(min=0)].permute(2, 0, 1)


def rotate_pairs(x, positions, dims, base):
    """Rotation of the entries (2i, 2i + 1), i < dims / 2, of the last axis; ``x [T, heads, D]``."""
    out = x.clone()
    for i in range(dims // 2):
        a = (positions.to(F64) * float(base) ** (-2.0 * i / dims))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def query_temperature(positions, coef, every):
    return 1.0 + coef * torch.log(((positions + 1) // every).to(F64) + 1.0)


def attend(q, k, v, scale, window=0, softcap=0.0, bias=None, sink=None):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``: query head h reads key head h // (H / G); token i sees j with
    0 <= i - j < window (no lower bound without a window); a sink adds exp(sink_h) to the softmax' denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    seen = (dist >= 0) if not window else (dist >= 0) & (dist < window)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        if softcap:
            s = cap(s, softcap)
        if bias is not None:
            s = s + bias[h]
        s = s.masked_fill(~seen, float("-inf"))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h].to(F64) - top)
        out[:, h] = (e / den) @ v[:, g]
    return out


def biased_attention(h, w, pre, m, eps):
    """Head norms, a query temperature and a learned bias by distance; no rotation."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = unit_rms(linear(w, pre + "q", h).view(T, H, D), eps) * get(w, pre + "q.norm")
    k = unit_rms(linear(w, pre + "k", h).view(T, G, D), eps) * get(w, pre + "k.norm")
    v = linear(w, pre + "v", h).view(T, G, m["vdim"])
    q = q * query_temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    o = attend(q, k, v, m["scale"], bias=distance_bias(w[pre + "rel"], m["bias_max"], T))
    return linear(w, pre + "o", o.reshape(T, -1))


def gated_window_attention(h, w, pre, m, eps):
    """Norms over the whole projections, rotation in adjacent pairs, capped scores, a window, sinks and an output gate."""
    T, H, G, D, pos = h.shape[0], m["heads"], m["kv_heads"], m["dim"], torch.arange(h.shape[0])
    q = (unit_rms(linear(w, pre + "q", h), eps) * get(w, pre + "q.norm")).view(T, H, D)
    k = (unit_rms(linear(w, pre + "k", h), eps) * get(w, pre + "k.norm")).view(T, G, D)
    q, k = (rotate_pairs(x, pos, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
    v = linear(w, pre + "v", h).view(T, G, m["vdim"])
    o = attend(q, k, v, m["scale"], m["mask"]["size"], m["softcap"], sink=w[pre + "sink"])
    return linear(w, pre + "o", o.reshape(T, -1) * sigmoid(linear(w, pre + "g", h)))


# ------------------------------------------------------------------ recurrences
def decayed_states(q, k, v, decay):
    """``q, k [T, H, D]``, ``v [T, H, V]``, ``decay [H]``: S <- decay S + k v^T, read-out S^T q."""
    S, o = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F64), []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(o)


def lightning(h, w, pre, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k = (silu(linear(w, pre + n, h)).view(T, H, m["dim"]) for n in "qk")
    v = silu(linear(w, pre + "v", h)).view(T, H, m["vdim"])
    o = decayed_states(q, k, v, torch.tensor(m["decay"], dtype=F64))
    o = unit_rms(o.reshape(T, -1), eps) * get(w, pre + "norm")
    return linear(w, pre + "o", o * sigmoid(linear(w, pre + "g", h)))


def short_conv(x, taps):
    """``x [T, C]``, ``taps [C, K]``: y[t] = sum_j taps[:, j] x[t - (K - 1) + j], zeros in front."""
    K = taps.shape[1]
    ext = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=F64), x])
    return sum(ext[j: j + x.shape[0]] * taps[:, j].to(F64) for j in range(K))


def delta_states(q, k, v, g, beta):
    """``q, k, g [T, H, D]``, ``v [T, H, V]``, ``beta [T, H]``: decay per key channel, then the delta rule, then the read-out."""
    T, H, D = q.shape
    S, o = torch.zeros(H, D, v.shape[2], dtype=F64), []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(o)


def gated_delta(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(linear(w, pre + n, h), w[f"{pre}{n}.conv"])) for n in "qkv")
    q, k, v = q.view(T, G, D), k.view(T, G, D), v.view(T, H, V)
    q, k = (x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6) for x in (q, k))
    q, k = (x.repeat_interleave(H // G, 1) for x in (q * D ** -0.5, k))
    beta = sigmoid(h @ get(w, pre + "b").t())
    a = (linear(w, pre + "a2", linear(w, pre + "a1", h)) + get(w, pre + "dt_bias")).view(T, H, D)
    g = torch.exp(-torch.exp(get(w, pre + "A_log"))[None, :, None] * softplus(a))
    o = unit_rms(delta_states(q, k, v, g, beta), eps) * get(w, pre + "norm")
    gate = sigmoid(linear(w, pre + "g2", linear(w, pre + "g1", h)))
    return linear(w, pre + "o", o.reshape(T, -1) * gate)


def memory_states(q, k, v, i, f):
    """``q, k [T, H, D]``, ``v [T, H, V]``, log gates ``i, f [T, H]``: the stabilised matrix memory with its normaliser."""
    T, H, D = q.shape
    S, n, top, out = torch.zeros(H, D, v.shape[2], dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64), []
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, add, top = torch.exp(f[t] + top - new), torch.exp(i[t] - new), new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out)


def matrix_memory(h, w, pre, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(w, pre + "q", h).view(T, H, D) * D ** -0.5
    k, v = linear(w, pre + "k", h).view(T, H, D), linear(w, pre + "v", h).view(T, H, V)
    i = cap(linear(w, pre + "i", h), m["gate_cap"])
    f = -softplus(-cap(linear(w, pre + "f", h), m["gate_cap"]))
    o = unit_rms(memory_states(q, k, v, i, f), eps).reshape(T, -1) * get(w, pre + "norm")
    return linear(w, pre + "o", o * sigmoid(linear(w, pre + "g", h)))


# ------------------------------------------------------------------ mixers, feed-forward
def mixer(h, w, pre, l, eps):
    m = l["mixer"]
    if l["type"] == "lightning":
        return lightning(h, w, pre, m, eps)
    left, right = {"parallel": (biased_attention, gated_delta),
                   "parallel_2": (gated_window_attention, matrix_memory)}[l["type"]]
    return (m["left_scale"] * left(h, w, pre + "left.", m["left"], eps)
            + m["right_scale"] * right(h, w, pre + "right.", m["right"], eps))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense(h, w, pre):
    return linear(w, pre + "down", gelu_tanh(linear(w, pre + "gate", h)) * linear(w, pre + "up", h))


def expert(h, w, pre, limit):
    g = torch.clamp(linear(w, pre + "gate", h), max=limit)
    u = torch.clamp(linear(w, pre + "up", h), -limit, limit)
    return linear(w, pre + "down", g * sigmoid(1.702 * g) * (u + 1.0))


def choose(z, top):
    """Router logits ``[n]`` -> [(expert, weight)]: the largest sigmoid scores, as they are."""
    s = sigmoid(z)
    return [(e, float(s[e])) for e in sorted(range(z.numel()), key=lambda e: (-float(s[e]), e))[:top]]


def experts(h, w, pre, f):
    z = linear(w, pre + "router", h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in choose(z[t], f["router"]["top"]):
            out[t] += expert(wt * h[t], w, f"{pre}e{e}.", f["expert"]["limit"])
    return out


# ------------------------------------------------------------------ model
def layer_runs(cfg):
    """``(layer, pass)`` in the order they run; ``pass`` is None outside the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(tokens, w, cfg, residuals=None):
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = x0 = get(w, "embed")[torch.as_tensor(tokens)]
    for i, t in layer_runs(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            x = linear(w, "loop.in", torch.cat([x, x0], -1)) + get(w, "loop.step")[t]
        p, l = f"l{i}.", cfg["layers"][i]
        x = x + mixer(layer_norm(x, w[p + "norm1"], eps), w, p + "mix.", l, eps)
        f = l.get("mlp")
        if f is not None:
            h = layer_norm(x, w[p + "norm2"], eps)
            x = x + (dense(h, w, p + "mlp.") if f["kind"] == "dense" else experts(h, w, p + "mlp.", f))
        if residuals is not None:
            residuals.append(x)
    return cap(layer_norm(x, w["final.norm"], eps) @ get(w, "embed").t(), float(cfg["logit_softcap"]))


# ------------------------------------------------------------------ checkpoints for tests
def tensor_shapes(cfg, low=lambda i: (6 + 2 * i, 5 + i, 11)):
    """``low(i)``: what the config does not carry - rows of layer i's distance bias, ranks of its decay and gate projections."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    if cfg.get("loop"):
        out.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l.get("mlp")
        out[p + "norm1"] = (W,)

        def linear_attention(pre, m, gated=True):
            k, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({pre + "q": (k, W), pre + "k": (k, W), pre + "v": (v, W), pre + "g": (v, W), pre + "o": (W, v),
                        pre + "norm": (v,)})

        if l["type"] == "lightning":
            linear_attention(p + "mix.", m)
        else:
            a, r, pre = m["left"], m["right"], p + "mix.left."
            q, k, v, o = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
            out.update({pre + "q": (q, W), pre + "k": (k, W), pre + "v": (v, W), pre + "o": (W, o)})
            rows, ra, rg = low(i)
            if l["type"] == "parallel":
                out.update({pre + "q.b": (q,), pre + "k.b": (k,), pre + "v.b": (v,), pre + "q.norm": (a["dim"],),
                            pre + "k.norm": (a["dim"],), pre + "rel": (rows, a["heads"])})
                pre = p + "mix.right."
                H, k, v = r["heads"], r["kv_heads"] * r["dim"], r["heads"] * r["vdim"]
                out.update({pre + "q": (k, W), pre + "k": (k, W), pre + "v": (v, W), pre + "q.conv": (k, r["conv"]),
                            pre + "k.conv": (k, r["conv"]), pre + "v.conv": (v, r["conv"]), pre + "b": (H, W),
                            pre + "A_log": (H,), pre + "norm": (r["vdim"],), pre + "a1": (ra, W), pre + "a2": (H * r["dim"], ra),
                            pre + "dt_bias": (H * r["dim"],), pre + "g1": (rg, W), pre + "g2": (v, rg), pre + "o": (W, v)})
            else:
                out.update({pre + "q.norm": (q,), pre + "k.norm": (k,), pre + "sink": (a["heads"],), pre + "g": (o, W)})
                pre, H = p + "mix.right.", r["heads"]
                linear_attention(pre, r)
                out.update({pre + "i": (H, W), pre + "i.b": (H,), pre + "f": (H, W), pre + "f.b": (H,)})
        if f is not None:
            out[p + "norm2"] = (W,)
            if f["kind"] == "dense":
                out.update({p + "mlp.gate": (f["ff"], W), p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
            else:
                out[p + "mlp.router"] = (f["router"]["experts"], W)
                for e in range(f["router"]["experts"]):
                    ff, q = f["expert"]["ff"], f"{p}mlp.e{e}."
                    out.update({q + "gate": (ff, W), q + "up": (ff, W), q + "down": (W, ff)})
    return out


def random_weights(cfg, seed=0, **kw):
    """bf16 tensors under the checkpoint's names; norm weights around one, biases of the forget gates that keep states alive,
    sinks and distance biases of the size of scores."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, **kw).items():
        t = torch.randn(*shape, generator=g)
        leaf = name.split(".")[-1]
        if "norm" in leaf:
            t = 1.0 + 0.3 * t
        elif leaf == "A_log":
            t = 0.5 * t - 1.0
        elif leaf == "dt_bias":
            t = t - 2.0
        elif name.endswith(".f.b"):
            t = t + 4.0
        elif leaf == "conv":
            t = 0.5 * t
        elif leaf in ("rel", "sink"):
            t = 1.5 * t
        elif leaf in ("step", "b") and len(shape) < 2 or name == "loop.step":
            t = 0.3 * t
        elif name != "embed":
            t = t * shape[-1] ** -0.5 * (2.0 if leaf == "router" else 1.0)
        out[name] = t.to(torch.bfloat16)
    return out
