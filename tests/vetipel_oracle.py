"""Plain statement of the Vetipel decoder, one function per mechanism, whole sequences at a time, in float64 on the CPU.

Nothing here uses the package: the tests compare the package with these functions.  ``w`` maps checkpoint tensor names to
tensors and ``cfg`` is the checkpoint's ``config.json`` as a dict.  Attention builds the full score matrix of a head, biases
come entry by entry, rotations pair by pair, streams one at a time.
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


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(w, name, x, eps):
    return unit_rms(x, eps) * (1.0 + get(w, name))


# ------------------------------------------------------------------ streams
def read_streams(streams, weights):
    """What a sublayer reads: one number per stream."""
    return sum(float(weights[s]) * x for s, x in enumerate(streams))


def write_streams(streams, mix, out, y):
    """The new streams, each made of all the streams before: ``mix[s, t]`` is what stream t takes of stream s."""
    return [sum(float(mix[s, t]) * x for s, x in enumerate(streams)) + float(out[t]) * y for t in range(len(streams))]


# ------------------------------------------------------------------ attention
def distances(T):
    i = torch.arange(T)
    return i[:, None] - i[None, :]


def window_mask(T, size):
    d = distances(T)
    return (d >= 0) & (d < size)


def chunk_mask(T, size):
    i = torch.arange(T)
    return (distances(T) >= 0) & (i[:, None] // size == i[None, :] // size)


def causal_mask(T):
    return distances(T) >= 0


def linear_bias(T, heads):
    """``[heads, T, T]``, taken off the scores: a slope per head, 2 ** (-8 (h + 1) / heads)."""
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)
    return slopes[:, None, None] * distances(T).clamp(min=0).to(F64)


def log_bias(T, r1, r2):
    """``[heads, T, T]``, taken off the scores: r1 ln(1 + r2 distance)."""
    d = distances(T).clamp(min=0).to(F64)
    return torch.stack([r1[h].to(F64) * torch.log(1.0 + r2[h].to(F64) * d) for h in range(len(r1))])


def softmax_weights(scores, seen, sink=None):
    """Over the seen keys; a sink is one more term of the denominator."""
    s = scores.masked_fill(~seen, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + math.e ** (float(sink) - top)
    return e / den


def sigmoid_weights(scores, seen, shift):
    return torch.where(seen, sigmoid(scores + float(shift)), torch.zeros_like(scores))


def attend(q, k, v, score, weigh):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``: query head h reads key head h // (H / G); ``score(h, q . k)`` and
    ``weigh(h, scores)`` make a head's weights."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        out.append(weigh(h, score(h, q[:, h] @ k[:, g].t())) @ v[:, g])
    return torch.stack(out, 1)


def head_gate(h, w, pre, o):
    """``o [T, H, Dv]`` times one number per head."""
    return o * sigmoid(linear(w, pre + "g", h))[:, :, None]


def sigmoid_attention(h, w, pre, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = linear(w, pre + "q", h).view(T, H, m["dim"]), linear(w, pre + "k", h).view(T, G, m["dim"])
    v = linear(w, pre + "v", h).view(T, G, m["vdim"])
    bias, seen = linear_bias(T, H), window_mask(T, m["mask"]["size"])
    o = attend(q, k, v, lambda i, s: s * m["scale"] - bias[i], lambda i, s: sigmoid_weights(s, seen, w[pre + "pb"][i]))
    return linear(w, pre + "o", head_gate(h, w, pre, o).reshape(T, -1))


def chunked_attention(h, w, pre, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = unit_rms(linear(w, pre + "q", h).view(T, H, m["dim"]), eps)
    k = unit_rms(linear(w, pre + "k", h).view(T, G, m["dim"]), eps)
    v = linear(w, pre + "v", h).view(T, G, m["vdim"])
    bias, seen = log_bias(T, w[pre + "r1"], w[pre + "r2"]), chunk_mask(T, m["mask"]["size"])
    temp, sink = get(w, pre + "temp"), w[pre + "sink"]
    o = attend(q, k, v, lambda i, s: s * m["scale"] * temp[i] - bias[i], lambda i, s: softmax_weights(s, seen, sink[i]))
    return linear(w, pre + "o", head_gate(h, w, pre, o).reshape(T, -1))


def rotate_pairs(x, positions, dims, base):
    """Rotation of the entries (2i, 2i + 1), i < dims / 2, of the last axis; ``x [T, heads, D]``."""
    out = x.clone()
    for i in range(dims // 2):
        a = (positions.to(F64) * float(base) ** (-2.0 * i / dims))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_attention(h, w, pre, m, eps):
    T, H, D, R, K, pos = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], torch.arange(h.shape[0])
    q = linear(w, pre + "q", h).view(T, H, D + R)
    down = linear(w, pre + "dkv", h)
    c = unit_rms(down[:, :K], eps) * get(w, pre + "dkv.norm")
    qr = rotate_pairs(q[..., D:], pos, m["rot"]["dims"], m["rot"]["base"])
    kr = rotate_pairs(down[:, None, K:], pos, m["rot"]["dims"], m["rot"]["base"])
    k = torch.cat([linear(w, pre + "uk", c).view(T, H, D), kr.expand(T, H, R)], -1)
    v = linear(w, pre + "uv", c).view(T, H, m["vdim"])
    seen = causal_mask(T)
    o = attend(torch.cat([q[..., :D], qr], -1), k, v, lambda i, s: s * m["scale"], lambda i, s: softmax_weights(s, seen))
    return linear(w, pre + "o", o.reshape(T, -1))


MIXERS = {"attention": sigmoid_attention, "latent_attention": latent_attention, "attention_2": chunked_attention}


# ------------------------------------------------------------------ feed-forward, model
def dense(h, w, pre):
    return linear(w, pre + "down", torch.clamp(linear(w, pre + "up", h), min=0.0) ** 2)


def sublayers(cfg, w):
    """Every sublayer in order: ``(name of its norm, name of its stream weights, function of the normed input, ends a layer)``."""
    eps = float(cfg["norm"]["eps"])
    for i, l in enumerate(cfg["layers"]):
        yield (f"l{i}.norm1", f"l{i}.hc1.", lambda h, l=l, i=i: MIXERS[l["type"]](h, w, f"l{i}.mix.", l["mixer"], eps),
               l.get("mlp") is None)
        if l.get("mlp") is not None:
            yield f"l{i}.norm2", f"l{i}.hc2.", lambda h, i=i: dense(h, w, f"l{i}.mlp."), True


def forward(tokens, w, cfg, residuals=None):
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = get(w, "embed")[torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    streams = [x.clone() for _ in range(int(cfg["streams"]))]
    for gain, hc, f, last in sublayers(cfg, w):
        y = f(norm(w, gain, read_streams(streams, w[hc + "in"]), eps))
        streams = write_streams(streams, w[hc + "mix"], w[hc + "out"], y)
        if last and residuals is not None:
            residuals.append(sum(streams))
    return norm(w, "final.norm", sum(streams), eps) @ get(w, "head").t()


# ------------------------------------------------------------------ checkpoints for tests
def tensor_shapes(cfg):
    W, S = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        subs, pre, H = [1] if l.get("mlp") is None else [1, 2], p + "mix.", m["heads"]
        for q in subs:
            out.update({f"{p}norm{q}": (W,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        if l["type"] == "latent_attention":
            K = m["kv_rank"]
            out.update({pre + "q": (H * (m["dim"] + m["rot_dim"]), W), pre + "dkv": (K + m["rot_dim"], W), pre + "dkv.norm": (K,),
                        pre + "uk": (H * m["dim"], K), pre + "uv": (H * m["vdim"], K)})
        else:
            G = m["kv_heads"]
            rows = {"q": H * m["dim"], "k": G * m["dim"], "v": G * m["vdim"], "g": H}
            out.update({pre + n: (r, W) for n, r in rows.items()})
            if l["type"] == "attention":
                out[pre + "pb"] = (H,)
            else:
                out.update({f"{pre}{n}.b": (rows[n],) for n in "qkv"})
                out.update({pre + n: (H,) for n in ("r1", "r2", "temp", "sink")})
        out[pre + "o"] = (W, H * m["vdim"])
        if l.get("mlp") is not None:
            out.update({p + "mlp.up": (l["mlp"]["ff"], W), p + "mlp.down": (W, l["mlp"]["ff"])})
    return out


def random_weights(cfg, seed=0):
    """bf16 tensors under the checkpoint's names; stored norm weights around zero (the latent's around one), mixes around the
    identity, biases of the size of scores."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        leaf = name.split(".")[-1]
        if name.endswith("dkv.norm"):
            t = 1.0 + 0.3 * t
        elif "norm" in leaf or leaf == "b":
            t = 0.3 * t
        elif leaf == "in":
            t = 1.0 / cfg["streams"] + 0.3 * t
        elif leaf in ("out", "temp"):
            t = 1.0 + 0.4 * t
        elif leaf == "mix":
            t = 0.8 * torch.eye(shape[0]) + 0.3 * t
        elif leaf in ("r1", "r2"):
            t = t.abs() + 0.1
        elif leaf == "pb":
            t = 0.7 * t - 2.0
        elif leaf == "sink":
            t = 1.5 * t
        elif name != "embed":
            t = t * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
