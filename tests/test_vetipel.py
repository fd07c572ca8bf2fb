"""The Vetipel model through the engine's own scheduler, block pool and step function, against the plain statement in
``vetipel_oracle.py``.  Every test makes its own small checkpoint (sizes that differ from layer to layer, also ones that are 1 or
not a multiple of anything) and runs on the CPU and, marked ``gpu``, through the kernels."""
import json
import os
import random
import subprocess
import sys

import pytest
import torch
from safetensors.torch import save_file

from tests import vetipel_oracle as O
from vllm_metax_b200 import LLM, SamplingParams
from vllm_metax_b200.entrypoints.trace_replay import TraceReplay

RUNS = [pytest.param("cpu", "float32"), pytest.param("cpu", "bfloat16"),
        pytest.param("cuda", "float32", marks=pytest.mark.gpu), pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
# rms of a position's logit error over the logits' rms: (a position, median of all).  A wrong key or a mask off by one gives 0.3
# and more.
LIMIT = {"float32": (1e-4, 2e-5), "bfloat16": (0.18, 4e-2)}
pytestmark = pytest.mark.usefixtures("kernel_status_ok")


def dense(ff):
    return {"kind": "dense", "ff": ff}


def window(heads, kv_heads, dim, vdim, size, mlp=None, scale=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                       "scale": scale or dim ** -0.5, "mask": {"size": size}}}


def chunked(heads, kv_heads, dim, vdim, size, mlp=None, scale=None):
    return {**window(heads, kv_heads, dim, vdim, size, mlp, scale or 1.5 * dim ** -0.5), "type": "attention_2"}


def latent(heads, dim, rot_dim, vdim, kv_rank, base, mlp=None, scale=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
        "scale": scale or (dim + rot_dim) ** -0.5}}


def config(vocab, width, streams, layers, eps=1e-5, scale=8.0, **extra):
    return {"architecture": "Vetipel", "vocab": vocab, "width": width, "streams": streams, "embedding": {"scale": scale},
            "norm": {"eps": eps}, "layers": layers, **extra}


CONFIGS = {
    # sizes the tensor-core paths take; feed-forwards and none
    "even": config(200, 96, 2, [window(4, 2, 64, 40, 37, dense(88)), latent(5, 24, 8, 40, 48, 700.0, dense(64)),
                                chunked(6, 2, 40, 56, 50, None), window(6, 6, 48, 64, 100, dense(40)),
                                chunked(8, 1, 104, 128, 64, dense(64)), latent(2, 64, 64, 128, 136, 5e4)]),
    # nothing divides by eight; one head, one stream, a window and chunks of one token
    "odd": config(101, 50, 1, [chunked(1, 1, 9, 11, 1, dense(13)), window(1, 1, 7, 5, 1), latent(1, 3, 2, 1, 5, 20.0, dense(9)),
                               chunked(3, 1, 10, 3, 23, dense(7)), window(3, 1, 6, 9, 11, dense(17))], eps=1e-3, scale=0.7),
    # wider heads and latents than the tensor-core tiles, many streams
    "wide": config(64, 64, 5, [chunked(2, 1, 200, 160, 70, dense(32)), latent(2, 136, 64, 144, 264, 1e4, dense(24)),
                               window(2, 2, 264, 40, 30), latent(1, 40, 16, 24, 600, 300.0), chunked(2, 2, 16, 264, 33)], eps=1e-6),
    # one layer without a feed-forward
    "single": config(88, 72, 4, [latent(3, 16, 8, 16, 40, 99.0)]),
}


def checkpoint(tmp_path, cfg, seed=1, weights=None):
    """Returns (path, weights, config)."""
    w = weights or O.random_weights(cfg, seed)
    d = tmp_path / "model"
    d.mkdir(exist_ok=True)
    save_file(w, str(d / "model.safetensors"))
    (d / "config.json").write_text(json.dumps(cfg))
    return str(d), w, cfg


def tokens(n, vocab, seed=0):
    return random.Random(seed * 1000 + n).choices(range(vocab), k=n)


def check(got, want, dtype, what=""):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    peak, mean = LIMIT[dtype]
    assert float(err.max()) < peak and float(err.median()) < mean, \
        f"{what}: error {float(err.max()):.3g} at position {int(err.argmax())}, median {float(err.median()):.3g}"


def feed(rp, rid, toks, sizes):
    """All logits of one request fed in portions of ``sizes`` (the last one repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(rp.step([{"id": rid, "tokens": toks[at: at + n], "want": list(range(n))}], [rid] if at + n == len(toks) else []))
        at, k = at + n, k + 1
    return torch.cat(out)


# ------------------------------------------------------------------ prompts, portions, decoding
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts(tmp_path, name, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name])
    rp = TraceReplay.open(path, dtype, 192, device, enforce_eager=True)
    for n in (1, 2, 3, 17, 65, 110):
        t = tokens(n, cfg["vocab"])
        check(feed(rp, f"r{n}", t, [n]), O.forward(t, w, cfg), dtype, f"{n} tokens")
    assert rp.engine.kv.num_free_blocks == 3


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens(tmp_path, name, device, dtype):
    """One sequence cut in many ways: token by token from the start, pairs, odd sizes, page-sized portions, a long prompt and
    then single tokens - all the same logits.  Pages are used again without being cleared."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=2)
    t = tokens(84, cfg["vocab"])
    want = O.forward(t, w, cfg)
    rp = TraceReplay.open(path, dtype, 128, device)
    whole = feed(rp, "x", t, [84])
    for sizes in ([1], [2], [3, 1, 2, 16], [5, 40, 1, 1, 30], [64], [63, 2, 65], [80, 2, 1]):
        got = feed(rp, "x", t, sizes)
        check(got, want, dtype, str(sizes))
        check(got, whole.double(), dtype, str(sizes))


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_passes_every_window_and_chunk(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["even"], seed=3)
    t = tokens(215, cfg["vocab"])
    rp = TraceReplay.open(path, dtype, 256, device)
    check(feed(rp, "x", t, [10, 1]), O.forward(t, w, cfg), dtype)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_context(tmp_path, device, dtype):
    """Short portions that see much more context than they have tokens, and several key tiles per window and chunk."""
    cfg = config(70, 64, 3, [window(2, 1, 64, 64, 300, dense(64)), latent(2, 32, 16, 32, 64, 1e4), chunked(4, 2, 64, 64, 280, dense(48))])
    path, w, _ = checkpoint(tmp_path, cfg, seed=6)
    t = tokens(777, 70)
    want = O.forward(t, w, cfg)
    rp = TraceReplay.open(path, dtype, 832, device)
    for sizes in ([777], [700, 2, 9, 1], [256, 130]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


# ------------------------------------------------------------------ batches, pages used again
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_equal_each_request_alone(tmp_path, name, device, dtype):
    """Up to four live requests in a pool that is nearly full all the time: portions beside single tokens, requests that sit
    out steps, pages handed on to the next request."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=4)
    rng = random.Random(5)
    lens = [1, 2, 100, 70, 33, 64, 66, 3]
    seqs = [tokens(n, cfg["vocab"], seed=7) for n in lens]
    got = [[] for _ in seqs]
    rp = TraceReplay.open(path, dtype, 320, device)
    pages = lambda i: -(-lens[i] // 64)
    waiting, live, at, used = list(range(len(seqs))), [], [0] * len(seqs), set()
    while waiting or live:
        while waiting and len(live) < 4 and sum(map(pages, live)) + pages(waiting[0]) <= 5:
            live.append(waiting.pop(0))
        step = [i for i in live if rng.random() < 0.8] or live[:1]
        rng.shuffle(step)
        entries, end = [], []
        for i in step:
            n = min(rng.choice([1, 1, 1, 2, 3, 17, 40]), lens[i] - at[i])
            entries.append({"id": i, "tokens": seqs[i][at[i]: at[i] + n], "want": list(range(n))})
            at[i] += n
            if at[i] == lens[i]:
                end.append(i)
        logits = rp.step(entries, [])
        used |= {b for r in rp.engine.scheduler.running for b in r.block_ids}
        rp.step([], end)
        for e in entries:
            n = len(e["tokens"])
            got[e["id"]].append(logits[:n])
            logits = logits[n:]
        live = [i for i in live if i not in end]
    for i, t in enumerate(seqs):
        check(torch.cat(got[i]), O.forward(t, w, cfg), dtype, f"request {i}")
    assert len(used) <= 5 < sum(map(pages, range(len(seqs)))) and rp.engine.kv.num_free_blocks == 5


# ------------------------------------------------------------------ keys at the edges, far keys
def differ(a, b):
    return float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt())


def needle(w, q, k, floor):
    """``(a, b)``: the pair of tokens whose score stands out most among those of query token a (its own aside)."""
    s = q @ k.t()
    s.fill_diagonal_(-float("inf"))
    top = s.topk(2, -1).values
    a = int((top[:, 0] - top[:, 1].clamp(min=floor)).argmax())
    return a, int(s[a].argmax()), float(top[a].mean())


def case(vocab, a, b, at, far, seed):
    """Token a at place ``at``, token b ``far`` places before it, and neither anywhere else."""
    t = random.Random(seed).choices([x for x in range(vocab) if x not in (a, b)], k=at + 4)
    t[at - far], t[at] = b, a
    return t


def edge_model(kind, size):
    """One layer, one head, whose query token a gives its weight to key token b alone."""
    make = window if kind == "window" else chunked
    cfg = config(60, 48, 2, [make(1, 1, 32, 40, size, scale=6.0)], eps=1e-6)
    w = O.random_weights(cfg, seed=11)
    w["l0.mix.g"].zero_()
    for n in "qkv":
        if f"l0.mix.{n}.b" in w:
            w[f"l0.mix.{n}.b"].zero_()
    h = O.norm(w, "l0.norm1", O.get(w, "embed") * cfg["embedding"]["scale"] * float(w["l0.hc1.in"].double().sum()), 1e-6)
    q, k = O.linear(w, "l0.mix.q", h), O.linear(w, "l0.mix.k", h)
    if kind == "chunk":
        q, k = O.unit_rms(q, 1e-6), O.unit_rms(k, 1e-6)
        w["l0.mix.temp"].fill_(1.0)
        w["l0.mix.r1"].fill_(0.125)
        w["l0.mix.sink"].fill_(20.0)
    a, b, mid = needle(w, q, k, 0.0)
    if kind == "window":
        w["l0.mix.pb"].fill_(-6.0 * mid + 2.0 ** -8 * size)
    w["l0.mix.o"] *= 8.0
    return cfg, w, a, b


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("size", [2, 16, 64, 65, 100])
def test_window_edges(tmp_path, size, device, dtype):
    """The one key that matters sits just inside or just outside the window of the query that wants it; queries fall on both
    sides of page borders, in whole prompts, portions and decoding."""
    cfg, w, a, b = edge_model("window", size)
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 256, device)
    for at in sorted({p for p in (size, size + 1, 63, 64, 65, 127, 128) if p >= size}):
        for far in (size - 1, size):
            t = case(60, a, b, at, far, at)
            want = O.forward(t, w, cfg)
            wrong = json.loads(json.dumps(cfg))
            wrong["layers"][0]["mixer"]["mask"]["size"] += -1 if far < size else 1
            assert differ(O.forward(t, w, wrong)[at], want[at]) > 0.3, "the case is blind"
            for sizes in ([len(t)], [max(1, at - 1), 1], [at, 2], [2]):
                check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("size", [2, 16, 63, 64, 100])
def test_chunk_edges(tmp_path, size, device, dtype):
    """The key is the first of the query's chunk or the last of the chunk before; the query is the first, second or last of its
    chunk.  Chunks are counted from the sequence's start, not from a portion's."""
    cfg, w, a, b = edge_model("chunk", size)
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 320, device)
    for n in {1, 2, -(-66 // size)}:
        for at in sorted({n * size, n * size + 1, n * size + size - 1}):
            for key in (n * size, n * size - 1):
                if key == at:
                    continue
                t = case(60, a, b, at, at - key, at)
                want = O.forward(t, w, cfg)
                wrong = json.loads(json.dumps(cfg))                    # everything seen, or no key but the query's own
                wrong["layers"][0]["mixer"]["mask"]["size"] = 1 if key == n * size else 1000
                assert differ(O.forward(t, w, wrong)[at], want[at]) > 0.3, "the case is blind"
                for sizes in ([len(t)], [max(1, at - 1), 1], [at, 2], [2]):
                    check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {key}, {sizes}")


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_keys_of_latent_attention(tmp_path, device, dtype):
    """A key far back that alone matters, at page borders and at the first token, through the latent."""
    cfg = config(60, 48, 2, [latent(1, 32, 8, 40, 40, 1e30, scale=4.0)], eps=1e-6)
    w = O.random_weights(cfg, seed=12)
    w["l0.mix.q"][32: 34], w["l0.mix.dkv"][40: 42] = 0, 0              # with a huge base only the first pair turns
    h = O.norm(w, "l0.norm1", O.get(w, "embed") * 8.0 * float(w["l0.hc1.in"].double().sum()), 1e-6)
    d = O.linear(w, "l0.mix.dkv", h)
    c = O.unit_rms(d[:, :40], 1e-6) * O.get(w, "l0.mix.dkv.norm")
    a, b, _ = needle(w, O.linear(w, "l0.mix.q", h), torch.cat([O.linear(w, "l0.mix.uk", c), d[:, 40:]], 1), -1e9)
    w["l0.mix.o"] *= 3.0
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 512, device)
    for at, far in ((400, 400), (320, 192), (299, 171), (65, 1)):
        t = case(60, a, b, at, far, at + far)
        want = O.forward(t, w, cfg)
        blind = O.forward([x if x != b else (a + 1 if a + 1 != b else a + 2) % 60 for x in t], w, cfg)
        assert differ(blind[at], want[at]) > 0.3, "the case is blind"
        for sizes in ([len(t)], [at, 1], [at // 2, at - at // 2 - 2, 2]):
            check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}")


@pytest.mark.parametrize("device,dtype", RUNS)
def test_sink_temperature_and_first_tokens(tmp_path, device, dtype):
    """A sink larger than every score leaves next to nothing of a head's output, one among the scores part of it, whatever the
    temperature; the first tokens of a sequence and of a chunk see the fewest keys."""
    cfg = config(40, 48, 3, [chunked(2, 1, 16, 16, 6), chunked(2, 2, 24, 16, 9, dense(32))])
    w = O.random_weights(cfg, seed=31)
    w["l0.mix.o"] *= 4.0
    t = tokens(20, 40)
    base = O.forward(t, w, cfg)
    for sink, temp in (([9.0, -9.0], [1.0, 1.0]), ([1.0, 2.0], [3.0, -2.0])):
        w["l0.mix.sink"], w["l0.mix.temp"] = torch.tensor(sink).to(torch.bfloat16), torch.tensor(temp).to(torch.bfloat16)
        want = O.forward(t, w, cfg)
        assert differ(want, base) > 0.1
        path, _, _ = checkpoint(tmp_path, cfg, weights=w)
        rp = TraceReplay.open(path, dtype, 64, device)
        for sizes in ([20], [1], [2, 9, 1]):
            check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


@pytest.mark.parametrize("device,dtype", RUNS)
def test_streams_mix_from_the_old_ones(tmp_path, device, dtype):
    """A mix that only hands each stream on to the next: read the other way round, or from streams already written, the logits
    are others."""
    cfg = config(50, 40, 3, [window(2, 1, 16, 24, 9, dense(24)), latent(2, 8, 8, 16, 24, 50.0, dense(24))], scale=0.5)
    w = O.random_weights(cfg, seed=21)
    shift = torch.roll(torch.eye(3), 1, 1)
    for name in [n for n in w if n.endswith(".mix") and ".hc" in n]:
        w[name] = (shift * torch.tensor([1.0, 0.5, 2.0])).to(torch.bfloat16)
        w[name.replace(".mix", ".out")] = torch.tensor([2.0, 0.0, -1.0]).to(torch.bfloat16)
    t = tokens(60, 50)
    want = O.forward(t, w, cfg)
    other = O.forward(t, {n: v.t() if n.endswith(".mix") and ".hc" in n else v for n, v in w.items()}, cfg)
    assert differ(other, want) > 0.3, "the case is blind"
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 64, device)
    for sizes in ([60], [33, 1], [2]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


# ------------------------------------------------------------------ generation through the engine's own entry point
def check_greedy(prompt, out, w, cfg, dtype, n):
    assert len(out) == n
    logits = O.forward(prompt + out[:-1], w, cfg)[len(prompt) - 1:]
    slack = (5e-4 if dtype == "float32" else 0.15) * logits.pow(2).mean().sqrt()
    for i, t in enumerate(out):
        assert logits[i, t] >= logits[i].max() - slack, f"token {i}: {t} is not the most likely one"


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name,blocks", [("even", 48), ("odd", 48), ("wide", 48), ("single", 7)])
def test_greedy_generation(tmp_path, name, blocks, device, dtype):
    """Chunked prompts beside decoding requests; with 7 blocks requests are pre-empted and computed again."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=8)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=blocks, max_num_seqs=3, max_model_len=112,
              max_num_batched_tokens=24)
    prompts = [tokens(n, cfg["vocab"], seed=n) for n in (1, 50, 45, 33, 2)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=16, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        check_greedy(p, list(o.outputs[0].token_ids), w, cfg, dtype, 16)
    assert (llm.engine.scheduler.num_preemptions > 0) == (blocks == 7)
    assert llm.engine.kv.num_free_blocks == blocks


@pytest.mark.parametrize("device,dtype", RUNS)
def test_prefix_caching(tmp_path, device, dtype):
    """All state is in pages, so a shared prefix is computed once."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS["even"], seed=9)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=48, max_num_seqs=2, max_model_len=160,
              enable_prefix_caching=True)
    shared = tokens(70, cfg["vocab"])
    for i, tail in enumerate((5, 9, 33)):
        p = shared + tokens(tail, cfg["vocab"], seed=tail)
        out = llm.generate([p], SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))[0]
        check_greedy(p, list(out.outputs[0].token_ids), w, cfg, dtype, 8)
        assert out.num_cached_tokens == (64 if i else 0)


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_sampling_and_scoring(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["odd"], seed=9)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=32, max_num_seqs=2, max_model_len=96)
    p = tokens(40, cfg["vocab"])
    sp = SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True)
    a, b = (llm.generate([p], sp)[0].outputs[0].token_ids for _ in range(2))
    assert list(a) == list(b)
    lp = llm.prompt_logprobs([p])[0]
    want = torch.log_softmax(O.forward(p, w, cfg), -1)
    for i in range(1, len(p)):
        assert abs(lp[i]["logprob"] - float(want[i - 1, p[i]])) < 1e-3


# ------------------------------------------------------------------ loading
def test_loader_reports_what_does_not_fit(tmp_path):
    cfg = CONFIGS["even"]
    _, good, _ = checkpoint(tmp_path, cfg)
    name = "l1.mix.uk"
    for change, message in (({name: None}, "missing"), ({"l0.mix.sink": good["l2.mix.sink"].clone()}, "unexpected"),
                            ({name: good[name].t().contiguous()}, "does not fit"), ({"l2.hc2.mix": good["l2.hc1.mix"].clone()}, "unexpected"),
                            ({"head": None}, "missing")):
        w = {k: v for k, v in {**good, **change}.items() if v is not None}
        path, _, _ = checkpoint(tmp_path, cfg, weights=w)
        with pytest.raises(ValueError, match=message):
            TraceReplay.open(path, "float32", 64, "cpu")


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][2].update(type="other"), "unknown mixer"), (lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "query heads"), (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.update(streams=9), "streams")])
def test_config_errors(tmp_path, change, message):
    cfg = json.loads(json.dumps(CONFIGS["even"]))
    change(cfg)
    path, _, _ = checkpoint(tmp_path, cfg, weights={"x": torch.zeros(1)})
    with pytest.raises(ValueError, match=message):
        TraceReplay.open(path, "float32", 64, "cpu")


def test_config_and_weight_update(tmp_path):
    from vllm_metax_b200 import ModelConfig
    from vllm_metax_b200.models import get_model_class

    cfg = CONFIGS["wide"]
    path, w, _ = checkpoint(tmp_path, cfg)
    mc = ModelConfig.from_pretrained(path)
    assert (mc.architecture, mc.vocab_size, mc.hidden_size, mc.num_hidden_layers) == ("Vetipel", 64, 64, 5)
    assert get_model_class("Vetipel").native_units == "streams" and mc.dtype == torch.bfloat16
    llm = LLM(path, device="cpu", dtype="float32", num_gpu_blocks=4, max_model_len=128, max_num_seqs=1)
    new = O.random_weights(cfg, seed=99)
    part = {k: v for k, v in new.items() if k.startswith(("l1.", "l0.hc2", "l0.mix.r1", "final.norm"))}
    assert llm.update_weights(part) == len(part)
    p = tokens(9, 64)
    check_greedy(p, list(llm.generate([p], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))[0].outputs[0].token_ids),
                 {**w, **part}, cfg, "float32", 6)


# ------------------------------------------------------------------ the replay program
@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[3]])
def test_trace_run_program(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["odd"], seed=5)
    a, b = tokens(70, cfg["vocab"], 1), tokens(3, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [65, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": [2]}, {"id": "a", "tokens": a[66:67], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[67:], "want": []}], "end": ["a"]}]
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, exe, "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "192",
                        "--device", device], input="\n".join(map(json.dumps, steps)) + "\n", text=True, capture_output=True,
                       timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    la, lb = O.forward(a, w, cfg), O.forward(b, w, cfg)
    read = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    check(read(0), la[[65, 3]], dtype)
    check(read(1), torch.stack([lb[2], la[66]]), dtype)
    assert not (out / "2.f32").exists()
