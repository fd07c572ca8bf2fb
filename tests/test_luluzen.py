"""The Luluzen model through the engine's own scheduler, block pool, state slots and step function, against the plain statement
in ``luluzen_oracle.py``.  Every test makes its own small checkpoint (sizes that differ from layer to layer, also ones that are 1
or not a multiple of anything) and runs on the CPU and, marked ``gpu``, through the kernels."""
import json
import os
import random
import subprocess
import sys

import pytest
import torch
from safetensors.torch import save_file

from tests import luluzen_oracle as O
from vllm_metax_b200 import LLM, SamplingParams
from vllm_metax_b200.entrypoints.trace_replay import TraceReplay

RUNS = [pytest.param("cpu", "float32"), pytest.param("cpu", "bfloat16"),
        pytest.param("cuda", "float32", marks=pytest.mark.gpu), pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
# rms of a position's logit error over the logits' rms: (a position, median of all).  A lost state or a wrong key gives 0.3 and
# more.
LIMIT = {"float32": (3e-4, 5e-5), "bfloat16": (0.2, 8e-2)}
pytestmark = pytest.mark.usefixtures("kernel_status_ok")


def lightning(heads, dim, vdim, decay, mlp=None):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def delta(left, right, scales=(0.7, 1.2), mlp=None, scale=None, temp=(0.35, 20), far=40):
    H, G, D, V = left
    h, g, d, v, conv = right
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale or D ** -0.5, "bias_max": far,
                 "q_temp": {"coef": temp[0], "every": temp[1]}},
        "right": {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "conv": conv}, "left_scale": scales[0], "right_scale": scales[1]}}


def memory(left, right, window, rot, scales=(1.3, 0.6), mlp=None, scale=None, cap=11.0, base=900.0, gate_cap=9.0):
    H, G, D, V = left
    h, d, v = right
    return {"type": "parallel_2", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale or D ** -0.5, "softcap": cap,
                 "mask": {"size": window}, "rot": {"base": base, "dims": rot}},
        "right": {"heads": h, "dim": d, "vdim": v, "gate_cap": gate_cap}, "left_scale": scales[0], "right_scale": scales[1]}}


def moe(experts, top, ff, limit=1.1):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, layers, loop=None, eps=1e-5, cap=25.0, **extra):
    c = {"architecture": "Luluzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers, **extra}
    return {**c, "loop": dict(zip(("start", "stop", "times"), loop))} if loop else c


CONFIGS = {
    # sizes the tensor-core paths take; a loop over four of six layers, feed-forwards of both kinds and none
    "even": config(200, 96, [
        memory((4, 4, 64, 24), (3, 24, 16), 37, 16, mlp=moe(6, 2, 40)),
        delta((6, 2, 48, 48), (4, 2, 32, 24, 4), mlp=moe(5, 3, 24, 0.7), far=33),
        lightning(3, 40, 24, [0.7, 0.95, 0.999], dense(88)),
        memory((6, 2, 40, 56), (2, 64, 40), 70, 40, mlp=None, base=5e4, cap=30.0),
        delta((4, 1, 104, 128), (2, 2, 72, 48, 2), (1.1, 0.4), dense(64), far=400),
        lightning(2, 16, 64, [0.9, 0.5], moe(4, 1, 16))], (1, 5, 2)),
    # nothing divides by eight; one head, one expert, one tap, a window of one token; the loop is the whole model
    "odd": config(101, 50, [
        memory((1, 1, 9, 11), (1, 7, 5), 1, 6, mlp=moe(1, 1, 7), scale=0.9),
        delta((3, 1, 10, 3), (3, 1, 9, 6, 1), mlp=dense(13), temp=(1.5, 1), far=21),
        lightning(1, 5, 3, [0.8]),
        delta((1, 1, 6, 5), (2, 2, 3, 1, 3), (1.0, 1.0), moe(3, 2, 9), far=12)], (0, 4, 3), eps=1e-3, cap=9.0),
    # wider heads than the tensor-core tiles; a loop of one layer that ends the model
    "wide": config(64, 64, [delta((2, 1, 200, 160), (2, 1, 136, 144, 4), mlp=dense(32)), lightning(1, 160, 136, [0.97]),
                            memory((2, 2, 264, 40), (1, 200, 24), 30, 48, mlp=moe(2, 1, 16))], (2, 3, 2), eps=1e-6),
    # no loop
    "plain": config(88, 72, [lightning(2, 24, 16, [0.99, 0.9], dense(40)), memory((2, 1, 32, 16), (2, 8, 8), 20, 8, mlp=dense(24)),
                             delta((2, 2, 16, 16), (2, 1, 16, 8, 5))], cap=40.0),
}


def checkpoint(tmp_path, cfg, seed=1, weights=None, dtype="float32"):
    """Returns (path, weights, config).  In bf16 a token may take another expert on a close call, and with it change everything
    after it: there every expert is taken, so that only the weights are left to the router."""
    cfg = json.loads(json.dumps(cfg))
    if dtype == "bfloat16":
        for l in cfg["layers"]:
            if l["mlp"] and l["mlp"]["kind"] == "moe":
                l["mlp"]["router"]["top"] = l["mlp"]["router"]["experts"]
    w = weights or O.random_weights(cfg, seed)
    d = tmp_path / "model"
    d.mkdir(exist_ok=True)
    save_file(w, str(d / "model.safetensors"))
    (d / "config.json").write_text(json.dumps(cfg))
    return str(d), w, cfg


def tokens(n, vocab, seed=0):
    return random.Random(seed * 1000 + n).choices(range(vocab), k=n)


def check(got, want, dtype, what="", at=None, loose=False):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    peak, mean = LIMIT[dtype]
    # a first token's read-out is normed whatever its size: where q . k is nearly nothing, 16 bits do not even tell its sign
    spare = len(err) // 10 if loose and dtype == "bfloat16" else 0
    assert at is None or float(err[at]) < peak, f"{what}: error {float(err[at]):.3g} at {at}"
    assert int((err >= peak).sum()) <= spare and float(err.median()) < mean, \
        f"{what}: error {float(err.max()):.3g} at position {int(err.argmax())}, {int((err >= peak).sum())} over, median {float(err.median()):.3g}"


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
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], dtype=dtype)
    rp = TraceReplay.open(path, dtype, 192, device, enforce_eager=True)
    got, want = [], []
    for n in (1, 2, 3, 17, 65, 110):
        t = tokens(n, cfg["vocab"])
        got.append(feed(rp, f"r{n}", t, [n]))
        want.append(O.forward(t, w, cfg))
        if dtype == "float32":
            check(got[-1], want[-1], dtype, f"{n} tokens")
    check(torch.cat(got), torch.cat(want), dtype, loose=True)
    assert rp.engine.kv.num_free_blocks == 3


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens(tmp_path, name, device, dtype):
    """One sequence cut in many ways: token by token from the start, pairs, odd sizes, page-sized portions, a long prompt and
    then single tokens - all the same logits.  State slots and pages are used again without being cleared."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=2, dtype=dtype)
    t = tokens(84, cfg["vocab"])
    want = O.forward(t, w, cfg)
    rp = TraceReplay.open(path, dtype, 128, device)
    whole = feed(rp, "x", t, [84])
    for sizes in ([1], [2], [3, 1, 2, 16], [5, 40, 1, 1, 30], [64], [63, 2, 65], [80, 2, 1]):
        got = feed(rp, "x", t, sizes)
        check(got, want, dtype, str(sizes), loose=True)
        check(got, whole.double(), dtype, str(sizes), loose=True)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_passes_every_window(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["even"], seed=3, dtype=dtype)
    t = tokens(150, cfg["vocab"])
    rp = TraceReplay.open(path, dtype, 192, device)
    check(feed(rp, "x", t, [10, 1]), O.forward(t, w, cfg), dtype, loose=True)


# ------------------------------------------------------------------ batches, pages and slots used again
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_equal_each_request_alone(tmp_path, name, device, dtype):
    """Up to four live requests in a pool that is nearly full all the time: portions beside single tokens, requests that sit
    out steps, pages and state slots handed on to the next request."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=4, dtype=dtype)
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
    got, want = [torch.cat(g) for g in got], [O.forward(t, w, cfg) for t in seqs]
    for i in range(len(seqs) if dtype == "float32" else 0):
        check(got[i], want[i], dtype, f"request {i}")
    check(torch.cat(got), torch.cat(want), dtype, loose=True)
    assert len(used) <= 5 < sum(map(pages, range(len(seqs)))) and rp.engine.kv.num_free_blocks == 5
    assert sorted(rp.engine.runner.free_state_slots) == list(range(4))


# ------------------------------------------------------------------ keys at the edge of a window, far keys, distances
def needle(cfg, w, vocab, pre, m, rotated):
    """Makes the left side of layer 0 a search for one key: large scores, no rotation in effect.  Returns the (query, key) pair of
    tokens that stands out most."""
    if rotated:                                                  # with a huge base only the first pair of a head turns
        w[pre + "q"][:2], w[pre + "k"][:2] = 0, 0
    for n in "qkv":
        if pre + n + ".b" in w:
            w[pre + n + ".b"].zero_()
    h = O.layer_norm(w["embed"].double(), w["l0.norm1"], 1e-6)
    q = O.unit_rms(O.linear(w, pre + "q", h), 1e-6) * w[pre + "q.norm"].double()
    k = O.unit_rms(O.linear(w, pre + "k", h), 1e-6) * w[pre + "k.norm"].double()
    s = q @ k.t()
    top = s.topk(2, -1).values
    a = int((top[:, 0] - top[:, 1]).argmax())
    return a, int(s[a].argmax())


def needle_case(vocab, a, b, at, far, seed):
    t = random.Random(seed).choices([x for x in range(vocab) if x not in (a, b)], k=at + 3)
    t[at - far], t[at] = b, a
    return t


def window_model(window):
    cfg = config(60, 48, [memory((1, 1, 32, 40), (1, 8, 8), window, 8, (3.0, 0.0), scale=3.0, cap=500.0, base=1e30)], eps=1e-6)
    w = O.random_weights(cfg, seed=11)
    w["l0.mix.left.sink"].fill_(-50.0)
    w["l0.mix.left.g"].zero_()
    return cfg, w, needle(cfg, w, 60, "l0.mix.left.", cfg["layers"][0]["mixer"]["left"], True)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("window", [2, 16, 64, 65, 100])
def test_window_edges(tmp_path, window, device, dtype):
    """The one key that matters sits just inside or just outside the window of the query that wants it; queries fall on both
    sides of page borders, in whole prompts, portions and decoding.  A window off by one changes these logits."""
    cfg, w, (a, b) = window_model(window)
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 256, device)
    for at in sorted({p for p in (window, window + 1, 63, 64, 65, 127, 128) if p >= window}):
        for far in (window - 1, window):
            if a == b and far == 0:
                continue
            t = needle_case(60, a, b, at, far, at)
            want = O.forward(t, w, cfg)
            wrong = json.loads(json.dumps(cfg))
            wrong["layers"][0]["mixer"]["left"]["mask"]["size"] += -1 if far < window else 1
            other = O.forward(t, w, wrong)
            assert (other[at] - want[at]).pow(2).mean().sqrt() > 0.2 * want.pow(2).mean().sqrt(), "the case is blind"
            for sizes in ([len(t)], [max(1, at - 1), 1], [max(1, at), 2], [2]):
                check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}", at=at, loose=True)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_far_keys_and_distance_buckets(tmp_path, device, dtype):
    """A key far back that alone matters, at page borders, at the first token and on both sides of a bucket's border, where
    neighbouring buckets differ by more than the other scores."""
    cfg = config(60, 48, [delta((1, 1, 32, 40), (1, 1, 8, 8, 2), (3.0, 0.0), scale=3.0, temp=(0.0, 5), far=300)], eps=1e-6)
    w = O.random_weights(cfg, seed=12, low=lambda i: (12, 5, 11))
    w["l0.mix.left.rel"].zero_()
    a, b = needle(cfg, w, 60, "l0.mix.left.", cfg["layers"][0]["mixer"]["left"], False)
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 512, device)
    for at, far in ((400, 400), (320, 192), (299, 171)):
        t = needle_case(60, a, b, at, far, at + far)
        want = O.forward(t, w, cfg)
        blind = O.forward([x if x != b else (a + 1 if a + 1 != b else a + 2) % 60 for x in t], w, cfg)
        assert (blind[at] - want[at]).pow(2).mean().sqrt() > 0.2 * want.pow(2).mean().sqrt(), "the case is blind"
        for sizes in ([len(t)], [at, 1], [256, 40, at - 296, 1]):
            check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}", at=at, loose=True)
    border = next(n for n in range(40, 300) if O.distance_bucket(n, 12, 300) != O.distance_bucket(n - 1, 12, 300))
    w["l0.mix.left.rel"][O.distance_bucket(border, 12, 300)] = -300.0      # the key is seen up to the border and not from it on
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 512, device)
    for at in (border + 1, 127, 128, 200):
        seen = [O.forward(needle_case(60, a, b, at, far, at), w, cfg) for far in (border - 1, border)]
        assert (seen[0][at] - seen[1][at]).pow(2).mean().sqrt() > 0.2 * seen[0].pow(2).mean().sqrt(), "the case is blind"
        for far, want in zip((border - 1, border), seen):
            t = needle_case(60, a, b, at, far, at)
            for sizes in ([len(t)], [at, 1], [at - 1, 3]):
                check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}", at=at, loose=True)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_sink_and_first_tokens(tmp_path, device, dtype):
    """A sink larger than every score leaves next to nothing of a head's output, one among the scores part of it; the first
    tokens see the fewest keys."""
    cfg = config(40, 48, [memory((2, 1, 16, 16), (1, 8, 8), 6, 8, (2.0, 0.1))])
    w = O.random_weights(cfg, seed=31)
    t = tokens(20, 40)
    for sink in ([9.0, -9.0], [1.0, 2.0]):
        w["l0.mix.left.sink"] = torch.tensor(sink).to(torch.bfloat16)
        want = O.forward(t, w, cfg)
        path, _, _ = checkpoint(tmp_path, cfg, weights=w)
        rp = TraceReplay.open(path, dtype, 64, device)
        for sizes in ([20], [1], [2, 9, 1]):
            check(feed(rp, "x", t, sizes), want, dtype, str(sizes), loose=True)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_passes_have_states_and_caches_of_their_own(tmp_path, device, dtype):
    """With a step vector that turns the stream around between two passes, a cache or state that both passes shared would hold
    the other pass's tokens."""
    cfg = config(50, 40, [delta((2, 1, 16, 24), (2, 1, 8, 8, 3), far=9), memory((2, 1, 16, 24), (1, 8, 8), 12, 8),
                          lightning(1, 8, 8, [0.9])], (0, 3, 2))
    w = O.random_weights(cfg, seed=21)
    w["loop.step"] = torch.stack([4.0 * torch.ones(40), -4.0 * torch.ones(40)]).mul(torch.linspace(-1, 1, 40)).to(torch.bfloat16)
    t = tokens(60, 50)
    want = O.forward(t, w, cfg)
    path, _, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 64, device)
    model = rp.engine.runner.model
    assert model.num_kv_layers() == len(rp.engine.runner.kv_caches) == 4
    assert model.layers[2].mixer.branches[0].state.shape[0] == 2
    for sizes in ([60], [33, 1], [2]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes), loose=True)


# ------------------------------------------------------------------ generation through the engine's own entry point
def check_greedy(prompt, out, w, cfg, dtype, n):
    assert len(out) == n
    logits = O.forward(prompt + out[:-1], w, cfg)[len(prompt) - 1:]
    slack = (2e-3 if dtype == "float32" else 0.4) * logits.pow(2).mean().sqrt()
    for i, t in enumerate(out):
        assert logits[i, t] >= logits[i].max() - slack, f"token {i}: {t} is not the most likely one"


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name,blocks", [("even", 48), ("odd", 48), ("wide", 48), ("plain", 7)])
def test_greedy_generation(tmp_path, name, blocks, device, dtype):
    """Chunked prompts beside decoding requests; with 7 blocks requests are pre-empted and computed again."""
    path, w, cfg = checkpoint(tmp_path, CONFIGS[name], seed=8, dtype=dtype)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=blocks, max_num_seqs=3, max_model_len=112,
              max_num_batched_tokens=24)
    prompts = [tokens(n, cfg["vocab"], seed=n) for n in (1, 50, 45, 33, 2)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=16, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        check_greedy(p, list(o.outputs[0].token_ids), w, cfg, dtype, 16)
    assert (llm.engine.scheduler.num_preemptions > 0) == (blocks == 7)
    assert llm.engine.kv.num_free_blocks == blocks


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_sampling_and_scoring(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["odd"], seed=9, dtype=dtype)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=32, max_num_seqs=2, max_model_len=96)
    p = tokens(40, cfg["vocab"])
    sp = SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True)
    a, b = (llm.generate([p], sp)[0].outputs[0].token_ids for _ in range(2))
    assert list(a) == list(b)
    lp = llm.prompt_logprobs([p])[0]
    want = torch.log_softmax(O.forward(p, w, cfg), -1)
    for i in range(1, len(p)):
        assert abs(lp[i]["logprob"] - float(want[i - 1, p[i]])) < 2e-3


# ------------------------------------------------------------------ loading
def test_loader_reports_what_does_not_fit(tmp_path):
    cfg = CONFIGS["even"]
    _, good, _ = checkpoint(tmp_path, cfg)
    name = "l1.mix.left.q"
    for change, message in (({name: None}, "missing"), ({"l2.mix.left.q": good[name].clone()}, "unexpected"),
                            ({name: good[name].t().contiguous()}, "does not fit"), ({"loop.step": None}, "missing")):
        w = {k: v for k, v in {**good, **change}.items() if v is not None}
        path, _, _ = checkpoint(tmp_path, cfg, weights=w)
        with pytest.raises(ValueError, match=message):
            TraceReplay.open(path, "float32", 64, "cpu")


@pytest.mark.parametrize("change,message", [
    (lambda c: c["loop"].update(stop=9), "loop"), (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["layers"][2].update(type="other"), "unknown mixer"), (lambda c: c["layers"][2]["mlp"].update(kind="other"), "feed-forward"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5]), "decays"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "query heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=3), "value heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(bias_max=3), "distance bias")])
def test_config_errors(tmp_path, change, message):
    cfg = json.loads(json.dumps(CONFIGS["even"]))
    change(cfg)
    path, _, _ = checkpoint(tmp_path, cfg, weights={"x": torch.zeros(1)})
    with pytest.raises(ValueError, match=message):
        TraceReplay.open(path, "float32", 64, "cpu")


def test_config_and_weight_update(tmp_path):
    from vllm_metax_b200 import ModelConfig
    from vllm_metax_b200.models import get_model_class

    cfg = CONFIGS["plain"]
    path, w, _ = checkpoint(tmp_path, cfg)
    mc = ModelConfig.from_pretrained(path)
    assert (mc.architecture, mc.vocab_size, mc.hidden_size, mc.num_hidden_layers) == ("Luluzen", 88, 72, 3)
    assert get_model_class("Luluzen").native_units == "parallel" and mc.dtype == torch.bfloat16
    llm = LLM(path, device="cpu", dtype="float32", num_gpu_blocks=4, max_model_len=128, max_num_seqs=1)
    new = O.random_weights(cfg, seed=99)
    part = {k: v for k, v in new.items() if k.startswith(("l1.", "l2.mix.left.rel", "l2.mix.right.A_log"))}
    assert llm.update_weights(part) == len(part)
    p = tokens(9, 88)
    check_greedy(p, list(llm.generate([p], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))[0].outputs[0].token_ids),
                 {**w, **part}, cfg, "float32", 6)


# ------------------------------------------------------------------ the replay program
@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[3]])
def test_trace_run_program(tmp_path, device, dtype):
    path, w, cfg = checkpoint(tmp_path, CONFIGS["odd"], seed=5, dtype=dtype)
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
