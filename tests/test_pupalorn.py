"""The Pupalorn model through the engine's own scheduler, block pool and step function, against the plain statement in
``pupalorn_oracle.py``.  Every test makes its own small checkpoint (sizes that differ from layer to layer, also ones that are 1
or not a multiple of anything) and runs on the CPU and, marked ``gpu``, through the kernels."""
import json
import os
import random
import subprocess
import sys

import pytest
import torch
from safetensors.torch import save_file

from tests import pupalorn_oracle as O
from vllm_metax_b200 import LLM, SamplingParams
from vllm_metax_b200.entrypoints.trace_replay import TraceReplay

RUNS = [pytest.param("cpu", "float32"), pytest.param("cpu", "bfloat16"),
        pytest.param("cuda", "float32", marks=pytest.mark.gpu), pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
# rms of a position's logit error over the logits' rms: (a position, median of all).  A lost page or a wrong key gives 0.3 and
# more.
LIMIT = {"float32": (2e-4, 5e-5), "bfloat16": (0.15, 6e-2)}
pytestmark = pytest.mark.usefixtures("kernel_status_ok")

LLAMA = {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 48}


def layer(heads, kv_heads, dim, vdim, window, rot, mlp=None, kv_from=None, base=700.0, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if window:
        m["mask"] = {"size": window}
    if scaling:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, identity=0):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff}}


def config(vocab, width, layers, eps=1e-5, mult=0.6, embed=5.0, **extra):
    return {"architecture": "Pupalorn", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "norm": {"eps": eps},
            "residual_mult": mult, "layers": layers, **extra}


CONFIGS = {
    # sizes the tensor-core paths take: grouped heads, key and value sizes of every tile, two sources of shared keys and
    # values whose readers look back further than they do
    "even": config(200, 96, [
        layer(6, 2, 48, 48, 37, 32, moe(6, 2, 40, 2), scaling=LLAMA),
        layer(4, 4, 64, 24, 70, 16, None, base=40.0),
        layer(6, 2, 48, 48, 90, 32, moe(5, 3, 24, 1), kv_from=0, scaling=LLAMA),
        layer(4, 1, 104, 128, 21, 96, moe(8, 1, 16)),
        layer(4, 4, 64, 24, 0, 16, moe(3, 2, 32, 3), kv_from=1, base=40.0),
        layer(8, 2, 136, 72, 50, 48, moe(4, 4, 16, 4), scaling=LLAMA, base=5e4)]),
    # nothing divides by eight; one head, one expert, a window of one token, every output an identity expert but one
    "odd": config(101, 50, [
        layer(1, 1, 9, 11, 5, 6, moe(3, 1, 10, 2), scale=0.9),
        layer(3, 1, 10, 3, 64, 10, moe(1, 2, 7, 4)),
        layer(1, 1, 9, 11, 1, 6, None, kv_from=0),
        layer(7, 7, 6, 5, 19, 2, moe(4, 4, 12), scaling=dict(LLAMA, factor=2.0))], eps=1e-3, mult=1.0, embed=1.0),
    # wider heads than the tensor-core tiles: prompts through the decode kernel, and the CUDA cores
    "wide": config(64, 64, [layer(2, 1, 200, 160, 33, 128, moe(2, 1, 16, 1)), layer(2, 2, 264, 40, 0, 48, None),
                            layer(2, 2, 264, 40, 30, 48, moe(2, 2, 16, 1), kv_from=1)], eps=1e-6, mult=0.3),
}


def checkpoint(tmp_path, cfg, seed=1, weights=None, dtype="float32"):
    """In bf16 a token may take another expert on a close call, and with it change everything after it: there the corrections
    alone decide, another choice for every layer."""
    w = weights or O.random_weights(cfg, seed, decisive=dtype == "bfloat16")
    d = tmp_path / "model"
    d.mkdir(exist_ok=True)
    save_file(w, str(d / "model.safetensors"))
    (d / "config.json").write_text(json.dumps(cfg))
    return str(d), w


def tokens(n, vocab, seed=0):
    return random.Random(seed * 1000 + n).choices(range(vocab), k=n)


def check(got, want, dtype, what="", loose=False, at=None):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    peak, mean = LIMIT[dtype]
    spare = len(err) // 10 if loose and dtype == "bfloat16" else 0
    assert at is None or float(err[at]) < peak, f"{what}: error {float(err[at]):.3g} at {at}"
    assert int((err >= peak).sum()) <= spare and float(err.median()) < mean, \
        f"{what}: error {float(err.max()):.3g} at position {int(err.argmax())}, {int((err >= peak).sum())} over, median {float(err.median()):.3g}"


def feed(rp, rid, toks, sizes, end=True):
    """All logits of one request fed in portions of ``sizes`` (the last one repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        done = end and at + n == len(toks)
        out.append(rp.step([{"id": rid, "tokens": toks[at: at + n], "want": list(range(n))}], [rid] if done else []))
        at, k = at + n, k + 1
    return torch.cat(out)


# ------------------------------------------------------------------ prompts, portions, decoding
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts(tmp_path, name, device, dtype):
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, dtype=dtype)
    rp = TraceReplay.open(path, dtype, 256, device, enforce_eager=True)
    for n in (1, 2, 3, 17, 64, 65, 150):
        t = tokens(n, cfg["vocab"])
        check(feed(rp, f"r{n}", t, [n]), O.forward(t, w, cfg), dtype, f"{n} tokens")
    assert rp.engine.kv.num_free_blocks == 4


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens(tmp_path, name, device, dtype):
    """One sequence cut in many ways: token by token from the start, pairs, odd sizes, page-sized portions, a long prompt and
    then single tokens - all the same logits."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=2, dtype=dtype)
    t = tokens(140, cfg["vocab"])
    want = O.forward(t, w, cfg)
    rp = TraceReplay.open(path, dtype, 192, device)
    whole = feed(rp, "x", t, [140])
    for sizes in ([1], [2], [3, 1, 2, 16], [5, 64, 1, 1, 30], [64], [63, 2, 65], [131, 2, 1]):
        got = feed(rp, "x", t, sizes)
        check(got, want, dtype, str(sizes))
        check(got, whole.double(), dtype, str(sizes))


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_passes_every_window(tmp_path, device, dtype):
    cfg = CONFIGS["even"]
    path, w = checkpoint(tmp_path, cfg, seed=3, dtype=dtype)
    t = tokens(210, cfg["vocab"])
    rp = TraceReplay.open(path, dtype, 256, device)
    check(feed(rp, "x", t, [10, 1]), O.forward(t, w, cfg), dtype)


# ------------------------------------------------------------------ batches and pages used again
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_equal_each_request_alone(tmp_path, name, device, dtype):
    """Up to four live requests in a pool that is nearly full all the time: portions beside single tokens, requests that sit
    out steps, pages handed on to the next request."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=4, dtype=dtype)
    rng = random.Random(5)
    lens = [1, 2, 130, 70, 33, 64, 100, 3, 90, 65]
    seqs = [tokens(n, cfg["vocab"], seed=7) for n in lens]
    want = [O.forward(t, w, cfg) for t in seqs]
    got = [[] for _ in seqs]
    rp = TraceReplay.open(path, dtype, 448, device)
    pages = lambda i: -(-lens[i] // 64)
    waiting, live, at = list(range(len(seqs))), [], [0] * len(seqs)
    used = set()
    while waiting or live:
        while waiting and len(live) < 4 and sum(map(pages, live)) + pages(waiting[0]) <= 7:
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
    for i in range(len(seqs)):
        check(torch.cat(got[i]), want[i], dtype, f"request {i}")
    assert len(used) <= 7 < sum(map(pages, range(len(seqs))))
    assert rp.engine.kv.num_free_blocks == 7


# ------------------------------------------------------------------ keys at the edge of a window, far keys
def needle_model(windows, rot=8):
    """One attention layer (with two windows: a second one that reads the first one's keys and values) without rotation whose
    scores are large: attention goes to the key that fits the query best.  Returns the checkpoint's weights and the (query,
    key) pair of tokens that stands out in the last layer."""
    ls = [layer(1, 1, 32, 40, windows[0], rot, base=1e30, scale=3.0)]
    if len(windows) > 1:
        ls.append(layer(1, 1, 32, 40, windows[1], rot, base=1e30, scale=3.0, kv_from=0))
    cfg = config(60, 48, ls, eps=1e-6, mult=1.0, embed=0.6)      # (the attention's output outweighs the embedding)
    w = O.random_weights(cfg, seed=11)
    w["l0.mix.q"][0], w["l0.mix.k"][0] = 0, 0                 # the one pair that turns (base^0) holds nothing
    w["l0.mix.q"][rot // 2], w["l0.mix.k"][rot // 2] = 0, 0
    if len(windows) > 1:
        w["l0.mix.o"].mul_(0.0)                               # the first layer only fills the cache
        w["l1.mix.q"], w["l1.mix.q.norm"] = w["l0.mix.q"].clone(), w["l0.mix.q.norm"].clone()
        w["l1.norm1"] = w["l0.norm1"].clone()
    h = O.norm_around_one(w["embed"].double() * 0.6, w["l0.norm1"], 1e-6)
    q = O.unit_rms(O.linear(w, "l0.mix.q", h), 1e-6) * w["l0.mix.q.norm"].double()
    k = O.unit_rms(O.linear(w, "l0.mix.k", h), 1e-6) * w["l0.mix.k.norm"].double()
    s = q @ k.t()
    top = s.topk(2, -1).values
    a = int((top[:, 0] - top[:, 1]).argmax())
    return cfg, w, a, int(s[a].argmax())


def needle_case(cfg, vocab, a, b, at, far, seed):
    t = random.Random(seed).choices([x for x in range(vocab) if x not in (a, b)], k=at + 3)
    t[at - far], t[at] = b, a
    return t


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("windows", [(1,), (2,), (16,), (64,), (65,), (100,), (9, 70), (70, 9)])
def test_window_edges(tmp_path, windows, device, dtype):
    """The one key that matters sits just inside or just outside the window of the query that wants it; queries fall on both
    sides of page borders, in whole prompts, portions and decoding.  A window off by one changes these logits; a layer that
    reads another layer's keys uses its own window."""
    cfg, w, a, b = needle_model(windows)
    path, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 256, device)
    window = windows[-1]
    wrong = []
    for d in (-1, 1):
        c = json.loads(json.dumps(cfg))
        c["layers"][-1]["mixer"]["mask"]["size"] = window + d
        wrong.append(c)
    for at in sorted({p for p in (window, window + 1, 63, 64, 65, 127, 128, 190) if p >= window}):
        for far in (window - 1, window):
            if a == b and far == 0:
                continue
            t = needle_case(cfg, 60, a, b, at, far, at)
            want = O.forward(t, w, cfg)
            if window > 1:
                other = O.forward(t, w, wrong[0 if far < window else 1])
                assert (other[at] - want[at]).pow(2).mean().sqrt() > 0.2 * want.pow(2).mean().sqrt(), "the case is blind"
            for sizes in ([len(t)], [max(1, at - 1), 1], [max(1, at), 2], [2]):
                check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}", loose=True, at=at)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("window", [0, 900])
def test_far_keys(tmp_path, window, device, dtype):
    """A key hundreds of tokens back that alone matters: on page borders, at the first token, in prompts and in decoding
    (where the context is split over several CTAs)."""
    cfg, w, a, b = needle_model((window,))
    path, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 1024, device)
    for at, far in ((700, 700), (820, 692), (899, 771), (899, 899), (840, 521)):
        t = needle_case(cfg, 60, a, b, at, far, at + far)
        want = O.forward(t, w, cfg)
        blind = O.forward([x if x != b else (a + 1 if a + 1 != b else a + 2) % 60 for x in t], w, cfg)
        assert (blind[at] - want[at]).pow(2).mean().sqrt() > 0.2 * want.pow(2).mean().sqrt(), "the case is blind"
        for sizes in ([len(t)], [at, 1], [512, 130, at - 642, 1]):
            check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}", loose=True, at=at)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_readers_see_the_source_layers_keys(tmp_path, device, dtype):
    """A reader of shared keys and values follows every change of its source's projections, and nothing of another layer's."""
    cfg = config(50, 40, [layer(2, 1, 16, 24, 12, 8), layer(2, 1, 16, 24, 30, 8), layer(4, 1, 16, 24, 18, 8, kv_from=0),
                          layer(2, 1, 16, 24, 25, 8, kv_from=1)])
    w = O.random_weights(cfg, seed=21)
    t = tokens(70, 50)
    base = O.forward(t, w, cfg)
    w["l0.mix.o"].zero_()                                    # layer 0 acts through its cache alone
    w["l0.mix.v"].mul_(-1.0)
    want = O.forward(t, w, cfg)
    assert (want - base).pow(2).mean().sqrt() > 0.2 * base.pow(2).mean().sqrt()
    path, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 128, device)
    assert rp.engine.runner.model.num_kv_layers() == 2 and len(rp.engine.runner.kv_caches) == 2
    for sizes in ([70], [33, 1], [2]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("which", ["identity", "real", "both"])
def test_identity_experts_in_the_model(tmp_path, which, device, dtype):
    """The correction forces every token to identity experts, to real ones, or to one of each: it moves the choice and not
    the weights."""
    cfg = config(40, 48, [layer(2, 2, 16, 16, 8, 8, moe(4, 2, 24, 3))], embed=2.0)
    w = O.random_weights(cfg, seed=31)
    c = {"identity": [0, 0, 0, 0, 9, 0, 8], "real": [0, 9, 8, 0, 0, 0, 0], "both": [0, 0, 9, 0, 0, 8, 0]}[which]
    w["l0.mlp.correction"] = torch.tensor(c).to(torch.bfloat16)
    t = tokens(40, 40)
    want = O.forward(t, w, cfg)
    path, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 64, device)
    for sizes in ([40], [9, 1]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


# ------------------------------------------------------------------ generation through the engine's own entry point
def check_greedy(prompt, out, w, cfg, dtype, n):
    assert len(out) == n
    logits = O.forward(prompt + out[:-1], w, cfg)[len(prompt) - 1:]
    slack = (1e-3 if dtype == "float32" else 0.3) * logits.pow(2).mean().sqrt()
    for i, t in enumerate(out):
        assert logits[i, t] >= logits[i].max() - slack, f"token {i}: {t} is not the most likely one"


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name,blocks", [("even", 64), ("odd", 64), ("wide", 64), ("even", 8)])
def test_greedy_generation(tmp_path, name, blocks, device, dtype):
    """Chunked prompts beside decoding requests; with 8 blocks requests are pre-empted and computed again."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=8, dtype=dtype)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=blocks, max_num_seqs=3, max_model_len=160,
              max_num_batched_tokens=24)
    prompts = [tokens(n, cfg["vocab"], seed=n) for n in (1, 60, 5, 33, 2, 48, 17)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=25, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        check_greedy(p, list(o.outputs[0].token_ids), w, cfg, dtype, 25)
    assert (llm.engine.scheduler.num_preemptions > 0) == (blocks == 8)
    assert llm.engine.kv.num_free_blocks == blocks


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_sampling_scoring_and_prefix_caching(tmp_path, device, dtype):
    cfg = CONFIGS["odd"]
    path, w = checkpoint(tmp_path, cfg, seed=9, dtype=dtype)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=32, max_num_seqs=2, max_model_len=96,
              enable_prefix_caching=True)
    p = tokens(40, cfg["vocab"])
    a = llm.generate([p], SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True))
    b = llm.generate([p], SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True))
    assert list(a[0].outputs[0].token_ids) == list(b[0].outputs[0].token_ids)
    out = llm.generate([p[:35]], SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))[0]
    assert out.num_cached_tokens == 32                        # two full blocks of the earlier prompt
    check_greedy(p[:35], list(out.outputs[0].token_ids), w, cfg, dtype, 8)
    lp = llm.prompt_logprobs([p])[0]
    want = torch.log_softmax(O.forward(p, w, cfg), -1)
    for i in range(1, len(p)):
        assert abs(lp[i]["logprob"] - float(want[i - 1, p[i]])) < 2e-3


# ------------------------------------------------------------------ loading
def test_loader_reports_what_does_not_fit(tmp_path):
    cfg = CONFIGS["even"]
    _, good = checkpoint(tmp_path, cfg)
    name = "l1.mix.k"
    for change, message in (({name: None}, "missing"), ({"l2.mix.k": good[name].clone()}, "unexpected"),
                            ({name: good[name].t().contiguous()}, "does not fit")):
        w = {k: v for k, v in {**good, **change}.items() if v is not None}
        path, _ = checkpoint(tmp_path, cfg, weights=w)
        with pytest.raises(ValueError, match=message):
            TraceReplay.open(path, "float32", 64, "cpu")


@pytest.mark.parametrize("change,message", [({"kv_from": 4}, "kv_from"), ({"kv_from": 2}, "kv_from"),
                                            ({"kv_from": 0, "vdim": 32}, "sizes"), ({"kv_heads": 5}, "query heads")])
def test_config_errors(tmp_path, change, message):
    cfg = json.loads(json.dumps(CONFIGS["even"]))
    cfg["layers"][2 if "kv_from" in change else 0]["mixer"].update(change)
    path, _ = checkpoint(tmp_path, cfg, weights={"x": torch.zeros(1)})
    with pytest.raises(ValueError, match=message):
        TraceReplay.open(path, "float32", 64, "cpu")


def test_config_and_weight_update(tmp_path):
    from vllm_metax_b200 import ModelConfig
    from vllm_metax_b200.models import get_model_class

    cfg = CONFIGS["even"]
    path, w = checkpoint(tmp_path, cfg)
    mc = ModelConfig.from_pretrained(path)
    assert (mc.architecture, mc.vocab_size, mc.hidden_size, mc.num_hidden_layers) == ("Pupalorn", 200, 96, 6)
    assert get_model_class("Pupalorn").native_units == "gqa" and mc.dtype == torch.bfloat16
    llm = LLM(path, device="cpu", dtype="float32", num_gpu_blocks=4, max_model_len=128, max_num_seqs=1)
    new = O.random_weights(cfg, seed=99)
    part = {k: v for k, v in new.items() if k.startswith(("l1.", "l4.", "head"))}
    assert llm.update_weights(part) == len(part)
    p = tokens(9, 200)
    check_greedy(p, list(llm.generate([p], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))[0].outputs[0].token_ids),
                 {**w, **part}, cfg, "float32", 6)


# ------------------------------------------------------------------ the replay program
@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[3]])
def test_trace_run_program(tmp_path, device, dtype):
    cfg = CONFIGS["odd"]
    path, w = checkpoint(tmp_path, cfg, seed=5, dtype=dtype)
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
