"""The Naguzen model through the engine's own scheduler, block pool, state slots and step function, against the plain
statement in ``naguzen_oracle.py``.  Every test makes its own small checkpoint (sizes that differ from layer to layer, also
ones that are 1 or not a multiple of anything) and runs on the CPU and, marked ``gpu``, through the kernels."""
import json
import os
import random
import subprocess
import sys

import pytest
import torch
from safetensors.torch import save_file

from tests import naguzen_oracle as O
from vllm_metax_b200 import LLM, SamplingParams
from vllm_metax_b200.entrypoints.trace_replay import TraceReplay

RUNS = [pytest.param("cpu", "float32"), pytest.param("cpu", "bfloat16"),
        pytest.param("cuda", "float32", marks=pytest.mark.gpu), pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)]
# rms of a position's logit error over the logits' rms: (any position, mean of all).  A lost state or a wrong key gives 0.3
# and more; bf16 activations of these small random models leave up to a tenth at single positions.
LIMIT = {"float32": (2e-4, 5e-5), "bfloat16": (0.2, 8e-2)}
pytestmark = pytest.mark.usefixtures("kernel_status_ok")


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, base=900.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale or (dim + rot_dim) ** -0.5}}


def gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff},
            "shared": {"ff": shared} if shared else None}


def config(vocab, width, taps, eps, layers, **extra):
    return {"architecture": "Naguzen", "vocab": vocab, "width": width, "canon": {"taps": taps}, "norm": {"eps": eps},
            "layers": [dict(l, mlp=f) for l, f in layers], **extra}


CONFIGS = {
    # sizes the tensor-core paths take, two windows, every feed-forward form
    "even": config(200, 96, 3, 1e-5, [
        (rglru(120, 3, 2), None), (latent(3, 24, 16, 40, 48, 32, 37), dense(136)),
        (gla(2, 40, 24, 5.0), moe(6, 2, 24, 0.6, 40)), (latent(5, 16, 8, 16, 40, 72, 70, base=40.0), moe(9, 3, 16, 2.0, None)),
        (rglru(64, 1, 4), dense(56))]),
    # nothing divides by eight; one head, one block, one expert per token, one tap
    "odd": config(101, 50, 1, 1e-3, [
        (latent(1, 9, 6, 11, 13, 15, 5), moe(3, 1, 10, 1.9, 6)), (gla(3, 7, 5, 1.0), dense(30)),
        (rglru(35, 5, 1), moe(4, 4, 12, 1.0, None)), (latent(7, 10, 2, 4, 22, 31, 64), None)]),
    # recurrent layers only: no layer owns pages
    "recurrent": config(64, 64, 5, 1e-6, [(gla(1, 136, 72, 3.0), dense(40)), (rglru(48, 2, 3), None)]),
}


def checkpoint(tmp_path, cfg, seed=1, weights=None, rank=None):
    cfg = dict(cfg, decay_rank=rank or 12)
    w = weights or O.random_weights(cfg, seed)
    d = tmp_path / "model"
    d.mkdir(exist_ok=True)
    save_file(w, str(d / "model.safetensors"))
    (d / "config.json").write_text(json.dumps({k: v for k, v in cfg.items() if k != "decay_rank"}))
    return str(d), w


def tokens(n, vocab, seed=0):
    return random.Random(seed * 1000 + n).choices(range(vocab), k=n)


def check(got, want, dtype, what=""):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    bad = int(err.argmax())
    peak, mean = LIMIT[dtype]
    assert float(err.max()) < peak and float(err.mean()) < mean, \
        f"{what}: error {float(err.max()):.3g} at position {bad}, mean {float(err.mean()):.3g}"


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
    path, w = checkpoint(tmp_path, cfg)
    rp = TraceReplay.open(path, dtype, 256, device, enforce_eager=True)
    for n in (1, 2, 3, 17, 64, 65, 150):
        t = tokens(n, cfg["vocab"])
        check(feed(rp, f"r{n}", t, [n]), O.forward(t, w, cfg), dtype, f"{n} tokens")
    assert rp.engine.kv.num_free_blocks == 4 and len(rp.engine.runner.state_slots) == 0


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens(tmp_path, name, device, dtype):
    """One sequence cut in many ways: token by token from the start, pairs, odd sizes, page- and chunk-sized portions, a
    long prompt and then single tokens - all the same logits."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=2)
    t = tokens(140, cfg["vocab"])
    want = O.forward(t, w, cfg)
    rp = TraceReplay.open(path, dtype, 192, device)
    for sizes in ([1], [2], [3, 1, 2, 16], [5, 64, 1, 1, 30], [17], [64], [63, 2, 65], [100, 1], [131, 2, 1], [1, 2, 137]):
        check(feed(rp, "x", t, sizes), want, dtype, str(sizes))


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_passes_every_window(tmp_path, device, dtype):
    cfg = CONFIGS["even"]
    path, w = checkpoint(tmp_path, cfg, seed=3)
    t = tokens(230, cfg["vocab"])
    rp = TraceReplay.open(path, dtype, 256, device)
    check(feed(rp, "x", t, [10, 1]), O.forward(t, w, cfg), dtype)


# ------------------------------------------------------------------ batches, pages and slots used again
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_equal_each_request_alone(tmp_path, name, device, dtype):
    """Up to four live requests in a pool that is nearly full all the time: portions beside single tokens, requests that
    sit out steps, pages and slots handed on to the next request."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=4)
    rng = random.Random(5)
    lens = [1, 2, 130, 70, 33, 64, 100, 3, 90, 65]
    seqs = [tokens(n, cfg["vocab"], seed=7) for n in lens]
    want = [O.forward(t, w, cfg) for t in seqs]
    got = [[] for _ in seqs]
    rp = TraceReplay.open(path, dtype, 448, device)
    pages = lambda i: -(-lens[i] // 64)
    waiting, live, at = list(range(len(seqs))), [], [0] * len(seqs)
    used_slots, used_pages = set(), set()
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
        used_slots |= set(rp.engine.runner.state_slots.values())
        used_pages |= {b for r in rp.engine.scheduler.running for b in r.block_ids}
        rp.step([], end)
        for e in entries:
            n = len(e["tokens"])
            got[e["id"]].append(logits[:n])
            logits = logits[n:]
        live = [i for i in live if i not in end]
    for i in range(len(seqs)):
        check(torch.cat(got[i]), want[i], dtype, f"request {i}")
    assert used_slots <= set(range(4)) and len(used_pages) <= 7 < sum(map(pages, range(len(seqs))))
    assert rp.engine.kv.num_free_blocks == 7


@pytest.mark.parametrize("device,dtype", RUNS)
def test_nothing_leaks_from_a_freed_slot(tmp_path, device, dtype):
    cfg = CONFIGS["even"]
    path, w = checkpoint(tmp_path, cfg, seed=6)
    rp = TraceReplay.open(path, dtype, 128, device, max_live=1)
    first, second = tokens(90, cfg["vocab"], 1), tokens(9, cfg["vocab"], 2)
    alone = feed(rp, "a", second, [9])
    for sizes in ([1], [2], [4, 1]):
        feed(rp, "b", first, [64, 1])
        again = feed(rp, "c", second, sizes)
        check(again, O.forward(second, w, cfg), dtype, str(sizes))
        check(again, alone.double(), dtype, str(sizes))


# ------------------------------------------------------------------ keys at the edge of a window
def needle_model(window):
    """One latent layer without rotation or convolution whose scores are large: attention goes to the key that fits the
    query best.  Returns the checkpoint's weights and a (query token, key token) pair that stands out."""
    cfg = config(60, 48, 2, 1e-6, [(latent(1, 32, 8, 40, 48, 40, window, scale=3.0), None)])
    w = O.random_weights(cfg, seed=11)
    w["l0.canon1"].zero_()
    w["l0.mix.uq"].view(1, 40, 48)[:, 32:] = 0               # no rotated part: a score depends on the two tokens only
    emb = w["embed"].double()
    cq = O.unit_rms(O.linear(w, "l0.mix.dq", emb), 1e-6) * w["l0.mix.dq.norm"].double()
    c = O.unit_rms(O.linear(w, "l0.mix.dkv", emb)[:, :40], 1e-6) * w["l0.mix.dkv.norm"].double()
    q, k = O.linear(w, "l0.mix.uq", cq)[:, :32], O.linear(w, "l0.mix.uk", c)
    s = q @ k.t()
    top = s.topk(2, -1).values
    a = int((top[:, 0] - top[:, 1]).argmax())
    b = int(s[a].argmax())
    return cfg, w, a, b


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("window", [1, 2, 16, 64, 65, 100])
def test_window_edges(tmp_path, window, device, dtype):
    """The one key that matters sits just inside or just outside the window of the query that wants it; queries fall on
    both sides of page borders, in whole prompts, portions and decoding.  A window off by one changes these logits."""
    cfg, w, a, b = needle_model(window)
    path, _ = checkpoint(tmp_path, cfg, weights=w)
    rp = TraceReplay.open(path, dtype, 256, device)
    filler = [t for t in range(cfg["vocab"]) if t not in (a, b)]
    wrong = [dict(cfg, layers=[latent(1, 32, 8, 40, 48, 40, window + d, scale=3.0) | {"mlp": None}]) for d in (-1, 1)]
    for at in sorted({p for p in (window, window + 1, 63, 64, 65, 127, 128, 190) if p >= window}):
        for far in (window - 1, window):
            if a == b and far == 0:
                continue
            t = random.Random(at).choices(filler, k=at + 3)
            t[at - far], t[at] = b, a
            want = O.forward(t, w, cfg)
            if window > 1:
                other = O.forward(t, w, wrong[0 if far < window else 1])
                assert (other[at] - want[at]).pow(2).mean().sqrt() > 0.2 * want.pow(2).mean().sqrt(), "the case is blind"
            for sizes in ([len(t)], [max(1, at - 1), 1], [max(1, at), 2], [2]):
                check(feed(rp, "x", t, sizes), want, dtype, f"query {at}, key {far} back, {sizes}")


# ------------------------------------------------------------------ generation through the engine's own entry point
def check_greedy(prompt, out, w, cfg, dtype, n):
    assert len(out) == n
    logits = O.forward(prompt + out[:-1], w, cfg)[len(prompt) - 1:]
    slack = (1e-3 if dtype == "float32" else 0.3) * logits.pow(2).mean().sqrt()
    for i, t in enumerate(out):
        assert logits[i, t] >= logits[i].max() - slack, f"token {i}: {t} is not the most likely one"


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name,blocks", [("even", 64), ("odd", 64), ("recurrent", 64), ("even", 8)])
def test_greedy_generation(tmp_path, name, blocks, device, dtype):
    """Chunked prompts beside decoding requests, more requests than state slots; with 8 blocks requests are pre-empted and
    computed again."""
    cfg = CONFIGS[name]
    path, w = checkpoint(tmp_path, cfg, seed=8)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=blocks, max_num_seqs=3, max_model_len=160,
              max_num_batched_tokens=24)
    prompts = [tokens(n, cfg["vocab"], seed=n) for n in (1, 60, 5, 33, 2, 48, 17)]
    outs = llm.generate(prompts, SamplingParams(max_tokens=25, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        check_greedy(p, list(o.outputs[0].token_ids), w, cfg, dtype, 25)
    assert (llm.engine.scheduler.num_preemptions > 0) == (blocks == 8)
    assert not llm.engine.runner.state_slots and llm.engine.kv.num_free_blocks == blocks


@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[2]])
def test_sampling_and_scoring(tmp_path, device, dtype):
    cfg = CONFIGS["odd"]
    path, w = checkpoint(tmp_path, cfg, seed=9)
    llm = LLM(path, device=device, dtype=dtype, block_size=16, num_gpu_blocks=32, max_num_seqs=2, max_model_len=96)
    p = tokens(20, cfg["vocab"])
    a = llm.generate([p], SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True))
    b = llm.generate([p], SamplingParams(max_tokens=12, temperature=0.8, top_k=20, seed=3, ignore_eos=True))
    assert list(a[0].outputs[0].token_ids) == list(b[0].outputs[0].token_ids)
    lp = llm.prompt_logprobs([p])[0]
    want = torch.log_softmax(O.forward(p, w, cfg), -1)
    for i in range(1, len(p)):
        assert abs(lp[i]["logprob"] - float(want[i - 1, p[i]])) < 2e-3


# ------------------------------------------------------------------ loading
def test_loader_reports_what_does_not_fit(tmp_path):
    cfg = CONFIGS["even"]
    _, good = checkpoint(tmp_path, cfg)
    name = "l1.mix.uk"
    for change, message in (({name: None}, "missing"), ({"l0.mix.extra": torch.zeros(3)}, "unexpected"),
                            ({name: good[name].t().contiguous()}, "does not fit")):
        w = {k: v for k, v in {**good, **change}.items() if v is not None}
        path, _ = checkpoint(tmp_path, cfg, weights=w)
        with pytest.raises(ValueError, match=message):
            TraceReplay.open(path, "float32", 64, "cpu")


def test_config_and_weight_update(tmp_path):
    from vllm_metax_b200 import ModelConfig
    from vllm_metax_b200.models import get_model_class

    cfg = CONFIGS["even"]
    path, w = checkpoint(tmp_path, cfg)
    mc = ModelConfig.from_pretrained(path)
    assert (mc.architecture, mc.vocab_size, mc.hidden_size, mc.num_hidden_layers) == ("Naguzen", 200, 96, 5)
    assert get_model_class("Naguzen").native_units == "hybrid" and mc.dtype == torch.bfloat16
    llm = LLM(path, device="cpu", dtype="float32", num_gpu_blocks=4, max_model_len=128, max_num_seqs=1)
    new = O.random_weights(dict(cfg, decay_rank=12), seed=99)
    part = {k: v for k, v in new.items() if k.startswith(("l1.", "l4.", "head"))}
    assert llm.update_weights(part) == len(part)
    p = tokens(9, 200)
    check_greedy(p, list(llm.generate([p], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))[0].outputs[0].token_ids),
                 {**w, **part}, cfg, "float32", 6)


@pytest.mark.parametrize("rank", [1, 5, 24])
def test_decay_rank_comes_from_the_checkpoint(tmp_path, rank):
    cfg = config(40, 24, 2, 1e-5, [(gla(2, 8, 8, 2.0), None), (rglru(16, 2, 2), dense(16))])
    path, w = checkpoint(tmp_path, cfg, rank=rank)
    t = tokens(12, 40)
    check(feed(TraceReplay.open(path, "float32", 64, "cpu"), "x", t, [5]), O.forward(t, w, cfg), "float32")


# ------------------------------------------------------------------ the replay program
@pytest.mark.parametrize("device,dtype", [RUNS[0], RUNS[3]])
def test_trace_run_program(tmp_path, device, dtype):
    cfg = CONFIGS["odd"]
    path, w = checkpoint(tmp_path, cfg, seed=5)
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
