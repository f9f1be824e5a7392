"""Doderax on the device against its float64 oracle: whole prompts, single tokens, portions, batches, reused pages and slots,
greedy generation through the public entry points. float32 models are compared tightly (they compute everything in true 32
bits), bfloat16 models within what bfloat16 rounding of weights-times-activations leaves."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from llaisys_b200.models import Doderax
from oracle import doderax as oracle
from tests import doderax_cases as cases

pytestmark = pytest.mark.gpu
DT = {"f32": llaisys.DataType.F32, "f16": llaisys.DataType.F16, "bf16": llaisys.DataType.BF16}
# relative rms error of a row of logits (mean taken off): float32 rounding; bfloat16 rounding through a few layers
TOL = {"f32": 2e-5, "f16": 0.01, "bf16": 0.06}


def make(cfg, w, dtype):
    return Doderax(config=cfg, state_dict=w, dtype=DT[dtype])


def row_errors(got, want):
    d = torch.as_tensor(got).double() - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / spread


def check(got, want, dtype, what=""):
    err = row_errors(got, want)
    assert err.max().item() <= TOL[dtype], f"{what}: row {int(err.argmax())} of {len(err)} is off by {err.max().item():.2e}"


@pytest.fixture(scope="module", params=sorted(cases.CASES))
def ready(request, cuda_device):
    """A case with the oracle's logits of one sequence."""
    cfg, w = cases.case(request.param)
    toks = cases.tokens(cfg, 150)
    logits, streams = oracle.forward(cfg, w, toks)
    return request.param, cfg, w, toks, logits, streams


@pytest.mark.parametrize("dtype", ["f32", "f16", "bf16"])
def test_whole_prompt_and_every_layer(ready, dtype):
    name, cfg, w, toks, logits, streams = ready
    model = make(cfg, w, dtype)
    model.configure_cache(2, 160)
    model.record_stream(True)
    got = model.step_rows([model.add_seq()], [toks], range(len(toks)))
    stream = torch.from_numpy(model.layer_stream()).double()
    assert stream.shape == streams.shape
    for run in range(len(streams)):
        err = (stream[run] - streams[run]).pow(2).mean().sqrt() / streams[run].pow(2).mean().sqrt()
        assert err.item() <= TOL[dtype], f"{name}: layer run {run}"
    check(got, logits, dtype, name)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 5], [16, 1, 17], [64, 15, 2, 33]])
def test_portions_and_single_tokens(ready, dtype, sizes):
    """The same sequence cut in different ways: portions down to two tokens and token by token (which replays captured
    steps from the third one on)."""
    name, cfg, w, toks, logits, _ = ready
    model = make(cfg, w, dtype)
    model.configure_cache(1, 160)
    seq, at, i, rows = model.add_seq(), 0, 0, []
    while at < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - at)
        rows.append(model.step_rows([seq], [toks[at:at + n]], range(n)))
        at, i = at + n, i + 1
    check(np.concatenate(rows), logits, dtype, f"{name} in portions of {sizes}")


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_mixed_batches_with_reused_pages_and_slots(ready, dtype):
    """Unequal requests join, pause, decode beside others' portions and leave; the pool is smaller than their sum, so pages
    and state slots of finished requests serve later ones."""
    name, cfg, w, toks, _, _ = ready
    model = make(cfg, w, dtype)
    lens = [90, 33, 47, 64, 18, 75, 2]
    seqs = [cases.tokens(cfg, n, seed=10 + i) for i, n in enumerate(lens)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    model.configure_cache(3, 96, 208)
    total_pages = model.free_pages
    rng = np.random.default_rng(5)
    waiting, live, got = list(range(len(seqs))), {}, {i: [] for i in range(len(seqs))}
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-lens[i] // 16) for i in [*live, waiting[0]]) <= total_pages:
            live[waiting.pop(0)] = [model.add_seq(), 0]
        batch = [i for i in live if rng.random() < 0.8] or [next(iter(live))]
        counts = {i: min(int(rng.choice([1, 1, 1, 2, 3, 16, 40])), lens[i] - live[i][1]) for i in batch}
        feed = [seqs[i][live[i][1]:live[i][1] + counts[i]] for i in batch]
        out = model.step_rows([live[i][0] for i in batch], feed, range(sum(map(len, feed))))
        at = 0
        for i in batch:
            got[i].append(out[at:at + counts[i]])
            at += counts[i]
            live[i][1] += counts[i]
            if live[i][1] == lens[i]:
                model.free_seq(live.pop(i)[0])
    assert model.free_pages == total_pages
    for i in range(len(seqs)):
        check(np.concatenate(got[i]), want[i], dtype, f"{name}, request {i}")


def test_logits_at_chosen_rows_only(ready):
    name, cfg, w, toks, logits, _ = ready
    model = make(cfg, w, "f32")
    model.configure_cache(2, 160)
    a, b = model.add_seq(), model.add_seq()
    assert model.step_rows([a, b], [toks[:20], toks[:7]], []).shape == (0, cfg["vocab"])
    got = model.step_rows([b, a], [toks[7:30], toks[20:22]], [24, 0, 5])
    check(got, logits[[21, 7, 12]], "f32", name)
    with pytest.raises(llaisys.LlaisysError):
        model.step_rows([a], [toks[22:24]], [2])
    with pytest.raises(llaisys.LlaisysError):
        model.step_rows([a], [[cfg["vocab"]]], [0])


def test_long_decoding(cuda_device):
    """Several windows' worth of decoded tokens, far past where the first keys left every window, on a device-resident loop
    and step by step: the same greedy tokens, and the logits still agree with the oracle at the end."""
    cfg, w = cases.case("mixed", seed=3)
    model = make(cfg, w, "f32")
    model.configure_cache(2, 400)
    prompt = cases.tokens(cfg, 5, seed=2)
    seq = model.add_seq()
    first = model.step([seq], [prompt])
    loop = model.decode_loop([seq], first, 300)[:, 0].tolist()
    history = prompt + first + loop[:-1]
    other = model.add_seq()
    assert model.step([other], [prompt]) == first
    tok, steps = first[0], []
    for _ in range(300):
        tok = model.step([other], [[tok]])[0]
        steps.append(tok)
    assert steps == loop
    check(model.last_logits(1), oracle.forward(cfg, w, history)[0][-1:], "f32")


def test_greedy_generation_and_engine(cuda_device):
    """generate() and the batching engine (unequal prompts, late arrivals, chunked prompts, fewer slots than requests) give
    the oracle's greedy tokens; a shared beginning is recomputed, never taken from another request's pages."""
    cfg, w = cases.case("mixed", seed=4)
    model = make(cfg, w, "f32")
    lens, max_new = [5, 40, 1, 64, 33], [12, 6, 9, 5, 8]
    prompts = [cases.tokens(cfg, n, seed=20 + i) for i, n in enumerate(lens)]
    prompts[4] = prompts[3][:33]
    want, margins = zip(*[oracle.greedy(cfg, w, p, n) for p, n in zip(prompts, max_new)])
    assert min(map(min, margins)) > 1e-4  # no near-ties, so the tokens are determined
    model.configure_cache(1, 128)
    for p, n, t in zip(prompts, max_new, want):
        assert model.generate(p, max_new_tokens=n)[len(p):] == t
    model.configure_cache(2, 96)
    engine = llaisys.Engine(model, max_batch=2, max_tokens_per_step=24, prefill_chunk=10)
    got = engine.run([(0, prompts[0], max_new[0]), (0, prompts[1], max_new[1]), (1, prompts[2], max_new[2]),
                      (4, prompts[3], max_new[3]), (6, prompts[4], max_new[4])])
    for i, t in enumerate(want):
        assert got[i] == t, f"request {i}"
    assert engine.counters["prompt_tokens_from_cache"] == 0
    engine.close()
    seq, covered = model.add_seq_with_prefix(prompts[3])
    assert covered == 0
    model.free_seq(seq)
    sampled = model.generate(prompts[1], max_new_tokens=8, top_k=5, temperature=0.9, seed=1)
    assert len(sampled) == len(prompts[1]) + 8 and sampled == model.generate(prompts[1], max_new_tokens=8, top_k=5,
                                                                             temperature=0.9, seed=1)


def test_loading_errors(cuda_device):
    cfg, w = cases.case("mixed")
    short = {k: v for k, v in w.items() if k != "l1.mix.left.k"}
    with pytest.raises(ValueError, match="l1.mix.left.k"):
        make(cfg, short, "f32")
    bad = dict(w, head=w["head"][:-1])
    with pytest.raises(ValueError, match="head"):
        make(cfg, bad, "f32")
    with pytest.raises(RuntimeError):
        Doderax(config=cfg, state_dict=w, device=llaisys.DeviceType.CPU)
    wrong = cases.case("mixed")[0]
    wrong["layers"][1]["mixer"]["left"]["kv_heads"] = 3  # does not divide the query heads
    with pytest.raises((RuntimeError, ValueError)):
        make(wrong, w, "f32")


def test_trace_replay(ready, tmp_path):
    """The replay class on a live model: what it returns are the oracle's logits at the wanted places."""
    from llaisys_b200.trace import TraceRunner

    name, cfg, w, toks, logits, _ = ready
    runner = TraceRunner(make(cfg, w, "f32"), 192)
    a = runner.step([{"id": "a", "tokens": toks[:50], "want": [0, 49]}])
    check(a, logits[[0, 49]], "f32", name)
    b = runner.step([{"id": "a", "tokens": toks[50:51], "want": [0]}, {"id": "b", "tokens": toks[:70], "want": [69]}], ["a"])
    check(b, logits[[50, 69]], "f32", name)
    c = runner.step([{"id": "a", "tokens": toks[:100], "want": [99]}, {"id": "b", "tokens": toks[70:72], "want": [0, 1]}], ["a", "b"])
    check(c, logits[[99, 70, 71]], "f32", name)


@pytest.mark.parametrize("cut", [None, 6, 7])
def test_the_previous_token_counts(cuda_device, cut):
    """The embedding of a token depends on the one before it, also when that came in an earlier step: with everything else
    silenced, logits are those of token and pair rows alone."""
    cfg, w = cases.case("mixed")
    for name in w:
        if name.endswith((".o", "mlp.down", ".out")):
            w[name] = np.zeros_like(w[name])
    toks = cases.tokens(cfg, 12, seed=7)
    toks[6] = toks[2]  # the same token behind another one
    model = make(cfg, w, "f32")
    model.configure_cache(2, 64)
    seq = model.add_seq()
    parts = [toks] if cut is None else [toks[:cut], [toks[cut]], toks[cut + 1:]]
    got = np.concatenate([model.step_rows([seq], [p], range(len(p))) for p in parts])
    x = oracle.to_f64(w["embed"])[toks] + oracle.to_f64(w["bigram"])[oracle.pair_rows(toks, cfg["embedding"]["bigram"])]
    want = cfg["logit_scale"] * (oracle.rms(x, cfg["norm"]["eps"]) * (1 + oracle.to_f64(w["final.norm"]))) @ oracle.to_f64(w["head"]).T
    check(got, want, "f32")
    assert row_errors(got[6:7], want[2:3]).item() > 0.1


def test_decoding_past_the_windows_on_the_fast_kernels(cuda_device):
    """bfloat16, head size 128: hundreds of tokens decoded in a batch of unequal sequences, so that pages between the kept tokens
    and the windows drop out one by one."""
    cfg, w = cases.case("head_dim_128", seed=2)
    model = make(cfg, w, "bf16")
    model.configure_cache(3, 320)
    seqs = [cases.tokens(cfg, n, seed=30 + n) for n in (300, 180, 75)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    ids, at = [model.add_seq() for _ in seqs], [20, 3, 64]
    model.step(ids, [s[:n] for s, n in zip(seqs, at)])
    got = [[] for _ in seqs]
    while any(a < len(s) for a, s in zip(at, seqs)):
        live = [i for i in range(3) if at[i] < len(seqs[i])]
        rows = model.step_rows([ids[i] for i in live], [[seqs[i][at[i]]] for i in live], range(len(live)))
        for r, i in enumerate(live):
            got[i].append(rows[r])
            at[i] += 1
    for i, start in enumerate([20, 3, 64]):
        check(np.stack(got[i]), want[i][start:], "bf16", f"sequence {i}")
