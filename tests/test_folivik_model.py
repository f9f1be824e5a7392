"""Folivik on the device against its float64 oracle: whole prompts, single tokens, portions, batches, reused pages and slots,
greedy generation through the public entry points. float32 models are compared tightly (they compute everything in true 32
bits), bfloat16 models within what bfloat16 rounding of weights-times-activations leaves."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from llaisys_b200.models import Folivik
from oracle import folivik as oracle
from tests import folivik_cases as cases

pytestmark = pytest.mark.gpu
DT = {"f32": llaisys.DataType.F32, "f16": llaisys.DataType.F16, "bf16": llaisys.DataType.BF16}
# relative rms error of a row of logits (mean taken off): float32 rounding; bfloat16 rounding through a few layers
TOL = {"f32": 2e-5, "f16": 0.01, "bf16": 0.06}


def make(cfg, w, dtype):
    return Folivik(config=cfg, state_dict=w, dtype=DT[dtype])


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
    """Hundreds of decoded tokens on a device-resident loop and step by step: the same greedy tokens, and the logits still agree with
    the oracle at the end."""
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


def test_pages_of_a_shared_beginning_are_reused_without_recurrent_layers(cuda_device):
    """A model whose layers are all attention finds a published prefix; logits behind it are those of the whole sequence."""
    cfg, w = cases.case("attention_only", seed=0)
    model = make(cfg, w, "f32")
    model.configure_cache(3, 96)
    toks = cases.tokens(cfg, 60, seed=4)
    a = model.add_seq()
    model.step_rows([a], [toks[:50]], [])
    b, covered = model.add_seq_with_prefix(toks)
    assert covered == 48
    check(model.step_rows([b], [toks[covered:]], range(60 - covered)), oracle.forward(cfg, w, toks)[0][covered:], "f32")
    model.free_seq(a)
    check(model.step_rows([b], [[7]], [0]), oracle.forward(cfg, w, toks + [7])[0][-1:], "f32")


def test_loading_errors(cuda_device):
    cfg, w = cases.case("mixed")
    short = {k: v for k, v in w.items() if k != "l1.mlp.e3.up"}
    with pytest.raises(ValueError, match="l1.mlp.e3.up"):
        make(cfg, short, "f32")
    bad = dict(w, head=w["head"][:-1])
    with pytest.raises(ValueError, match="head"):
        make(cfg, bad, "f32")
    with pytest.raises(RuntimeError):
        Folivik(config=cfg, state_dict=w, device=llaisys.DeviceType.CPU)
    wrong = cases.case("mixed")[0]
    wrong["layers"][2]["mixer"]["kv_heads"] = 4  # does not divide the query heads
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


def test_positions_and_latents_far_away(cuda_device):
    """Thousands of tokens of context in front of the queries, in a prompt and decoded: turned parts at far positions, pages of
    latents far back, a window that has passed most of them."""
    cfg, w = cases.case("attention_only", seed=0)
    toks = cases.tokens(cfg, 1500, seed=8)
    model = make(cfg, w, "f32")
    model.configure_cache(1, 1520)
    seq = model.add_seq()
    model.step_rows([seq], [toks[:900]], [])
    got = [model.step_rows([seq], [toks[900:1490]], [0, 100, 589])] + [model.step_rows([seq], [[t]], [0]) for t in toks[1490:]]
    want = oracle.forward(cfg, w, toks)[0][[900, 1000, 1489, *range(1490, 1500)]]
    check(np.concatenate(got), want, "f32")
    model = make(cfg, w, "bf16")
    model.configure_cache(1, 1520)
    seq = model.add_seq()
    got = [model.step_rows([seq], [toks[:1490]], [900, 1000, 1489])] + [model.step_rows([seq], [[t]], [0]) for t in toks[1490:]]
    check(np.concatenate(got), want, "bf16")


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_a_far_token_decides(cuda_device, dtype):
    """The first token, hundreds of tokens back, is what every later query's latent attention reads: the logits follow the oracle,
    and change when that token changes."""
    cfg, w = cases.case("attention_only", seed=0)
    w = {n: v.copy() for n, v in w.items()}
    # token 3 has a direction of its own in the stream; the latent's first channel reads it, and so does every head's key
    e = oracle.to_f64(w["embed"]).numpy()
    e[:, 8] = 0.0
    e[3], e[4] = 0.0, 0.0
    e[3, 3 % cases.CLASSES] = e[4, 4 % cases.CLASSES] = 0.8 * cfg["width"] ** 0.5
    e[3, 8] = e[4, 9] = 12.0
    w["embed"] = cases.bf16_words(e.astype(np.float32))
    dkv = oracle.to_f64(w["l0.mix.dkv"]).numpy() * 0.3
    dkv[0] = 0.0
    dkv[0, 8] = 6.0
    w["l0.mix.dkv"] = cases.bf16_words(dkv.astype(np.float32))
    uk = oracle.to_f64(w["l0.mix.uk"]).numpy()
    uk[:, 0] = 2.0
    w["l0.mix.uk"] = cases.bf16_words(uk.astype(np.float32))
    toks = [3] + [t % 50 + 5 for t in cases.tokens(cfg, 420, seed=9)]
    logits, _ = oracle.forward(cfg, w, toks)
    other, _ = oracle.forward(cfg, w, [4] + toks[1:])
    assert row_errors(other[-1:], logits[-1:]).item() > 2 * TOL["bf16"]
    model = make(cfg, w, dtype)
    model.configure_cache(2, 448)
    a = model.add_seq()
    got = [model.step_rows([a], [toks[:300]], range(300))] + [model.step_rows([a], [[t]], [0]) for t in toks[300:]]
    check(np.concatenate(got), logits, dtype)


def test_a_batch_of_unequal_sequences_decodes(cuda_device):
    """bfloat16, head size 128: tokens decoded in a batch of unequal sequences, some leaving early."""
    cfg, w = cases.case("head_dim_128", seed=1)
    model = make(cfg, w, "bf16")
    model.configure_cache(3, 224)
    seqs = [cases.tokens(cfg, n, seed=30 + n) for n in (200, 150, 75)]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    ids, at = [model.add_seq() for _ in seqs], [120, 3, 64]
    model.step(ids, [s[:n] for s, n in zip(seqs, at)])
    got = [[] for _ in seqs]
    while any(a < len(s) for a, s in zip(at, seqs)):
        live = [i for i in range(3) if at[i] < len(seqs[i])]
        rows = model.step_rows([ids[i] for i in live], [[seqs[i][at[i]]] for i in live], range(len(live)))
        for r, i in enumerate(live):
            got[i].append(rows[r])
            at[i] += 1
    for i, start in enumerate([120, 3, 64]):
        check(np.stack(got[i]), want[i][start:], "bf16", f"sequence {i}")


def test_long_prompts_beside_single_tokens(cuda_device):
    """bfloat16, sizes of the fast kernels: a long portion, a short one and decoded tokens in one step, from contexts of every kind."""
    cfg, w = cases.case("head_dim_128", seed=1)
    model = make(cfg, w, "bf16")
    model.configure_cache(4, 640)
    lens = [600, 330, 140, 259]
    seqs = [cases.tokens(cfg, n, seed=50 + n) for n in lens]
    want = [oracle.forward(cfg, w, s)[0] for s in seqs]
    ids, at = [model.add_seq() for _ in seqs], [0] * 4
    plan = [[257, 1, 130, 0], [1, 300, 1, 3], [300, 1, 2, 255], [42, 28, 7, 1]]
    for counts in plan:
        who = [i for i in range(4) if counts[i]]
        rows = model.step_rows([ids[i] for i in who], [seqs[i][at[i]:at[i] + counts[i]] for i in who], range(sum(counts)))
        offset = 0
        for i in who:
            check(rows[offset:offset + counts[i]], want[i][at[i]:at[i] + counts[i]], "bf16", f"sequence {i} at {at[i]}")
            offset += counts[i]
            at[i] += counts[i]
    assert at == lens
