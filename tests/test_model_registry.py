"""Host side of the model package: the class a config selects, configurations and their weights, the safetensors reader, the
trace protocol and the command line. No GPU."""
import io
import json
import struct
import sys

import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from llaisys_b200 import trace
from llaisys_b200.models import Doderax, Folivik, Lilovik, Qwen2, Vozozen, load_model, model_class
from llaisys_b200.models import doderax as dx
from llaisys_b200.models import folivik as fk
from llaisys_b200.models import lilovik as lk
from llaisys_b200.models import vozozen as vz
from llaisys_b200.models.weights import SafetensorsFile, checkpoint_files
from oracle import doderax as doderax_oracle
from oracle import folivik as folivik_oracle
from oracle import lilovik as lilovik_oracle
from oracle import vozozen as oracle
from tests import doderax_cases, folivik_cases, lilovik_cases
from tests import vozozen_cases as cases


def write_safetensors(path, tensors):
    header, blob = {"__metadata__": {"format": "pt"}}, b""
    for name, a in tensors.items():
        kind = {np.dtype(np.uint16): "BF16", np.dtype(np.float32): "F32", np.dtype(np.int32): "I32"}[a.dtype]
        header[name] = {"dtype": kind, "shape": list(a.shape), "data_offsets": [len(blob), len(blob) + a.nbytes]}
        blob += a.tobytes()
    text = json.dumps(header).encode()
    path.write_bytes(struct.pack("<Q", len(text)) + text + blob)


def test_class_by_config():
    assert model_class({"architecture": "Vozozen"}) is Vozozen
    assert model_class({"architecture": "Doderax"}) is Doderax
    assert model_class({"architecture": "Lilovik"}) is Lilovik
    assert model_class({"architecture": "Folivik"}) is Folivik
    assert model_class({"architectures": ["Qwen2ForCausalLM"], "model_type": "qwen2"}) is Qwen2
    assert model_class({"model_type": "qwen2"}) is Qwen2
    with pytest.raises(ValueError, match="Mamba"):
        model_class({"architecture": "Mamba"})


def test_qwen2_checkpoint_through_the_registry(tmp_path):
    """A directory with config.json and safetensors becomes a running model (CPU) without naming its class."""
    import safetensors.torch
    from tests.test_qwen2_model import hf_greedy, hf_model

    cfg, hf = hf_model(seed=5)
    (tmp_path / "config.json").write_text(json.dumps({**cfg, "model_type": "qwen2", "dtype": "float32"}))
    state = {k: v.contiguous().clone() for k, v in hf.state_dict().items()}
    safetensors.torch.save_file(state, str(tmp_path / "model.safetensors"))
    model = load_model(tmp_path, llaisys.DeviceType.CPU)
    assert isinstance(model, Qwen2)
    assert model.generate([3, 1, 4], max_new_tokens=5) == hf_greedy(hf, [3, 1, 4], 5)
    # logits at chosen rows, and a pool smaller than slots x length, on the shared step
    model.configure_cache(2, 64, 64)
    assert model.free_pages == 4
    toks = list(range(20))
    got = model.step_rows([model.add_seq()], [toks], [4, 19])
    with torch.no_grad():
        want = hf(torch.tensor([toks])).logits[0, [4, 19]].float().numpy()
    assert np.abs(got - want).max() < 2e-4


def test_safetensors_reader(tmp_path):
    a = np.arange(6, dtype=np.float32).reshape(2, 3)
    b = cases.bf16_words(np.array([1.0, -2.5, 3.14159], dtype=np.float32))
    c = np.array([7, 8], dtype=np.int32)
    write_safetensors(tmp_path / "x.safetensors", {"a": a, "b": b, "c": c})
    f = SafetensorsFile(tmp_path / "x.safetensors")
    assert f.names() == ["a", "b", "c"] and f.shape("a") == (2, 3) and f.dtype("b") == "BF16"
    assert np.array_equal(f.array("a"), a) and np.array_equal(f.array("b"), b) and np.array_equal(f.array("c"), c)
    assert oracle.to_f64(f.array("b"))[1] == -2.5
    (tmp_path / "short.safetensors").write_bytes(b"abc")
    with pytest.raises(ValueError):
        SafetensorsFile(tmp_path / "short.safetensors")
    with pytest.raises(FileNotFoundError):
        list(checkpoint_files(tmp_path / "nowhere"))


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_configuration_reaches_the_library(name):
    cfg, ranks = cases.CASES[name]
    meta = vz.build_meta(cfg, ranks, llaisys.DataType.BF16)
    assert meta.nlayer == len(cfg["layers"]) and meta.width == cfg["width"] and meta.voc == cfg["vocab"]
    for i, entry in enumerate(cfg["layers"]):
        got, left, right = meta.layers[i], entry["mixer"]["left"], entry["mixer"]["right"]
        assert (got.left.heads, got.left.kv_heads, got.left.dim, got.left.vdim, got.left.window) == (
            left["heads"], left["kv_heads"], left["dim"], left["vdim"], left["mask"]["size"])
        assert (got.right.heads, got.right.dim, got.right.vdim, got.right.rank) == (
            right["heads"], right["dim"], right["vdim"], ranks[i])
        assert got.right.tau == pytest.approx(right["tau"]) and got.left.scale == pytest.approx(left["scale"])
        assert got.left_scale == pytest.approx(entry["mixer"]["left_scale"])
        assert got.right_scale == pytest.approx(entry["mixer"]["right_scale"])
        assert got.ff == (entry["mlp"]["ff"] if entry["mlp"] else 0)
    assert meta.logit_softcap == pytest.approx(cfg["logit_softcap"]) and meta.eps == pytest.approx(cfg["norm"]["eps"])
    assert meta.embed_scale == pytest.approx(cfg["embedding"]["scale"])
    loop = cfg["loop"]
    assert (meta.loop_start, meta.loop_stop, meta.loop_times) == ((loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0))


def test_unknown_parts_of_a_configuration_are_refused():
    cfg, ranks = cases.case("looped")[0], cases.CASES["looped"][1]
    cfg["layers"][0]["type"] = "serial"
    with pytest.raises(ValueError, match="serial"):
        vz.build_meta(cfg, ranks, llaisys.DataType.BF16)
    cfg = cases.case("looped")[0]
    cfg["layers"][0]["mlp"]["kind"] = "experts"
    with pytest.raises(ValueError, match="experts"):
        vz.build_meta(cfg, ranks, llaisys.DataType.BF16)


@pytest.mark.parametrize("name", sorted(doderax_cases.CASES))
def test_doderax_configuration_reaches_the_library(name):
    cfg, ranks = doderax_cases.CASES[name]
    shapes = dx.weight_shapes(cfg, ranks)
    assert dx.low_ranks(cfg, shapes) == ranks
    meta = dx.build_meta(cfg, ranks, llaisys.DataType.BF16)
    pairs = cfg["embedding"]["bigram"]
    assert (meta.nlayer, meta.width, meta.voc) == (len(cfg["layers"]), cfg["width"], cfg["vocab"])
    assert (meta.pair_buckets, meta.pair_mul_prev, meta.pair_mul_cur) == (pairs["buckets"], pairs["mul_prev"], pairs["mul_cur"])
    assert meta.eps == pytest.approx(cfg["norm"]["eps"]) and meta.logit_scale == pytest.approx(cfg["logit_scale"])
    for i, entry in enumerate(cfg["layers"]):
        got, mixer = meta.layers[i], entry["mixer"]
        assert got.ff == (entry["mlp"]["ff"] if entry["mlp"] else 0) and bool(got.parallel) == (entry["type"] == "parallel")
        delta = mixer["right"] if got.parallel else mixer
        assert (got.delta.heads, got.delta.kv_heads, got.delta.dim, got.delta.vdim, got.delta.taps, got.delta.decay_rank,
                got.delta.gate_rank) == (*(delta[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")), *ranks[i])
        if got.parallel:
            a, left = got.attn, mixer["left"]
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.rot_dims) == (
                left["heads"], left["kv_heads"], left["dim"], left["vdim"], left["mask"]["size"], left["mask"]["keep_first"],
                left["rot"]["dims"])
            assert a.rot_base == left["rot"]["base"] and a.scale == pytest.approx(left["scale"])


def test_unknown_parts_of_a_doderax_configuration_are_refused():
    cfg, _ = doderax_cases.case("mixed")
    ranks = doderax_cases.CASES["mixed"][1]
    cfg["layers"][0]["type"] = "serial"
    with pytest.raises(ValueError, match="serial"):
        dx.build_meta(cfg, ranks, llaisys.DataType.BF16)
    cfg, w = doderax_cases.case("mixed")
    cfg["layers"][1]["mlp"]["kind"] = "experts"
    with pytest.raises(ValueError, match="experts"):
        dx.build_meta(cfg, ranks, llaisys.DataType.BF16)
    cfg, w = doderax_cases.case("mixed")
    with pytest.raises(ValueError, match="l0.mix.a1"):
        Doderax(config=cfg, state_dict={k: v for k, v in w.items() if k != "l0.mix.a1"}, device=llaisys.DeviceType.CPU)
    with pytest.raises(RuntimeError, match="NVIDIA"):
        Doderax(config=cfg, state_dict=w, device=llaisys.DeviceType.CPU)


def test_doderax_oracle_mechanisms_agree_with_closed_forms():
    torch.manual_seed(1)
    T, H, d, dv = 10, 2, 6, 5
    q, k, v = torch.randn(T, H, d).double(), torch.nn.functional.normalize(torch.randn(T, H, d).double(), dim=-1), torch.randn(T, H, dv).double()
    none, one = torch.zeros(T, H, d).double(), torch.ones(T, H).double()
    # orthogonal keys: nothing to correct, plain sums of outer products
    basis = torch.eye(d).double()[[0, 1, 2, 3, 4, 5]].unsqueeze(1).expand(d, H, d)
    _, S = doderax_oracle.delta_rule(q[:d], basis, v[:d], none[:d], one[:d])
    assert torch.allclose(S, v[:d].transpose(0, 1))
    # full write strength: the newest key reads its own value back, with any decay
    log = doderax_oracle.decay_log(torch.tensor(0.3).double(), torch.randn(T, H, d).double())
    y, S = doderax_oracle.delta_rule(k, k, v, log, one)
    assert torch.allclose(y, v) and (log < 0).all()
    # no write strength: the state only decays
    _, S1 = doderax_oracle.delta_rule(q, k, v, log, 0 * one, state=S)
    assert torch.allclose(S1, S * torch.exp(log.sum(0)).unsqueeze(2))
    assert torch.allclose(doderax_oracle.decay_log(torch.zeros(1).double(), torch.zeros(1).double()), -torch.tensor([2.0]).double().log())
    # rotation: lengths stay, equal distances give equal products, position 0 and the unrotated dims pass
    x = torch.randn(1, 1, 8).double().expand(9, 1, 8)
    r = doderax_oracle.rotate(x, 6, 50.0)
    assert torch.allclose(r.norm(dim=-1), x.norm(dim=-1)) and torch.allclose(r[0], x[0]) and torch.equal(r[..., 6:], x[..., 6:])
    dots = torch.einsum("ihd,jhd->ij", r, r)
    assert torch.allclose(dots[2, 0], dots[8, 6])
    # a window that covers everything, and one of a single token beside kept ones
    args = q, k, v
    full = doderax_oracle.sink_attention(*args, 0.7, T, 0)
    assert torch.allclose(full, doderax_oracle.sink_attention(*args, 0.7, 1, T)) and torch.allclose(full, oracle.window_attention(*args, 0.7, T))
    assert torch.allclose(doderax_oracle.sink_attention(*args, 0.7, 1, 0), v)
    w = torch.zeros(3, 4).double()
    w[:, -1] = 1.0
    y = torch.randn(7, 3).double()
    assert torch.allclose(doderax_oracle.short_conv(y, w), oracle.silu(y))
    assert doderax_oracle.pair_rows([3, 4, 3], {"buckets": 10, "mul_prev": 2, "mul_cur": 5}) == [10, 6, 3]
    assert torch.allclose(doderax_oracle.gelu(y), torch.nn.functional.gelu(y, approximate="tanh"))


@pytest.mark.parametrize("name", sorted(lilovik_cases.CASES))
def test_lilovik_configuration_reaches_the_library(name):
    cfg, w = lilovik_cases.case(name)
    assert set(w) == set(lk.weight_shapes(cfg)) and all(w[n].shape == s for n, s in lk.weight_shapes(cfg).items())
    meta = lk.build_meta(cfg, llaisys.DataType.F32)
    assert (meta.nlayer, meta.width, meta.voc, meta.end_token) == (len(cfg["layers"]), cfg["width"], cfg["vocab"], -1)
    assert meta.eps == pytest.approx(cfg["norm"]["eps"]) and meta.logit_scale == pytest.approx(cfg["logit_scale"])
    for i, entry in enumerate(cfg["layers"]):
        got, m = meta.layers[i], entry["mixer"]
        assert got.ff == (entry["mlp"]["ff"] if entry["mlp"] else 0) and got.recurrent == (entry["type"] == "mingru")
        if got.recurrent:
            assert got.gru_width == m["width"]
            continue
        temp = m.get("q_temp")
        assert (got.attn.heads, got.attn.kv_heads, got.attn.dim, got.attn.vdim) == (m["heads"], m["kv_heads"], m["dim"], m["vdim"])
        assert got.attn.scale == pytest.approx(m["scale"]) and got.attn.softcap == pytest.approx(m.get("softcap", 0.0))
        assert got.attn.temp_coef == pytest.approx(temp["coef"] if temp else 0.0)
        assert temp is None or got.attn.temp_every == temp["every"]


def test_unknown_parts_of_a_lilovik_configuration_are_refused():
    cfg, w = lilovik_cases.case("mixed")
    cfg["layers"][0]["type"] = "serial"
    with pytest.raises(ValueError, match="serial"):
        lk.build_meta(cfg, llaisys.DataType.BF16)
    cfg, w = lilovik_cases.case("mixed")
    cfg["layers"][1]["mlp"]["kind"] = "experts"
    with pytest.raises(ValueError, match="experts"):
        lk.build_meta(cfg, llaisys.DataType.BF16)
    with pytest.raises(RuntimeError, match="NVIDIA"):
        Lilovik(config=lilovik_cases.case("mixed")[0], state_dict=w, device=llaisys.DeviceType.CPU)


def test_lilovik_oracle_mechanisms_agree_with_closed_forms():
    torch.manual_seed(2)
    T, H, G, d, dv = 9, 4, 2, 6, 5
    q, k, v = torch.randn(T, H, d).double(), torch.randn(T, G, d).double(), torch.randn(T, G, dv).double()
    none, eye = torch.zeros(H).double(), torch.eye(H).double()
    # slopes halve from head to head at eight heads; a query far behind its keys sees sigmoid(score - slope distance + bias)
    assert torch.allclose(lilovik_oracle.slopes(8), 0.5 ** torch.arange(1, 9).double())
    a = lilovik_oracle.gates(q, k, 0.3, None, none + 0.7)
    assert torch.allclose(a[1, 5, 2], torch.sigmoid(0.3 * (q[5, 1] @ k[2, 0]) - 3 * 2.0 ** -4 + 0.7))
    assert (torch.triu(a, 1) == 0).all() and torch.allclose(a[:, 4:6, :], lilovik_oracle.gates(q[4:6], k, 0.3, None, none + 0.7, first=4))
    # a wide cap is none, and nothing passes a cap
    assert torch.allclose(lilovik_oracle.gates(q, k, 0.3, 1e6, none), lilovik_oracle.gates(q, k, 0.3, None, none), atol=1e-9)
    assert lilovik_oracle.gates(q, k, 50.0, 2.0, none)[:, range(T), range(T)].max() <= torch.sigmoid(torch.tensor(2.0).double())
    # mixing with the identity changes nothing, with a permutation it moves heads; unweighted values add up
    assert torch.allclose(lilovik_oracle.mix_heads(a, eye), a) and torch.allclose(lilovik_oracle.mix_heads(a, eye[[2, 0, 1, 3]]), a[[2, 0, 1, 3]])
    ones = torch.tril(torch.ones(H, T, T)).double()
    assert torch.allclose(lilovik_oracle.weigh_values(ones, v), v.cumsum(0).repeat_interleave(H // G, 1))
    # the query factor steps where position + 1 reaches a multiple
    f = lilovik_oracle.query_factors([0, 6, 7, 14, 15], {"coef": 0.5, "every": 8})
    assert torch.allclose(f, 1 + 0.5 * torch.tensor([1.0, 1.0, 2.0, 2.0, 3.0]).double().log()) and (lilovik_oracle.query_factors([3], None) == 1).all()
    # position 0 is (0, 1, 0, 1, ..); the pair's distance to another position depends on the difference only
    p = lilovik_oracle.position_vectors([0, 3, 7, 10], 8)
    assert torch.equal(p[0], torch.tensor([0.0, 1.0] * 4).double()) and torch.allclose(p[0] @ p[1], p[2] @ p[3])
    # a closed gate keeps the state, an open one takes the candidate, which is continuous at zero
    z, u, o = (torch.randn(T, 3).double() for _ in range(3))
    start = torch.randn(3).double()
    y, S = lilovik_oracle.min_gru(z * 0 - 1e3, u, o, start)
    assert torch.allclose(S, start) and torch.allclose(y, start * lilovik_oracle.silu(o))
    _, S = lilovik_oracle.min_gru(z * 0 + 1e3, u.abs(), o, start)
    assert torch.allclose(S, u[-1].abs() + 0.5)
    _, S = lilovik_oracle.min_gru(z * 0 + 1e3, torch.tensor([[0.0, -1e-9, -50.0]]).double().expand(T, 3), o, start)
    assert torch.allclose(S, torch.tensor([0.5, 0.5, 0.0]).double())


@pytest.mark.parametrize("name", sorted(folivik_cases.CASES))
def test_folivik_configuration_becomes_the_c_description(name):
    cfg = folivik_cases.CASES[name]
    meta = fk.build_meta(cfg, llaisys.DataType.BF16, 77)
    assert (meta.nlayer, meta.width, meta.voc, meta.maxseq, meta.end_token) == (len(cfg["layers"]), cfg["width"], cfg["vocab"], 77, -1)
    assert meta.eps == pytest.approx(cfg["norm"]["eps"])
    for got, entry in zip(meta._layers, cfg["layers"]):
        m, mlp = entry["mixer"], entry["mlp"]
        part = {"latent_attention": got.latent, "attention": got.attn, "mamba2": got.ssm}[entry["type"]]
        assert got.mixer == fk.LAYER_TYPES.index(entry["type"]) and part.heads == m["heads"] and part.vdim == m["vdim"]
        if entry["type"] == "latent_attention":
            assert (part.dim, part.rot_dim, part.q_rank, part.kv_rank) == (m["dim"], m["rot_dim"], m["q_rank"], m["kv_rank"])
            assert part.rot_base == m["rot"]["base"] and part.scale == pytest.approx(m["scale"])
        elif entry["type"] == "attention":
            assert (part.kv_heads, part.dim, part.window) == (m["kv_heads"], m["dim"], m["mask"]["size"])
        else:
            assert (part.groups, part.state, part.taps, part.norm_groups) == (m["groups"], m["state"], m["conv"], m["norm_groups"])
        if mlp is None:
            assert got.mlp.top == 0
            continue
        r, groups = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
        assert (got.mlp.experts, got.mlp.identity, got.mlp.top) == (r["experts"], r["identity"], r["top"])
        assert (got.mlp.groups, got.mlp.keep, got.mlp.ff) == (groups["count"], groups["keep"], mlp["expert"]["ff"])
        assert got.mlp.shared_ff == (mlp["shared"]["ff"] if mlp.get("shared") else 0) and got.mlp.scale == pytest.approx(r["scale"])
    shapes = fk.weight_shapes(cfg)
    assert shapes["l0.norm1"] == () and shapes["head"] == (cfg["vocab"], cfg["width"])


def test_unknown_parts_of_a_folivik_configuration_are_refused():
    def broken(change):
        cfg = folivik_cases.case("mixed")[0]
        change(cfg["layers"])
        return cfg

    for change, words in ((lambda l: l[0].update(type="serial"), "serial"), (lambda l: l[1]["mlp"].update(kind="dense"), "dense"),
                          (lambda l: l[1]["mixer"]["rot"].update(dims=8), "rotated part"),
                          (lambda l: l[0]["mlp"]["router"].update(groups={"count": 3, "keep": 1}), "do not fit"),
                          (lambda l: l[0]["mlp"]["router"].update(top=7), "do not fit"),
                          (lambda l: l[0]["mlp"]["router"].update(groups={"count": 4, "keep": 5}), "do not fit")):
        with pytest.raises(ValueError, match=words):
            fk.build_meta(broken(change), llaisys.DataType.BF16)
    cfg, w = folivik_cases.case("recurrence_only")
    with pytest.raises(RuntimeError, match="NVIDIA"):
        Folivik(config=cfg, state_dict=w, device=llaisys.DeviceType.CPU)


def test_folivik_oracle_mechanisms_agree_with_closed_forms():
    torch.manual_seed(3)
    o = folivik_oracle
    T, H, G, d, dv = 9, 4, 2, 6, 5
    q, k, v = torch.randn(T, H, d).double(), torch.randn(T, G, d).double(), torch.randn(T, G, dv).double()
    ones, none = torch.ones(H).double(), torch.zeros(H).double()
    full = o.softmax_attention(q, k, v, 0.3)
    # a window of one token returns its value; a wide one is none; a penalty of zero and a factor of one change nothing
    assert torch.allclose(o.softmax_attention(q, k, v, 0.3, window=1), v.repeat_interleave(2, 1))
    assert torch.allclose(o.softmax_attention(q, k, v, 0.3, window=T, temp=ones, bias=(none, ones)), full)
    assert torch.allclose(o.softmax_attention(q[4:], k, v, 0.3, first=4), full[4:])
    # with equal scores the penalty leaves weights (1 + b distance)^(-a)
    w = (1 + 0.5 * torch.arange(T - 1, -1, -1).double()) ** -2.0
    got = o.softmax_attention(q, k * 0, v, 0.3, bias=(2 * ones, 0.5 * ones))[-1, 0]
    assert torch.allclose(got, (w / w.sum()) @ v[:, 0])
    # a turn keeps lengths, depends on the difference of positions in products, and is none at position 0
    a, b = torch.randn(2, 1, 8).double()
    at = lambda x, p: o.turn_pairs(x, [p], 100.0)[0]  # noqa: E731
    assert torch.allclose(at(a, 0), a[0]) and torch.allclose(at(a, 5).norm(), a.norm())
    assert torch.allclose(at(a, 7) @ at(b, 3), at(a, 14) @ at(b, 10))
    # queries multiplied into the latents' space score like expanded keys
    c, z, uk, uv = torch.randn(T, 7).double(), torch.randn(T, 2).double(), torch.randn(H * d, 7).double(), torch.randn(H * dv, 7).double()
    kk, vv = o.latent_keys_values(c, z, uk, uv, H)
    qq = torch.randn(T, H, d + 2).double()
    wide = torch.cat([torch.einsum("thd,hdr->thr", qq[..., :d], uk.view(H, d, 7)), qq[..., d:]], dim=-1)
    rows = torch.cat([c, z], dim=1).unsqueeze(1)
    over = o.softmax_attention(wide, rows, c.unsqueeze(1), 0.4)
    assert torch.allclose(torch.einsum("thr,hvr->thv", over, uv.view(H, dv, 7)), o.softmax_attention(qq, kk, vv, 0.4))
    # a convolution whose only tap is the current token's; the inputs ahead of a portion stand in for its beginning
    x, taps, bias = torch.randn(T, 3).double(), torch.randn(3, 4).double(), torch.randn(3).double()
    last = torch.cat([torch.zeros(3, 3), torch.ones(3, 1)], dim=1).double()
    assert torch.allclose(o.convolve(x, last, bias), o.silu(x + bias))
    assert torch.allclose(o.convolve(x[5:], taps, bias, before=x[2:5]), o.convolve(x, taps, bias)[5:])
    # no decay sums everything written; total decay keeps the newest token alone; a state carries over
    xs, B, C, dt = torch.randn(T, 2, 4).double(), torch.randn(T, 1, 3).double(), torch.randn(T, 1, 3).double(), torch.rand(T, 2).double()
    D = torch.randn(2).double()
    _, S = o.state_space(xs, B, C, dt, torch.full((2,), -60.0).double(), D)
    assert torch.allclose(S, torch.einsum("th,tn,thp->hnp", dt, B[:, 0], xs))
    y, _ = o.state_space(xs, B, C, dt + 1, torch.full((2,), 8.0).double(), D)
    assert torch.allclose(y[-1], ((B[-1, 0] @ C[-1, 0]) * (dt[-1] + 1) + D).unsqueeze(1) * xs[-1])
    A = torch.randn(2).double()
    y, S = o.state_space(xs, B, C, dt, A, D)
    _, S5 = o.state_space(xs[:5], B[:5], C[:5], dt[:5], A, D)
    y2, S2 = o.state_space(xs[5:], B[5:], C[5:], dt[5:], A, D, S5)
    assert torch.allclose(y2, y[5:]) and torch.allclose(S2, S)
    # parts of a norm are normed on their own
    n = o.gated_parts_norm(torch.randn(2, 8).double() * torch.tensor([1.0] * 4 + [100.0] * 4).double(), torch.ones(2, 8).double(),
                           torch.ones(8).double(), 2, 0.0)
    assert torch.allclose(n.view(2, 2, 4).pow(2).mean(-1), torch.ones(2, 2).double())
    # routing: the correction moves the choice and not the weights; refused groups stay out however low the others are
    router = {"top": 2, "scale": 3.0, "groups": {"count": 2, "keep": 1}}
    logits = torch.tensor([3.0, 2.0, 1.0, 0.0]).double()
    chosen, weight = o.route(logits, torch.tensor([0.0, 0.0, -9.0, 1.0]).double(), router)
    assert sorted(chosen.tolist()) == [2, 3] and weight.sum() == pytest.approx(3.0)
    s = torch.softmax(logits, 0)
    assert float(weight[chosen.tolist().index(2)]) == pytest.approx(float(3 * s[2] / (s[2] + s[3])))


def test_no_host_stand_in():
    cfg, w = cases.case("looped")
    with pytest.raises(RuntimeError, match="NVIDIA"):
        Vozozen(config=cfg, state_dict=w, device=llaisys.DeviceType.CPU)
    with pytest.raises(ValueError, match="a1"):
        Vozozen(config=cfg, state_dict={k: v for k, v in w.items() if not k.endswith("a1")}, device=llaisys.DeviceType.CPU)


def test_oracle_mechanisms_agree_with_closed_forms():
    """The plain functions the device is compared with, on cases whose answers are known."""
    torch.manual_seed(0)
    q, k, v = (torch.randn(12, 2, 4, dtype=torch.float64) for _ in range(3))
    ones = torch.ones(12, 2, 4, dtype=torch.float64)
    out, S = oracle.gated_linear(q, k, v, ones)  # no decay: plain sums of outer products
    want = torch.stack([sum((q[t, 1] @ k[s, 1]) * v[s, 1] for s in range(t + 1)) for t in range(12)])
    assert torch.allclose(out[:, 1], want) and torch.allclose(S[0], torch.einsum("td,te->de", k[:, 0], v[:, 0]))
    assert torch.allclose(oracle.key_decay(torch.tensor([0.0]).double(), 1.0), torch.tensor([0.5]).double())
    assert torch.allclose(oracle.window_attention(q, k, v, 1.0, 1), v)  # each token sees itself only
    full = torch.nn.functional.scaled_dot_product_attention(*(x.transpose(0, 1) for x in (q, k, v)), is_causal=True, scale=0.7)
    assert torch.allclose(oracle.window_attention(q, k, v, 0.7, 12), full.transpose(0, 1))
    cfg = cases.CASES["looped"][0]
    assert oracle.run_order(cfg) == [(0, False), (1, True), (2, False), (1, True), (2, False)]


class FakeModel:
    """Stands in for a model: counts slots and 'logits' = (sequence, position, token)."""
    vocab = 3

    def configure_cache(self, seqs, tokens, pool):
        self.sizes, self.free, self.len = (seqs, tokens, pool), list(range(seqs)), {}

    def add_seq(self):
        s = self.free.pop()
        self.len[s] = 0
        return s

    def free_seq(self, s):
        self.free.append(s)

    def step_rows(self, seqs, tokens, rows):
        assert len(set(seqs)) == len(seqs)
        flat = []
        for s, toks in zip(seqs, tokens):
            for t in toks:
                flat.append((s, self.len[s], t))
                self.len[s] += 1
        return np.array([flat[r] for r in rows], dtype=np.float32).reshape(len(rows), 3)


def test_trace_runner_slots_and_rows():
    model = FakeModel()
    runner = trace.TraceRunner(model, 640)
    assert model.sizes == (trace.MAX_LIVE, 640, 640)
    a = runner.step([{"id": "x", "tokens": [5, 6, 7], "want": [2]}, {"id": "y", "tokens": [9], "want": [0]}])
    assert a[:, 1:].tolist() == [[2, 7], [0, 9]]
    b = runner.step([{"id": "y", "tokens": [1, 2], "want": []}], ["x"])
    assert b.shape == (0, 3) and len(model.free) == trace.MAX_LIVE - 1
    c = runner.step([{"id": "x", "tokens": [4], "want": [0]}, {"id": "y", "tokens": [3], "want": [0]}], ["x", "y"])
    assert c[:, 1:].tolist() == [[0, 4], [3, 3]] and len(model.free) == trace.MAX_LIVE


def test_trace_main_protocol(tmp_path, monkeypatch, capsys):
    import llaisys_b200.models as models

    monkeypatch.setattr(models, "load_model", lambda path, dtype: FakeModel())
    lines = [{"step": 0, "entries": [{"id": "q", "tokens": [1, 2], "want": [1, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": [2], "want": []}], "end": ["q"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(map(json.dumps, lines)) + "\n"))
    rc = trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"])
    assert rc == 0 and capsys.readouterr().out.split("\n")[:2] == ["done 0", "done 1"]
    got = np.fromfile(tmp_path / "0.f32", dtype="<f4").reshape(2, 3)
    assert got[:, 1:].tolist() == [[1, 2], [0, 1]] and not (tmp_path / "1.f32").exists()


def test_command_line_generates(tmp_path, capsys):
    """python -m llaisys_b200 generate, on a Qwen2 checkpoint (CPU): several prompts through the batching engine."""
    import safetensors.torch
    from llaisys_b200.cli import main
    from tests.test_qwen2_model import hf_greedy, hf_model

    cfg, hf = hf_model(seed=6)
    (tmp_path / "config.json").write_text(json.dumps({**cfg, "model_type": "qwen2"}))
    safetensors.torch.save_file({k: v.contiguous().clone() for k, v in hf.state_dict().items()}, str(tmp_path / "model.safetensors"))
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert "Qwen2" in capsys.readouterr().out
    assert main(["generate", "--model", str(tmp_path), "--device", "cpu", "--dtype", "float32", "--max-new-tokens", "4",
                 "--prompt", "3,1,4", "--prompt", "1,5,9,2,6"]) == 0
    out = [json.loads(line) for line in capsys.readouterr().out.strip().split("\n")]
    for row, p in zip(out, ([3, 1, 4], [1, 5, 9, 2, 6])):
        assert row["prompt"] == p and row["tokens"] == hf_greedy(hf, p, 4)[len(p):]
    assert main(["generate", "--model", str(tmp_path), "--device", "cpu", "--dtype", "float32", "--max-new-tokens", "3",
                 "--prompt", "7", "--top-k", "4", "--seed", "2"]) == 0
    assert len(json.loads(capsys.readouterr().out)["tokens"]) == 3
