"""bench.py --workload vozozen | doderax | lilovik | folivik: a design beside its closest relative at equal size, one GPU -- Vozozen
beside Qwen2, Doderax beside Vozozen, Lilovik beside Qwen2, Folivik beside Vozozen.

Two parts, one JSON line:
  models   prefill and decode throughput of whole models with random weights. Equal size: the same width, query and kv heads,
           layers and vocabulary, and an MLP of as many parameters (two matrices have an inner size 1.5 times that of Qwen2's
           three). Vozozen's second mixer (gated linear attention) comes on top of Qwen2's attention; Doderax has as many heads of
           the delta rule in every layer, and attention in every other one. Lilovik has Qwen2's attention heads and MLP sizes, and in
           every other layer a minGRU of as many parameters instead of the attention. Folivik has a Mamba-2 state space in every other
           layer and latent or windowed attention in the others, and experts of which a token passes as many parameters as an MLP has.
  kernels  every new kernel alone next to the like kernel of the relative, each as a fraction of its own roofline: CUDA graphs of
           launches over rotating buffers larger than L2, the median of the replays.
"""
from __future__ import annotations

import json
import statistics

import numpy as np

SIZES = {
    "1.5B-like": dict(width=1536, heads=12, kv_heads=2, gla_heads=6, ff=8960, layers=8, vocab=32768, window=1024),
    "8B-like": dict(width=4096, heads=32, kv_heads=8, gla_heads=16, ff=14336, layers=4, vocab=32768, window=1024),
}
D = 128
PREFILL = {"one prompt of 8192": [8192], "eight prompts of 1024": [1024] * 8}
DECODE_SEQS, DECODE_CTX, DECODE_STEPS = 64, 2048, 64
KEEP_FIRST, TAPS, LOW_RANK = 64, 4, 128  # Doderax: kept first tokens, convolution taps, ranks of its decay and gate projections
EXPERTS, IDENTITY, TOP, GROUPS, KEPT = 32, 4, 4, 4, 2  # Folivik
KV_RANK, ROT, STATE, STATE_V = 512, 64, 128, 64


def vozozen_config(s: dict) -> dict:
    mixer = {"left": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": D, "vdim": D, "mask": {"size": s["window"]},
                      "scale": D ** -0.5},
             "right": {"heads": s["gla_heads"], "dim": D, "vdim": D, "tau": 16.0}, "left_scale": 0.7, "right_scale": 0.7}
    layer = {"type": "parallel", "mixer": mixer, "mlp": {"kind": "dense", "ff": s["ff"] * 3 // 2}}
    return {"architecture": "Vozozen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0}, "logit_softcap": 30.0, "loop": None, "layers": [layer] * s["layers"]}


def qwen2_config(s: dict) -> dict:
    return {"hidden_size": s["width"], "num_attention_heads": s["heads"], "num_key_value_heads": s["kv_heads"], "head_dim": D,
            "intermediate_size": s["ff"], "num_hidden_layers": s["layers"], "vocab_size": s["vocab"], "rms_norm_eps": 1e-6,
            "rope_theta": 1e6}


def doderax_config(s: dict) -> dict:
    def delta(kv_heads):
        return {"heads": s["gla_heads"], "kv_heads": kv_heads, "dim": D, "vdim": D, "conv": TAPS}

    left = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": D, "vdim": D, "mask": {"size": s["window"], "keep_first": KEEP_FIRST},
            "rot": {"dims": D, "base": 1e6}, "scale": D ** -0.5}
    mlp = {"kind": "dense", "ff": s["ff"] * 3 // 2}
    layers = [{"type": "channel_delta", "mixer": delta(s["gla_heads"]), "mlp": mlp},
              {"type": "parallel", "mixer": {"left": left, "right": delta(s["gla_heads"] // 2)}, "mlp": mlp}]
    return {"architecture": "Doderax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 10007, "mul_cur": 257}}, "layers": layers * (s["layers"] // 2)}


def lilovik_config(s: dict) -> dict:
    attn = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": D, "vdim": D, "scale": D ** -0.5, "softcap": 30.0,
            "q_temp": {"coef": 0.1, "every": 1024}}
    mlp = {"kind": "dense", "ff": s["ff"]}
    layers = [{"type": "attention", "mixer": attn, "mlp": mlp}, {"type": "mingru", "mixer": {"width": gru_width(s)}, "mlp": mlp}]
    return {"architecture": "Lilovik", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "logit_scale": 0.5,
            "layers": layers * (s["layers"] // 2)}


def expert_ff(s: dict) -> int:
    """Four chosen experts and a shared one have about the parameters of the MLP."""
    return s["ff"] // (TOP + 1) // 128 * 128


def state_heads(s: dict) -> int:
    return 2 * s["width"] // STATE_V


def folivik_config(s: dict) -> dict:
    ff = expert_ff(s)
    mlp = {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": ff},
           "router": {"experts": EXPERTS, "top": TOP, "scale": 1.0, "identity": IDENTITY, "groups": {"count": GROUPS, "keep": KEPT}}}
    mamba = {"type": "mamba2", "mixer": {"heads": state_heads(s), "vdim": STATE_V, "state": STATE, "groups": s["kv_heads"],
                                         "norm_groups": s["kv_heads"], "conv": TAPS}}
    latent = {"type": "latent_attention", "mixer": {"heads": s["heads"], "dim": D, "rot_dim": ROT, "vdim": D, "q_rank": s["width"] // 2,
                                                    "kv_rank": KV_RANK, "rot": {"base": 1e4, "dims": ROT}, "scale": (D + ROT) ** -0.5}}
    attn = {"type": "attention", "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": D, "vdim": D, "mask": {"size": s["window"]},
                                           "scale": D ** -0.5}}
    layers = [{**e, "mlp": mlp} for e in (mamba, latent, mamba, attn)]
    return {"architecture": "Folivik", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers * (s["layers"] // 4)}


def gru_width(s: dict) -> int:
    """Channels of a minGRU with as many parameters as the attention."""
    return (s["heads"] + s["kv_heads"]) * D // 2


def attention_layers(family: str, s: dict) -> int:
    return s["layers"] // 2 if family in ("doderax", "lilovik") else s["layers"]


def build_model(torch, llaisys, family: str, s: dict):
    """-> the model, bytes of weights a decode step reads, parameters of the matrices applied to every token"""
    if family == "qwen2":
        from bench import qwen2_random_weights

        cfg = qwen2_config(s)
        model = llaisys.models.Qwen2(config=cfg, device=llaisys.DeviceType.NVIDIA, dtype=llaisys.DataType.BF16,
                                     max_seq_len=DECODE_CTX + 256)
        total = per_token = 0
        for name, value in qwen2_random_weights(cfg, 4, "cuda"):
            model.load_tensor(name, value)
            if "embed_tokens" not in name:
                total += value.numel() * 2
                per_token += value.numel() if value.ndim == 2 and name != "lm_head.weight" else 0
        return model, total, per_token
    if family == "doderax":
        from llaisys_b200.models.doderax import weight_shapes

        cfg = doderax_config(s)
        shapes = weight_shapes(cfg, [(LOW_RANK, LOW_RANK)] * s["layers"])
    elif family == "lilovik":
        from llaisys_b200.models.lilovik import weight_shapes

        cfg = lilovik_config(s)
        shapes = weight_shapes(cfg)
    elif family == "folivik":
        from llaisys_b200.models.folivik import weight_shapes

        cfg = folivik_config(s)
        shapes = weight_shapes(cfg)
    else:
        from llaisys_b200.models.vozozen import weight_shapes

        cfg = vozozen_config(s)
        shapes = weight_shapes(cfg, [16] * s["layers"])
    g = torch.Generator(device="cuda").manual_seed(4)
    weights, total, per_token = {}, 0, 0
    for name, shape in shapes.items():
        if family == "lilovik" and name.endswith(("talk", "pb", ".b")):
            w = torch.eye(shape[0]) + 0.1 if name.endswith("talk") else torch.full(shape, -3.0 if name.endswith("pb") else 0.0)
        elif name.endswith(("norm", "norm1", "norm2", "norm1b", "norm2b", ".out", "temp", ".D")):
            w = torch.ones(shape)
        elif name.endswith(("r1", "r2", "correction", "conv.b")):
            w = torch.full(shape, 0.1 if name.endswith(("r1", "r2")) else 0.0)
        elif name.endswith(("a2.b", "dt_bias")):
            w = torch.full(shape, 3.0 if family == "vozozen" else -5.0)
        elif name.endswith("A_log"):
            w = torch.zeros(shape)
        elif name.endswith(".conv"):
            w = torch.randn(shape, generator=g, device="cuda") * 0.5
        else:
            w = torch.randn(shape, generator=g, device="cuda") * 0.02
        weights[name] = w.bfloat16().cpu().view(torch.int16).numpy().view(np.uint16)
        if name not in ("embed", "bigram"):
            total += w.numel() * 2
            share = TOP / (EXPERTS + IDENTITY) if ".mlp.e" in name else 1.0  # of the tokens that pass an expert
            per_token += int(w.numel() * share) if w.ndim == 2 and name != "head" and not name.endswith(".conv") else 0
    cls = getattr(llaisys.models, family.capitalize())
    model = cls(config=cfg, state_dict=weights, dtype=llaisys.DataType.BF16)
    return model, total, per_token


def visible(n: int, window: int | None, keep: int = 0) -> int:
    """(query, key) pairs of a causal run of n tokens from an empty cache"""
    full = n * (n + 1) // 2
    if window is None or window >= n:
        return full
    out = n - window  # queries behind a full window; the i-th of them misses i tokens, `keep` of which it sees all the same
    kept = sum(min(i, keep) for i in range(1, min(out, keep) + 1)) + max(out - keep, 0) * keep
    return full - out * (out + 1) // 2 + kept


def prefill_flops(family: str, s: dict, lens: list[int], per_token: int) -> float:
    tokens = sum(lens)
    flops = 2.0 * tokens * per_token + 2.0 * len(lens) * s["vocab"] * s["width"]
    if family == "folivik":  # (W_uk and W_uv, applied to every token, are among per_token)
        latent = sum(visible(n, None) for n in lens) * 2.0 * (2 * D + ROT)
        windowed = sum(visible(n, s["window"]) for n in lens) * 4.0 * D
        return flops + s["layers"] // 4 * (s["heads"] * (latent + windowed) + 2 * state_heads(s) * tokens * 4.0 * STATE * STATE_V)
    window, keep = (None if family in ("qwen2", "lilovik") else s["window"]), (KEEP_FIRST if family == "doderax" else 0)
    flops += attention_layers(family, s) * s["heads"] * 4.0 * D * sum(visible(n, window, keep) for n in lens)
    if family not in ("qwen2", "lilovik"):  # state update and read-out, and the delta rule's correction
        flops += s["layers"] * s["gla_heads"] * tokens * (6.0 if family == "doderax" else 4.0) * D * D
    return flops


def measure_model(torch, llaisys, stream, family: str, s: dict, repeats: int) -> dict:
    from bench import _peaks

    hbm, _, sustained, kind = _peaks()
    model, weight_bytes, per_token = build_model(torch, llaisys, family, s)
    model.configure_cache(DECODE_SEQS, max(8192, DECODE_CTX + 2 * DECODE_STEPS), DECODE_SEQS * (DECODE_CTX + 2 * DECODE_STEPS + 16))
    rng = np.random.default_rng(0)
    rec = {"parameters_per_token": per_token, "prefill": {}, "decode": {}}
    for what, lens in PREFILL.items():
        prompts = [rng.integers(0, s["vocab"], n).tolist() for n in lens]
        times = []
        for r in range(3 + repeats):
            seqs = [model.add_seq() for _ in lens]
            a, b = (torch.cuda.Event(enable_timing=True) for _ in range(2))
            a.record(stream)
            model.step(seqs, prompts)
            b.record(stream)
            b.synchronize()
            if r >= 3:
                times.append(a.elapsed_time(b))
            for q in seqs:
                model.free_seq(q)
        ms, flops = statistics.median(times), prefill_flops(family, s, lens, per_token)
        rec["prefill"][what] = {"tokens_per_s": sum(lens) * 1e3 / ms, "ms": ms, "ms_min": min(times), "ms_max": max(times),
                                "tflops": flops / ms / 1e9, "frac_of_sustained_gemm": flops / ms / 1e9 / sustained}
    seqs = [model.add_seq() for _ in range(DECODE_SEQS)]
    nxt = []
    for i in range(0, DECODE_SEQS, 4):
        nxt += model.step(seqs[i:i + 4], [rng.integers(0, s["vocab"], DECODE_CTX).tolist() for _ in range(4)])
    nxt = model.decode_loop(seqs, nxt, 8)[-1].tolist()
    model.decode_loop(seqs, nxt, DECODE_STEPS + 1)
    ms = model.last_loop_ms
    keys = DECODE_CTX + DECODE_STEPS // 2
    if family not in ("qwen2", "lilovik"):
        keys = min(keys, s["window"] + (KEEP_FIRST if family == "doderax" else 0))
    kv = attention_layers(family, s) * DECODE_SEQS * keys * s["kv_heads"] * 2 * D * 2
    state = 2 * s["layers"] * DECODE_SEQS * s["gla_heads"] * D * D * 4 if family not in ("qwen2", "lilovik") else 0
    if family == "folivik":
        full = DECODE_CTX + DECODE_STEPS // 2
        kv = s["layers"] // 4 * DECODE_SEQS * 2 * (full * (KV_RANK + ROT) + min(full, s["window"]) * s["kv_heads"] * 2 * D)
        state = 2 * (s["layers"] // 2) * DECODE_SEQS * state_heads(s) * STATE * STATE_V * 4
    if family == "lilovik":
        state = 2 * (s["layers"] // 2) * DECODE_SEQS * gru_width(s) * 4
    moved = weight_bytes + kv + state
    rec["decode"] = {"tokens_per_s": DECODE_SEQS * 1e3 / ms, "ms_per_step": ms, "bytes": {"weights": weight_bytes, "kv": kv, "state": state},
                     "gb_per_s": moved / ms / 1e6, "frac_of_copy": moved / ms / 1e6 / hbm, "peak_kind": kind}
    model.close()
    return rec


# ---- kernels ----------------------------------------------------------------------------------------------------------------


class Kernels:
    """Timed launches of single kernels on the library's stream."""

    def __init__(self, torch, llaisys, stream, repeats: int):
        from bench import _peaks

        self.torch, self.ll, self.stream, self.repeats = torch, llaisys, stream, repeats
        self.cs = llaisys.context_stream()
        self.hbm, self.burst, _, self.kind = _peaks()
        self.gen = torch.Generator(device="cuda").manual_seed(1)

    def rand(self, *shape, scale=1.0):
        return (self.torch.randn(*shape, generator=self.gen, device="cuda") * scale).bfloat16()

    def i32(self, values):
        return self.torch.tensor(values, dtype=self.torch.int32, device="cuda")

    def time(self, launch, per_graph: int = 8) -> float:
        """Median microseconds per launch(i)"""
        from bench import replay_times

        torch = self.torch
        for i in range(3):
            launch(i)
        self.stream.synchronize()
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=self.stream):
            for i in range(per_graph):
                launch(i)
        return statistics.median(replay_times(torch, self.stream, graph, self.repeats)) * 1e3 / per_graph

    def memory(self, us: float, nbytes: int) -> dict:
        return {"us": us, "bytes": nbytes, "tb_per_s": nbytes / us / 1e6, "frac": nbytes / us / 1e3 / self.hbm, "of": f"{self.kind} copy"}

    def tensor(self, us: float, flops: float) -> dict:
        return {"us": us, "tflops": flops / us / 1e6, "frac": flops / us / 1e6 / self.burst, "of": f"{self.kind} burst bf16 GEMM"}

    def fading(self, heads: int, kv_heads: int, window: int, layers: int = 3) -> dict:
        """Windowed attention with a distance penalty and without, and the position-wise kernel with factors on the query heads and without."""
        torch, ll = self.torch, self.ll
        out = {}
        cache = ll.PagedKVCache(64 * 2 * window // 16, kv_heads, D, nlayer=layers, dtype=ll.DataType.BF16, device=ll.DeviceType.NVIDIA,
                                max_seqs=64, max_pages_per_seq=8192 // 16)
        cache.set_launch_overlap(True)
        a, b, temp = (torch.rand(heads, device="cuda") + 0.1 for _ in range(3))
        width, qn, kn = (heads + 2 * kv_heads) * D, self.rand(D), self.rand(D)
        for what, lens, q_lens in (("decode, 64 sequences", [2 * window] * 64, [1] * 64), ("one chunk of 8192", [8192], [8192]),
                                   ("eight chunks of 1024", [1024] * 8, [1024] * 8)):
            seqs, n = [cache.add_seq() for _ in lens], sum(q_lens)
            for q, length in zip(seqs, lens):
                cache.reserve(q, length)
            cache.flush()
            for layer in range(layers):  # every page holds something
                for q, length in zip(seqs, lens):
                    k, v = self.rand(length, kv_heads, D), self.rand(length, kv_heads, D)
                    cache.append_dev(layer, k, v, self.i32([q] * length), self.i32(list(range(length))), length, self.cs)
                    self.stream.synchronize()
            q, o = self.rand(n, heads, D), self.rand(n, heads, D)
            ids, kv = self.i32(seqs), self.i32(lens)
            starts = None if max(q_lens) == 1 else self.i32([0, *np.cumsum(q_lens).tolist()])
            common = dict(n_seqs=len(lens), total_q=n, max_q_len=max(q_lens), max_kv_len=max(lens), nh=heads, scale=D ** -0.5, stream=self.cs,
                          window=window)
            fade = self.time(lambda i: cache.fade_dev(i % layers, o, q, ids, starts, kv, fade_a=a, fade_b=b, **common))
            plain = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, starts, kv, **common))
            for name, us in (("window attention with penalty, ", fade), ("window attention, Vozozen, ", plain)):
                out[name + what] = self.memory(us, len(lens) * window * kv_heads * 2 * D * 2 + 2 * n * heads * D * 2) if starts is None else \
                    self.tensor(us, 4.0 * D * heads * sum(visible(x, window) for x in lens))
            if what != "eight chunks of 1024":
                ids_n = self.i32([s for s, c in zip(seqs, q_lens) for _ in range(c)])
                pos_n = self.i32([length - c + t for length, c in zip(lens, q_lens) for t in range(c)])
                proj = [self.rand(n, width) for _ in range(layers)]
                for name, factor in ((f"norm, factors + append, {n} rows", temp), (f"norm + append, Vozozen, {n} rows", None)):
                    us = self.time(lambda i: cache.norm_append_dev(
                        i % layers, self.cs, proj=proj[i % layers], row_stride=width, q_at=0, k_at=heads * D, v_at=(heads + kv_heads) * D,
                        gate_at=-1, q_norm=qn, k_norm=kn, eps=1e-6, gate_scale=1.0, q_out=q, row_scale=None, seq_ids_dev=ids_n,
                        positions_dev=pos_n, n_rows=n, nh=heads, head_scale=factor))
                    out[name] = self.memory(us, n * 2 * width * 2)
            for s in seqs:
                cache.free_seq(s)
        cache.check()
        cache.close()
        return out

    def latents(self, heads: int, kv_heads: int, q_rank: int, ctx: int = 2048, layers: int = 3) -> dict:
        """Attention over latents beside Qwen2's attention with as many heads: decode over 64 sequences, short chunks, and long chunks over
        keys and values made of the latents; the append in front."""
        torch, ll = self.torch, self.ll
        out, row = {}, KV_RANK + ROT
        lat = ll.PagedKVCache.with_latents(64 * ctx // 16, [(KV_RANK, ROT)] * layers, dtype=ll.DataType.BF16, max_seqs=64,
                                           max_pages_per_seq=8192 // 16)
        kv_cache = ll.PagedKVCache(64 * ctx // 16, kv_heads, D, nlayer=layers, dtype=ll.DataType.BF16, device=ll.DeviceType.NVIDIA,
                                   max_seqs=64, max_pages_per_seq=8192 // 16)
        kv_cache.set_launch_overlap(True)
        width = (q_rank + row + heads + 7) // 8 * 8
        qn, cn = self.rand(q_rank), self.rand(KV_RANK)
        for what, lens, q_lens in (("decode, 64 sequences", [ctx] * 64, [1] * 64), ("sixteen chunks of 32 behind 2016", [ctx] * 16, [32] * 16),
                                   ("one chunk of 8192", [8192], [8192]), ("eight chunks of 1024", [1024] * 8, [1024] * 8)):
            n, long, single = sum(q_lens), q_lens == lens, max(q_lens) == 1
            sets = []
            for cache in (lat, kv_cache):
                seqs = [cache.add_seq() for _ in lens]
                for q, length in zip(seqs, lens):
                    cache.reserve(q, length)
                cache.flush()
                sets.append(seqs)
            for layer in range(layers):  # every page holds something
                for i, length in enumerate(lens):
                    pos = self.i32(list(range(length)))
                    k, v = self.rand(length, kv_heads, D), self.rand(length, kv_heads, D)
                    kv_cache.append_dev(layer, k, v, self.i32([sets[1][i]] * length), pos, length, self.cs)
                    proj, table, ql = self.rand(length, width), torch.rand(length, ROT // 2, 2, device="cuda"), self.rand(length, q_rank)
                    lat.latent_append_dev(layer, self.cs, proj=proj, row_stride=width, q_at=0, kv_at=q_rank, gate_at=-1, q_rank=q_rank, rank=KV_RANK,
                                          rot_dims=ROT, nh=heads, q_norm=qn, kv_norm=cn, eps=1e-6, rot_table=table, q_latent=ql,
                                          q_latent_stride=q_rank, row_scale=None, seq_ids_dev=self.i32([sets[0][i]] * length), positions_dev=pos,
                                          n_rows=length)
                    self.stream.synchronize()
            starts = None if single else self.i32([0, *np.cumsum(q_lens).tolist()])
            kv, factor = self.i32(lens), torch.rand(n, heads, device="cuda")
            common = dict(n_seqs=len(lens), total_q=n, max_q_len=max(q_lens), max_kv_len=max(lens), nh=heads, stream=self.cs)
            q, o, ids = self.rand(n, heads, D), self.rand(n, heads, D), self.i32(sets[1])
            us = self.time(lambda i: kv_cache.attention_dev(i % layers, o, q, ids, starts, kv, scale=D ** -0.5, **common))
            seen = sum(visible(x, None) - visible(x - c, None) for x, c in zip(lens, q_lens))
            out["attention, Qwen2, " + what] = self.memory(us, sum(lens) * kv_heads * 2 * D * 2 + 2 * n * heads * D * 2) if single else \
                self.tensor(us, 4.0 * D * heads * seen)
            ids = self.i32(sets[0])
            if long:
                tokens = sum(lens) + 64
                context = torch.zeros(tokens, row, dtype=torch.bfloat16, device="cuda")
                pages = self.i32([int(x) // 16 for x in np.cumsum([0, *lens[:-1]])])
                us = self.time(lambda i: lat.latent_gather_dev(i % layers, context, row, ids, pages, kv, len(lens), max(lens), self.cs))
                out["gather of latents, " + what] = self.memory(us, 2 * sum(lens) * row * 2)
                keys, values = ([self.rand(tokens, heads, D) for _ in range(2)] for _ in range(2))
                q, o = self.rand(n, heads, D + ROT), self.rand(n, heads, D)
                us = self.time(lambda i: lat.expanded_dev(
                    self.cs, q=q, k=keys[i % 2], k_shared=context.data_ptr() + KV_RANK * 2, v=values[i % 2], shared_stride=row, tokens=tokens,
                    nh=heads, dim=D, rot_dim=ROT, vdim=D, page_starts_dev=pages, q_starts_dev=starts, kv_lens_dev=kv, n_seqs=len(lens),
                    scale=(D + ROT) ** -0.5, out=o, out_stride=heads * D, row_scale=factor))
                out["expanded latent attention, " + what] = self.tensor(us, 2.0 * (2 * D + ROT) * heads * seen)
                del keys, values
            else:
                q, o = self.rand(n, heads, row), self.rand(n, heads, KV_RANK)
                us = self.time(lambda i: lat.attention_dev(i % layers, o, q, ids, starts, kv, scale=(D + ROT) ** -0.5, row_scale=factor, **common))
                out["latent attention, " + what] = self.memory(us, sum(lens) * row * 2 + n * heads * (row + KV_RANK) * 2)
                out["latent attention, " + what]["tflops"] = 2.0 * (row + KV_RANK) * heads * seen / us / 1e6
            if single or what == "one chunk of 8192":
                pos = self.i32([length - c + t for length, c in zip(lens, q_lens) for t in range(c)])
                ids_n = self.i32([s for s, c in zip(sets[0], q_lens) for _ in range(c)])
                proj, table = [self.rand(n, width) for _ in range(layers)], torch.rand(n, ROT // 2, 2, device="cuda")
                ql = self.rand(n, q_rank)
                us = self.time(lambda i: lat.latent_append_dev(
                    i % layers, self.cs, proj=proj[i % layers], row_stride=width, q_at=0, kv_at=q_rank, gate_at=q_rank + row, q_rank=q_rank,
                    rank=KV_RANK, rot_dims=ROT, nh=heads, q_norm=qn, kv_norm=cn, eps=1e-6, rot_table=table, q_latent=ql, q_latent_stride=q_rank,
                    row_scale=factor, seq_ids_dev=ids_n, positions_dev=pos, n_rows=n))
                out[f"latent append, {n} rows"] = self.memory(us, n * (2 * (q_rank + row) * 2 + heads * 6 + ROT * 4))
            for cache, seqs in zip((lat, kv_cache), sets):
                for s in seqs:
                    cache.free_seq(s)
        for cache in (lat, kv_cache):
            cache.check()
            cache.close()
        return out

    def state_space(self, heads: int, groups: int, lens: list[int], copies: int = 3) -> dict:
        torch, ll = self.torch, self.ll
        decode, rows, inner = max(lens) == 1, sum(lens), heads * STATE_V
        channels = inner + 2 * groups * STATE
        width = (inner + channels + heads + 7) // 8 * 8
        copies = copies if decode or rows * width * 2 < 300e6 else 2
        proj = [self.rand(rows, width, scale=0.7) for _ in range(copies)]
        floats, n_scratch, n_seg = ll.state_space_sizes(ll.DataType.BF16, rows, heads, groups, STATE, STATE_V, TAPS)
        floats = (floats + 3) // 4 * 4
        state = [torch.zeros(len(lens), floats, device="cuda") for _ in range(copies)]
        conv, cb, norm = self.rand(channels, TAPS, scale=0.5), self.rand(channels, scale=0.1), self.rand(inner)
        a_log, bias, skip = torch.zeros(heads, device="cuda"), torch.full((heads,), -4.0, device="cuda"), torch.ones(heads, device="cuda")
        out, scratch, seg = self.rand(rows, inner), torch.empty(n_scratch, device="cuda"), torch.empty(n_seg, device="cuda")
        ids, starts = self.i32(list(range(len(lens)))), self.i32([0, *np.cumsum(lens).tolist()])
        kv = self.i32([x + 100 for x in lens])
        us = self.time(lambda i: ll.state_space_dev(
            ll.DataType.BF16, decode=decode, stream=self.cs, proj=proj[i % copies], row_stride=width, z_at=0, x_at=inner, dt_at=inner + channels,
            conv_w=conv, conv_b=cb, norm_w=norm, a_log=a_log, dt_bias=bias, d_skip=skip, taps=TAPS, heads=heads, groups=groups, dk=STATE,
            dv=STATE_V, norm_groups=groups, eps=1e-6, state=state[i % copies], slot_stride=floats, seq_ids_dev=ids, q_starts_dev=starts,
            kv_lens_dev=kv, n_seqs=len(lens), n_rows=rows, max_q_len=max(lens), out=out, out_stride=inner, scratch=scratch,
            scratch_floats=n_scratch, scratch_segments=seg, scratch_segment_floats=n_seg))
        rec = self.memory(us, rows * (width + inner) * 2 + 2 * len(lens) * floats * 4)
        if not decode:
            rec["f32_tflops_of_the_recurrence"] = rows * heads * 4.0 * STATE * STATE_V / us / 1e6
        return rec

    def experts(self, width: int, ff: int, rows: int, dense_ff: int) -> dict:
        """Choice, experts' products and weighted sum beside the products and activation of an MLP (the library's, as every model here runs
        them); parts of the experts' time are in between."""
        torch, ll = self.torch, self.ll
        copies, n = 2, EXPERTS + IDENTITY
        gate_up = [self.rand(EXPERTS, 2 * ff, width, scale=0.02) for _ in range(copies)]
        down = [self.rand(EXPERTS, width, ff, scale=0.02) for _ in range(copies)]
        h, nxt = self.rand(rows, width), self.rand(rows, width)
        x, logits = torch.randn(rows, width, device="cuda"), torch.randn(rows, n, device="cuda")
        ints = [torch.zeros(rows * TOP, dtype=torch.int32, device="cuda") for _ in range(3)]
        weights, counts = torch.zeros(rows * TOP, device="cuda"), torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
        line, act, out = self.rand(rows * TOP, width), self.rand(rows * TOP, ff), self.rand(rows * TOP, width)
        correction, gain = torch.zeros(n, device="cuda"), torch.ones((), device="cuda")
        us = self.time(lambda i: ll.experts_dev(
            ll.DataType.BF16, stream=self.cs, experts=EXPERTS, identity=IDENTITY, top=TOP, groups=GROUPS, keep=KEPT, width=width, ff=ff,
            n_rows=rows, scale=1.0, eps=1e-6, gate_up=gate_up[i % copies], down=down[i % copies], correction=correction, logits=logits,
            gain=gain, h=h, chosen=ints[0], weights=weights, place=ints[1], counts=counts, line=ints[2], rows=line, act=act, out=out, x=x,
            next=nxt))
        chosen = ints[0].view(rows, TOP)
        passed, used = int((chosen < EXPERTS).sum()), int(torch.unique(chosen[chosen < EXPERTS]).numel())
        rec = {}
        name = f"experts, {rows} rows"
        if rows <= 256:
            rec[name] = self.memory(us, used * 3 * ff * width * 2 + passed * (2 * width + 2 * ff) * 2)
        else:
            rec[name] = self.tensor(us, 6.0 * passed * width * ff)
        del gate_up, down
        w1, w2 = ([self.rand(a, b, scale=0.02) for _ in range(copies)] for a, b in ((2 * dense_ff, width), (width, dense_ff)))
        gu, u, y = self.rand(rows, 2 * dense_ff), self.rand(rows, dense_ff), torch.randn(rows, width, device="cuda").bfloat16()

        def dense(i):
            torch.mm(h, w1[i % copies].T, out=gu)
            torch.mul(gu[:, :dense_ff], gu[:, dense_ff:], out=u)
            torch.mm(u, w2[i % copies].T, out=y)

        us = self.time(dense)
        name = f"MLP, library products, {rows} rows"
        rec[name] = self.memory(us, 3 * dense_ff * width * 2) if rows <= 256 else self.tensor(us, 6.0 * rows * width * dense_ff)
        return rec

    def attention(self, heads: int, kv_heads: int, window: int, layers: int = 3, design: str = "vozozen") -> dict:
        """Decode over 64 sequences and one chunk of 8192 tokens, with the window and without one at equal visible keys /
        at full length (doderax: with kept first tokens and without); the position-wise kernel in front of each."""
        torch, ll = self.torch, self.ll
        out = {}
        n_seqs, ctx, rows = 64, 2 * window, 8192
        pages = max(n_seqs * ctx, rows) // 16
        cache = ll.PagedKVCache(pages, kv_heads, D, nlayer=layers, dtype=ll.DataType.BF16, device=ll.DeviceType.NVIDIA,
                                max_seqs=n_seqs, max_pages_per_seq=max(ctx, rows) // 16)
        seqs = [cache.add_seq() for _ in range(n_seqs)]
        for q in seqs:
            cache.reserve(q, ctx)
        cache.flush()
        cache.set_launch_overlap(True)
        width = (heads + 2 * kv_heads) * D
        for layer in range(layers):  # every page holds something
            for lo in range(0, n_seqs, 8):
                part = seqs[lo:lo + 8]
                ids, pos = self.i32([q for q in part for _ in range(ctx)]), self.i32(list(range(ctx)) * len(part))
                k, v = self.rand(len(part) * ctx, kv_heads, D), self.rand(len(part) * ctx, kv_heads, D)
                cache.append_dev(layer, k, v, ids, pos, len(part) * ctx, self.cs)
                self.stream.synchronize()
        q, o = self.rand(n_seqs, heads, D), self.rand(n_seqs, heads, D)
        factor = torch.rand(n_seqs, heads, device="cuda")
        ids, full, short = self.i32(seqs), self.i32([ctx] * n_seqs), self.i32([window] * n_seqs)
        kv_bytes = n_seqs * window * kv_heads * 2 * D * 2 + 2 * n_seqs * heads * D * 2
        common = dict(n_seqs=n_seqs, nh=heads, scale=D ** -0.5, stream=self.cs)
        us = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, None, full, total_q=n_seqs, max_q_len=1, max_kv_len=ctx,
                                                     window=window, row_scale=factor, **common))
        out["decode attention, window"] = self.memory(us, kv_bytes)
        if design == "doderax":
            us = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, None, full, total_q=n_seqs, max_q_len=1, max_kv_len=ctx,
                                                         window=window, keep_first=KEEP_FIRST, **common))
            out["decode attention, window and kept tokens"] = self.memory(us, kv_bytes * (window + KEEP_FIRST) // window)
        else:
            us = self.time(lambda i: cache.decode_dev(i % layers, o, q, ids, short, n_seqs, window, heads, D ** -0.5, self.cs))
            out["decode attention, Qwen2, as many keys"] = self.memory(us, kv_bytes)

        qn, kn = self.rand(D), self.rand(D)
        wide = width + heads  # the gate behind q | k | v
        for n in (n_seqs, rows):
            if n == rows:
                for s in seqs:
                    cache.free_seq(s)
                long = cache.add_seq()
                cache.reserve(long, rows)
                cache.flush()
                ids_n, pos_n = self.i32([long] * rows), self.i32(list(range(rows)))
            else:
                ids_n, pos_n = ids, self.i32([ctx - 1] * n_seqs)
            proj = [self.rand(n, (wide + 7) // 8 * 8) for _ in range(layers)]
            qo, fac = self.rand(n, heads, D), torch.empty(n, heads, device="cuda")
            moved = n * (2 * width * 2 + heads * 6)
            us = self.time(lambda i: cache.norm_append_dev(
                i % layers, self.cs, proj=proj[i % layers], row_stride=proj[0].shape[1], q_at=0, k_at=heads * D,
                v_at=(heads + kv_heads) * D, gate_at=width, q_norm=qn, k_norm=kn, eps=1e-6, gate_scale=0.7, q_out=qo, row_scale=fac,
                seq_ids_dev=ids_n, positions_dev=pos_n, n_rows=n, nh=heads))
            out[f"norm + append, {n} rows"] = self.memory(us, moved)
            if design == "doderax":
                table = torch.rand(n, D // 2, 2, device="cuda")
                us = self.time(lambda i: cache.norm_append_dev(
                    i % layers, self.cs, proj=proj[i % layers], row_stride=proj[0].shape[1], q_at=0, k_at=heads * D,
                    v_at=(heads + kv_heads) * D, gate_at=-1, q_norm=None, k_norm=None, eps=1e-6, gate_scale=1.0, q_out=qo, row_scale=None,
                    seq_ids_dev=ids_n, positions_dev=pos_n, n_rows=n, nh=heads, rot_dims=D, rot_table=table))
                out[f"rotation + append, {n} rows"] = self.memory(us, n * (2 * width * 2 + D * 4))
                continue
            packed = [self.rand(n, width) for _ in range(layers)]
            bias = self.rand(width)
            us = self.time(lambda i: self._rope_append(cache, i % layers, qo, packed[i % layers], bias, ids_n, pos_n, n, heads))
            out[f"rope + append, Qwen2, {n} rows"] = self.memory(us, n * 2 * width * 2)
        q, o = self.rand(rows, heads, D), self.rand(rows, heads, D)
        factor = torch.rand(rows, heads, device="cuda")
        ids, starts, lens = self.i32([long]), self.i32([0, rows]), self.i32([rows])
        common = dict(n_seqs=1, total_q=rows, max_q_len=rows, max_kv_len=rows, nh=heads, scale=D ** -0.5, stream=self.cs)
        us = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, starts, lens, window=window, row_scale=factor, **common))
        out["chunk attention, window, 8192 tokens"] = self.tensor(us, 4.0 * D * heads * visible(rows, window))
        if design == "doderax":
            us = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, starts, lens, window=window, keep_first=KEEP_FIRST, **common))
            out["chunk attention, window and kept tokens, 8192 tokens"] = self.tensor(us, 4.0 * D * heads * visible(rows, window, KEEP_FIRST))
        else:
            us = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, starts, lens, **common))
            out["chunk attention, Qwen2, 8192 tokens"] = self.tensor(us, 4.0 * D * heads * visible(rows, None))
        cache.check()
        cache.close()
        return out

    def _rope_append(self, cache, layer, qo, packed, bias, ids, pos, n, heads):
        lib = self.ll.libllaisys.LIB_LLAISYS
        rc = lib.llaisysPagedKVRopeAppendDev(cache._kv, layer, qo.data_ptr(), packed.data_ptr(), bias.data_ptr(), ids.data_ptr(),
                                             pos.data_ptr(), n, heads, 1e6, self.cs)
        assert rc == 0

    def gates(self, heads: int, kv_heads: int, ctx: int = 2048, layers: int = 3) -> dict:
        """Attention without a softmax beside Qwen2's on the same pages: decode over 64 sequences, one chunk of 8192 tokens, eight of
        1024; the position-wise kernel in front of each."""
        torch, ll = self.torch, self.ll
        out = {}
        n_seqs, rows = 64, 8192
        cache = ll.PagedKVCache(max(n_seqs * ctx, rows) // 16, kv_heads, D, nlayer=layers, dtype=ll.DataType.BF16,
                                device=ll.DeviceType.NVIDIA, max_seqs=n_seqs, max_pages_per_seq=max(ctx, rows) // 16)
        cache.set_launch_overlap(True)
        width = (heads + 2 * kv_heads) * D
        opt = dict(softcap=30.0, slopes=torch.tensor([2.0 ** (-8 * (h + 1) / heads) for h in range(heads)], device="cuda"),
                   bias=self.rand(heads) - 3, talk=(torch.eye(heads, device="cuda") + 0.1).bfloat16())
        bias, qn, kn = self.rand(width), self.rand(heads * D), self.rand(kv_heads * D)
        for what, lens, q_lens in (("decode", [ctx] * n_seqs, [1] * n_seqs), ("one chunk of 8192", [rows], [rows]),
                                   ("eight chunks of 1024", [1024] * 8, [1024] * 8)):
            seqs, n = [cache.add_seq() for _ in lens], sum(q_lens)
            for q, length in zip(seqs, lens):
                cache.reserve(q, length)
            cache.flush()
            for layer in range(layers):  # every page holds something
                for q, length in zip(seqs, lens):
                    k, v = self.rand(length, kv_heads, D), self.rand(length, kv_heads, D)
                    cache.append_dev(layer, k, v, self.i32([q] * length), self.i32(list(range(length))), length, self.cs)
                    self.stream.synchronize()
            q, o = self.rand(n, heads, D), self.rand(n, heads, D)
            ids, kv = self.i32(seqs), self.i32(lens)
            starts = None if what == "decode" else self.i32([0, *np.cumsum(q_lens).tolist()])
            common = dict(n_seqs=len(lens), total_q=n, max_q_len=max(q_lens), max_kv_len=max(lens), nh=heads, scale=D ** -0.5, stream=self.cs)
            gates = self.time(lambda i: cache.gates_dev(i % layers, o, q, ids, starts, kv, **common, **opt))
            soft = self.time(lambda i: cache.attention_dev(i % layers, o, q, ids, starts, kv, **common))
            for name, us in (("gated attention, ", gates), ("softmax attention, Qwen2, ", soft)):
                out[name + what] = self.memory(us, sum(lens) * kv_heads * 2 * D * 2 + 2 * n * heads * D * 2) if what == "decode" else \
                    self.tensor(us, 4.0 * D * heads * sum(visible(x, None) for x in lens))
            if what != "eight chunks of 1024":
                ids_n = self.i32([s for s, c in zip(seqs, q_lens) for _ in range(c)])
                pos_n = self.i32([length - c + t for length, c in zip(lens, q_lens) for t in range(c)])
                proj = [self.rand(n, width) for _ in range(layers)]
                us = self.time(lambda i: cache.norm_append_dev(
                    i % layers, self.cs, proj=proj[i % layers], row_stride=width, q_at=0, k_at=heads * D, v_at=(heads + kv_heads) * D,
                    gate_at=-1, q_norm=qn, k_norm=kn, eps=1e-6, gate_scale=1.0, q_out=q, row_scale=None, seq_ids_dev=ids_n,
                    positions_dev=pos_n, n_rows=n, nh=heads, row_norm=1, bias=bias, temp_coef=0.1, temp_every=1024.0))
                out[f"row norm + append, {n} rows"] = self.memory(us, n * 2 * width * 2)
                us = self.time(lambda i: self._rope_append(cache, i % layers, q, proj[i % layers], bias, ids_n, pos_n, n, heads))
                out[f"rope + append, Qwen2, {n} rows"] = self.memory(us, n * 2 * width * 2)
            for s in seqs:
                cache.free_seq(s)
        cache.check()
        cache.close()
        return out

    def min_gru(self, width: int, lens: list[int], copies: int = 6) -> dict:
        torch, ll = self.torch, self.ll
        rows = sum(lens)
        copies = copies if rows * width * 6 < 30e6 else 3
        proj = [self.rand(rows, 3 * width) for _ in range(copies)]
        state = [torch.zeros(len(lens), width, device="cuda") for _ in range(copies)]
        n_scratch = ll.min_gru_scratch_floats(rows, width)
        scratch = torch.empty(n_scratch, device="cuda")
        bz, bx, out = self.rand(width), self.rand(width), [self.rand(rows, width) for _ in range(copies)]
        ids, starts, kv = self.i32(list(range(len(lens)))), self.i32([0, *np.cumsum(lens).tolist()]), self.i32([x + 100 for x in lens])
        us = self.time(lambda i: ll.min_gru_dev(
            ll.DataType.BF16, decode=max(lens) == 1, stream=self.cs, proj=proj[i % copies], row_stride=3 * width, z_at=0, x_at=width,
            g_at=2 * width, bias_z=bz, bias_x=bx, width=width, state=state[i % copies], slot_stride=width, seq_ids_dev=ids,
            q_starts_dev=starts, kv_lens_dev=kv, n_seqs=len(lens), n_rows=rows, max_q_len=max(lens), out=out[i % copies], out_stride=width,
            scratch=scratch, scratch_floats=n_scratch))
        return self.memory(us, rows * 4 * width * 2 + 2 * len(lens) * width * 4)

    def gated_linear(self, heads: int, lens: list[int], rank: int = 16, copies: int = 3) -> dict:
        torch, ll = self.torch, self.ll
        decode, rows, n = max(lens) == 1, sum(lens), heads * D
        at = dict(q_at=0, k_at=n, v_at=2 * n, g_at=3 * n, z_at=4 * n)
        width = 4 * n + rank
        copies = copies if decode or rows * width * 2 < 300e6 else 2
        proj = [self.rand(rows, width, scale=0.7) for _ in range(copies)]
        state = [torch.zeros(len(lens), heads * D * D, device="cuda") for _ in range(copies)]
        w, b, norm = self.rand(n, rank, scale=0.3), self.rand(n) + 3, self.rand(D)
        out = self.rand(rows, n)
        raw = torch.empty(4, device="cuda")  # (the tensor-core form uses neither scratch at 128 value columns)
        floats = ll.gated_linear_segment_floats(ll.DataType.BF16, heads, D, D)
        seg = torch.empty(floats, device="cuda")
        ids, starts = self.i32(list(range(len(lens)))), self.i32([0, *np.cumsum(lens).tolist()])
        kv = self.i32([x + 100 for x in lens])
        us = self.time(lambda i: ll.gated_linear_dev(
            ll.DataType.BF16, decode=decode, stream=self.cs, proj=proj[i % copies], row_stride=width, **at, decay_w=w, decay_b=b,
            norm_w=norm, tau=16.0, q_scale=D ** -0.5, eps=1e-6, out_scale=0.7, heads=heads, dk=D, dv=D, rank=rank,
            state=state[i % copies], slot_stride=heads * D * D, seq_ids_dev=ids, q_starts_dev=starts, kv_lens_dev=kv,
            n_seqs=len(lens), n_rows=rows, max_q_len=max(lens), out=out, out_stride=n, scratch_raw=raw, scratch_decay=raw,
            scratch_segments=seg, scratch_segment_floats=floats))
        rec = self.memory(us, rows * (width + n) * 2 + 2 * len(lens) * heads * D * D * 4)
        if not decode:
            rec["f32_tflops_of_the_recurrence"] = rows * heads * 4.0 * D * D / us / 1e6
        return rec


    def gated_delta(self, heads: int, kv_heads: int, lens: list[int], rank: int, copies: int = 3) -> dict:
        """rank 0: one decay per head"""
        torch, ll = self.torch, self.ll
        decode, rows, nq, nv = max(lens) == 1, sum(lens), kv_heads * D, heads * D
        at, width = {}, 0
        for name, n in (("q", nq), ("k", nq), ("v", nv), ("b", heads), ("a", rank or heads), ("g", nv)):
            at[name], width = width, width + (n + 7) // 8 * 8
        copies = copies if decode or rows * width * 2 < 300e6 else 2
        proj = [self.rand(rows, width, scale=0.7) for _ in range(copies)]
        floats, n_scratch, n_seg = ll.gated_delta_sizes(ll.DataType.BF16, rows, heads, kv_heads, D, D, TAPS)
        state = [torch.zeros(len(lens), floats, device="cuda") for _ in range(copies)]
        conv = {f"conv_{n}": self.rand(m, TAPS, scale=0.5) for n, m in (("q", nq), ("k", nq), ("v", nv))}
        w = self.rand(nv, rank, scale=0.3) if rank else None
        bias, a_log, norm = self.rand(nv if rank else heads) - 5, self.rand(heads, scale=0.1), self.rand(D)
        out, scratch, seg = self.rand(rows, nv), torch.empty(n_scratch, device="cuda"), torch.empty(n_seg, device="cuda")
        ids, starts = self.i32(list(range(len(lens)))), self.i32([0, *np.cumsum(lens).tolist()])
        kv = self.i32([x + 100 for x in lens])
        us = self.time(lambda i: ll.gated_delta_dev(
            ll.DataType.BF16, decode=decode, stream=self.cs, proj=proj[i % copies], row_stride=width, q_at=at["q"], k_at=at["k"],
            v_at=at["v"], b_at=at["b"], a_at=at["a"], **conv, decay_w=w, decay_ld=rank, a_log=a_log, dt_bias=bias, norm_w=norm,
            gate=proj[i % copies].data_ptr() + at["g"] * 2, gate_stride=width, gate_silu=1, q_scale=D ** -0.5, eps=1e-6, unit_eps=1e-6,
            taps=TAPS, heads=heads, kv_heads=kv_heads, dk=D, dv=D, rank=rank, state=state[i % copies], slot_stride=floats,
            seq_ids_dev=ids, q_starts_dev=starts, kv_lens_dev=kv, n_seqs=len(lens), n_rows=rows, max_q_len=max(lens), out=out,
            out_stride=nv, scratch=scratch, scratch_floats=n_scratch, scratch_segments=seg, scratch_segment_floats=n_seg))
        rec = self.memory(us, rows * (width + nv) * 2 + 2 * len(lens) * floats * 4)
        if not decode:
            rec["f32_tflops_of_the_recurrence"] = rows * heads * 6.0 * D * D / us / 1e6
        return rec


def run(args) -> None:
    from bench import ClockSampler, _init_device

    torch, llaisys, rank, local_rank, world, _ = _init_device()
    if world != 1:
        raise SystemExit(f"--workload {args.workload} runs on one GPU")
    handle = llaisys.context_stream()
    stream = torch.cuda.ExternalStream(int(getattr(handle, "value", handle)))
    repeats = 10 if args.repeats == 100 else max(3, args.repeats)
    design = args.workload
    relative = {"vozozen": "qwen2", "doderax": "vozozen", "lilovik": "qwen2", "folivik": "vozozen"}[design]
    chunks = {"one run of 8192": [8192], "eight runs of 1024": [1024] * 8}
    models, kernels = {}, {}
    with ClockSampler(local_rank) as clocks:
        for name, s in SIZES.items():
            models[name] = {"size": s, **{f: measure_model(torch, llaisys, stream, f, s, repeats) for f in (design, relative)}}
            k = Kernels(torch, llaisys, stream, max(30, repeats))
            h = s["gla_heads"]
            if design == "lilovik":
                kernels[name] = k.gates(s["heads"], s["kv_heads"])
                kernels[name]["minGRU decode, 64 sequences"] = k.min_gru(gru_width(s), [1] * 64)
                for what, lens in chunks.items():
                    kernels[name]["minGRU chunk, " + what] = k.min_gru(gru_width(s), lens)
            elif design == "folivik":
                kernels[name] = k.fading(s["heads"], s["kv_heads"], s["window"]) | k.latents(s["heads"], s["kv_heads"], s["width"] // 2)
                for rows in (64, 8192):
                    kernels[name] |= k.experts(s["width"], expert_ff(s), rows, s["ff"])
                kernels[name]["state space decode, 64 sequences"] = k.state_space(state_heads(s), s["kv_heads"], [1] * 64)
                for what, lens in chunks.items():
                    kernels[name]["state space chunk, " + what] = k.state_space(state_heads(s), s["kv_heads"], lens)
            else:
                kernels[name] = k.attention(s["heads"], s["kv_heads"], s["window"], design=design)
            kernels[name]["gated linear decode, 64 sequences"] = k.gated_linear(h, [1] * 64)
            if design == "doderax":
                kernels[name]["gated delta decode, decay per channel, 64 sequences"] = k.gated_delta(h, h, [1] * 64, 16)
                kernels[name][f"gated delta decode, decay per channel of rank {LOW_RANK}, 64 sequences"] = k.gated_delta(h, h, [1] * 64, LOW_RANK)
                kernels[name]["gated delta decode, decay per head, 64 sequences"] = k.gated_delta(h, h // 2, [1] * 64, 0)
            for what, lens in chunks.items():
                kernels[name]["gated linear chunk, " + what] = k.gated_linear(h, lens)
                if design == "doderax":
                    kernels[name]["gated delta chunk, decay per channel, " + what] = k.gated_delta(h, h, lens, 16)
                    kernels[name][f"gated delta chunk, decay per channel of rank {LOW_RANK}, " + what] = k.gated_delta(h, h, lens, LOW_RANK)
                    kernels[name]["gated delta chunk, decay per head, " + what] = k.gated_delta(h, h // 2, lens, 0)
    decode = models["8B-like"][design]["decode"]
    print(json.dumps({
        "metric": f"decode tokens/s ({design.capitalize()}, 8B-like layers, greedy)", "value": decode["tokens_per_s"], "unit": "tokens/s",
        "n_gpus": 1, "steps": DECODE_STEPS, "warmup": 8, "ms_per_step": decode["ms_per_step"], "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, random-token prompts)",
        "config": {"workload": design, "decode": f"{DECODE_SEQS} sequences, {DECODE_CTX}-token prompts", "prefill": list(PREFILL),
                   "l2": "weights, caches and rotated kernel buffers are larger than L2"},
        "models": models, "kernels": kernels, "clocks": clocks.summary(),
        "timing": "CUDA events: prefill around step(), decode around the library's graph replays, kernels around graph replays (median)",
    }), flush=True)
