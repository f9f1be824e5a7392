"""Small random Folivik models for the tests: configurations of several shapes and seeded weights."""
from __future__ import annotations

import copy
import functools

import numpy as np
import torch

from llaisys_b200.models.folivik import weight_shapes
from oracle import folivik as oracle
from tests.vozozen_cases import bf16_words, tokens  # noqa: F401

CLASSES = 4  # leading columns of the stream that only the embedding writes


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, *, scale=None, base=1e4):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}}


def attn(heads, kv_heads, dim, vdim, window, *, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                                           "scale": scale if scale is not None else dim ** -0.5}}


def mamba(heads, vdim, state, groups, norm_groups, taps):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups,
                                        "conv": taps}}


def moe(experts, top, ff, *, identity=0, groups=None, scale=1.0, shared=None):
    router = {"experts": experts, "top": top, "scale": scale, "identity": identity}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def config(layers, *, vocab=131, width=80, eps=1e-5):
    """layers: (mixer entry, mlp or None)"""
    return {"architecture": "Folivik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{**copy.deepcopy(entry), "mlp": copy.deepcopy(mlp)} for entry, mlp in layers]}


# name -> config
CASES = {
    "mixed": config([(mamba(4, 24, 48, 2, 1, 4), moe(6, 2, 40, identity=2, groups=(4, 3), scale=1.3, shared=56)),
                     (latent(3, 24, 16, 40, 48, 56, scale=0.2), moe(10, 3, 24, identity=2, groups=(2, 1), scale=2.0, shared=24)),
                     (attn(6, 2, 32, 24, 21), None),
                     (mamba(3, 40, 16, 3, 3, 2), moe(5, 1, 64, scale=0.7)),
                     (attn(4, 4, 16, 48, 1000, scale=0.4), moe(4, 4, 32, shared=40))]),
    "odd_sizes": config([(latent(5, 7, 6, 9, 11, 13), moe(7, 3, 19, identity=1, groups=(4, 2), shared=21)),
                         (mamba(5, 9, 11, 1, 5, 3), moe(3, 2, 13, identity=3, groups=(3, 3), scale=1.7, shared=5)),
                         (attn(3, 1, 13, 10, 17, scale=0.5), moe(9, 2, 27, scale=0.9))], vocab=97, width=51, eps=1e-3),
    "head_dim_128": config([(attn(8, 2, 128, 128, 40), moe(8, 2, 128, identity=0, groups=(2, 2), scale=1.2, shared=64)),
                            (latent(4, 128, 64, 128, 96, 128), moe(10, 3, 64, identity=2, groups=(4, 2), scale=1.1, shared=128)),
                            (mamba(4, 64, 128, 2, 2, 4), moe(8, 2, 64)),
                            (latent(16, 64, 64, 128, 64, 256, base=5e5), None),
                            (attn(12, 4, 128, 128, 130, scale=0.15), None)], width=128, vocab=77),
    "attention_only": config([(latent(4, 32, 32, 32, 40, 64), moe(6, 2, 40, identity=1, shared=16)),
                              (attn(2, 2, 64, 48, 33), moe(5, 3, 24, scale=1.4))], vocab=60, width=64),
    "recurrence_only": config([(mamba(8, 16, 32, 4, 2, 4), moe(6, 2, 48, shared=32)), (mamba(2, 8, 8, 1, 1, 1), None)], width=48, vocab=50),
    "single_choices": config([(mamba(1, 64, 64, 1, 1, 4), moe(3, 1, 32, identity=1)), (attn(1, 1, 32, 32, 1), moe(1, 1, 24)),
                              (latent(1, 16, 2, 16, 8, 24), moe(2, 1, 16, identity=2, groups=(2, 1)))], width=72, vocab=83),
}


def weights(cfg, seed=0):
    """Seeded weights (bfloat16 words). The choice of experts depends on the token and is clear in every precision: the stream's first
    columns hold the token's class, which the embedding writes and no layer's product changes, and routers read them alone. States
    of the recurrences last from a few tokens to hundreds."""
    rng = np.random.default_rng(seed)
    width = cfg["width"]
    out = {}
    for name, shape in weight_shapes(cfg).items():
        w = np.asarray(rng.standard_normal(shape))
        if name == "embed":
            w[:, :CLASSES] = 0.0
            w[np.arange(shape[0]), np.arange(shape[0]) % CLASSES] = 0.8 * width ** 0.5
        elif name.endswith(".router"):
            w[:, CLASSES:] = 0.0
            w[:, :CLASSES] = rng.permuted(np.tile(np.linspace(-0.5, 0.5, shape[0]), (CLASSES, 1)), axis=1).T
        elif name.endswith(".correction"):
            w = 0.03 * w
        elif name.endswith(("norm1", "norm2", "final.norm")):
            w = 1.0 + 0.2 * w
        elif name.endswith("norm"):
            w = 1.0 + 0.2 * w
        elif name.endswith(("temp", ".D")):
            w = 1.0 + 0.3 * w
        elif name.endswith(("r1", "r2")):
            w = 0.3 * np.abs(w) + 0.05
        elif name.endswith("A_log"):
            w = 0.5 * w
        elif name.endswith("dt_bias"):
            w = -3.0 + 1.5 * w
        elif name.endswith("conv.b"):
            w = 0.3 * w
        else:
            w = w * (1.2 / shape[-1] ** 0.5)
            if name.endswith((".o", ".down")):
                w[:CLASSES] = 0.0
        out[name] = bf16_words(w.astype(np.float32)).reshape(shape)
    return out


def choice_gap(logits, correction, router):
    """How far the last chosen and the first refused output are apart (choice scores; group scores too) for one token."""
    s = torch.softmax(logits, 0) + correction
    groups = router.get("groups") or {"count": 1, "keep": 1}
    score = s.view(groups["count"], -1)
    best = score.max(1).values.sort(descending=True)
    gap = float(best.values[groups["keep"] - 1] - best.values[groups["keep"]]) if groups["keep"] < groups["count"] else float("inf")
    among = score[best.indices[:groups["keep"]]].flatten().sort(descending=True).values
    return min(gap, float(among[router["top"] - 1] - among[router["top"]])) if router["top"] < len(among) else gap


def routing_gaps(cfg, w, toks):
    """The closest call of every layer with experts."""
    gaps, plain = [], oracle.route

    def watched(logits, correction, router):
        gaps.append(choice_gap(logits, correction, router))
        return plain(logits, correction, router)

    oracle.route = watched
    try:
        oracle.forward(cfg, w, toks)
    finally:
        oracle.route = plain
    return [min(gaps[i:i + len(toks)]) for i in range(0, len(gaps), len(toks))]


@functools.lru_cache(maxsize=None)
def _case(name, seed):
    cfg = copy.deepcopy(CASES[name])
    w = weights(cfg, seed)
    layers = [i for i, e in enumerate(cfg["layers"]) if e.get("mlp")]
    for attempt in range(1, 100): # routers whose choices are close are drawn again
        close = [i for i, gap in zip(layers, routing_gaps(cfg, w, tokens(cfg, 40))) if gap < 0.01]
        if not close:
            return cfg, w
        other = weights(cfg, seed + 1000 * attempt)
        for i in close:
            for part in ("router", "correction"):
                w[f"l{i}.mlp.{part}"] = other[f"l{i}.mlp.{part}"]
    raise AssertionError(f"{name}: no clear choice of experts")


def case(name, seed=0):
    cfg, w = _case(name, seed)
    return copy.deepcopy(cfg), dict(w)
