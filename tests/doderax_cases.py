"""Small random Doderax models for the tests: configurations of several shapes and seeded weights."""
from __future__ import annotations

import copy

import numpy as np

from llaisys_b200.models.doderax import weight_shapes
from tests.vozozen_cases import bf16_words, tokens  # noqa: F401


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attn(heads, kv_heads, dim, vdim, window, keep_first, rot_dims, base=10000.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep_first},
            "rot": {"dims": rot_dims, "base": base}, "scale": scale if scale is not None else dim ** -0.5}


def config(layers, *, vocab=131, width=80, buckets=53, mul_prev=11, mul_cur=5, logit_scale=0.6, eps=1e-5):
    """layers: (delta mixer, ff or None) or (attention, delta mixer, ff or None)"""
    entries = []
    for *mixer, ff in layers:
        kind = "channel_delta" if len(mixer) == 1 else "parallel"
        entries.append({"type": kind, "mixer": mixer[0] if len(mixer) == 1 else {"left": mixer[0], "right": mixer[1]},
                        "mlp": None if ff is None else {"kind": "dense", "ff": ff}})
    return {"architecture": "Doderax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": entries}


# name -> (config, (decay rank, gate rank) per layer)
def _cases():
    yield "mixed", config([(delta(4, 2, 24, 20, 4), 112), (attn(4, 2, 32, 20, 24, 5, 8), delta(3, 3, 16, 12, 3), 72),
                           (delta(3, 1, 16, 32, 2), None), (attn(6, 2, 12, 28, 40, 18, 12, 500.0, 0.4), delta(6, 2, 20, 8, 5), None)]), \
        [(12, 7), (0, 0), (5, 9), (0, 0)]
    yield "tiles", config([(attn(2, 1, 40, 24, 33, 1, 20, 77.0), delta(4, 2, 64, 32, 3), 96), (delta(3, 1, 40, 48, 4), 104),
                           (delta(2, 2, 96, 136, 2), 40)], width=96, buckets=7, mul_prev=1, mul_cur=1, logit_scale=1.0), \
        [(0, 0), (16, 24), (33, 8)]
    yield "odd_sizes", config([(delta(5, 5, 13, 9, 1), 37), (attn(3, 1, 10, 7, 17, 0, 6), delta(2, 1, 6, 7, 5), 50)], vocab=97, width=52,
                              buckets=1009, mul_prev=100003, mul_cur=-7, eps=1e-3), [(3, 5), (0, 0)]
    yield "head_dim_128", config([(delta(2, 1, 128, 128, 4), 96), (attn(6, 2, 128, 128, 40, 20, 128), delta(2, 1, 128, 128, 4), 128),
                                  (attn(8, 1, 128, 128, 130, 65, 32, 1e6), delta(1, 1, 64, 128, 3), None)], width=64), \
        [(16, 16), (0, 0), (0, 0)]
    yield "delta_only", config([(delta(2, 1, 144, 40, 7), 64), (delta(6, 3, 8, 8, 3), None)], width=64, vocab=71), [(4, 4), (40, 1)]


CASES = {name: (cfg, ranks) for name, cfg, ranks in _cases()}


def weights(cfg, ranks, seed=0, bias=-2.0):
    """Seeded weights (bfloat16 words). Decay biases spread, so that heads and channels forget at different rates."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(cfg, ranks).items():
        if name.endswith("norm1") or name == "final.norm":
            w = 0.2 * rng.standard_normal(shape)
        elif name.endswith(("norm", ".out")):
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith("A_log"):
            w = 0.7 * rng.standard_normal(shape)
        elif name.endswith("dt_bias"):
            w = bias + 2.0 * rng.standard_normal(shape)
        elif name in ("embed", "bigram"):
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) * (1.2 / shape[-1] ** 0.5)
        out[name] = bf16_words(w.astype(np.float32))
    return out


def case(name, seed=0):
    cfg, ranks = CASES[name]
    return copy.deepcopy(cfg), weights(cfg, ranks, seed)
