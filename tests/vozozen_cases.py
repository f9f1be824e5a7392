"""Small random Vozozen models for the tests: configurations of several shapes and seeded weights."""
from __future__ import annotations

import copy

import numpy as np

from llaisys_b200.models.vozozen import weight_shapes


def mixer(heads, kv_heads, dim, vdim, window, r_heads, r_dim, r_vdim, tau, scale=None, left_scale=0.8, right_scale=0.7):
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                     "scale": scale if scale is not None else dim ** -0.5},
            "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "tau": tau},
            "left_scale": left_scale, "right_scale": right_scale}


def config(layers, *, vocab=131, width=80, loop=None, softcap=20.0, embed_scale=3.0, eps=1e-5):
    """layers: (mixer, ff or None) pairs"""
    return {"architecture": "Vozozen", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "logit_softcap": softcap, "loop": loop,
            "layers": [{"type": "parallel", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
                       for m, ff in layers]}


def _cases():
    base = mixer(4, 2, 32, 32, 24, 3, 32, 48, 8.0)
    yield "looped", config([(base, 112), (mixer(6, 3, 16, 24, 9, 2, 16, 32, 4.0, scale=0.4), None), (base, 56)],
                           loop={"start": 1, "stop": 3, "times": 2}), [12, 7, 12]
    yield "one_pass_odd_sizes", config([(mixer(3, 1, 20, 12, 17, 1, 10, 14, 1.0), 37), (mixer(2, 2, 13, 9, 33, 5, 6, 7, 2.5), 50)],
                                       vocab=97, width=52, loop={"start": 0, "stop": 2, "times": 1}, softcap=9.0), [3, 5]
    yield "no_loop_window_1", config([(mixer(2, 1, 24, 24, 1, 2, 24, 24, 16.0, left_scale=1.0, right_scale=1.0), None),
                                      (mixer(4, 4, 8, 16, 1000, 1, 72, 80, 3.0), 64)], embed_scale=1.0), [16, 8]
    yield "head_dim_128", config([(mixer(6, 2, 128, 128, 40, 2, 128, 128, 12.0), 96), (mixer(8, 1, 128, 128, 130, 3, 64, 128, 16.0), 128)],
                                 width=64, loop={"start": 0, "stop": 1, "times": 3}), [16, 16]


CASES = {name: (cfg, ranks) for name, cfg, ranks in _cases()}


def bf16_words(x: np.ndarray) -> np.ndarray:
    """float32 -> bfloat16 words, to nearest even"""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def weights(cfg, ranks, seed=0, decay_bias=2.0):
    """Seeded weights (bfloat16 words). Norms around 1; decay biases spread, so that channels forget at different rates."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(cfg, ranks).items():
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("norm2"):
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith("a2.b"):
            w = decay_bias + 2.0 * rng.standard_normal(shape)
        elif name.endswith("embed"):
            w = rng.standard_normal(shape) / 3.0
        else:
            w = rng.standard_normal(shape) * (1.2 / shape[-1] ** 0.5)
        out[name] = bf16_words(w.astype(np.float32))
    return out


def case(name, seed=0):
    cfg, ranks = CASES[name]
    return copy.deepcopy(cfg), weights(cfg, ranks, seed)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).tolist()
