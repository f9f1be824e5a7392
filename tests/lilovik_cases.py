"""Small random Lilovik models for the tests: configurations of several shapes and seeded weights."""
from __future__ import annotations

import copy

import numpy as np

from llaisys_b200.models.lilovik import weight_shapes
from tests.vozozen_cases import bf16_words, tokens  # noqa: F401


def attn(heads, kv_heads, dim, vdim, *, scale=None, softcap=None, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if softcap is not None:
        m["softcap"] = softcap
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def gru(width):
    return {"width": width}


def config(layers, *, vocab=131, width=80, logit_scale=0.6, eps=1e-5):
    """layers: (mixer, ff or None)"""
    entries = [{"type": "mingru" if "width" in mixer else "attention", "mixer": mixer,
                "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for mixer, ff in layers]
    return {"architecture": "Lilovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": entries}


# name -> config
CASES = {
    "mixed": config([(attn(6, 2, 32, 16, scale=0.3, softcap=7.0, temp=(0.4, 20)), 112), (gru(72), 56), (gru(40), None),
                     (attn(4, 1, 48, 64, softcap=3.0, temp=(0.7, 1)), None), (attn(3, 3, 16, 32, temp=(-0.2, 33)), 72)]),
    "head_dim_128": config([(attn(8, 2, 128, 128, scale=0.15, softcap=12.0, temp=(0.2, 50)), 96), (gru(200), 64),
                            (attn(12, 1, 128, 96, scale=0.2, softcap=30.0), None)], width=64, vocab=77),
    "odd_sizes": config([(gru(37), 29), (attn(5, 5, 13, 9, softcap=5.0, temp=(0.5, 7)), 37), (attn(3, 1, 10, 7, scale=0.5), None)], vocab=97,
                        width=51, eps=1e-3, logit_scale=1.0),
    "attention_only": config([(attn(20, 4, 16, 16, scale=0.4, softcap=9.0, temp=(1.0, 3)), 64), (attn(2, 2, 64, 48, softcap=1.5), 40)],
                             vocab=60, width=48),
    "recurrence_only": config([(gru(96), 48), (gru(8), None)], width=32, vocab=50, logit_scale=2.0),
}


def weights(cfg, seed=0):
    """Seeded weights (bfloat16 words). Score biases keep most attention weights small, so that single keys matter; update gates
    lean towards keeping, so that early tokens last."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(cfg).items():
        w = rng.standard_normal(shape)
        if name.endswith((".q.norm", ".k.norm")):
            w = 1.0 + 0.2 * w
        elif "norm" in name:
            w = 0.2 * w
        elif name.endswith("talk"):
            w = 0.8 * np.eye(shape[0]) + 0.4 * w / shape[0] ** 0.5
        elif name.endswith("pb"):
            w = -2.0 + w
        elif name.endswith("z.b"):
            w = -2.5 + 1.5 * w
        elif name.endswith(".b"):
            w = 0.5 * w
        elif name != "embed":
            w = w * (1.2 / shape[-1] ** 0.5)
        out[name] = bf16_words(w.astype(np.float32))
    return out


def case(name, seed=0):
    cfg = copy.deepcopy(CASES[name])
    return cfg, weights(cfg, seed)
