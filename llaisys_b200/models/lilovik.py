"""Lilovik on the C model API (include/llaisys/models/lilovik.h): norms before and after each sublayer, and layers that mix tokens by
attention without a softmax (weights mixed over the heads) or by a minGRU. Runs on NVIDIA devices, in bfloat16, float16 or float32.
"""
from __future__ import annotations

from typing import Mapping

from ..libllaisys import DataType, LlaisysGatesAttentionMeta, LlaisysLilovikLayerMeta, LlaisysLilovikMeta
from .base import NamedWeightsLM

LAYER_TYPES = ("attention", "mingru")


def _layer_meta(index: int, entry: Mapping) -> LlaisysLilovikLayerMeta:
    if entry.get("type") not in LAYER_TYPES:
        raise ValueError(f"layer {index}: unknown layer type {entry.get('type')!r}")
    mixer, mlp = entry["mixer"], entry.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
    ff = int(mlp["ff"]) if mlp else 0
    if entry["type"] == "mingru":
        return LlaisysLilovikLayerMeta(recurrent=1, gru_width=int(mixer["width"]), ff=ff)
    temp = mixer.get("q_temp")
    attn = LlaisysGatesAttentionMeta(
        heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]), vdim=int(mixer["vdim"]),
        scale=float(mixer["scale"]), softcap=float(mixer.get("softcap") or 0.0), temp_coef=float(temp["coef"]) if temp else 0.0,
        temp_every=float(temp["every"]) if temp else 1.0)
    return LlaisysLilovikLayerMeta(recurrent=0, attn=attn, ff=ff)


def build_meta(config: Mapping, dtype: DataType, max_seq_len: int | None = None) -> LlaisysLilovikMeta:
    """The C description of a model."""
    entries = config["layers"]
    layers = (LlaisysLilovikLayerMeta * len(entries))(*[_layer_meta(i, e) for i, e in enumerate(entries)])
    eos, logit_scale = config.get("eos_token_id"), config.get("logit_scale")
    meta = LlaisysLilovikMeta(
        dtype=int(dtype), nlayer=len(entries), layers=layers, width=int(config["width"]), voc=int(config["vocab"]),
        maxseq=int(max_seq_len or config.get("max_position_embeddings", 4096)), eps=float(config["norm"]["eps"]),
        logit_scale=1.0 if logit_scale is None else float(logit_scale), end_token=-1 if eos is None else int(eos))
    meta._layers = layers  # keeps the array alive as long as the struct
    return meta


def weight_shapes(config: Mapping) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a model's weights."""
    width, vocab = int(config["width"]), int(config["vocab"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (vocab, width)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        shapes |= {p + "norm1": (width,), p + "norm1b": (width,)}
        if entry["type"] == "mingru":
            n = m["width"]
            shapes |= {p + "mix.z": (n, width), p + "mix.z.b": (n,), p + "mix.x": (n, width), p + "mix.x.b": (n,), p + "mix.g": (n, width),
                       p + "mix.o": (width, n)}
        else:
            rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for name, n in rows.items():
                shapes |= {p + f"mix.{name}": (n, width), p + f"mix.{name}.b": (n,)}
            shapes |= {p + "mix.q.norm": (rows["q"],), p + "mix.k.norm": (rows["k"],), p + "mix.talk": (m["heads"], m["heads"]),
                       p + "mix.pb": (m["heads"],), p + "mix.o": (width, m["heads"] * m["vdim"])}
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            shapes |= {p + "norm2": (width,), p + "norm2b": (width,), p + "mlp.gate": (ff, width), p + "mlp.up": (ff, width),
                       p + "mlp.down": (width, ff)}
    return shapes | {"final.norm": (width,), "head": (vocab, width)}


class Lilovik(NamedWeightsLM):
    create = "llaisysLilovikModelCreate"

    def meta_of(self, config, shapes, dtype, max_seq_len):
        return build_meta(config, dtype, max_seq_len)
