"""Vozozen on the C model API (include/llaisys/models/vozozen.h): layers of sliding-window attention and gated linear
attention side by side, with a range of layers run several times over. Runs on NVIDIA devices, in bfloat16 or float32.
"""
from __future__ import annotations

from typing import Mapping

from ..libllaisys import (DataType, LlaisysGatedLinearMeta, LlaisysVozozenLayerMeta, LlaisysVozozenMeta,
                          LlaisysWindowAttentionMeta)
from .base import NamedWeightsLM, tensor_rows


def _layer_meta(index: int, entry: Mapping, decay_rank: int) -> LlaisysVozozenLayerMeta:
    if entry.get("type") != "parallel":
        raise ValueError(f"layer {index}: unknown layer type {entry.get('type')!r}")
    mixer, mlp = entry["mixer"], entry.get("mlp")
    left, right = mixer["left"], mixer["right"]
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
    return LlaisysVozozenLayerMeta(
        left=LlaisysWindowAttentionMeta(heads=int(left["heads"]), kv_heads=int(left["kv_heads"]), dim=int(left["dim"]),
                                        vdim=int(left["vdim"]), window=int(left["mask"]["size"]), scale=float(left["scale"])),
        right=LlaisysGatedLinearMeta(heads=int(right["heads"]), dim=int(right["dim"]), vdim=int(right["vdim"]),
                                     rank=decay_rank, tau=float(right["tau"])),
        left_scale=float(mixer["left_scale"]), right_scale=float(mixer["right_scale"]), ff=int(mlp["ff"]) if mlp else 0)


def build_meta(config: Mapping, decay_ranks: list[int], dtype: DataType, max_seq_len: int | None = None) -> LlaisysVozozenMeta:
    """The C description of a model. decay_ranks: rows of every layer's `mix.right.a1` (a size only the weights hold)."""
    entries = config["layers"]
    layers = (LlaisysVozozenLayerMeta * len(entries))(*[_layer_meta(i, e, decay_ranks[i]) for i, e in enumerate(entries)])
    loop = config.get("loop")
    eos = config.get("eos_token_id")
    meta = LlaisysVozozenMeta(
        dtype=int(dtype), nlayer=len(entries), layers=layers, width=int(config["width"]), voc=int(config["vocab"]),
        maxseq=int(max_seq_len or config.get("max_position_embeddings", 4096)),
        embed_scale=float(config["embedding"]["scale"]), eps=float(config["norm"]["eps"]),
        logit_softcap=float(config.get("logit_softcap") or 0.0),
        loop_start=int(loop["start"]) if loop else 0, loop_stop=int(loop["stop"]) if loop else 0,
        loop_times=int(loop["times"]) if loop else 0, end_token=-1 if eos is None else int(eos))
    meta._layers = layers  # keeps the array alive as long as the struct
    return meta


def weight_shapes(config: Mapping, decay_ranks: list[int]) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a model's weights."""
    width, vocab = int(config["width"]), int(config["vocab"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (vocab, width)}
    if config.get("loop"):
        shapes["loop.in"] = (width, 2 * width)
    for i, entry in enumerate(config["layers"]):
        left, right, rank = entry["mixer"]["left"], entry["mixer"]["right"], decay_ranks[i]
        h, g, d, dv = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
        rh, rd, rv = right["heads"], right["dim"], right["vdim"]
        ml, mr = f"l{i}.mix.left.", f"l{i}.mix.right."
        shapes |= {f"l{i}.norm1": (width,), ml + "q": (h * d, width), ml + "k": (g * d, width), ml + "v": (g * dv, width),
                   ml + "q.norm": (d,), ml + "k.norm": (d,), ml + "g": (h, width), ml + "o": (width, h * dv),
                   mr + "q": (rh * rd, width), mr + "k": (rh * rd, width), mr + "v": (rh * rv, width),
                   mr + "g": (rh * rv, width), mr + "o": (width, rh * rv), mr + "norm": (rv,), mr + "a1": (rank, width),
                   mr + "a2": (rh * rd, rank), mr + "a2.b": (rh * rd,)}
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            shapes |= {f"l{i}.norm2": (width,), f"l{i}.mlp.up": (ff, width), f"l{i}.mlp.down": (width, ff)}
    return shapes | {"final.norm": (width,), "head": (vocab, width)}


class Vozozen(NamedWeightsLM):
    create = "llaisysVozozenModelCreate"

    def meta_of(self, config, shapes, dtype, max_seq_len):
        ranks = tensor_rows(shapes, [f"l{i}.mix.right.a1" for i in range(len(config["layers"]))])
        return build_meta(config, ranks, dtype, max_seq_len)

    def layer_runs(self) -> int:
        loop = self.config.get("loop")
        return len(self.config["layers"]) + ((loop["stop"] - loop["start"]) * (loop["times"] - 1) if loop else 0)
