"""Doderax on the C model API (include/llaisys/models/doderax.h): layers whose mixer (a gated delta rule, or windowed attention
with rotary positions and kept first tokens beside one) and MLP read one norm, and an embedding of token pairs. Runs on NVIDIA
devices, in bfloat16, float16 or float32.
"""
from __future__ import annotations

from typing import Mapping

from ..libllaisys import (DataType, LlaisysDeltaMixerMeta, LlaisysDoderaxLayerMeta, LlaisysDoderaxMeta, LlaisysSinkAttentionMeta)
from .base import NamedWeightsLM, tensor_rows

LAYER_TYPES = ("parallel", "channel_delta")


def _delta_meta(mixer: Mapping, decay_rank: int, gate_rank: int) -> LlaisysDeltaMixerMeta:
    return LlaisysDeltaMixerMeta(heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]),
                                 vdim=int(mixer["vdim"]), taps=int(mixer["conv"]), decay_rank=decay_rank, gate_rank=gate_rank)


def _layer_meta(index: int, entry: Mapping, ranks: tuple[int, int]) -> LlaisysDoderaxLayerMeta:
    """ranks: of the decay and gate projections (channel_delta; sizes only the weights hold)."""
    if entry.get("type") not in LAYER_TYPES:
        raise ValueError(f"layer {index}: unknown layer type {entry.get('type')!r}")
    mixer, mlp = entry["mixer"], entry.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {mlp.get('kind')!r}")
    ff = int(mlp["ff"]) if mlp else 0
    if entry["type"] == "channel_delta":
        return LlaisysDoderaxLayerMeta(parallel=0, delta=_delta_meta(mixer, *ranks), ff=ff)
    left = mixer["left"]
    rot = left.get("rot")
    attn = LlaisysSinkAttentionMeta(
        heads=int(left["heads"]), kv_heads=int(left["kv_heads"]), dim=int(left["dim"]), vdim=int(left["vdim"]),
        window=int(left["mask"]["size"]), keep_first=int(left["mask"]["keep_first"]), rot_dims=int(rot["dims"]) if rot else 0,
        rot_base=float(rot["base"]) if rot else 0.0, scale=float(left["scale"]))
    return LlaisysDoderaxLayerMeta(parallel=1, attn=attn, delta=_delta_meta(mixer["right"], 0, 0), ff=ff)


def low_ranks(config: Mapping, shapes: Mapping[str, tuple[int, ...]]) -> list[tuple[int, int]]:
    """Ranks of every layer's decay and gate projections, (0, 0) where it has none."""
    return [tuple(tensor_rows(shapes, [f"l{i}.mix.a1", f"l{i}.mix.g1"])) if e.get("type") == "channel_delta" else (0, 0)
            for i, e in enumerate(config["layers"])]


def build_meta(config: Mapping, ranks: list[tuple[int, int]], dtype: DataType, max_seq_len: int | None = None) -> LlaisysDoderaxMeta:
    """The C description of a model; ranks as low_ranks gives them."""
    entries = config["layers"]
    layers = (LlaisysDoderaxLayerMeta * len(entries))(*[_layer_meta(i, e, ranks[i]) for i, e in enumerate(entries)])
    pairs = (config.get("embedding") or {}).get("bigram")
    eos, logit_scale = config.get("eos_token_id"), config.get("logit_scale")
    meta = LlaisysDoderaxMeta(
        dtype=int(dtype), nlayer=len(entries), layers=layers, width=int(config["width"]), voc=int(config["vocab"]),
        maxseq=int(max_seq_len or config.get("max_position_embeddings", 4096)),
        pair_buckets=int(pairs["buckets"]) if pairs else 0, pair_mul_prev=int(pairs["mul_prev"]) if pairs else 0,
        pair_mul_cur=int(pairs["mul_cur"]) if pairs else 0, eps=float(config["norm"]["eps"]),
        logit_scale=1.0 if logit_scale is None else float(logit_scale), end_token=-1 if eos is None else int(eos))
    meta._layers = layers  # keeps the array alive as long as the struct
    return meta


def weight_shapes(config: Mapping, ranks: list[tuple[int, int]]) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a model's weights."""
    width, vocab = int(config["width"]), int(config["vocab"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (vocab, width)}
    pairs = (config.get("embedding") or {}).get("bigram")
    if pairs:
        shapes["bigram"] = (int(pairs["buckets"]) + 1, width)

    def delta(p: str, m: Mapping) -> dict[str, tuple[int, ...]]:
        nq, nv, taps = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["conv"]
        return {p + "q": (nq, width), p + "q.conv": (nq, taps), p + "k": (nq, width), p + "k.conv": (nq, taps), p + "v": (nv, width),
                p + "v.conv": (nv, taps), p + "b": (m["heads"], width), p + "A_log": (m["heads"],), p + "norm": (m["vdim"],),
                p + "o": (width, nv)}

    for i, entry in enumerate(config["layers"]):
        p, mixer = f"l{i}.mix.", entry["mixer"]
        shapes[f"l{i}.norm1"] = (width,)
        if entry["type"] == "channel_delta":
            nk, nv, (decay, gate) = mixer["heads"] * mixer["dim"], mixer["heads"] * mixer["vdim"], ranks[i]
            shapes |= delta(p, mixer) | {p + "a1": (decay, width), p + "a2": (nk, decay), p + "dt_bias": (nk,),
                                         p + "g1": (gate, width), p + "g2": (nv, gate)}
        else:
            left, right = mixer["left"], mixer["right"]
            h, g, d, dv = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
            pl, pr = p + "left.", p + "right."
            shapes |= {pl + "q": (h * d, width), pl + "k": (g * d, width), pl + "v": (g * dv, width), pl + "o": (width, h * dv),
                       pl + "out": (width,)}
            shapes |= delta(pr, right) | {pr + "a": (right["heads"], width), pr + "dt_bias": (right["heads"],),
                                          pr + "g": (right["heads"] * right["vdim"], width), pr + "out": (width,)}
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            shapes |= {f"l{i}.mlp.up": (ff, width), f"l{i}.mlp.down": (width, ff)}
    return shapes | {"final.norm": (width,), "head": (vocab, width)}


class Doderax(NamedWeightsLM):
    create = "llaisysDoderaxModelCreate"

    def meta_of(self, config, shapes, dtype, max_seq_len):
        return build_meta(config, low_ranks(config, shapes), dtype, max_seq_len)
