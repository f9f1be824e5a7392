"""Folivik on the C model API (include/llaisys/models/folivik.h): layers of attention over latents, windowed attention with a
logarithmic distance penalty, or a Mamba-2 state space, each followed by a mixture of experts. Runs on NVIDIA devices, in bfloat16,
float16 or float32.
"""
from __future__ import annotations

from typing import Mapping

from ..libllaisys import (DataType, LlaisysExpertLayerMeta, LlaisysFadingAttentionMeta, LlaisysFolivikLayerMeta, LlaisysFolivikMeta,
                          LlaisysLatentAttentionMeta, LlaisysStateSpaceMixerMeta)
from .base import NamedWeightsLM

LAYER_TYPES = ("latent_attention", "attention", "mamba2")  # in the order of the C enumeration


def _check_rotation(where: str, mixer: Mapping) -> None:
    if mixer["rot"]["dims"] != mixer["rot_dim"]:
        raise ValueError(f"{where}: the whole rotated part turns ({mixer['rot_dim']} dims), not {mixer['rot']['dims']}")


def _experts_meta(where: str, mlp: Mapping | None) -> LlaisysExpertLayerMeta:
    if mlp is None:
        return LlaisysExpertLayerMeta()
    if mlp.get("kind") != "moe":
        raise ValueError(f"{where}: unknown feed-forward kind {mlp.get('kind')!r}")
    router, shared = mlp["router"], mlp.get("shared")
    groups = router.get("groups") or {"count": 1, "keep": 1}
    experts, identity = int(router["experts"]), int(router.get("identity") or 0)
    count, keep, top = int(groups["count"]), int(groups["keep"]), int(router["top"])
    if count < 1 or (experts + identity) % count or not 1 <= keep <= count or not 1 <= top <= keep * ((experts + identity) // count):
        raise ValueError(f"{where}: {experts} + {identity} router outputs in {count} groups, {keep} kept, {top} chosen do not fit together")
    scale = router.get("scale")
    return LlaisysExpertLayerMeta(experts=experts, identity=identity, top=top, groups=count, keep=keep, ff=int(mlp["expert"]["ff"]),
                                  shared_ff=int(shared["ff"]) if shared else 0, scale=1.0 if scale is None else float(scale))


def _layer_meta(index: int, entry: Mapping) -> LlaisysFolivikLayerMeta:
    where, kind, m = f"layer {index}", entry.get("type"), entry["mixer"]
    if kind not in LAYER_TYPES:
        raise ValueError(f"{where}: unknown layer type {kind!r}")
    layer = LlaisysFolivikLayerMeta(mixer=LAYER_TYPES.index(kind), mlp=_experts_meta(where, entry.get("mlp")))
    if kind == "latent_attention":
        _check_rotation(where, m)
        layer.latent = LlaisysLatentAttentionMeta(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                                  q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), rot_base=float(m["rot"]["base"]),
                                                  scale=float(m["scale"]))
    elif kind == "attention":
        layer.attn = LlaisysFadingAttentionMeta(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                                window=int(m["mask"]["size"]), scale=float(m["scale"]))
    else:
        layer.ssm = LlaisysStateSpaceMixerMeta(heads=int(m["heads"]), groups=int(m["groups"]), state=int(m["state"]), vdim=int(m["vdim"]),
                                               taps=int(m["conv"]), norm_groups=int(m["norm_groups"]))
    return layer


def build_meta(config: Mapping, dtype: DataType, max_seq_len: int | None = None) -> LlaisysFolivikMeta:
    """The C description of a model."""
    entries = config["layers"]
    layers = (LlaisysFolivikLayerMeta * len(entries))(*[_layer_meta(i, e) for i, e in enumerate(entries)])
    eos = config.get("eos_token_id")
    meta = LlaisysFolivikMeta(dtype=int(dtype), nlayer=len(entries), layers=layers, width=int(config["width"]), voc=int(config["vocab"]),
                              maxseq=int(max_seq_len or config.get("max_position_embeddings", 4096)), eps=float(config["norm"]["eps"]),
                              end_token=-1 if eos is None else int(eos))
    meta._layers = layers  # keeps the array alive as long as the struct
    return meta


def weight_shapes(config: Mapping) -> dict[str, tuple[int, ...]]:
    """Names and shapes of a model's weights."""
    width, vocab = int(config["width"]), int(config["vocab"])
    shapes: dict[str, tuple[int, ...]] = {"embed": (vocab, width)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.mix.", entry["mixer"]
        h = m["heads"]
        shapes[f"l{i}.norm1"] = ()
        if entry["type"] == "latent_attention":
            q, r = m["q_rank"], m["kv_rank"]
            shapes |= {p + "dq": (q, width), p + "dq.norm": (q,), p + "uq": (h * (m["dim"] + m["rot_dim"]), q),
                       p + "dkv": (r + m["rot_dim"], width), p + "dkv.norm": (r,), p + "uk": (h * m["dim"], r), p + "uv": (h * m["vdim"], r),
                       p + "g": (h, width), p + "o": (width, h * m["vdim"])}
        elif entry["type"] == "attention":
            g, d, dv = m["kv_heads"], m["dim"], m["vdim"]
            shapes |= {p + "q": (h * d, width), p + "k": (g * d, width), p + "v": (g * dv, width), p + "q.norm": (d,), p + "k.norm": (d,),
                       p + "temp": (h,), p + "r1": (h,), p + "r2": (h,), p + "o": (width, h * dv)}
        else:
            inner, shared = h * m["vdim"], 2 * m["groups"] * m["state"]
            shapes |= {p + "in": (2 * inner + shared + h, width), p + "conv": (inner + shared, m["conv"]), p + "conv.b": (inner + shared,),
                       p + "dt_bias": (h,), p + "A_log": (h,), p + "D": (h,), p + "norm": (inner,), p + "o": (width, inner)}
        mlp = entry.get("mlp")
        if mlp:
            f, router = f"l{i}.mlp.", mlp["router"]
            n = router["experts"] + (router.get("identity") or 0)
            shapes |= {f"l{i}.norm2": (), f + "router": (n, width), f + "correction": (n,)}
            units = [(f"e{e}", mlp["expert"]["ff"]) for e in range(router["experts"])]
            for name, ff in units + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                shapes |= {f"{f}{name}.gate": (ff, width), f"{f}{name}.up": (ff, width), f"{f}{name}.down": (width, ff)}
    return shapes | {"final.norm": (), "head": (vocab, width)}


class Folivik(NamedWeightsLM):
    create = "llaisysFolivikModelCreate"

    def meta_of(self, config, shapes, dtype, max_seq_len):
        return build_meta(config, dtype, max_seq_len)
