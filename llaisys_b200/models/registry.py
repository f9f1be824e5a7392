"""Which class runs a checkpoint: chosen by its config.json."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Mapping

from .base import CausalLM
from .doderax import Doderax
from .folivik import Folivik
from .lilovik import Lilovik
from .qwen2 import Qwen2
from .vozozen import Vozozen

# architecture name (config "architecture", an entry of "architectures", or "model_type") -> class
MODELS: dict[str, type[CausalLM]] = {"qwen2": Qwen2, "Qwen2ForCausalLM": Qwen2, "Vozozen": Vozozen, "vozozen": Vozozen,
                                   "Doderax": Doderax, "doderax": Doderax, "Lilovik": Lilovik, "lilovik": Lilovik,
                                   "Folivik": Folivik, "folivik": Folivik}


def model_class(config: Mapping) -> type[CausalLM]:
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for name in names:
        if name in MODELS:
            return MODELS[name]
    raise ValueError(f"no model class for architecture {[n for n in names if n]}; known: {sorted(MODELS)}")


def load_model(model_path, device=None, **kwargs) -> CausalLM:
    """The model of a checkpoint directory (config.json + *.safetensors). device: NVIDIA if there is one, else CPU, when
    not given; other arguments as the class's constructor."""
    from ..libllaisys import DeviceType
    from ..runtime import RuntimeAPI

    config = json.loads((Path(model_path) / "config.json").read_text())
    if device is None:
        device = DeviceType.NVIDIA if RuntimeAPI(DeviceType.NVIDIA).get_device_count() > 0 else DeviceType.CPU
    return model_class(config).from_pretrained(model_path, device, **kwargs)
