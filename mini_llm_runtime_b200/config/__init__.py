from .bopilorn import BopilornConfig, BopilornLayer, bopilorn_model_spec
from .qwen2 import Qwen2Config, qwen2_model_spec
from .ratilorn import RatilornConfig, RatilornLayer, ratilorn_model_spec
from .registry import (Architecture, architecture_of, config_from_dict, known_architectures,
                       load_config, register_architecture, unregister_architecture)
from .rozesun import RozesunConfig, RozesunLayer, rozesun_model_spec
from .spec import LayerSpec, ModelSpec, PartSpec, RunStep
from .vetevik import VetevikConfig, VetevikLayer, vetevik_model_spec
from .zazasun import ZazasunConfig, ZazasunLayer, zazasun_model_spec
from .zugarax import ZugaraxConfig, ZugaraxLayer, zugarax_model_spec

__all__ = [
    "Architecture", "BopilornConfig", "BopilornLayer", "LayerSpec", "ModelSpec", "PartSpec", "Qwen2Config", "RatilornConfig", "RatilornLayer", "RozesunConfig", "RozesunLayer",
    "RunStep", "VetevikConfig", "VetevikLayer", "ZazasunConfig", "ZazasunLayer", "ZugaraxConfig", "ZugaraxLayer",
    "architecture_of", "bopilorn_model_spec", "config_from_dict", "known_architectures", "load_config",
    "qwen2_model_spec", "ratilorn_model_spec", "register_architecture", "rozesun_model_spec", "unregister_architecture", "vetevik_model_spec", "zazasun_model_spec", "zugarax_model_spec",
]
