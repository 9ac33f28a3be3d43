"""Model registry: which classes serve a checkpoint folder, by its config.json."""
from typing import Optional

from . import _native as N
from . import synthetic
from ._native import Oxg4Error
from .gemma4 import Device, Gemma4ForCausalLM
from .nozurax import NozuraxForCausalLM
from .pabovik import PabovikForCausalLM

# `architecture` (or `model_type`) of config.json -> model class
MODELS = {
    "Nozurax": NozuraxForCausalLM,
    "Pabovik": PabovikForCausalLM,
    "gemma4": Gemma4ForCausalLM,
    "gemma4_text": Gemma4ForCausalLM,
}


def model_class(config: dict):
    for key in ("architecture", "model_type"):
        if config.get(key) in MODELS:
            return MODELS[config[key]]
    raise Oxg4Error(7, f"no model for architecture `{config.get('architecture', config.get('model_type'))}`")


def load_pretrained(directory: str, device: Device, weight_dtype: Optional[int] = None, kv_dtype: Optional[int] = None):
    """The model of `directory`. `weight_dtype`: F32 runs a BF16 checkpoint in f32 throughout (None: as stored)."""
    cls = model_class(synthetic.read_config(directory))
    model = cls.from_pretrained(directory, device, kv_dtype)
    if weight_dtype is not None:
        model = cls(model.config(), model._weights, device, weight_dtype, directory,
                    kv_dtype if kv_dtype is not None else weight_dtype)
    return model
