"""B200-native token generation: the reference's Gemma4 API (gemma4.py) and models of listed layers (layered.py,
pabovik.py, nozurax.py).

The directory name carries a hyphen, so import it with
    importlib.import_module("oxide-beta_b200")
from the repository root.
"""
from . import _native, synthetic
from ._native import BF16, F32, INACTIVE, Oxg4Error, library_path
from . import models
from .gemma4 import (Device, Gemma4CudaCacheTable, Gemma4CudaState, Gemma4ForCausalLM, Gemma4TextConfig,
                     Gemma4TpCacheTable, Gemma4TpState, GenerationConfig, sample_token, sample_topk_candidates,
                     tp_shard)

from .models import MODELS, load_pretrained
from .layered import LayeredConfig, LayeredCudaState, LayeredForCausalLM
from .nozurax import NozuraxConfig, NozuraxCudaState, NozuraxForCausalLM
from .pabovik import PabovikConfig, PabovikCudaState, PabovikForCausalLM

__all__ = ["MODELS", "load_pretrained", "LayeredConfig", "LayeredCudaState", "LayeredForCausalLM", "NozuraxConfig",
           "NozuraxCudaState", "NozuraxForCausalLM", "PabovikConfig", "PabovikCudaState", "PabovikForCausalLM",
           "BF16", "F32", "INACTIVE", "Oxg4Error", "Device", "Gemma4CudaCacheTable", "Gemma4CudaState",
           "Gemma4ForCausalLM", "Gemma4TextConfig", "Gemma4TpCacheTable", "Gemma4TpState", "GenerationConfig",
           "sample_token", "sample_topk_candidates", "synthetic", "library_path", "tp_shard"]
