"""Nozurax: retention (linear attention with a fixed decay per head and rotated queries and keys) and grouped-query attention
without rotation (whole-projection query and key norms, a query factor that grows with the logarithm of the position, a
learned sink), one mixer per listed layer. Mixer and feed-forward run in parallel behind one norm whose weight is stored
around zero (layered.py has what the designs of listed layers share).
"""
from . import _native as N
from ._native import Oxg4Error
from .layered import LayeredConfig, LayeredCudaState, LayeredForCausalLM


class NozuraxConfig(LayeredConfig):
    """config.json of a Nozurax model."""

    DESIGN = "Nozurax"
    MIXERS = ("retention", "attention")
    BLOCK = N.BLOCK_PARALLEL
    ACT = "relu"
    NORM_WEIGHT_OFFSET = 1

    def mixer_spec(self, layer: dict, s: N.LayerSpec):
        c = layer["mixer"]
        if layer["type"] == "retention":
            s.rot_dims, s.rot_base = int(c["rot"]["dims"]), float(c["rot"]["base"])
            c["decay"]                       # required
        else:
            s.kv_heads, s.scale = int(c["kv_heads"]), float(c["scale"])
            s.q_temp_coef, s.q_temp_every = float(c["q_temp"]["coef"]), int(c["q_temp"]["every"])
            if s.q_temp_every != c["q_temp"]["every"]:
                raise Oxg4Error(1, "q_temp.every must be a whole number of positions")


class NozuraxCudaState(LayeredCudaState):
    """Device weights and plan of a Nozurax model."""


class NozuraxForCausalLM(LayeredForCausalLM):
    """Checkpoint adapter + generate loop of a Nozurax model."""

    CONFIG = NozuraxConfig
    STATE = NozuraxCudaState
