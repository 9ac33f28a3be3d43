"""Pabovik: latent attention, lightning attention and RWKV-style time mixing, one mixer per listed layer; norms stand
before and after every sublayer (layered.py has what the designs of listed layers share).
"""
from . import _native as N
from .layered import LayeredConfig, LayeredCudaState, LayeredForCausalLM


class PabovikConfig(LayeredConfig):
    """config.json of a Pabovik model."""

    DESIGN = "Pabovik"
    MIXERS = ("latent_attention", "lightning", "wkv")

    def mixer_spec(self, layer: dict, s: N.LayerSpec):
        c = layer["mixer"]
        if layer["type"] == "latent_attention":
            s.q_rank, s.kv_rank, s.rot_dim = int(c["q_rank"]), int(c["kv_rank"]), int(c["rot_dim"])
            s.rot_dims, s.rot_base = int(c["rot"]["dims"]), float(c["rot"]["base"])
            s.scale = float(c["scale"])


class PabovikCudaState(LayeredCudaState):
    """Device weights and plan of a Pabovik model."""


class PabovikForCausalLM(LayeredForCausalLM):
    """Checkpoint adapter + generate loop of a Pabovik model."""

    CONFIG = PabovikConfig
    STATE = PabovikCudaState

    def _expected_shape(self, name: str, shape: tuple) -> tuple:
        """The low rank of the time mixing's decay is a size of the checkpoint only."""
        if name.endswith(("mix.w1", "mix.w2")):
            w1 = self._weights.get(name[:-1] + "1")
            rank = -1 if w1 is None else w1.shape[0]
            return (rank, shape[1]) if name.endswith("w1") else (shape[0], rank)
        return shape
