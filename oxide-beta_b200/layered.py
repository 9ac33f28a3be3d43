"""Models whose config.json lists the layers one by one: what the designs share. Every layer names a mixer, the mixer's
sizes and an optional gated feed-forward, and may use the tensors of another layer. Steps, cache tables, sampling and
generation are those of gemma4.py; a design adds its mixers, its block (how mixer and feed-forward meet the residual
stream) and its tensor names (synthetic.layered_weight_names).
"""
import ctypes as C
import os
from typing import Optional

import numpy as np

from . import _native as N
from . import synthetic
from ._native import Oxg4Error
from .gemma4 import Device, Gemma4CudaState, Gemma4ForCausalLM


class LayeredConfig:
    """config.json of a model of listed layers."""

    DESIGN = ""                  # `architecture` of config.json
    MIXERS = ()
    BLOCK = N.BLOCK_SANDWICH
    ACT = "silu"                 # of the feed-forward's gate
    NORM_WEIGHT_OFFSET = 0       # 1: the weights of the block and final norms are stored around zero

    def __init__(self, d: dict):
        self.raw = d
        try:
            self.vocab_size = int(d["vocab"])
            self.hidden_size = int(d["width"])
            self.norm_eps = float(d["norm"]["eps"])
            self.layers = [dict(layer) for layer in d["layers"]]
        except (KeyError, TypeError) as e:
            raise Oxg4Error(1, f"invalid {self.DESIGN} configuration: {e}")
        self.num_hidden_layers = len(self.layers)
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in self.MIXERS:
                raise Oxg4Error(7, f"layer {i}: unknown mixer `{layer.get('type')}`")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise Oxg4Error(7, f"layer {i}: unknown feed-forward `{mlp['kind']}`")

    def to_dict(self) -> dict:
        return self.raw

    def weights_layer(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        for _ in range(self.num_hidden_layers):
            j = self.layers[i].get("weights_of")
            if j is None:
                return i
            if not 0 <= j < self.num_hidden_layers:
                break
            i = j
        raise Oxg4Error(2, f"layer {i}: invalid weights_of")

    def mixer_spec(self, layer: dict, s: N.LayerSpec):
        """Fills in what only this layer's mixer has, beyond heads, sizes and decays."""

    def native(self, weight_dtype: int):
        """oxg4_layered_config plus the arrays it points into."""
        specs = (N.LayerSpec * self.num_hidden_layers)()
        keep = [specs]
        for i, layer in enumerate(self.layers):
            c, s = layer["mixer"], specs[i]
            s.mixer = N.MIXERS[layer["type"]]
            try:
                s.heads, s.dim = int(c["heads"]), int(c["dim"])
                s.vdim = int(c.get("vdim", c["dim"]))
                s.ff = int(layer["mlp"]["ff"]) if layer.get("mlp") else 0
                self.mixer_spec(layer, s)
            except (KeyError, TypeError) as e:
                raise Oxg4Error(1, f"layer {i}: invalid {self.DESIGN} configuration: {e}")
            j = self.weights_layer(i)
            s.weights_of = -1 if j == i else j
            if "decay" in c:
                decay = np.ascontiguousarray(c["decay"], dtype=np.float32)
                if decay.size != s.heads:
                    raise Oxg4Error(1, f"layer {i}: one decay per head is required")
                keep.append(decay)
                s.decay = decay.ctypes.data_as(C.POINTER(C.c_float))
        return N.LayeredConfig(self.vocab_size, self.hidden_size, self.num_hidden_layers, self.norm_eps, weight_dtype, self.BLOCK,
                               N.ACTIVATIONS[self.ACT], self.NORM_WEIGHT_OFFSET, specs), keep


class LayeredCudaState(Gemma4CudaState):
    """Device weights and plan of a model of listed layers."""

    def __init__(self, config: LayeredConfig, device_index: int = 0, weight_dtype: int = N.BF16):
        self.config = config
        c, self._keep = config.native(weight_dtype)
        self._h = C.c_void_p()
        self.weight_dtype = weight_dtype
        N.check(N.lib().oxg4_model_create_layered(C.byref(c), device_index, C.byref(self._h)))


class LayeredForCausalLM(Gemma4ForCausalLM):
    """Checkpoint adapter + generate loop. `weight_dtype` F32 runs a BF16 checkpoint in f32 throughout; the cache has the
    weights' type unless `kv_dtype` says otherwise."""

    CONFIG = LayeredConfig
    STATE = LayeredCudaState

    def __init__(self, config: LayeredConfig, weights: dict, device: Device, weight_dtype: int,
                 checkpoint_directory: Optional[str] = None, kv_dtype: Optional[int] = None):
        super().__init__(config, weights, device, weight_dtype, checkpoint_directory,
                         weight_dtype if kv_dtype is None else kv_dtype)

    @classmethod
    def from_pretrained(cls, directory: str, device: Device, kv_dtype: Optional[int] = None, weight_dtype: Optional[int] = None):
        config = cls.CONFIG(synthetic.read_config(directory))
        weights = synthetic.read_tensors(os.path.join(directory, "model.safetensors"))
        return cls(config, weights, device, N.BF16 if weight_dtype is None else weight_dtype, directory, kv_dtype)

    @classmethod
    def from_weights(cls, cfg: dict, weights: dict, device: Device, kv_dtype: Optional[int] = None, weight_dtype: int = N.BF16):
        return cls(cls.CONFIG(cfg), weights, device, weight_dtype, None, kv_dtype)

    def _expected_shape(self, name: str, shape: tuple) -> tuple:
        """Shape of a tensor; a design whose checkpoint alone names a size reads it from there."""
        return shape

    def _validate_checkpoint(self):
        for name, shape, _ in synthetic.layered_weight_names(self._config.to_dict()):
            if name not in self._weights:
                raise Oxg4Error(2, f"checkpoint is missing `{name}`")
            shape = self._expected_shape(name, shape)
            if tuple(self._weights[name].shape) != shape:
                raise Oxg4Error(1, f"tensor `{name}` has shape {tuple(self._weights[name].shape)}, expected {shape}")

    def embed(self, input_ids) -> np.ndarray:
        """CPU helper: embedding rows widened to f32."""
        ids = np.asarray(input_ids, dtype=np.int64)
        if ids.size and ids.max() >= self._config.vocab_size:
            raise Oxg4Error(2, "token id exceeds embedding vocabulary")
        e = self._weights["embed"][ids]
        return synthetic.bf16_bits_to_f32(e) if e.dtype == np.uint16 else np.asarray(e, dtype=np.float32)

    def prepare_cuda(self) -> LayeredCudaState:
        if not self._device.is_cuda():
            raise Oxg4Error(2, f"{self._config.DESIGN} generate requires Device::Cuda")
        names = [n for n, _, _ in synthetic.layered_weight_names(self._config.to_dict())]
        return self.STATE.load(self._config, [(n, self._weights[n]) for n in names], self._device.index, self._weight_dtype)
