"""Pabovik: a decoder whose config lists its layers one by one. Every layer names a mixer (latent attention, lightning
attention or RWKV-style time mixing), the mixer's sizes and an optional dense feed-forward; norms stand before and after
every sublayer. Steps, cache tables, sampling and generation are those of gemma4.py: only the configuration, the
checkpoint's tensor names and the creation of the device model differ.
"""
import ctypes as C
import os
from typing import Optional

import numpy as np

from . import _native as N
from . import synthetic
from ._native import Oxg4Error
from .gemma4 import Device, Gemma4CudaState, Gemma4ForCausalLM


class PabovikConfig:
    """config.json of a Pabovik model."""

    def __init__(self, d: dict):
        self.raw = d
        try:
            self.vocab_size = int(d["vocab"])
            self.hidden_size = int(d["width"])
            self.norm_eps = float(d["norm"]["eps"])
            self.layers = [dict(layer) for layer in d["layers"]]
        except (KeyError, TypeError) as e:
            raise Oxg4Error(1, f"invalid Pabovik configuration: {e}")
        self.num_hidden_layers = len(self.layers)
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in N.MIXERS:
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

    def native(self, weight_dtype: int):
        """oxg4_layered_config plus the arrays it points into."""
        specs = (N.LayerSpec * self.num_hidden_layers)()
        keep = [specs]
        for i, layer in enumerate(self.layers):
            c, s = layer["mixer"], specs[i]
            s.mixer = N.MIXERS[layer["type"]]
            s.heads, s.dim = int(c["heads"]), int(c["dim"])
            s.vdim = int(c.get("vdim", c["dim"]))
            s.ff = int(layer["mlp"]["ff"]) if layer.get("mlp") else 0
            j = self.weights_layer(i)
            s.weights_of = -1 if j == i else j
            if layer["type"] == "latent_attention":
                s.q_rank, s.kv_rank, s.rot_dim = int(c["q_rank"]), int(c["kv_rank"]), int(c["rot_dim"])
                s.rot_dims, s.rot_base = int(c["rot"]["dims"]), float(c["rot"]["base"])
                s.scale = float(c["scale"])
            elif layer["type"] == "lightning":
                decay = np.ascontiguousarray(c["decay"], dtype=np.float32)
                if decay.size != s.heads:
                    raise Oxg4Error(1, f"layer {i}: one decay per head is required")
                keep.append(decay)
                s.decay = decay.ctypes.data_as(C.POINTER(C.c_float))
        return N.LayeredConfig(self.vocab_size, self.hidden_size, self.num_hidden_layers, self.norm_eps, weight_dtype, specs), keep


class PabovikCudaState(Gemma4CudaState):
    """Device weights and plan of a Pabovik model."""

    def __init__(self, config: PabovikConfig, device_index: int = 0, weight_dtype: int = N.BF16):
        self.config = config
        c, self._keep = config.native(weight_dtype)
        self._h = C.c_void_p()
        self.weight_dtype = weight_dtype
        N.check(N.lib().oxg4_model_create_layered(C.byref(c), device_index, C.byref(self._h)))


class PabovikForCausalLM(Gemma4ForCausalLM):
    """Checkpoint adapter + generate loop. `weight_dtype` F32 runs a BF16 checkpoint in f32 throughout; the cached
    latents have the weights' type unless `kv_dtype` says otherwise."""

    def __init__(self, config: PabovikConfig, weights: dict, device: Device, weight_dtype: int,
                 checkpoint_directory: Optional[str] = None, kv_dtype: Optional[int] = None):
        super().__init__(config, weights, device, weight_dtype, checkpoint_directory,
                         weight_dtype if kv_dtype is None else kv_dtype)

    @classmethod
    def from_pretrained(cls, directory: str, device: Device, kv_dtype: Optional[int] = None, weight_dtype: Optional[int] = None):
        config = PabovikConfig(synthetic.read_config(directory))
        weights = synthetic.read_tensors(os.path.join(directory, "model.safetensors"))
        return cls(config, weights, device, N.BF16 if weight_dtype is None else weight_dtype, directory, kv_dtype)

    @classmethod
    def from_weights(cls, cfg: dict, weights: dict, device: Device, kv_dtype: Optional[int] = None, weight_dtype: int = N.BF16):
        return cls(PabovikConfig(cfg), weights, device, weight_dtype, None, kv_dtype)

    def _validate_checkpoint(self):
        low = {n[:-len("mix.w1")]: a.shape[0] for n, a in self._weights.items() if n.endswith("mix.w1")}
        for name, shape, _ in synthetic.layered_weight_names(self._config.to_dict()):
            if name not in self._weights:
                raise Oxg4Error(2, f"checkpoint is missing `{name}`")
            p = name[:name.find("mix.")]
            if name.endswith("mix.w1"):
                shape = (low[p], shape[1])
            elif name.endswith("mix.w2"):
                shape = (shape[0], low.get(p, -1))
            if tuple(self._weights[name].shape) != shape:
                raise Oxg4Error(1, f"tensor `{name}` has shape {tuple(self._weights[name].shape)}, expected {shape}")

    def embed(self, input_ids) -> np.ndarray:
        """CPU helper: embedding rows widened to f32."""
        ids = np.asarray(input_ids, dtype=np.int64)
        if ids.size and ids.max() >= self._config.vocab_size:
            raise Oxg4Error(2, "token id exceeds embedding vocabulary")
        e = self._weights["embed"][ids]
        return synthetic.bf16_bits_to_f32(e) if e.dtype == np.uint16 else np.asarray(e, dtype=np.float32)

    def prepare_cuda(self) -> PabovikCudaState:
        if not self._device.is_cuda():
            raise Oxg4Error(2, "Pabovik generate requires Device::Cuda")
        names = [n for n, _, _ in synthetic.layered_weight_names(self._config.to_dict())]
        return PabovikCudaState.load(self._config, [(n, self._weights[n]) for n in names], self._device.index, self._weight_dtype)
