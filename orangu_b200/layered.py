"""Models given as a list of layers (``ob_layered_desc``), each layer with its own token mixer.  A design's reader (fenipel.py,
nenodra.py, senuvik.py, filorax.py) turns its configuration and tensors into blocks; this class owns the description and the handle."""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

from . import capi
from .model import DeviceModel
from .safetensors import SafetensorsFile, from_bf16, to_bf16


class Describer:
    """Fills C descriptions and keeps the arrays they point to alive until the model has been made."""

    def __init__(self):
        self.keep = []

    def matrix(self, bits: np.ndarray) -> capi.MatrixDesc:
        a = np.ascontiguousarray(bits, np.uint16)
        self.keep.append(a)
        return capi.MatrixDesc(a.ctypes.data, capi.TYPE_BF16, a.shape[1], a.shape[0])

    def matrices(self, items):
        each = [self.matrix(bits) for bits in items]
        arr = (capi.MatrixDesc * len(each))(*each)
        self.keep.append(arr)
        return arr

    def doubles(self, v) -> int:
        a = np.ascontiguousarray(v, np.float64)
        self.keep.append(a)
        return a.ctypes.data

    def vector(self, v) -> int:
        a = np.ascontiguousarray(v, np.float32)
        self.keep.append(a)
        return a.ctypes.data


class TensorDict:
    """The reader's interface over a dict: uint16 arrays are bfloat16 bits, other arrays floats."""

    def __init__(self, tensors: dict):
        self._t = tensors

    def _get(self, name, shape):
        if name not in self._t:
            raise ValueError(f"no tensor {name}")
        a = np.asarray(self._t[name])
        if shape is not None and a.shape != tuple(shape):
            raise ValueError(f"{name} is {list(a.shape)}, expected {list(shape)}")
        return a

    def bf16(self, name, shape=None):
        a = self._get(name, shape)
        return a if a.dtype == np.uint16 else to_bf16(a)

    def f32(self, name, shape=None):
        a = self._get(name, shape)
        return from_bf16(a) if a.dtype == np.uint16 else np.array(a, np.float32, order="C")


def tensor_source(tensors):
    return TensorDict(tensors) if isinstance(tensors, dict) else tensors


class LayeredModel(DeviceModel):
    """``dtype``: "bfloat16" (activations and cache; accumulation and everything a design wants in 32 bits is fp32) or "float32"."""

    @classmethod
    def from_folder(cls, backend, path: str, **sizing):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        return cls(backend, config, SafetensorsFile(os.path.join(path, "model.safetensors")), **sizing)

    @staticmethod
    def size(desc: capi.LayeredDesc, dtype: str, max_seq_len: int, max_batch_tokens: int, kv_pool_tokens: int, state_slots: int) -> None:
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype}: bfloat16 or float32")
        desc.compute_f32 = dtype == "float32"
        desc.max_seq_len, desc.max_batch_tokens, desc.kv_pool_tokens, desc.n_state_slots = max_seq_len, max_batch_tokens, kv_pool_tokens, state_slots

    def __init__(self, backend, desc: capi.LayeredDesc, blocks):
        self.backend, self._lib = backend, backend._lib
        self._mixers = [b.mixer for b in blocks]
        self._states = [b.mixer2 if b.mixer2.kind and b.mixer.kind == capi.MIXER_ATTENTION else b.mixer for b in blocks]
        self._inputs = [(1 + (b.n_ff > 0), max(desc.conv_taps, 1) - 1, desc.n_embd) for b in blocks]
        arr = (capi.BlockDesc * len(blocks))(*blocks)
        desc.layers = arr
        self._h = C.c_void_p()
        capi.check(backend._h, self._lib.ob_layered_model_create(backend._h, C.byref(desc), C.byref(self._h)))
        self.cfg = {"n_vocab": desc.n_vocab, "n_embd": desc.n_embd, "n_layer": desc.n_layer}
        self.n_vocab, self.max_batch_tokens = desc.n_vocab, desc.max_batch_tokens

    def cache_widths(self, layer: int):
        m = self._mixers[layer]
        if m.kind == capi.MIXER_ATTENTION:
            return m.n_kv_head * m.n_map * m.dim, m.n_kv_head * m.vdim
        return m.kv_rank, m.rot_dim

    def state_shape(self, layer: int):
        m = self._states[layer]
        if m.kind in (capi.MIXER_ATTENTION, capi.MIXER_LATENT_ATTENTION):
            return self._inputs[layer]  # last inputs of the sublayers' convolutions, the oldest first
        return m.n_head, m.dim, m.vdim
