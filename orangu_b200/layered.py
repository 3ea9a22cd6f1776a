"""Models given as a list of layers (``ob_layered_desc``), each layer with its own token mixer.  A design's reader (fenipel.py)
turns its configuration and tensors into blocks; this class owns the description and the handle."""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import capi
from .model import DeviceModel


class Describer:
    """Fills C descriptions and keeps the arrays they point to alive until the model has been made."""

    def __init__(self):
        self.keep = []

    def matrix(self, bits: np.ndarray) -> capi.MatrixDesc:
        a = np.ascontiguousarray(bits, np.uint16)
        self.keep.append(a)
        return capi.MatrixDesc(a.ctypes.data, capi.TYPE_BF16, a.shape[1], a.shape[0])

    def vector(self, v) -> int:
        a = np.ascontiguousarray(v, np.float32)
        self.keep.append(a)
        return a.ctypes.data


class LayeredModel(DeviceModel):
    def __init__(self, backend, desc: capi.LayeredDesc, blocks):
        self.backend, self._lib = backend, backend._lib
        self._mixers = [(b.mixer.kind, b.mixer.n_head, b.mixer.dim, b.mixer.vdim, b.mixer.kv_rank, b.mixer.rot_dim) for b in blocks]
        arr = (capi.BlockDesc * len(blocks))(*blocks)
        desc.layers = arr
        self._h = C.c_void_p()
        capi.check(backend._h, self._lib.ob_layered_model_create(backend._h, C.byref(desc), C.byref(self._h)))
        self.cfg = {"n_vocab": desc.n_vocab, "n_embd": desc.n_embd, "n_layer": desc.n_layer}
        self.n_vocab, self.max_batch_tokens = desc.n_vocab, desc.max_batch_tokens

    def cache_widths(self, layer: int):
        return self._mixers[layer][4], self._mixers[layer][5]

    def state_shape(self, layer: int):
        return self._mixers[layer][1:4]
