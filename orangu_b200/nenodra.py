"""Nenodra: a decoder whose layers attend within sliding windows -- differential attention with biases, or gated attention whose
values are its keys -- followed by a feed-forward with a squared relu or a mixture of experts that scales an expert's input.
Sublayers read the residual itself; what they add is normed.

Reads the design's config.json and tensors into ``ob_layered_desc``; what runs is the library's layered model."""
from __future__ import annotations

import numpy as np

from . import capi
from .layered import Describer, LayeredModel, tensor_source


def _attention(d: Describer, t, at: str, mx: dict, width: int, maps: int) -> capi.MixerDesc:
    """What both kinds share: grouped heads, query and key norms, rotation of halves, window."""
    H, G, dim, rot = mx["heads"], mx["kv_heads"], mx["dim"], mx["rot"]
    if H % G:
        raise ValueError(f"{at[:-1]}: {H} heads over {G} key/value heads")
    m = capi.MixerDesc()
    m.kind, m.n_head, m.n_kv_head, m.n_map, m.dim, m.vdim = capi.MIXER_ATTENTION, H, G, maps, dim, mx["vdim"]
    m.window, m.scale = mx["mask"]["size"], mx["scale"]
    m.rot_dims, m.rot_interleaved, m.rot_base = rot["dims"], 0, rot["base"]
    m.wq = d.matrix(t.bf16(at + "q", (H * maps * dim, width)))
    m.wk = d.matrix(t.bf16(at + "k", (G * maps * dim, width)))
    m.q_norm, m.k_norm = d.vector(t.f32(at + "q.norm", (dim,))), d.vector(t.f32(at + "k.norm", (dim,)))
    m.wo = d.matrix(t.bf16(at + "o", (width, H * mx["vdim"])))
    return m


def _differential_attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    H, G, dim, vdim, diff = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["diff"]
    m = _attention(d, t, at, mx, width, 2)
    m.wv = d.matrix(t.bf16(at + "v", (G * vdim, width)))
    m.q_bias, m.k_bias = d.vector(t.f32(at + "q.b", (H * 2 * dim,))), d.vector(t.f32(at + "k.b", (G * 2 * dim,)))
    m.v_bias, m.o_bias = d.vector(t.f32(at + "v.b", (G * vdim,))), d.vector(t.f32(at + "o.b", (width,)))
    lq1, lk1, lq2, lk2 = (t.f32(at + n, (dim,)).astype(np.float64) for n in ("lq1", "lk1", "lq2", "lk2"))
    m.map_weight, m.head_gain = float(np.exp(lq1 @ lk1) - np.exp(lq2 @ lk2) + diff), 1.0 - diff
    return m


def _gated_attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    if mx["vdim"] != mx["dim"]:
        raise ValueError(f"{at[:-1]}: keys of {mx['dim']} cannot be values of {mx['vdim']}")
    m = _attention(d, t, at, mx, width, 1)
    m.w_gate = d.matrix(t.bf16(at + "g", (mx["heads"] * mx["vdim"], width)))
    return m


MIXERS = {"attention": _differential_attention, "attention_2": _gated_attention}


class NenodraModel(LayeredModel):
    """``config`` is the parsed config.json, ``tensors`` a SafetensorsFile or a dict of arrays under the file's names."""

    ARCHITECTURE = "Nenodra"

    def __init__(self, backend, config: dict, tensors, dtype: str = "bfloat16", max_seq_len: int = 4096, max_batch_tokens: int = 512,
                 kv_pool_tokens: int = 0, state_slots: int = 0):
        t = tensor_source(tensors)
        d, width, vocab = Describer(), config["width"], config["vocab"]
        blocks = [self._block(d, t, i, layer, width) for i, layer in enumerate(config["layers"])]
        desc = capi.LayeredDesc()
        desc.n_vocab, desc.n_embd, desc.n_layer = vocab, width, len(blocks)
        desc.rms_eps, desc.residual_mult = config["norm"]["eps"], config["residual_mult"]
        desc.final_norm, desc.final_gain = self._gain(d, t, "final.norm", width), config["logit_scale"]  # the scale goes through the head
        self.size(desc, dtype, max_seq_len, max_batch_tokens, kv_pool_tokens, state_slots)
        desc.token_embd = d.matrix(t.bf16("embed", (vocab, width)))
        desc.output = d.matrix(t.bf16("head", (vocab, width)))
        super().__init__(backend, desc, blocks)
        self.config = config

    @staticmethod
    def _gain(d: Describer, t, name: str, width: int) -> int:
        return d.vector(1.0 + t.f32(name, (width,)))  # stored around zero

    @classmethod
    def _block(cls, d: Describer, t, i: int, layer: dict, width: int) -> capi.BlockDesc:
        if layer["type"] not in MIXERS:
            raise ValueError(f"layer {i}: no mixer {layer['type']}")
        at, b = f"l{i}.", capi.BlockDesc()
        b.mixer = MIXERS[layer["type"]](d, t, at + "mix.", layer["mixer"], width)
        b.post_norm1 = cls._gain(d, t, at + "norm1", width)
        mlp = layer.get("mlp")
        if mlp is None:
            return b
        b.post_norm2 = cls._gain(d, t, at + "norm2", width)
        if mlp["kind"] == "dense":
            b.ff_kind, b.n_ff = capi.FF_RELU2, mlp["ff"]
            b.w_up = d.matrix(t.bf16(at + "mlp.up", (b.n_ff, width)))
            b.w_down = d.matrix(t.bf16(at + "mlp.down", (width, b.n_ff)))
        elif mlp["kind"] == "moe":
            n, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            if not 1 <= mlp["router"]["top"] <= n:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {n} experts")
            b.ff_kind, b.n_ff, b.n_expert, b.n_expert_used = capi.FF_EXPERTS, ff, n, mlp["router"]["top"]
            b.w_router = d.matrix(t.bf16(at + "mlp.router", (n, width)))
            b.expert_gate, b.expert_up, b.expert_down = (
                d.matrices(t.bf16(f"{at}mlp.e{e}.{name}", shape) for e in range(n))
                for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))
        else:
            raise ValueError(f"layer {i}: no feed-forward {mlp['kind']}")
        return b
