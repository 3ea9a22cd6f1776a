"""Fenipel: a decoder whose layers are latent attention within a sliding window or retention, each in parallel with a clamped
gated feed-forward, followed by a per-layer token input; norms of the residual have a single number as gain.

Reads the design's config.json and tensors into ``ob_layered_desc``; what runs is the library's layered model."""
from __future__ import annotations

from . import capi
from .layered import Describer, LayeredModel, tensor_source

GLU_ALPHA = 1.702  # slope of the sigmoid in the feed-forward's gate, fixed by the design


def _latent_attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    H, dim, rot, vdim, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    m = capi.MixerDesc()
    m.kind, m.n_head, m.dim, m.vdim, m.rot_dim, m.kv_rank = capi.MIXER_LATENT_ATTENTION, H, dim, vdim, rot, rank
    m.window, m.scale = mx["mask"]["size"], mx["scale"]
    m.rot_dims, m.rot_interleaved, m.rot_base = mx["rot"]["dims"], 1, mx["rot"]["base"]
    m.wq = d.matrix(t.bf16(at + "q", (H * (dim + rot), width)))
    m.w_dkv = d.matrix(t.bf16(at + "dkv", (rank + rot, width)))
    m.kv_norm = d.vector(t.f32(at + "dkv.norm", (rank,)))
    m.w_uk = d.matrix(t.bf16(at + "uk", (H * dim, rank)))
    m.w_uv = d.matrix(t.bf16(at + "uv", (H * vdim, rank)))
    m.w_gate = d.matrix(t.bf16(at + "g", (H, width)))
    m.wo = d.matrix(t.bf16(at + "o", (width, H * vdim)))
    return m


def _retention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    H, dim, vdim = mx["heads"], mx["dim"], mx["vdim"]
    if len(mx["decay"]) != H:
        raise ValueError(f"{at}decay names {len(mx['decay'])} heads of {H}")
    m = capi.MixerDesc()
    m.kind, m.n_head, m.dim, m.vdim = capi.MIXER_RETENTION, H, dim, vdim
    m.rot_dims, m.rot_interleaved, m.rot_base = mx["rot"]["dims"], 0, mx["rot"]["base"]
    m.decay = d.vector(mx["decay"])
    m.wq = d.matrix(t.bf16(at + "q", (H * dim, width)))
    m.wk = d.matrix(t.bf16(at + "k", (H * dim, width)))
    m.wv = d.matrix(t.bf16(at + "v", (H * vdim, width)))
    m.w_gate = d.matrix(t.bf16(at + "g", (H * vdim, width)))
    m.wo = d.matrix(t.bf16(at + "o", (width, H * vdim)))
    return m


MIXERS = {"latent_attention": _latent_attention, "retention": _retention}


class FenipelModel(LayeredModel):
    """``config`` is the parsed config.json, ``tensors`` a SafetensorsFile or a dict of arrays under the file's names.
    ``dtype``: "bfloat16" (activations and cache; accumulation and everything the design wants in 32 bits is fp32) or "float32"."""

    ARCHITECTURE = "Fenipel"

    def __init__(self, backend, config: dict, tensors, dtype: str = "bfloat16", max_seq_len: int = 4096, max_batch_tokens: int = 512,
                 kv_pool_tokens: int = 0, state_slots: int = 0):
        t = tensor_source(tensors)
        d, width, vocab = Describer(), config["width"], config["vocab"]
        side = config.get("token_side")
        side_dim = side["dim"] if side else 0
        blocks = [self._block(d, t, i, layer, width, side_dim) for i, layer in enumerate(config["layers"])]
        desc = capi.LayeredDesc()
        desc.n_vocab, desc.n_embd, desc.n_layer, desc.side_dim = vocab, width, len(blocks), side_dim
        desc.rms_eps, desc.final_gain = config["norm"]["eps"], float(t.f32("final.norm", ()).reshape(()))
        self.size(desc, dtype, max_seq_len, max_batch_tokens, kv_pool_tokens, state_slots)
        desc.token_embd = d.matrix(t.bf16("embed", (vocab, width)))
        desc.output = d.matrix(t.bf16("head", (vocab, width)))
        if side_dim:
            desc.side_embd = d.matrix(t.bf16("side.embed", (vocab, len(blocks) * side_dim)))
        super().__init__(backend, desc, blocks)
        self.config = config

    @staticmethod
    def _block(d: Describer, t, i: int, layer: dict, width: int, side_dim: int) -> capi.BlockDesc:
        if layer["type"] not in MIXERS:
            raise ValueError(f"layer {i}: no mixer {layer['type']}")
        at, b = f"l{i}.", capi.BlockDesc()
        b.norm_gain = float(t.f32(at + "norm1", ()).reshape(()))
        b.mixer = MIXERS[layer["type"]](d, t, at + "mix.", layer["mixer"], width)
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: no feed-forward {mlp['kind']}")
            ff = mlp["ff"]
            b.n_ff, b.glu_limit, b.glu_alpha = ff, mlp["limit"], GLU_ALPHA
            b.w_gate = d.matrix(t.bf16(at + "mlp.gate", (ff, width)))
            b.w_up = d.matrix(t.bf16(at + "mlp.up", (ff, width)))
            b.w_down = d.matrix(t.bf16(at + "mlp.down", (width, ff)))
        if side_dim:
            b.side_gate = d.matrix(t.bf16(at + "side.gate", (side_dim, width)))
            b.side_proj = d.matrix(t.bf16(at + "side.proj", (width, side_dim)))
            b.side_norm = d.vector(t.f32(at + "side.norm", (width,)))
        return b
