"""Filorax: a decoder whose layers are latent attention in three forms (within a window without positions, with or without sink and
output gate; causal with a rotated key part), each followed by a mixture of experts in groups with a shared one.  A sublayer reads
the residual normed in groups plus a short convolution of it over time; a layer's result is averaged with those of the layers before.

Reads the design's config.json and tensors into ``ob_layered_desc``; what runs is the library's layered model."""
from __future__ import annotations

from typing import NamedTuple

from . import capi
from .layered import Describer, LayeredModel, tensor_source


class Form(NamedTuple):
    rotated: bool  # a rotated key part and no window, else a window and no positions
    sink: bool
    gated: bool


MIXERS = {
    "latent_attention": Form(rotated=False, sink=True, gated=True),
    "latent_attention_2": Form(rotated=True, sink=True, gated=True),
    "latent_attention_3": Form(rotated=False, sink=False, gated=False),
}


def _latent_attention(d: Describer, t, at: str, mx: dict, width: int, form: Form) -> capi.MixerDesc:
    H, dim, vdim, rank = mx["heads"], mx["dim"], mx["vdim"], mx["kv_rank"]
    rot = mx["rot_dim"] if form.rotated else 0
    m = capi.MixerDesc()
    m.kind, m.n_head, m.dim, m.vdim, m.rot_dim, m.kv_rank = capi.MIXER_LATENT_ATTENTION, H, dim, vdim, rot, rank
    m.scale = mx["scale"]
    if form.rotated:
        m.rot_dims, m.rot_interleaved, m.rot_base = mx["rot"]["dims"], 0, mx["rot"]["base"]
    else:
        m.window = mx["mask"]["size"]
    m.wq = d.matrix(t.bf16(at + "q", (H * (dim + rot), width)))
    m.w_dkv = d.matrix(t.bf16(at + "dkv", (rank + rot, width)))
    m.kv_norm = d.vector(t.f32(at + "dkv.norm", (rank,)))
    m.w_uk = d.matrix(t.bf16(at + "uk", (H * dim, rank)))
    m.w_uv = d.matrix(t.bf16(at + "uv", (H * vdim, rank)))
    if form.sink:
        m.sink = d.vector(t.f32(at + "sink", (H,)))
    if form.gated:
        m.w_gate = d.matrix(t.bf16(at + "g", (H * vdim, width)))
    m.wo = d.matrix(t.bf16(at + "o", (width, H * vdim)))
    return m


class FiloraxModel(LayeredModel):
    """``config`` is the parsed config.json, ``tensors`` a SafetensorsFile or a dict of arrays under the file's names."""

    ARCHITECTURE = "Filorax"

    def __init__(self, backend, config: dict, tensors, dtype: str = "bfloat16", max_seq_len: int = 4096, max_batch_tokens: int = 512,
                 kv_pool_tokens: int = 0, state_slots: int = 0):
        t = tensor_source(tensors)
        d, width, vocab, taps = Describer(), config["width"], config["vocab"], config["canon"]["taps"]
        if width % config["norm"]["groups"]:
            raise ValueError(f"{config['norm']['groups']} norm groups do not divide a width of {width}")
        blocks = [self._block(d, t, i, layer, width, taps) for i, layer in enumerate(config["layers"])]
        desc = capi.LayeredDesc()
        desc.n_vocab, desc.n_embd, desc.n_layer = vocab, width, len(blocks)
        desc.rms_eps, desc.residual_mult = config["norm"]["eps"], config["residual_mult"]
        desc.norm_groups, desc.conv_taps = config["norm"]["groups"], taps
        desc.final_norm, desc.final_gain = d.vector(t.f32("final.norm", (width,))), 1.0
        self.size(desc, dtype, max_seq_len, max_batch_tokens, kv_pool_tokens, state_slots)
        desc.token_embd = d.matrix(t.bf16("embed", (vocab, width)))
        desc.output = d.matrix(t.bf16("head", (vocab, width)))
        super().__init__(backend, desc, blocks)
        self.config = config

    @classmethod
    def _block(cls, d: Describer, t, i: int, layer: dict, width: int, taps: int) -> capi.BlockDesc:
        if layer["type"] not in MIXERS:
            raise ValueError(f"layer {i}: no mixer {layer['type']}")
        at, b = f"l{i}.", capi.BlockDesc()
        b.mixer = _latent_attention(d, t, at + "mix.", layer["mixer"], width, MIXERS[layer["type"]])
        b.pre_norm1, b.conv1 = d.vector(t.f32(at + "norm1", (width,))), d.vector(t.f32(at + "canon1", (width, taps)))
        b.depth = d.vector(t.f32(at + "dwa", (i + 2,)))
        mlp = layer.get("mlp")
        if mlp is not None:
            b.pre_norm2, b.conv2 = d.vector(t.f32(at + "norm2", (width,))), d.vector(t.f32(at + "canon2", (width, taps)))
            cls._feed_forward(b, d, t, i, at + "mlp.", mlp, width)
        return b

    @staticmethod
    def _feed_forward(b: capi.BlockDesc, d: Describer, t, i: int, at: str, mlp: dict, width: int) -> None:
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {i}: no feed-forward {mlp['kind']}")
        router, ff = mlp["router"], mlp["expert"]["ff"]
        n, top, groups = router["experts"], router["top"], router.get("groups") or {"count": 1, "keep": 1}
        if n % groups["count"] or not 1 <= groups["keep"] <= groups["count"]:
            raise ValueError(f"layer {i}: {groups['keep']} of {groups['count']} groups of {n} experts")
        if not 1 <= top <= n // groups["count"] * groups["keep"]:
            raise ValueError(f"layer {i}: {top} experts of {groups['keep']} groups of {n // groups['count']}")
        b.ff_kind, b.n_ff, b.n_expert, b.n_expert_used = capi.FF_EXPERTS, ff, n, top
        b.router_softmax, b.router_scale = capi.ROUTER_SOFTMAX_ALL, router["scale"]
        b.n_expert_group, b.n_group_used = groups["count"], groups["keep"]
        b.w_router = d.matrix(t.bf16(at + "router", (n, width)))
        b.expert_gate, b.expert_up, b.expert_down = (
            d.matrices(t.bf16(f"{at}e{e}.{name}", shape) for e in range(n))
            for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))
        if mlp.get("shared"):
            s = b.shared_ff = mlp["shared"]["ff"]
            b.shared_gate, b.shared_up, b.shared_down = (
                d.matrix(t.bf16(f"{at}shared.{name}", shape)) for name, shape in (("gate", (s, width)), ("up", (s, width)), ("down", (width, s))))
            b.w_shared_scale = d.matrix(t.bf16(at + "shared.sg", (1, width)))
