"""Senuvik: a decoder whose layers are attention within a window that keeps the first tokens, a state-space layer, or causal
attention beside a time-mixing layer, each followed by a gated feed-forward or a mixture of experts with a shared one.  Sublayers
read the norm of the residual; what they add is normed and scaled.

Reads the design's config.json and tensors into ``ob_layered_desc``; what runs is the library's layered model."""
from __future__ import annotations

import math

import numpy as np

from . import capi
from .layered import Describer, LayeredModel, tensor_source


def plain_frequencies(rot: dict) -> np.ndarray:
    return float(rot["base"]) ** (-2.0 * np.arange(rot["dims"] // 2) / max(rot["dims"], 1))


def linear_frequencies(rot: dict) -> np.ndarray:
    """Positions stretched by a factor."""
    return plain_frequencies(rot) / float((rot.get("scaling") or {}).get("factor", 1.0))


def yarn_frequencies(rot: dict):
    """YaRN (Peng et al., "YaRN: Efficient Context Window Extension of Large Language Models"): pairs that turn at least `fast`
    times within the original length keep their frequency, those that turn at most `slow` times are stretched, a ramp between.
    Frequencies and the factor of cos and sin."""
    f, s, n = plain_frequencies(rot), rot.get("scaling"), rot["dims"]
    if not s:
        return f, 1.0

    def pair(turns):  # the (fractional) number of the pair that turns so often
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo, hi = max(math.floor(pair(s["fast"])), 0), min(math.ceil(pair(s["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def _attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    """What both kinds share."""
    H, G = mx["heads"], mx["kv_heads"]
    if H % G:
        raise ValueError(f"{at[:-1]}: {H} heads over {G} key/value heads")
    m = capi.MixerDesc()
    m.kind, m.n_head, m.n_kv_head, m.n_map, m.dim, m.vdim = capi.MIXER_ATTENTION, H, G, 1, mx["dim"], mx["vdim"]
    m.scale, m.rot_dims, m.rot_base = mx["scale"], mx["rot"]["dims"], mx["rot"]["base"]
    m.wq = d.matrix(t.bf16(at + "q", (H * m.dim, width)))
    m.wo = d.matrix(t.bf16(at + "o", (width, H * m.vdim)))
    return m


def _rotation(d: Describer, m: capi.MixerDesc, freqs: np.ndarray, gain: float = 1.0) -> None:
    m.rot_freqs, m.rot_gain = d.doubles(freqs), gain


def _window_attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    m = _attention(d, t, at, mx, width)
    H, G, dim, vdim = m.n_head, m.n_kv_head, m.dim, m.vdim
    m.window, m.keep_first, m.rot_interleaved = mx["mask"]["size"], mx["mask"].get("keep_first", 0), 1
    _rotation(d, m, linear_frequencies(mx["rot"]))
    m.qk_norm_whole = 1
    m.q_bias, m.q_norm = d.vector(t.f32(at + "q.b", (H * dim,))), d.vector(t.f32(at + "q.norm", (H * dim,)))
    m.sink = d.vector(t.f32(at + "sink", (H,)))
    if mx.get("kv_from") is not None:
        m.kv_layer = mx["kv_from"] + 1
        return m
    m.wk, m.wv = d.matrix(t.bf16(at + "k", (G * dim, width))), d.matrix(t.bf16(at + "v", (G * vdim, width)))
    m.k_bias, m.v_bias = d.vector(t.f32(at + "k.b", (G * dim,))), d.vector(t.f32(at + "v.b", (G * vdim,)))
    m.k_norm = d.vector(t.f32(at + "k.norm", (G * dim,)))
    return m


def _capped_attention(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    m = _attention(d, t, at, mx, width)
    m.softcap = mx["softcap"]
    _rotation(d, m, *yarn_frequencies(mx["rot"]))
    m.wk, m.wv = d.matrix(t.bf16(at + "k", (m.n_kv_head * m.dim, width))), d.matrix(t.bf16(at + "v", (m.n_kv_head * m.vdim, width)))
    m.w_gate = d.matrix(t.bf16(at + "g", (m.n_head, width)))
    return m


def _state_space(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    H, V, N, G, taps = mx["heads"], mx["vdim"], mx["state"], mx["groups"], mx["conv"]
    if H % G or H * V % mx["norm_groups"]:
        raise ValueError(f"{at[:-1]}: {H} heads of {V} over {G} groups and {mx['norm_groups']} normed parts")
    inner = H * V
    channels = inner + 2 * G * N
    m = capi.MixerDesc()
    m.kind, m.n_head, m.dim, m.vdim, m.n_group, m.n_norm_group, m.conv_taps = capi.MIXER_STATE_SPACE, H, N, V, G, mx["norm_groups"], taps
    m.w_in = d.matrix(t.bf16(at + "in", (inner + channels + H, width)))
    m.conv_w, m.conv_b = d.vector(t.f32(at + "conv", (channels, taps))), d.vector(t.f32(at + "conv.b", (channels,)))
    m.dt_bias, m.a_log, m.d_skip = (d.vector(t.f32(at + n, (H,))) for n in ("dt_bias", "A_log", "D"))
    m.out_norm = d.vector(t.f32(at + "norm", (inner,)))
    m.wo = d.matrix(t.bf16(at + "o", (width, inner)))
    return m


def _time_mixing(d: Describer, t, at: str, mx: dict, width: int) -> capi.MixerDesc:
    H, dim = mx["heads"], mx["dim"]
    n = H * dim
    m = capi.MixerDesc()
    m.kind, m.n_head, m.dim, m.vdim = capi.MIXER_TIME_MIXING, H, dim, dim
    m.wq, m.wk, m.wv, m.w_gate = (d.matrix(t.bf16(at + c, (n, width))) for c in "rkvg")
    m.mu_r, m.mu_k, m.mu_v, m.mu_g, m.mu_w = (d.vector(t.f32(at + "mu." + c, (width,))) for c in "rkvgw")
    low = t.bf16(at + "w1")  # its rows are the rank of the decay
    m.w_decay1 = d.matrix(t.bf16(at + "w1", (low.shape[0], width)))
    m.w_decay2 = d.matrix(t.bf16(at + "w2", (n, low.shape[0])))
    m.decay0, m.bonus = d.vector(t.f32(at + "w0", (n,))), d.vector(t.f32(at + "u", (H, dim)))
    m.out_norm = d.vector(t.f32(at + "norm", (n,)))
    m.wo = d.matrix(t.bf16(at + "o", (width, n)))
    return m


class SenuvikModel(LayeredModel):
    """``config`` is the parsed config.json, ``tensors`` a SafetensorsFile or a dict of arrays under the file's names."""

    ARCHITECTURE = "Senuvik"

    def __init__(self, backend, config: dict, tensors, dtype: str = "bfloat16", max_seq_len: int = 4096, max_batch_tokens: int = 512,
                 kv_pool_tokens: int = 0, state_slots: int = 0):
        t = tensor_source(tensors)
        d, width, vocab = Describer(), config["width"], config["vocab"]
        blocks = [self._block(d, t, i, layer, width) for i, layer in enumerate(config["layers"])]
        desc = capi.LayeredDesc()
        desc.n_vocab, desc.n_embd, desc.n_layer = vocab, width, len(blocks)
        desc.rms_eps, desc.residual_mult = config["norm"]["eps"], 1.0
        desc.final_norm, desc.final_gain = d.vector(t.f32("final.norm", (width,))), 1.0
        self.size(desc, dtype, max_seq_len, max_batch_tokens, kv_pool_tokens, state_slots)
        desc.token_embd = d.matrix(t.bf16("embed", (vocab, width)))
        desc.output = d.matrix(t.bf16("head", (vocab, width)))
        super().__init__(backend, desc, blocks)
        self.config = config

    @classmethod
    def _block(cls, d: Describer, t, i: int, layer: dict, width: int) -> capi.BlockDesc:
        at, mx, b = f"l{i}.", layer["mixer"], capi.BlockDesc()

        def added(norm: str, scale: str) -> int:  # factors of what a sublayer adds: its norm's and the layer scale
            return d.vector(t.f32(at + norm, (width,)) * t.f32(at + scale, (width,)))

        if layer["type"] == "attention":
            b.mixer = _window_attention(d, t, at + "mix.", mx, width)
        elif layer["type"] == "mamba2":
            b.mixer = _state_space(d, t, at + "mix.", mx, width)
        elif layer["type"] == "parallel":
            b.mixer, b.mixer_scale = _capped_attention(d, t, at + "mix.left.", mx["left"], width), mx["left_scale"]
            b.mixer2, b.mixer2_scale = _time_mixing(d, t, at + "mix.right.", mx["right"], width), mx["right_scale"]
        else:
            raise ValueError(f"layer {i}: no mixer {layer['type']}")
        b.pre_norm1, b.post_norm1 = d.vector(t.f32(at + "norm1", (width,))), added("norm1b", "ls1")
        mlp = layer.get("mlp")
        if mlp is not None:
            b.pre_norm2, b.post_norm2 = d.vector(t.f32(at + "norm2", (width,))), added("norm2b", "ls2")
            cls._feed_forward(b, d, t, i, at + "mlp.", mlp, width)
        return b

    @staticmethod
    def _feed_forward(b: capi.BlockDesc, d: Describer, t, i: int, at: str, mlp: dict, width: int) -> None:
        def part(prefix: str, ff: int):
            return [d.matrix(t.bf16(at + prefix + name, shape)) for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))]

        if mlp["kind"] == "dense":
            b.ff_kind, b.n_ff = capi.FF_GELU_GLU, mlp["ff"]
            b.w_gate, b.w_up, b.w_down = part("", b.n_ff)
        elif mlp["kind"] == "moe":
            n, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            if not 1 <= mlp["router"]["top"] <= n:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {n} experts")
            b.ff_kind, b.n_ff, b.n_expert, b.n_expert_used, b.router_softmax = capi.FF_EXPERTS, ff, n, mlp["router"]["top"], 1
            b.w_router = d.matrix(t.bf16(at + "router", (n, width)))
            b.expert_gate, b.expert_up, b.expert_down = (
                d.matrices(t.bf16(f"{at}e{e}.{name}", shape) for e in range(n))
                for name, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))
            if mlp.get("shared"):
                b.shared_ff = mlp["shared"]["ff"]
                b.shared_gate, b.shared_up, b.shared_down = part("shared.", b.shared_ff)
                b.w_shared_scale = d.matrix(t.bf16(at + "shared.sg", (1, width)))
        else:
            raise ValueError(f"layer {i}: no feed-forward {mlp['kind']}")
