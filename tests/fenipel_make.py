"""Small Fenipel configurations with random weights for the tests."""
import numpy as np


def latent(heads=3, dim=24, rot_dim=16, vdim=20, kv_rank=40, window=11, base=3000.0, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
        "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def retention(heads=3, dim=24, vdim=36, rot_dims=16, base=7000.0, decay=None):
    return {"type": "retention", "mixer": {
        "heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
        "decay": [float(1.0 - 2.0 ** -(3 + 2 * h)) for h in range(heads)] if decay is None else decay}}


def config(layers, width=88, vocab=96, side=12, eps=1e-5, ff=104, limit=0.9):
    """ff: feed-forward size of every layer, None for none, or a list with one per layer."""
    ffs = ff if isinstance(ff, list) else [ff] * len(layers)
    return {"architecture": "Fenipel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "token_side": {"dim": side} if side else None,
            "layers": [dict(x, mlp=None if f is None else {"kind": "dense", "ff": f, "limit": limit}) for x, f in zip(layers, ffs)]}


def bf16_bits(a):
    u = np.array(a, np.float32, order="C").view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_values(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def weights(cfg, seed, gain=1.0):
    """Tensors as bfloat16 bits under the design's names.  Rows are scaled to keep products near one; `gain` multiplies the
    attention queries, so that scores spread and single keys stand out."""
    r = np.random.default_rng(seed)
    E, V, L = cfg["width"], cfg["vocab"], len(cfg["layers"])
    w = {"embed": r.normal(size=(V, E)), "head": r.normal(size=(V, E)) * E ** -0.5, "final.norm": np.array(1.3)}
    side = cfg.get("token_side")
    if side:
        w["side.embed"] = r.normal(size=(V, L * side["dim"]))
    lin = lambda o, i: r.normal(size=(o, i)) * i ** -0.5
    for n, layer in enumerate(cfg["layers"]):
        m, at = layer["mixer"], f"l{n}."
        H = m["heads"]
        w[at + "norm1"] = np.array(r.uniform(0.7, 1.4))
        if layer["type"] == "latent_attention":
            w[at + "mix.q"] = gain * lin(H * (m["dim"] + m["rot_dim"]), E)
            w[at + "mix.dkv"] = lin(m["kv_rank"] + m["rot_dim"], E)
            w[at + "mix.dkv.norm"] = r.uniform(0.6, 1.5, m["kv_rank"])
            w[at + "mix.uk"] = lin(H * m["dim"], m["kv_rank"])
            w[at + "mix.uv"] = lin(H * m["vdim"], m["kv_rank"])
            w[at + "mix.g"] = lin(H, E)
        else:
            w[at + "mix.q"], w[at + "mix.k"] = lin(H * m["dim"], E), lin(H * m["dim"], E)
            w[at + "mix.v"], w[at + "mix.g"] = lin(H * m["vdim"], E), lin(H * m["vdim"], E)
        w[at + "mix.o"] = lin(E, H * m["vdim"])
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[at + "mlp.gate"], w[at + "mlp.up"], w[at + "mlp.down"] = lin(ff, E), lin(ff, E), lin(E, ff)
        if side:
            w[at + "side.gate"], w[at + "side.proj"] = lin(side["dim"], E), lin(E, side["dim"])
            w[at + "side.norm"] = r.uniform(0.2, 0.6, E)
    return {k: bf16_bits(v) for k, v in w.items()}


def values(w):
    """The same tensors as numbers, for the plain statement."""
    return {k: bf16_values(v) for k, v in w.items()}


def tokens(cfg, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]
