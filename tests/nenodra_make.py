"""Small Nenodra configurations with random weights for the tests."""
import numpy as np

from fenipel_make import bf16_bits, bf16_values, tokens, values  # noqa: F401


def differential(heads=4, kv_heads=2, dim=24, vdim=20, window=11, rot_dims=16, base=3000.0, scale=None, diff=0.35):
    return {"type": "attention", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": {"base": base, "dims": rot_dims},
        "scale": dim ** -0.5 if scale is None else scale, "diff": diff}}


def gated(heads=6, kv_heads=3, dim=40, window=17, rot_dims=40, base=9000.0, scale=None):
    return {"type": "attention_2", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window}, "rot": {"base": base, "dims": rot_dims},
        "scale": dim ** -0.5 if scale is None else scale}}


def dense(ff=104):
    return {"kind": "dense", "ff": ff}


def experts(n=7, top=2, ff=36):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}


def config(layers, ff=None, width=88, vocab=96, eps=1e-5, mult=0.7, logit_scale=0.4):
    """ff: feed-forward of every layer, None for none, or a list with one per layer."""
    ffs = ff if isinstance(ff, list) else [ff] * len(layers)
    return {"architecture": "Nenodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale,
            "layers": [dict(x, mlp=f) for x, f in zip(layers, ffs)]}


def weights(cfg, seed, gain=1.0):
    """Tensors as bfloat16 bits under the design's names.  Rows are scaled to keep products near one; `gain` multiplies the query
    norms, so that scores spread and single keys stand out.

    Rounding must not decide which experts a token gets: the first entries of the residual, one per expert, hold a ladder of
    well-separated values, in an order of its own for every token; nothing else is added to them (their norm weights are -1), and
    routers read little else."""
    r = np.random.default_rng(seed)
    E, V = cfg["width"], cfg["vocab"]
    codes = max([x["mlp"]["router"]["experts"] for x in cfg["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe"], default=0)
    assert codes < E
    embed = r.normal(size=(V, E))
    for t in range(V):
        embed[t, :codes] = r.permutation(np.linspace(-2.0 - 0.05 * codes, 2.0 + 0.05 * codes, codes))

    def norm():
        w = r.normal(size=E) * 0.3
        w[:codes] = -1.0
        return w

    lin = lambda o, i: r.normal(size=(o, i)) * i ** -0.5
    w = {"embed": embed, "head": lin(V, E), "final.norm": r.normal(size=E) * 0.3}
    for n, layer in enumerate(cfg["layers"]):
        m, at = layer["mixer"], f"l{n}."
        H, G, D, D2 = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        maps = 2 if layer["type"] == "attention" else 1
        w[at + "norm1"] = norm()
        w[at + "mix.q"], w[at + "mix.k"] = lin(H * maps * D, E), lin(G * maps * D, E)
        w[at + "mix.q.norm"], w[at + "mix.k.norm"] = gain * r.uniform(0.5, 1.5, D), r.uniform(0.5, 1.5, D)
        w[at + "mix.o"] = lin(E, H * D2)
        if maps == 2:
            w[at + "mix.v"] = lin(G * D2, E)
            for name, size in (("q", H * 2 * D), ("k", G * 2 * D), ("v", G * D2), ("o", E)):
                w[at + f"mix.{name}.b"] = r.normal(size=size) * 0.5
            for name in ("lq1", "lk1", "lq2", "lk2"):
                w[at + "mix." + name] = r.normal(size=D) * 0.7 * D ** -0.5
        else:
            w[at + "mix.g"] = lin(H * D2, E)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        w[at + "norm2"] = norm()
        if mlp["kind"] == "dense":
            w[at + "mlp.up"], w[at + "mlp.down"] = lin(mlp["ff"], E), lin(E, mlp["ff"])
        else:
            X, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            z = r.normal(size=(X, E)) * 0.004
            for e, c in enumerate(r.permutation(codes)[:X]):
                z[e, c] += 1.0
            w[at + "mlp.router"] = z
            for e in range(X):
                w[at + f"mlp.e{e}.gate"], w[at + f"mlp.e{e}.up"], w[at + f"mlp.e{e}.down"] = lin(ff, E), lin(ff, E), lin(E, ff)
    return {k: bf16_bits(v) for k, v in w.items()}
