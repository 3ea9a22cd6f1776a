"""Small Filorax configurations with random weights for the tests."""
import numpy as np

from fenipel_make import bf16_bits, bf16_values, tokens, values  # noqa: F401


def window(heads=3, dim=24, vdim=20, kv_rank=40, size=11, scale=None, plain=False):
    """plain: without sink and gate."""
    return {"type": "latent_attention_3" if plain else "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": size}, "scale": dim ** -0.5 if scale is None else scale}}


def causal(heads=3, dim=24, rot_dim=16, vdim=20, kv_rank=40, base=3000.0, scale=None):
    return {"type": "latent_attention_2", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
        "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def experts(n=8, top=3, ff=36, groups=4, keep=2, scale=1.7, shared=20):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale},
            "shared": {"ff": shared} if shared else None}


def config(layers, ff=None, width=96, groups=3, taps=4, vocab=90, eps=1e-5, mult=0.7):
    """ff: feed-forward of every layer, None for none, or a list with one per layer."""
    ffs = ff if isinstance(ff, list) else [ff] * len(layers)
    return {"architecture": "Filorax", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "canon": {"taps": taps}, "residual_mult": mult,
            "layers": [dict(x, mlp=f) for x, f in zip(layers, ffs)]}


def weights(cfg, seed, gain=1.0, conv=True):
    """Tensors as bfloat16 bits under the design's names.  Rows are scaled to keep products near one; `gain` multiplies the queries,
    so that scores spread and single keys stand out.  conv False: only the current token's tap of the input convolutions.

    Rounding must not decide which experts a token gets: the first entries of the residual, one per expert, hold a ladder of
    well-separated values, in an order of its own for every token; nothing is added to them, no other token is mixed in, the factors
    of the average over depth sum to one, and routers read little else."""
    r = np.random.default_rng(seed)
    E, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    codes = max([x["mlp"]["router"]["experts"] for x in cfg["layers"] if x["mlp"]], default=0)
    assert codes < E
    embed = r.normal(size=(V, E))
    for t in range(V):
        embed[t, :codes] = r.permutation(np.linspace(-2.0 - 0.05 * codes, 2.0 + 0.05 * codes, codes))
    lin = lambda o, i: r.normal(size=(o, i)) * i ** -0.5

    def factors(n, keep=0):
        f = r.uniform(0.5, 1.5, n)
        f[:keep] = 1.0
        return f

    def added(i):
        w = lin(E, i)
        w[:codes] = 0.0
        return w

    def taps_of():
        w = r.normal(size=(E, taps)) * 0.4
        w[:codes] = 0.0
        if not conv:
            w[:, :-1] = 0.0
        return w

    w = {"embed": embed, "head": lin(V, E), "final.norm": factors(E)}
    for n, layer in enumerate(cfg["layers"]):
        m, at = layer["mixer"], f"l{n}."
        H, D, D2, K, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m.get("rot_dim", 0)
        mix = at + "mix."
        w[at + "norm1"], w[at + "canon1"] = factors(E, codes), taps_of()
        depth = np.append(r.normal(size=n + 1) * 0.4 / (n + 1), 1.0)
        w[at + "dwa"] = depth / depth.sum()
        w[mix + "q"], w[mix + "dkv"] = gain * lin(H * (D + R), E), lin(K + R, E)
        w[mix + "dkv.norm"], w[mix + "uk"], w[mix + "uv"] = factors(K), lin(H * D, K), lin(H * D2, K)
        if layer["type"] != "latent_attention_3":
            w[mix + "sink"], w[mix + "g"] = r.normal(size=H) + 1.0, 2.0 * lin(H * D2, E)
        w[mix + "o"] = 2.5 * added(H * D2)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        w[at + "norm2"], w[at + "canon2"] = factors(E, codes), taps_of()

        def feed(prefix, ff):
            w[prefix + "gate"], w[prefix + "up"], w[prefix + "down"] = lin(ff, E), lin(ff, E), added(ff)

        X = mlp["router"]["experts"]
        z = r.normal(size=(X, E)) * 0.004
        for e, c in enumerate(r.permutation(codes)[:X]):
            z[e, c] += 1.0
        w[at + "mlp.router"] = z
        for e in range(X):
            feed(f"{at}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp["shared"]:
            feed(at + "mlp.shared.", mlp["shared"]["ff"])
            w[at + "mlp.shared.sg"] = 2.0 * lin(1, E)
    return {k: bf16_bits(v) for k, v in w.items()}
