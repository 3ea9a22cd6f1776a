"""Small Senuvik configurations with random weights for the tests."""
import numpy as np

from fenipel_make import bf16_bits, bf16_values, tokens, values  # noqa: F401


def window(heads=4, kv_heads=2, dim=24, vdim=20, size=11, keep=3, rot_dims=16, base=3000.0, factor=2.5, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
         "rot": {"base": base, "dims": rot_dims, "scaling": {"factor": factor}}, "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": m if kv_from is None else dict(m, kv_from=kv_from)}


def space(heads=6, vdim=12, state=20, groups=3, norm_groups=4, conv=4):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def beside(heads=4, kv_heads=2, dim=24, vdim=20, rot_dims=20, base=9000.0, factor=3.0, original=40, fast=8.0, slow=0.5, softcap=4.0, scale=None,
           left=0.8, right=1.3, time_heads=3, time_dim=18):
    """Causal attention beside time mixing."""
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": softcap, "scale": dim ** -0.5 if scale is None else scale,
                 "rot": {"base": base, "dims": rot_dims, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}},
        "right": {"heads": time_heads, "dim": time_dim}, "left_scale": left, "right_scale": right}}


def dense(ff=104):
    return {"kind": "dense", "ff": ff}


def experts(n=7, top=2, ff=36, shared=None):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}, "shared": {"ff": ff if shared is None else shared}}


def config(layers, ff=None, width=88, vocab=96, eps=1e-5):
    """ff: feed-forward of every layer, None for none, or a list with one per layer."""
    ffs = ff if isinstance(ff, list) else [ff] * len(layers)
    return {"architecture": "Senuvik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(x, mlp=f) for x, f in zip(layers, ffs)]}


def weights(cfg, seed, gain=1.0, rank=10):
    """Tensors as bfloat16 bits under the design's names.  Rows are scaled to keep products near one; `gain` multiplies the
    queries, so that scores spread and single keys stand out.  rank: of the time mixing's decay.

    Rounding must not decide which experts a token gets: the first entries of the residual, one per expert, hold a ladder of
    well-separated values, in an order of its own for every token; nothing else is added to them (the factors of what is added are
    zero there), and routers read little else."""
    r = np.random.default_rng(seed)
    E, V = cfg["width"], cfg["vocab"]
    codes = max([x["mlp"]["router"]["experts"] for x in cfg["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe"], default=0)
    assert codes < E
    embed = r.normal(size=(V, E))
    for t in range(V):
        embed[t, :codes] = r.permutation(np.linspace(-2.0 - 0.05 * codes, 2.0 + 0.05 * codes, codes))
    lin = lambda o, i: r.normal(size=(o, i)) * i ** -0.5
    factors = lambda n: r.uniform(0.5, 1.5, n)

    def added():
        w = r.normal(size=E) * 0.9
        w[:codes] = 0.0
        return w

    def read():
        w = factors(E)
        w[:codes] = 1.0
        return w

    w = {"embed": embed, "head": lin(V, E), "final.norm": factors(E)}
    for n, layer in enumerate(cfg["layers"]):
        m, at = layer["mixer"], f"l{n}."
        mix = at + "mix."
        w[at + "norm1"], w[at + "norm1b"], w[at + "ls1"] = read(), added(), factors(E)
        if layer["type"] == "attention":
            H, G, D, D2 = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w[mix + "q"], w[mix + "q.b"], w[mix + "q.norm"] = lin(H * D, E), 0.5 * r.normal(size=H * D), gain * factors(H * D)
            w[mix + "sink"] = r.normal(size=H) + 1.0
            w[mix + "o"] = lin(E, H * D2)
            if m.get("kv_from") is None:
                w[mix + "k"], w[mix + "k.b"], w[mix + "k.norm"] = lin(G * D, E), 0.5 * r.normal(size=G * D), factors(G * D)
                w[mix + "v"], w[mix + "v.b"] = lin(G * D2, E), 0.5 * r.normal(size=G * D2)
        elif layer["type"] == "mamba2":
            H, D2, S, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner, channels = H * D2, H * D2 + 2 * G * S
            w[mix + "in"], w[mix + "o"] = lin(inner + channels + H, E), lin(E, inner)
            w[mix + "conv"], w[mix + "conv.b"] = r.normal(size=(channels, m["conv"])) * m["conv"] ** -0.5, 0.3 * r.normal(size=channels)
            w[mix + "dt_bias"], w[mix + "A_log"], w[mix + "D"] = r.normal(size=H) - 1.0, r.normal(size=H), r.normal(size=H)
            w[mix + "norm"] = factors(inner)
        else:
            a, b = m["left"], m["right"]
            H, G, D, D2 = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w[mix + "left.q"], w[mix + "left.k"], w[mix + "left.v"] = gain * lin(H * D, E), lin(G * D, E), lin(G * D2, E)
            w[mix + "left.g"], w[mix + "left.o"] = lin(H, E), lin(E, H * D2)
            N = b["heads"] * b["dim"]
            for c in "rkvg":
                w[mix + "right." + c] = lin(N, E)
            for c in "rkvgw":
                w[mix + "right.mu." + c] = r.uniform(0.0, 1.0, E)
            w[mix + "right.w1"], w[mix + "right.w2"], w[mix + "right.w0"] = lin(rank, E), lin(N, rank), 1.5 * r.normal(size=N) - 1.5
            w[mix + "right.u"], w[mix + "right.norm"], w[mix + "right.o"] = r.normal(size=(b["heads"], b["dim"])), factors(N), lin(E, N)
        mlp = layer["mlp"]
        if mlp is None:
            continue
        w[at + "norm2"], w[at + "norm2b"], w[at + "ls2"] = read(), added(), factors(E)

        def feed(prefix, ff):
            w[prefix + "gate"], w[prefix + "up"], w[prefix + "down"] = lin(ff, E), lin(ff, E), lin(E, ff)

        if mlp["kind"] == "dense":
            feed(at + "mlp.", mlp["ff"])
        else:
            X = mlp["router"]["experts"]
            z = r.normal(size=(X, E)) * 0.004
            for e, c in enumerate(r.permutation(codes)[:X]):
                z[e, c] += 1.0
            w[at + "mlp.router"] = z
            for e in range(X):
                feed(f"{at}mlp.e{e}.", mlp["expert"]["ff"])
            feed(at + "mlp.shared.", mlp["shared"]["ff"])
            w[at + "mlp.shared.sg"] = 2.0 * lin(1, E)
    return {k: bf16_bits(v) for k, v in w.items()}
