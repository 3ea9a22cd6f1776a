"""Plain, slow statement of the Filorax design in float64, one function per mechanism.  It is what the tests compare the framework
with and shares no code with it.

Weights are a dict of numpy arrays under the file's tensor names; a configuration is the parsed config.json."""
import numpy as np


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def over_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def grouped_norm(x, w, groups, eps):
    """Each of `groups` equal consecutive parts over its own root mean square, then the factors."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return over_rms(parts, eps).reshape(x.shape) * w


def input_conv(h, w):
    """h [n, width] plus its causal convolution over time, channel by channel; w [width, taps], the last tap meets the current token."""
    out, taps = np.array(h), w.shape[1]
    for t in range(len(h)):
        for back in range(min(taps, t + 1)):
            out[t] = out[t] + w[:, taps - 1 - back] * h[t - back]
    return out


def depth_average(outputs, a):
    """outputs: the embedding and every layer's result so far; a has one number for each."""
    x = np.zeros_like(outputs[0])
    for weight, o in zip(a, outputs, strict=True):
        x = x + weight * o
    return x


def rotate(x, pos, base):
    """All of x [..., n] turns by position, entry i with entry i + n/2."""
    n = x.shape[-1]
    out = np.array(x, np.float64)
    for i in range(n // 2):
        a = pos * float(base) ** (-2.0 * i / n)
        u, v = x[..., i], x[..., i + n // 2]
        out[..., i], out[..., i + n // 2] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def visible(i, j, window=None):
    """Does position i see position j?  window None: everything up to itself."""
    return 0 <= i - j and (window is None or i - j < window)


def attend(q, k, v, scale, window=None, sink=None):
    """q, k [n, heads, d], v [n, heads, d2] -> [n, heads, d2].  A head's sink is one more term of its denominator, exp(sink), that
    brings no value."""
    n, heads = q.shape[:2]
    out = np.zeros((n, heads, v.shape[2]))
    for i in range(n):
        js = [j for j in range(n) if visible(i, j, window)]
        for a in range(heads):
            s = (k[js, a] @ q[i, a]) * scale
            top = s.max() if sink is None else max(s.max(), sink[a])
            p = np.exp(s - top)
            total = p.sum() + (0.0 if sink is None else np.exp(sink[a] - top))
            out[i, a] = p @ v[js, a] / total
    return out


def latent(h, w, mx, eps):
    """What a token leaves in the cache: the normed latent and the rotated key part all heads share (before rotation)."""
    both = h @ w["dkv"].T
    K = mx["kv_rank"]
    return over_rms(both[:, :K], eps) * w["dkv.norm"], both[:, K:]


def latent_attention(h, w, mx, eps, rotated, sink, gated):
    """Mixer over a whole sequence h [n, width]; keys and values are rebuilt from the latent."""
    H, D, V, n = mx["heads"], mx["dim"], mx["vdim"], len(h)
    R = mx["rot_dim"] if rotated else 0
    window = mx["mask"]["size"] if not rotated else None
    q = (h @ w["q"].T).reshape(n, H, D + R)
    c, kr = latent(h, w, mx, eps)
    k = (c @ w["uk"].T).reshape(n, H, D)
    v = (c @ w["uv"].T).reshape(n, H, V)
    if R:
        q = np.concatenate([q[..., :D], np.stack([rotate(q[p, :, D:], p, mx["rot"]["base"]) for p in range(n)])], -1)
        shared = np.stack([rotate(kr[p], p, mx["rot"]["base"]) for p in range(n)])
        k = np.concatenate([k, np.repeat(shared[:, None], H, 1)], -1)
    o = attend(q, k, v, mx["scale"], window, w["sink"] if sink else None).reshape(n, H * V)
    if gated:
        o = o * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


MIXERS = {  # rotated and causal, or without positions and within a window; with a sink; gated
    "latent_attention": dict(rotated=False, sink=True, gated=True),
    "latent_attention_2": dict(rotated=True, sink=True, gated=True),
    "latent_attention_3": dict(rotated=False, sink=False, gated=False),
}


def expert(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def route(z, router):
    """One token's logits -> chosen experts and their weights: the softmax over all experts, only the groups with the largest single
    scores, the largest scores among those, times a constant."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    count, keep = router["groups"]["count"], router["groups"]["keep"]
    size = len(s) // count
    groups = sorted(range(count), key=lambda g: -s[g * size:(g + 1) * size].max())[:keep]
    allowed = [e for e in range(len(s)) if e // size in groups]
    chosen = sorted(allowed, key=lambda e: -s[e])[:router["top"]]
    return chosen, [s[e] * router["scale"] for e in chosen]


def mixture(h, w, mlp):
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, weight in zip(*route(w["router"] @ h[t], mlp["router"])):
            out[t] += weight * expert(h[t:t + 1], w, f"e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ w["shared.sg"].T) * expert(h, w, "shared.")
    return out


def part(weights, prefix):
    return {k[len(prefix):]: np.asarray(v, np.float64) for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, inputs=None):
    """Logits [n, vocab] at every position of one sequence, and the residual after every layer [layers, n, width].  inputs: gets the
    normed inputs of every layer's sublayers before their convolution."""
    eps, groups, mult = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    get = lambda name: np.asarray(weights[name], np.float64)
    x = get("embed")[np.asarray(tokens)]
    outputs, hidden = [x], []
    for i, layer in enumerate(cfg["layers"]):
        at = f"l{i}."
        h = grouped_norm(x, get(at + "norm1"), groups, eps)
        if inputs is not None:
            inputs.append([h])
        x = x + mult * latent_attention(input_conv(h, get(at + "canon1")), part(weights, at + "mix."), layer["mixer"], eps, **MIXERS[layer["type"]])
        if layer["mlp"] is not None:
            h = grouped_norm(x, get(at + "norm2"), groups, eps)
            if inputs is not None:
                inputs[-1].append(h)
            x = x + mult * mixture(input_conv(h, get(at + "canon2")), part(weights, at + "mlp."), layer["mlp"])
        outputs.append(x)
        x = depth_average(outputs, get(at + "dwa"))
        hidden.append(x)
    return grouped_norm(x, get("final.norm"), groups, eps) @ get("head").T, np.array(hidden)
