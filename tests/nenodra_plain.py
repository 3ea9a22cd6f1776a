"""Plain, slow statement of the Nenodra design in float64, one function per mechanism.  It is what the tests compare the framework
with and shares no code with it.

Weights are a dict of numpy arrays under the file's tensor names; a configuration is the parsed config.json."""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def over_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """Norm of the residual's width; the weight is stored around zero."""
    return over_rms(x, eps) * (1.0 + w)


def rotate(x, pos, base, dims):
    """x [..., n]: entries i and i + dims/2 of the first `dims` turn by pos * base^(-2i/dims), the others stay."""
    out = np.array(x, np.float64)
    half = dims // 2
    for i in range(half):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * np.cos(a) - v * np.sin(a)
        out[..., i + half] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(i, j, window):
    """Does position i see position j?  (j may be an array.)"""
    return (i - j >= 0) & (i - j < window)


def normed_rotated(x, w, mx, eps):
    """Queries or keys [n, ..., dim] of consecutive positions from 0: norm per vector, then rotation."""
    y = over_rms(x, eps) * w
    return np.stack([rotate(y[p], p, mx["rot"]["base"], mx["rot"]["dims"]) for p in range(len(y))])


def softmax_average(q, k, v, scale, window):
    """One map of one head: q, k [n, dim], v [n, vdim] -> [n, vdim]."""
    out = np.zeros((len(q), v.shape[1]))
    for i in range(len(q)):
        js = np.flatnonzero(visible(i, np.arange(len(k)), window))
        s = (k[js] @ q[i]) * scale
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[js]
    return out


def differential_weight(w, diff):
    return np.exp(np.sum(w["lq1"] * w["lk1"])) - np.exp(np.sum(w["lq2"] * w["lk2"])) + diff


def differential_attention(h, w, mx, eps):
    """Two maps per head over the same values; their difference over its root mean square."""
    n, H, G, D, V, win = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["mask"]["size"]
    q = normed_rotated((h @ w["q"].T + w["q.b"]).reshape(n, H, 2, D), w["q.norm"], mx, eps)
    k = normed_rotated((h @ w["k"].T + w["k.b"]).reshape(n, G, 2, D), w["k.norm"], mx, eps)
    v = (h @ w["v"].T + w["v.b"]).reshape(n, G, V)
    lam = differential_weight(w, mx["diff"])
    o = np.zeros((n, H, V))
    for hd in range(H):
        g = hd // (H // G)
        a1, a2 = (softmax_average(q[:, hd, m], k[:, g, m], v[:, g], mx["scale"], win) for m in (0, 1))
        o[:, hd] = over_rms(a1 - lam * a2, eps) * (1.0 - mx["diff"])
    return o.reshape(n, -1) @ w["o"].T + w["o.b"]


def gated_attention(h, w, mx, eps):
    """Values are the keys as projected; the heads are gated element by element."""
    n, H, G, D, win = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["mask"]["size"]
    kp = (h @ w["k"].T).reshape(n, G, D)
    q = normed_rotated((h @ w["q"].T).reshape(n, H, D), w["q.norm"], mx, eps)
    k = normed_rotated(kp, w["k.norm"], mx, eps)
    o = np.stack([softmax_average(q[:, hd], k[:, hd // (H // G)], kp[:, hd // (H // G)], mx["scale"], win) for hd in range(H)], axis=1)
    return (o.reshape(n, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def dense(h, w):
    return np.maximum(h @ w["up"].T, 0.0) ** 2 @ w["down"].T


def chosen_experts(h, w, router):
    """Experts of every token, best first, and their scores: [n, top] each."""
    s = sigmoid(h @ w["router"].T)
    best = np.argsort(-s, axis=1, kind="stable")[:, :router["top"]]
    return best, np.take_along_axis(s, best, axis=1)


def mixture(h, w, mlp):
    """A chosen expert reads its score times the input."""
    best, score = chosen_experts(h, w, mlp["router"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(best[t], score[t]):
            z = s * h[t]
            out[t] += w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ z) * (w[f"e{e}.up"] @ z))
    return out


def feed_forward(h, w, mlp):
    return mixture(h, w, mlp) if mlp["kind"] == "moe" else dense(h, w)


def part(weights, prefix):
    return {k[len(prefix):]: np.asarray(v, np.float64) for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"attention": differential_attention, "attention_2": gated_attention}


def forward(cfg, weights, tokens):
    """Logits [n, vocab] at every position of one sequence, and the residual stream after every layer [layers, n, width]."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = np.asarray(weights["embed"], np.float64)[np.asarray(tokens)]
    hidden = []
    for i, layer in enumerate(cfg["layers"]):
        w = part(weights, f"l{i}.")
        x = x + m * norm(MIXERS[layer["type"]](x, part(weights, f"l{i}.mix."), layer["mixer"], eps), w["norm1"], eps)
        if layer["mlp"] is not None:
            x = x + m * norm(feed_forward(x, part(weights, f"l{i}.mlp."), layer["mlp"]), w["norm2"], eps)
        hidden.append(x)
    h = norm(x, np.asarray(weights["final.norm"], np.float64), eps)
    return h @ np.asarray(weights["head"], np.float64).T * cfg["logit_scale"], np.array(hidden)
