"""Plain, slow statement of the Fenipel design in float64, one function per mechanism, token by token where the design is
stated that way.  It is what the tests compare the framework with and shares no code with it.

Weights are a dict of numpy arrays under the file's tensor names; a configuration is the parsed config.json."""
import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def over_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotate(x, pos, base, dims, interleaved):
    """x [..., n]: the first `dims` entries rotated by position, the others as they are."""
    out = np.array(x, np.float64)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * np.cos(a) - v * np.sin(a)
        out[..., iv] = v * np.cos(a) + u * np.sin(a)
    return out


def retention(h, w, mx, eps):
    """Mixer over a whole sequence h [n, width], one token after the other; returns (out, final state [heads, dim, vdim])."""
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    decay = np.asarray(mx["decay"], np.float64)
    S = np.zeros((H, D, V))
    outs = []
    for p in range(h.shape[0]):
        q = rotate((w["q"] @ h[p]).reshape(H, D), p, mx["rot"]["base"], mx["rot"]["dims"], False)
        k = rotate((w["k"] @ h[p]).reshape(H, D), p, mx["rot"]["base"], mx["rot"]["dims"], False) * D ** -0.5
        v = (w["v"] @ h[p]).reshape(H, V)
        S = decay[:, None, None] * S + k[:, :, None] * v[:, None, :]
        o = over_rms(np.einsum("hd,hdv->hv", q, S), eps)
        outs.append(w["o"] @ (o.reshape(-1) * silu(w["g"] @ h[p])))
    return np.array(outs), S


def visible(i, j, window):
    """Does position i see position j?"""
    return 0 <= i - j < window


def latent_attention(h, w, mx, eps):
    """Mixer over a whole sequence h [n, width]: keys and values rebuilt from the latent, a softmax per (position, head)."""
    H, D, R, V, K = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    base, win, n = mx["rot"]["base"], mx["mask"]["size"], h.shape[0]
    q = (h @ w["q"].T).reshape(n, H, D + R)
    dkv = h @ w["dkv"].T
    c = over_rms(dkv[:, :K], eps) * w["dkv.norm"]
    kn = (c @ w["uk"].T).reshape(n, H, D)
    v = (c @ w["uv"].T).reshape(n, H, V)
    kr = np.stack([rotate(dkv[p, K:], p, base, R, True) for p in range(n)])
    gate = sigmoid(h @ w["g"].T)
    outs = []
    for i in range(n):
        qn, qr = q[i, :, :D], rotate(q[i, :, D:], i, base, R, True)
        js = [j for j in range(n) if visible(i, j, win)]
        o = np.zeros((H, V))
        for hd in range(H):
            s = (kn[js, hd] @ qn[hd] + kr[js] @ qr[hd]) * mx["scale"]
            p = np.exp(s - s.max())
            o[hd] = (p / p.sum()) @ v[js, hd] * gate[i, hd]
        outs.append(w["o"] @ o.reshape(-1))
    return np.array(outs)


def feed_forward(h, w, mlp):
    lim = mlp["limit"]
    g = np.minimum(h @ w["gate"].T, lim)
    u = np.clip(h @ w["up"].T, -lim, lim)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def token_side(x, e, w, eps):
    """Per-layer token input: what is added to x [n, width]; e [n, dim] is the layer's part of the side table."""
    y = (gelu_tanh(x @ w["gate"].T) * e) @ w["proj"].T
    return over_rms(y, eps) * w["norm"]


def part(weights, prefix):
    return {k[len(prefix):]: np.asarray(v, np.float64) for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"retention": lambda *a: retention(*a)[0], "latent_attention": latent_attention}


def forward(cfg, weights, tokens):
    """Logits [n, vocab] at every position of one sequence, and the residual stream after every layer [layers, n, width]."""
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = np.asarray(weights["embed"], np.float64)[tokens]
    side = cfg.get("token_side")
    hidden = []
    for i, layer in enumerate(cfg["layers"]):
        w = part(weights, f"l{i}.")
        h = over_rms(x, eps) * w["norm1"]
        y = MIXERS[layer["type"]](h, part(weights, f"l{i}.mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, part(weights, f"l{i}.mlp."), layer["mlp"])
        x = x + y
        if side:
            e = np.asarray(weights["side.embed"], np.float64)[tokens][:, i * side["dim"]:(i + 1) * side["dim"]]
            x = x + token_side(x, e, part(weights, f"l{i}.side."), eps)
        hidden.append(x)
    logits = (over_rms(x, eps) * np.float64(weights["final.norm"])) @ np.asarray(weights["head"], np.float64).T
    return logits, np.array(hidden)
