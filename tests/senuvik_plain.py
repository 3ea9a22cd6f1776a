"""Plain, slow statement of the Senuvik design in float64, one function per mechanism.  It is what the tests compare the framework
with and shares no code with it.

Weights are a dict of numpy arrays under the file's tensor names; a configuration is the parsed config.json."""
import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    return over_rms(x, eps) * w


# ---- rotation ---------------------------------------------------------------------------------------------------------------------
def plain_frequencies(rot):
    return np.array([float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])


def linear_frequencies(rot):
    """Every frequency over the factor."""
    return plain_frequencies(rot) / rot["scaling"]["factor"], 1.0


def yarn_frequencies(rot):
    """Pairs that turn often within the original length keep their frequency, slow ones are divided by the factor, a ramp between;
    and the gain of cos and sin."""
    s, n = rot["scaling"], rot["dims"]

    def pair_with_turns(t):
        return n * np.log(s["original"] / (2.0 * np.pi * t)) / (2.0 * np.log(rot["base"]))

    lo, hi = max(np.floor(pair_with_turns(s["fast"])), 0.0), min(np.ceil(pair_with_turns(s["slow"])), n - 1.0)
    f = plain_frequencies(rot)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(s["factor"]) + 1.0


def rotate(x, pos, freq, gain, interleaved):
    """The first 2 len(freq) entries of x [..., n] turn; pairs (2i, 2i+1) or (i, i + len(freq))."""
    out, half = np.array(x, np.float64), len(freq)
    for i in range(half):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        c, s = gain * np.cos(pos * freq[i]), gain * np.sin(pos * freq[i])
        out[..., a], out[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s
    return out


def rotate_all(x, freq, gain, interleaved):
    return np.stack([rotate(x[p], p, freq, gain, interleaved) for p in range(len(x))])


# ---- softmax attention ------------------------------------------------------------------------------------------------------------
def visible(i, j, size=None, keep=0):
    """Does position i see position j?  (j may be an array.)  Within the last `size`, or among the first `keep`."""
    j = np.asarray(j)
    return (j <= i) & ((i - j < size) | (j < keep) if size is not None else True)


def attend(q, k, v, scale, size=None, keep=0, sink=None, softcap=None):
    """One head: q, k [n, dim], v [n, vdim] -> [n, vdim]."""
    out = np.zeros((len(q), v.shape[1]))
    for i in range(len(q)):
        js = np.flatnonzero(visible(i, np.arange(len(k)), size, keep))
        s = (k[js] @ q[i]) * scale
        if softcap is not None:
            s = softcap * np.tanh(s / softcap)
        top = s.max() if sink is None else max(s.max(), sink)
        p = np.exp(s - top)
        out[i] = p @ v[js] / (p.sum() + (0.0 if sink is None else np.exp(sink - top)))
    return out


def window_keys_values(h, w, mx, eps):
    """Keys [n, G, dim] as the cache holds them, and values [n, G, vdim]."""
    n, G, D, V = len(h), mx["kv_heads"], mx["dim"], mx["vdim"]
    k = norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps).reshape(n, G, D)
    return rotate_all(k, *linear_frequencies(mx["rot"]), True), (h @ w["v"].T + w["v.b"]).reshape(n, G, V)


def window_attention(h, w, mx, eps, keys=None):
    """Window with kept first tokens, sink, norm over the whole projection; `keys`: another layer's keys and values."""
    n, H, G, D, mask = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["mask"]
    q = norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).reshape(n, H, D)
    q = rotate_all(q, *linear_frequencies(mx["rot"]), True)
    k, v = keys if keys is not None else window_keys_values(h, w, mx, eps)
    o = [attend(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], mx["scale"], mask["size"], mask["keep_first"], w["sink"][a]) for a in range(H)]
    return np.concatenate(o, axis=1) @ w["o"].T


def capped_attention(h, w, mx):
    """Causal attention over everything with a soft cap and a gate per head."""
    n, H, G, D, V = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    turn = yarn_frequencies(mx["rot"])
    q = rotate_all((h @ w["q"].T).reshape(n, H, D), *turn, False)
    k = rotate_all((h @ w["k"].T).reshape(n, G, D), *turn, False)
    v = (h @ w["v"].T).reshape(n, G, V)
    g = sigmoid(h @ w["g"].T)
    o = [attend(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], mx["scale"], softcap=mx["softcap"]) * g[:, a:a + 1] for a in range(H)]
    return np.concatenate(o, axis=1) @ w["o"].T


# ---- recurrences ------------------------------------------------------------------------------------------------------------------
def causal_conv(u, taps, bias):
    """u [n, channels]; the last column of taps [channels, K] meets the current token."""
    n, K = len(u), taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, u.shape[1])), u])
    return sum(padded[i:i + n] * taps[:, i] for i in range(K)) + bias


def state_space(x, B, C, dt, A_log, D, heads, groups):
    """x [n, heads, vdim], B and C [n, groups, N], dt [n, heads] -> outputs like x, and the last state [heads, N, vdim]."""
    S = np.zeros((heads, B.shape[2], x.shape[2]))
    y = np.zeros_like(x)
    for t in range(len(x)):
        for a in range(heads):
            g = a // (heads // groups)
            S[a] = np.exp(-np.exp(A_log[a]) * dt[t, a]) * S[a] + dt[t, a] * np.outer(B[t, g], x[t, a])
            y[t, a] = S[a].T @ C[t, g] + D[a] * x[t, a]
    return y, S


def mamba2(h, w, mx, eps, states=None):
    n, H, V, N, G = len(h), mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * V
    p = h @ w["in"].T
    z, dt = p[:, :inner], softplus(p[:, -H:] + w["dt_bias"])
    u = silu(causal_conv(p[:, inner:-H], w["conv"], w["conv.b"]))
    x, B, C = u[:, :inner], u[:, inner:inner + G * N], u[:, inner + G * N:]
    y, S = state_space(x.reshape(n, H, V), B.reshape(n, G, N), C.reshape(n, G, N), dt, w["A_log"], w["D"], H, G)
    if states is not None:
        states.append(S)
    y = y.reshape(n, inner) * silu(z)
    y = over_rms(y.reshape(n, mx["norm_groups"], -1), eps).reshape(n, inner)
    return (y * w["norm"]) @ w["o"].T


def decayed_outer_products(r, k, v, decay, u):
    """One head: r, k, decay [n, dim], v [n, dim], u [dim] -> [n, dim] and the last state [dim, dim]."""
    S = np.zeros((r.shape[1], v.shape[1]))
    o = np.zeros((len(r), v.shape[1]))
    for t in range(len(r)):
        kv = np.outer(k[t], v[t])
        o[t] = (S + u[:, None] * kv).T @ r[t]
        S = decay[t][:, None] * S + kv
    return o, S


def time_mixing(h, w, mx, eps, states=None):
    n, H, D = len(h), mx["heads"], mx["dim"]
    before = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])
    mix = {c: h + (before - h) * w["mu." + c] for c in "rkvgw"}
    r, k, v = ((mix[c] @ w[c].T).reshape(n, H, D) for c in "rkv")
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(n, H, D)
    heads = [decayed_outer_products(r[:, a], k[:, a], v[:, a], decay[:, a], w["u"][a]) for a in range(H)]
    if states is not None:
        states.append(np.stack([S for _, S in heads]))
    o = np.concatenate([over_rms(o, eps) for o, _ in heads], axis=1)
    return (o * w["norm"] * silu(mix["g"] @ w["g"].T)) @ w["o"].T


# ---- feed-forwards ----------------------------------------------------------------------------------------------------------------
def gated_ff(h, w, act):
    return (act(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def chosen_experts(h, w, router):
    """Experts of every token, best first, and their weights: [n, top] each."""
    z = h @ w["router"].T
    best = np.argsort(-z, axis=1, kind="stable")[:, :router["top"]]
    p = np.take_along_axis(z, best, axis=1)
    p = np.exp(p - p.max(axis=1, keepdims=True))
    return best, p / p.sum(axis=1, keepdims=True)


def mixture(h, w, mlp):
    best, weight = chosen_experts(h, w, mlp["router"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(best[t], weight[t]):
            out[t] += s * gated_ff(h[t], part(w, f"e{e}."), silu)
    return out + sigmoid(h @ w["shared.sg"].T) * gated_ff(h, part(w, "shared."), silu)


def feed_forward(h, w, mlp):
    return mixture(h, w, mlp) if mlp["kind"] == "moe" else gated_ff(h, w, gelu)


def part(weights, prefix):
    return {k[len(prefix):]: np.asarray(v, np.float64) for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, states=None):
    """Logits [n, vocab] at every position of one sequence, and the residual stream after every layer [layers, n, width].
    states (a list) gets every recurrent layer's last state."""
    eps = cfg["norm"]["eps"]
    x = np.asarray(weights["embed"], np.float64)[np.asarray(tokens)]
    hidden, cached = [], {}
    for i, layer in enumerate(cfg["layers"]):
        w, at, mx = part(weights, f"l{i}."), f"l{i}.mix.", layer["mixer"]
        h = norm(x, w["norm1"], eps)
        if layer["type"] == "attention":
            cached[i] = cached[mx["kv_from"]] if mx.get("kv_from") is not None else window_keys_values(h, part(weights, at), mx, eps)
            y = window_attention(h, part(weights, at), mx, eps, cached[i])
        elif layer["type"] == "mamba2":
            y = mamba2(h, part(weights, at), mx, eps, states)
        else:
            y = mx["left_scale"] * capped_attention(h, part(weights, at + "left."), mx["left"]) + \
                mx["right_scale"] * time_mixing(h, part(weights, at + "right."), mx["right"], eps, states)
        x = x + norm(y, w["norm1b"], eps) * w["ls1"]
        if layer.get("mlp") is not None:
            y = feed_forward(norm(x, w["norm2"], eps), part(weights, f"l{i}.mlp."), layer["mlp"])
            x = x + norm(y, w["norm2b"], eps) * w["ls2"]
        hidden.append(x)
    h = norm(x, np.asarray(weights["final.norm"], np.float64), eps)
    return h @ np.asarray(weights["head"], np.float64).T, np.array(hidden)
