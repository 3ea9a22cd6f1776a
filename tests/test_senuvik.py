"""Senuvik without a GPU: configuration and weight reading, the registry, and the plain statement the GPU tests lean on."""
import json

import numpy as np
import pytest

import senuvik_make as S
import senuvik_plain as P
from test_fenipel import FakeBackend

CFG = S.config([S.window(), S.space(), S.beside(), S.window(size=30, keep=5, kv_from=0), S.beside(heads=1, kv_heads=1)],
               ff=[S.dense(40), S.experts(5, 3, 20, shared=50), None, S.experts(4, 1, 30, shared=12), S.dense(24)])


def test_description_follows_the_configuration(monkeypatch):
    import ctypes as C

    from orangu_b200 import capi, senuvik
    from orangu_b200.senuvik import SenuvikModel

    described = senuvik.Describer()
    monkeypatch.setattr(senuvik, "Describer", lambda: described)  # keeps the arrays behind the description alive
    be, w = FakeBackend(), S.weights(CFG, 1)
    m = SenuvikModel(be, CFG, w, dtype="float32", max_seq_len=70, max_batch_tokens=9, kv_pool_tokens=64, state_slots=3)
    d, (a, b, c, e, f) = be._lib.desc, be._lib.blocks
    floats = lambda p, n: np.ctypeslib.as_array(C.cast(p, C.POINTER(C.c_float)), (n,))
    doubles = lambda p, n: np.ctypeslib.as_array(C.cast(p, C.POINTER(C.c_double)), (n,))
    v = S.values(w)
    assert (d.n_vocab, d.n_embd, d.n_layer, d.side_dim, d.compute_f32) == (96, 88, 5, 0, 1)
    assert (d.max_seq_len, d.max_batch_tokens, d.kv_pool_tokens, d.n_state_slots) == (70, 9, 64, 3)
    assert d.rms_eps == pytest.approx(1e-5) and d.residual_mult == 1.0 and d.final_gain == 1.0
    np.testing.assert_allclose(floats(d.final_norm, 88), v["final.norm"])
    np.testing.assert_allclose(floats(a.pre_norm1, 88), v["l0.norm1"])
    np.testing.assert_allclose(floats(a.post_norm1, 88), v["l0.norm1b"] * v["l0.ls1"], rtol=1e-6)
    np.testing.assert_allclose(floats(b.post_norm2, 88), v["l1.norm2b"] * v["l1.ls2"], rtol=1e-6)
    x = a.mixer
    assert (x.kind, x.n_head, x.n_kv_head, x.n_map, x.dim, x.vdim, x.window, x.keep_first) == (capi.MIXER_ATTENTION, 4, 2, 1, 24, 20, 11, 3)
    assert (x.rot_dims, x.rot_interleaved, x.qk_norm_whole, x.kv_layer, x.softcap) == (16, 1, 1, 0, 0.0)
    np.testing.assert_allclose(doubles(x.rot_freqs, 8), P.linear_frequencies(CFG["layers"][0]["mixer"]["rot"])[0])
    np.testing.assert_allclose(floats(x.sink, 4), v["l0.mix.sink"])
    np.testing.assert_allclose(floats(x.k_norm, 48), v["l0.mix.k.norm"])
    assert (a.ff_kind, a.n_ff, a.w_gate.out_dim, a.w_down.in_dim) == (capi.FF_GELU_GLU, 40, 40, 40) and not a.mixer2.kind
    x = b.mixer
    assert (x.kind, x.n_head, x.dim, x.vdim, x.n_group, x.n_norm_group, x.conv_taps) == (capi.MIXER_STATE_SPACE, 6, 20, 12, 3, 4, 4)
    assert x.w_in.out_dim == 72 + 72 + 120 + 6
    np.testing.assert_allclose(floats(x.conv_w, 192 * 4), v["l1.mix.conv"].reshape(-1))
    assert (b.ff_kind, b.n_ff, b.n_expert, b.n_expert_used, b.router_softmax, b.shared_ff) == (capi.FF_EXPERTS, 20, 5, 3, 1, 50)
    assert (b.shared_up.out_dim, b.shared_down.in_dim, b.w_shared_scale.out_dim) == (50, 50, 1)
    x, y = c.mixer, c.mixer2
    freqs, gain = P.yarn_frequencies(CFG["layers"][2]["mixer"]["left"]["rot"])
    np.testing.assert_allclose(doubles(x.rot_freqs, 10), freqs)
    assert x.rot_gain == pytest.approx(gain) and x.softcap == 4.0 and x.window == 0 and x.w_gate.out_dim == 4 and not x.q_norm and not x.sink
    assert (y.kind, y.n_head, y.dim, y.vdim, y.w_decay1.out_dim, y.w_decay2.in_dim) == (capi.MIXER_TIME_MIXING, 3, 18, 18, 10, 10)
    np.testing.assert_allclose(floats(y.mu_g, 88), v["l2.mix.right.mu.g"])
    assert (c.mixer_scale, c.mixer2_scale) == (pytest.approx(0.8), pytest.approx(1.3)) and not c.n_ff and not c.pre_norm2
    x = e.mixer
    assert (x.kv_layer, x.window, x.keep_first) == (1, 30, 5) and not x.wk.data and not x.wv.data and not x.k_norm and x.q_norm
    assert e.shared_ff == 12
    assert m.cache_widths(0) == (48, 40) and m.state_shape(1) == (6, 20, 12) and m.state_shape(2) == (3, 18, 18)


@pytest.mark.parametrize("change, message", [
    (lambda c, w: c["layers"][0].update(type="other"), "no mixer"),
    (lambda c, w: c["layers"][1]["mlp"].update(kind="other"), "no feed-forward"),
    (lambda c, w: w.pop("l0.mix.v.b"), "no tensor l0.mix.v.b"),
    (lambda c, w: w.pop("l1.mlp.shared.sg"), "no tensor l1.mlp.shared.sg"),
    (lambda c, w: w.pop("l2.mix.right.mu.w"), "no tensor l2.mix.right.mu.w"),
    (lambda c, w: c["layers"][0]["mixer"].update(dim=32), "expected"),
    (lambda c, w: c["layers"][1]["mixer"].update(state=32), "expected"),
    (lambda c, w: c["layers"][1]["mixer"].update(groups=4), "over 4 groups"),
    (lambda c, w: c["layers"][1]["mixer"].update(norm_groups=5), "5 normed parts"),
    (lambda c, w: c["layers"][2]["mixer"]["left"].update(kv_heads=3), "4 heads over 3"),
    (lambda c, w: c["layers"][1]["mlp"]["router"].update(top=6), "6 of 5 experts"),
])
def test_what_does_not_fit_is_refused(change, message):
    from orangu_b200.senuvik import SenuvikModel

    c, w = json.loads(json.dumps(CFG)), S.weights(CFG, 1)
    change(c, w)
    with pytest.raises(ValueError, match=message):
        SenuvikModel(FakeBackend(), c, w)


def test_registry_chooses_by_architecture(tmp_path):
    from orangu_b200 import registry

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert registry.model_class(str(tmp_path)) is registry.SenuvikModel


def test_frequencies():
    """The reader's frequencies are the statement's, also at the ends of the ramp."""
    from orangu_b200 import senuvik

    for dims, base, original, fast, slow, factor in ((20, 9000.0, 40, 8.0, 0.5, 3.0), (64, 1e4, 4096, 32.0, 1.0, 16.0), (8, 100.0, 7, 1.0, 1.0, 1.0), (2, 50.0, 1000, 20.0, 0.01, 4.0)):
        rot = {"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
        (a, b), (c, d) = senuvik.yarn_frequencies(rot), P.yarn_frequencies(rot)
        np.testing.assert_allclose(a, c, rtol=1e-14)
        assert b == pytest.approx(d)
        np.testing.assert_allclose(senuvik.linear_frequencies(rot), P.linear_frequencies(rot)[0], rtol=1e-14)
    f, g = P.yarn_frequencies({"dims": 64, "base": 1e4, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}})
    plain = P.plain_frequencies({"dims": 64, "base": 1e4})
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 8) and (np.diff(f) < 0).all() and g == pytest.approx(1.2079, abs=1e-4)
    f, g = P.yarn_frequencies({"dims": 64, "base": 1e4, "scaling": {"factor": 1.0, "original": 2048, "fast": 32.0, "slow": 1.0}})
    np.testing.assert_allclose(f, plain)
    assert g == 1.0


# ---- the plain statement itself
def test_plain_mask_sink_and_cap():
    assert [j for j in range(12) if P.visible(9, j, 4, 2)] == [0, 1, 6, 7, 8, 9] and [j for j in range(6) if P.visible(1, j, 4, 3)] == [0, 1]
    assert [j for j in range(12) if P.visible(5, j)] == [0, 1, 2, 3, 4, 5]
    q, k, v = np.zeros((3, 2)), np.ones((3, 2)), np.array([[3.0], [6.0], [9.0]])
    np.testing.assert_allclose(P.attend(q, k, v, 1.0), [[3.0], [4.5], [6.0]])
    np.testing.assert_allclose(P.attend(q, k, v, 1.0, sink=np.log(3.0)), [[0.75], [9 / 5], [3.0]])  # the sink weighs as much as three keys
    q = np.array([[0.0], [0.0], [100.0]])
    k = np.array([[1.0], [2.0], [-1.0]])
    got = P.attend(q, k, v, 1.0, softcap=2.0)[2, 0]  # scores 2, 2 and -2
    assert got == pytest.approx((3 * np.e ** 2 + 6 * np.e ** 2 + 9 * np.e ** -2) / (2 * np.e ** 2 + np.e ** -2))


def test_plain_rotation_layouts():
    one = np.array([1.0])
    np.testing.assert_allclose(P.rotate(np.eye(4)[0], 1, np.array([1.0, 0.1]), 1.0, False), [np.cos(1), 0, np.sin(1), 0], atol=1e-12)
    np.testing.assert_allclose(P.rotate(np.eye(4)[0], 1, np.array([1.0, 0.1]), 2.0, True), [2 * np.cos(1), 2 * np.sin(1), 0, 0], atol=1e-12)
    np.testing.assert_allclose(P.rotate(np.array([1.0, 2.0, 7.0]), 3, one, 1.0, True)[2], 7.0)


def test_plain_recurrences():
    """Against sums over all earlier tokens."""
    r = np.random.default_rng(3)
    n, N, V = 6, 4, 3
    x, B, C, dt = r.normal(size=(n, 2, V)), r.normal(size=(n, 1, N)), r.normal(size=(n, 1, N)), r.uniform(0.1, 1.0, (n, 2))
    A, D = r.normal(size=2), r.normal(size=2)
    y, S = P.state_space(x, B, C, dt, A, D, 2, 1)
    for a in range(2):
        for t in range(n):
            want = D[a] * x[t, a]
            for s in range(t + 1):
                want = want + np.exp(-np.exp(A[a]) * dt[s + 1:t + 1, a].sum()) * dt[s, a] * (C[t, 0] @ B[s, 0]) * x[s, a]
            np.testing.assert_allclose(y[t, a], want)
    q, k, v, w, u = r.normal(size=(n, N)), r.normal(size=(n, N)), r.normal(size=(n, N)), r.uniform(0.2, 1.0, (n, N)), r.normal(size=N)
    o, S = P.decayed_outer_products(q, k, v, w, u)
    for t in range(n):
        want = (q[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (q[t] * w[s + 1:t].prod(0) * k[s]).sum() * v[s]
        np.testing.assert_allclose(o[t], want)
    taps = np.array([[2.0, 3.0, 5.0]])
    np.testing.assert_allclose(P.causal_conv(np.array([[1.0], [10.0], [100.0]]), taps, np.array([0.5]))[:, 0], [5.5, 53.5, 532.5])


def test_plain_experts():
    mlp = S.experts(4, 2, 5, shared=9)
    w, h = P.part(S.values(S.weights(S.config([S.window()], ff=mlp), 7)), "l0.mlp."), np.random.default_rng(8).normal(size=(3, 88))
    got = P.mixture(h, w, mlp)
    ff = lambda p, x: w[p + "down"] @ (x_silu(w[p + "gate"] @ x) * (w[p + "up"] @ x))
    x_silu = lambda z: z / (1 + np.exp(-z))
    for t in range(3):
        z = w["router"] @ h[t]
        a, b = np.argsort(-z)[:2]
        s = 1 / (1 + np.exp(z[b] - z[a]))
        want = s * ff(f"e{a}.", h[t]) + (1 - s) * ff(f"e{b}.", h[t]) + ff("shared.", h[t]) / (1 + np.exp(-(w["shared.sg"] @ h[t])))
        np.testing.assert_allclose(got[t], want)
