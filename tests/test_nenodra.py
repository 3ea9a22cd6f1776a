"""Nenodra without a GPU: configuration and weight reading, the registry, and the plain statement the GPU tests lean on."""
import json

import numpy as np
import pytest

import nenodra_make as N
import nenodra_plain as P
from test_fenipel import FakeBackend

CFG = N.config([N.differential(), N.gated(), N.gated(heads=2, kv_heads=1)], ff=[N.dense(40), N.experts(5, 3, 20), None])


def test_description_follows_the_configuration(monkeypatch):
    import ctypes as C

    from orangu_b200 import capi, nenodra
    from orangu_b200.nenodra import NenodraModel

    described = nenodra.Describer()
    monkeypatch.setattr(nenodra, "Describer", lambda: described)  # keeps the arrays behind the description alive
    be, w = FakeBackend(), N.weights(CFG, 1)
    m = NenodraModel(be, CFG, w, dtype="float32", max_seq_len=70, max_batch_tokens=9, kv_pool_tokens=64)
    d, (a, b, c) = be._lib.desc, be._lib.blocks
    floats = lambda p, n: np.ctypeslib.as_array(C.cast(p, C.POINTER(C.c_float)), (n,))
    v = N.values(w)
    assert (d.n_vocab, d.n_embd, d.n_layer, d.side_dim, d.compute_f32) == (96, 88, 3, 0, 1)
    assert (d.max_seq_len, d.max_batch_tokens, d.kv_pool_tokens) == (70, 9, 64)
    assert d.rms_eps == pytest.approx(1e-5) and d.residual_mult == pytest.approx(0.7) and d.final_gain == pytest.approx(0.4)
    np.testing.assert_allclose(floats(d.final_norm, 88), 1 + v["final.norm"], rtol=1e-6, atol=1e-6)
    x = a.mixer
    assert (x.kind, x.n_head, x.n_kv_head, x.n_map, x.dim, x.vdim, x.window) == (capi.MIXER_ATTENTION, 4, 2, 2, 24, 20, 11)
    assert (x.rot_dims, x.rot_interleaved, x.rot_base) == (16, 0, 3000.0) and x.scale == pytest.approx(24 ** -0.5)
    lam = np.exp((v["l0.mix.lq1"] * v["l0.mix.lk1"]).sum()) - np.exp((v["l0.mix.lq2"] * v["l0.mix.lk2"]).sum()) + 0.35
    assert x.map_weight == pytest.approx(lam, rel=1e-6) and x.head_gain == pytest.approx(0.65)
    assert (x.wq.out_dim, x.wk.out_dim, x.wv.out_dim, x.wo.in_dim) == (4 * 48, 2 * 48, 40, 80) and not x.w_gate.data
    np.testing.assert_allclose(floats(x.k_bias, 96), v["l0.mix.k.b"], rtol=1e-6)
    np.testing.assert_allclose(floats(a.post_norm1, 88), 1 + v["l0.norm1"], rtol=1e-6, atol=1e-6)
    assert (a.ff_kind, a.n_ff, a.w_up.out_dim, a.w_down.in_dim) == (capi.FF_RELU2, 40, 40, 40) and not a.w_gate.data
    y = b.mixer
    assert (y.n_map, y.n_head, y.n_kv_head, y.vdim, y.w_gate.out_dim) == (1, 6, 3, 40, 240) and not y.wv.data and not y.q_bias and not y.o_bias
    assert (b.ff_kind, b.n_ff, b.n_expert, b.n_expert_used, b.w_router.out_dim) == (capi.FF_EXPERTS, 20, 5, 3, 5)
    assert [(b.expert_up[e].out_dim, b.expert_down[e].out_dim) for e in range(5)] == [(20, 88)] * 5
    got = np.ctypeslib.as_array(C.cast(b.expert_gate[4].data, C.POINTER(C.c_uint16)), (20, 88))
    assert (got == w["l1.mlp.e4.gate"]).all()
    assert c.n_ff == 0 and not c.post_norm2 and c.post_norm1
    assert m.cache_widths(0) == (96, 40) and m.cache_widths(1) == (120, 120)


@pytest.mark.parametrize("change, message", [
    (lambda c, w: c["layers"][0].update(type="other"), "no mixer"),
    (lambda c, w: c["layers"][1]["mlp"].update(kind="other"), "no feed-forward"),
    (lambda c, w: w.pop("l0.mix.v.b"), "no tensor l0.mix.v.b"),
    (lambda c, w: w.pop("l1.mlp.e3.up"), "no tensor l1.mlp.e3.up"),
    (lambda c, w: c["layers"][0]["mixer"].update(dim=32), "expected"),
    (lambda c, w: c["layers"][1]["mixer"].update(vdim=32), "cannot be values"),
    (lambda c, w: c["layers"][1]["mixer"].update(kv_heads=4), "6 heads over 4"),
    (lambda c, w: c["layers"][1]["mlp"]["router"].update(top=6), "6 of 5 experts"),
])
def test_what_does_not_fit_is_refused(change, message):
    from orangu_b200.nenodra import NenodraModel

    c, w = json.loads(json.dumps(CFG)), N.weights(CFG, 1)
    change(c, w)
    with pytest.raises(ValueError, match=message):
        NenodraModel(FakeBackend(), c, w)


def test_registry_chooses_by_architecture(tmp_path):
    from orangu_b200 import registry

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert registry.model_class(str(tmp_path)) is registry.NenodraModel


# ---- the plain statement itself
def test_plain_difference_of_maps():
    """With equal maps and a weight of one nothing is left; with a weight of zero the second map does not count."""
    cfg = N.config([N.differential(heads=2, kv_heads=1, dim=8, vdim=6, window=5, rot_dims=4, diff=0.0)], width=16)
    mx, r = cfg["layers"][0]["mixer"], np.random.default_rng(3)
    w, h = P.part(N.values(N.weights(cfg, 4)), "l0.mix."), r.normal(size=(7, 16))
    w["lq1"], w["lq2"] = np.zeros(8), np.zeros(8)
    assert P.differential_weight(w, 0.0) == 0.0 and P.differential_weight(w, 0.25) == 0.25
    a = P.differential_attention(h, w, mx, 1e-5)
    other = dict(w, q=np.where(np.arange(32)[:, None] % 16 < 8, w["q"], r.normal(size=(32, 16))))  # another second map
    np.testing.assert_allclose(P.differential_attention(h, other, mx, 1e-5), a)
    q, k = w["q"].reshape(2, 2, 8, 16), w["k"].reshape(1, 2, 8, 16)
    qb, kb = w["q.b"].reshape(2, 2, 8), w["k.b"].reshape(1, 2, 8)
    same = dict(w, q=np.repeat(q[:, :1], 2, 1).reshape(32, 16), k=np.repeat(k[:, :1], 2, 1).reshape(16, 16), lq1=np.ones(8), lk1=np.full(8, np.log(2) / 8))
    same["q.b"], same["k.b"] = np.repeat(qb[:, :1], 2, 1).reshape(-1), np.repeat(kb[:, :1], 2, 1).reshape(-1)
    assert P.differential_weight(same, 0.0) == pytest.approx(1.0)
    np.testing.assert_allclose(P.differential_attention(h, same, mx, 1e-5), np.broadcast_to(w["o.b"], (7, 16)), atol=1e-9)


def test_plain_values_are_unrotated_keys():
    """With a window of one a head's output is the gated projection of its own key."""
    cfg = N.config([N.gated(heads=2, kv_heads=1, dim=6, window=1, rot_dims=6)], width=16)
    w, h = P.part(N.values(N.weights(cfg, 5)), "l0.mix."), np.random.default_rng(6).normal(size=(4, 16))
    k = h @ w["k"].T
    want = (np.concatenate([k, k], 1) / (1 + np.exp(-(h @ w["g"].T)))) @ w["o"].T
    np.testing.assert_allclose(P.gated_attention(h, w, cfg["layers"][0]["mixer"], 1e-5), want)


def test_plain_experts_scale_their_input():
    mlp = N.experts(4, 2, 5)
    cfg = N.config([N.gated()], ff=mlp)
    w, h = P.part(N.values(N.weights(cfg, 7)), "l0.mlp."), np.random.default_rng(8).normal(size=(3, 88))
    got = P.mixture(h, w, mlp)
    for t in range(3):
        z = w["router"] @ h[t]
        want = np.zeros(88)
        for e in np.argsort(-z)[:2]:
            s = 1 / (1 + np.exp(-z[e]))
            g, u = w[f"e{e}.gate"] @ h[t] * s, w[f"e{e}.up"] @ h[t] * s
            want += w[f"e{e}.down"] @ (g / (1 + np.exp(-g)) * u)
        np.testing.assert_allclose(got[t], want)


def test_plain_window_and_rotation():
    assert [j for j in range(12) if P.visible(9, j, 4)] == [6, 7, 8, 9]
    x = np.random.default_rng(9).normal(size=(2, 10))
    a, b = P.rotate(x, 7, 100.0, 6), P.rotate(x, 3, 100.0, 6)
    np.testing.assert_allclose(a[:, 6:], x[:, 6:])
    np.testing.assert_allclose((a[0] * b[1]).sum(), (P.rotate(x, 4, 100.0, 6)[0] * x[1]).sum())  # only the distance counts
    np.testing.assert_allclose(P.rotate(np.eye(4)[0], 1, 5.0, 4), [np.cos(1), 0, np.sin(1), 0], atol=1e-12)  # entry 0 pairs with entry 2
