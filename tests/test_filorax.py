"""Filorax without a GPU: configuration and weight reading, the registry, and the plain statement the GPU tests lean on."""
import json

import numpy as np
import pytest

import filorax_make as S
import filorax_plain as P
from test_fenipel import FakeBackend

CFG = S.config([S.window(), S.causal(heads=2), S.window(plain=True, size=30), S.causal()],
               ff=[S.experts(), None, S.experts(6, 1, 20, groups=1, keep=1, shared=None), S.experts(10, 4, 30, groups=5, keep=2, shared=50)])


def test_description_follows_the_configuration(monkeypatch):
    import ctypes as C

    from orangu_b200 import capi, filorax
    from orangu_b200.filorax import FiloraxModel

    described = filorax.Describer()
    monkeypatch.setattr(filorax, "Describer", lambda: described)  # keeps the arrays behind the description alive
    be, w = FakeBackend(), S.weights(CFG, 1)
    m = FiloraxModel(be, CFG, w, dtype="float32", max_seq_len=70, max_batch_tokens=9, kv_pool_tokens=64, state_slots=3)
    d, (a, b, c, e) = be._lib.desc, be._lib.blocks
    floats = lambda p, n: np.ctypeslib.as_array(C.cast(p, C.POINTER(C.c_float)), (n,))
    v = S.values(w)
    assert (d.n_vocab, d.n_embd, d.n_layer, d.side_dim, d.compute_f32, d.norm_groups, d.conv_taps) == (90, 96, 4, 0, 1, 3, 4)
    assert (d.max_seq_len, d.max_batch_tokens, d.kv_pool_tokens, d.n_state_slots) == (70, 9, 64, 3)
    assert (d.rms_eps, d.residual_mult, d.final_gain) == (pytest.approx(1e-5), pytest.approx(0.7), 1.0)
    np.testing.assert_allclose(floats(d.final_norm, 96), v["final.norm"])
    np.testing.assert_allclose(floats(a.pre_norm1, 96), v["l0.norm1"])
    np.testing.assert_allclose(floats(a.conv2, 96 * 4), v["l0.canon2"].reshape(-1))
    np.testing.assert_allclose(floats(e.depth, 5), v["l3.dwa"])
    assert not a.post_norm1 and not a.post_norm2
    x = a.mixer
    assert (x.kind, x.n_head, x.dim, x.rot_dim, x.vdim, x.kv_rank, x.window, x.rot_dims) == (capi.MIXER_LATENT_ATTENTION, 3, 24, 0, 20, 40, 11, 0)
    assert (x.w_gate.out_dim, x.wq.out_dim, x.w_dkv.out_dim) == (60, 72, 40) and x.scale == pytest.approx(24 ** -0.5)
    np.testing.assert_allclose(floats(x.sink, 3), v["l0.mix.sink"])
    x = b.mixer
    assert (x.n_head, x.rot_dim, x.window, x.rot_dims, x.rot_interleaved, x.rot_base) == (2, 16, 0, 16, 0, 3000.0)
    assert (x.wq.out_dim, x.w_dkv.out_dim) == (80, 56) and x.sink and x.w_gate.data and not b.n_ff and not b.conv2
    x = c.mixer
    assert x.window == 30 and not x.sink and not x.w_gate.data
    assert (a.ff_kind, a.n_ff, a.n_expert, a.n_expert_used, a.router_softmax) == (capi.FF_EXPERTS, 36, 8, 3, capi.ROUTER_SOFTMAX_ALL)
    assert (a.n_expert_group, a.n_group_used, a.shared_ff) == (4, 2, 20) and a.router_scale == pytest.approx(1.7)
    assert (c.n_expert_group, c.n_group_used, c.shared_ff) == (1, 1, 0) and e.shared_ff == 50
    assert m.cache_widths(1) == (40, 16) and m.cache_widths(0) == (40, 0) and m.state_shape(0) == (2, 3, 96) and m.state_shape(1) == (1, 3, 96)


@pytest.mark.parametrize("change, message", [
    (lambda c, w: c["layers"][0].update(type="other"), "no mixer"),
    (lambda c, w: c["layers"][0]["mlp"].update(kind="dense"), "no feed-forward"),
    (lambda c, w: w.pop("l1.mix.g"), "no tensor l1.mix.g"),
    (lambda c, w: w.pop("l0.mlp.shared.sg"), "no tensor l0.mlp.shared.sg"),
    (lambda c, w: w.pop("l2.canon2"), "no tensor l2.canon2"),
    (lambda c, w: w.update({"l2.dwa": w["l1.dwa"]}), "expected"),
    (lambda c, w: c["layers"][1]["mixer"].update(rot_dim=32), "expected"),
    (lambda c, w: c["canon"].update(taps=3), "expected"),
    (lambda c, w: c["norm"].update(groups=5), "do not divide"),
    (lambda c, w: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups of 8 experts"),
    (lambda c, w: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "5 of 4 groups"),
    (lambda c, w: c["layers"][0]["mlp"]["router"].update(top=5), "5 experts of 2 groups"),
])
def test_what_does_not_fit_is_refused(change, message):
    from orangu_b200.filorax import FiloraxModel

    c, w = json.loads(json.dumps(CFG)), S.weights(CFG, 1)
    change(c, w)
    with pytest.raises(ValueError, match=message):
        FiloraxModel(FakeBackend(), c, w)


def test_registry_chooses_by_architecture(tmp_path):
    from orangu_b200 import registry

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert registry.model_class(str(tmp_path)) is registry.FiloraxModel


# ---- the plain statement itself
def test_plain_mask_and_sink():
    assert [j for j in range(12) if P.visible(9, j, 4)] == [6, 7, 8, 9] and [j for j in range(6) if P.visible(3, j)] == [0, 1, 2, 3]
    q, k, v = np.zeros((3, 1, 2)), np.ones((3, 1, 2)), np.array([3.0, 6.0, 9.0]).reshape(3, 1, 1)
    np.testing.assert_allclose(P.attend(q, k, v, 1.0)[:, 0], [[3.0], [4.5], [6.0]])
    np.testing.assert_allclose(P.attend(q, k, v, 1.0, window=2)[:, 0], [[3.0], [4.5], [7.5]])
    np.testing.assert_allclose(P.attend(q, k, v, 1.0, sink=[np.log(3.0)])[:, 0], [[0.75], [9 / 5], [3.0]])  # the sink weighs as much as three keys


def test_plain_rotation():
    np.testing.assert_allclose(P.rotate(np.eye(4)[0], 1, 100.0), [np.cos(1), 0, np.sin(1), 0], atol=1e-12)
    np.testing.assert_allclose(P.rotate(np.eye(4)[3], 2, 100.0), [0, -np.sin(0.2), 0, np.cos(0.2)], atol=1e-12)


def test_plain_norm_convolution_and_average():
    np.testing.assert_allclose(P.grouped_norm(np.array([3.0, 4.0, 0.0, 2.0]), np.array([1.0, 2.0, 1.0, 1.0]), 2, 0.0), np.array([3, 8, 0, 0]) / np.sqrt(12.5) + [0, 0, 0, np.sqrt(2)])
    np.testing.assert_allclose(P.input_conv(np.array([[1.0], [10.0], [100.0]]), np.array([[2.0, 3.0, 5.0]]))[:, 0], [6.0, 63.0, 632.0])
    np.testing.assert_allclose(P.depth_average([np.array([1.0]), np.array([10.0])], [0.5, 2.0]), [20.5])


def test_plain_routing():
    """Groups by their best expert, then experts within the best groups; weights are not made to sum to anything."""
    router = {"top": 3, "scale": 2.0, "groups": {"count": 3, "keep": 2}}
    z = np.array([5.0, -9.0, 4.0, 3.9, 1.0, 0.0])
    chosen, weights = P.route(z, router)
    assert chosen == [0, 2, 3]
    np.testing.assert_allclose(weights, 2.0 * np.exp(z[[0, 2, 3]]) / np.exp(z).sum())
    assert P.route(z, dict(router, groups={"count": 3, "keep": 1}, top=2))[0] == [0, 1]
    assert P.route(z, dict(router, groups={"count": 1, "keep": 1}))[0] == [0, 2, 3]
    assert P.route(z, dict(router, groups={"count": 6, "keep": 4}, top=4))[0] == [0, 2, 3, 4]


def test_plain_experts():
    mlp = S.experts(4, 2, 5, groups=2, keep=1, shared=9)
    w, h = P.part(S.values(S.weights(S.config([S.window()], ff=mlp), 7)), "l0.mlp."), np.random.default_rng(8).normal(size=(3, 96))
    got = P.mixture(h, w, mlp)
    ff = lambda p, x: w[p + "down"] @ ((lambda z: z / (1 + np.exp(-z)))(w[p + "gate"] @ x) * (w[p + "up"] @ x))
    for t in range(3):
        z = w["router"] @ h[t]
        g = int(np.argmax(z)) // 2
        s = 1.7 * np.exp(z) / np.exp(z).sum()
        want = s[2 * g] * ff(f"e{2 * g}.", h[t]) + s[2 * g + 1] * ff(f"e{2 * g + 1}.", h[t]) + ff("shared.", h[t]) / (1 + np.exp(-(w["shared.sg"] @ h[t])))
        np.testing.assert_allclose(got[t], want)
