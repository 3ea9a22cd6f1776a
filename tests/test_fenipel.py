"""Fenipel without a GPU: configuration and weight reading, the registry, and the plain statement the GPU tests lean on."""
import json
import os

import numpy as np
import pytest

import fenipel_make as F
import fenipel_plain as P


class FakeLib:
    """Stands in for the library: keeps the description it is given."""

    def ob_layered_model_create(self, ctx, desc, out):
        from orangu_b200 import capi

        d = desc._obj
        self.blocks = [d.layers[i] for i in range(d.n_layer)]
        self.desc, self.capi = d, capi
        return 0

    def ob_model_destroy(self, h):
        pass


class FakeBackend:
    def __init__(self):
        self._h, self._lib = None, FakeLib()


CFG = F.config([F.latent(heads=2, window=5), F.retention(heads=4, rot_dims=8)], ff=[None, 40])


def test_description_follows_the_configuration():
    from orangu_b200.fenipel import GLU_ALPHA, FenipelModel

    be = FakeBackend()
    m = FenipelModel(be, CFG, F.weights(CFG, 1), dtype="float32", max_seq_len=70, max_batch_tokens=9, kv_pool_tokens=64, state_slots=3)
    d, (a, b) = be._lib.desc, be._lib.blocks
    assert (d.n_vocab, d.n_embd, d.n_layer, d.side_dim, d.compute_f32) == (96, 88, 2, 12, 1)
    assert (d.max_seq_len, d.max_batch_tokens, d.kv_pool_tokens, d.n_state_slots) == (70, 9, 64, 3)
    assert d.rms_eps == pytest.approx(1e-5) and d.final_gain == pytest.approx(1.3, rel=4e-3)
    assert (a.mixer.n_head, a.mixer.dim, a.mixer.rot_dim, a.mixer.vdim, a.mixer.kv_rank, a.mixer.window) == (2, 24, 16, 20, 40, 5)
    assert (a.mixer.rot_dims, a.mixer.rot_interleaved, a.mixer.rot_base) == (16, 1, 3000.0) and a.n_ff == 0
    assert (a.mixer.wq.out_dim, a.mixer.wq.in_dim, a.mixer.w_dkv.out_dim) == (2 * 40, 88, 56)
    assert (b.mixer.n_head, b.mixer.dim, b.mixer.vdim, b.mixer.rot_dims, b.mixer.rot_interleaved) == (4, 24, 36, 8, 0)
    assert b.n_ff == 40 and b.glu_limit == pytest.approx(0.9) and b.glu_alpha == pytest.approx(GLU_ALPHA)
    assert m.cache_widths(0) == (40, 16) and m.state_shape(1) == (4, 24, 36)


@pytest.mark.parametrize("change, message", [
    (lambda c, w: c["layers"][0].update(type="other"), "no mixer"),
    (lambda c, w: c["layers"][1]["mlp"].update(kind="other"), "no feed-forward"),
    (lambda c, w: w.pop("l1.mix.k"), "no tensor l1.mix.k"),
    (lambda c, w: c["layers"][0]["mixer"].update(kv_rank=48), "expected"),
    (lambda c, w: c["layers"][1]["mixer"].update(decay=[0.5]), "heads of 4"),
])
def test_what_does_not_fit_is_refused(change, message):
    from orangu_b200.fenipel import FenipelModel

    c, w = json.loads(json.dumps(CFG)), F.weights(CFG, 1)
    change(c, w)
    with pytest.raises(ValueError, match=message):
        FenipelModel(FakeBackend(), c, w)


def test_safetensors_round_trip_and_damage(tmp_path):
    from orangu_b200.safetensors import SafetensorsFile, from_bf16, save, to_bf16

    p = str(tmp_path / "m.safetensors")
    x = np.random.default_rng(0).normal(size=(3, 5)).astype(np.float32)
    save(p, {"a": to_bf16(x), "b": x, "i": np.arange(4, dtype=np.int32), "s": to_bf16(np.float32(0.75)).reshape(())})
    t = SafetensorsFile(p)
    assert (t.bf16("a") == t.bf16("b")).all() and (t.bf16("a", (3, 5)) == F.bf16_bits(x)).all()
    assert (t.f32("b") == x).all() and (t.raw("i") == np.arange(4)).all() and t.f32("s", ()).shape == () and float(t.f32("s")) == 0.75
    assert (from_bf16(t.bf16("a")) == t.f32("a")).all() and "c" not in t
    with pytest.raises(ValueError, match="expected"):
        t.raw("a", (5, 3))
    with pytest.raises(ValueError, match="no tensor"):
        t.raw("c")
    blob = open(p, "rb").read()
    open(p, "wb").write(blob[:-8])
    with pytest.raises(ValueError, match="offsets"):
        SafetensorsFile(p).raw("s")
    open(p, "wb").write(b"\xff" * 16)
    with pytest.raises(ValueError, match="header"):
        SafetensorsFile(p)


def test_registry_chooses_by_architecture(tmp_path):
    from orangu_b200 import registry
    from orangu_b200.gguf import write_gguf
    from orangu_b200 import synth

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert registry.model_class(str(tmp_path)) is registry.FenipelModel
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="Unheard"):
        registry.model_class(str(tmp_path))
    g = str(tmp_path / "m.gguf")
    write_gguf(g, synth.CONFIGS["tiny"], synth.model_tensors(synth.CONFIGS["tiny"], seed=1))
    assert registry.model_class(g) is registry.LlamaModel


def test_command_lines_explain_themselves():
    import subprocess, sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for cmd in (["-m", "orangu_b200", "generate", "--help"], ["-m", "orangu_b200", "trace", "--help"], [os.path.join(root, "bin", "trace_run"), "--help"]):
        r = subprocess.run([sys.executable, *cmd], cwd=root, capture_output=True, text=True)
        assert r.returncode == 0 and "--model" in r.stdout


def test_library_without_the_quantized_kernels(tmp_path):
    """The part a layered model needs links, loads and exports everything; what is left out answers with a status."""
    import subprocess, sys

    from orangu_b200 import build

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    lib = build.build_cuda(quantized=False)
    code = ("import ctypes as C, sys\nfrom orangu_b200 import capi\ncapi.select(sys.argv[1])\nL = capi.load()\n"
            "d, h = capi.ModelDesc(), C.c_void_p()\n"
            "assert L.ob_model_create(None, C.byref(d), C.byref(h)) == -2 and b'without the quantized' in L.ob_last_error(None)\n"
            "assert L.ob_layered_model_create(None, None, C.byref(h)) == -1 and L.ob_quantize_act(None, None, 1, 0, None, None, None) == -2\n"
            "print(capi.lib_path())")
    r = subprocess.run([sys.executable, "-c", code, lib], cwd=root, capture_output=True, text=True)
    assert r.returncode == 0 and r.stdout.strip() == lib, r.stderr


# ---- the plain statement itself
def test_plain_retention_equals_its_unrolled_sum():
    cfg = F.config([F.retention(heads=2, dim=8, vdim=6, rot_dims=4)], width=16, ff=None, side=0)
    w, mx = P.part(F.values(F.weights(cfg, 3)), "l0.mix."), cfg["layers"][0]["mixer"]
    h = np.random.default_rng(4).normal(size=(9, 16))
    out, _ = P.retention(h, w, mx, 1e-5)
    rot = lambda x, p: P.rotate(x, p, mx["rot"]["base"], 4, False)
    for t in range(9):
        o = np.zeros((2, 6))
        for s in range(t + 1):
            q, k = rot((w["q"] @ h[t]).reshape(2, 8), t), rot((w["k"] @ h[s]).reshape(2, 8), s) * 8 ** -0.5
            o += (np.array(mx["decay"]) ** (t - s) * (q * k).sum(1))[:, None] * (w["v"] @ h[s]).reshape(2, 6)
        g = w["g"] @ h[t]
        want = w["o"] @ (P.over_rms(o, 1e-5).reshape(-1) * g / (1 + np.exp(-g)))
        np.testing.assert_allclose(out[t], want, rtol=1e-9, atol=1e-12)


def test_plain_window_and_rotation():
    assert [j for j in range(12) if P.visible(9, j, 4)] == [6, 7, 8, 9] and [j for j in range(4) if P.visible(2, j, 9)] == [0, 1, 2]
    x = np.random.default_rng(5).normal(size=(2, 10))
    for inter in (False, True):
        a, b = P.rotate(x, 7, 100.0, 6, inter), P.rotate(x, 3, 100.0, 6, inter)
        np.testing.assert_allclose(a[:, 6:], x[:, 6:])
        np.testing.assert_allclose((a[0] * b[1]).sum(), (P.rotate(x, 4, 100.0, 6, inter)[0] * x[1]).sum())  # only the distance counts
        assert not np.allclose(a, P.rotate(x, 7, 100.0, 6, not inter))
