"""Host-side parts of the Givozen design: the oracle's own consistency and the configuration."""

import numpy as np
import pytest

from oracle import givozen as OG
import givozen_cases as GC


def test_rotation_pairs_halves_and_depends_on_distance():
    r = {"base": 500.0, "dims": 12}
    x = np.zeros((1, 1, 16))
    x[..., 1] = 1.0                               # the second pair: dimensions 1 and 7
    y = OG.rotate(x, r, 3)
    a = 3 * 500.0 ** (-1 / 6)
    np.testing.assert_allclose(y[0, 0, [1, 7]], [np.cos(a), np.sin(a)])
    assert not np.any(np.delete(y[0, 0], [1, 7]))
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal((1, 1, 16)), rng.standard_normal((1, 1, 16))
    s = [float((OG.rotate(q, r, 40 + a) * OG.rotate(k, r, 33 + a))[..., :12].sum()) for a in (0, 7)]
    assert s[0] == pytest.approx(s[1])
    np.testing.assert_array_equal(OG.rotate(q, r, 9)[..., 12:], q[..., 12:])


def test_scaling_by_wavelength_has_three_ranges():
    r = {"base": 10000.0, "dims": 32}
    f = OG.rope_frequencies(r)
    g = OG.rope_frequencies(dict(r, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1024}))
    turns = 1024 * f / (2 * np.pi)
    np.testing.assert_allclose(g[turns > 4], f[turns > 4])
    np.testing.assert_allclose(g[turns < 1], f[turns < 1] / 8)
    mid = (turns > 1) & (turns < 4)
    assert mid.any() and np.all((g[mid] < f[mid]) & (g[mid] > f[mid] / 8))
    np.testing.assert_allclose(g[mid], f[mid] / 8 + (turns[mid] - 1) / 3 * (f[mid] - f[mid] / 8))


def test_temperatures_sharpen_flatten_and_turn_around():
    q = np.ones((2, 3, 1))
    k, v = np.array([[[0.0]], [[1.0]]]), np.array([[[0.0]], [[1.0]]])
    out = OG.softmax_attention(q, k, v, 2.0, np.array([0.0, 1.0, -1.0]))[1, :, 0]
    np.testing.assert_allclose(out, [0.5, 1 / (1 + np.exp(-2)), 1 / (1 + np.exp(2))])


def test_poly_norm():
    z = np.array([[1.0, -2.0, 0.5]])
    want = 2 * z / np.sqrt(5.25 / 3) + 3 * z ** 2 / np.sqrt((1 + 16 + 0.0625) / 3) - z ** 3 / np.sqrt((1 + 64 + 0.015625) / 3) + 0.25
    np.testing.assert_allclose(OG.poly_norm(z, (2, 3, -1, 0.25), 0.0), want)
    np.testing.assert_allclose(OG.poly_norm(np.zeros((1, 4)), (2, 3, -1, 0.25), 1e-6), 0.25)


def test_clamped_gate():
    g, u = np.array([9.0, -9.0, 1.0, 1.0]), np.array([0.5, 0.5, 9.0, -9.0])
    s = lambda x: 1 / (1 + np.exp(-x))
    np.testing.assert_allclose(OG.clamped_gate(g, u, 1.5), [1.5 * s(1.702 * 1.5) * 1.5, -9 * s(-1.702 * 9) * 1.5, s(1.702) * 2.5, s(1.702) * -0.5])


def test_weights_are_sigmoids_and_multiply_the_input():
    z = np.array([[2.0, -1.0, 3.0, 0.0]])
    chosen, w = OG.route(z, 2)
    assert chosen.tolist() == [[2, 0]]
    np.testing.assert_allclose(w, [[1 / (1 + np.exp(-3)), 1 / (1 + np.exp(-2))]])
    h = np.array([[1.0, -2.0]])
    W = {"router": np.array([[1.0, 0.0]]), "e0.gate": np.eye(2), "e0.up": np.eye(2) * 2, "e0.down": np.eye(2)}
    x = h / (1 + np.exp(-1))
    np.testing.assert_allclose(OG.mixture(h, W, {"router": {"experts": 1, "top": 1}, "expert": {"limit": 9.0}}), x / (1 + np.exp(-1.702 * x)) * (2 * x + 1))


def test_passes_begin_by_adding():
    """With results of nothing (norms behind the sublayers of factor 0) the stream is what the entries add."""
    cfg = GC.config([GC.attention(mlp=None)] * 3, loop=(1, 2, 3))
    sd = GC.weights(cfg)
    for n in sd:
        if n.endswith("norm1b"):
            sd[n] = sd[n] * 0 - 1
    runs = []
    OG.forward(sd, cfg, [5], runs)
    x0, step = sd["embed"][5:6].astype(float), sd["loop.step"].astype(float)
    want = [x0, x0 + step[0], 2 * x0 + step[0] + step[1], 3 * x0 + step.sum(0), 3 * x0 + step.sum(0)]
    assert len(runs) == 5
    for a, b in zip(runs, want):
        np.testing.assert_allclose(a, np.broadcast_to(b, a.shape))


@pytest.mark.parametrize("name", GC.MODELS)
def test_oracle_is_causal_and_uses_every_tensor(name):
    cfg = GC.MODELS[name]
    sd = GC.weights(cfg)
    toks = GC.prompt(cfg, 24)
    full = OG.forward(sd, cfg, toks)
    np.testing.assert_allclose(OG.forward(sd, cfg, toks[:13]), full[:13], rtol=1e-9, atol=1e-9)
    for n in sd:
        if ".mlp.e" in n or (n[0] == "l" and ".norm2" in n and not cfg["layers"][int(n[1:n.index(".")])]["mlp"]):
            continue                                          # an expert that nobody chose; a norm that nobody needs
        if n.endswith("mlp.act") and cfg["layers"][int(n[1:n.index(".")])]["mlp"]["ff"] == 1:
            continue                                          # nothing but signs is left of one column
        if n.endswith("mix.k.b") and not cfg["layers"][int(n[1:n.index(".")])]["mixer"]["rot"]:
            continue                                          # without rotation the same for all keys of a query
        rng = np.random.default_rng(3)
        changed = dict(sd, **{n: sd[n] * 1.5 + 0.1 * rng.standard_normal(sd[n].shape)})
        assert np.max(np.abs(OG.forward(changed, cfg, toks) - full)) > 1e-5, n


def test_clear_tokens_choose_many_experts():
    """The prompts that the device tests use reach most experts, although close calls are left out."""
    cfg = GC.MODELS["plain"]
    sd = GC.weights(cfg, seed=5)
    toks = GC.prompt(cfg, 170, sd=sd)
    assert len(set(toks)) > 20
    seen, plain = [], OG.route
    OG.route = lambda *a: seen.append(plain(*a)) or seen[-1]
    try:
        OG.forward(sd, cfg, toks)
    finally:
        OG.route = plain
    assert [len(np.unique(c)) >= 4 for c, _ in seen] == [True] * 4


def test_configuration_is_translated():
    from versenext_b200.givozen import composed_config
    out = composed_config(GC.MODELS["plain"], {})
    assert out["post_norm"] is True and out["tie_weights"] is True and out["norm_eps"] == 1e-4 and "norm_weight" not in out
    assert out["loop"] == {"start": 1, "stop": 3, "times": 2, "entry": "add"}
    a, b, c, d = out["layers"]
    assert a == {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 24, "vdim": 16, "scale": 0.3, "bias": True, "out_bias": False,
                 "temperature": True, "output_gate": "head", "mlp_hidden": 48, "mlp_act": "poly_norm",
                 "rope": {"dims": 16, "base": 1000.0, "scaling": {"kind": "wavelength", "factor": 3.0, "low": 1.0, "high": 4.0, "original": 200.0}}}
    assert b["experts"] == {"count": 7, "top": 3, "score": "sigmoid", "weight": "input", "shared": {"hidden": 40, "limit": 2.1}}
    assert (b["mlp_hidden"], b["mlp_act"], b["mlp_limit"]) == (24, "clamped", 1.2)
    assert c["heads"] == 2 and "mlp_hidden" not in d
    ones = composed_config(GC.MODELS["ones"], {})
    assert "shared" not in ones["layers"][1]["experts"] and "rope" not in ones["layers"][1] and ones["loop"]["times"] == 1
    assert "loop" not in composed_config(GC.MODELS["no_loop"], {})
    assert composed_config(GC.MODELS["other_order"], {})["layers"][0]["rope"]["scaling"] is None
    with pytest.raises(ValueError):
        composed_config(GC.config([dict(GC.attention(), type="other")]), {})
    with pytest.raises(ValueError):
        composed_config(GC.config([GC.attention(mlp={"kind": "sparse", "ff": 8})]), {})


def test_registry():
    import versenext_b200 as vn
    assert vn.registry.model_class("Givozen") is vn.GivozenLM and "Givozen" in vn.registry.architectures()
