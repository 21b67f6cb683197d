"""Host-side parts of the Musutar design: the oracle's own consistency and the configuration."""

import numpy as np
import pytest

from oracle import musutar as OM
import musutar_cases as MC


def test_state_continues_and_decays():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 5)), rng.standard_normal((9, 5)), rng.standard_normal((9, 2))
    o, S = OM.decayed_state(q, k, v, 0.7)
    o1, S1 = OM.decayed_state(q[:4], k[:4], v[:4], 0.7)
    o2, S2 = OM.decayed_state(q[4:], k[4:], v[4:], 0.7, S1)
    np.testing.assert_allclose(np.concatenate([o1, o2]), o, rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)
    # the closed form: o_t = sum_j decay^(t - j) (q_t . k_j) v_j, the token itself undecayed
    want = [sum(0.7 ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)) for t in range(9)]
    np.testing.assert_allclose(o, want, rtol=1e-10)


def test_rotation_depends_on_distance_only_and_keeps_the_rest():
    rng = np.random.default_rng(1)
    rot = {"base": 500.0, "dims": 12, "scaling": MC.yarn()}
    f, amp = OM.rope_frequencies(rot)
    assert len(f) == 6 and amp == pytest.approx(0.1 * np.log(3.0) + 1)
    # fast pairs keep their frequency, slow ones are divided by the factor
    plain = 500.0 ** (-2.0 * np.arange(6) / 12)
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 3.0) and np.all(np.diff(f) < 0)
    q, k = rng.standard_normal((1, 1, 16)), rng.standard_normal((1, 1, 16))
    s = [float((OM.rotate(q, rot, 40 + a) * OM.rotate(k, rot, 33 + a))[..., :12].sum()) for a in (0, 7)]
    assert s[0] == pytest.approx(s[1])
    np.testing.assert_array_equal(OM.rotate(q, rot, 9)[..., 12:], q[..., 12:])


def test_window_counts_itself():
    q = np.zeros((5, 1, 2))
    v = np.arange(5.0)[:, None, None]
    out = OM.windowed_attention(q, np.zeros((5, 1, 2)), v, 1.0, 2)[:, 0, 0]
    np.testing.assert_allclose(out, [0, 0.5, 1.5, 2.5, 3.5])


def test_streams_are_mixed_from_to():
    xs = np.stack([np.full((1, 2), 1.0), np.full((1, 2), 10.0)])
    mix = np.array([[1.0, 5.0], [0.0, 1.0]])                  # stream 0 also goes to stream 1
    got = OM.write_streams(xs, mix, np.array([0.0, 2.0]), np.full((1, 2), 100.0))
    np.testing.assert_allclose(got[:, 0, 0], [1.0, 215.0])
    assert OM.read_streams(xs, np.array([1.0, 0.5]))[0, 0] == 6.0


@pytest.mark.parametrize("name", MC.MODELS)
def test_oracle_is_causal_and_uses_every_tensor(name):
    cfg = MC.MODELS[name]
    sd = MC.weights(cfg)
    toks = MC.prompt(cfg, 24)
    full = OM.forward(sd, cfg, toks)
    np.testing.assert_allclose(OM.forward(sd, cfg, toks[:13]), full[:13], rtol=1e-9, atol=1e-9)
    for n in sd:
        if cfg["layers"][0]["mixer"].get("mask") == {"size": 1} and n.startswith("l0.mix.") and n[7] in "qk":
            continue                                          # a window of one: the keys do not matter
        changed = dict(sd, **{n: sd[n] * 1.5 + 0.1})
        assert np.max(np.abs(OM.forward(changed, cfg, toks) - full)) > 1e-5, n


def test_configuration_is_translated():
    from versenext_b200.musutar import composed_config
    out = composed_config(MC.MODELS["plain"], {})
    assert out["norm"] == "layer" and out["norm_eps"] == 1e-4 and out["streams"] == 3 and out["input_conv"] == 3 and out["residual_gate"]
    a, b = out["layers"][1], out["layers"][2]
    assert a == {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 24, "vdim": 16, "scale": 0.25, "output_gate": True, "window": 37,
                 "conv": 3, "rope": {"base": 1000.0, "dims": 16, "scaling": MC.yarn()}, "mlp_hidden": 48, "mlp_act": "relu2"}
    assert b["kv_from"] == 1 and b["window"] == 9 and "mlp_hidden" not in b
    assert out["layers"][0]["decay"] == MC.MODELS["plain"]["layers"][0]["mixer"]["decay"]
    with pytest.raises(ValueError):
        composed_config(MC.config([dict(MC.lightning(), type="other")]), {})
    with pytest.raises(ValueError):
        composed_config(MC.config([dict(MC.lightning(), mlp={"kind": "sparse", "ff": 8})]), {})


def test_registry():
    import versenext_b200 as vn
    assert vn.registry.model_class("Musutar") is vn.MusutarLM and "Musutar" in vn.registry.architectures()
