"""Host-side parts of the Bozasun design: the oracle's own consistency and the configuration."""

import numpy as np
import pytest

from oracle import bozasun as OB
import bozasun_cases as BC


def test_recurrence_continues_and_has_a_closed_form():
    rng = np.random.default_rng(0)
    x, B, C, dt = rng.standard_normal((9, 3)), rng.standard_normal((9, 5)), rng.standard_normal((9, 5)), rng.uniform(0.1, 1, 9)
    y, S = OB.ssm(x, B, C, dt, -0.7, 0.4)
    y1, S1 = OB.ssm(x[:4], B[:4], C[:4], dt[:4], -0.7, 0.4)
    y2, S2 = OB.ssm(x[4:], B[4:], C[4:], dt[4:], -0.7, 0.4, S1)
    np.testing.assert_allclose(np.concatenate([y1, y2]), y, rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)
    run = np.cumsum(-0.7 * dt)                    # the token's own decay does not touch its own contribution
    want = [0.4 * x[t] + sum(np.exp(run[t] - run[j]) * dt[j] * (C[t] @ B[j]) * x[j] for j in range(t + 1)) for t in range(9)]
    np.testing.assert_allclose(y, want, rtol=1e-10)


def test_rotation_is_interleaved_scaled_and_depends_on_distance():
    rot = {"base": 500.0, "dims": 12, "scaling": {"factor": 4.0}}
    np.testing.assert_allclose(OB.rope_frequencies(rot), 500.0 ** (-np.arange(6) / 6) / 4)
    x = np.zeros((1, 1, 16))
    x[..., 2] = 1.0                               # the second pair's first member turns into both members
    y = OB.rotate(x, rot, 3)
    a = 3 * 500.0 ** (-1 / 6) / 4
    np.testing.assert_allclose(y[0, 0, 2:4], [np.cos(a), np.sin(a)])
    assert not np.any(np.delete(y[0, 0], [2, 3]))
    rng = np.random.default_rng(1)
    q, k = rng.standard_normal((1, 1, 16)), rng.standard_normal((1, 1, 16))
    s = [float((OB.rotate(q, rot, 40 + a) * OB.rotate(k, rot, 33 + a))[..., :12].sum()) for a in (0, 7)]
    assert s[0] == pytest.approx(s[1])
    np.testing.assert_array_equal(OB.rotate(q, rot, 9)[..., 12:], q[..., 12:])


def test_chunks_begin_anew():
    assert OB.same_chunk(5, 2).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    v = np.arange(5.0)[:, None, None]
    out = OB.softmax_attention(np.zeros((5, 1, 2)), np.zeros((5, 1, 2)), v, 1.0, OB.same_chunk(5, 3))[:, 0, 0]
    np.testing.assert_allclose(out, [0, 0.5, 1, 3, 3.5])


def test_scores_are_capped():
    q, k, v = np.full((2, 1, 1), 100.0), np.array([[[1.0]], [[-1.0]]]), np.array([[[0.0]], [[1.0]]])
    out = OB.softmax_attention(q, k, v, 1.0, OB.causal(2), 2.0)[1, 0, 0]
    assert out == pytest.approx(np.exp(-2) / (np.exp(2) + np.exp(-2)))


def test_router_groups_correction_and_weights():
    p = np.array([[0.30, 0.05, 0.22, 0.20, 0.13, 0.10]])
    z, none = np.log(p), np.zeros(6)
    chosen, w = OB.route(z, none, 2, 1, 1)
    assert chosen.tolist() == [[0, 2]] and w[0] == pytest.approx([0.30, 0.22])
    # two of three groups of neighbours (best members 0.30, 0.22, 0.13): the last one is out
    assert OB.route(z, none, 4, 3, 2)[0].tolist() == [[0, 2, 3, 1]]
    # the correction moves the choice, also between groups, but not the weights
    chosen, w = OB.route(z, np.array([-0.4, 0, 0, 0, 0, 0.5]), 2, 3, 2)
    assert chosen.tolist() == [[5, 2]] and w[0] == pytest.approx([0.10, 0.22])
    # negative choice scores still beat those of groups that are out
    assert OB.route(z, np.full(6, -1.0), 2, 3, 1)[0].tolist() == [[0, 1]]


def test_identity_experts_return_their_input():
    h = np.array([[1.0, -2.0]])
    W = {"router": np.array([[0.0, 0.0], [5.0, 0.0]]), "correction": np.zeros(2), "e0.gate": np.ones((3, 2)), "e0.up": np.ones((3, 2)), "e0.down": np.ones((2, 3))}
    cfg = {"router": {"experts": 1, "identity": 1, "top": 1, "groups": {"count": 1, "keep": 1}}}
    np.testing.assert_allclose(OB.experts(h, W, cfg), h / (1 + np.exp(-5)))


def test_gate_comes_before_the_norm_of_each_part():
    y = OB.grouped_rms(np.array([[3.0, 3.0, 0.5, -0.5]]), 2, 0.0)
    np.testing.assert_allclose(y, [[1, 1, 1, -1]])


@pytest.mark.parametrize("name", BC.MODELS)
def test_oracle_is_causal_and_uses_every_tensor(name):
    cfg = BC.MODELS[name]
    sd = BC.weights(cfg)
    toks = BC.prompt(cfg, 24)
    full = OB.forward(sd, cfg, toks)
    np.testing.assert_allclose(OB.forward(sd, cfg, toks[:13]), full[:13], rtol=1e-9, atol=1e-9)
    for n in sd:
        layer = cfg["layers"][int(n[1:n.index(".")])] if n[0] == "l" else {"mixer": {}}
        if (layer["mixer"].get("mask") or {}).get("size") == 1 and n[3:].startswith(("mix.q", "mix.k")):
            continue                                          # a chunk of one: the keys do not matter
        if ".mlp.e" in n or n.endswith("correction"):
            continue                                          # an expert that nobody chose; see the next test
        changed = dict(sd, **{n: sd[n] * 1.5 + 0.1})
        assert np.max(np.abs(OB.forward(changed, cfg, toks) - full)) > 1e-5, n


def test_clear_tokens_choose_many_experts():
    """The prompts that the device tests use reach every kind of expert, although close calls are left out."""
    cfg = BC.MODELS["plain"]
    sd = BC.weights(cfg, seed=5)
    toks = BC.prompt(cfg, 170, sd=sd)
    assert len(set(toks)) > 20
    seen, plain = [], OB.route
    OB.route = lambda *a: seen.append(plain(*a)) or seen[-1]
    try:
        OB.forward(sd, cfg, toks)
    finally:
        OB.route = plain
    assert all(len(np.unique(c)) >= 5 and c.max() >= n for (c, _), n in zip(seen, (7, 5)))


def test_configuration_is_translated():
    from versenext_b200.bozasun import composed_config
    out = composed_config(BC.MODELS["plain"], {})
    assert out["norm_weight"] == "plain" and out["norm_eps"] == 1e-4 and out["token_side"] == 10
    a, b, c, d = out["layers"]
    assert a == {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 24, "vdim": 16, "scale": 0.3, "bias": True, "qk_norm": True, "chunk": 37,
                 "softcap": 6.0, "rope": {"dims": 16, "base": 1000.0, "interleaved": True, "scaling": {"kind": "linear", "factor": 2.5}},
                 "mlp_hidden": 48, "mlp_act": "silu"}
    assert b == {"mixer": "mamba2", "heads": 6, "vdim": 20, "state": 12, "groups": 3, "norm_groups": 2, "conv": 4, "mlp_hidden": 24, "mlp_act": "silu",
                 "experts": {"count": 7, "identity": 3, "top": 3, "groups": 5, "keep": 2, "correction": True}}
    assert c["rot_dim"] == 8 and c["output_gate"] == "element" and not c["sink"] and c["rope"]["dims"] == 8 and c["rope"]["scaling"] is None
    assert "mlp_hidden" not in d and d["chunk"] == 64
    with pytest.raises(ValueError):
        composed_config(BC.config([dict(BC.latent(), type="other")]), {})
    with pytest.raises(ValueError):
        composed_config(BC.config([dict(BC.latent(), mlp={"kind": "sparse", "ff": 8})]), {})


def test_registry():
    import versenext_b200 as vn
    assert vn.registry.model_class("Bozasun") is vn.BozasunLM and "Bozasun" in vn.registry.architectures()
