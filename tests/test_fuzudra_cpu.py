"""Host-side parts of the Fuzudra design: the oracle's own consistency, configuration, weights files, scheduling."""

import json
import struct

import numpy as np
import pytest

from oracle import fuzudra as OF
import fuzudra_cases as FC


def test_recurrences_continue_from_their_state():
    """A scan cut in two, the second half started from the first one's state, is the whole scan."""
    rng = np.random.default_rng(0)
    x, dt, B, C = rng.standard_normal((9, 4)), rng.random((9, 4)), rng.standard_normal((9, 3)), rng.standard_normal((9, 3))
    A, D = -rng.random((4, 3)), rng.standard_normal(4)
    y, S = OF.selective_scan(x, dt, B, C, A, D)
    y1, S1 = OF.selective_scan(x[:5], dt[:5], B[:5], C[:5], A, D)
    y2, S2 = OF.selective_scan(x[5:], dt[5:], B[5:], C[5:], A, D, S1)
    np.testing.assert_allclose(np.concatenate([y1, y2]), y, rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)
    q, k, v = rng.standard_normal((9, 5)), rng.standard_normal((9, 5)), rng.standard_normal((9, 2))
    g, b = rng.random((9, 5)), rng.random(9)
    o, S = OF.delta_rule(q, k, v, g, b)
    o1, S1 = OF.delta_rule(q[:4], k[:4], v[:4], g[:4], b[:4])
    o2, S2 = OF.delta_rule(q[4:], k[4:], v[4:], g[4:], b[4:], S1)
    np.testing.assert_allclose(np.concatenate([o1, o2]), o, rtol=1e-12)
    np.testing.assert_allclose(S2, S, rtol=1e-12)


def test_delta_rule_reads_back_what_it_wrote():
    """beta = 1, no decay, orthonormal keys: the read-out of a key is the value written under it, its own token included."""
    k = np.eye(4)
    v = np.arange(8.0).reshape(4, 2) + 1
    o, S = OF.delta_rule(k, k, v, np.ones((4, 4)), np.ones(4))
    np.testing.assert_allclose(o, v)
    np.testing.assert_allclose(S, v)


@pytest.mark.parametrize("name", FC.MODELS)
def test_oracle_is_causal_and_uses_every_tensor(name):
    cfg = FC.MODELS[name]
    sd = FC.weights(cfg)
    toks = FC.prompt(cfg, 24)
    full = OF.forward(sd, cfg, toks)
    np.testing.assert_allclose(OF.forward(sd, cfg, toks[:13]), full[:13], rtol=1e-9, atol=1e-9)
    for n in sd:
        changed = dict(sd, **{n: sd[n] * 1.5 + 0.1})
        assert np.max(np.abs(OF.forward(changed, cfg, toks) - full)) > 1e-4, n


def test_layer_runs_of_a_loop():
    cfg = FC.MODELS["loop_inside"]
    assert OF.layer_runs(cfg) == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2), (3, None)]
    assert OF.layer_runs(FC.MODELS["plain"]) == [(0, None), (1, None), (2, None)]


def test_configuration_is_translated():
    from versenext_b200.fuzudra import composed_config
    cfg = FC.MODELS["loop_inside"]
    sd = FC.weights(cfg, rank_a=9, rank_g=17)
    out = composed_config(cfg, {n: a.shape for n, a in sd.items()})
    assert out["loop"] == {"start": 1, "stop": 3, "times": 3} and out["dim"] == 64 and out["norm_eps"] == 1e-4
    assert out["layers"][0] == {"mixer": "channel_delta", "heads": 4, "kv_heads": 2, "dim": 32, "vdim": 20, "conv": 3,
                                "decay_rank": 9, "gate_rank": 17, "mlp_hidden": 40, "mlp_act": "gelu_tanh"}
    assert out["layers"][1]["window"] == 5 and "mlp_hidden" not in out["layers"][2]
    bad = FC.config([dict(FC.mamba(), type="other")])
    with pytest.raises(ValueError):
        composed_config(bad, {})


def write_model(path, cfg, sd):
    """A model directory: config.json and bfloat16 tensors."""
    head, blobs, at = {}, [], 0
    for n, a in sd.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[n] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        at += len(raw)
        blobs.append(raw)
    h = json.dumps(head).encode()
    (path / "config.json").write_text(json.dumps(cfg))
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def test_safetensors_file(tmp_path):
    from versenext_b200.safetensors_file import SafetensorsFile
    cfg = FC.MODELS["unaligned"]
    sd = FC.weights(cfg)
    write_model(tmp_path, cfg, sd)
    with SafetensorsFile(str(tmp_path / "model.safetensors")) as f:
        assert f.shapes() == {n: a.shape for n, a in sd.items()}
        for _ in range(2):
            got = dict(f)
            assert set(got) == set(sd)
            for n in sd:
                np.testing.assert_array_equal(got[n], sd[n])


def test_registry():
    import versenext_b200 as vn
    assert vn.registry.model_class("Fuzudra") is vn.FuzudraLM
    with pytest.raises(ValueError):
        vn.registry.model_class("NoSuchDesign")


class FakeModel:
    """A next-token rule instead of a model: token t after a prefix of n tokens is (sum of the prefix + n) mod 50."""
    vocab_size = 50

    class ctx:
        pass

    def __init__(self):
        self.text = {}
        self.calls = []

    def new_cache(self, max_batch, max_seq, pool_tokens=0):
        model = self

        class Cache:
            pages = (pool_tokens // 64 if pool_tokens else max_batch * -(-max_seq // 64), 0)

            def reset_seq(self, slot):
                model.text[slot] = []
        return Cache()

    def forward_ragged(self, cache, slots, counts, tokens, rows):
        self.calls.append(list(counts))
        out, r0 = [], 0
        for s, n in zip(slots, counts):
            for i in range(n):
                self.text[s].append(int(tokens[r0 + i]))
                if r0 + i in rows:
                    out.append((sum(self.text[s]) + len(self.text[s])) % 50)
            r0 += n
        return np.eye(50, dtype=np.float32)[out] if out else None

    def check(self):
        pass


def test_scheduler_mixes_portions_and_single_tokens(monkeypatch):
    from versenext_b200 import sampling, serving

    class Arr(np.ndarray):
        def numpy(self):
            return np.asarray(self)
    monkeypatch.setattr(sampling, "argmax", lambda ctx, lg: np.argmax(lg, -1).view(Arr))
    prompts = [list(range(1, n + 1)) for n in (5, 1, 30, 12, 7)]
    limits = [4, 9, 3, 1, 6]

    def stream(p, n, eos=None):
        t = list(p)
        for _ in range(n):
            t.append((sum(t) + len(t)) % 50)
            if t[-1] == eos:
                break
        return t[len(p):]
    for slots, pool, budget in ((2, 0, 8), (5, 0, 2048), (3, 128, 6), (1, 0, 2)):
        m = FakeModel()
        eng = serving.BatchEngine(m, max_batch=slots, max_seq=64, pool_tokens=pool, step_tokens=budget)
        got = eng.run(prompts, limits)
        assert [list(g) for g in got] == [stream(p, n) for p, n in zip(prompts, limits)]
        assert all(sum(c) <= budget and len(c) <= slots for c in m.calls)
        assert any(1 in c and max(c) > 1 for c in m.calls) or slots == 1
        assert eng.free_slots == slots and not eng.live
    eos = stream(prompts[4], 6)[2]
    eng = serving.BatchEngine(FakeModel(), max_batch=2, max_seq=64)
    assert [list(g) for g in eng.run(prompts, 6, eos_id=eos)] == [stream(p, 6, eos) for p in prompts]
    with pytest.raises(RuntimeError):
        eng.run([list(range(60))], 10)
    eng = serving.BatchEngine(FakeModel(), max_batch=2, max_seq=256, pool_tokens=64)
    with pytest.raises(RuntimeError):
        eng.run([list(range(80))], 4)


def test_step_runner_rejects_bad_steps():
    from versenext_b200.serving import StepRunner
    r = StepRunner(FakeModel(), max_batch=2, max_seq=64)
    with pytest.raises(ValueError):
        r.step([("a", [1], []), ("a", [2], [])])
    with pytest.raises(ValueError):
        r.step([("a", [], [])])
    with pytest.raises(RuntimeError):
        r.step([("a", [1], []), ("b", [2], []), ("c", [3], [])])
    r.step([("a", [1, 2], []), ("b", [2], [])])
    assert r.length == {"a": 2, "b": 1} and r.free_slots == 0
    r.end("a")
    assert r.live == ["b"] and r.free_slots == 1
