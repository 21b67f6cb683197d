"""The Fuzudra design on the device against the plain NumPy restatement (oracle/fuzudra.py), in fp32 and bf16."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import fuzudra as OF
import fuzudra_cases as FC
from fuzudra_cases import TOL, Expected, build, err, prompt
from test_fuzudra_cpu import write_model

pytestmark = pytest.mark.gpu
DTYPES = ["f32", "bf16"]


def whole(m, toks):
    """Logits of every position from one forward over an empty cache."""
    out = m.forward_cached(np.asarray(toks)[None], m.new_cache(1, len(toks))).numpy()[0]
    m.check()
    return out


def in_portions(m, toks, sizes):
    cache = m.new_cache(1, len(toks))
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - at)
        out.append(m.forward_ragged(cache, [0], [n], toks[at:at + n], range(n)).numpy())
        at, i = at + n, i + 1
    m.check()
    return np.concatenate(out)


MECHANISMS = {
    "latent": FC.latent(), "latent_one_head": FC.latent(heads=1, dim=5, vdim=7, kv_rank=3, window=2),
    "latent_wide": FC.latent(heads=6, dim=64, vdim=48, kv_rank=160, window=100, scale=0.125, ff=0),
    "latent_rank_beyond_tiles": FC.latent(heads=2, dim=16, vdim=16, kv_rank=520, window=20),
    "latent_many_heads": FC.latent(heads=20, dim=16, vdim=16, kv_rank=96, window=65),
    "mamba": FC.mamba(), "mamba_one_tap": FC.mamba(conv=1), "mamba_long_filter": FC.mamba(inner=48, conv=9, state=1, dt_rank=17),
    "mamba_wide_state": FC.mamba(inner=40, state=65, dt_rank=2, ff=16), "mamba_16": FC.mamba(inner=128, state=16, dt_rank=8),
    "delta": FC.delta(), "delta_wide": FC.delta(heads=2, kv_heads=1, dim=128, vdim=72), "delta_one_tap": FC.delta(conv=1, dim=9, vdim=5),
    "delta_dim_160": FC.delta(heads=1, kv_heads=1, dim=160, vdim=33, conv=6), "delta_dim_96": FC.delta(heads=2, kv_heads=2, dim=96, vdim=96, ff=20),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_alone(name, dtype):
    cfg = FC.config([MECHANISMS[name]])
    sd = FC.weights(cfg, seed=3)
    toks = prompt(cfg, 150)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [70, 1, 2, 1, 40, 1]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", FC.MODELS)
def test_models_whole_portions_and_decoding(name, dtype):
    cfg = FC.MODELS[name]
    sd = FC.weights(cfg, seed=5)
    toks = prompt(cfg, 170)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    res = m.residuals(toks)
    assert len(res) == len(want.runs)
    for i, (a, b, tol) in enumerate(zip(res, want.runs, want.run_tol)):
        assert err(a, b) < tol[dtype], i
    want.check(whole(m, toks), dtype)
    for sizes in ([2], [1], [3, 2, 61, 1, 5], [64], [63, 65], [127, 1, 1, 40], [100] + [1] * 70):
        want.check(in_portions(m, toks, sizes), dtype, what=sizes)


ASKS, ANSWERS, FILLER = 95, 96, 90


def edge_model(window):
    """One latent layer in which token ASKS finds token ANSWERS and nothing else: the first half of an embedding is what
    a token asks for, the second half what it offers, and these two share one vector."""
    cfg = FC.config([FC.latent(heads=2, dim=32, vdim=32, kv_rank=64, window=window, scale=1.0, ff=0)], width=64)
    sd = FC.weights(cfg, seed=9)
    eye, off = np.eye(32, dtype=np.float32), np.zeros((32, 32), np.float32)
    sd["embed"] = OF.bf16(sd["embed"] * 8)                          # the position vector is small beside it
    sd["embed"][ANSWERS, 32:] = sd["embed"][ASKS, :32]
    sd["l0.norm1"] = sd["l0.norm1"] * 0
    sd["l0.mix.q"] = np.tile(np.concatenate([eye, off], 1), (2, 1))
    sd["l0.mix.dkv"] = np.eye(64, dtype=np.float32)
    sd["l0.mix.dkv.norm"] = np.ones(64, np.float32)
    sd["l0.mix.uk"] = np.tile(np.concatenate([off, eye], 1), (2, 1))
    sd["l0.mix.sink"] = np.array([3.0, 4.0], np.float32)
    sd["l0.mix.o"] = OF.bf16(sd["l0.mix.o"] * 8)
    return cfg, sd


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100])
def test_window_edges(window, dtype):
    """The answer at the last distance that is seen, and just beyond it: in a prompt, in a portion, and when the asking
    token is decoded alone, which stands at several offsets from a page's border."""
    cfg, sd = edge_model(window)
    m = build(cfg, sd, dtype)
    base = prompt(cfg, 2 * window + 140) % FILLER
    for q in (window + 62, window + 63, window + 64, window + 70):
        logits = {}
        for dist in (window - 1, window):
            toks = base[:q + 1].copy()
            toks[q] = ASKS
            if dist > 0:
                toks[q - dist] = ANSWERS
            want = Expected(sd, cfg, toks)
            for got in (whole(m, toks)[-1:], in_portions(m, toks, [q, 1])[-1:], in_portions(m, toks, [q - 4, 5])[-1:]):
                want.check(got, dtype, slice(q, q + 1), (q, dist))
            logits[dist] = want.logits[-1:]
        if window > 1:      # the case means something: the answer weighs
            assert err(logits[window - 1], logits[window]) > 3 * want.tol["bf16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_counts_once_and_unscaled(dtype):
    """Sinks far above, near and far below the scores, and a scale far from one."""
    cfg = FC.config([FC.latent(heads=4, dim=16, vdim=16, kv_rank=32, window=20, scale=0.05)])
    sd = FC.weights(cfg, seed=4)
    sd["l0.mix.sink"] = np.array([-20.0, 0.0, 4.0, 25.0], np.float32)
    toks = prompt(cfg, 40)
    m = build(cfg, sd, dtype)
    want = Expected(sd, cfg, toks)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [1]), dtype)
    for wrong in (0.05, 0.0):
        other = OF.forward(dict(sd, **{"l0.mix.sink": sd["l0.mix.sink"] * wrong}), cfg, toks)
        assert err(other, want.logits) > 3 * want.tol["bf16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_layers_and_long_prompts(dtype):
    """Widths at which the bf16 model takes the many-row tensor-core route, a prompt over several row segments, and more
    rows of decoding than one key page."""
    cfg = FC.config([FC.latent(heads=4, dim=64, vdim=64, kv_rank=128, window=150, scale=0.125, ff=512),
                     FC.mamba(inner=256, state=16, dt_rank=16), FC.delta(heads=4, kv_heads=2, dim=64, vdim=64, ff=256)],
                    width=256, vocab=300, loop={"start": 0, "stop": 2, "times": 2})
    sd = FC.weights(cfg, seed=6, rank_a=64, rank_g=32)
    toks = prompt(cfg, 640)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [560] + [1] * 80), dtype)
    want.check(in_portions(m, toks, [300, 7, 333]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_slots_and_pages_are_used_again(dtype):
    """Unequal requests that come and go over a pool that holds only a part of them: every position equals the request
    alone; portions beside single tokens; requests that pause; a slot used by a longer request before."""
    import versenext_b200 as vn
    cfg = FC.MODELS["loop_inside"]
    sd = FC.weights(cfg, seed=7)
    m = build(cfg, sd, dtype)
    rng = np.random.default_rng(11)
    reqs = {f"r{i}": prompt(cfg, n, seed=20 + i) for i, n in enumerate((130, 1, 64, 2, 65, 190, 33, 100, 7))}
    want = {r: Expected(sd, cfg, t) for r, t in reqs.items()}
    run = vn.StepRunner(m, max_batch=3, max_seq=192, pool_tokens=448)
    at = {r: 0 for r in reqs}
    waiting, live = list(reqs), []
    pages = {r: -(-len(t) // 64) for r, t in reqs.items()}
    while waiting or live:
        while waiting and len(live) < 3 and sum(pages[r] for r in live) + pages[waiting[0]] <= 7:
            live.append(waiting.pop(0))
        entries = []
        for r in live:
            left = len(reqs[r]) - at[r]
            n = min(left, int(rng.choice([0, 1, 1, 2, 3, 17, 64, 90])))
            if n:
                entries.append((r, reqs[r][at[r]:at[r] + n], list(range(n))))
        if not entries:
            continue
        got = run.step(entries).numpy()
        r0 = 0
        for r, t, _ in entries:
            want[r].check(got[r0:r0 + len(t)], dtype, slice(at[r], at[r] + len(t)), (r, at[r]))
            r0 += len(t)
            at[r] += len(t)
            if at[r] == len(reqs[r]):
                run.end(r)
                live.remove(r)
    m.check()
    assert run.cache.pages == (7, 7) and run.free_slots == 3


def test_a_batch_changes_nothing():
    """The same request alone and inside a batch: equal up to the order of sums (fp32 1e-5), every position."""
    cfg = FC.MODELS["plain"]
    m = build(cfg, FC.weights(cfg), "f32")
    a, b, c = prompt(cfg, 40, 1), prompt(cfg, 90, 2), prompt(cfg, 3, 3)
    cache = m.new_cache(3, 128)
    got = m.forward_ragged(cache, [2, 0, 1], [40, 90, 3], np.concatenate([a, b, c]), range(133)).numpy()
    assert err(got[:40], whole(m, a)) < 1e-5 and err(got[40:130], whole(m, b)) < 1e-5 and err(got[130:], whole(m, c)) < 1e-5
    got = m.forward_ragged(cache, [0, 2], [1, 5], np.concatenate([a[:1], b[:5]]), [0, 5]).numpy()
    assert err(got[:1], whole(m, np.concatenate([b, a[:1]]))[-1:]) < 1e-5
    assert err(got[1:], whole(m, np.concatenate([a, b[:5]]))[-1:]) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(dtype):
    """Batches wide enough for the kernels' many-sequence shapes, as a prompt, as short portions that could be cut back,
    and as single tokens."""
    cfg = FC.config([FC.delta(heads=8, kv_heads=4, dim=64, vdim=64), FC.mamba(inner=96, state=16, dt_rank=8),
                     FC.delta(heads=10, kv_heads=10, dim=128, vdim=72, conv=4), FC.latent(heads=8, dim=16, vdim=16, kv_rank=64, window=7)],
                    width=64)
    sd = FC.weights(cfg, seed=15)
    m = build(cfg, sd, dtype)
    B, T = 40, 29
    toks = np.stack([prompt(cfg, T, seed=200 + b) for b in range(B)])
    want = [Expected(sd, cfg, t) for t in toks[::13]]
    cache = m.new_cache(B, 32, max_pending=3)
    at, got = 0, []
    for n in (19, 2, 1, 3, 1, 3):
        got.append(m.forward_cached(toks[:, at:at + n], cache).numpy())
        cache.commit(n, np.full(B, n, np.int32))
        at += n
    got = np.concatenate(got, axis=1)
    for i, w in enumerate(want):
        w.check(got[13 * i], dtype)
    cache = m.new_cache(B, 32)
    got = m.forward_ragged(cache, list(range(B)), [T] * B, toks.reshape(-1), range(B * T)).numpy().reshape(B, T, -1)
    for i, w in enumerate(want):
        w.check(got[13 * i], dtype)
    m.check()


def greedy(sd, cfg, toks, n):
    toks = list(toks)
    for _ in range(n):
        toks.append(int(np.argmax(OF.forward(sd, cfg, toks)[-1])))
    return toks[-n:]


def test_greedy_generation_through_the_scheduler():
    import versenext_b200 as vn
    cfg = FC.MODELS["plain"]
    sd = FC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    prompts = [prompt(cfg, n, seed=40 + n) for n in (20, 1, 70, 5)]
    want = [greedy(sd, cfg, p, 12) for p in prompts]
    assert [list(x) for x in m.generate(prompts, 12)] == want
    eng = vn.BatchEngine(m, max_batch=2, max_seq=128, pool_tokens=192, step_tokens=11)
    assert [list(x) for x in eng.run(prompts, 12)] == want
    assert eng.cache.pages == (3, 3)
    eos = want[2][3]
    first = [w.index(eos) + 1 if eos in w else 12 for w in want]
    assert [list(x) for x in eng.run(prompts, 12, eos_id=eos)] == [w[:f] for w, f in zip(want, first)]
    sampled = eng.run(prompts, 6, temperature=0.9, top_k=5, seed=3)
    assert [len(x) for x in sampled] == [6] * 4 and all(0 <= t < cfg["vocab"] for x in sampled for t in x)


def test_long_decoding():
    """Hundreds of single tokens: the window has left the prompt behind, states have been handed on at every step."""
    cfg = FC.MODELS["loop_all"]
    sd = FC.weights(cfg, seed=12)
    toks = prompt(cfg, 420)
    want = Expected(sd, cfg, toks)
    for dtype in DTYPES:
        want.check(in_portions(build(cfg, sd, dtype), toks, [2] + [1] * 418), dtype)


@pytest.mark.parametrize("graph", [False, True])
def test_speculative_rounds_roll_recurrent_states_back(graph):
    """A composed model as target and another one as draft: the committed stream is the target's greedy stream, although
    most proposals are rejected and their states dropped."""
    import versenext_b200 as vn
    cfg = FC.MODELS["plain"]
    sd = FC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    near = {n: OF.bf16(a + 0.02 * np.random.default_rng(1).standard_normal(a.shape).astype(np.float32)) for n, a in sd.items()}
    prompts = np.stack([prompt(cfg, 9, seed=s) for s in (60, 61, 62)])
    want = [greedy(sd, cfg, p, 16) for p in prompts]
    for other in (near, FC.weights(cfg, seed=99)):
        d = build(cfg, other, "f32")
        for k in (1, 4):
            eng = vn.SpecEngine(m, d, max_batch=3, max_seq=64, k=k, graph=graph)
            out, stats = eng.generate(prompts, 16)
            assert [list(r) for r in out[:, 9:]] == want, k
    assert [list(r) for r in m.generate([p for p in prompts], 16, draft=d)] == want


def test_cut_back_and_refused_operations():
    cfg = FC.MODELS["plain"]
    sd = FC.weights(cfg)
    m = build(cfg, sd, "f32")
    toks, other = prompt(cfg, 30, 1), prompt(cfg, 30, 2)
    want = OF.forward(sd, cfg, toks)
    cache = m.new_cache(2, 64, max_pending=3)
    one = lambda n: np.array([n, n], np.int32)
    m.forward_cached(np.stack([toks[:20]] * 2), cache, want_logits=False, want_hidden=True, last_only=True)
    cache.commit(20, one(20))
    m.forward_cached(np.stack([np.r_[toks[20:21], other[:2]]] * 2), cache)       # one of three is right
    cache.commit(3, one(1))
    m.forward_cached(np.stack([other[:3]] * 2), cache)                           # none is right
    cache.commit(3, one(0))
    got = m.forward_cached(np.stack([toks[21:24]] * 2), cache).numpy()
    assert err(got[0], want[21:24]) < TOL["f32"] and err(got[1], want[21:24]) < TOL["f32"]
    cache.commit(3, one(3))
    np.testing.assert_array_equal(cache.per_seq_lens, [24, 24])
    # proposals forwarded one by one behind uncommitted ones
    for i in range(3):
        got = m.forward_cached(np.stack([toks[24 + i:25 + i]] * 2), cache, slot_offset=i).numpy()
        assert err(got[:, 0], want[24 + i][None].repeat(2, 0)) < TOL["f32"]
    cache.commit(3, np.array([2, 3], np.int32))
    got = m.forward_ragged(cache, [0, 1], [1, 1], [toks[26], toks[27]], [0, 1]).numpy()
    assert err(got, want[26:28]) < TOL["f32"]
    m.check()
    with pytest.raises(ValueError):
        m.forward_cached(np.stack([toks[:1]] * 2), cache, slot_offset=3)
    with pytest.raises(NotImplementedError):
        m.forward_cached(np.stack([toks[:2]] * 2), cache, parents=[-1, 0])
    with pytest.raises(NotImplementedError):
        cache.set_lengths([5, 5])
    m.forward_cached(np.stack([toks[:10]] * 2), cache)
    cache.commit(10, one(4))                                                     # more rows than there are states for
    with pytest.raises(ValueError):
        m.check()
    with pytest.raises(RuntimeError):
        m.forward_cached(np.stack([toks] * 2 )[:, :30].repeat(2, 1), cache)
    cache.reset()
    got = m.forward_cached(np.stack([toks] * 2), cache).numpy()
    assert err(got[1], want) < TOL["f32"]
    with pytest.raises(IndexError):
        m.forward_cached(np.full((1, 2), cfg["vocab"]), m.new_cache(1, 8))
        m.check()
    pool = m.new_cache(2, 192, pool_tokens=128)
    m.forward_ragged(pool, [0], [100], np.resize(toks, 100), [])
    with pytest.raises(RuntimeError):
        m.forward_ragged(pool, [1], [1], toks[:1], [0])
    pool.reset_seq(0)
    assert err(m.forward_ragged(pool, [1], [30], toks, range(30)).numpy(), want) < TOL["f32"]


def test_loading_is_checked():
    import versenext_b200 as vn
    cfg = FC.MODELS["plain"]
    sd = FC.weights(cfg)
    shapes = {n: a.shape for n, a in sd.items()}
    m = vn.FuzudraLM(cfg, shapes, dtype="f32")
    for n in list(sd)[:-1]:
        m.load_tensor(n, sd[n])
    with pytest.raises(ValueError):
        m.finalize()
    with pytest.raises(ValueError):
        m.load_tensor("l0.mix.unknown", sd["head"])
    with pytest.raises(ValueError):
        m.load_tensor("head", sd["head"][:-1])
    m.load_tensor(list(sd)[-1], sd[list(sd)[-1]])
    m.finalize()
    toks = prompt(cfg, 10)
    assert err(whole(m, toks), OF.forward(sd, cfg, toks)) < TOL["f32"]
    again = dict(sd, **{"l1.mix.uk": OF.bf16(sd["l1.mix.uk"] * 2), "l0.mix.x": OF.bf16(sd["l0.mix.x"] * 0.5)})
    for n in ("l1.mix.uk", "l0.mix.x"):                              # a tensor loaded anew is honoured
        m.load_tensor(n, again[n])
    m.finalize()
    assert err(whole(m, toks), OF.forward(again, cfg, toks)) < TOL["f32"]


def test_step_runner_serves_the_other_models_too():
    """A VerseNexLM behind the same step-wise interface."""
    import versenext_b200 as vn
    from oracle import model as OM
    cfg = OM.Config(vocab_size=64, dim=32, n_layer=2, n_head=4, use_alibi=False, use_rope=True, max_seq_len=64)
    sd = OM.init_state_dict(cfg, seed=1)
    kw = cfg.to_dict()
    kw.pop("init_std")
    m = vn.VerseNexLM(dtype="f32", **kw)
    m.load_state_dict(sd)
    a, b = np.arange(20) % 64, (np.arange(9) * 7) % 64
    wa, wb = OM.forward(sd, cfg, a[None])[0][0], OM.forward(sd, cfg, b[None])[0][0]
    run = vn.StepRunner(m, max_batch=2, max_seq=64)
    run.step([("a", a[:12], []), ("b", b[:3], [])])
    got = run.step([("a", a[12:20], [0, 7]), ("b", b[3:4], [0])]).numpy()
    assert err(got, np.stack([wa[12], wa[19], wb[3]])) < 1e-3


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(tmp_path, dtype):
    cfg = FC.MODELS["loop_all"]
    sd = FC.weights(cfg, seed=13)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir()
    out.mkdir()
    write_model(model, cfg, sd)
    a, b, c = prompt(cfg, 80, 1).tolist(), prompt(cfg, 30, 2).tolist(), prompt(cfg, 5, 3).tolist()
    steps = [([("a", a[:70], [0, 69])], []), ([("a", a[70:71], [0]), ("b", b[:20], [19])], []), ([("b", b[20:], [])], ["b"]),
             ([("c", c, [4]), ("a", a[71:], [8])], ["a", "c"]), ([("b2", b, [29])], ["b2"])]
    text = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in e], "end": end}) + "\n"
                   for i, (e, end) in enumerate(steps))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "192"], input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not (out / "2.f32").exists()
    A, Bw, Cw = (Expected(sd, cfg, t) for t in (a, b, c))
    want = {0: [(A, 0), (A, 69)], 1: [(A, 70), (Bw, 19)], 3: [(Cw, 4), (A, 79)], 4: [(Bw, 29)]}
    for i, rows in want.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert len(got) == len(rows)
        for g, (e, p) in zip(got, rows):
            e.check(g[None], "bf16" if dtype == "bfloat16" else "f32", slice(p, p + 1), (i, p))


def test_command_line(tmp_path):
    cfg = FC.MODELS["plain"]
    sd = FC.weights(cfg, seed=8)
    write_model(tmp_path, cfg, sd)
    p = prompt(cfg, 6)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-m", "versenext_b200", "generate", "--model", str(tmp_path), "--dtype", "f32", "--prompt",
                        ",".join(map(str, p)), "--max-new-tokens", "5"], capture_output=True, text=True, timeout=300, cwd=root)
    assert r.returncode == 0, r.stderr
    assert json.loads(r.stdout.splitlines()[-1]) == greedy(sd, cfg, p, 5)
