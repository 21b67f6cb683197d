"""The Musutar design on the device against the plain NumPy restatement (oracle/musutar.py), in fp32 and bf16."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import musutar as OM
from oracle.fuzudra import bf16
import fuzudra_cases as FC
import musutar_cases as MC
from musutar_cases import Expected, build, err, greedy, prompt
from test_fuzudra_cpu import write_model
from test_fuzudra_gpu import in_portions, whole

pytestmark = pytest.mark.gpu
DTYPES = ["f32", "bf16"]

A, L = MC.attention, MC.lightning
MECHANISMS = {
    "attention": A(), "attention_one_head": A(heads=1, kv_heads=1, dim=5, vdim=7, rot=4, conv=2, window=2),
    "attention_no_rotation_left": A(dim=32, vdim=32, rot=32, window=64), "attention_unscaled": A(scaling=None, window=65),
    "attention_wide": A(heads=4, kv_heads=1, dim=128, vdim=96, rot=64, window=100, scale=0.1),
    "attention_many_heads_per_key": A(heads=20, kv_heads=1, dim=16, vdim=24, rot=8, window=50),
    "attention_dim_192": A(heads=2, kv_heads=1, dim=180, vdim=64, rot=90, scale=0.08), "attention_dim_256": A(heads=2, kv_heads=2, dim=40, vdim=250, conv=6),
    "attention_dim_300": A(heads=1, kv_heads=1, dim=300, vdim=20, scale=0.06), "attention_dim_96": A(dim=80, vdim=90, heads=2, kv_heads=1, conv=1),
    "attention_no_window": A(window=None), "lightning": L(), "lightning_one_head": L(heads=1, dim=3, vdim=5, decay=[0.5]),
    "lightning_wide": L(heads=2, dim=128, vdim=128), "lightning_dim_160": L(heads=1, dim=160, vdim=40), "lightning_dim_300": L(heads=1, dim=300, vdim=12),
    "lightning_vdim_150": L(heads=2, dim=72, vdim=150, ff=0), "lightning_slow_and_fast": L(heads=4, dim=16, vdim=16, decay=[0.9995, 0.99, 0.2, 1e-3]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_alone(name, dtype):
    cfg = MC.config([MECHANISMS[name]])
    sd = MC.weights(cfg, seed=3)
    toks = prompt(cfg, 150)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [70, 1, 2, 1, 40, 1]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MC.MODELS)
def test_models_whole_portions_and_decoding(name, dtype):
    cfg = MC.MODELS[name]
    sd = MC.weights(cfg, seed=5)
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


@pytest.mark.parametrize("part", ["canon1", "hc1.mix", "hc1.in", "hc2.out", "rg1", "rg2.b", "mix.q.conv", "mix.v.conv", "mlp.up"])
def test_single_parts_scaled_up(part):
    """One part of a layer made the dominant one, in turn: an error in it cannot hide behind the others."""
    cfg = MC.config([A(window=20), A(kv_from=0, window=12)], streams=4, taps=5)
    sd = MC.weights(cfg, seed=21)
    for n in sd:
        if n == "l0." + part:
            sd[n] = bf16(sd[n] * 3)
    toks = prompt(cfg, 80)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, "f32")
    want.check(whole(m, toks), "f32")
    want.check(in_portions(m, toks, [30, 1, 1, 2]), "f32")


ASKS, ANSWERS, FILLER = 95, 96, 90


def edge_model(window, shared):
    """Attention in which token ASKS finds token ANSWERS and nothing else: the first half of an embedding is what a token
    asks for, the second half what it offers, and these two share one vector.  shared: the asking layer reads the keys of a
    layer whose own window is narrower."""
    layers = [A(heads=2, kv_heads=1, dim=32, vdim=32, window=window, rot=2, scale=1.0, conv=3, ff=0, scaling=None)]
    if shared:
        layers = [A(heads=2, kv_heads=1, dim=32, vdim=32, window=1, rot=2, scale=1.0, conv=3, ff=0, scaling=None)] + layers
        layers[1]["mixer"]["kv_from"] = 0
    cfg = MC.config(layers, width=64)
    sd = MC.weights(cfg, seed=9)
    eye, off = np.eye(32, dtype=np.float32), np.zeros((32, 32), np.float32)
    sd["embed"][ANSWERS, 32:] = sd["embed"][ASKS, :32]
    own, ask = "l0.", f"l{len(layers) - 1}."
    last_tap = lambda w: np.eye(1, 3, 2, dtype=np.float32).repeat(w, 0)
    for p in {own, ask}:
        sd[p + "norm1"] = np.ones(64, np.float32)
        sd[p + "canon1"] = sd[p + "canon1"] * 0
        sd[p + "hc1.mix"] = np.eye(3, dtype=np.float32)
        sd[p + "hc1.in"] = np.ones(3, np.float32)
    if shared:
        sd[own + "hc1.out"] = np.zeros(3, np.float32)
    sd[ask + "mix.q"] = bf16(np.tile(np.concatenate([eye, off], 1), (2, 1)))
    sd[ask + "mix.q.conv"] = last_tap(64)
    sd[ask + "mix.o"] = bf16(sd[ask + "mix.o"] * 8)
    sd[own + "mix.k"] = np.concatenate([off, eye], 1)
    sd[own + "mix.k.conv"] = last_tap(32)
    sd[own + "mix.v.conv"] = last_tap(32)
    return cfg, sd


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 63, 64, 65, 100])
def test_window_edges(window, shared, dtype):
    """The answer at the last distance that is seen, and just beyond it: in a prompt, in a portion, and when the asking
    token is decoded alone, which stands at several offsets from a page's border."""
    cfg, sd = edge_model(window, shared)
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
def test_far_keys_at_page_borders(dtype):
    """No window: the answer hundreds of tokens back, at the first token and around page borders, while the asking token is
    decoded; many key ranges are merged."""
    cfg, sd = edge_model(None, False)
    m = build(cfg, sd, dtype)
    base = prompt(cfg, 700, seed=4) % FILLER
    for at in (0, 1, 63, 64, 65, 511, 512, 640):
        toks = base.copy()
        toks[at], toks[-1] = ANSWERS, ASKS
        want = Expected(sd, cfg, toks)
        for got in (whole(m, toks)[-1:], in_portions(m, toks, [699, 1])[-1:], in_portions(m, toks, [300, 395, 5])[-1:]):
            want.check(got, dtype, slice(699, 700), at)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_state_carries_a_far_token(dtype):
    """Slow decay: the first token's share of the state is still there hundreds of tokens later, across portions, chunks and
    decoded tokens."""
    cfg = MC.config([L(heads=2, dim=24, vdim=24, decay=[0.999, 0.9], ff=0)], width=64)
    sd = MC.weights(cfg, seed=31)
    sd["embed"][7] *= 30                                             # after the norm a token of its own kind
    sd["l0.hc1.out"] = sd["l0.hc1.out"] * 4
    toks = prompt(cfg, 500, seed=2) % 90 + 8
    for first in (7, 8):
        t = toks.copy()
        t[0] = first
        want = Expected(sd, cfg, t)
        m = build(cfg, sd, dtype)
        want.check(whole(m, t)[-1:], dtype, slice(499, 500))
        want.check(in_portions(m, t, [64, 1, 63, 2, 150, 200, 1])[-1:], dtype, slice(499, 500))


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_layers_and_long_prompts(dtype):
    """Widths at which the bf16 model takes the many-row tensor-core route, a prompt over several row and state segments, and
    more rows of decoding than one key page."""
    cfg = MC.config([L(heads=4, dim=64, vdim=48, ff=512), A(heads=8, kv_heads=2, dim=64, vdim=64, rot=64, window=150, scale=0.125, ff=384),
                     L(heads=3, dim=128, vdim=128, ff=256), A(heads=8, kv_heads=2, dim=64, vdim=64, rot=64, window=90, scale=0.125, ff=0, kv_from=1)],
                    width=256, vocab=300)
    sd = MC.weights(cfg, seed=6)
    toks = prompt(cfg, 840)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [760] + [1] * 80), dtype)
    want.check(in_portions(m, toks, [300, 7, 533]), dtype)
    want.check(in_portions(m, toks, [270, 570]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["plain", "shared"])
def test_batches_slots_and_pages_are_used_again(name, dtype):
    """Unequal requests that come and go over a pool that holds only a part of them: every position equals the request
    alone; portions beside single tokens; requests that pause; a slot used by a longer request before."""
    import versenext_b200 as vn
    cfg = MC.MODELS[name]
    sd = MC.weights(cfg, seed=7)
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
    cfg = MC.MODELS["plain"]
    m = build(cfg, MC.weights(cfg), "f32")
    a, b, c = prompt(cfg, 40, 1), prompt(cfg, 90, 2), prompt(cfg, 3, 3)
    cache = m.new_cache(3, 128)
    got = m.forward_ragged(cache, [2, 0, 1], [40, 90, 3], np.concatenate([a, b, c]), range(133)).numpy()
    assert err(got[:40], whole(m, a)) < 1e-5 and err(got[40:130], whole(m, b)) < 1e-5 and err(got[130:], whole(m, c)) < 1e-5
    got = m.forward_ragged(cache, [0, 2], [1, 5], np.concatenate([a[:1], b[:5]]), [0, 5]).numpy()
    assert err(got[:1], whole(m, np.concatenate([b, a[:1]]))[-1:]) < 1e-5
    assert err(got[1:], whole(m, np.concatenate([a, b[:5]]))[-1:]) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(dtype):
    """Batches wide enough for the kernels' many-sequence shapes, as a prompt, as short portions that could be cut back, and
    as single tokens; more single tokens than the split-K route takes."""
    cfg = MC.config([L(heads=8, dim=64, vdim=64), A(heads=8, kv_heads=4, dim=64, vdim=64, rot=64, window=7), L(heads=10, dim=128, vdim=72),
                     A(heads=8, kv_heads=4, dim=64, vdim=64, rot=64, window=20, kv_from=1)], width=64)
    sd = MC.weights(cfg, seed=15)
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
    B = 260
    cache = m.new_cache(B, 4)
    for t in range(3):
        rows = np.array([toks[b % 40, t] for b in range(B)])
        got = m.forward_ragged(cache, list(range(B)), [1] * B, rows, range(B)).numpy()
        for b in (0, 13, 255, 259):
            Expected(sd, cfg, toks[b % 40][:3]).check(got[b:b + 1], dtype, slice(t, t + 1), (b, t))
    m.check()


def test_greedy_generation_through_the_scheduler():
    import versenext_b200 as vn
    cfg = MC.MODELS["plain"]
    sd = MC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    prompts = [prompt(cfg, n, seed=40 + n) for n in (20, 1, 70, 5)]
    want = [greedy(sd, cfg, p, 12) for p in prompts]
    assert [list(x) for x in m.generate(prompts, 12)] == want
    eng = vn.BatchEngine(m, max_batch=2, max_seq=128, pool_tokens=192, step_tokens=11)
    assert [list(x) for x in eng.run(prompts, 12)] == want
    assert eng.cache.pages == (3, 3)
    sampled = eng.run(prompts, 6, temperature=0.9, top_k=5, seed=3)
    assert [len(x) for x in sampled] == [6] * 4 and all(0 <= t < cfg["vocab"] for x in sampled for t in x)


def test_long_decoding():
    """Hundreds of single tokens: the windows have left the prompt behind, states have been handed on at every step."""
    cfg = MC.MODELS["shared"]
    sd = MC.weights(cfg, seed=12)
    toks = prompt(cfg, 420)
    want = Expected(sd, cfg, toks)
    for dtype in DTYPES:
        want.check(in_portions(build(cfg, sd, dtype), toks, [2] + [1] * 418), dtype)


@pytest.mark.parametrize("graph", [False, True])
def test_speculative_rounds_roll_states_back(graph):
    """A Musutar model as target and another one as draft: the committed stream is the target's greedy stream, although most
    proposals are rejected and their states and convolution inputs dropped."""
    import versenext_b200 as vn
    cfg = MC.MODELS["plain"]
    sd = MC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    near = {n: bf16(a + 0.02 * np.random.default_rng(1).standard_normal(a.shape).astype(np.float32)) for n, a in sd.items()}
    prompts = np.stack([prompt(cfg, 9, seed=s) for s in (60, 61, 62)])
    want = [greedy(sd, cfg, p, 16) for p in prompts]
    for other in (near, MC.weights(cfg, seed=99)):
        d = build(cfg, other, "f32")
        for k in (1, 4):
            eng = vn.SpecEngine(m, d, max_batch=3, max_seq=64, k=k, graph=graph)
            out, stats = eng.generate(prompts, 16)
            assert [list(r) for r in out[:, 9:]] == want, k


def test_mechanisms_in_other_arrangements():
    """Streams, gates and input convolutions around the other layer kinds, grouped-query attention on the plain residual:
    the parts are not tied to one design."""
    import versenext_b200 as vn
    from oracle import fuzudra as OF
    D, V, eps = 48, 60, 1e-4
    # (1) plain residual, RMS norms around zero, gated feed-forward, attention without gate, rotation or convolution
    cfg = {"vocab_size": V, "dim": D, "norm_eps": eps, "layers": [
        {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.3, "window": 11, "mlp_hidden": 40, "mlp_act": "silu"}]}
    rng = np.random.default_rng(3)
    w = lambda *s: bf16((rng.standard_normal(s) / np.sqrt(s[-1])).astype(np.float32))
    sd = {"embed": w(V, D) * 4, "head": w(V, D), "final.norm": w(D), "l0.norm1": w(D), "l0.norm2": w(D), "l0.mix.q": w(48, D) * 2, "l0.mix.k": w(24, D) * 2,
          "l0.mix.v": w(24, D), "l0.mix.o": w(D, 48), "l0.mlp.gate": w(40, D), "l0.mlp.up": w(40, D), "l0.mlp.down": w(D, 40)}
    toks = rng.integers(0, V, 50)
    F = np.float64
    x = sd["embed"].astype(F)[toks]
    h = OF.norm(x, sd["l0.norm1"], eps)
    o = OM.windowed_attention((h @ sd["l0.mix.q"].T).reshape(50, 4, 12), (h @ sd["l0.mix.k"].T).reshape(50, 2, 12), (h @ sd["l0.mix.v"].T).reshape(50, 2, 12), 0.3, 11)
    x = x + o.reshape(50, 48) @ sd["l0.mix.o"].T
    h = OF.norm(x, sd["l0.norm2"], eps)
    x = x + (OF.silu(h @ sd["l0.mlp.gate"].T) * (h @ sd["l0.mlp.up"].T)) @ sd["l0.mlp.down"].T
    want = OF.norm(x, sd["final.norm"], eps) @ sd["head"].T
    m = vn.ComposedLM(cfg, dtype="f32")
    m.load_state_dict(sd)
    assert err(whole(m, toks), want) < 3e-5 and err(in_portions(m, toks, [20, 1, 2]), want) < 3e-5
    # (2) two streams, RMS norms, an input convolution and result gates around a delta rule layer with a gated feed-forward
    fz = FC.config([FC.delta(heads=2, kv_heads=1, dim=16, vdim=12, ff=24)], width=D, vocab=V, eps=eps)
    sd = FC.weights(fz, seed=2)
    from versenext_b200.fuzudra import composed_config
    cfg = dict(composed_config(fz, {n: a.shape for n, a in sd.items()}), positions="", streams=2, input_conv=3, residual_gate=True)
    for q in (1, 2):
        sd.update({f"l0.hc{q}.in": w(2) + 1, f"l0.hc{q}.out": w(2) + 1, f"l0.hc{q}.mix": bf16(np.eye(2) + 0.2 * w(2, 2)), f"l0.rg{q}": w(D, D), f"l0.rg{q}.b": w(D)})
    sd["l0.canon1"] = w(D, 3)
    sd = {n: bf16(np.asarray(a, np.float32)) for n, a in sd.items()}
    W = {n[3:]: a.astype(F) for n, a in sd.items() if n.startswith("l0.")}
    xs = np.stack([sd["embed"].astype(F)[toks]] * 2)
    h = OF.norm(OM.read_streams(xs, W["hc1.in"]), W["norm1"], eps)
    y = OF.channel_delta(h + OF.causal_conv(h, W["canon1"]), {n[4:]: a for n, a in W.items() if n.startswith("mix.")}, fz["layers"][0]["mixer"], eps)
    xs = OM.write_streams(xs, W["hc1.mix"], W["hc1.out"], y * OF.sigmoid(h @ W["rg1"].T + W["rg1.b"]))
    h = OF.norm(OM.read_streams(xs, W["hc2.in"]), W["norm2"], eps)
    y = OF.feed_forward(h, {n[4:]: a for n, a in W.items() if n.startswith("mlp.")})
    xs = OM.write_streams(xs, W["hc2.mix"], W["hc2.out"], y * OF.sigmoid(h @ W["rg2"].T + W["rg2.b"]))
    want = OF.norm(xs.sum(0), sd["final.norm"], eps) @ sd["head"].T
    m = vn.ComposedLM(cfg, dtype="f32")
    m.load_state_dict(sd)
    assert err(whole(m, toks), want) < 3e-5 and err(in_portions(m, toks, [20, 1, 2]), want) < 3e-5


def test_loading_is_checked():
    import versenext_b200 as vn
    cfg = MC.MODELS["plain"]
    sd = MC.weights(cfg)
    m = vn.MusutarLM(cfg, {n: a.shape for n, a in sd.items()}, dtype="f32")
    for n in list(sd)[:-1]:
        m.load_tensor(n, sd[n])
    with pytest.raises(ValueError):
        m.finalize()
    with pytest.raises(ValueError):
        m.load_tensor("l2.mix.k", sd["l1.mix.k"])                    # a layer that reads another one's keys has none
    with pytest.raises(ValueError):
        m.load_tensor("l0.hc1.mix", sd["l0.hc1.mix"][:, :-1])
    m.load_tensor(list(sd)[-1], sd[list(sd)[-1]])
    m.finalize()
    toks = prompt(cfg, 10)
    assert err(whole(m, toks), OM.forward(sd, cfg, toks)) < 3e-5
    for bad in ({"kv_from": 2}, {"kv_from": 0}, {"heads": 3}, {"kv_heads": 1, "kv_from": 1}):
        other = json.loads(json.dumps(cfg))
        other["layers"][2]["mixer"].update(bad)
        with pytest.raises(ValueError):
            vn.MusutarLM(other, {}, dtype="f32")


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_and_command_line(tmp_path, dtype):
    cfg = MC.MODELS["shared"]
    sd = MC.weights(cfg, seed=13)
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
    EA, EB, EC = (Expected(sd, cfg, t) for t in (a, b, c))
    want = {0: [(EA, 0), (EA, 69)], 1: [(EA, 70), (EB, 19)], 3: [(EC, 4), (EA, 79)], 4: [(EB, 29)]}
    for i, rows in want.items():
        got = np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert len(got) == len(rows)
        for g, (e, p) in zip(got, rows):
            e.check(g[None], "bf16" if dtype == "bfloat16" else "f32", slice(p, p + 1), (i, p))
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "versenext_b200", "generate", "--model", str(model), "--dtype", "f32", "--prompt",
                            ",".join(map(str, c)), "--max-new-tokens", "5"], capture_output=True, text=True, timeout=300, cwd=root)
        assert r.returncode == 0, r.stderr
        assert json.loads(r.stdout.splitlines()[-1]) == greedy(sd, cfg, c, 5)
