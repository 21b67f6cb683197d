"""The Givozen design on the device against the plain NumPy restatement (oracle/givozen.py), in fp32 and bf16."""

import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import givozen as OG
from oracle import bozasun as OB
from oracle import fuzudra as OF
from oracle.fuzudra import bf16
import givozen_cases as GC
from givozen_cases import Expected, build, err, greedy, prompt
from test_fuzudra_cpu import write_model
from test_fuzudra_gpu import in_portions, whole

pytestmark = pytest.mark.gpu
DTYPES = ["f32", "bf16"]

A, E, R, D = GC.attention, GC.moe, GC.rot, GC.dense
MECHANISMS = {
    "attention": A(mlp=None), "attention_one_head": A(heads=1, kv_heads=1, dim=5, vdim=7, rot=R(4), mlp=None), "attention_all_rotated": A(dim=32, vdim=32, rot=R(32), mlp=None),
    "attention_not_rotated": A(rot=None, mlp=None), "attention_not_scaled": A(rot=R(24, 50.0, None), mlp=None), "attention_all_slow": A(rot=R(original=4), mlp=None),
    "attention_all_fast": A(rot=R(base=4.0, original=9000), mlp=None), "attention_mixed_wavelengths": A(dim=64, vdim=64, scale=0.2, rot=R(64, 10000.0, 8.0, 1.5, 6.0, 300), mlp=None),
    "attention_wide": A(heads=4, kv_heads=1, dim=128, vdim=96, rot=R(64), scale=0.1, mlp=None), "attention_many_heads_per_key": A(heads=20, kv_heads=1, dim=16, vdim=24, rot=R(8), mlp=None),
    "attention_33_heads_per_key": A(heads=66, kv_heads=2, dim=8, vdim=8, rot=R(8), mlp=None), "attention_narrow": A(heads=5, kv_heads=5, dim=8, vdim=4, rot=R(4), mlp=None),
    "attention_dim_180": A(heads=2, kv_heads=1, dim=180, vdim=64, rot=R(90), scale=0.08, mlp=None), "attention_vdim_250": A(heads=2, kv_heads=2, dim=40, vdim=250, mlp=None),
    "attention_dim_300": A(heads=1, kv_heads=1, dim=300, vdim=20, scale=0.06, mlp=None), "attention_odd_widths": A(heads=3, kv_heads=1, dim=21, vdim=13, rot=R(10), mlp=None),
    "poly_norm_1100": A(mlp=D(1100)), "poly_norm_2050": A(mlp=D(2050)), "poly_norm_4500": A(mlp=D(4500)), "poly_norm_9001": A(mlp=D(9001)), "poly_norm_one": A(mlp=D(1)),
    "moe": A(mlp=E()), "moe_no_shared": A(mlp=E(shared_ff=None)), "moe_one_chosen": A(mlp=E(top=1)), "moe_one_expert": A(mlp=E(experts=1, top=1)), "moe_all": A(mlp=E(experts=4, top=4, ff=9, shared_ff=7)),
    "moe_many": A(mlp=E(experts=40, top=6, ff=40, shared_ff=80)), "moe_no_limits": A(mlp=E(limit=50.0, shared_limit=60.0)), "moe_low_limits": A(mlp=E(limit=0.3, shared_limit=0.1)),
    "moe_300_experts": A(heads=1, kv_heads=1, mlp=E(experts=300, top=3, ff=8, shared_ff=8)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", MECHANISMS)
def test_each_mechanism_alone(name, dtype):
    cfg = GC.config([MECHANISMS[name]])
    sd = GC.weights(cfg, seed=3)
    toks = prompt(cfg, 150, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [70, 1, 2, 1, 40, 1]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", GC.MODELS)
def test_models_whole_portions_and_decoding(name, dtype):
    cfg = GC.MODELS[name]
    sd = GC.weights(cfg, seed=5)
    toks = prompt(cfg, 170, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    res = m.residuals(toks)
    assert len(res) == len(want.runs)
    for i, (a, b, tol) in enumerate(zip(res, want.runs, want.run_tol)):
        assert err(a, b) < tol[dtype], i
    want.check(whole(m, toks), dtype)
    for sizes in ([2], [1], [3, 2, 61, 1, 5], [64], [63, 65], [127, 1, 1, 40], [100] + [1] * 70):
        want.check(in_portions(m, toks, sizes), dtype, what=sizes)


@pytest.mark.parametrize("part", ["mix.q.b", "mix.k.b", "mix.v.b", "mix.temp", "mix.g", "norm1b", "norm2b", "mlp.act", "mlp.shared.sg", "mlp.shared.up", "mlp.router", "mlp.e2.up",
                                  "mlp.e1.gate", "loop.step"])
def test_single_parts_scaled_up(part):
    """One part of a model made the dominant one, in turn: an error in it cannot hide behind the others."""
    cfg = GC.config([A(mlp=E(experts=5, top=3)), A(mlp=D(60))], loop=(0, 2, 2))
    sd = GC.weights(cfg, seed=21)
    name = part if part == "loop.step" else ("l1." if part == "mlp.act" else "l0.") + part
    sd[name] = bf16(3 * sd[name])
    if part.startswith("norm"):
        sd[name][-GC.CODE:] = -1
    toks = prompt(cfg, 80, sd=sd)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, "f32")
    want.check(whole(m, toks), "f32")
    want.check(in_portions(m, toks, [30, 1, 1, 2]), "f32")


@pytest.mark.parametrize("dtype", DTYPES)
def test_temperatures_of_either_sign(dtype):
    """Heads that attend evenly, sharply, and to what fits least."""
    cfg = GC.config([A(heads=6, kv_heads=2, mlp=None)])
    sd = GC.weights(cfg, seed=17)
    sd["l0.mix.temp"] = bf16(np.array([0.0, 3.0, -1.0, 0.1, -0.02, 1.0], np.float32))
    toks = prompt(cfg, 140, seed=3)
    want = Expected(sd, cfg, toks)
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [1, 100]), dtype)


ASKS, ANSWERS, FILLER = 95, 96, 90


def asking_model():
    """Attention in which token ASKS finds token ANSWERS and nothing else: the first half of an embedding is what a token
    asks for, the second half what it offers, and these two share one vector."""
    cfg = GC.config([A(heads=2, kv_heads=1, dim=32, vdim=32, rot=R(2, factor=None), scale=0.4, mlp=None)], width=64)
    sd = GC.weights(cfg, seed=9)
    eye, off = np.eye(32, dtype=np.float32), np.zeros((32, 32), np.float32)
    sd["embed"][ANSWERS, 32:] = sd["embed"][ASKS, :32]
    sd["l0.norm1"] = sd["l0.norm1"] * 0
    sd["l0.mix.temp"] = bf16(np.array([1.0, 1.25], np.float32))
    for n in ("q", "k"):
        sd[f"l0.mix.{n}.b"] = sd[f"l0.mix.{n}.b"] * 0
    sd["l0.mix.q"], sd["l0.mix.k"] = np.tile(np.concatenate([eye, off], 1), (2, 1)), np.concatenate([off, eye], 1)
    sd["l0.norm1b"] = sd["l0.norm1b"] * 0 + 1
    return cfg, sd


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_at_page_borders(dtype):
    """The answer hundreds of tokens back, at the first token, around page borders and right before the asking token, which is
    decoded, or ends a portion, or a prompt; many key ranges are merged."""
    cfg, sd = asking_model()
    m = build(cfg, sd, dtype)
    base = prompt(cfg, 700, seed=4) % FILLER
    plain = None
    for at in (None, 0, 1, 63, 64, 65, 511, 512, 640, 697, 698):
        toks = base.copy()
        toks[-1] = ASKS
        if at is not None:
            toks[at] = ANSWERS
        want = Expected(sd, cfg, toks)
        plain = want.logits[-1:] if at is None else plain
        assert at is None or err(want.logits[-1:], plain) > 2 * want.tol["bf16"]
        for got in (whole(m, toks)[-1:], in_portions(m, toks, [699, 1])[-1:], in_portions(m, toks, [300, 395, 5])[-1:], in_portions(m, toks, [512, 186, 2])[-1:]):
            want.check(got, dtype, slice(699, 700), at)


@pytest.mark.parametrize("dtype", DTYPES)
def test_what_comes_later_is_not_seen(dtype):
    """An answer behind the asking token, in the same portion and the same page, changes nothing."""
    cfg, sd = asking_model()
    m = build(cfg, sd, dtype)
    toks = prompt(cfg, 80, seed=6) % FILLER
    for q in (0, 14, 15, 62, 63):
        t = toks.copy()
        t[q], t[q + 1] = ASKS, ANSWERS
        want = Expected(sd, cfg, t)
        want.check(whole(m, t)[q:q + 1], dtype, slice(q, q + 1), q)
        want.check(in_portions(m, t, [q + 2])[q:q + 1], dtype, slice(q, q + 1), q)


@functools.lru_cache(None)
def wide_case():
    cfg = GC.config([A(heads=8, kv_heads=2, dim=64, vdim=64, rot=R(64, original=500), scale=0.15, mlp=E(experts=6, top=3, ff=192, shared_ff=320)),
                     A(heads=4, kv_heads=4, dim=128, vdim=64, rot=R(64, original=500), scale=0.1, mlp=D(384)),
                     A(heads=6, kv_heads=3, dim=64, vdim=128, rot=R(32), scale=0.1, mlp=E(experts=10, top=2, ff=128, shared_ff=128))], width=256, vocab=300, loop=(1, 3, 2))
    sd = GC.weights(cfg, seed=6)
    toks = prompt(cfg, 540, sd=sd)
    return cfg, sd, toks, Expected(sd, cfg, toks)


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_layers_and_long_prompts(dtype):
    """Widths at which the bf16 model takes the many-row tensor-core route, a prompt over several row segments and several
    pieces of an expert's rows, and more rows of decoding than one key page."""
    cfg, sd, toks, want = wide_case()
    m = build(cfg, sd, dtype)
    want.check(whole(m, toks), dtype)
    want.check(in_portions(m, toks, [460] + [1] * 80), dtype)
    want.check(in_portions(m, toks, [300, 7, 233]), dtype)
    want.check(in_portions(m, toks, [258, 282]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["plain", "other_order"])
def test_batches_slots_and_pages_are_used_again(name, dtype):
    """Unequal requests that come and go over a pool that holds only a part of them: every position equals the request
    alone; portions beside single tokens; requests that pause; a slot used by a longer request before."""
    import versenext_b200 as vn
    cfg = GC.MODELS[name]
    sd = GC.weights(cfg, seed=7)
    m = build(cfg, sd, dtype)
    rng = np.random.default_rng(11)
    reqs = {f"r{i}": prompt(cfg, n, seed=20 + i, sd=sd) for i, n in enumerate((130, 1, 64, 2, 65, 190, 33, 100, 7))}
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
    cfg = GC.MODELS["plain"]
    sd = GC.weights(cfg)
    m = build(cfg, sd, "f32")
    a, b, c = prompt(cfg, 40, 1, sd), prompt(cfg, 90, 2, sd), prompt(cfg, 3, 3, sd)
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
    cfg = GC.config([A(heads=8, kv_heads=4, dim=64, vdim=64, rot=R(64), scale=0.15, mlp=E(ff=32)), A(heads=4, kv_heads=1, dim=32, vdim=32, mlp=D(64)),
                     A(heads=2, kv_heads=2, mlp=E(experts=5, top=4, ff=40, shared_ff=24))], width=64, loop=(0, 2, 2))
    sd = GC.weights(cfg, seed=15)
    m = build(cfg, sd, dtype)
    B, T = 40, 29
    checked = range(0, B, 13)
    toks = np.stack([prompt(cfg, T, seed=200 + b, sd=sd if b in checked else None) for b in range(B)])
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
        for b in (0, 13, 253, 259):
            if b % 40 in checked:
                want[(b % 40) // 13].check(got[b:b + 1], dtype, slice(t, t + 1), (b, t))
    m.check()


def test_greedy_generation_through_the_scheduler():
    import versenext_b200 as vn
    cfg = GC.MODELS["plain"]
    sd = GC.weights(cfg, seed=8)
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
    """Hundreds of single tokens over several pages of every pass."""
    cfg = GC.MODELS["other_order"]
    sd = GC.weights(cfg, seed=12)
    toks = prompt(cfg, 420, sd=sd)
    want = Expected(sd, cfg, toks)
    for dtype in DTYPES:
        want.check(in_portions(build(cfg, sd, dtype), toks, [2] + [1] * 418), dtype)


@pytest.mark.parametrize("graph", [False, True])
def test_speculative_rounds(graph):
    """A Givozen model as target and another one as draft: the committed stream is the target's greedy stream, although most
    proposals are rejected and their keys and values cut back."""
    import versenext_b200 as vn
    cfg = GC.MODELS["plain"]
    sd = GC.weights(cfg, seed=8)
    m = build(cfg, sd, "f32")
    near = {n: bf16(a + 0.02 * np.random.default_rng(1).standard_normal(a.shape).astype(np.float32)) for n, a in sd.items()}
    prompts = np.stack([prompt(cfg, 9, seed=s) for s in (60, 61, 62)])
    want = [greedy(sd, cfg, p, 16) for p in prompts]
    for other in (near, GC.weights(cfg, seed=99)):
        d = build(cfg, other, "f32")
        for k in (1, 4):
            eng = vn.SpecEngine(m, d, max_batch=3, max_seq=64, k=k, graph=graph)
            out, stats = eng.generate(prompts, 16)
            assert [list(r) for r in out[:, 9:]] == want, k


@pytest.mark.parametrize("D", [48, 50])
@pytest.mark.parametrize("dtype", DTYPES)
def test_mechanisms_in_other_arrangements(D, dtype):
    """The parts are not tied to one design: temperatures and gates per head with norms of the heads, interleaved pairs, a window
    and an output bias; sigmoid scores with a correction and groups, weights on the result; weights on the input of GELU experts
    beside a shared one; PolyNorm and an entry that adds without norms behind the sublayers, short prompts and long ones."""
    import versenext_b200 as vn
    V, eps, T, F = 60, 1e-4, 300, np.float64
    rng = np.random.default_rng(3)
    w = lambda *s: bf16((rng.standard_normal(s) / np.sqrt(s[-1])).astype(np.float32))
    rope = {"dims": 8, "base": 300.0, "interleaved": True}
    cfg = {"vocab_size": V, "dim": D, "norm_eps": eps, "loop": {"start": 1, "stop": 3, "times": 2, "entry": "add"}, "layers": [
        {"mixer": "attention", "heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.3, "window": 40, "qk_norm": True, "output_gate": "head", "temperature": True,
         "out_bias": True, "rope": rope, "mlp_hidden": 20, "mlp_act": "gelu_tanh", "experts": {"count": 6, "top": 2, "groups": 3, "keep": 2, "correction": True, "score": "sigmoid"}},
        {"mixer": "attention", "heads": 2, "kv_heads": 1, "dim": 16, "vdim": 8, "scale": 0.3, "output_gate": "element", "temperature": True,
         "mlp_hidden": 18, "mlp_act": "gelu_tanh", "experts": {"count": 3, "top": 2, "weight": "input", "shared": {"hidden": 10}}},
        {"mixer": "attention", "heads": 2, "kv_heads": 2, "dim": 8, "vdim": 16, "scale": 0.4, "mlp_hidden": 40, "mlp_act": "poly_norm"}]}
    sd = {"embed": w(V, D) * 4, "head": w(V, D), "final.norm": w(D), "loop.step": w(2, D) * 3}
    for i, (H, G, d, v) in enumerate(((4, 2, 12, 12), (2, 1, 16, 8), (2, 2, 8, 16))):
        p = f"l{i}."
        sd.update({p + "norm1": w(D), p + "norm2": w(D), p + "mix.q": w(H * d, D) * 2, p + "mix.k": w(G * d, D) * 2, p + "mix.v": w(G * v, D), p + "mix.o": w(D, H * v)})
    sd.update({"l0.mix.g": w(4, D) * 2, "l0.mix.temp": 1 + w(4), "l0.mix.q.norm": 1 + w(12), "l0.mix.k.norm": 1 + w(12), "l0.mix.o.b": w(D), "l0.mlp.router": w(6, D) * 2,
               "l0.mlp.correction": w(6) * 0.3, "l1.mix.g": w(16, D) * 2, "l1.mix.temp": 1 + w(2), "l1.mlp.router": w(3, D) * 2, "l1.mlp.shared.sg": w(1, D) * 2,
               "l2.mlp.up": w(40, D), "l2.mlp.down": w(D, 40), "l2.mlp.act": np.array([0.5, -0.7, 0.6, 0.3])})
    for p, f in [(f"l0.mlp.e{e}.", 20) for e in range(6)] + [(f"l1.mlp.e{e}.", 18) for e in range(3)] + [("l1.mlp.shared.", 10)]:
        sd.update({p + "gate": w(f, D) * 2, p + "up": w(f, D) * 2, p + "down": w(D, f) * 2})
    sd = {n: bf16(np.asarray(a, np.float32)) for n, a in sd.items()}
    W = {n: a.astype(F) for n, a in sd.items()}
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    gelu = lambda h, p: (OF.gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T

    def heads(h, p, H, G, d, v):
        return ((h @ W[p + "mix.q"].T).reshape(-1, H, d), (h @ W[p + "mix.k"].T).reshape(-1, G, d), (h @ W[p + "mix.v"].T).reshape(-1, G, v))

    def attend(q, k, v, scale, temp, seen):
        o = np.zeros((T, q.shape[1], v.shape[2]))
        for a in range(q.shape[1]):
            g = a // (q.shape[1] // k.shape[1])
            s = np.where(seen, q[:, a] @ k[:, g].T * scale * temp[a], -np.inf)
            e = np.exp(s - s.max(1, keepdims=True))
            o[:, a] = e @ v[:, g] / e.sum(1, keepdims=True)
        return o

    def clear(z, top):                     # how far the choice is from another one
        z = -np.sort(-z, axis=1)
        return z[:, top - 1] - z[:, top]

    def forward(toks):
        gap = np.full(T, np.inf)
        x = x0 = W["embed"][toks]
        h = OF.norm(x, W["l0.norm1"], eps)
        q, k, v = heads(h, "l0.", 4, 2, 12, 12)
        q, k = (OB.rotate(OB.norm(y, W[f"l0.mix.{n}.norm"], eps), rope) for y, n in ((q, "q"), (k, "k")))
        o = attend(q, k, v, 0.3, W["l0.mix.temp"], (j <= i) & (i - j < 40)) * OF.sigmoid(h @ W["l0.mix.g"].T)[:, :, None]
        x = x + o.reshape(T, -1) @ W["l0.mix.o"].T + W["l0.mix.o.b"]
        h = OF.norm(x, W["l0.norm2"], eps)
        s = OF.sigmoid(h @ W["l0.mlp.router"].T)
        c = s + W["l0.mlp.correction"]
        best = c.reshape(T, 3, 2).max(2)
        gap = np.minimum(gap, clear(best, 2))
        c = np.where(np.repeat(best >= -np.sort(-best, axis=1)[:, 1:2], 2, axis=1), c, -np.inf)
        gap = np.minimum(gap, clear(c, 2))
        y = np.zeros_like(x)
        for e in range(6):
            on = np.argsort(-c, axis=1)[:, :2] == e
            y += (on.any(1) * s[:, e])[:, None] * gelu(h, f"l0.mlp.e{e}.")
        x = x + y
        for t in range(2):
            x = (x + x0 if t else x) + W["loop.step"][t]
            h = OF.norm(x, W["l1.norm1"], eps)
            o = attend(*heads(h, "l1.", 2, 1, 16, 8), 0.3, W["l1.mix.temp"], j <= i).reshape(T, -1) * OF.sigmoid(h @ W["l1.mix.g"].T)
            x = x + o @ W["l1.mix.o"].T
            h = OF.norm(x, W["l1.norm2"], eps)
            z = h @ W["l1.mlp.router"].T
            s = np.exp(z) / np.exp(z).sum(1, keepdims=True)
            gap = np.minimum(gap, clear(s, 2))
            y = OF.sigmoid(h @ W["l1.mlp.shared.sg"].T) * gelu(h, "l1.mlp.shared.")
            for e in range(3):
                on = (np.argsort(-s, axis=1)[:, :2] == e).any(1)
                y += on[:, None] * gelu(s[:, e:e + 1] * h, f"l1.mlp.e{e}.")
            x = x + y
            h = OF.norm(x, W["l2.norm1"], eps)
            x = x + attend(*heads(h, "l2.", 2, 2, 8, 16), 0.4, np.ones(2), j <= i).reshape(T, -1) @ W["l2.mix.o"].T
            h = OF.norm(x, W["l2.norm2"], eps)
            x = x + OG.poly_norm(h @ W["l2.mlp.up"].T, W["l2.mlp.act"], eps) @ W["l2.mlp.down"].T
        return OF.norm(x, W["final.norm"], eps) @ W["head"].T, gap
    toks = rng.integers(0, V, T)
    for _ in range(200):                                   # tokens whose experts are clear, so far as there are some
        gap = forward(toks)[1]
        if (gap > 0.02).all():
            break
        toks = np.where(gap > 0.02, toks, rng.integers(0, V, T))
    want, gap = forward(toks)
    m = vn.ComposedLM(cfg, dtype=dtype)
    m.load_state_dict(sd)
    clean = gap > (1e-4 if dtype == "f32" else 0.02)
    assert clean.mean() > 0.7
    tol = 3e-5 if dtype == "f32" else 3e-2
    for got in (whole(m, toks), in_portions(m, toks, [20, 1, 2]), in_portions(m, toks, [290, 1])):
        if dtype == "f32":
            assert err(got[clean], want[clean]) < tol
        else:                                              # a close choice that went the other way reaches later tokens a little
            d = np.sqrt(np.mean((got - want) ** 2, axis=1)) / np.std(want)
            assert np.median(d[clean]) < tol and np.mean(d[clean] < 3 * tol) > 0.95


def test_loading_is_checked():
    import versenext_b200 as vn
    cfg = GC.MODELS["plain"]
    sd = GC.weights(cfg)
    m = vn.GivozenLM(cfg, {n: a.shape for n, a in sd.items()}, dtype="f32")
    for n in list(sd)[:-1]:
        m.load_tensor(n, sd[n])
    with pytest.raises(ValueError):
        m.finalize()
    for name, a in (("l1.mlp.e7.gate", sd["l1.mlp.e0.gate"]), ("l3.mlp.up", sd["l0.mlp.up"]), ("l2.mix.sink", np.zeros(2, np.float32)), ("head", sd["embed"]),
                    ("l1.mlp.shared.sg", sd["l1.mlp.router"]), ("l0.mlp.act", np.zeros(3, np.float32)), ("l0.mlp.gate", sd["l0.mlp.up"]),
                    ("l0.mix.g", sd["l0.mix.v"]), ("l0.mix.o.b", np.zeros(72, np.float32)), ("loop.in", np.zeros((72, 144), np.float32)), ("loop.step", sd["loop.step"][:1])):
        with pytest.raises(ValueError):
            m.load_tensor(name, a)
    m.load_tensor(list(sd)[-1], sd[list(sd)[-1]])
    m.finalize()
    toks = prompt(cfg, 10)
    assert err(whole(m, toks), OG.forward(sd, cfg, toks)) < 3e-5
    for layer, part, bad in ((0, "mixer", {"heads": 3}), (0, "mixer", {"rot": R(26)}), (1, "mlp", {"router": {"experts": 7, "top": 8}}), (1, "mlp", {"router": {"experts": 0, "top": 0}})):
        other = json.loads(json.dumps(cfg))
        other["layers"][layer][part].update(bad)
        with pytest.raises(ValueError):
            vn.GivozenLM(other, {}, dtype="f32")
    with pytest.raises(ValueError):
        vn.GivozenLM(dict(cfg, loop={"start": 1, "stop": 5, "times": 2}), {}, dtype="f32")


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_and_command_line(tmp_path, dtype):
    cfg = GC.MODELS["other_order"]
    sd = GC.weights(cfg, seed=13)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir()
    out.mkdir()
    write_model(model, cfg, sd)
    a, b, c = prompt(cfg, 80, 1, sd).tolist(), prompt(cfg, 30, 2, sd).tolist(), prompt(cfg, 5, 3, sd).tolist()
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
